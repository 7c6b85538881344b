"""Small Nopozen configurations for the tests, which differ from each other in every size, constant and order of layers, and
helpers to write their folders with random weights and to ask the plain model.

The weights are drawn here so that a fault shows: biases and norm weights away from 0 and 1, router biases that change the
choice, convolution taps of weight on every lag, gates away from one half; linear attention's queries lean on its keys.
"""

from __future__ import annotations

import random

import numpy as np
import torch

from paged_llm_b200.config.registry import parse_model_config
from paged_llm_b200.models.causal_lm import build_model
from tests import plain_nopozen
from tests.rokarax_cases import make_folder as _write_folder
from tests.rokarax_cases import read_folder  # noqa: F401  (re-exported)


def rot(dims, base, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def attention(heads, kv, dim, vdim, rotation, chunk=None, scale=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": rotation, "scale": dim ** -0.5 if scale is None else scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return m


def convolved(heads, kv, dim, vdim, rotation, taps, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": rotation, "scale": dim ** -0.5 if scale is None else scale,
            "conv": taps}


def lightning(dim, vdim, *decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, loop=None, eps=1e-5):
    cfg = {"architecture": "Nopozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: begins inside the loop, which runs three times; a chunk of 11 and partial rotation whose band of frequencies is blended;
# values longer and shorter than keys; a feed-forward of every kind and a layer without one; four taps; one decay of 1 (nothing
# is forgotten) and one of 0 (nothing is kept).
CASE_A = model(131, 64, [
    layer("lightning", lightning(16, 24, 0.5, 1.0, 0.93), moe(24, 6, 2)),
    layer("attention", attention(4, 2, 16, 24, rot(12, 10000.0, (4.0, 1.0, 4.0, 40.0)), 11), dense(72)),
    layer("attention_2", convolved(2, 2, 32, 16, rot(8, 500.0), 4, scale=0.3), None),
    layer("lightning", lightning(8, 8, 0.0, 0.8), moe(16, 5, 5)),
], loop=(0, 2, 3))

# B: no loop; attention over everything (no mask) with six heads on one kv head; two taps; a linear attention whose sizes fill
# neither the lanes of a column nor a quad; one expert per token; a width that is no multiple of eight.
CASE_B = model(77, 92, [
    layer("attention_2", convolved(6, 1, 16, 16, rot(16, 30.5), 2), moe(20, 4, 1)),
    layer("lightning", lightning(20, 13, 0.9, 0.99), dense(50)),
    layer("attention", attention(3, 3, 8, 40, rot(4, 1000.0), scale=0.5), moe(56, 8, 3)),
    layer("lightning", lightning(6, 20, 0.7), None),
], eps=1e-6)

# C: heads of 64 and 128 (the tensor-core prefill kernels), chunks around a tile's size, one tap (no history), eight query
# heads on two kv heads, a single layer that loops twice in the middle, four of sixteen experts.
CASE_C = model(300, 128, [
    layer("attention", attention(8, 2, 64, 64, rot(64, 10000.0, (8.0, 1.0, 4.0, 128.0)), 65), moe(64, 16, 4)),
    layer("attention_2", convolved(4, 1, 64, 64, rot(16, 10000.0), 1), dense(96)),
    layer("lightning", lightning(64, 64, 0.97, 0.995), moe(32, 8, 2)),
    layer("attention", attention(2, 1, 128, 128, rot(32, 100.0), 100), moe(64, 4, 2)),
], loop=(1, 2, 2))

# D: every layer in one pass of the loop (times 1): the join runs all the same.
CASE_D = model(90, 48, [
    layer("attention", attention(2, 1, 16, 16, rot(16, 10000.0, (2.0, 1.0, 2.0, 16.0)), 1), dense(40)),
    layer("attention_2", convolved(4, 2, 24, 8, rot(24, 77.0), 7), moe(8, 3, 2)),
    layer("lightning", lightning(12, 36, 0.6, 0.99, 0.999), dense(24)),
], loop=(0, 3, 1))

CASES = {"A": (CASE_A, 61), "B": (CASE_B, 62), "C": (CASE_C, 63), "D": (CASE_D, 64)}


def _drawn_mlp(rng, ffs):
    if rng.random() < 0.15:
        return None
    if rng.random() < 0.3:
        return dense(rng.choice(ffs))
    experts = rng.choice([1, 3, 4, 8, 12])
    return moe(rng.choice(ffs), experts, rng.randint(1, min(experts, 4)))


def _drawn_rot(rng, dim):
    scaling = rng.choice([None, (rng.choice([2.0, 8.0]), 1.0, rng.choice([2.0, 4.0]), rng.choice([16.0, 60.0, 300.0]))])
    return rot(rng.choice([dim, 2 * max(1, dim // 4), 2]), rng.choice([50.0, 10000.0, 500000.0]), scaling)


def _drawn_loop(rng, n):
    if rng.random() < 0.2:
        return None
    start = rng.randrange(n)
    return start, rng.randint(start + 1, n), rng.choice([1, 2, 2, 3])


def _drawn_layers(rng, count, kv_choices, dims, vdims, light_dims, ffs, chunks):
    layers = []
    for _ in range(count):
        kind = rng.choice(["attention", "attention_2", "lightning"])
        if kind == "lightning":
            decay = [rng.choice([0.3, 0.8, 0.95, 0.99, 0.999]) for _ in range(rng.choice([1, 2, 3, 5]))]
            m = lightning(rng.choice(light_dims), rng.choice(light_dims), *decay)
        else:
            kv, dim = rng.choice(kv_choices), rng.choice(dims)
            heads, vdim, scale = kv * rng.choice([1, 2, 4]), rng.choice([dim] + vdims), rng.choice([0.7, 1.0, 1.4]) * dim ** -0.5
            if kind == "attention":
                m = attention(heads, kv, dim, vdim, _drawn_rot(rng, dim), rng.choice(chunks), scale)
            else:
                m = convolved(heads, kv, dim, vdim, _drawn_rot(rng, dim), rng.choice([1, 2, 3, 5]), scale)
        layers.append(layer(kind, m, _drawn_mlp(rng, ffs)))
    return layers


def generated_case(seed: int) -> dict:
    """A configuration drawn from a seed: widths, head counts and sizes, chunks, rotations, decays, taps, the experts, the loop
    and the order of layers all vary, within what the design allows."""
    rng = random.Random(seed)
    layers = _drawn_layers(rng, rng.randint(2, 4), [1, 2, 3], [8, 16, 24, 64], [8, 40], [4, 8, 20, 36, 64], [8, 24, 64], [None, 1, 5, 16, 31, 64])
    return model(rng.choice([50, 131, 300, 777]), rng.choice([48, 64, 90, 160]), layers, _drawn_loop(rng, len(layers)),
                 eps=rng.choice([1e-6, 1e-5]))


def wide_case(seed: int) -> dict:
    """A drawn configuration at widths of 256 to 512 with heads of 32 to 128: the sizes at which the tensor-core kernels,
    four-element accesses and the larger builds of the attention kernels run."""
    rng = random.Random(seed)
    layers = _drawn_layers(rng, rng.randint(3, 5), [1, 2, 4], [32, 64, 128], [48, 96], [32, 64, 128], [32, 64, 128], [None, 20, 64, 90])
    return model(rng.choice([320, 1000]), rng.choice([256, 384, 512]), layers, _drawn_loop(rng, len(layers)), eps=rng.choice([1e-6, 1e-5]))


def draw_weights(hf_cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Every tensor the model expects, in float32 with values that bfloat16 holds exactly."""
    arch, cfg = parse_model_config(hf_cfg)
    specs = build_model(arch.build_spec(cfg)).tensor_specs()
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name in sorted(specs):
        shape = specs[name].shape
        r = torch.randn(shape, generator=g)
        if name.endswith(".router.b"):
            t = 0.7 * r                                            # of the size of the logits' spread: changes choices
        elif name.endswith(".b"):
            t = 0.5 * r
        elif name.endswith(".conv"):
            t = 0.6 * r
        elif "norm" in name:
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = r
        elif name.endswith(".router"):
            t = r * (2.0 / np.sqrt(shape[-1]))
        elif name.endswith(".mix.q") and not name + ".b" in specs and not name + ".conv" in specs:
            # linear attention's queries lean towards its keys: the norm behind a nearly empty state keeps only the sign of
            # q . k of the first tokens, which stays away from zero this way also in bfloat16
            t = out[name[:-1] + "k"] + 0.4 * r * (1.2 / np.sqrt(shape[-1]))
        else:
            t = r * (1.2 / np.sqrt(shape[-1]))                     # matrices: outputs of the order of their inputs
        out[name] = t.to(torch.bfloat16).float().contiguous()
    return out


def make_folder(path, hf_cfg: dict, seed: int, dtype: str = "bfloat16", weights=None) -> str:
    return _write_folder(path, hf_cfg, seed, dtype, weights if weights is not None else draw_weights(hf_cfg, seed))


def case_folder(tmp_path_factory, name: str) -> str:
    hf, seed = CASES[name]
    return make_folder(tmp_path_factory.mktemp(f"nopozen{name}"), hf, seed)


def plain_logits(folder: str, tokens) -> np.ndarray:
    cfg, w = read_folder(folder)
    with torch.no_grad():
        return plain_nopozen.forward(cfg, w, tokens)[0].to(torch.float32).numpy()


def rounding_error(folder: str, tokens, dtype=torch.float32) -> np.ndarray:
    """Per position, the root mean square over the vocabulary of the difference between the plain model run in `dtype`
    and in float64: what rounding alone does to these weights."""
    cfg, w = read_folder(folder)
    with torch.no_grad():
        exact = plain_nopozen.forward(cfg, w, tokens)[0]
        with plain_nopozen.precision(dtype):
            rounded = plain_nopozen.forward(cfg, w, tokens)[0]
    return (rounded.double() - exact).pow(2).mean(dim=1).sqrt().numpy()


def clear_requests(folder: str, vocab: int, lengths, seed: int = 0, margin: float = 0.1) -> dict[str, list[int]]:
    """Random requests on which no router of the model comes close to a tie (the last chosen expert's logit leads the next by
    `margin` at every token): a bfloat16 engine then chooses the experts the plain model chooses, and the two differ by
    rounding only.  From its first close call on a request is drawn again, until there is none; one that does not get there is
    cut in front of it."""
    cfg, w = read_folder(folder)
    out = {}
    for i, n in enumerate(lengths):
        g = torch.Generator().manual_seed(seed * 100003 + i * 401)
        toks = torch.randint(0, vocab, (n,), generator=g).tolist()
        for attempt in range(60):
            margins: list[float] = []
            with torch.no_grad():
                plain_nopozen.forward(cfg, w, toks, margins)
            close = (np.array(margins).reshape(-1, n).min(axis=0) < margin) if margins else np.zeros(n, bool)
            if not close.any():
                break
            first = int(np.argmax(close))
            toks[first:] = torch.randint(0, vocab, (n - first,), generator=g).tolist()
        else:
            toks = toks[:first]
        if not toks:
            raise AssertionError("no request without a close call, however short")
        out[f"r{i}"] = toks
    return out


def plain_greedy(folder: str, prompt, n: int) -> list[int]:
    cfg, w = read_folder(folder)
    with torch.no_grad():
        return plain_nopozen.greedy_generate(cfg, w, prompt, n)
