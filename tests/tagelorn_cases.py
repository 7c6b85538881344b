"""Small Tagelorn configurations for the tests, which differ from each other in every size, constant and order of
layers, and helpers to write their folders with random weights and to ask the plain model.

The weights are drawn here so that a fault shows: bias tables of a few units, sinks of the size of the scores, biases and
norm weights away from 0 and 1, convolution taps of weight, decays between about 0.55 and 0.99 per token, corrections that
change the routers' choices; the delta rule's r leans on its k (see `draw_weights`).
"""

from __future__ import annotations

import random

import numpy as np
import torch

from paged_llm_b200.config.registry import parse_model_config
from paged_llm_b200.models.causal_lm import build_model
from tests import plain_tagelorn
from tests.rokarax_cases import make_folder as _write_folder
from tests.rokarax_cases import read_folder  # noqa: F401  (re-exported)


def attention(heads, kv, dim, vdim, bias_max, mask=None, scale=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
         "bias_max": bias_max}
    if mask is not None:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return m


def delta(heads, dim):
    return {"heads": heads, "dim": dim}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale=1.0, groups=None, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, taps, side, layers, eps=1e-5, scale=1.0, cap=10.0):
    return {"architecture": "Tagelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "canon": {"taps": taps}, "token_side": {"dim": side}, "logit_softcap": cap, "layers": layers}


# A: starts with the delta rule; a window of 9 beside three kept tokens and, in the same model, one of 24 beside none;
# values longer and shorter than keys; a feed-forward of every kind and a layer without one; four taps.
CASE_A = model(131, 64, 4, 12, [
    layer("general_delta", delta(3, 16), moe(24, 6, 2, 1.5, (3, 2), shared=40)),
    layer("attention", attention(4, 2, 16, 24, 40, (9, 3)), dense(72)),
    layer("attention", attention(2, 2, 32, 16, 64, (24, 0), scale=0.3), None),
    layer("general_delta", delta(2, 8), moe(16, 5, 3, 0.7, shared=8)),
], scale=3.0)

# B: starts with attention over everything, six query heads on one kv head; two taps; a delta rule whose key size fills
# neither the lanes of a column nor the columns of a block; one expert per token out of one group, no shared expert; a side
# vector and a width that are no multiples of eight; kept tokens that straddle pages (21 beside a window of 5).
CASE_B = model(77, 92, 2, 5, [
    layer("attention", attention(6, 1, 16, 16, 30.5), moe(20, 4, 1, 2.5, (1, 1))),
    layer("general_delta", delta(2, 20), dense(50)),
    layer("attention", attention(3, 3, 8, 40, 100, (5, 21), scale=0.5), moe(56, 8, 3, 1.0, (4, 2), shared=24)),
], eps=1e-6, scale=0.5, cap=30.0)

# C: heads of 64 and 128 (the tensor-core prefill kernels) with windows around a tile's size; one tap (no history); eight
# query heads on two kv heads; four of sixteen experts out of two of four groups.
CASE_C = model(300, 128, 1, 16, [
    layer("attention", attention(8, 2, 64, 64, 128, (65, 6)), moe(64, 16, 4, 1.8, (4, 2), shared=32)),
    layer("general_delta", delta(2, 64), dense(96)),
    layer("attention", attention(2, 1, 128, 128, 50, (100, 70)), moe(32, 8, 2, 1.0, (2, 1), shared=64)),
], scale=8.0, cap=20.0)

CASES = {"A": (CASE_A, 51), "B": (CASE_B, 52), "C": (CASE_C, 53)}


def _drawn_mlp(rng, ffs):
    if rng.random() < 0.15:
        return None
    if rng.random() < 0.25:
        return dense(rng.choice(ffs))
    count, per = rng.choice([1, 2, 3, 4]), rng.choice([1, 2, 3])
    keep = rng.randint(1, count)
    groups = rng.choice([None, (count, keep), (count, keep)])
    allowed = count * per if groups is None else keep * per
    return moe(rng.choice(ffs), count * per, rng.randint(1, min(allowed, 4)), rng.choice([1.0, 2.0, 0.4]), groups,
               shared=rng.choice([None] + list(ffs)))


def generated_case(seed: int) -> dict:
    """A configuration drawn from a seed: widths, head counts and sizes, windows and kept tokens, tables' ranges, taps, the
    experts, their groups and the order of layers all vary, within what the design allows."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(2, 4)):
        if rng.random() < 0.55:
            kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 16, 24, 64])
            m = attention(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([dim, 8, 40]), rng.choice([17, 33.5, 64, 200]),
                          rng.choice([None, (rng.choice([1, 2, 7, 16, 31]), rng.choice([0, 1, 4, 19]))]),
                          scale=rng.choice([0.7, 1.0, 1.4]) * dim ** -0.5)
            layers.append(layer("attention", m, _drawn_mlp(rng, [8, 24, 64])))
        else:
            layers.append(layer("general_delta", delta(rng.choice([1, 2, 5]), rng.choice([4, 8, 20, 36, 64])), _drawn_mlp(rng, [8, 24, 64])))
    return model(rng.choice([50, 131, 300, 777]), rng.choice([48, 64, 90, 160]), rng.choice([1, 2, 3, 5]), rng.choice([3, 8, 20]), layers,
                 eps=rng.choice([1e-6, 1e-5]), scale=rng.choice([0.5, 1.0, 6.0]), cap=rng.choice([5.0, 15.0, 50.0]))


def wide_case(seed: int) -> dict:
    """A drawn configuration at widths of 256 to 512 with heads of 32 to 128, three to five layers: the sizes at which the
    tensor-core kernels, four-element accesses and the larger builds of the attention kernels run."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(3, 5)):
        if rng.random() < 0.55:
            kv, dim = rng.choice([1, 2, 4]), rng.choice([32, 64, 128])
            m = attention(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([dim, dim, 48, 96]), rng.choice([64, 128, 300]),
                          rng.choice([None, (rng.choice([20, 64, 90]), rng.choice([0, 4, 17, 66]))]),
                          scale=rng.choice([0.8, 1.0]) * dim ** -0.5)
            layers.append(layer("attention", m, _drawn_mlp(rng, [32, 64, 128])))
        else:
            layers.append(layer("general_delta", delta(rng.choice([2, 4]), rng.choice([32, 64, 128])), _drawn_mlp(rng, [32, 64, 128])))
    return model(rng.choice([320, 1000]), rng.choice([256, 384, 512]), rng.choice([2, 3, 4]), rng.choice([16, 24, 40]), layers,
                 eps=rng.choice([1e-6, 1e-5]), scale=rng.choice([1.0, 10.0]), cap=rng.choice([15.0, 30.0]))


def draw_weights(hf_cfg: dict, seed: int, rel_rows: int = 16) -> dict[str, torch.Tensor]:
    """Every tensor the model expects, in float32 with values that bfloat16 holds exactly."""
    arch, cfg = parse_model_config(hf_cfg)
    specs = build_model(arch.build_spec(cfg)).tensor_specs()
    g = torch.Generator().manual_seed(seed)
    rng = random.Random(seed)
    out = {}
    for name in sorted(specs):
        if specs[name].optional:
            continue                                               # the head is the embedding
        shape = list(specs[name].draw_shape or specs[name].shape)
        if name.endswith(".rel"):
            shape[0] = rng.choice([4, 8, rel_rows])                # the table's rows are the checkpoint's
        if name.endswith(".mix.w1"):
            rank = rng.choice([3, 8, 20])                          # and so is the decay's rank
            shape[0] = rank
        if name.endswith(".mix.w2"):
            shape[1] = rank
        r = torch.randn(shape, generator=g)
        if name.endswith(".sink"):
            t = 1.0 + r                                            # of the size of the scores: leaving it out shows
        elif name.endswith(".rel"):
            t = 1.5 * r
        elif name.endswith(".w0"):
            t = -2.0 + 1.5 * r                                     # most decays close to one, some far from it
        elif name.endswith((".q.b", ".k.b", ".v.b", ".a.b")):
            t = 0.5 * r
        elif name.endswith(".correction"):
            t = 0.15 * r
        elif name.endswith(".canon1"):
            t = 0.4 * r
        elif "norm" in name:
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = 0.5 * r
        elif name.endswith(".router"):
            t = r * (2.0 / np.sqrt(shape[-1]))                     # scores spread over (0, 1)
        elif name.endswith(".mix.r"):
            # the delta rule's r leans towards its own k: the norm behind a nearly empty state keeps only the sign of r . k
            # of the first tokens, which stays away from zero this way also in bfloat16
            t = out[name[:-1] + "k"] + 0.4 * r * (1.2 / np.sqrt(shape[-1]))
        else:
            t = r * (1.2 / np.sqrt(shape[-1]))                     # matrices: outputs of the order of their inputs
        out[name] = t.to(torch.bfloat16).float().contiguous()
    return out


def make_folder(path, hf_cfg: dict, seed: int, dtype: str = "bfloat16", weights=None) -> str:
    return _write_folder(path, hf_cfg, seed, dtype, weights if weights is not None else draw_weights(hf_cfg, seed))


def case_folder(tmp_path_factory, name: str) -> str:
    hf, seed = CASES[name]
    return make_folder(tmp_path_factory.mktemp(f"tagelorn{name}"), hf, seed)


def plain_logits(folder: str, tokens) -> np.ndarray:
    cfg, w = read_folder(folder)
    with torch.no_grad():
        return plain_tagelorn.forward(cfg, w, tokens)[0].to(torch.float32).numpy()


def rounding_error(folder: str, tokens, dtype=torch.float32) -> np.ndarray:
    """Per position, the root mean square over the vocabulary of the difference between the plain model run in `dtype`
    and in float64: what rounding alone does to these weights."""
    cfg, w = read_folder(folder)
    with torch.no_grad():
        exact = plain_tagelorn.forward(cfg, w, tokens)[0]
        with plain_tagelorn.precision(dtype):
            rounded = plain_tagelorn.forward(cfg, w, tokens)[0]
    return (rounded.double() - exact).pow(2).mean(dim=1).sqrt().numpy()


def clear_requests(folder: str, vocab: int, lengths, seed: int = 0, margin: float = 0.01) -> dict[str, list[int]]:
    """Random requests on which no router of the model comes close to a tie (the last kept group and the last chosen
    expert lead the next by `margin` at every token): a bfloat16 engine then chooses the experts the plain model
    chooses, and the two differ by rounding only.  A length for which 40 draws find no such request is shortened."""
    cfg, w = read_folder(folder)
    out = {}
    for i, n in enumerate(lengths):
        while f"r{i}" not in out:
            for attempt in range(40):
                g = torch.Generator().manual_seed(seed * 100003 + i * 401 + attempt)
                toks = torch.randint(0, vocab, (n,), generator=g).tolist()
                margins: list[float] = []
                with torch.no_grad():
                    plain_tagelorn.forward(cfg, w, toks, margins)
                if min(margins, default=1.0) >= margin:
                    out[f"r{i}"] = toks
                    break
            else:
                if n <= 2:
                    raise AssertionError("no request without a close call, however short")
                n = max(2, n * 2 // 3)
    return out


def plain_greedy(folder: str, prompt, n: int) -> list[int]:
    cfg, w = read_folder(folder)
    with torch.no_grad():
        return plain_tagelorn.greedy_generate(cfg, w, prompt, n)
