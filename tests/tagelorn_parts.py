"""The Tagelorn mechanisms one at a time, against the plain functions, for any kernel library: the host tests run these
checks with the tensor-code stand-in on the CPU, the GPU tests with the CUDA kernels in both precisions.

Every check builds one part of the package with weights of its own, feeds requests of unequal length through it several
ways (whole; in portions; a portion and then token by token; portions of two tokens; all requests in one batch) and
compares each with the plain function on the whole sequence."""

from __future__ import annotations

import types

import numpy as np
import torch

from paged_llm_b200.parts.base import FEED_FORWARDS, MIXERS, PartSpec, make_part, materialize
from tests import plain_tagelorn as plain
from tests.munazen_parts import load, rand, run_mixer, tol  # noqa: F401  (the harness is the same for every design)

F64 = torch.float64
WAYS = ("whole", (0.6, 0.4), (0.25, 0.05, 0.7), "decode", ("every", 2))


def _mat(rows, cols, seed):
    return rand(rows, cols, seed=seed, std=1.2 / np.sqrt(cols))


def _compare(ops, device, part, hs, dtype, want, ways, ps, scale_tol):
    for way, got in zip(ways, run_mixer(ops, device, part, hs, dtype, ps=ps, ways=ways)):
        err = (got.double() - want).abs().max().item()
        assert err <= tol(dtype, scale_tol) * max(1.0, want.abs().max().item()), (way, err)
    return want


# ---------------------------------------------------------------- attention
def attention_weights(W, m, seed, rows=8):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"a.q": _mat(H * d, W, seed), "a.k": _mat(G * d, W, seed + 1), "a.v": _mat(G * dv, W, seed + 2), "a.o": _mat(W, H * dv, seed + 3),
            "a.q.b": rand(H * d, seed=seed + 4, std=0.5), "a.k.b": rand(G * d, seed=seed + 5, std=0.5),
            "a.v.b": rand(G * dv, seed=seed + 6, std=0.5), "a.rel": rand(rows, H, seed=seed + 7, std=1.5),
            "a.sink": 1.0 + rand(H, seed=seed + 8)}


def attention_part(W, m, w, eps, dtype, device):
    names = {x + "_proj": "a." + x for x in "qkvo"}
    names.update({x + "_proj_bias": f"a.{x}.b" for x in "qkv"}, rel="a.rel", sink="a.sink")
    mask = m.get("mask") or {}
    part = MIXERS["gated_attention"](
        weights=names, hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"],
        scale=m["scale"], eps=eps, window=mask.get("size"), keep_first=mask.get("keep_first", 0), distance_bias=True,
        bias_far=m["bias_max"], gate=False, sink=True, head_norm=True, bias=True)
    return load(part, w, dtype, device)


def check_attention(ops, device, dtype, W, m, lens, seed=0, eps=1e-5, weights=None, hs=None, ways=WAYS, ps=8, scale_tol=3.0, rows=8):
    w = weights if weights is not None else attention_weights(W, m, seed, rows)
    hs = hs if hs is not None else [rand(n, W, seed=seed + 20 + i) for i, n in enumerate(lens)]
    part = attention_part(W, m, w, eps, dtype, device)
    wd = {k: v.double() for k, v in w.items()}
    want = torch.cat([plain.attention(h.double(), wd, "a.", m, eps) for h in hs])
    return _compare(ops, device, part, hs, dtype, want, ways, ps, scale_tol)


def loud_key(W, m, n, loud, seed=0, rows=8):
    """Weights and inputs on which position `loud` holds the one key that every later query of every head answers to:
    hidden unit 0 is on at `loud` only and turns its key towards the queries, which unit 1 turns the same way everywhere; all
    other keys point elsewhere.  The value at `loud` is marked through unit 0 as well."""
    w = attention_weights(W, m, seed, rows)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = rand(n, W, seed=seed + 31, std=0.05)
    h[:, 0], h[:, 1] = 0.0, 1.0
    h[loud, 0] = 6.0
    for name in ("a.q", "a.k", "a.v"):
        w[name] = w[name] * 0.05
        w[name][:, :2] = 0.0
        w[name + ".b"][:] = 0.0
    for g in range(G):
        w["a.k"][g * d, 0] = 8.0
        w["a.k"][g * d + 1, 1] = 4.0                        # every other key points along its second element
        w["a.v"][g * dv, 0] = 4.0
    for hh in range(H):
        w["a.q"][hh * d, 1] = 8.0
    w["a.rel"][:] = w["a.rel"] * 0.2
    w["a.sink"][:] = 0.0
    return w, h


# ---------------------------------------------------------------- the generalized delta rule
def delta_weights(W, m, seed, rank=5, w0=None):
    C = m["heads"] * m["dim"]
    k = _mat(C, W, seed + 1)
    return {"d.r": k + 0.4 * _mat(C, W, seed), "d.k": k, "d.v": _mat(C, W, seed + 2), "d.g": _mat(C, W, seed + 3), "d.a": _mat(C, W, seed + 4),
            "d.a.b": rand(C, seed=seed + 5, std=0.5), "d.w1": _mat(rank, W, seed + 6), "d.w2": _mat(C, rank, seed + 7),
            "d.w0": -1.5 + rand(C, seed=seed + 8, std=1.5) if w0 is None else torch.full((C,), float(w0)),
            "d.norm": 1.0 + rand(C, seed=seed + 9, std=0.2), "d.o": _mat(W, C, seed + 10)}


DELTA_NAMES = {"r_proj": "d.r", "k_proj": "d.k", "v_proj": "d.v", "g_proj": "d.g", "removal_proj": "d.a", "removal_bias": "d.a.b",
               "decay_down": "d.w1", "decay_up": "d.w2", "decay_bias": "d.w0", "norm": "d.norm", "o_proj": "d.o"}


def delta_part(W, m, w, eps, dtype, device):
    part = MIXERS["general_delta"](weights=DELTA_NAMES, hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], eps=eps)
    return load(part, w, dtype, device)


def check_delta(ops, device, dtype, W, m, lens, seed=0, eps=1e-5, weights=None, hs=None, ways=WAYS, scale_tol=3.0, rank=5):
    w = weights if weights is not None else delta_weights(W, m, seed, rank)
    hs = hs if hs is not None else [rand(n, W, seed=seed + 20 + i) for i, n in enumerate(lens)]
    part = delta_part(W, m, w, eps, dtype, device)
    wd = {k: v.double() for k, v in w.items()}
    want = torch.cat([plain.general_delta(h.double(), wd, "d.", m, eps) for h in hs])
    return _compare(ops, device, part, hs, dtype, want, ways, 8, scale_tol)


# ---------------------------------------------------------------- the convolution in front of a mixer
def check_input_convolution(ops, device, dtype, W, taps, inner, m, lens, seed=0, eps=1e-5, ways=WAYS, scale_tol=3.0):
    """In front of either mixer: the request keeps the convolution's inputs beside what the mixer keeps."""
    conv = rand(W, taps, seed=seed + 90, std=0.5)
    if inner == "general_delta":
        w = delta_weights(W, m, seed)
        spec = PartSpec("general_delta", dict(hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], eps=eps), DELTA_NAMES)
        mixer = lambda h, wd: plain.general_delta(h, wd, "d.", m, eps)      # noqa: E731
    else:
        w = attention_weights(W, m, seed)
        mask = m.get("mask") or {}
        spec = PartSpec("gated_attention", dict(
            hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"],
            eps=eps, window=mask.get("size"), keep_first=mask.get("keep_first", 0), distance_bias=True, bias_far=m["bias_max"],
            gate=False, sink=True, head_norm=True, bias=True),
            {**{x + "_proj": "a." + x for x in "qkvo"}, **{x + "_proj_bias": f"a.{x}.b" for x in "qkv"}, "rel": "a.rel", "sink": "a.sink"})
        mixer = lambda h, wd: plain.attention(h, wd, "a.", m, eps)          # noqa: E731
    part = make_part(MIXERS, "mixer", PartSpec("input_convolution", dict(hidden_size=W, taps=taps, mixer=spec), {"conv": "c"}))
    load(part, {**w, "c": conv}, dtype, device)
    hs = [rand(n, W, seed=seed + 20 + i) for i, n in enumerate(lens)]
    wd = {k: v.double() for k, v in w.items()}
    want = torch.cat([mixer(plain.input_convolution(h.double(), conv.double()), wd) for h in hs])
    return _compare(ops, device, part, hs, dtype, want, ways, 8, scale_tol)


# ---------------------------------------------------------------- routed experts
def experts_weights(W, mlp, seed):
    E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
    w = {"m.router": rand(E, W, seed=seed, std=2.0 / np.sqrt(W)), "m.correction": rand(E, seed=seed + 1, std=0.15)}
    for e in range(E):
        w[f"m.e{e}.up"], w[f"m.e{e}.down"] = _mat(F, W, seed + 2 * e + 2), _mat(W, F, seed + 2 * e + 3)
    if mlp.get("shared"):
        s = mlp["shared"]["ff"]
        w["m.shared.up"], w["m.shared.down"] = _mat(s, W, seed + 300), _mat(W, s, seed + 301)
    return w


def experts_part(W, mlp, w, dtype, device):
    E, r, g = mlp["router"]["experts"], mlp["router"], mlp["router"].get("groups")
    shared = mlp.get("shared")
    names = {"router": "m.router", "correction": "m.correction"}
    for prefix in [f"e{e}" for e in range(E)] + (["shared"] if shared else []):
        for x in ("up", "down"):
            names[f"{prefix}.{x}"] = f"m.{prefix}.{x}"
    part = FEED_FORWARDS["routed_mlp"](
        weights=names, hidden_size=W, expert_size=mlp["expert"]["ff"], num_experts=E, top_k=r["top"], activation="relu2", gated=False,
        shared_size=shared["ff"] if shared else None, shared_gate=False, scoring="softmax", correction=True,
        groups=(g["count"], g["keep"]) if g else None, group_score_top=1, renorm=True, weight_scale=r["scale"])
    return load(part, w, dtype, device)


def clear_rows(W, mlp, w, rows, seed, margin=0.01):
    """Inputs on which the router has no close call (the plain router's smallest gap is at least `margin`)."""
    keep = []
    s = seed
    while len(keep) < rows:
        h = rand(4 * rows, W, seed=s)
        s += 1
        for i in range(h.shape[0]):
            margins: list[float] = []
            plain.router(h[i:i + 1].double(), w["m.router"].double(), w["m.correction"].double(), mlp["router"], margins)
            if min(margins, default=1.0) >= margin and len(keep) < rows:
                keep.append(h[i])
    return torch.stack(keep)


def check_experts(ops, device, dtype, W, mlp, rows, seed=0, scale_tol=3.0):
    w = experts_weights(W, mlp, seed)
    part = experts_part(W, mlp, w, dtype, device)
    h = clear_rows(W, mlp, w, rows, seed + 500)
    ops.set_compute_dtype(dtype)
    got = part.forward(h.to(dtype).to(device).contiguous(), types.SimpleNamespace(ops=ops)).float().cpu()
    want = plain.routed_experts(h.double(), {k: v.double() for k, v in w.items()}, "m.", mlp)
    err = (got.double() - want).abs().max().item()
    assert err <= tol(dtype, scale_tol) * max(1.0, want.abs().max().item()), err


# ---------------------------------------------------------------- token input, sinusoids, cap
class _Branch:
    """A mixer that hands on a fixed branch (and a block around it without a feed-forward)."""

    accepts_lazy_input, capturable = True, True

    def __init__(self, branch):
        self.branch = branch

    def tensor_specs(self):
        return {}

    def load(self, tensors):
        pass

    def forward(self, h, ctx, cache):
        return self.branch


def check_token_side(ops, device, dtype, W, dim, layers, which, rows, vocab=37, seed=0, eps=1e-5):
    """One layer's token input behind a branch, then the norm of the next layer: stream and norm against the equations."""
    from paged_llm_b200.parts.block import TokenSideBlock
    from paged_llm_b200.parts.norm import RMSNorm
    ops.set_compute_dtype(dtype)
    w = {"t": rand(vocab, layers * dim, seed=seed), "s.gate": _mat(dim, W, seed + 1), "s.proj": _mat(W, dim, seed + 2),
         "s.norm": 1.0 + rand(W, seed=seed + 3, std=0.2), "n1": 1.0 + rand(W, seed=seed + 4, std=0.2), "n2": 1.0 + rand(W, seed=seed + 5, std=0.2)}
    x, branch = rand(rows, W, seed=seed + 6, std=2.0), rand(rows, W, seed=seed + 7)
    ids = torch.randint(0, vocab, (rows,), generator=torch.Generator().manual_seed(seed))
    blk = TokenSideBlock(_Branch(branch.to(dtype).to(device).contiguous()), None, {"input": RMSNorm({"weight": "n1"}, W, eps)},
                         {"table": "t", "gate": "s.gate", "proj": "s.proj", "norm": "s.norm"}, W, vocab, dim, which * dim, layers * dim, eps)
    nxt = RMSNorm({"weight": "n2"}, W, eps)
    tensors = {k: v.to(dtype if v.dim() == 2 else torch.float32).to(device) for k, v in w.items()}
    blk.load(tensors)
    nxt.load(tensors)
    ctx = types.SimpleNamespace(ops=ops, input_ids=ids.to(torch.int32).to(device))
    xd = x.to(device).clone()
    _, pending = blk.forward(xd, None, ctx, None)
    alone = materialize(pending, ops).float().cpu()
    y = ops.materialize(nxt.add_forward(xd, pending, ctx)).float().cpu()
    wd = {k: v.double() for k, v in w.items()}
    mid = x.double() + branch.double()
    add = plain.token_side(mid, wd["t"][ids][:, which * dim:(which + 1) * dim], wd, "s.", eps)
    assert (alone.double() - add).abs().max() < tol(dtype, 3.0) * max(1.0, add.abs().max().item())
    assert (xd.cpu().double() - mid - add).abs().max() < tol(dtype, 3.0) * max(1.0, (mid + add).abs().max().item())
    want = plain.rms(mid + add, wd["n2"], eps)
    assert (y.double() - want).abs().max() < tol(dtype, 4.0) * max(1.0, want.abs().max().item())


def check_sinusoids(ops, device, dtype, W, scale, positions, vocab=19, seed=0):
    """The scaled embedding plus the position's vector, also far out (the phase keeps its precision)."""
    from paged_llm_b200.parts.embedding import SinusoidalEncoding
    enc = SinusoidalEncoding({}, W)
    enc.prepare(0, torch.device(device), ops)
    table = rand(vocab, W, seed=seed)
    ids = torch.randint(0, vocab, (len(positions),), generator=torch.Generator().manual_seed(seed))
    got = ops.embedding_sinusoid(table.to(dtype).to(device), ids.to(torch.int32).to(device), scale, enc.turns,
                                 torch.tensor(positions, dtype=torch.int32, device=device)).cpu().double()
    for row, p in enumerate(positions):
        for e in {0, 1, 2, 3, W // 2, W - 2, W - 1}:
            ang = p * 10000.0 ** (-(e - e % 2) / W)
            want = table[ids[row], e].item() * scale + (np.sin(ang) if e % 2 == 0 else np.cos(ang))
            assert abs(got[row, e].item() - want) < 2e-6 * max(1.0, abs(want)), (p, e)
