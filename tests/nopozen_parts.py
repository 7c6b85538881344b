"""The Nopozen mechanisms one at a time, against the plain functions, for any kernel library: the host tests run these checks
with the tensor-code stand-in on the CPU, the GPU tests with the CUDA kernels in both precisions.

Every check builds one part of the package with weights of its own, feeds requests of unequal length through it several ways
(whole; in portions; a portion and then token by token; portions of two tokens; all requests in one batch) and compares each
with the plain function on the whole sequence."""

from __future__ import annotations

import types

import numpy as np
import torch

from paged_llm_b200.models.nopozen import _feed_forward, _mixer, _Positions
from paged_llm_b200.config.nopozen import _MIXERS, NopozenMLP
from paged_llm_b200.models.causal_lm import _resolve_positions
from paged_llm_b200.parts.base import FEED_FORWARDS, MIXERS, POSITION_ENCODINGS, STREAM_JOINS, LazyLinear, LazySum, PartSpec, make_part, materialize
from tests import plain_nopozen as plain
from tests.munazen_parts import load, rand, run_mixer, tol  # noqa: F401  (the harness is the same for every design)

WAYS = ("whole", (0.6, 0.4), (0.25, 0.05, 0.7), "decode", ("every", 2))


def _mat(rows, cols, seed):
    return rand(rows, cols, seed=seed, std=1.2 / np.sqrt(cols))


def mixer_weights(kind, W, m, seed):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)
    w = {"a.q": _mat(H * d, W, seed), "a.k": _mat(G * d, W, seed + 1), "a.v": _mat(G * dv, W, seed + 2), "a.o": _mat(W, H * dv, seed + 3),
         "a.g": _mat(H if kind == "attention" else H * dv, W, seed + 4)}
    if kind == "attention":
        w.update({"a.q.b": rand(H * d, seed=seed + 5, std=0.5), "a.k.b": rand(G * d, seed=seed + 6, std=0.5),
                  "a.v.b": rand(G * dv, seed=seed + 7, std=0.5), "a.o.b": rand(W, seed=seed + 8, std=0.5),
                  "a.q.norm": 1.0 + rand(d, seed=seed + 9, std=0.3), "a.k.norm": 1.0 + rand(d, seed=seed + 10, std=0.3)})
    elif kind == "attention_2":
        w.update({f"a.{x}.conv": rand(w["a." + x].shape[0], m["conv"], seed=seed + 11 + i, std=0.6) for i, x in enumerate("qkv")})
    else:
        w["a.norm"] = 1.0 + rand(H * dv, seed=seed + 14, std=0.2)
        w["a.q"] = w["a.k"] + 0.4 * w["a.q"]
        w["a.q"] = w["a.q"].to(torch.bfloat16).float()
    return w


def mixer_part(kind, W, m, w, eps, dtype, device, ops, length=4096):
    """The part as the model's spec names it, with its position table prepared."""
    positions = _Positions()
    spec = _mixer(W, eps, kind, _MIXERS[kind].from_dict(m, "test"), "a.", positions)
    tables = {name: make_part(POSITION_ENCODINGS, "position encoding", ps) for name, ps in positions.specs.items()}
    for t in tables.values():
        t.prepare(length, device, ops)
    spec, extra = _resolve_positions(spec, tables)
    return load(make_part(MIXERS, "mixer", spec, **extra), w, dtype, device)


def check_mixer(kind, ops, device, dtype, W, m, lens, seed=0, eps=1e-5, weights=None, hs=None, ways=WAYS, ps=8, scale_tol=3.0):
    w = weights if weights is not None else mixer_weights(kind, W, m, seed)
    hs = hs if hs is not None else [rand(n, W, seed=seed + 30 + i) for i, n in enumerate(lens)]
    part = mixer_part(kind, W, m, w, eps, dtype, device, ops)
    wd = {k: v.double() for k, v in w.items()}
    want = torch.cat([plain.MIXERS[kind](h.double(), wd, "a.", m, eps) for h in hs])
    for way, got in zip(ways, run_mixer(ops, device, part, hs, dtype, ps=ps, ways=ways)):
        err = (got.double() - want).abs().max().item()
        assert err <= tol(dtype, scale_tol) * max(1.0, want.abs().max().item()), (way, err)
    return want


def loud_key(kind, W, m, n, loud, seed=0):
    """Weights and inputs on which position `loud` holds the one key that every later query of every head answers to: hidden
    unit 0 is on at `loud` only and turns its key towards the queries, which unit 1 turns the same way everywhere; all other
    keys point elsewhere.  The key's element lies behind the rotated ones, so distance does not dim it.  The value at `loud`
    is marked through unit 0 as well."""
    w = mixer_weights(kind, W, m, seed)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    assert m["rot"]["dims"] <= d - 2
    h = rand(n, W, seed=seed + 31, std=0.05)
    h[:, 0], h[:, 1] = 0.0, 1.0
    h[loud, 0] = 6.0
    for name in ("a.q", "a.k", "a.v"):
        w[name] = w[name] * 0.05
        w[name][:, :2] = 0.0
        if name + ".b" in w:
            w[name + ".b"][:] = 0.0
        if name + ".conv" in w:
            w[name + ".conv"] = w[name + ".conv"] * 0.01
            w[name + ".conv"][:, -1] = 1.0
    for g in range(G):
        w["a.k"][g * d + d - 1, 0] = 8.0
        w["a.k"][g * d + d - 2, 1] = 4.0                    # every other key points along another element
        w["a.v"][g * dv, 0] = 4.0
    for hh in range(H):
        w["a.q"][hh * d + d - 1, 1] = 8.0
    w["a.g"][:] = w["a.g"] * 0.2
    return w, h


def far_effect(kind, W, m, w, h, at, want):
    """How much the plain output at every position changes when unit 0 is off at position `at`."""
    other = h.clone()
    other[at, 0] = 0.0
    quiet = plain.MIXERS[kind](other.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    return (want - quiet).abs().amax(1)


# ---------------------------------------------------------------- feed-forwards
def mlp_weights(W, f, seed):
    if f["kind"] == "dense":
        return {"m.up": _mat(f["ff"], W, seed), "m.down": _mat(W, f["ff"], seed + 1)}
    E, F = f["router"]["experts"], f["expert"]["ff"]
    w = {"m.router": rand(E, W, seed=seed, std=2.0 / np.sqrt(W)), "m.router.b": rand(E, seed=seed + 1, std=0.7)}
    for e in range(E):
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"] = (_mat(F, W, seed + 3 * e + 2), _mat(F, W, seed + 3 * e + 3),
                                                                 _mat(W, F, seed + 3 * e + 4))
    return w


def mlp_part(W, f, w, dtype, device):
    return load(make_part(FEED_FORWARDS, "feed-forward", _feed_forward(W, NopozenMLP.from_dict(f, "test"), "m.")), w, dtype, device)


def clear_rows(W, f, w, rows, seed, margin=0.02):
    """Inputs on which the router has no close call."""
    keep, s = [], seed
    while len(keep) < rows:
        h = rand(4 * rows, W, seed=s)
        s += 1
        if f["kind"] == "dense" or f["router"]["top"] == f["router"]["experts"]:
            return h[:rows]
        margins: list[float] = []
        plain.router(h.double(), w["m.router"].double(), w["m.router.b"].double(), f["router"]["top"], margins)
        keep += [r for r, gap in zip(h, margins) if gap >= margin][:rows - len(keep)]
    return torch.stack(keep)


def check_mlp(ops, device, dtype, W, f, rows, seed=0, scale_tol=3.0):
    """The feed-forward alone (its sum formed), some of its rows (as for the wanted logits), and beside a projection with a
    bias in front of the norm that follows."""
    w = mlp_weights(W, f, seed)
    part = mlp_part(W, f, w, dtype, device)
    h = clear_rows(W, f, w, rows, seed + 500)
    ops.set_compute_dtype(dtype)
    ctx = types.SimpleNamespace(ops=ops)
    want = plain.feed_forward(h.double(), {k: v.double() for k, v in w.items()}, "m.", f)
    hd = h.to(dtype).to(device).contiguous()
    limit = tol(dtype, scale_tol) * max(1.0, want.abs().max().item())
    out = part.forward(hd, ctx)
    assert (materialize(out, ops).float().cpu().double() - want).abs().max() <= limit
    pick = [rows - 1, 0, rows // 2]
    idx = torch.tensor(pick, dtype=torch.int32, device=device)
    some = out.rows(ops, idx) if hasattr(out, "rows") else ops.gather_rows(out, idx)
    assert (materialize(some, ops).float().cpu().double() - want[pick]).abs().max() <= limit
    # the sum of both branches of a layer, the stream and the next norm
    a, wa, ba = rand(rows, 24, seed=seed + 600), _mat(W, 24, seed + 601), rand(W, seed=seed + 602, std=0.5)
    x, nw = rand(rows, W, seed=seed + 603, std=2.0), 1.0 + rand(W, seed=seed + 604, std=0.2)
    first = LazyLinear(a.to(dtype).to(device), wa.to(dtype).to(device), ba.to(device))
    xd = x.to(device).clone()
    both = LazySum((first, part.forward(hd, ctx)))
    stream = x.double() + a.double() @ wa.double().T + ba.double() + want
    top = max(1.0, stream.abs().max().item())
    alone = materialize(both, ops).float().cpu().double()
    assert (alone - (stream - x.double())).abs().max() <= tol(dtype, scale_tol) * top
    y = ops.branches_add_rms_norm(xd, list(both.parts), nw.to(device), 1e-5)
    assert (xd.cpu().double() - stream).abs().max() <= tol(dtype, scale_tol) * top
    normed = plain.rms(stream, nw.double(), 1e-5)
    assert (ops.materialize(y).float().cpu().double() - normed).abs().max() <= tol(dtype, scale_tol) * max(1.0, normed.abs().max().item())
    xd = x.to(device).clone()
    copy = ops.add_copy(xd, both).float().cpu().double()
    assert (copy - stream).abs().max() <= tol(dtype, scale_tol) * top and (xd.cpu().double() - stream).abs().max() <= tol(dtype, scale_tol) * top
    # behind the last layer only the wanted rows are finished
    got = both.rows(ops, idx)
    xr = x[pick].to(device).clone()
    y = ops.materialize(ops.branches_add_rms_norm(xr, list(got.parts), nw.to(device), 1e-5)).float().cpu().double()
    assert (y - normed[pick]).abs().max() <= tol(dtype, scale_tol) * max(1.0, normed.abs().max().item())


def check_join(ops, device, dtype, W, rows, times=3, seed=0):
    """`times` joins in a row, with a branch pending in front of each, against W_in [x; x0]."""
    from paged_llm_b200.parts.norm import RMSNorm
    ops.set_compute_dtype(dtype)
    w = {"j": _mat(W, 2 * W, seed), "n": 1.0 + rand(W, seed=seed + 1, std=0.2)}
    join = make_part(STREAM_JOINS, "stream join", PartSpec("linear_join", dict(hidden_size=W), {"weight": "j"}))
    norm = RMSNorm({"weight": "n"}, W, 1e-5)
    load(join, {"j": w["j"]}, dtype, device)
    norm.load({"n": w["n"].to(device)})
    ctx = types.SimpleNamespace(ops=ops)
    x0 = rand(rows, W, seed=seed + 2)
    xd, pending = x0.to(device).clone(), None
    want = x0.double()
    shared = join.start(xd, times, ctx)
    for t in range(times):
        xd, pending = join.forward(xd, pending, shared, ctx)
        want = torch.cat([want, x0.double()], dim=1) @ w["j"].double().T
        y = ops.materialize(norm.add_forward(xd, pending, ctx)).float().cpu().double()
        top = max(1.0, want.abs().max().item())
        assert (xd.cpu().double() - want).abs().max() <= tol(dtype, 2.0) * top, t
        assert (y - plain.rms(want, w["n"].double(), 1e-5)).abs().max() <= tol(dtype, 4.0) * 4.0, t
        branch = rand(rows, W, seed=seed + 10 + t)
        pending = LazySum((branch.to(dtype).to(device).contiguous(),))
        want = want + branch.double()
