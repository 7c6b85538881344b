"""The Nopozen decoder on the GPU: each new kernel and each mixer alone against the plain functions, then the engine under
every schedule in both precisions against the plain model."""

from __future__ import annotations

import copy
import json
import os
import subprocess
import sys
import types

import numpy as np
import pytest
import torch

from tests import nopozen_parts as parts
from tests import plain_nopozen as plain
from tests import schedules
from tests.helpers import requests_for
from tests.nopozen_cases import (CASE_A, CASE_B, CASE_C, CASES, attention, case_folder, clear_requests, convolved, dense, generated_case, lightning,
                                 make_folder, moe, plain_greedy, plain_logits, rot, rounding_error, wide_case)

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
F32_TOL, BF16_TOL = 2e-5, 4e-2


@pytest.fixture(scope="module")
def ops():
    from paged_llm_b200.kernels.ops import CudaOps
    return CudaOps("cuda")


def close(got, want, dtype, what, rounding=None):
    """float32: the largest difference within F32_TOL of the largest logit, or the position's root mean square error
    within 10 times what float32 alone does to the plain model there.  bfloat16: within BF16_TOL of the largest logit, or
    (`rounding` then measured in bfloat16) a root mean square error within 3 times what bfloat16 alone does there, or
    within what it does at the request's worst position (one run in bfloat16 is one draw of a position's error)."""
    assert got.shape == want.shape, what
    assert np.isfinite(got).all(), what
    err = np.abs(got - want)
    top = max(1.0, float(np.abs(want).max()))
    if dtype == "bfloat16":
        bad = err.max(axis=1) > BF16_TOL * top
        if rounding is not None:
            rms = np.sqrt((err.astype(np.float64) ** 2).mean(axis=1))
            bad &= (rms > 3.0 * rounding) & (rms > rounding.max())
    else:
        bad = err.max(axis=1) > F32_TOL * top
        if rounding is not None:
            bad &= np.sqrt((err.astype(np.float64) ** 2).mean(axis=1)) > 10.0 * rounding
    assert not bad.any(), f"{what}: max |diff| {err.max():.3e}, first bad row {int(np.argmax(bad))} ({err[int(np.argmax(bad))].max():.3e})"


# ---------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("f,W,rows", [(dense(24), 32, 9), (dense(96), 128, 2100), (dense(20), 37, 5), (moe(16, 6, 2), 32, 40), (moe(24, 4, 1), 32, 9),
                                      (moe(8, 5, 5), 40, 33), (moe(8, 1, 1), 36, 16), (moe(64, 8, 4), 64, 300), (moe(40, 64, 6), 64, 50),
                                      (moe(64, 12, 2), 128, 2100), (moe(12, 6, 2), 36, 21)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_alone(ops, dtype, f, W, rows):
    """In every form of the products (few tokens, tiles of 16 and 64 pairs, the grouped tcgen05 form, FFMA chains), its sum formed
    beside the other branch of a layer and the next norm."""
    parts.check_mlp(ops, "cuda", dtype, W, f, rows, seed=13, scale_tol=4.0)


@pytest.mark.parametrize("rows", [1, 9, 16, 17, 300])
@pytest.mark.parametrize("W", [32, 20, 96, 1024])
@pytest.mark.parametrize("dtype", DTYPES)
def test_join_alone(ops, dtype, W, rows):
    parts.check_join(ops, "cuda", dtype, W, rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [8, 30, 1023, 2048, 5000, 9000])
def test_norm_over_a_row_with_a_gate(ops, dtype, W):
    o, proj, w = parts.rand(7, W, seed=1), parts.rand(7, W + 24, seed=2), 1.0 + parts.rand(W, seed=3, std=0.2)
    got = ops.row_norm_gate(o.cuda(), proj.to(dtype).cuda(), 16, w.cuda(), 1e-5).float().cpu().double()
    want = plain.rms(o.double(), w.double(), 1e-5) * torch.sigmoid(proj.double()[:, 16:16 + W])
    assert (got - want).abs().max() < parts.tol(dtype) * 4.0


@pytest.mark.parametrize("W", [64, 6, 1028, 4100, 12000])
def test_sum_of_branches(ops, W):
    """Rows in either type and experts' rows with and without places and weights, at widths with and without the vector form."""
    from paged_llm_b200.parts.base import LazyExperts, LazySum
    ops.set_compute_dtype(torch.bfloat16)
    rows, top = 5, 3
    x, a, nw = parts.rand(rows, W, seed=1), parts.rand(rows, W, seed=2), 1.0 + parts.rand(W, seed=3, std=0.1)
    e, wt = parts.rand(40, W, seed=4), torch.rand(rows, top, generator=torch.Generator().manual_seed(5))
    place = torch.randperm(40, generator=torch.Generator().manual_seed(6))[:rows * top].to(torch.int32)
    for kind in ("placed", "plain"):
        if kind == "placed":
            ex = LazyExperts(e.bfloat16().cuda(), top, place.cuda(), wt.reshape(-1).cuda(), rows)
            want_e = (e[place.long()].view(rows, top, W).double() * wt.double()[:, :, None]).sum(1)
        else:
            ex = LazyExperts(e[:rows * top].cuda().contiguous(), top, None, None, rows)
            want_e = e[:rows * top].view(rows, top, W).double().sum(1)
        both = LazySum((a.bfloat16().cuda(), ex))
        want = a.double() + want_e
        assert (both.materialize(ops).cpu().double() - want).abs().max() < 1e-4
        xd = x.cuda().clone()
        y = ops.branches_add_rms_norm(xd, list(both.parts), nw.cuda(), 1e-5).float().cpu().double()
        assert (xd.cpu().double() - x.double() - want).abs().max() < 1e-4
        assert (y - plain.rms(x.double() + want, nw.double(), 1e-5)).abs().max() < 4e-2


# ---------------------------------------------------------------- mixers alone
LENS = [1, 137, 70, 2]
MIXERS = [
    ("attention", 48, attention(4, 2, 16, 24, rot(12, 10000.0, (4.0, 1.0, 4.0, 40.0)), 11), 16),
    ("attention", 32, attention(6, 1, 8, 40, rot(8, 30.5), None, scale=0.4), 16),
    ("attention", 40, attention(3, 3, 32, 16, rot(2, 100.0), 8), 8),
    ("attention", 24, attention(2, 1, 16, 16, rot(16, 20.0), 1), 16),
    ("attention", 64, attention(8, 2, 64, 64, rot(64, 10000.0, (8.0, 1.0, 4.0, 128.0)), 65), 16),      # tcgen05 prefill
    ("attention", 64, attention(4, 1, 128, 128, rot(32, 100.0), 33, scale=0.05), 32),
    ("attention", 64, attention(2, 2, 64, 64, rot(6, 100.0), 50), 12),                                 # pages that TMA boxes do not fit
    ("attention", 64, attention(2, 1, 200, 256, rot(200, 5000.0), 90), 8),
    ("attention", 33, attention(3, 1, 10, 6, rot(10, 50.0), 20), 16),                                  # sizes that fill no quad
    ("attention", 48, attention(20, 1, 16, 16, rot(8, 50.0), 64), 8),
    ("attention_2", 48, convolved(4, 2, 16, 24, rot(12, 10000.0), 4), 16),
    ("attention_2", 24, convolved(2, 2, 16, 16, rot(16, 20.0), 1), 16),
    ("attention_2", 40, convolved(6, 1, 12, 8, rot(2, 100.0), 9, scale=0.5), 8),
    ("attention_2", 64, convolved(8, 2, 64, 64, rot(16, 10000.0), 3), 16),
    ("attention_2", 64, convolved(4, 1, 128, 128, rot(128, 100.0), 2, scale=0.05), 32),
    ("attention_2", 64, convolved(2, 1, 256, 200, rot(256, 5000.0), 5), 8),                            # a rotation over both of a lane's quads
    ("attention_2", 33, convolved(3, 1, 10, 6, rot(10, 50.0), 3), 16),
    ("attention_2", 64, convolved(1, 1, 32, 32, rot(24, 50.0), 64), 16),                               # the longest history
    ("lightning", 48, lightning(16, 24, 0.5, 1.0, 0.93), 8),
    ("lightning", 32, lightning(20, 6, 0.0, 0.99), 8),
    ("lightning", 40, lightning(3, 40, 0.9), 8),
    ("lightning", 64, lightning(64, 64, 0.8, 0.99), 8),
    ("lightning", 64, lightning(128, 128, 0.95, 0.999), 8),
    ("lightning", 64, lightning(100, 72, 0.95), 8),
    ("lightning", 64, lightning(256, 136, 0.9), 8),
    ("lightning", 48, lightning(33, 5, 0.7, 0.99), 8),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,W,m,ps", MIXERS)
def test_mixer_alone(ops, dtype, kind, W, m, ps):
    parts.check_mixer(kind, ops, "cuda", dtype, W, m, LENS, seed=3, ps=ps, ways=("whole", (0.6, 0.4), (0.25, 0.05, 0.7), "decode", ("every", 2), ("every", 19)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims,vdim", [(32, 32), (128, 128), (80, 160)])
def test_lightning_over_many_chunks(ops, dtype, dims, vdim):
    """Portions that end before, at and behind the borders of chunks and half chunks, several requests beside each other."""
    m = lightning(dims, vdim, 0.6, 0.99, 0.9999)
    parts.check_mixer("lightning", ops, "cuda", dtype, 32, m, [530, 128, 64, 65, 127, 129, 9, 256, 257], seed=5, scale_tol=4.0,
                      ways=("whole", (0.3, 0.7), (0.49, 0.02, 0.49), ("every", 64), ("every", 100), ("every", 9)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_decay_of_one_sums_everything(ops, dtype):
    """decay 1, keys and queries all alike: the state is the plain sum of what came, over a long prompt and decoding."""
    m = lightning(16, 16, 1.0)
    w = parts.mixer_weights("lightning", 16, m, 6)
    h = parts.rand(400, 16, seed=2)
    parts.check_mixer("lightning", ops, "cuda", dtype, 16, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 31)), scale_tol=4.0)


def test_steps_of_a_padded_graph_take_any_portions(ops):
    """A step captured for mixed items is replayed with other portions: what the kernels are launched for must not depend on the
    portions at hand.  The step is told it is padded, and its longest portion is given wrongly short."""
    ops.set_compute_dtype(torch.bfloat16)
    m = lightning(32, 32, 0.9, 0.99)
    H, d = 2, 32
    lens = [300, 5, 70]
    proj = parts.rand(sum(lens), 4 * H * d, seed=3).bfloat16().cuda()
    decay = torch.tensor(m["decay"]).cuda()
    dev = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")        # noqa: E731
    outs = []
    for padded, longest in ((False, 300), (True, 1)):
        ctx = types.SimpleNamespace(num_seqs=3, cu_seqlens_q=dev([0, 300, 305, 375]), state_slots=dev([2, 0, 1]), max_q_len=longest, padded=padded)
        state = torch.zeros(3, H * d * d, device="cuda")
        outs.append((ops.fixed_decay_attention(proj.clone(), H, d, d, decay, state, ctx).cpu(), state.cpu()))     # (silu is in place)
    assert torch.equal(outs[0][0], outs[1][0]) and torch.equal(outs[0][1], outs[1][1])


def test_gated_linear_attention_in_a_padded_step(ops):
    """The same for the linear attention with a decay per channel, whose long prompts run in segments."""
    ops.set_compute_dtype(torch.bfloat16)
    H, d = 2, 16
    lens = [500, 12]
    proj = parts.rand(sum(lens), 3 * H * d, seed=3).bfloat16().cuda()
    bias = parts.rand(H * d, seed=4).cuda()
    dev = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")        # noqa: E731
    outs = []
    for padded, longest in ((False, 500), (True, 256)):
        ctx = types.SimpleNamespace(num_seqs=2, cu_seqlens_q=dev([0, 500, 512]), state_slots=dev([1, 0]), max_q_len=longest, padded=padded)
        state = torch.zeros(2, H * d * d, device="cuda")
        z = parts.rand(sum(lens), H * d, seed=5).cuda()
        outs.append((ops.linear_attention_scan(proj, z, bias, H, d, d, 16.0, 0.25, state, ctx).cpu(), state.cpu()))
    assert (outs[0][0] - outs[1][0]).abs().max() < 1e-5 * outs[0][0].abs().max() and (outs[0][1] - outs[1][1]).abs().max() < 1e-5 * outs[0][1].abs().max()


# ---------------------------------------------------------------- weights made so that a fault shows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim", [(2, 1, 8), (4, 2, 64), (2, 1, 128)])
@pytest.mark.parametrize("kind,loud", [("attention", 5), ("attention", 63), ("attention_2", 15), ("attention_2", 16), ("attention_2", 64)])
def test_one_far_key_among_hundreds(ops, dtype, heads, kv, dim, kind, loud):
    """One key that every head answers to, on both sides of page and tile borders, seen from hundreds of tokens on, in a prompt's
    portions and decoding (every attention kernel form)."""
    scale = (8 / dim) ** 0.5 if kind == "attention" else 0.3
    m = attention(heads, kv, dim, dim, rot(4, 50.0), None, scale) if kind == "attention" else convolved(heads, kv, dim, dim, rot(4, 50.0), 3, scale)
    w, h = parts.loud_key(kind, 16, m, 600, loud, seed=1)
    want = parts.check_mixer(kind, ops, "cuda", dtype, 16, m, None, weights=w, hs=[h], ps=16, ways=("whole", "decode", (0.5, 0.5), (0.02, 0.98)),
                             scale_tol=4.0)
    assert parts.far_effect(kind, 16, m, w, h, loud, want)[-1] > 0.05, "the far key shows"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64, 128])
@pytest.mark.parametrize("size,loud", [(31, 61), (32, 64), (33, 65), (63, 125), (64, 64), (65, 129), (100, 100), (128, 127), (77, 80)])
def test_the_chunks_edge(ops, dtype, dim, size, loud):
    """A loud key shows up to the last position of its chunk and not behind it, at the chunk's start, inside and at its end."""
    m = attention(2, 1, dim, dim, rot(4, 50.0), size, (8 / dim) ** 0.5)
    w, h = parts.loud_key("attention", 16, m, 260, loud, seed=2)
    want = parts.check_mixer("attention", ops, "cuda", dtype, 16, m, None, weights=w, hs=[h], ps=16, ways=("whole", "decode", (0.3, 0.7)), scale_tol=4.0)
    diff = parts.far_effect("attention", 16, m, w, h, loud, want)
    end = min(260, loud - loud % size + size)
    assert diff[loud:end].min() > 0.05 and (end == 260 or diff[end:].max() < 1e-9)


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_in_the_denominator(ops, dtype):
    """Scores near zero and few keys: leaving the 1 out, counting it per split or scaling it would show at once."""
    m = convolved(2, 1, 16, 16, rot(8, 50.0), 2, 0.01)
    w = parts.mixer_weights("attention_2", 16, m, 2)
    h = parts.rand(700, 16, seed=3)
    want = parts.check_mixer("attention_2", ops, "cuda", dtype, 16, m, None, weights=w, hs=[h], ps=16, ways=("whole", "decode", (0.3, 0.7), ("every", 2)))
    assert want[0].abs().max() > 0.02


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
def test_a_far_token_through_the_state(ops, dtype, dim):
    m = lightning(dim, dim, 0.999, 0.5)
    w = parts.mixer_weights("lightning", 16, m, 4)
    h = 0.3 * parts.rand(300, 16, seed=8)
    h[0] = 4.0 * parts.rand(16, seed=9)
    h = h.to(torch.bfloat16).float()
    want = parts.check_mixer("lightning", ops, "cuda", dtype, 16, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 2)), scale_tol=4.0)
    h2 = h.clone()
    h2[0] = -h2[0]
    other = plain.lightning(h2.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    assert (want[-1] - other[-1]).abs().max() > 1e-2, "the first token does not show"


# ---------------------------------------------------------------- the engine against the plain model
LENGTHS = {"A": (1, 30, 77, 49, 2, 60), "B": (5, 41, 120, 13, 80), "C": (3, 270, 33, 141), "D": (2, 66, 35)}


def rounding_of(folder, toks, dtype):
    return rounding_error(folder, toks, torch.bfloat16 if dtype == "bfloat16" else torch.float32)


def replay(folder, dtype, steps, max_tokens, block_size=16, slots=4, **kw):
    from paged_llm_b200.engine.replay import TraceReplayer

    rp = TraceReplayer(folder, dtype, max_tokens, block_size=block_size, poison=float("nan"), max_num_seqs=slots, **kw)
    for state in rp.storage._state_tensors():
        state.fill_(float("nan"))                     # a slot that is not zeroed at a request's start shows
    outputs = {}
    for rec in steps:
        out = rp.step(rec)
        if out is not None:
            outputs[rec["step"]] = out
    assert not rp.live, "requests left alive at the end of the trace"
    rp.cm.check_invariants([])
    for g in range(len(rp.cm.pools)):
        assert rp.cm.num_free_in_group(g) == rp.cm.pools[g].num_pages, "pages were lost"
    assert rp.cm.num_free_state_slots == rp.cm.num_state_slots
    return outputs, rp


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: case_folder(tmp_path_factory, name) for name in CASES}


@pytest.fixture(scope="module")
def drawn(folders):
    """Requests by (case, precision, lengths, seed), drawn once: float32 takes any, bfloat16 those on which no router has a
    close call."""
    seen = {}

    def get(name, dtype, lengths=None, seed=None):
        lengths = lengths or (LENGTHS[name] if dtype == "float32" or name != "C" else (3, 150, 33, 80))
        seed = ord(name) if seed is None else seed
        key = (name, dtype, lengths, seed)
        if key not in seen:
            vocab = CASES[name][0]["vocab"]
            seen[key] = requests_for(vocab, lengths, seed=seed) if dtype == "float32" else clear_requests(folders[name], vocab, lengths, seed=seed)
        return seen[key]

    return get


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
@pytest.mark.parametrize("schedule", ["whole", "tail", "portions", "mixed"])
def test_schedule_matches_plain(folders, drawn, name, dtype, schedule):
    reqs = drawn(name, dtype)
    steps, max_tokens = getattr(schedules, schedule)(reqs)
    outputs, rp = replay(folders[name], dtype, steps, max_tokens, block_size=8 if name == "B" else 16)
    got = schedules.collect(steps, outputs)
    for rid, toks in reqs.items():
        close(got[rid], plain_logits(folders[name], toks), dtype, f"{schedule}/{name}/{rid}", rounding_of(folders[name], toks, dtype))
    if schedule == "tail":
        assert rp.runner.num_graph_steps > 0, "decode steps replay graphs: every part of the model can be captured"


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_bfloat16_against_the_float32_engine(folders, drawn, name):
    reqs = drawn(name, "bfloat16")
    steps, max_tokens = schedules.mixed(reqs)
    a, _ = replay(folders[name], "float32", steps, max_tokens)
    b, _ = replay(folders[name], "bfloat16", steps, max_tokens)
    a, b = schedules.collect(steps, a), schedules.collect(steps, b)
    for rid, toks in reqs.items():
        close(b[rid], a[rid], "bfloat16", f"{name}/{rid}", rounding_of(folders[name], toks, "bfloat16"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_graph_and_eager_decode_agree(folders, drawn, dtype):
    reqs = drawn("A", dtype, (66, 90), 5)
    steps, max_tokens = schedules.tail(reqs, last=45)
    a, rp_a = replay(folders["A"], dtype, steps, max_tokens)
    b, rp_b = replay(folders["A"], dtype, steps, max_tokens, enforce_eager=True)
    assert rp_a.runner.num_graph_steps > 0 and rp_b.runner.num_graph_steps == 0
    for k in a:
        close(a[k], b[k], dtype, f"graph vs eager step {k}")


def test_long_decoding(folders, tmp_path):
    """Three hundred tokens one by one behind a short prompt, beside a second request that does the same; every chunk of the
    models passes over decoded tokens.  In bfloat16 on case A with dense feed-forwards, whose requests need no drawing."""
    hf = copy.deepcopy(CASE_A)
    for lay in hf["layers"]:
        lay["mlp"] = dense(40)
    plain_folder = make_folder(tmp_path, hf, 7)
    for folder, vocab, dtype in ((folders["A"], CASE_A["vocab"], "float32"), (folders["C"], CASE_C["vocab"], "float32"),
                                 (plain_folder, hf["vocab"], "bfloat16")):
        reqs = requests_for(vocab, (330, 311), seed=12)
        steps, max_tokens = schedules.mixed(reqs, live=2, seed=3, prompt_fraction=0.08)
        outputs, _ = replay(folder, dtype, steps, max_tokens, block_size=8, slots=2)
        got = schedules.collect(steps, outputs)
        for rid, toks in reqs.items():
            close(got[rid], plain_logits(folder, toks), dtype, f"long decoding {dtype}/{rid}", rounding_of(folder, toks, dtype))


def test_mixed_steps_replay_one_graph_with_other_portions(folders):
    """Steps of the same 64-token bucket whose portions differ from step to step (a long one beside short ones, then several
    alike): they replay one captured graph."""
    reqs = requests_for(CASE_C["vocab"], (330, 120, 60), seed=21)
    cuts = {"r0": (20, 40, 100, 30, 9, 120, 11), "r1": (40, 20, 10, 30, 20), "r2": (4, 4, 10, 40, 2)}
    steps, at = [], {k: 0 for k in reqs}
    for i in range(7):
        entries, ended = [], []
        for rid, toks in reqs.items():
            if i >= len(cuts[rid]):
                continue
            n = cuts[rid][i]
            entries.append({"id": rid, "tokens": toks[at[rid]:at[rid] + n], "want": [n - 1]})
            at[rid] += n
            if i == len(cuts[rid]) - 1:
                ended.append(rid)
        steps.append({"step": i, "entries": entries, "end": ended})
    assert all(at[r] == len(t) for r, t in reqs.items())
    for dtype in ("float32", "bfloat16"):
        outputs, rp = replay(folders["C"], dtype, steps, 640)
        got, pos = schedules.collect(steps, outputs), schedules.wanted_positions(steps)
        other, _ = replay(folders["C"], dtype, steps, 640, enforce_eager=True)
        other = schedules.collect(steps, other)
        assert rp.runner.num_graph_steps >= 2
        for rid, toks in reqs.items():
            close(got[rid], other[rid], dtype, f"graphs against launches {dtype}/{rid}")
            if dtype == "float32":
                close(got[rid], plain_logits(folders["C"], toks)[pos[rid]], dtype, rid, rounding_of(folders["C"], toks, dtype)[pos[rid]])


def test_first_tokens(folders):
    """Requests of one and two tokens, alone and in one batch."""
    for name in sorted(CASES):
        reqs = requests_for(CASES[name][0]["vocab"], (1, 2, 1, 2), seed=3)
        steps = [{"step": 0, "entries": [{"id": k, "tokens": t, "want": list(range(len(t)))} for k, t in reqs.items()], "end": list(reqs)}]
        outputs, _ = replay(folders[name], "float32", steps, 256)
        got = schedules.collect(steps, outputs)
        for rid, toks in reqs.items():
            close(got[rid], plain_logits(folders[name], toks), "float32", f"first tokens {name}/{rid}")


@pytest.mark.parametrize("seed", range(10))
def test_generated_configurations(tmp_path, seed):
    hf = generated_case(300 + seed)
    folder = make_folder(tmp_path, hf, seed)
    for dtype in ("float32", "bfloat16"):
        lengths = (2, 50, 21, 70, 9, 130)
        reqs = requests_for(hf["vocab"], lengths, seed=seed) if dtype == "float32" else clear_requests(folder, hf["vocab"], lengths, seed=seed)
        steps, max_tokens = schedules.mixed(reqs, live=3, seed=seed)
        outputs, _ = replay(folder, dtype, steps, max_tokens, slots=3)
        got = schedules.collect(steps, outputs)
        for rid, toks in reqs.items():
            close(got[rid], plain_logits(folder, toks), dtype, f"generated {seed}/{dtype}/{rid}", rounding_of(folder, toks, dtype))


@pytest.mark.parametrize("seed", [1, 3])
def test_wide_generated_configurations(tmp_path, seed):
    """Drawn configurations at widths of 256 to 512 under a mixed schedule, float32 against the plain model and bfloat16
    against the float32 engine (which is measured against the plain model in the same test)."""
    hf = wide_case(seed)
    folder = make_folder(tmp_path, hf, seed)
    reqs = clear_requests(folder, hf["vocab"], (3, 90, 1, 33, 140), seed=seed)
    steps, max_tokens = schedules.mixed(reqs, live=4, seed=seed)
    a, _ = replay(folder, "float32", steps, max_tokens)
    b, _ = replay(folder, "bfloat16", steps, max_tokens)
    a, b = schedules.collect(steps, a), schedules.collect(steps, b)
    for rid, toks in reqs.items():
        close(a[rid], plain_logits(folder, toks), "float32", f"wide {seed}/float32/{rid}", rounding_of(folder, toks, "float32"))
        close(b[rid], a[rid], "bfloat16", f"wide {seed}/bfloat16/{rid}", rounding_of(folder, toks, "bfloat16"))


def test_greedy_generation_through_the_engine(folders):
    from paged_llm_b200 import LLMEngine, SamplingParams
    prompts = list(requests_for(CASE_A["vocab"], (3, 22, 47, 9, 31), seed=60).values())
    eng = LLMEngine(folders["A"], dtype="float32", block_size=16, num_gpu_blocks=24, max_model_len=96,
                    max_num_batched_tokens=16, max_num_seqs=3)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12))
    for p, o in zip(prompts, outs):
        assert o.token_ids == plain_greedy(folders["A"], p, 12)
    assert eng.block_manager.num_free_state_slots == 3


def test_generation_with_preemption_restarts_the_state(folders):
    from paged_llm_b200 import LLMEngine, SamplingParams
    prompts = list(requests_for(CASE_C["vocab"], (30, 26, 21, 12), seed=70).values())
    eng = LLMEngine(folders["C"], dtype="float32", block_size=8, num_gpu_blocks=11, max_model_len=88,
                    max_num_batched_tokens=24, max_num_seqs=4)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=16))
    assert sum(o.num_preemptions for o in outs) > 0, "the pool was meant to run out"
    for p, o in zip(prompts, outs):
        assert o.token_ids == plain_greedy(folders["C"], p, 16)
    assert eng.block_manager.num_free_state_slots == 4


def test_trace_runner_as_a_program(folders, tmp_path):
    """bin/trace_run on case B: two requests in portions and single tokens, the files it writes against the plain model."""
    reqs = requests_for(CASE_B["vocab"], (40, 23), seed=9)
    steps, max_tokens = schedules.mixed(reqs, live=2, seed=1)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["B"], "--dtype", "float32", "--out",
                        str(out), "--max-tokens", str(max_tokens), "--max-requests", "2"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == [f"done {s['step']}" for s in steps]
    outputs = {s["step"]: np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, CASE_B["vocab"]) for s in steps
               if any(e["want"] for e in s["entries"])}
    got = schedules.collect(steps, outputs)
    for rid, toks in reqs.items():
        close(got[rid], plain_logits(folders["B"], toks), "float32", f"trace_run {rid}")
