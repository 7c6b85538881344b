"""The Tagelorn decoder on the GPU: each new kernel and each mixer alone against the plain functions, then the engine
under every schedule in both precisions against the plain model."""

from __future__ import annotations

import copy
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import plain_tagelorn as plain
from tests import schedules
from tests import tagelorn_parts as parts
from tests.helpers import requests_for
from tests.tagelorn_cases import (CASE_A, CASE_B, CASE_C, CASES, attention, case_folder, clear_requests, delta, dense, generated_case, make_folder,
                                  moe, plain_greedy, plain_logits, rounding_error, wide_case)

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
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,scale", [(64, 2.0), (7, 1.0), (2050, 12.5)])
def test_sinusoids(ops, dtype, W, scale):
    parts.check_sinusoids(ops, "cuda", dtype, W, scale, [0, 1, 2, 63, 1000, 65537, 1000003])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,dim,layers,which,rows", [(32, 12, 3, 1, 9), (48, 8, 1, 0, 1), (20, 5, 4, 3, 17), (1024, 64, 2, 1, 300), (288, 40, 3, 2, 16),
                                                     (5000, 32, 2, 0, 3)])
def test_token_input(ops, dtype, W, dim, layers, which, rows):
    """The stream takes the branch and the normed token input in, and the next norm reads the result; widths that four-element
    accesses do not fit and widths beyond what a block keeps in registers.  (The seed: the norm of a projected vector that
    nearly vanishes would magnify bfloat16's rounding of it.)"""
    parts.check_token_side(ops, "cuda", dtype, W, dim, layers, which, rows, seed=2)


def test_capped_logits(ops):
    x = 30.0 * parts.rand(7, 333, seed=1)
    got = ops.softcap(x.cuda().clone(), 12.5).cpu().double()
    assert (got - 12.5 * torch.tanh(x.double() / 12.5)).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,K,N", [(5, 64, 48), (16, 128, 40), (40, 64, 24), (2100, 128, 72), (3, 20, 12)])
def test_square_of_relu_behind_a_product(ops, dtype, rows, K, N):
    """In the epilogue of the weight-streaming and the tcgen05 product, and as a kernel behind the others."""
    ops.set_compute_dtype(dtype)
    h, w = parts.rand(rows, K, seed=1), parts.rand(N, K, seed=2, std=K ** -0.5)
    got = ops.relu2_linear(h.to(dtype).cuda(), w.to(dtype).cuda()).float().cpu().double()
    want = (h.double() @ w.double().T).clamp(min=0.0) ** 2
    assert (got - want).abs().max() < parts.tol(dtype, 2.0) * max(1.0, want.max().item())


@pytest.mark.parametrize("mlp,W,rows", [(moe(16, 6, 2, 1.5, (3, 2), shared=24), 32, 40), (moe(24, 4, 1, 1.0, (1, 1)), 32, 9),
                                        (moe(8, 5, 3, 0.5, shared=8), 40, 33), (moe(64, 8, 4, 2.0, (4, 2), shared=64), 64, 300),
                                        (moe(40, 64, 6, 1.0, (8, 3), shared=20), 64, 50), (moe(64, 12, 2, 2.5, (3, 1), shared=128), 128, 2100),
                                        (moe(12, 6, 2, 1.0, shared=20), 36, 21)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_alone(ops, dtype, mlp, W, rows):
    """Corrected softmax scores, groups by their largest, experts of one matrix and the square of relu, in every form of the
    products (tiles of 16 and 64 pairs, the grouped tcgen05 form from 2,048 pairs on, FFMA chains)."""
    parts.check_experts(ops, "cuda", dtype, W, mlp, rows, seed=13, scale_tol=4.0)


# ---------------------------------------------------------------- mixers alone
LENS = [1, 137, 70, 2]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,m,rows,ps", [
    (48, attention(4, 2, 16, 24, 40, (9, 3)), 8, 16),
    (32, attention(6, 1, 8, 40, 30.5, scale=0.4), 4, 16),                     # no window
    (40, attention(3, 3, 32, 16, 100, (5, 21)), 16, 8),                       # more kept tokens than the window holds
    (24, attention(2, 1, 16, 16, 20, (1, 1)), 8, 16),
    (64, attention(8, 2, 64, 64, 128, (65, 6)), 16, 16),                      # tcgen05 prefill, head size 64
    (64, attention(4, 2, 64, 64, 128, (20, 70)), 16, 16),                     # kept tokens over two tiles
    (64, attention(4, 1, 128, 128, 60, (33, 4), scale=0.05), 8, 32),          # head size 128
    (64, attention(2, 2, 64, 64, 90, (50, 10)), 8, 12),                       # pages that TMA boxes do not fit
    (64, attention(20, 1, 16, 16, 40, (30, 2)), 8, 16),
    (64, attention(2, 1, 200, 256, 40, (30, 2)), 8, 16),
    (48, attention(4, 2, 64, 64, 40, (24, 0)), 8, 16),
    (48, attention(8, 1, 64, 64, 70, (90, 3)), 8, 16),                        # the largest group whose biases are staged,
    (48, attention(9, 1, 64, 64, 70, (90, 3)), 8, 16),                        # and one beyond it
    (48, attention(3, 1, 128, 128, 70.5), 16, 16),
    (48, attention(14, 2, 64, 64, 300), 16, 16),
])
def test_attention_alone(ops, dtype, W, m, rows, ps):
    parts.check_attention(ops, "cuda", dtype, W, m, LENS, seed=3, rows=rows, ps=ps)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,m,rank", [(48, delta(3, 16), 5), (32, delta(2, 20), 8), (40, delta(1, 40), 1), (64, delta(2, 64), 16), (64, delta(1, 128), 24),
                                      (64, delta(1, 200), 8), (40, delta(2, 6), 3), (32, delta(2, 33), 3)])
def test_delta_rule_alone(ops, dtype, W, m, rank):
    """Every form of the recurrence's kernels (key sizes up to 32, 64, 128, 256), sizes that fill neither lanes nor columns."""
    parts.check_delta(ops, "cuda", dtype, W, m, LENS, seed=7, rank=rank, ways=("whole", (0.6, 0.4), (0.25, 0.05, 0.7), "decode", ("every", 2), ("every", 19)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,taps,inner,m", [(32, 4, "general_delta", delta(2, 8)), (24, 2, "attention", attention(2, 1, 8, 8, 40, (5, 2))),
                                            (24, 1, "attention", attention(2, 2, 8, 8, 40)), (20, 7, "general_delta", delta(1, 12)),
                                            (27, 3, "general_delta", delta(1, 8)), (288, 5, "general_delta", delta(2, 16))])
def test_input_convolution_alone(ops, dtype, W, taps, inner, m):
    parts.check_input_convolution(ops, "cuda", dtype, W, taps, inner, m, [1, 3, 70, 33], seed=9)


# ---------------------------------------------------------------- weights made so that a fault shows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim", [(2, 1, 8), (4, 2, 64), (2, 1, 128)])
@pytest.mark.parametrize("loud,mask", [(5, None), (63, None), (15, (16, 16)), (16, (16, 16)), (17, (100, 18)), (18, (100, 18)), (63, (70, 64)), (64, (70, 64)),
                                       (69, (33, 70)), (70, (33, 70))])
def test_one_far_key_among_hundreds(ops, dtype, heads, kv, dim, loud, mask):
    """One key that every head answers to, as the last kept token and the first that is not, on both sides of page and tile
    borders, in a prompt's portions and decoding (every attention kernel form: the float32 kernel, mma.sync tiles, tcgen05
    at head sizes 64 and 128, decode as clusters)."""
    W, m = 16, attention(heads, kv, dim, dim, 128, mask, scale=0.9 * (8 / dim) ** 0.5)
    w, h = parts.loud_key(W, m, 600, loud, seed=1)
    want = parts.check_attention(ops, "cuda", dtype, W, m, None, weights=w, hs=[h], ps=16, ways=("whole", "decode", (0.5, 0.5), (0.02, 0.98)),
                                 scale_tol=4.0)
    other = h.clone()
    other[loud, 0] = 0.0
    quiet = plain.attention(other.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    moved = (want[-1] - quiet[-1]).abs().max().item()
    seen = mask is None or loud < mask[1]
    assert moved > 0.1 if seen else moved < 1e-9, "the far key shows exactly if it is kept"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64, 128])
@pytest.mark.parametrize("size,keep", [(31, 2), (32, 2), (33, 2), (63, 5), (64, 5), (65, 0), (128, 1)])
def test_the_windows_edge(ops, dtype, dim, size, keep):
    """A loud key at the last distance inside the window shows, one step later it does not."""
    W, m = 16, attention(2, 1, dim, dim, 80, (size, keep), scale=0.9 * (8 / dim) ** 0.5)
    loud = 77
    w, h = parts.loud_key(W, m, 260, loud, seed=2)
    want = parts.check_attention(ops, "cuda", dtype, W, m, None, weights=w, hs=[h], ps=16, ways=("whole", "decode", (0.3, 0.7)), scale_tol=4.0)
    other = h.clone()
    other[loud, 0] = 0.0
    quiet = plain.attention(other.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    diff = (want - quiet).abs().amax(1)
    assert diff[loud + size - 1] > 0.1 and diff[loud + size:].max() < 1e-9


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_large_sink_takes_the_weight(ops, dtype):
    """sink = 12 against scores near zero: leaving the sink out, counting it per split or scaling it would show at once."""
    W, m = 16, attention(2, 1, 16, 16, 50, None, scale=0.02)
    w = parts.attention_weights(W, m, seed=2)
    w["a.rel"][:] = 0.0
    w["a.sink"][:] = 12.0
    h = parts.rand(700, W, seed=3)
    want = parts.check_attention(ops, "cuda", dtype, W, m, None, weights=w, hs=[h], ps=16, ways=("whole", "decode", (0.3, 0.7)))
    assert want.abs().max() < 0.1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
def test_a_far_token_through_the_delta_state(ops, dtype, dim):
    W, m = 16, delta(2, dim)
    w = parts.delta_weights(W, m, seed=4, w0=-8.0)
    w["d.w2"] = w["d.w2"] * 0.1
    w["d.a"], w["d.a.b"] = w["d.a"] * 0.1, torch.full((2 * dim,), -7.0)
    h = parts.rand(300, W, seed=8)
    want = parts.check_delta(ops, "cuda", dtype, W, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 2)), scale_tol=4.0)
    h2 = h.clone()
    h2[0] = -3.0 * h2[0]
    other = plain.general_delta(h2.double(), {k: v.double() for k, v in w.items()}, "d.", m, 1e-5)
    assert (want[-1] - other[-1]).abs().max() > 1e-2, "the first token does not show"


@pytest.mark.parametrize("dim", [16, 64, 100])
def test_fast_decays_and_full_removal(ops, dim):
    """Every decay at its fastest (0.545 per token) and every removal rate near one, over a long prompt in float32."""
    W, m = 24, delta(2, dim)
    w = parts.delta_weights(W, m, seed=6, w0=9.0)
    w["d.a.b"] = torch.full((2 * dim,), 6.0)
    parts.check_delta(ops, "cuda", torch.float32, W, m, [530, 97], weights=w, ways=("whole", (0.33, 0.67), ("every", 50)))


# ---------------------------------------------------------------- the engine against the plain model
LENGTHS = {"A": (1, 30, 77, 49, 2, 60, 90, 35), "B": (5, 41, 120, 13, 80, 55), "C": (3, 270, 33, 190, 18, 141)}


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
@pytest.mark.parametrize("name", ["A", "B", "C"])
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
    """Three hundred tokens one by one behind a short prompt, beside a second request that does the same; every window of
    the models passes over decoded tokens.  In bfloat16 on case A with dense feed-forwards, whose requests need no drawing."""
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


def test_first_tokens(folders):
    """Requests of one and two tokens, alone and in one batch."""
    for name in ("A", "B", "C"):
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
    import json
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
