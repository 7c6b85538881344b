"""The Nopozen decoder on the host: configuration, the model as data, each mechanism by hand and alone and the engine's host
logic (runner, cache manager, state slots, replay, scheduler) with the kernel library replaced by the tensor-code stand-in,
against the plain implementation."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

from paged_llm_b200.config.model import ConfigError
from paged_llm_b200.config.nopozen import NopozenConfig
from paged_llm_b200.config.registry import parse_model_config
from paged_llm_b200.models.causal_lm import build_model
from paged_llm_b200.parts.base import FixedState, PagedKV
from tests import nopozen_parts as parts
from tests import plain_nopozen as plain
from tests import schedules
from tests.helpers import requests_for
from tests.nopozen_cases import (CASE_A, CASE_B, CASES, attention, case_folder, convolved, dense, generated_case, lightning, make_folder, moe,
                                 plain_greedy, plain_logits, read_folder, rot, rounding_error)
from tests.torch_ops import TorchOps

F32_TOL = 2e-5
F32 = torch.float32


def close(got, want, what, rounding=None):
    """Largest difference within F32_TOL of the largest logit; with `rounding` (per position, the root mean square of what
    float32 alone does to the plain model) a position passes too if its root mean square error is within 10 times that."""
    assert got.shape == want.shape, what
    assert np.isfinite(got).all(), what
    err = np.abs(got - want)
    bad = err.max(axis=1) > F32_TOL * max(1.0, float(np.abs(want).max()))
    if rounding is not None:
        bad &= np.sqrt((err.astype(np.float64) ** 2).mean(axis=1)) > 10.0 * rounding
    assert not bad.any(), f"{what}: max |diff| {err.max():.3e}, first bad row {int(np.argmax(bad))} ({err[int(np.argmax(bad))].max():.3e})"


def replay(folder, steps, max_tokens, block_size=8, slots=4):
    from paged_llm_b200.engine.replay import TraceReplayer

    rp = TraceReplayer(folder, "float32", max_tokens, device="cpu", ops=TorchOps(), block_size=block_size, max_num_seqs=slots,
                       poison=float("nan"))
    for state in rp.storage._state_tensors():
        state.fill_(float("nan"))                      # a slot that is not zeroed at a request's start shows
    outputs = {}
    for rec in steps:
        out = rp.step(rec)
        if out is not None:
            outputs[rec["step"]] = out
    assert not rp.live
    rp.cm.check_invariants([])
    for g in range(len(rp.cm.pools)):
        assert rp.cm.num_free_in_group(g) == rp.cm.pools[g].num_pages, "pages were lost"
    assert rp.cm.num_free_state_slots == rp.cm.num_state_slots, "state slots were lost"
    return outputs, rp


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: case_folder(tmp_path_factory, name) for name in CASES}


@pytest.fixture(scope="module")
def ops():
    return TorchOps()


# ---------------------------------------------------------------- configuration
def test_configuration_round_trip():
    for hf, _ in CASES.values():
        arch, cfg = parse_model_config(hf)
        assert arch.name == "Nopozen"
        assert NopozenConfig.from_hf_dict(cfg.to_hf_dict()) == cfg
        back = cfg.to_hf_dict()
        back.pop("torch_dtype")
        assert back == hf
        specs = build_model(arch.build_spec(cfg)).tensor_specs()
        assert cfg.num_parameters == sum(int(np.prod(s.shape)) for s in specs.values())
        assert cfg.layer_runs() == plain.layer_runs(hf)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "not implemented"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=9.0), "low"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"].update(mask={"size": 4}), "mask"),
    (lambda c: c["layers"][0]["mixer"]["decay"].pop(), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5, 0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(dim=0), "dim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "dense and moe only"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("width"), "width"),
])
def test_configuration_refusals(change, message):
    hf = copy.deepcopy(CASE_A)
    change(hf)
    with pytest.raises(ConfigError, match=message):
        parse_model_config(hf)


def test_the_model_as_data():
    """Case A: every run of a looped layer keeps a cache of its own; the convolved attention keeps its last three projected
    values beside its pages; attention caches heads padded to the larger of key and value size, within its chunk."""
    arch, cfg = parse_model_config(CASE_A)
    model = build_model(arch.build_spec(cfg))
    lit, att = FixedState((3 * 16 * 24,)), PagedKV(2, 32, None, 11)
    assert [s.requirement for s in model.cache_slots()] == [lit, att] * 3 + [
        (FixedState((3 * (2 * 32 + 2 * 32 + 2 * 16),)), PagedKV(2, 32)), FixedState((2 * 8 * 8,))]
    assert [e.join_embedding for e in model.schedule] == [True, False] * 3 + [False, False]
    specs = model.tensor_specs()
    assert {"embed", "head", "loop.in", "final.norm", "l1.mix.q.norm", "l1.mix.o.b", "l1.mix.g", "l2.mix.v.conv", "l0.mix.norm",
            "l0.mlp.router.b", "l0.mlp.e5.gate", "l1.mlp.down"} <= set(specs)
    assert specs["loop.in"].shape == (64, 128) and specs["l1.mix.g"].shape == (4, 64) and specs["l2.mix.g"].shape == (32, 64)
    assert not any(n.startswith("l2.mlp") or n.endswith("norm2") for n in specs)
    assert not any(s.optional for s in specs.values()) and model.has_fixed_state
    # one tap leaves nothing to keep, and without a loop nothing is joined
    hf = copy.deepcopy(CASE_A)
    hf["layers"] = hf["layers"][1:3]
    hf["layers"][1]["mixer"]["conv"] = 1
    hf.pop("loop")
    arch, cfg = parse_model_config(hf)
    model = build_model(arch.build_spec(cfg))
    assert not model.has_fixed_state and "loop.in" not in model.tensor_specs()


# ---------------------------------------------------------------- mechanisms by hand
def test_scaled_frequencies_by_hand():
    """Base 16, four dims: the frequencies 1 and 1/4 have waves of 2 pi and 8 pi.  Against 50 positions with low 1 and high 4
    the first turns 8 times (kept), the second 1.99 times (blended: s = (50 / (8 pi) - 1) / 3); against 20 positions the
    second turns less than once (divided)."""
    from paged_llm_b200.parts.rope import RotaryEncoding
    s = (50.0 / (8.0 * math.pi) - 1.0) / 3.0
    for original, second in ((50.0, (1.0 - s) * 0.25 / 8.0 + s * 0.25), (20.0, 0.25 / 8.0), (200.0, 0.25)):
        first = 1.0
        if original == 20.0:
            u = (20.0 / (2.0 * math.pi) - 1.0) / 3.0
            first = (1.0 - u) / 8.0 + u
        r = rot(4, 16.0, (8.0, 1.0, 4.0, original))
        assert np.allclose(plain.frequencies(r), [first, second], rtol=1e-12)
        enc = RotaryEncoding({}, head_dim=4, theta=16.0, exact=True, scaling=dict(
            type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_position_embeddings=original))
        assert np.allclose(enc.inv_freq().numpy(), [first, second], rtol=1e-7)


def _silent(kind, W, m):
    """Scores all zero, gates of one half, output = the first value element times 2."""
    w = parts.mixer_weights(kind, W, m, 1)
    for name, t in w.items():
        if not name.endswith("norm"):
            t[:] = 0.0
    w["a.v"][0, 0] = 1.0
    w["a.o"][0, 0] = 2.0
    return w


def test_chunks_by_hand(ops):
    """Every visible key weighs the same; values are the position itself, so the output is the mean of the visible positions:
    chunks of three, counted from position 0 however the prompt is cut."""
    W, m = 4, attention(1, 1, 4, 2, rot(2, 10.0), 3)
    w = _silent("attention", W, m)
    h = torch.zeros(10, W)
    h[:, 0] = torch.arange(10.0)
    want = np.array([np.mean(range(i - i % 3, i + 1)) for i in range(10)])
    assert np.allclose(plain.chunked_attention(h.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)[:, 0], want)
    part = parts.mixer_part("attention", W, m, w, 1e-5, F32, "cpu", ops)
    for out in parts.run_mixer(ops, "cpu", part, [h], F32, ps=2, ways=("whole", "decode", ("every", 2), ("every", 4))):
        assert np.allclose(out[:, 0], want, atol=1e-5)


def test_one_in_the_denominator_by_hand(ops):
    """Scores all zero over i + 1 keys and one more term of e^0: the output is the sum of the values over i + 2."""
    W, m = 4, convolved(1, 1, 4, 2, rot(2, 10.0), 2)
    w = _silent("attention_2", W, m)
    for x in "qkv":
        w[f"a.{x}.conv"][:, 0], w[f"a.{x}.conv"][:, 1] = 10.0, 1.0          # y_t = u_t + 10 u_(t-1)
    h = torch.zeros(7, W)
    h[:, 0] = torch.arange(1.0, 8.0)
    v = np.array([t + 10.0 * (t - 1) for t in range(1, 8)])
    want = np.cumsum(v) / (np.arange(7) + 2.0)
    assert np.allclose(plain.convolved_attention(h.double(), {k: t.double() for k, t in w.items()}, "a.", m, 1e-5)[:, 0], want)
    part = parts.mixer_part("attention_2", W, m, w, 1e-5, F32, "cpu", ops)
    for out in parts.run_mixer(ops, "cpu", part, [h], F32, ps=2, ways=("whole", "decode", ("every", 2))):
        assert np.allclose(out[:, 0], want, rtol=1e-5)


def test_scale_of_a_heads_projection_does_not_matter():
    W, m = 16, attention(4, 2, 8, 8, rot(8, 100.0), 6)
    w = {k: v.double() for k, v in parts.mixer_weights("attention", W, m, seed=4).items()}
    h = parts.rand(11, W, seed=5).double()
    a = plain.chunked_attention(h, w, "a.", m, 1e-12)
    w2 = dict(w)
    for name, rows in (("a.q", slice(8, 16)), ("a.k", slice(0, 8))):
        for t in (name, name + ".b"):
            w2[t] = w2[t].clone()
            w2[t][rows] *= 7.0
    assert (plain.chunked_attention(h, w2, "a.", m, 1e-12) - a).abs().max() < 1e-9


def test_lightning_by_hand(ops):
    """Two heads of one channel and one value each: S <- decay S + k v, o = S q, both heads under one norm."""
    W, m = 3, lightning(1, 1, 0.5, 1.0)
    w = parts.mixer_weights("lightning", W, m, 0)
    w.update({"a.q": torch.tensor([[0.0, 0, 1.0], [0, 0, 1.0]]), "a.k": torch.tensor([[1.0, 0, 0], [1.0, 0, 0]]),
              "a.v": torch.tensor([[0, 1.0, 0], [0, 1.0, 0]]), "a.g": torch.tensor([[0, 0, 1.0], [0, 0, 0]]),
              "a.norm": torch.tensor([1.5, 0.5]), "a.o": torch.tensor([[1.0, 0], [0, 1.0], [0, 0]])})
    h = torch.tensor([[2.0, 1.0, 0.5], [-1.0, 3.0, -0.5], [0.5, -2.0, 1.0]])
    sig = lambda z: 1 / (1 + math.exp(-z))      # noqa: E731
    silu = lambda z: z * sig(z)                 # noqa: E731
    eps, S, want = 1e-3, [0.0, 0.0], []
    for a, b, c in h.tolist():
        S = [dec * s + silu(a) * silu(b) for dec, s in zip((0.5, 1.0), S)]
        o = [s * silu(c) for s in S]
        f = 1.0 / math.sqrt((o[0] ** 2 + o[1] ** 2) / 2 + eps)
        want.append([o[0] * f * 1.5 * sig(c), o[1] * f * 0.5 * 0.5])
    got = plain.lightning(h.double(), {k: v.double() for k, v in w.items()}, "a.", m, eps)
    assert np.allclose(got[:, :2].numpy(), want, rtol=1e-9)
    part = parts.mixer_part("lightning", W, m, w, eps, F32, "cpu", ops)
    for out in parts.run_mixer(ops, "cpu", part, [h], F32, ways=("whole", "decode")):
        assert np.allclose(out[:, :2].numpy(), want, rtol=1e-4)


def test_router_by_hand():
    """Logits 1, 3, 2 with biases 2.5, -1, 0: 3.5, 2, 2 + a hair for the third; the two largest take the token."""
    one = torch.ones(1, 1, dtype=torch.float64)
    z, b = torch.tensor([[1.0], [3.0], [2.001]], dtype=torch.float64), torch.tensor([2.5, -1.0, 0.0], dtype=torch.float64)
    idx, wt = plain.router(one, z, b, 2)
    assert idx[0].tolist() == [0, 2]
    e = math.exp(2.001 - 3.5)
    assert np.allclose(wt[0].tolist(), [1 / (1 + e), e / (1 + e)])
    assert plain.router(one, z, 0 * b, 2)[0][0].tolist() == [1, 2], "the bias changes the choice"


# ---------------------------------------------------------------- each mechanism alone, through prompts and decoding
MIXERS = [
    ("attention", 48, attention(4, 2, 16, 24, rot(12, 10000.0, (4.0, 1.0, 4.0, 40.0)), 11)),
    ("attention", 32, attention(6, 1, 8, 40, rot(8, 30.5), None, scale=0.4)),                     # no mask
    ("attention", 40, attention(3, 3, 32, 16, rot(2, 100.0), 8)),                                 # chunks on page borders
    ("attention", 24, attention(2, 1, 16, 16, rot(16, 20.0), 1)),                                 # a chunk of the token itself
    ("attention_2", 48, convolved(4, 2, 16, 24, rot(12, 10000.0), 4)),
    ("attention_2", 24, convolved(2, 2, 16, 16, rot(16, 20.0), 1)),                               # one tap: nothing to keep
    ("attention_2", 40, convolved(6, 1, 12, 8, rot(2, 100.0), 9, scale=0.5)),
    ("lightning", 48, lightning(16, 24, 0.5, 1.0, 0.93)),
    ("lightning", 32, lightning(20, 6, 0.0, 0.99)),
    ("lightning", 40, lightning(3, 40, 0.9)),
]


@pytest.mark.parametrize("kind,W,m", MIXERS)
def test_mixer_alone(ops, kind, W, m):
    parts.check_mixer(kind, ops, "cpu", F32, W, m, (1, 2, 21, 61), seed=3)


@pytest.mark.parametrize("f", [dense(24), moe(16, 6, 2), moe(24, 4, 1), moe(8, 5, 5), moe(8, 1, 1)])
def test_feed_forward_alone(ops, f):
    parts.check_mlp(ops, "cpu", F32, 32, f, 17, seed=11)


@pytest.mark.parametrize("times", [1, 3])
def test_join_alone(ops, times):
    parts.check_join(ops, "cpu", F32, 20, 9, times=times)


@pytest.mark.parametrize("kind,m", [("attention", attention(2, 1, 8, 8, rot(4, 50.0), None, 1.0)), ("attention_2", convolved(2, 1, 8, 8, rot(4, 50.0), 3, 0.3))])
def test_one_far_key_among_hundreds(ops, kind, m):
    """One position holds the key every head answers to: seen from hundreds of tokens on."""
    w, h = parts.loud_key(kind, 16, m, 320, 5, seed=1)
    want = parts.check_mixer(kind, ops, "cpu", F32, 16, m, None, weights=w, hs=[h], ways=("whole", "decode", (0.5, 0.5)))
    assert parts.far_effect(kind, 16, m, w, h, 5, want)[-1] > 0.05


@pytest.mark.parametrize("size", [7, 8, 9])
@pytest.mark.parametrize("loud", [21, 24, 27])
def test_the_chunks_edge(ops, size, loud):
    """A loud key shows up to the last position of its chunk and not behind it (pages of 8)."""
    m = attention(2, 1, 8, 8, rot(4, 50.0), size, 1.0)
    w, h = parts.loud_key("attention", 16, m, 44, loud, seed=2)
    want = parts.check_mixer("attention", ops, "cpu", F32, 16, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 2), (0.3, 0.7)))
    diff = parts.far_effect("attention", 16, m, w, h, loud, want)
    end = loud - loud % size + size
    assert diff[loud:end].min() > 0.05 and diff[end:].max() < 1e-9


def test_a_far_token_through_the_state(ops):
    """A decay close to one: what the first token wrote still shows 300 tokens later."""
    m = lightning(16, 16, 0.999, 0.5)
    w = parts.mixer_weights("lightning", 16, m, 4)
    h = 0.3 * parts.rand(300, 16, seed=8)
    h[0] = 4.0 * parts.rand(16, seed=9)
    want = parts.check_mixer("lightning", ops, "cpu", F32, 16, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 2)))
    h2 = h.clone()
    h2[0] = -h2[0]
    other = plain.lightning(h2.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    assert (want[-1] - other[-1]).abs().max() > 1e-2, "the first token does not show"


# ---------------------------------------------------------------- the engine
@pytest.mark.parametrize("case", sorted(CASES))
@pytest.mark.parametrize("schedule", ["whole", "tail", "portions", "mixed"])
def test_schedules_against_the_plain_model(folders, case, schedule):
    hf, _ = CASES[case]
    reqs = requests_for(hf["vocab"], (1, 2, 23, 41), seed=7)
    steps, max_tokens = getattr(schedules, schedule)(reqs)
    outputs, rp = replay(folders[case], steps, max_tokens)
    got = schedules.collect(steps, outputs)
    for rid, toks in reqs.items():
        close(got[rid], plain_logits(folders[case], toks), f"{case} {schedule} {rid}", rounding_error(folders[case], toks))


def test_the_stream_after_every_layer(folders):
    """The residual stream of the engine after every run of a layer against the plain model's."""
    from paged_llm_b200.engine.replay import TraceReplayer
    from paged_llm_b200.parts.base import materialize
    for case in ("A", "B"):
        cfg, w = read_folder(folders[case])
        toks = requests_for(cfg["vocab"], (29,), seed=2)["r0"]
        rp = TraceReplayer(folders[case], "float32", 64, device="cpu", ops=TorchOps(), block_size=8, max_num_seqs=2)
        seen = []
        for blk in rp.model.blocks:
            def wrap(f):
                def g(x, pending, ctx, cache):
                    x, p = f(x, pending, ctx, cache)
                    p = materialize(p, ctx.ops)
                    seen.append((x + p.float()).clone())
                    return x, p
                return g
            blk.forward = wrap(blk.forward)
        rp.step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": [0]}], "end": ["a"]})
        with torch.no_grad():
            after = plain.forward(cfg, w, toks)[1]
        assert len(seen) == len(after)
        for i, s in enumerate(seen):
            assert (s.double() - after[i]).abs().max() < 2e-5 * max(1.0, float(after[i].abs().max())), f"{case}: run {i}"


def test_state_does_not_leak_between_requests(folders):
    """Two live requests in two slots, then a third that takes over a freed slot and freed pages: each matches its plain run."""
    hf, _ = CASES["A"]
    reqs = requests_for(hf["vocab"], (17, 9, 13), seed=3)
    a, b, c = reqs["r0"], reqs["r1"], reqs["r2"]
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:10], "want": list(range(10))}, {"id": "b", "tokens": b[:4], "want": list(range(4))}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[4:], "want": list(range(5))}], "end": ["b"]},           # a sits out
        {"step": 2, "entries": [{"id": "a", "tokens": a[10:12], "want": [0, 1]}, {"id": "c", "tokens": c[:2], "want": [0, 1]}], "end": []},
        {"step": 3, "entries": [{"id": "c", "tokens": c[2:], "want": list(range(11))}, {"id": "a", "tokens": a[12:], "want": list(range(5))}],
         "end": ["a", "c"]},
    ]
    outputs, _ = replay(folders["A"], steps, 128, slots=2)
    got = schedules.collect(steps, outputs)
    for rid, toks in (("a", a), ("b", b), ("c", c)):
        close(got[rid], plain_logits(folders["A"], toks), rid)


@pytest.mark.parametrize("seed", range(8))
def test_generated_configurations(tmp_path, seed):
    hf = generated_case(100 + seed)
    folder = make_folder(tmp_path, hf, 200 + seed)
    reqs = requests_for(hf["vocab"], (2, 19, 33), seed=seed)
    steps, max_tokens = schedules.mixed(reqs, live=3, seed=seed)
    outputs, _ = replay(folder, steps, max_tokens, slots=3)
    got = schedules.collect(steps, outputs)
    for rid, toks in reqs.items():
        close(got[rid], plain_logits(folder, toks), f"seed {seed} {rid}", rounding_error(folder, toks))


def _engine(folder, **kw):
    from paged_llm_b200 import LLMEngine
    return LLMEngine(folder, dtype="float32", device="cpu", ops=TorchOps(), block_size=8, max_model_len=96, **kw)


@pytest.mark.parametrize("case", ["A", "B"])
def test_greedy_generation_through_the_engine(folders, case):
    from paged_llm_b200 import SamplingParams
    hf, _ = CASES[case]
    prompts = list(requests_for(hf["vocab"], (3, 11, 26), seed=5).values())
    eng = _engine(folders[case], num_gpu_blocks=40, max_num_seqs=4, max_num_batched_tokens=16)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6))
    for p, o in zip(prompts, outs):
        assert o.token_ids == plain_greedy(folders[case], p, 6)


def test_generation_under_preemption(folders):
    """So few pages that requests are preempted and start again, their state slots zeroed anew."""
    from paged_llm_b200 import SamplingParams
    prompts = list(requests_for(CASE_B["vocab"], (14, 15, 13), seed=6).values())
    eng = _engine(folders["B"], num_gpu_blocks=7, max_num_seqs=3, max_num_batched_tokens=32)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10))
    assert sum(o.num_preemptions for o in outs) > 0, "the pool was meant to run out"
    for p, o in zip(prompts, outs):
        assert o.token_ids == plain_greedy(folders["B"], p, 10)


def test_random_weights_mode(tmp_path):
    """A folder written by the random-weights mode loads and runs."""
    from paged_llm_b200.weights.random_init import write_model_folder
    arch, cfg = parse_model_config(CASE_A)
    folder = write_model_folder(str(tmp_path), cfg, seed=1, std=0.1, norm_std=0.1)
    outputs, _ = replay(folder, *schedules.whole({"r": [1, 2, 3, 4, 5]}))
    assert np.isfinite(outputs[0]).all()
