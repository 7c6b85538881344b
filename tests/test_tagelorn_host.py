"""The Tagelorn decoder on the host: configuration, the model as data, the cache's needs, each mechanism by hand and alone
and the engine's host logic (runner, cache manager, state slots, replay, scheduler) with the kernel library replaced by the
tensor-code stand-in, against the plain implementation."""

from __future__ import annotations

import copy
import math
import types

import numpy as np
import pytest
import torch

from paged_llm_b200.cache.manager import CacheManager, GroupSpec
from paged_llm_b200.config.model import ConfigError
from paged_llm_b200.config.registry import parse_model_config
from paged_llm_b200.config.sampling import SamplingParams
from paged_llm_b200.config.tagelorn import TagelornConfig
from paged_llm_b200.engine.sequence import NO_PAGE, Sequence
from paged_llm_b200.kernels.plan import plan_attention, visible_keys
from paged_llm_b200.models.causal_lm import build_model
from paged_llm_b200.parts.base import FixedState, PagedKV
from tests import plain_tagelorn as plain
from tests import schedules
from tests import tagelorn_parts as parts
from tests.helpers import requests_for
from tests.tagelorn_cases import (CASE_A, CASE_B, CASES, attention, case_folder, delta, generated_case, make_folder, moe, plain_greedy,
                                  plain_logits, read_folder, rounding_error)
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
        assert arch.name == "Tagelorn"
        assert TagelornConfig.from_hf_dict(cfg.to_hf_dict()) == cfg
        back = cfg.to_hf_dict()
        back.pop("torch_dtype")
        assert back == hf
        specs = build_model(arch.build_spec(cfg)).tensor_specs()
        assert cfg.num_parameters == sum(int(np.prod(s.draw_shape or s.shape)) for s in specs.values() if not s.optional)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "not implemented"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(bias_max=1), "bias_max"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"].update(dim=0), "dim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "dense and moe only"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["canon"].update(taps=0), "taps"),
    (lambda c: c["token_side"].pop("dim"), "dim"),
    (lambda c: c.update(logit_softcap=0.0), "softcap"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("width"), "width"),
])
def test_configuration_refusals(change, message):
    hf = copy.deepcopy(CASE_A)
    change(hf)
    with pytest.raises(ConfigError, match=message):
        parse_model_config(hf)


def test_the_model_as_data():
    """Case A: every mixer keeps the last three inputs of its convolution; attention caches heads padded to the larger of key
    and value size, with its window and kept tokens; the head is the embedding; a layer has no feed-forward."""
    arch, cfg = parse_model_config(CASE_A)
    model = build_model(arch.build_spec(cfg))
    conv = FixedState((3 * 64,))
    assert [s.requirement for s in model.cache_slots()] == [
        (conv, FixedState((3 * 16 * 16,))),
        (conv, PagedKV(2, 32, 9, keep_first=3)),                                       # 16 and 24 -> 32
        (conv, PagedKV(2, 32, 24)),
        (conv, FixedState((2 * 8 * 8,))),
    ]
    specs = model.tensor_specs()
    assert {"embed", "side.embed", "final.norm", "l1.mix.q.b", "l1.mix.rel", "l2.mix.sink", "l0.mix.w1", "l0.mix.a.b", "l0.canon1",
            "l0.mlp.correction", "l0.mlp.e5.down", "l0.mlp.shared.up", "l3.side.norm"} <= set(specs)
    assert specs["head"].optional and specs["side.embed"].shape == (131, 4 * 12)
    assert not any(n.startswith(("l2.mlp", "l2.norm2")) for n in specs), "a layer without a feed-forward"
    assert not any(n.endswith((".gate", "q.norm", "k.norm")) for n in specs if n.startswith(("l0.mlp", "l1.mix")))
    assert model.has_fixed_state
    # one tap leaves nothing to keep: a model of attention alone then has no state of fixed size
    hf = copy.deepcopy(CASE_A)
    hf["canon"]["taps"] = 1
    hf["layers"] = hf["layers"][1:3]
    arch, cfg = parse_model_config(hf)
    assert not build_model(arch.build_spec(cfg)).has_fixed_state


# ---------------------------------------------------------------- the cache: first pages stay beside a window
def test_kept_pages_stay_and_the_gap_is_given_back():
    cm = CacheManager([GroupSpec(32, window=6, keep_first=5), GroupSpec(32, window=6), GroupSpec(32)], 4)
    seq = Sequence(list(range(40)), SamplingParams())
    assert cm.allocate_slots(seq, 40) is not None
    seq.num_computed_tokens = 21
    # the next query (position 21) sees 16..21 and the first five: pages 2 and 3 go, pages 0 and 1 hold kept tokens
    assert cm.release_behind_window(seq) == 2 + 4
    kept, plain_window, everything = seq.block_tables
    assert [p == NO_PAGE for p in kept[:5]] == [False, False, True, True, False]
    assert [p == NO_PAGE for p in plain_window[:5]] == [True, True, True, True, False]
    assert NO_PAGE not in everything
    seq.num_computed_tokens = 22                                  # position 22 sees 17..: page 4 (16..19) stays
    assert cm.release_behind_window(seq) == 0
    seq.num_computed_tokens = 25                                  # position 25 sees 20..: page 4 goes in both
    assert cm.release_behind_window(seq) == 2
    cm.check_invariants([seq])
    cm.free(seq)
    cm.check_invariants([])
    assert all(cm.num_free_in_group(g) == 32 for g in range(3))


def test_planned_keys_count_the_kept_tokens():
    assert visible_keys(100, 101, 10, None, 4) == 10 + 4
    assert visible_keys(3, 4, 10, None, 4) == 4
    assert visible_keys(12, 15, 10, None, 4) == 12 + 3             # keys 3..14 and 0..2
    assert visible_keys(100, 101, None, None, 4) == 101
    plan = plan_attention([1], [3000], 2, 1, 512, small_rows=16, large_rows=64, min_split_keys=128, num_sms=148, keep_first=640)
    assert len(plan["small"]) // 4 == -(-(512 + 640) // 128)


# ---------------------------------------------------------------- mechanisms by hand
def test_buckets_by_hand():
    """Eight rows, farthest distance 64: 0..3 have a row each; 4 -> 4, then every factor of two a row: 8 -> 5, 16 -> 6,
    32 -> 7, and everything beyond stays there."""
    assert [plain.bias_bucket(n, 8, 64) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]


def test_window_and_kept_tokens_by_hand(ops):
    """Scores all zero, no bias, no sink to speak of (e^-40): every visible key weighs the same.  Window 3 beside two kept
    tokens; values are the position itself, so the output is the mean of the visible positions."""
    W, m = 4, attention(1, 1, 2, 2, 50, (3, 2), scale=1.0)
    w = parts.attention_weights(W, m, seed=1)
    for name in ("a.q", "a.k", "a.q.b", "a.k.b", "a.v.b", "a.rel"):
        w[name][:] = 0.0
    w["a.sink"][:] = -40.0
    w["a.v"] = torch.tensor([[1.0, 0, 0, 0], [0, 0, 0, 0]])
    w["a.o"] = torch.tensor([[1.0, 0], [0, 0], [0, 0], [0, 0]])
    h = torch.zeros(9, W)
    h[:, 0] = torch.arange(9.0)
    seen = [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 3, 4, 5], [0, 1, 4, 5, 6], [0, 1, 5, 6, 7], [0, 1, 6, 7, 8]]
    want = torch.tensor([sum(s) / len(s) for s in seen], dtype=torch.float64)
    got = plain.attention(h.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    assert (got[:, 0] - want).abs().max() < 1e-9
    part = parts.attention_part(W, m, w, 1e-5, F32, "cpu")
    for out in parts.run_mixer(ops, "cpu", part, [h], F32, ps=2, ways=("whole", "decode", ("every", 2))):
        assert (out[:, 0].double() - want).abs().max() < 1e-5


def test_a_kept_token_keeps_its_distance(ops):
    """The bias of a kept token is the one of its true distance, far beyond the window: position 0 under a table whose far
    rows are loud."""
    W, m = 4, attention(1, 1, 2, 2, 16, (2, 1), scale=1.0)
    w = parts.attention_weights(W, m, seed=1, rows=4)
    for name in ("a.q", "a.k", "a.q.b", "a.k.b", "a.v.b"):
        w[name][:] = 0.0
    w["a.rel"] = torch.tensor([[0.0], [0.0], [1.0], [3.0]])                          # rows for 0, 1, 2..5, 6..
    w["a.sink"][:] = -40.0
    w["a.v"] = torch.tensor([[1.0, 0, 0, 0], [0, 0, 0, 0]])
    w["a.o"] = torch.tensor([[1.0, 0], [0, 0], [0, 0], [0, 0]])
    h = torch.zeros(12, W)
    h[0, 0] = 1.0                                                                     # only position 0 has a value
    want = [1.0, 0.5]
    for i in range(2, 12):
        row = min(3, 2 + math.floor(math.log(i / 2) / math.log(16 / 2) * 2))
        e = math.exp([0, 0, 1.0, 3.0][row])
        want.append(e / (e + 2.0))
    got = plain.attention(h.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    assert np.allclose(got[:, 0].numpy(), want, atol=1e-9)
    part = parts.attention_part(W, m, w, 1e-5, F32, "cpu")
    for out in parts.run_mixer(ops, "cpu", part, [h], F32, ps=2, ways=("whole", "decode", ("every", 2))):
        assert np.allclose(out[:, 0].numpy(), want, atol=1e-5)


def test_unit_heads_by_hand():
    """q and k are divided by their root mean square over the head: scaling a head's projection changes nothing."""
    W, m = 16, attention(4, 2, 8, 8, 40, (6, 2))
    w = {k: v.double() for k, v in parts.attention_weights(W, m, seed=4).items()}
    h = parts.rand(11, W, seed=5).double()
    a = plain.attention(h, w, "a.", m, 1e-12)
    w2 = dict(w)
    for name, rows in (("a.q", slice(8, 16)), ("a.k", slice(0, 8))):
        for t in (name, name + ".b"):
            w2[t] = w2[t].clone()
            w2[t][rows] *= 7.0
    assert (plain.attention(h, w2, "a.", m, 1e-12) - a).abs().max() < 1e-9


def test_delta_rule_by_hand(ops):
    """One head of one channel: u = k / |k| = +-1, so S <- w S - a S + k v and o = S r; the norm over one value."""
    W, m = 3, delta(1, 1)
    w = parts.delta_weights(W, m, seed=0, rank=1)
    w.update({"d.r": torch.tensor([[0.0, 0, 1.0]]), "d.k": torch.tensor([[1.0, 0, 0]]), "d.v": torch.tensor([[0, 1.0, 0]]),
              "d.g": torch.tensor([[0, 0, 1.0]]), "d.a": torch.tensor([[0, 1.0, 0]]), "d.a.b": torch.tensor([0.5]),
              "d.w1": torch.tensor([[1.0, 0, 0]]), "d.w2": torch.tensor([[2.0]]), "d.w0": torch.tensor([-0.25]),
              "d.norm": torch.tensor([1.5]), "d.o": torch.tensor([[1.0], [0], [0]])})
    h = torch.tensor([[2.0, 1.0, 0.5], [-1.0, 3.0, -0.5], [0.5, -2.0, 1.0]])
    sig = lambda z: 1 / (1 + math.exp(-z))      # noqa: E731
    eps, S, want = 1e-3, 0.0, []
    for a, b, c in h.tolist():
        decay = math.exp(-math.exp(-0.5) * sig(2.0 * math.tanh(a) - 0.25))
        u = a / math.sqrt(a * a + 1e-6)
        S = decay * S - sig(b + 0.5) * u * (u * S) + a * b
        o = S * c
        want.append(o / math.sqrt(o * o + eps) * 1.5 * sig(c))
    got = plain.general_delta(h.double(), {k: v.double() for k, v in w.items()}, "d.", m, eps)
    assert np.allclose(got[:, 0].numpy(), want, rtol=1e-9)
    part = parts.delta_part(W, m, w, eps, F32, "cpu")
    for out in parts.run_mixer(ops, "cpu", part, [h], F32, ways=("whole", "decode")):
        assert np.allclose(out[:, 0].numpy(), want, rtol=1e-5)


def test_router_by_hand(ops):
    """Six experts in three groups of two, two groups stay, two experts are chosen.  Softmax scores 0.30 0.05 | 0.20 0.15 |
    0.25 0.05 with corrections 0 0 | 0.2 0 | -0.2 -0.3: choice scores 0.30 0.05 | 0.40 0.15 | 0.05 -0.25, the largest of each
    group 0.30, 0.40, 0.05 -> the first two stay; experts 2 and 0 are chosen and weigh 0.20 and 0.30 over their sum, times 3."""
    s = torch.tensor([0.30, 0.05, 0.20, 0.15, 0.25, 0.05], dtype=torch.float64)
    corr = torch.tensor([0.0, 0.0, 0.2, 0.0, -0.2, -0.3], dtype=torch.float64)
    r = {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 2}}
    one = torch.ones(1, 1, dtype=torch.float64)
    idx, wt = plain.router(one, torch.log(s)[:, None], corr, r)
    assert idx[0].tolist() == [2, 0] and np.allclose(wt[0].tolist(), [1.2, 1.8])
    # without the groups expert 4 still loses by its correction; without the correction it would be chosen
    assert sorted(plain.router(one, torch.log(s)[:, None], corr, {"experts": 6, "top": 2, "scale": 1.0})[0][0].tolist()) == [0, 2]
    assert sorted(plain.router(one, torch.log(s)[:, None], 0 * corr, {"experts": 6, "top": 2, "scale": 1.0})[0][0].tolist()) == [0, 4]
    # a single group whose choice scores are all negative: the excluded groups' experts are never taken instead
    low = torch.tensor([-2.0, -2.1, -3.0, -3.0, -3.0, -3.0], dtype=torch.float64)
    assert sorted(plain.router(one, torch.log(s)[:, None], low, {"experts": 6, "top": 2, "scale": 1.0, "groups": {"count": 3, "keep": 1}})[0][0].tolist()) == [0, 1]
    # the same through the part
    W, mlp = 8, moe(8, 6, 2, 3.0, (3, 2), shared=4)
    w = parts.experts_weights(W, mlp, seed=2)
    w["m.router"] = torch.zeros(6, W)
    w["m.router"][:, 0] = torch.log(s).float()
    w["m.correction"] = corr.float()
    h = torch.zeros(1, W)
    h[0, 0] = 1.0
    got = parts.experts_part(W, mlp, w, F32, "cpu").forward(h, types.SimpleNamespace(ops=ops)).double()
    wd = {k: v.double() for k, v in w.items()}
    want = 1.2 * plain.expert(h.double(), wd, "m.e2.") + 1.8 * plain.expert(h.double(), wd, "m.e0.") + plain.expert(h.double(), wd, "m.shared.")
    assert (got - want).abs().max() < 1e-5


def test_input_convolution_by_hand():
    h = torch.tensor([[1.0], [2.0], [4.0], [8.0]], dtype=torch.float64)
    got = plain.input_convolution(h, torch.tensor([[0.5, 10.0, 100.0]], dtype=torch.float64))
    assert got[:, 0].tolist() == [1 + 100, 2 + 200 + 10, 4 + 400 + 20 + 0.5, 8 + 800 + 40 + 1.0]


def test_sinusoids_by_hand(ops):
    s = plain.sinusoids(4, 6)
    assert s[0].tolist() == [0, 1, 0, 1, 0, 1]
    assert np.allclose(s[3, 2:4].tolist(), [math.sin(3 * 10000 ** (-1 / 3)), math.cos(3 * 10000 ** (-1 / 3))])
    parts.check_sinusoids(ops, "cpu", F32, 64, 2.0, [0, 1, 7, 1000, 123457])
    parts.check_sinusoids(ops, "cpu", F32, 7, 1.0, [0, 5, 99])


# ---------------------------------------------------------------- each mechanism alone, through prompts and decoding
@pytest.mark.parametrize("W,m,rows", [
    (48, attention(4, 2, 16, 24, 40, (9, 3)), 8),
    (32, attention(6, 1, 8, 40, 30.5, scale=0.4), 4),                    # no window
    (40, attention(3, 3, 32, 16, 100, (5, 21)), 16),                     # more kept tokens than the window holds
    (24, attention(2, 1, 16, 16, 20, (1, 1)), 8),                        # a window of the token itself
    (24, attention(2, 2, 16, 16, 20, (12, 0)), 8),
])
def test_attention_alone(ops, W, m, rows):
    parts.check_attention(ops, "cpu", F32, W, m, (1, 2, 21, 61), seed=3, rows=rows)


@pytest.mark.parametrize("W,m,rank", [(48, delta(3, 16), 5), (32, delta(2, 20), 8), (40, delta(1, 40), 1)])
def test_delta_rule_alone(ops, W, m, rank):
    parts.check_delta(ops, "cpu", F32, W, m, (1, 2, 4, 23), seed=7, rank=rank)


@pytest.mark.parametrize("W,taps,inner,m", [(32, 4, "general_delta", delta(2, 8)), (24, 2, "attention", attention(2, 1, 8, 8, 40, (5, 2))),
                                            (24, 1, "attention", attention(2, 2, 8, 8, 40)), (20, 7, "general_delta", delta(1, 12))])
def test_input_convolution_alone(ops, W, taps, inner, m):
    parts.check_input_convolution(ops, "cpu", F32, W, taps, inner, m, (1, 3, 18), seed=9)


@pytest.mark.parametrize("mlp", [moe(16, 6, 2, 1.5, (3, 2), shared=24), moe(24, 4, 1, 1.0, (1, 1)), moe(8, 5, 3, 0.5, shared=8), moe(16, 8, 4, 2.0, (4, 2))])
def test_experts_alone(ops, mlp):
    parts.check_experts(ops, "cpu", F32, 32, mlp, 24, seed=11)


@pytest.mark.parametrize("W,dim,layers,which", [(32, 12, 3, 1), (48, 8, 1, 0), (20, 5, 4, 3)])
def test_token_input_alone(ops, W, dim, layers, which):
    parts.check_token_side(ops, "cpu", F32, W, dim, layers, which, 9)


@pytest.mark.parametrize("loud,mask", [(5, None), (2, (16, 3)), (3, (16, 3))])
def test_one_far_key_among_hundreds(ops, loud, mask):
    """One position holds the key every head answers to: seen from hundreds of tokens on without a window and as a kept
    token, and not at all as the first token that is not kept."""
    W, m = 16, attention(2, 1, 8, 8, 64, mask, scale=1.0)
    w, h = parts.loud_key(W, m, 320, loud, seed=1)
    want = parts.check_attention(ops, "cpu", F32, W, m, None, weights=w, hs=[h], ways=("whole", "decode", (0.5, 0.5)))
    other = h.clone()
    other[loud, 0] = 0.0
    quiet = plain.attention(other.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    moved = (want[-1] - quiet[-1]).abs().max().item()
    assert moved < 1e-9 if loud == 3 else moved > 0.05


@pytest.mark.parametrize("size", [7, 8, 9])
def test_the_windows_edge(ops, size):
    """A loud key exactly at the last distance inside the window shows, one step later it does not (pages of 8)."""
    W, m = 16, attention(2, 1, 8, 8, 64, (size, 1), scale=1.0)
    loud = 21
    w, h = parts.loud_key(W, m, 40, loud, seed=2)
    want = parts.check_attention(ops, "cpu", F32, W, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 2), (0.3, 0.7)))
    other = h.clone()
    other[loud, 0] = 0.0
    quiet = plain.attention(other.double(), {k: v.double() for k, v in w.items()}, "a.", m, 1e-5)
    diff = (want - quiet).abs().amax(1)
    assert diff[loud + size - 1] > 0.05 and diff[loud + size:].max() < 1e-9


def test_a_far_token_through_the_delta_state(ops):
    """Decays close to one and removal rates close to zero: what the first token wrote still shows 300 tokens later."""
    W, m = 16, delta(2, 16)
    w = parts.delta_weights(W, m, seed=4, w0=-8.0)
    w["d.w2"] = w["d.w2"] * 0.1
    w["d.a"], w["d.a.b"] = w["d.a"] * 0.1, torch.full((32,), -7.0)
    h = parts.rand(300, W, seed=8)
    want = parts.check_delta(ops, "cpu", F32, W, m, None, weights=w, hs=[h], ways=("whole", "decode", ("every", 2)))
    h2 = h.clone()
    h2[0] = -3.0 * h2[0]
    other = plain.general_delta(h2.double(), {k: v.double() for k, v in w.items()}, "d.", m, 1e-5)
    assert (want[-1] - other[-1]).abs().max() > 1e-2, "the first token does not show"


# ---------------------------------------------------------------- the engine
@pytest.mark.parametrize("case", sorted(CASES))
@pytest.mark.parametrize("schedule", ["whole", "tail", "portions", "mixed"])
def test_schedules_against_the_plain_model(folders, case, schedule):
    hf, _ = CASES[case]
    reqs = requests_for(hf["vocab"], (1, 2, 23, 41, 70), seed=7)
    steps, max_tokens = getattr(schedules, schedule)(reqs)
    outputs, rp = replay(folders[case], steps, max_tokens)
    got = schedules.collect(steps, outputs)
    for rid, toks in reqs.items():
        close(got[rid], plain_logits(folders[case], toks), f"{case} {schedule} {rid}", rounding_error(folders[case], toks))


def test_pages_between_the_kept_tokens_and_the_window_are_used_again(folders):
    """Case A's window of 9 beside 3 kept tokens: a request of 70 tokens decoded in a pool of its own holds few pages of that
    group, and another request takes over what it gave back while both live."""
    from paged_llm_b200.engine.replay import TraceReplayer
    reqs = requests_for(131, (70, 33), seed=4)
    a, b = reqs["r0"], reqs["r1"]
    rp = TraceReplayer(folders["A"], "float32", 128, device="cpu", ops=TorchOps(), block_size=4, max_num_seqs=2, poison=float("nan"))
    got = {"a": [], "b": []}
    feed = [("a", a[:50])] + [("a", [t]) for t in a[50:60]] + [("b", b[:20])] + [("a", [t]) for t in a[60:]] + [("b", b[20:])]
    for i, (rid, toks) in enumerate(feed):
        got[rid].append(rp.step({"step": i, "entries": [{"id": rid, "tokens": toks, "want": list(range(len(toks)))}], "end": []}))
        if rid == "a" and i == 10:
            group = next(g for g, spec in enumerate(rp.cm.group_specs) if spec.keep_first == 3)
            held = [p for p in rp.live["a"].block_tables[group] if p != NO_PAGE]
            assert len(held) <= 1 + 3, "one page of kept tokens and those of the window"
    for rid, toks in (("a", a), ("b", b)):
        close(np.concatenate(got[rid]), plain_logits(folders["A"], toks), rid, rounding_error(folders["A"], toks))


def test_the_stream_after_every_layer(folders):
    """The residual stream of the engine after every layer against the plain model's."""
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
        for i, s in enumerate(seen):
            assert (s.double() - after[i]).abs().max() < 2e-5 * max(1.0, float(after[i].abs().max())), f"{case}: layer {i}"


def test_state_does_not_leak_between_requests(folders):
    """Two live requests in two slots, then a third that takes over a freed slot: each matches its plain run."""
    hf, _ = CASES["B"]
    reqs = requests_for(hf["vocab"], (17, 9, 13), seed=3)
    a, b, c = reqs["r0"], reqs["r1"], reqs["r2"]
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:10], "want": list(range(10))}, {"id": "b", "tokens": b[:4], "want": list(range(4))}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[4:], "want": list(range(5))}], "end": ["b"]},           # a sits out
        {"step": 2, "entries": [{"id": "a", "tokens": a[10:12], "want": [0, 1]}, {"id": "c", "tokens": c[:2], "want": [0, 1]}], "end": []},
        {"step": 3, "entries": [{"id": "c", "tokens": c[2:], "want": list(range(11))}, {"id": "a", "tokens": a[12:], "want": list(range(5))}],
         "end": ["a", "c"]},
    ]
    outputs, _ = replay(folders["B"], steps, 128, slots=2)
    got = schedules.collect(steps, outputs)
    for rid, toks in (("a", a), ("b", b), ("c", c)):
        close(got[rid], plain_logits(folders["B"], toks), rid)


@pytest.mark.parametrize("seed", range(10))
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


@pytest.mark.parametrize("case", sorted(CASES))
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
