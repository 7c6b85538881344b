"""Headline benchmark: decode tokens per second of the TinyLlama-1.1B-sized Llama
(random bfloat16 weights) at batch 8 with 512-token prompts, on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A step is one decode step.  The timed region is exactly K steps after W warm-up
steps, timed with CUDA events on the launching stream.  One JSON line is
printed; beside `value` (device-timed loop: tokens stay on the device) it holds

* `e2e`: the same through `LLMEngine.step()`: host token ids in, host token ids
  out, every step (metadata host-to-device from pinned memory, sampled ids
  device-to-host);
* `prefill`: one step of a 2,048-token prompt, with the fraction of the bf16 peak;
* `roofline`: bytes a decode step must read (weights once, the live cache)
  divided by its time, against the measured HBM bandwidth;
* `points`: decode tokens per second at batch 1 and 64;
* `clocks`: SM clock and throttle reasons sampled during the timed region;
* `gpu_launches`: kernels of this package launched in the timed region.

Weights (2.2 GB) are larger than the 126 MB L2, so every step re-reads them from
HBM; no L2 flush is needed between iterations.

`--impl reference` runs the unmodified reference (xiyiji/paged-llm, installed
under baseline/_ref) through its own `LLMEngine` on the same model folder and
prints the same line with "impl": "reference".
"""

from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}

SIZES = {
    # TinyLlama 1.1B layer sizes (22 layers, 32 query / 4 kv heads of 64, hidden 2048, context 2048)
    "tinyllama-1.1b": dict(vocab_size=32000, hidden_size=2048, intermediate_size=5632, num_hidden_layers=22,
                           num_attention_heads=32, num_key_value_heads=4, head_dim=64, rope_theta=10000.0,
                           rms_norm_eps=1e-5, tie_word_embeddings=False, max_position_embeddings=2048),
    # Llama-3.2-1B layer sizes (16 layers, 32 query / 8 kv heads of 64, llama3 rotary scaling, tied head)
    "llama-3.2-1b": dict(vocab_size=128256, hidden_size=2048, intermediate_size=8192, num_hidden_layers=16,
                         num_attention_heads=32, num_key_value_heads=8, head_dim=64, rope_theta=500000.0,
                         rope_scaling=dict(rope_type="llama3", factor=32.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                           original_max_position_embeddings=8192),
                         rms_norm_eps=1e-5, tie_word_embeddings=True, max_position_embeddings=8192),
    # Llama-3-8B layer sizes (32 layers, 32 query / 8 kv heads of 128, hidden 4096); about 16 GB at full depth
    "llama-3-8b": dict(vocab_size=128256, hidden_size=4096, intermediate_size=14336, num_hidden_layers=32,
                       num_attention_heads=32, num_key_value_heads=8, head_dim=128, rope_theta=500000.0,
                       rms_norm_eps=1e-5, tie_word_embeddings=False, max_position_embeddings=8192),
    # for trying the script out on small hardware; never the default
    "tiny-a": dict(vocab_size=256, hidden_size=64, intermediate_size=172, num_hidden_layers=2,
                   num_attention_heads=4, num_key_value_heads=2, head_dim=16, max_position_embeddings=4096),
}
# Layer sizes for `--only pomisun`: the Pomisun decoder (dense and routed-expert layers in turn, the first two run
# twice, chunked mask, score cap, YaRN) beside a Llama of the same width, heads, dense inner size and number of
# layer runs.
POMISUN_SIZES = {
    "p-2k": dict(vocab=32000, width=2048, heads=16, kv_heads=4, dim=128, ff=8192, experts=32, top=4, expert_ff=1024,
                 shared_ff=2048, chunk=1024, layers=4, loop=dict(start=0, stop=2, times=2)),
    "p-4k": dict(vocab=32000, width=4096, heads=32, kv_heads=8, dim=128, ff=14336, experts=64, top=6, expert_ff=1408,
                 shared_ff=2816, chunk=2048, layers=4, loop=None),
    # for trying the option out quickly; never a result
    "p-tiny": dict(vocab=256, width=128, heads=4, kv_heads=2, dim=32, ff=256, experts=4, top=2, expert_ff=64,
                   shared_ff=64, chunk=64, layers=2, loop=None),
}
# Layer sizes for `--only rokarax`: the Rokarax decoder (state-space layers, windowed attention with a bias by distance
# and an output gate, one of them reading the other's keys and values, and attention through latents) beside a Llama of
# the same width, heads, head size, dense inner size and number of layers.
ROKARAX_SIZES = {
    "r-2k": dict(vocab=32000, width=2048, heads=16, kv_heads=4, dim=128, ff=8192, window=1024, q_rank=768, kv_rank=192,
                 rot_dim=64, ssm_heads=64, ssm_dim=64, state=128, groups=1, conv=4),
    "r-4k": dict(vocab=32000, width=4096, heads=32, kv_heads=8, dim=128, ff=14336, window=2048, q_rank=1536, kv_rank=192,
                 rot_dim=64, ssm_heads=128, ssm_dim=64, state=128, groups=1, conv=4),
    # for trying the option out quickly; never a result
    "r-tiny": dict(vocab=256, width=128, heads=4, kv_heads=2, dim=32, ff=256, window=64, q_rank=48, kv_rank=32,
                   rot_dim=16, ssm_heads=8, ssm_dim=16, state=16, groups=2, conv=3),
}
# Munazen at the layer sizes of a 2k- and a 4k-wide model: attention beside a gated recurrence of the model's width, and
# gated linear attention with keys half and values once the model's width
MUNAZEN_SIZES = {
    "m-2k": dict(vocab=32000, width=2048, heads=16, kv_heads=4, dim=128, ff=8192, rec_width=2048, rec_blocks=16, conv=4,
                 gla_heads=8, gla_dim=128, gla_vdim=256, streams=2, norm_groups=2),
    "m-4k": dict(vocab=32000, width=4096, heads=32, kv_heads=8, dim=128, ff=14336, rec_width=4096, rec_blocks=16, conv=4,
                 gla_heads=16, gla_dim=128, gla_vdim=256, streams=4, norm_groups=4),
    # for trying the option out quickly; never a result
    "m-tiny": dict(vocab=256, width=128, heads=4, kv_heads=2, dim=32, ff=256, rec_width=96, rec_blocks=3, conv=3,
                   gla_heads=2, gla_dim=16, gla_vdim=32, streams=2, norm_groups=2),
}
# Pirerax at the layer sizes of a 2k- and a 4k-wide model: attention with a sink, latent attention, attention beside the
# gated delta rule, routed experts on every layer (the Llama beside it gets top * expert_ff as its inner size)
PIRERAX_SIZES = {
    "x-2k": dict(vocab=32000, width=2048, heads=16, kv_heads=4, dim=128, rot_dim=64, kv_rank=192, delta_heads=16, delta_kv=8,
                 delta_dim=128, delta_vdim=128, conv=4, experts=32, top=4, groups=(8, 4), expert_ff=1024),
    "x-4k": dict(vocab=32000, width=4096, heads=32, kv_heads=8, dim=128, rot_dim=64, kv_rank=192, delta_heads=32, delta_kv=16,
                 delta_dim=128, delta_vdim=128, conv=4, experts=64, top=6, groups=(8, 4), expert_ff=1408),
    # for trying the option out quickly; never a result
    "x-tiny": dict(vocab=256, width=128, heads=4, kv_heads=2, dim=32, rot_dim=16, kv_rank=32, delta_heads=4, delta_kv=2,
                   delta_dim=16, delta_vdim=32, conv=3, experts=8, top=2, groups=(4, 2), expert_ff=64),
}
# Tagelorn at the layer sizes of a 2k- and a 4k-wide model: windowed attention with kept tokens, a bias table and a sink, the
# generalized delta rule, routed experts of one matrix in front of the activation beside a shared one (the Pirerax beside it
# gets the same widths, heads, delta-rule heads and experts)
TAGELORN_SIZES = {
    "t-2k": dict(vocab=32000, width=2048, heads=16, kv_heads=4, dim=128, window=1024, keep_first=4, delta_heads=16, delta_dim=128,
                 ff=8192, experts=32, top=4, groups=(8, 4), expert_ff=1024, shared_ff=1024, taps=3, side_dim=128),
    "t-4k": dict(vocab=32000, width=4096, heads=32, kv_heads=8, dim=128, window=1024, keep_first=4, delta_heads=32, delta_dim=128,
                 ff=14336, experts=64, top=6, groups=(8, 4), expert_ff=1408, shared_ff=1408, taps=3, side_dim=256),
    # heads of 64 in both mixers
    "t-2k-64": dict(vocab=32000, width=2048, heads=32, kv_heads=8, dim=64, window=1024, keep_first=4, delta_heads=32, delta_dim=64,
                    ff=8192, experts=32, top=4, groups=(8, 4), expert_ff=1024, shared_ff=1024, taps=3, side_dim=128),
    # for trying the option out quickly; never a result
    "t-tiny": dict(vocab=256, width=128, heads=4, kv_heads=2, dim=32, window=64, keep_first=4, delta_heads=4, delta_dim=16, ff=256,
                   experts=8, top=2, groups=(4, 2), expert_ff=64, shared_ff=64, taps=3, side_dim=24),
}
# Nopozen at the layer sizes of a 2k- and a 4k-wide model: chunked attention, linear attention with a fixed decay, convolved
# attention; the first feed-forward dense, the others routed experts; layers 1 to 3 run twice.  The Pomisun beside it gets the
# same widths, heads, chunk, experts and loop (attention only); the Munazen the same widths, heads and linear-attention heads
# (its linear attention has a decay per channel), as many layers as the Nopozen has runs, and top * expert_ff as inner size
NOPOZEN_SIZES = {
    "n-2k": dict(vocab=32000, width=2048, heads=16, kv_heads=4, dim=128, chunk=1024, lin_heads=16, lin_dim=128, taps=3, ff=8192,
                 experts=32, top=4, expert_ff=1024, rec_blocks=16),
    "n-4k": dict(vocab=32000, width=4096, heads=32, kv_heads=8, dim=128, chunk=1024, lin_heads=32, lin_dim=128, taps=3, ff=14336,
                 experts=64, top=6, expert_ff=1408, rec_blocks=16),
    # heads of 64 in every mixer
    "n-2k-64": dict(vocab=32000, width=2048, heads=32, kv_heads=8, dim=64, chunk=1024, lin_heads=32, lin_dim=64, taps=3, ff=8192,
                    experts=32, top=4, expert_ff=1024, rec_blocks=16),
    # for trying the option out quickly; never a result
    "n-tiny": dict(vocab=256, width=128, heads=4, kv_heads=2, dim=32, chunk=64, lin_heads=4, lin_dim=16, taps=3, ff=256, experts=8,
                   top=2, expert_ff=64, rec_blocks=4),
}
PROMPT_LEN, DECODE_LEN, PREFILL_TOKENS, BLOCK_SIZE = 512, 256, 2048, 16
RAGGED_PROMPTS, RAGGED_OUTPUTS = (128, 4096), (64, 512)      # the ragged serving workload: lengths drawn uniformly


def load_peaks() -> dict:
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                raw = json.load(f)
            flat = {}

            def walk(d):
                for k, v in d.items():
                    if isinstance(v, dict):
                        walk(v)
                    elif isinstance(v, (int, float)):
                        flat.setdefault(k, float(v))
            walk(raw)
            out = {"source": "measured"}
            out["hbm_gbs"] = flat.get("hbm_gbs") or FALLBACK_PEAKS["hbm_gbs"]
            out["bf16_tflops"] = flat.get("bf16_tflops") or FALLBACK_PEAKS["bf16_tflops"]
            if "bf16_tflops_sustained" in flat:
                out["bf16_tflops_sustained"] = flat["bf16_tflops_sustained"]
            return out
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """nvidia-smi in a loop during the timed region (reads settings, changes none)."""

    QUERY = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self, device_index: int = 0):
        self.proc = None
        self.path = None
        self.uuid = None
        try:
            import torch
            self.uuid = "GPU-" + str(torch.cuda.get_device_properties(device_index).uuid)
        except Exception:
            self.uuid = None

    def __enter__(self):
        try:
            fd, self.path = tempfile.mkstemp(suffix=".csv")
            os.close(fd)
            cmd = ["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100"]
            if self.uuid:
                cmd += ["-i", self.uuid]
            self.proc = subprocess.Popen(cmd, stdout=open(self.path, "w"), stderr=subprocess.DEVNULL)
        except OSError:
            self.proc = None
        return self

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self) -> dict:
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        try:
            with open(self.path) as f:
                for line in f:
                    parts = [p.strip() for p in line.split(",")]
                    if len(parts) < 7:
                        continue
                    try:
                        sm.append(float(parts[0]))
                        mx.append(float(parts[1]))
                    except ValueError:
                        continue
                    for name, flag in zip(names, parts[3:7]):
                        if flag.lower().startswith("active"):
                            reasons.add(name)
            os.unlink(self.path)
        except (OSError, TypeError):
            pass
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "reasons": sorted(reasons), "samples": len(sm)}


def write_tokenizer(folder: str, vocab: int) -> None:
    """A word-level tokenizer over token names t0..tN, only so that the
    reference's engine, which loads a tokenizer unconditionally, starts."""
    from tokenizers import Tokenizer, models, pre_tokenizers

    tok = Tokenizer(models.WordLevel({f"t{i}": i for i in range(vocab)}, unk_token="t0"))
    tok.pre_tokenizer = pre_tokenizers.Whitespace()
    tok.save(os.path.join(folder, "tokenizer.json"))
    with open(os.path.join(folder, "tokenizer_config.json"), "w") as f:
        json.dump({"tokenizer_class": "PreTrainedTokenizerFast", "unk_token": "t0", "eos_token": "t1"}, f)


STUB_ABOVE_PARAMS = 2_000_000_000      # larger models get their random weights drawn on the device


def make_model(folder: str, size: str, layers: int | None, with_tokenizer: bool = False, on_device: bool | None = None):
    """Writes a model folder of the named layer sizes with random weights N(0, 0.02), seed 0.  Models of
    more than two billion parameters (or `on_device`) get a folder without tensors whose weights the
    engine draws on the device (weights/random_init.py: write_random_stub); the reference arm always
    gets tensors."""
    from paged_llm_b200.config.registry import parse_model_config
    from paged_llm_b200.weights import write_model_folder, write_random_stub

    hf = {"architectures": ["LlamaForCausalLM"], **SIZES[size]}
    full_layers = hf["num_hidden_layers"]
    if layers:
        hf["num_hidden_layers"] = layers
    _, cfg = parse_model_config(hf)          # the architecture named in the configuration decides the config class
    if on_device is None:
        on_device = cfg.num_parameters > STUB_ABOVE_PARAMS and not with_tokenizer
    if on_device:
        write_random_stub(folder, cfg, seed=0, std=0.02, dtype="bfloat16")
    else:
        write_model_folder(folder, cfg, seed=0, std=0.02, dtype="bfloat16")
    if with_tokenizer:
        write_tokenizer(folder, cfg.vocab_size)
    return cfg, full_layers


def prompts_for(vocab: int, batch: int, length: int, seed: int = 0):
    import torch
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (length,), generator=g).tolist() for _ in range(batch)]


def step_flops(cfg, tokens: int, context_start: int = 0) -> float:
    """Multiply-adds x 2 of one step of `tokens` new tokens of one request."""
    h, d = cfg.hidden_size, cfg.head_dim
    per_layer = (cfg.num_attention_heads + 2 * cfg.num_key_value_heads) * d * h + cfg.num_attention_heads * d * h \
        + 3 * cfg.intermediate_size * h
    gemm = 2.0 * tokens * per_layer * cfg.num_hidden_layers + 2.0 * cfg.vocab_size * h
    keys = sum(context_start + i + 1 for i in range(tokens))
    attn = 4.0 * cfg.num_attention_heads * d * keys * cfg.num_hidden_layers
    return gemm + attn


# ------------------------------------------------------------------------------ ours

def device_decode_loop(engine, batch: int, steps: int, warmup: int, prompt_len: int):
    """Prefills `batch` requests, then times `steps` decode steps on the device:
    sampled tokens stay on the device and feed the next step.  Returns
    (ms per step, launches per step, context length at the middle of the run)."""
    import torch
    from paged_llm_b200.config import SamplingParams
    from paged_llm_b200.engine.runner import StepItem
    from paged_llm_b200.engine.sequence import Sequence

    cm, runner, ops = engine.block_manager, engine.runner, engine.ops
    vocab = engine.model_config.vocab_size
    seqs = [Sequence(p, SamplingParams(temperature=0.0, max_tokens=steps + warmup + 2))
            for p in prompts_for(vocab, batch, prompt_len, seed=batch)]
    for s in seqs:
        assert cm.acquire_state_slot(s), "too few state slots for the benchmark"      # (models with state of fixed size)
    chunk = max(1, engine.config.max_num_batched_tokens // prompt_len)
    for i in range(0, batch, chunk):
        group = seqs[i:i + chunk]
        for s in group:
            ok = cm.allocate_slots(s, prompt_len)
            assert ok is not None, "pool too small for the benchmark"
        logits = runner.step([StepItem(s, prompt_len, (prompt_len - 1,)) for s in group])
        toks = ops.argmax(logits).tolist()
        for s, t in zip(group, toks):
            s.num_computed_tokens = prompt_len
            s.append_token(t)
    items = [StepItem(s, 1, (0,)) for s in seqs]

    def one_step(first: bool):
        for s in seqs:
            ok = cm.allocate_slots(s, 1)
            assert ok is not None, "pool too small for the benchmark"
        logits = runner.step(items)
        nxt = ops.argmax(logits)
        for s in seqs:
            s.num_computed_tokens += 1
            s.token_ids.append(0)            # the id lives on the device; the host list only keeps the length
        return nxt

    # device-resident feedback: the ids section of the next step's metadata is overwritten on the device
    def run(n):
        nonlocal last
        for _ in range(n):
            if last is not None:
                runner.next_ids_override = last
            last = one_step(False)

    last = None
    run(warmup)
    torch.cuda.synchronize()
    launches0 = ops.launches + runner.graph_launches
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    ctx_mid = seqs[0].num_computed_tokens + steps // 2
    start.record()
    run(steps)
    end.record()
    torch.cuda.synchronize()
    ms = start.elapsed_time(end) / steps
    launches = (ops.launches + runner.graph_launches - launches0) / steps
    for s in seqs:
        cm.free(s)
    return ms, launches, ctx_mid


def decode_kernel_times(engine, batch: int, steps: int, warmup: int, prompt_len: int) -> dict:
    """Device time of every kernel inside replayed decode steps (torch's profiler, i.e. CUPTI activity
    records of the real step, not serialised launches): name -> [launches per step, mean microseconds].
    Kernels launched with programmatic dependent launch overlap, so the sum can exceed the step."""
    import collections
    import torch
    from torch.profiler import ProfilerActivity, profile

    device_decode_loop(engine, batch, steps, warmup, prompt_len)            # graphs captured, caches warm
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        _, launches, _ = device_decode_loop(engine, batch, steps, warmup, prompt_len)
        torch.cuda.synchronize()
    events = sorted((e for e in prof.events() if e.device_type == torch.autograd.DeviceType.CUDA),
                    key=lambda e: e.time_range.start)
    # the decode steps are the tail of the record: per step the package's kernels, the library's, and two copies
    per_step = collections.Counter()
    tail = events[-int(round(launches + 4)) * steps:]
    total = collections.defaultdict(float)
    for e in tail:
        name = e.name.replace("(anonymous namespace)::", "").replace("<unnamed>::", "").replace("void ", "")
        name = name.split("(")[0][:72]
        per_step[name] += 1
        total[name] += e.time_range.end - e.time_range.start
    return {k: [round(per_step[k] / steps, 1), round(total[k] / per_step[k], 2)]
            for k in sorted(total, key=lambda k: -total[k])[:24]}


def prefill_kernel_times(engine, tokens: int) -> dict:
    """The same for one prompt portion of `tokens` tokens: name -> [launches in the step, mean microseconds]."""
    import collections
    import torch
    from torch.profiler import ProfilerActivity, profile

    prefill_once(engine, tokens, iters=1, warmup=3)                          # graph captured, caches warm
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        prefill_once(engine, tokens, iters=1, warmup=0)
        torch.cuda.synchronize()
    count, total = collections.Counter(), collections.defaultdict(float)
    for e in prof.events():
        if e.device_type != torch.autograd.DeviceType.CUDA:
            continue
        name = e.name.replace("(anonymous namespace)::", "").replace("<unnamed>::", "").replace("void ", "")
        name = name.split("(")[0][:72]
        count[name] += 1
        total[name] += e.time_range.end - e.time_range.start
    return {k: [count[k], round(total[k] / count[k], 2)] for k in sorted(total, key=lambda k: -total[k])[:24]}


def e2e_decode(engine, batch: int, steps: int, warmup: int, prompt_len: int):
    """The same decode steps through the public `LLMEngine.step()`: token ids
    come back to the host every step."""
    import torch
    from paged_llm_b200.config import SamplingParams

    vocab = engine.model_config.vocab_size
    # no request ends inside the timed steps (the requests of the second prefill step are a token
    # behind the others): all of them are steady decoding of the whole batch
    sp = SamplingParams(temperature=0.0, max_tokens=steps + warmup + 8, ignore_eos=True)
    for p in prompts_for(vocab, batch, prompt_len, seed=100 + batch):
        engine.add_request(p, sp)
    while any(not s.is_prefill_done or s.num_generated_tokens == 0 for s in engine.scheduler.running) \
            or engine.scheduler.waiting:
        engine.step()
    for _ in range(warmup):
        engine.step()
    torch.cuda.synchronize()
    h2d0 = engine.runner.h2d_bytes
    t0 = time.perf_counter()
    n_tokens = 0
    for _ in range(steps):
        n_tokens += sum(1 for o in engine.step() if o.new_token is not None)
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    h2d = (engine.runner.h2d_bytes - h2d0) / steps
    while engine.has_unfinished_requests:
        engine.step()
    return n_tokens / dt, h2d, batch * 4


def ragged_generate(engine, num_requests: int, prompt_range, output_range, seed: int = 0):
    """Ragged requests through the public `LLMEngine.generate`: prompt and output lengths drawn
    uniformly, uniform token ids, greedy, prompts cut into portions under the token budget while
    others decode.  Wall-clock seconds around the call, tokens counted from what comes back."""
    import random
    from paged_llm_b200.config import SamplingParams

    rng = random.Random(seed)
    vocab = engine.model_config.vocab_size
    prompts, params = [], []
    for _ in range(num_requests):
        n = rng.randint(*prompt_range)
        prompts.append([rng.randrange(vocab) for _ in range(n)])
        params.append(SamplingParams(temperature=0.0, max_tokens=rng.randint(*output_range), ignore_eos=True))
    steps0, pre0 = engine.stats.num_steps, engine.stats.num_preemptions
    graph0 = engine.runner.num_graph_steps
    t0 = time.perf_counter()
    outs = engine.generate(prompts, params)
    dt = time.perf_counter() - t0
    generated = sum(len(o.token_ids) for o in outs)
    assert generated == sum(p.max_tokens for p in params), "every request runs to its own length"
    return {"seconds": round(dt, 3), "requests": num_requests, "prompt_tokens": sum(map(len, prompts)),
            "generated_tokens": generated, "generated_tok_s": round(generated / dt, 1),
            "total_tok_s": round((generated + sum(map(len, prompts))) / dt, 1),
            "steps": engine.stats.num_steps - steps0,
            "graph_steps": engine.runner.num_graph_steps - graph0, "preemptions": engine.stats.num_preemptions - pre0}


def prefill_once(engine, tokens: int, iters: int = 5, warmup: int = 3):
    import torch
    from paged_llm_b200.config import SamplingParams
    from paged_llm_b200.engine.runner import StepItem
    from paged_llm_b200.engine.sequence import Sequence

    cm, runner = engine.block_manager, engine.runner
    vocab = engine.model_config.vocab_size
    times = []
    for i in range(warmup + iters):
        seq = Sequence(prompts_for(vocab, 1, tokens, seed=7 + i)[0], SamplingParams())
        assert cm.acquire_state_slot(seq), "too few state slots for the benchmark"
        ok = cm.allocate_slots(seq, tokens)
        assert ok is not None, "pool too small for the benchmark"
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        runner.step([StepItem(seq, tokens, (tokens - 1,))])
        end.record()
        torch.cuda.synchronize()
        if i >= warmup:
            times.append(start.elapsed_time(end))
        cm.free(seq)
    return statistics.median(times)


def mixed_step(engine, batch: int, portion: int, context: int, iters: int = 5, warmup: int = 3):
    """One step that carries `batch` decoding requests (context `context`) beside one prompt portion of
    `portion` tokens of a new request: the step a serving engine runs while a long prompt arrives.
    Returns the median milliseconds of the step (CUDA events)."""
    import torch
    from paged_llm_b200.config import SamplingParams
    from paged_llm_b200.engine.runner import StepItem
    from paged_llm_b200.engine.sequence import Sequence

    cm, runner, ops = engine.block_manager, engine.runner, engine.ops
    vocab = engine.model_config.vocab_size
    seqs = [Sequence(p, SamplingParams()) for p in prompts_for(vocab, batch, context, seed=3)]
    for s in seqs:
        assert cm.acquire_state_slot(s), "too few state slots for the benchmark"
    chunk = max(1, engine.config.max_num_batched_tokens // context)
    for i in range(0, batch, chunk):
        group = seqs[i:i + chunk]
        for s in group:
            ok = cm.allocate_slots(s, context)
            assert ok is not None, "pool too small for the benchmark"
        runner.step([StepItem(s, context, ()) for s in group])
        for s in group:
            s.num_computed_tokens = context
            s.append_token(1)
    times = []
    for i in range(warmup + iters):
        new = Sequence(prompts_for(vocab, 1, portion, seed=50 + i)[0], SamplingParams())
        assert cm.acquire_state_slot(new), "too few state slots for the benchmark"
        ok = cm.allocate_slots(new, portion)
        assert ok is not None
        for s in seqs:
            ok = cm.allocate_slots(s, 1)
            assert ok is not None
        items = [StepItem(s, 1, (0,)) for s in seqs] + [StepItem(new, portion, (portion - 1,))]
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        ops.argmax(runner.step(items))
        end.record()
        torch.cuda.synchronize()
        if i >= warmup:
            times.append(start.elapsed_time(end))
        for s in seqs:
            s.num_computed_tokens += 1
            s.append_token(1)
        cm.free(new)
    for s in seqs:
        cm.free(s)
    return statistics.median(times)


def chunked_prefill(engine, tokens: int, iters: int = 3, warmup: int = 2):
    """One prompt of `tokens` tokens through the public `LLMEngine.generate` with one output token: the
    scheduler cuts it into portions of `max_num_batched_tokens`.  Median wall-clock milliseconds."""
    import torch
    from paged_llm_b200.config import SamplingParams

    vocab = engine.model_config.vocab_size
    times = []
    for i in range(warmup + iters):
        prompt = prompts_for(vocab, 1, tokens, seed=20 + i)[0]
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        engine.generate([prompt], SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True))
        torch.cuda.synchronize()
        if i >= warmup:
            times.append((time.perf_counter() - t0) * 1e3)
    return statistics.median(times)


def sampling_times(args) -> dict:
    """Microseconds per call of the sampler's kernels on `--batch` rows of a vocabulary of the named size: the
    calls are issued back to back (each with its one copy of parameters from pinned memory) and timed with CUDA
    events, so a call that takes the device less than the host takes to issue it shows the host's time."""
    import numpy as np
    import torch
    from paged_llm_b200.kernels.ops import CudaOps

    ops = CudaOps(torch.device("cuda:0"))
    rows, vocab = args.batch, SIZES[args.size]["vocab_size"]
    logits = torch.randn(rows, vocab, device="cuda") * 2.0

    def timed(fn, n=50):
        for _ in range(5):
            fn()
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        for _ in range(n):
            fn()
        end.record()
        torch.cuda.synchronize()
        return round(start.elapsed_time(end) / n * 1e3, 1)

    out = {"only": "sample", "size": args.size, "rows": rows, "vocab": vocab, "unit": "us per call",
           "argmax": timed(lambda: ops.argmax(logits))}
    for name, k, p in (("temperature", 0, 1.0), ("top_k_50", 50, 1.0), ("top_p_0.9", 0, 0.9), ("top_k_50_top_p_0.9", 50, 0.9)):
        arrays = (np.full(rows, 0.7, np.float32), np.full(rows, k, np.int32), np.full(rows, p, np.float32),
                  np.arange(rows, dtype=np.uint64), np.arange(rows, dtype=np.uint64))
        out[name] = timed(lambda: ops.sample(logits, *arrays))
    return out


def validate(args) -> dict:
    """The float32 validation run at the benchmark's layer sizes: the same trace (a 2,048-token
    portion, 32 decoded tokens, portions of changing size, a mixed batch) through the bfloat16 engine
    and the true-float32 engine on the same weight values, and the float32 engine against the plain
    implementation of tests/plain_llama.py on a shorter request.  Reports the largest differences
    relative to the largest logit."""
    import numpy as np
    from paged_llm_b200.engine.replay import TraceReplayer
    from tests import plain_llama, schedules
    from tests.tiny import random_tokens, read_folder

    with tempfile.TemporaryDirectory() as folder:
        cfg, full_layers = make_model(folder, args.size, args.layers, on_device=False)
        V = cfg.vocab_size
        long_req = random_tokens(V, 2048 + 32, 1)
        reqs = {"w": long_req, "p": random_tokens(V, 700, 2), "q": random_tokens(V, 333, 3), "r": random_tokens(V, 90, 4)}
        # whole + tail for the long request, portions and a mixed batch for the others
        steps = [{"step": 0, "entries": [{"id": "w", "tokens": long_req[:2048], "want": [0, 1, 511, 1024, 2047]}], "end": []}]
        for i in range(2048, len(long_req)):
            steps.append({"step": len(steps), "entries": [{"id": "w", "tokens": [long_req[i]], "want": [0]}],
                          "end": ["w"] if i == len(long_req) - 1 else []})
        more, _ = schedules.mixed({k: reqs[k] for k in "pqr"}, live=3, seed=1, choices=(2, 5, 16, 40, 64, 130, 257))
        more = schedules.keep_wanted(more, lambda rid, p: p % 16 == 0 or p >= len(reqs[rid]) - 4)
        for rec in more:
            steps.append({**rec, "step": len(steps)})
        max_tokens = 2112 + sum(schedules._round64(len(reqs[k])) for k in "pqr")
        out = {}
        for dtype in ("float32", "bfloat16"):
            rp = TraceReplayer(folder, dtype, max_tokens)
            res = {rec["step"]: o for rec in steps if (o := rp.step(rec)) is not None}
            out[dtype] = schedules.collect(steps, res)
            del rp
        worst16 = max(float(np.abs(out["bfloat16"][k] - out["float32"][k]).max() / np.abs(out["float32"][k]).max())
                      for k in out["float32"])
        hf, w = read_folder(folder)
        rows = schedules.wanted_positions(steps)["q"]
        want = plain_llama.forward_logits(hf, w, reqs["q"], rows=rows).numpy()
        worst32 = float(np.abs(out["float32"]["q"] - want).max() / max(1.0, np.abs(want).max()))
    return {"only": "validate", "size": args.size, "layers": cfg.num_hidden_layers, "layers_full": full_layers,
            "positions_compared": int(sum(len(v) for v in out["float32"].values())),
            "bf16_vs_f32_engine_rel": round(worst16, 6), "f32_engine_vs_plain_rel": round(worst32, 8),
            "trace": "2,048-token portion + 32 decoded tokens; three requests of 700/333/90 tokens mixed, portions of 2 to 257 tokens"}


def pomisun_configs(name: str):
    """(Pomisun configuration dict, Llama configuration dict of equal size, number of layer runs)."""
    s = POMISUN_SIZES[name]
    mixer = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
             "softcap": 30.0, "mask": {"size": s["chunk"]},
             "rot": {"dims": s["dim"], "base": 500000.0,
                     "scaling": {"factor": 4.0, "original": 4096, "fast": 16.0, "slow": 2.0}}}
    dense = {"kind": "dense", "ff": s["ff"]}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"]}, "router": {"experts": s["experts"], "top": s["top"]},
           "shared": {"ff": s["shared_ff"]}}
    layers = [{"type": "attention", "mixer": mixer, "mlp": dense if i % 2 == 0 else moe} for i in range(s["layers"])]
    pom = {"architecture": "Pomisun", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "layers": layers}
    runs = s["layers"]
    if s["loop"]:
        pom["loop"] = dict(s["loop"])
        runs += (s["loop"]["stop"] - s["loop"]["start"]) * (s["loop"]["times"] - 1)
    llama = {"architectures": ["LlamaForCausalLM"], "vocab_size": s["vocab"], "hidden_size": s["width"],
             "intermediate_size": s["ff"], "num_hidden_layers": runs, "num_attention_heads": s["heads"],
             "num_key_value_heads": s["kv_heads"], "head_dim": s["dim"], "rope_theta": 500000.0, "rms_norm_eps": 1e-6,
             "tie_word_embeddings": True, "max_position_embeddings": 8192}
    return pom, llama, runs


def rokarax_configs(name: str):
    """(Rokarax configuration dict, Llama configuration dict of equal size, number of layers)."""
    s = ROKARAX_SIZES[name]
    attention = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
                 "bias_max": float(s["window"]), "mask": {"size": s["window"]}}
    latent = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot_dim"], "vdim": s["dim"], "q_rank": s["q_rank"],
              "kv_rank": s["kv_rank"], "scale": (s["dim"] + s["rot_dim"]) ** -0.5, "mask": {"size": s["window"]},
              "rot": {"dims": s["rot_dim"], "base": 500000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    ssm = {"heads": s["ssm_heads"], "vdim": s["ssm_dim"], "state": s["state"], "groups": s["groups"], "conv": s["conv"],
           "norm_groups": s["groups"]}
    dense = {"kind": "dense", "ff": s["ff"]}
    order = [("mamba2", ssm), ("attention", attention), ("mamba2", ssm), ("latent_attention", latent), ("mamba2", ssm),
             ("attention", dict(attention, kv_from=1))]
    rok = {"architecture": "Rokarax", "vocab": s["vocab"], "width": s["width"], "embedding": {"scale": s["width"] ** 0.5},
           "norm": {"eps": 1e-6}, "layers": [{"type": t, "mixer": m, "mlp": dense} for t, m in order]}
    llama = {"architectures": ["LlamaForCausalLM"], "vocab_size": s["vocab"], "hidden_size": s["width"],
             "intermediate_size": s["ff"], "num_hidden_layers": len(order), "num_attention_heads": s["heads"],
             "num_key_value_heads": s["kv_heads"], "head_dim": s["dim"], "rope_theta": 500000.0, "rms_norm_eps": 1e-6,
             "tie_word_embeddings": False, "max_position_embeddings": 8192}
    return rok, llama, len(order)


def munazen_configs(name: str):
    """(Munazen configuration dict, Llama configuration dict of equal size, number of layers)."""
    return munazen_configs_of(MUNAZEN_SIZES[name])


def munazen_configs_of(s: dict):
    """The same for sizes that no name stands for."""
    left = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
            "rot": {"dims": s["dim"], "base": 500000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    par = {"left": left, "right": {"width": s["rec_width"], "blocks": s["rec_blocks"], "conv": s["conv"]},
           "left_scale": 1.0, "right_scale": 1.0}
    gla = {"heads": s["gla_heads"], "dim": s["gla_dim"], "vdim": s["gla_vdim"], "tau": 16.0}
    dense = {"kind": "dense", "ff": s["ff"]}
    order = [("parallel", par), ("gla", gla), ("parallel", par), ("parallel", par), ("gla", gla), ("parallel", par)]
    mun = {"architecture": "Munazen", "vocab": s["vocab"], "width": s["width"], "streams": s["streams"],
           "norm": {"eps": 1e-6, "groups": s["norm_groups"]},
           "layers": [{"type": t, "mixer": m, "mlp": dense} for t, m in order]}
    llama = {"architectures": ["LlamaForCausalLM"], "vocab_size": s["vocab"], "hidden_size": s["width"],
             "intermediate_size": s["ff"], "num_hidden_layers": len(order), "num_attention_heads": s["heads"],
             "num_key_value_heads": s["kv_heads"], "head_dim": s["dim"], "rope_theta": 500000.0, "rms_norm_eps": 1e-6,
             "tie_word_embeddings": False, "max_position_embeddings": 8192}
    return mun, llama, len(order)


def pirerax_configs(name: str):
    """(Pirerax configuration dict, Llama configuration dict of equal size, number of layers)."""
    s = PIRERAX_SIZES[name]
    heads = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5}
    attention = dict(heads, q_temp={"coef": 0.5, "every": 1024})
    latent = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot_dim"], "vdim": s["dim"], "kv_rank": s["kv_rank"],
              "scale": (s["dim"] + s["rot_dim"]) ** -0.5, "rot": {"dims": s["rot_dim"], "base": 20000.0}}
    par = {"left": dict(heads, rot={"dims": s["dim"] // 2, "base": 500000.0}),
           "right": {"heads": s["delta_heads"], "kv_heads": s["delta_kv"], "dim": s["delta_dim"], "vdim": s["delta_vdim"],
                     "conv": s["conv"]}}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"], "limit": 7.0},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["groups"][0], "keep": s["groups"][1]}}}
    order = [("parallel", par), ("latent_attention", latent), ("attention", attention), ("attention", attention), ("parallel", par),
             ("latent_attention", latent)]
    pir = {"architecture": "Pirerax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
           "layers": [{"type": t, "mixer": m, "mlp": moe} for t, m in order]}
    llama = {"architectures": ["LlamaForCausalLM"], "vocab_size": s["vocab"], "hidden_size": s["width"],
             "intermediate_size": s["top"] * s["expert_ff"], "num_hidden_layers": len(order), "num_attention_heads": s["heads"],
             "num_key_value_heads": s["kv_heads"], "head_dim": s["dim"], "rope_theta": 500000.0, "rms_norm_eps": 1e-6,
             "tie_word_embeddings": False, "max_position_embeddings": 8192}
    return pir, llama, len(order)


def tagelorn_configs(name: str):
    """(Tagelorn configuration dict, Pirerax configuration dict of equal size, number of layers)."""
    s = TAGELORN_SIZES[name]
    heads = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5}
    attention = dict(heads, bias_max=float(s["window"]), mask={"size": s["window"], "keep_first": s["keep_first"]})
    delta = {"heads": s["delta_heads"], "dim": s["delta_dim"]}
    groups = {"count": s["groups"][0], "keep": s["groups"][1]}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"]}, "router": {"experts": s["experts"], "top": s["top"], "scale": 2.0, "groups": groups},
           "shared": {"ff": s["shared_ff"]}}
    order = [("attention", attention, {"kind": "dense", "ff": s["ff"]}), ("general_delta", delta, moe), ("attention", attention, moe),
             ("general_delta", delta, moe), ("attention", attention, moe), ("general_delta", delta, moe)]
    tag = {"architecture": "Tagelorn", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
           "embedding": {"scale": s["width"] ** 0.5}, "canon": {"taps": s["taps"]}, "token_side": {"dim": s["side_dim"]},
           "logit_softcap": 30.0, "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in order]}
    par = {"left": dict(heads, rot={"dims": s["dim"] // 2, "base": 500000.0}),
           "right": {"heads": s["delta_heads"], "kv_heads": s["delta_heads"], "dim": s["delta_dim"], "vdim": s["delta_dim"], "conv": s["taps"]}}
    pmoe = {"kind": "moe", "expert": {"ff": s["expert_ff"], "limit": 7.0}, "router": {"experts": s["experts"], "top": s["top"], "groups": groups}}
    pir = {"architecture": "Pirerax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
           "layers": [{"type": t, "mixer": m, "mlp": pmoe} for t, m in [("attention", heads), ("parallel", par)] * 3]}
    return tag, pir, len(order)


def nopozen_configs(name: str):
    """(Nopozen, Pomisun and Munazen configuration dicts of equal size, number of layer runs)."""
    s = NOPOZEN_SIZES[name]
    heads = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5}
    rot = {"dims": s["dim"], "base": 500000.0}
    chunked = dict(heads, mask={"size": s["chunk"]}, rot=dict(rot, scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}))
    convolved = dict(heads, rot=dict(rot, dims=s["dim"] // 2), conv=s["taps"])
    linear = {"heads": s["lin_heads"], "dim": s["lin_dim"], "vdim": s["lin_dim"],
              "decay": [1.0 - 2.0 ** (-2.0 - 6.0 * i / s["lin_heads"]) for i in range(s["lin_heads"])]}
    dense = {"kind": "dense", "ff": s["ff"]}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
    loop = {"start": 1, "stop": 4, "times": 2}
    order = [("attention", chunked, dense), ("lightning", linear, moe), ("attention_2", convolved, moe), ("attention", chunked, moe),
             ("lightning", linear, moe), ("attention_2", convolved, moe)]
    top = {"vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}}
    nop = dict(top, architecture="Nopozen", layers=[{"type": t, "mixer": m, "mlp": f} for t, m, f in order], loop=loop)
    pom_mixer = dict(heads, mask={"size": s["chunk"]}, rot=dict(rot, scaling={"factor": 4.0, "original": 4096, "fast": 16.0, "slow": 2.0}))
    pom = dict(top, architecture="Pomisun", layers=[{"type": "attention", "mixer": pom_mixer, "mlp": f} for _, _, f in order], loop=loop)
    mun, _, _ = munazen_configs_of(dict(vocab=s["vocab"], width=s["width"], heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"],
                                        ff=s["top"] * s["expert_ff"], rec_width=s["width"], rec_blocks=s["rec_blocks"], conv=s["taps"],
                                        gla_heads=s["lin_heads"], gla_dim=s["lin_dim"], gla_vdim=s["lin_dim"], streams=1, norm_groups=1))
    kinds = mun["layers"][:2]                       # attention beside the recurrence, linear attention
    mun["layers"] = [kinds[i] for i in (0, 1, 0) * 3]
    return nop, pom, mun, len(order) + 3


def compare_with_llama(args, label: str, size: str, sizes: dict, model: dict, llama: dict, runs: int, beside: str = "llama",
                       more: tuple = ()) -> dict:
    """Prefill and decode of another decoder at layer sizes of a real model (random weights drawn on the
    device) beside a Llama (or the model named by `beside`, and those in `more`) of equal width, heads and layer runs:
    device-timed with CUDA events, with the device time of every kernel inside the steps for the roofline of each."""
    import torch
    from paged_llm_b200 import EngineConfig, LLMEngine
    from paged_llm_b200.config.registry import parse_model_config
    from paged_llm_b200.weights import write_random_stub

    pre = args.prefill_tokens or PREFILL_TOKENS
    ctx_len = args.context or PROMPT_LEN
    steps = min(args.steps, 64)
    batches = (8, 64) if args.batch == 8 else (args.batch,)
    max_len = max(ctx_len + steps + args.warmup + 16, pre) + 64
    out = {"only": label, "size": size, "layer_runs": runs, "prefill_tokens": pre, "context": ctx_len,
           "sizes": sizes, "peaks": load_peaks()}
    for arm, hf in ((label, model), (beside, llama), *more):
        with tempfile.TemporaryDirectory() as folder:
            _, cfg = parse_model_config(hf)
            write_random_stub(folder, cfg, seed=0, std=0.02, dtype="bfloat16")
            seqs = max(batches)
            engine = LLMEngine(folder, EngineConfig(
                dtype="bfloat16", block_size=BLOCK_SIZE, max_model_len=max_len, max_num_seqs=max(seqs, 64),
                max_num_batched_tokens=max(2048, pre), enable_prefix_caching=False,
                num_gpu_blocks=seqs * (-(-max_len // BLOCK_SIZE)) + 64))
        res = {"params": cfg.num_parameters, "weight_bytes_per_decode_step": engine.model.weight_bytes_per_step()}
        ms = prefill_once(engine, pre)
        res["prefill_ms"] = round(ms, 3)
        res["prefill_tokens_per_s"] = round(pre * 1000.0 / ms, 1)
        if args.kernel_times:
            res["prefill_kernels"] = prefill_kernel_times(engine, pre)
        for B in batches:
            ms, launches, ctx_mid = device_decode_loop(engine, B, steps, args.warmup, ctx_len)
            res[f"decode_b{B}"] = {"ms_per_step": round(ms, 4), "tokens_per_s": round(B * 1000.0 / ms, 1),
                                   "launches_per_step": launches, "context": ctx_mid}
            if args.kernel_times:
                res[f"decode_b{B}"]["kernels"] = decode_kernel_times(engine, B, min(steps, 8), args.warmup, ctx_len)
        engine.ops.check_kernels()
        out[arm] = res
        del engine
        torch.cuda.empty_cache()
    return out


def pomisun_compare(args) -> dict:
    pom, llama, runs = pomisun_configs(args.pomisun_size)
    return compare_with_llama(args, "pomisun", args.pomisun_size, POMISUN_SIZES[args.pomisun_size], pom, llama, runs)


def rokarax_compare(args) -> dict:
    rok, llama, runs = rokarax_configs(args.rokarax_size)
    return compare_with_llama(args, "rokarax", args.rokarax_size, ROKARAX_SIZES[args.rokarax_size], rok, llama, runs)


def munazen_compare(args) -> dict:
    mun, llama, runs = munazen_configs(args.munazen_size)
    return compare_with_llama(args, "munazen", args.munazen_size, MUNAZEN_SIZES[args.munazen_size], mun, llama, runs)


def pirerax_compare(args) -> dict:
    pir, llama, runs = pirerax_configs(args.pirerax_size)
    return compare_with_llama(args, "pirerax", args.pirerax_size, PIRERAX_SIZES[args.pirerax_size], pir, llama, runs)


def tagelorn_compare(args) -> dict:
    tag, pir, runs = tagelorn_configs(args.tagelorn_size)
    return compare_with_llama(args, "tagelorn", args.tagelorn_size, TAGELORN_SIZES[args.tagelorn_size], tag, pir, runs, beside="pirerax")


def nopozen_compare(args) -> dict:
    nop, pom, mun, runs = nopozen_configs(args.nopozen_size)
    return compare_with_llama(args, "nopozen", args.nopozen_size, NOPOZEN_SIZES[args.nopozen_size], nop, pom, runs, beside="pomisun",
                              more=(("munazen", mun),))


def run_ours(args) -> dict:
    import torch
    from paged_llm_b200 import EngineConfig, LLMEngine

    peaks = load_peaks()
    if args.only == "pomisun":
        return pomisun_compare(args)
    if args.only == "rokarax":
        return rokarax_compare(args)
    if args.only == "munazen":
        return munazen_compare(args)
    if args.only == "pirerax":
        return pirerax_compare(args)
    if args.only == "tagelorn":
        return tagelorn_compare(args)
    if args.only == "nopozen":
        return nopozen_compare(args)
    if args.only == "validate":
        return validate(args)
    if args.only == "sample":
        return sampling_times(args)
    with tempfile.TemporaryDirectory() as folder:
        cfg, full_layers = make_model(folder, args.size, args.layers)
        prompt_len = args.context if args.only in ("decode", "mixed") and args.context else PROMPT_LEN
        pre_tokens = args.prefill_tokens if args.only in ("prefill", "mixed") and args.prefill_tokens else PREFILL_TOKENS
        max_len = max(prompt_len + args.steps + args.warmup + DECODE_LEN, pre_tokens) + 64
        if args.only == "ragged":
            p_hi = int(args.prompt_range.split(",")[1]) if args.prompt_range else RAGGED_PROMPTS[1]
            o_hi = int(args.output_range.split(",")[1]) if args.output_range else RAGGED_OUTPUTS[1]
            max_len = max(p_hi, 512) + max(o_hi, 32) + 64          # (the untimed first requests are up to 512 + 32 long)
        seqs = max(args.batch, 64) if prompt_len == PROMPT_LEN else args.batch
        if args.only == "mixed":
            max_len = max(max_len, prompt_len + 64, pre_tokens + 64)
            seqs = args.batch + 2
        engine = LLMEngine(folder, EngineConfig(
            dtype="bfloat16", block_size=BLOCK_SIZE, max_model_len=max_len, max_num_seqs=max(seqs, 64),
            max_num_batched_tokens=args.chunk if args.only == "prefill" and args.chunk else max(2048, pre_tokens),
            enable_prefix_caching=False,
            num_gpu_blocks=seqs * (-(-max_len // BLOCK_SIZE)) + 64))
    B = args.batch
    if args.only == "ragged":            # 64 ragged requests under a 2,048-token budget, end to end
        engine.warm_up()
        ragged_generate(engine, 8, (128, 512), (16, 32), seed=1)          # untimed: first-use costs
        # untimed too: the same workload with other lengths and tokens, so that the graphs of its batch buckets
        # and context classes exist (a server runs for longer than its first two seconds)
        n_req = args.requests
        p_range = tuple(int(v) for v in args.prompt_range.split(",")) if args.prompt_range else RAGGED_PROMPTS
        o_range = tuple(int(v) for v in args.output_range.split(",")) if args.output_range else RAGGED_OUTPUTS
        ragged_generate(engine, n_req, p_range, o_range, seed=1)
        return {"only": "ragged", "size": args.size, "layers": cfg.num_hidden_layers,
                "prompt_range": list(p_range), "output_range": list(o_range),
                **ragged_generate(engine, n_req, p_range, o_range, seed=0)}
    if args.only == "decode":            # a short run of one part, for profilers and other context lengths
        ms, launches, ctx_mid = device_decode_loop(engine, B, args.steps, args.warmup, prompt_len)
        step_bytes = engine.model.weight_bytes_per_step() + B * ctx_mid * (engine.kv_cache.page_bytes() // BLOCK_SIZE)
        gbs = step_bytes / (ms * 1e-3) / 1e9
        extra = {"kernel_times": decode_kernel_times(engine, B, min(args.steps, 8), args.warmup, prompt_len)} \
            if args.kernel_times else {}
        return {**extra, "only": "decode", "size": args.size, "batch": B, "context": ctx_mid, "ms_per_step": round(ms, 4),
                "tokens_per_s": round(B * 1000.0 / ms, 1), "launches_per_step": launches,
                "layers": cfg.num_hidden_layers, "layers_full": full_layers, "gb_per_s": round(gbs, 1),
                "frac": round(gbs / peaks["hbm_gbs"], 4), "peaks_source": peaks["source"]}
    if args.only == "mixed":             # B decoding requests beside one prompt portion, in one step
        portion = args.prefill_tokens or PREFILL_TOKENS
        ms = mixed_step(engine, B, portion, prompt_len, iters=max(3, min(args.steps, 10)), warmup=args.warmup)
        flops = step_flops(cfg, portion) + B * step_flops(cfg, 1, prompt_len)
        return {"only": "mixed", "size": args.size, "layers": cfg.num_hidden_layers, "layers_full": full_layers,
                "decoding_requests": B, "context": prompt_len, "portion": portion, "ms": round(ms, 3),
                "tokens_per_s": round((portion + B) * 1000.0 / ms, 1),
                "tflops": round(flops / (ms * 1e-3) / 1e12, 1),
                "frac": round(flops / (ms * 1e-3) / 1e12 / peaks["bf16_tflops"], 4), "peaks_source": peaks["source"]}
    if args.only == "prefill" and args.chunk:
        ms = chunked_prefill(engine, pre_tokens, iters=max(1, args.steps), warmup=args.warmup)
        tflops = step_flops(cfg, pre_tokens) / (ms * 1e-3) / 1e12
        return {"only": "prefill", "size": args.size, "tokens": pre_tokens, "portions_of": args.chunk, "ms": round(ms, 3),
                "through": "LLMEngine.generate, one output token, wall clock", "layers": cfg.num_hidden_layers,
                "layers_full": full_layers, "tokens_per_s": round(pre_tokens * 1000.0 / ms, 1), "tflops": round(tflops, 1),
                "frac": round(tflops / peaks["bf16_tflops"], 4), "peaks_source": peaks["source"]}
    if args.only == "prefill":
        pre_ms = prefill_once(engine, pre_tokens, iters=max(1, args.steps), warmup=args.warmup)
        tflops = step_flops(cfg, pre_tokens) / (pre_ms * 1e-3) / 1e12
        extra = {"kernel_times": prefill_kernel_times(engine, pre_tokens)} if args.kernel_times else {}
        return {**extra, "only": "prefill", "size": args.size, "tokens": pre_tokens, "ms": round(pre_ms, 3),
                "layers": cfg.num_hidden_layers, "tflops": round(tflops, 1),
                "frac": round(tflops / peaks["bf16_tflops"], 4), "peaks_source": peaks["source"]}
    weight_bytes = engine.model.weight_bytes_per_step()
    kv_bytes_per_token = engine.kv_cache.page_bytes() // BLOCK_SIZE

    with ClockSampler() as clocks:
        ms, launches, ctx_mid = device_decode_loop(engine, B, args.steps, args.warmup, PROMPT_LEN)
    clock_summary = clocks.summary()
    value = B * 1000.0 / ms
    step_bytes = weight_bytes + B * ctx_mid * kv_bytes_per_token
    achieved = step_bytes / (ms * 1e-3) / 1e9

    e2e_value, h2d, d2h = e2e_decode(engine, B, args.steps, args.warmup, PROMPT_LEN)
    points = {}
    for b in (1, 64):
        pms, _, _ = device_decode_loop(engine, b, min(args.steps, 128), args.warmup, PROMPT_LEN)
        points[f"decode_b{b}"] = round(b * 1000.0 / pms, 1)
    pre_ms = prefill_once(engine, PREFILL_TOKENS)
    flops = step_flops(cfg, PREFILL_TOKENS)
    peak_flops = peaks["bf16_tflops"] * 1e12

    return {
        "metric": "decode tok/s at batch 8 (TinyLlama 1.1B sizes, 512-token prompts, bf16, one B200)",
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: random weights N(0, 0.02) seed 0, uniform random token ids",
        "impl": "ours",
        "config": {
            "model": "TinyLlama-1.1B layer sizes" if args.size == "tinyllama-1.1b" else args.size,
            "global_batch": B, "seq_len": PROMPT_LEN + DECODE_LEN, "prompt_len": PROMPT_LEN,
            "decode_len": DECODE_LEN, "parallelism": "single GPU", "layers": cfg.num_hidden_layers,
            "layers_full": full_layers, "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads,
            "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size,
            "vocab": cfg.vocab_size, "block_size": BLOCK_SIZE, "params": cfg.num_parameters,
            "l2": "weights (2.2 GB) exceed the 126 MB L2: no flush between iterations",
            "peaks": peaks["source"], "cuda_graphs": not engine.config.enforce_eager,
        },
        "e2e": {"value": round(e2e_value, 1), "unit": "tokens/s", "h2d_bytes_per_step": int(h2d),
                "d2h_bytes_per_step": int(d2h)},
        "gpu_launches": int(round(launches * args.steps)),
        "clocks": clock_summary,
        "prefill": {"value": round(PREFILL_TOKENS * 1000.0 / pre_ms, 1), "tokens": PREFILL_TOKENS,
                    "ms": round(pre_ms, 3), "frac": round(flops / (pre_ms * 1e-3) / peak_flops, 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / peaks["hbm_gbs"], 4)},
        "points": points,
    }


# ------------------------------------------------------------------------------ reference

def run_reference(args) -> dict:
    ref_dir = os.path.join(ROOT, "baseline", "_ref")
    if not os.path.isdir(os.path.join(ref_dir, "pagedllm")):
        return {"impl": "reference", "unavailable": "baseline/_ref holds no installed reference (pip install --target failed or was not run)"}
    try:
        import torch
        if not torch.cuda.is_available():
            return {"impl": "reference", "unavailable": "no CUDA device"}
        sys.path.insert(0, ref_dir)
        from pagedllm import EngineConfig, SamplingParams
        from pagedllm.engine import LLMEngine
    except Exception as e:                                            # noqa: BLE001
        return {"impl": "reference", "unavailable": f"import of the reference failed: {type(e).__name__}: {e}"[:300]}
    B = args.batch
    try:
        with tempfile.TemporaryDirectory() as folder:
            cfg, full_layers = make_model(folder, args.size, args.layers, with_tokenizer=True)
            max_len = PROMPT_LEN + args.steps + args.warmup + DECODE_LEN + 64
            engine = LLMEngine(folder, EngineConfig(
                dtype="bfloat16", block_size=BLOCK_SIZE, max_model_len=max_len, max_num_seqs=64,
                max_num_batched_tokens=4096, enable_prefix_caching=False,
                num_gpu_blocks=64 * (-(-max_len // BLOCK_SIZE)) + 64))
        sp = SamplingParams(temperature=0.0, max_tokens=args.steps + args.warmup + 1, ignore_eos=True)
        for p in prompts_for(cfg.vocab_size, B, PROMPT_LEN, seed=100 + B):
            engine.add_request(p, sp)
        while engine.scheduler.waiting or any(s.num_generated_tokens == 0 for s in engine.scheduler.running):
            engine.step()
        for _ in range(args.warmup):
            engine.step()
        torch.cuda.synchronize()
        with ClockSampler() as clocks:
            t0 = time.perf_counter()
            n = 0
            for _ in range(args.steps):
                n += sum(1 for o in engine.step() if o.new_token is not None)
            torch.cuda.synchronize()
            dt = time.perf_counter() - t0
        value = n / dt
        return {
            "metric": "decode tok/s at batch 8 (TinyLlama 1.1B sizes, 512-token prompts, bf16, one B200)",
            "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": round(dt * 1000.0 / args.steps, 4), "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random weights, uniform random token ids",
            "impl": "reference",
            "config": {"model": "TinyLlama-1.1B layer sizes" if args.size == "tinyllama-1.1b" else args.size,
                       "global_batch": B, "seq_len": PROMPT_LEN + DECODE_LEN, "prompt_len": PROMPT_LEN,
                       "layers": cfg.num_hidden_layers, "layers_full": full_layers, "parallelism": "single GPU",
                       "attention": engine.attention_backend, "timing": "wall clock around LLMEngine.step()"},
            "e2e": {"value": round(value, 1), "unit": "tokens/s"},
            "clocks": clocks.summary(),
        }
    except Exception as e:                                            # noqa: BLE001
        return {"impl": "reference", "unavailable": f"the reference failed to run: {type(e).__name__}: {e}"[:300]}


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", choices=["ours", "reference"], default="ours")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=None,
                    help="with --only decode or mixed: prompt length of the decoding requests instead of 512")
    ap.add_argument("--prefill-tokens", type=int, default=None,
                    help="with --only prefill: length of the prompt (one step) instead of 2,048")
    ap.add_argument("--size", choices=sorted(SIZES), default="tinyllama-1.1b")
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the named size (reported in config)")
    ap.add_argument("--chunk", type=int, default=None,
                    help="with --only prefill: the prompt goes through LLMEngine.generate in portions of this many tokens")
    ap.add_argument("--requests", type=int, default=64, help="with --only ragged: number of requests")
    ap.add_argument("--prompt-range", default=None, help="with --only ragged: LO,HI prompt lengths (default 128,4096)")
    ap.add_argument("--output-range", default=None, help="with --only ragged: LO,HI output lengths (default 64,512)")
    ap.add_argument("--kernel-times", action="store_true",
                    help="with --only decode or --only prefill: add the device time of every kernel inside the replayed steps")
    ap.add_argument("--pomisun-size", choices=sorted(POMISUN_SIZES), default="p-2k",
                    help="with --only pomisun: the layer sizes (the Llama beside it gets the same)")
    ap.add_argument("--rokarax-size", choices=sorted(ROKARAX_SIZES), default="r-2k",
                    help="with --only rokarax: the layer sizes (the Llama beside it gets the same)")
    ap.add_argument("--munazen-size", choices=sorted(MUNAZEN_SIZES), default="m-2k",
                    help="with --only munazen: the layer sizes (the Llama beside it gets the same)")
    ap.add_argument("--pirerax-size", choices=sorted(PIRERAX_SIZES), default="x-2k",
                    help="with --only pirerax: the layer sizes (the Llama beside it gets the same)")
    ap.add_argument("--tagelorn-size", choices=sorted(TAGELORN_SIZES), default="t-2k",
                    help="with --only tagelorn: the layer sizes (the Pirerax beside it gets the same)")
    ap.add_argument("--nopozen-size", choices=sorted(NOPOZEN_SIZES), default="n-2k",
                    help="with --only nopozen: the layer sizes (the Pomisun and the Munazen beside it get the same)")
    ap.add_argument("--only", choices=["decode", "prefill", "ragged", "mixed", "validate", "sample", "pomisun", "rokarax", "munazen",
                                       "pirerax", "tagelorn", "nopozen"], default=None,
                    help="run only the decode loop, only the prefill step, the ragged serving workload through "
                         "LLMEngine.generate, one mixed step (--batch decoding requests of --context tokens beside one "
                         "portion of --prefill-tokens), the float32 validation run, the sampler's kernels on --batch rows, or "
                         "prefill and decode of the Pomisun, the Rokarax, the Munazen or the Pirerax decoder beside a Llama of equal size "
                         "(--pomisun-size, --rokarax-size, --munazen-size, --pirerax-size), or of the Tagelorn decoder beside a Pirerax of "
                         "equal size (--tagelorn-size), or of the Nopozen decoder beside a Pomisun and a Munazen of equal size "
                         "(--nopozen-size), and print "
                         "a short line")
    args = ap.parse_args()
    if args.gpus != 1 or int(os.environ.get("WORLD_SIZE", "1")) > 1:
        if int(os.environ.get("RANK", "0")) == 0:
            print(json.dumps({"unavailable": f"this engine runs on one GPU; --gpus {args.gpus} is not supported",
                              "n_gpus": args.gpus}))
        return 2
    if args.warmup < 3:
        args.warmup = 3
    line = run_reference(args) if args.impl == "reference" else run_ours(args)
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
