"""The Nopozen decoder as data: `NopozenConfig` -> `ModelSpec`.

Tensor names: `embed`, `head` (a matrix of its own), `final.norm`, `loop.in` (joins the stream and the embedding's output),
and per layer i the norm `l<i>.norm1`, the mixer under `l<i>.mix.` and the feed-forward under `l<i>.mlp.`.  Matrices are
stored [out, in].

A layer is parallel: with h = norm1(x), x += mixer(h) + ff(h) (or the mixer alone).  The mixer is "attention"
(`mix.{q,k,v,o}` with biases `.b`, `q.norm`, `k.norm`, `g`): grouped-query heads with a weighted RMS norm per head, rotary
positions on the first dims with Llama-3.1 scaling, a chunked mask and a gate per head; "attention_2" (`mix.{q,k,v}` with
`.conv`, `g`, `o`): a short convolution on queries, keys and values, rotary positions, 1 in the softmax's denominator and a
gate per element; or "lightning" (`mix.{q,k,v,g,norm,o}`): linear attention with a fixed decay per head.  The feed-forward
is W_down relu(W_up h)^2 or SiLU-gated routed experts with a bias on the router's logits.  A span of layers may run several
times in a row with the same weights; each run has a cache of its own, and every pass begins with W_in [x; x0], x0 the
embedding's output.
"""

from __future__ import annotations

from ..config.nopozen import NopozenConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

# The design fixes this: attention_2's softmax counts one key more, whose score is 0 and which has no value.
SINK_SCORE = 0.0


class _Positions:
    """Rotary tables by their parameters: layers with the same rotation share one."""

    def __init__(self):
        self.specs: dict[str, PartSpec] = {}

    def name(self, rot, head_dim: int) -> str | None:
        if rot is None:
            return None
        scaling = None
        if rot.scaling is not None:
            factor, low, high, original = rot.scaling
            scaling = dict(type="llama3", factor=factor, low_freq_factor=low, high_freq_factor=high,
                           original_max_position_embeddings=original)
        spec = PartSpec("rotary", dict(head_dim=rot.dims, theta=rot.base, pairing="half", scaling=scaling, exact=True))
        for name, known in self.specs.items():
            if known.params == spec.params:
                return name
        name = f"rotary{len(self.specs)}"
        self.specs[name] = spec
        return name


def _mixer(w: int, eps: float, kind: str, m, p: str, positions: _Positions) -> PartSpec:
    if kind == "lightning":
        return PartSpec("fixed_decay_attention", dict(hidden_size=w, num_heads=m.heads, head_dim=m.dim, value_dim=m.vdim, decay=m.decay,
                                                      eps=eps),
                        {**{x + "_proj": p + x for x in ("q", "k", "v", "g", "o")}, "norm": p + "norm"})
    sizes = dict(hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
                 position=positions.name(m.rot, m.dim))
    names = {x + "_proj": p + x for x in ("q", "k", "v", "g", "o")}
    if kind == "attention":
        names.update({x + "_proj_bias": f"{p}{x}.b" for x in ("q", "k", "v", "o")}, q_norm=p + "q.norm", k_norm=p + "k.norm")
        return PartSpec("gated_attention", dict(sizes, chunk=m.chunk, gate="head", head_norm=True, head_norm_weight=True, bias=True,
                                                out_bias=True), names)
    names.update({x + "_conv": f"{p}{x}.conv" for x in ("q", "k", "v")})
    return PartSpec("convolved_attention", dict(sizes, taps=m.taps, gate=True, sink_score=SINK_SCORE), names)


def _feed_forward(w: int, f, p: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("ungated_mlp", dict(hidden_size=w, intermediate_size=f.ff, activation="relu2"),
                        {x + "_proj": p + x for x in ("up", "down")})
    names = {"router": p + "router", "router_bias": p + "router.b"}
    for e in range(f.experts):
        for x in ("gate", "up", "down"):
            names[f"e{e}.{x}"] = f"{p}e{e}.{x}"
    return PartSpec("routed_mlp", dict(hidden_size=w, expert_size=f.ff, num_experts=f.experts, top_k=f.top, activation="silu",
                                       router_bias=True, defer_sum=True), names)


def nopozen_spec(cfg: NopozenConfig) -> ModelSpec:
    w, eps, vocab = cfg.hidden_size, cfg.norm_eps, cfg.vocab_size

    def norm(name: str) -> PartSpec:
        return PartSpec("rms_norm", dict(dim=w, eps=eps), {"weight": name})

    positions, layers = _Positions(), []
    for i, lay in enumerate(cfg.layers):
        p = f"l{i}."
        layers.append(LayerSpec("parallel_norm", _mixer(w, eps, lay.type, lay.mixer, p + "mix.", positions),
                                _feed_forward(w, lay.mlp, p + "mlp.") if lay.mlp is not None else None, {"input": norm(p + "norm1")}))
    return ModelSpec(
        hidden_size=w,
        vocab_size=vocab,
        embedding=PartSpec("embedding", dict(vocab_size=vocab, hidden_size=w), {"weight": "embed"}),
        layers=layers,
        schedule=[ScheduleEntry(i, join_embedding=begins) for i, begins in cfg.layer_runs()],
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(vocab_size=vocab, hidden_size=w), {"weight": "head"}),
        positions=positions.specs,
        stream_join=PartSpec("linear_join", dict(hidden_size=w), {"weight": "loop.in"}) if cfg.loop is not None else None,
    )
