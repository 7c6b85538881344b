"""The Tagelorn decoder as data: `TagelornConfig` -> `ModelSpec`.

Tensor names: `embed` (also the head), `side.embed` (a vector per token and layer, side by side), `final.norm`, and per
layer i the norms `l<i>.norm1` / `l<i>.norm2`, the input convolution `l<i>.canon1`, the mixer under `l<i>.mix.`, the
feed-forward under `l<i>.mlp.` and the token input `l<i>.side.{gate,proj,norm}`.  Matrices are stored [out, in].

The stream starts as the scaled embedding plus a sinusoidal vector of the position.  A layer is pre-norm: x += mixer(c),
c the normed input plus its causal convolution; then (unless the layer has no feed-forward) x += ff(norm2(x)); then the
token's own vector of the layer, gated by the stream, projected and normed, is added.  The mixer is "attention"
(`mix.{q,k,v}` with biases `.b`, `rel`, `sink`, `o`): grouped-query heads with unit-RMS queries and keys, a learned bias by
distance, a window beside which the first tokens stay visible, and a sink; or "general_delta" (`mix.{r,k,v,g,a,a.b,w0,w1,w2,
norm,o}`).  The feed-forward is a gated one with GELU, or routed experts of one matrix, the square of relu and another
matrix beside a shared expert of the same form.  The head caps its logits.
"""

from __future__ import annotations

from ..config.tagelorn import TagelornConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

# The design fixes these: the sinusoids' base, and a group of experts scores its largest choice score.
SINUSOID_BASE = 10000.0
GROUP_SCORE_TOP = 1


def _mixer(w: int, eps: float, kind: str, m, p: str) -> PartSpec:
    if kind == "attention":
        names = {"rel": p + "rel", "sink": p + "sink", "o_proj": p + "o"}
        for x in ("q", "k", "v"):
            names[x + "_proj"], names[x + "_proj_bias"] = p + x, p + x + ".b"
        return PartSpec("gated_attention", dict(
            hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
            window=m.window, keep_first=m.keep_first, distance_bias=True, bias_far=m.bias_max, gate=False, sink=True,
            head_norm=True, bias=True), names)
    return PartSpec("general_delta", dict(hidden_size=w, num_heads=m.heads, head_dim=m.dim, eps=eps), {
        "r_proj": p + "r", "k_proj": p + "k", "v_proj": p + "v", "g_proj": p + "g", "removal_proj": p + "a",
        "removal_bias": p + "a.b", "decay_down": p + "w1", "decay_up": p + "w2", "decay_bias": p + "w0", "norm": p + "norm",
        "o_proj": p + "o"})


def _feed_forward(w: int, f, p: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("gated_mlp", dict(hidden_size=w, intermediate_size=f.ff, activation="gelu_tanh"),
                        {x + "_proj": p + x for x in ("gate", "up", "down")})
    names = {"router": p + "router", "correction": p + "correction"}
    for prefix in [f"e{e}" for e in range(f.experts)] + (["shared"] if f.shared_ff is not None else []):
        for x in ("up", "down"):
            names[f"{prefix}.{x}"] = f"{p}{prefix}.{x}"
    return PartSpec("routed_mlp", dict(
        hidden_size=w, expert_size=f.ff, num_experts=f.experts, top_k=f.top, activation="relu2", gated=False,
        shared_size=f.shared_ff, shared_gate=False, scoring="softmax", correction=True, groups=f.groups,
        group_score_top=GROUP_SCORE_TOP, renorm=True, weight_scale=f.scale), names)


def tagelorn_spec(cfg: TagelornConfig) -> ModelSpec:
    w, eps, vocab = cfg.hidden_size, cfg.norm_eps, cfg.vocab_size

    def norm(name: str) -> PartSpec:
        return PartSpec("rms_norm", dict(dim=w, eps=eps), {"weight": name})

    layers, unused = [], []
    for i, lay in enumerate(cfg.layers):
        p = f"l{i}."
        mixer = PartSpec("input_convolution", dict(hidden_size=w, taps=cfg.taps, mixer=_mixer(w, eps, lay.type, lay.mixer, p + "mix.")),
                         {"conv": p + "canon1"})
        norms, ffn = {"input": norm(p + "norm1")}, None
        if lay.mlp is not None:
            norms["post_mixer"] = norm(p + "norm2")
            ffn = _feed_forward(w, lay.mlp, p + "mlp.")
        else:
            unused.append(p + "norm2")          # (a checkpoint may carry the norm of a feed-forward that is not there)
        block = PartSpec("pre_norm_token_side", dict(
            hidden_size=w, vocab_size=vocab, dim=cfg.side_dim, offset=i * cfg.side_dim, table_width=len(cfg.layers) * cfg.side_dim,
            eps=eps), {"table": "side.embed", "gate": p + "side.gate", "proj": p + "side.proj", "norm": p + "side.norm"})
        layers.append(LayerSpec(block, mixer, ffn, norms))
    return ModelSpec(
        hidden_size=w,
        vocab_size=vocab,
        embedding=PartSpec("embedding", dict(vocab_size=vocab, hidden_size=w, scale=cfg.embedding_scale, position="sinusoidal"),
                           {"weight": "embed"}),
        layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(layers))],
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(vocab_size=vocab, hidden_size=w, tied_to="embed", softcap=cfg.logit_softcap), {"weight": "head"}),
        positions={"sinusoidal": PartSpec("sinusoidal", dict(width=w, base=SINUSOID_BASE))},
        ignored_tensors=tuple(unused),
    )
