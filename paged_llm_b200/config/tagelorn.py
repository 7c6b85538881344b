"""Typed configuration of the Tagelorn decoder, read from a checkpoint's config.json.

config.json gives every size and every constant that may differ between models of the design:

    architecture     "Tagelorn"
    vocab, width     vocabulary and width of the residual stream
    norm.eps         epsilon of every RMS norm
    embedding.scale  factor on the embedding's rows
    canon.taps       taps of the convolution in front of every mixer
    token_side.dim   size of a layer's own vector per token
    logit_softcap    cap c on the logits, c tanh(logits / c) (absent: none)
    layers           one entry per layer: `type` (the mixer), `mixer` (its sizes and constants) and `mlp` (null for none)

Mixers by `type`:

    "attention"      heads, kv_heads, dim (query/key head), vdim (value head), scale, bias_max (farthest distance of the
                     bias table), mask {size (window), keep_first} (absent: every earlier token is seen)
    "general_delta"  heads, dim

Feed-forwards by `mlp.kind`:

    "dense"          ff
    "moe"            expert {ff}, router {experts, top, scale, groups {count, keep} (absent: none)}, shared {ff} (absent: none)

What the engine does not compute is refused here with a message, never computed wrongly.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

from .model import ConfigError, ModelConfig
from .pirerax import _heads, _scale
from .rokarax import _need, _positive_int

MIXER_TYPES = ("attention", "general_delta")


@dataclass(frozen=True)
class TagelornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    window: int | None = None
    keep_first: int = 0

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "TagelornAttention":
        heads, kv = _heads(d, where)
        dim = _positive_int(d, "dim", where)
        vdim = int(d.get("vdim", dim))
        if vdim < 1:
            raise ConfigError(f"{where}: vdim={vdim} must be positive")
        far = float(_need(d, "bias_max", where))
        if not (far > 1 and math.isfinite(far)):
            raise ConfigError(f"{where}: bias_max={far} must be above 1")
        window, keep = None, 0
        mask = d.get("mask")
        if mask is not None:
            window = _positive_int(mask, "size", where + ".mask")
            keep = int(mask.get("keep_first", 0))
            if keep < 0:
                raise ConfigError(f"{where}.mask: keep_first={keep} must not be negative")
        return cls(heads, kv, dim, vdim, _scale(d, where), far, window, keep)

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale, "bias_max": int(self.bias_max) if self.bias_max.is_integer() else self.bias_max}
        if self.window is not None:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return d


@dataclass(frozen=True)
class TagelornDelta:
    heads: int
    dim: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "TagelornDelta":
        return cls(_positive_int(d, "heads", where), _positive_int(d, "dim", where))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim}


_MIXERS = {"attention": TagelornAttention, "general_delta": TagelornDelta}


@dataclass(frozen=True)
class TagelornMLP:
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    scale: float = 1.0
    groups: tuple | None = None         # (count, keep)
    shared_ff: int | None = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "TagelornMLP":
        kind = _need(d, "kind", where)
        if kind == "dense":
            return cls(kind, _positive_int(d, "ff", where))
        if kind != "moe":
            raise ConfigError(f"{where}: kind={kind!r} is not implemented (dense and moe only)")
        ro = _need(d, "router", where)
        experts, top = _positive_int(ro, "experts", where + ".router"), _positive_int(ro, "top", where + ".router")
        scale = float(_need(ro, "scale", where + ".router"))
        if not math.isfinite(scale):
            raise ConfigError(f"{where}.router: scale={scale}")
        groups, allowed = ro.get("groups"), experts
        if groups is not None:
            count, keep = _positive_int(groups, "count", where + ".router.groups"), _positive_int(groups, "keep", where + ".router.groups")
            if experts % count or keep > count:
                raise ConfigError(f"{where}.router.groups: {experts} experts in {count} groups of which {keep} are kept")
            groups, allowed = (count, keep), experts // count * keep
        if top > allowed:
            raise ConfigError(f"{where}.router: top={top} of {allowed} experts that may be chosen")
        shared = d.get("shared")
        return cls(kind, _positive_int(_need(d, "expert", where), "ff", where + ".expert"), experts, top, scale, groups,
                   _positive_int(shared, "ff", where + ".shared") if shared is not None else None)

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        router: dict[str, Any] = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if self.groups is not None:
            router["groups"] = {"count": self.groups[0], "keep": self.groups[1]}
        out = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class TagelornLayer:
    type: str
    mixer: Any
    mlp: TagelornMLP | None


@dataclass(frozen=True)
class TagelornConfig(ModelConfig):
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    taps: int = 1
    side_dim: int = 1
    logit_softcap: float | None = None
    layers: tuple = ()

    @classmethod
    def from_hf_dict(cls, cfg: dict[str, Any], architecture: str = "Tagelorn") -> "TagelornConfig":
        top = "the top level"
        vocab, width = _positive_int(cfg, "vocab", top), _positive_int(cfg, "width", top)
        eps = float(_need(_need(cfg, "norm", top), "eps", "norm"))
        if not (eps > 0 and math.isfinite(eps)):
            raise ConfigError(f"norm.eps must be positive, got {eps}")
        scale = float(_need(_need(cfg, "embedding", top), "scale", "embedding"))
        if not math.isfinite(scale):
            raise ConfigError(f"embedding.scale={scale}")
        cap = cfg.get("logit_softcap")
        if cap is not None and not (float(cap) > 0 and math.isfinite(float(cap))):
            raise ConfigError(f"logit_softcap={cap} must be positive")
        raw = _need(cfg, "layers", top)
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, lay in enumerate(raw):
            where = f"layers[{i}]"
            kind = _need(lay, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}: type={kind!r} is not implemented ({', '.join(MIXER_TYPES)} only)")
            mlp = lay.get("mlp")
            layers.append(TagelornLayer(kind, _MIXERS[kind].from_dict(_need(lay, "mixer", where), where + ".mixer"),
                                        TagelornMLP.from_dict(mlp, where + ".mlp") if mlp is not None else None))
        return cls(architecture=architecture, vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers),
                   max_position_embeddings=int(cfg.get("max_positions", 1 << 20)),
                   torch_dtype=str(cfg.get("torch_dtype") or cfg.get("dtype") or "bfloat16"),
                   norm_eps=eps, embedding_scale=scale, taps=_positive_int(_need(cfg, "canon", top), "taps", "canon"),
                   side_dim=_positive_int(_need(cfg, "token_side", top), "dim", "token_side"),
                   logit_softcap=float(cap) if cap is not None else None, layers=tuple(layers))

    def to_hf_dict(self) -> dict:
        out = {
            "architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
            "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "canon": {"taps": self.taps},
            "token_side": {"dim": self.side_dim},
            "layers": [{"type": lay.type, "mixer": lay.mixer.to_dict(),
                        "mlp": lay.mlp.to_dict() if lay.mlp is not None else None} for lay in self.layers],
            "torch_dtype": self.torch_dtype,
        }
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    @property
    def num_parameters(self) -> int:
        from ..models.causal_lm import build_model
        from ..models.tagelorn import tagelorn_spec

        total = 0
        for spec in build_model(tagelorn_spec(self)).tensor_specs().values():
            if spec.optional and spec.alias_of is not None:
                continue
            n = 1
            for e in spec.draw_shape or spec.shape:
                n *= e
            total += n
        return total
