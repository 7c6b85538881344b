"""Typed configuration of the Nopozen decoder, read from a checkpoint's config.json.

config.json gives every size and every constant that may differ between models of the design:

    architecture  "Nopozen"
    vocab, width  vocabulary and width of the residual stream
    norm.eps      epsilon of every RMS norm
    layers        one entry per layer: `type` (the mixer), `mixer` (its sizes and constants) and `mlp` (null for none)
    loop          {start, stop, times}: layers start .. stop-1 run `times` times in a row with the same weights, and every
                  pass begins by joining the stream with the embedding's output (absent: every layer runs once)

Mixers by `type`:

    "attention"    heads, kv_heads, dim (query/key head), vdim (value head), scale, rot {base, dims, scaling {factor, low,
                   high, original} (absent: none)}, mask {size (the chunk)} (absent: every earlier token is seen)
    "attention_2"  heads, kv_heads, dim, vdim, scale, rot, conv (taps of the convolution on queries, keys and values)
    "lightning"    heads, dim, vdim, decay (one factor per head)

Feed-forwards by `mlp.kind`:

    "dense"        ff
    "moe"          expert {ff}, router {experts, top}

What the engine does not compute is refused here with a message, never computed wrongly.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

from .model import ConfigError, ModelConfig
from .pirerax import _heads, _scale
from .rokarax import _need, _positive_int

MIXER_TYPES = ("attention", "attention_2", "lightning")


@dataclass(frozen=True)
class NopozenRotary:
    dims: int
    base: float
    scaling: tuple | None = None         # (factor, low, high, original)

    @classmethod
    def from_dict(cls, d: dict, head_dim: int, where: str) -> "NopozenRotary":
        dims, base = int(_need(d, "dims", where)), float(_need(d, "base", where))
        if dims < 2 or dims % 2 or dims > head_dim:
            raise ConfigError(f"{where}: dims={dims} must be even and at most the head size {head_dim}")
        if not (base > 0 and math.isfinite(base)):
            raise ConfigError(f"{where}: base={base} must be positive")
        sc = d.get("scaling")
        if sc is not None:
            sc = tuple(float(_need(sc, k, where + ".scaling")) for k in ("factor", "low", "high", "original"))
            if not all(v > 0 and math.isfinite(v) for v in sc) or sc[1] > sc[2]:
                raise ConfigError(f"{where}.scaling: factor, low, high and original must be positive, and low at most high")
        return cls(dims, base, sc)

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"dims": self.dims, "base": self.base}
        if self.scaling is not None:
            d["scaling"] = dict(zip(("factor", "low", "high", "original"), self.scaling))
        return d


def _rotary(d: dict, dim: int, where: str) -> NopozenRotary | None:
    rot = d.get("rot")
    return NopozenRotary.from_dict(rot, dim, where + ".rot") if rot is not None else None


def _value_dim(d: dict, dim: int, where: str) -> int:
    return _positive_int(d, "vdim", where) if "vdim" in d else dim


@dataclass(frozen=True)
class NopozenAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: NopozenRotary | None = None
    chunk: int | None = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "NopozenAttention":
        heads, kv = _heads(d, where)
        dim = _positive_int(d, "dim", where)
        mask = d.get("mask")
        chunk = _positive_int(mask, "size", where + ".mask") if mask is not None else None
        return cls(heads, kv, dim, _value_dim(d, dim, where), _scale(d, where), _rotary(d, dim, where), chunk)

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.chunk is not None:
            d["mask"] = {"size": self.chunk}
        return d


@dataclass(frozen=True)
class NopozenConvolvedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    taps: int
    rot: NopozenRotary | None = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "NopozenConvolvedAttention":
        if d.get("mask") is not None:
            raise ConfigError(f"{where}: a mask goes with the mixer 'attention' only")
        heads, kv = _heads(d, where)
        dim = _positive_int(d, "dim", where)
        return cls(heads, kv, dim, _value_dim(d, dim, where), _scale(d, where), _positive_int(d, "conv", where), _rotary(d, dim, where))

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                             "conv": self.taps}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class NopozenLightning:
    heads: int
    dim: int
    vdim: int
    decay: tuple

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "NopozenLightning":
        heads, dim = _positive_int(d, "heads", where), _positive_int(d, "dim", where)
        decay = tuple(float(v) for v in _need(d, "decay", where))
        if len(decay) != heads or not all(0.0 <= v <= 1.0 for v in decay):
            raise ConfigError(f"{where}: decay needs {heads} factors between 0 and 1, got {list(decay)}")
        return cls(heads, dim, _value_dim(d, dim, where), decay)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


_MIXERS = {"attention": NopozenAttention, "attention_2": NopozenConvolvedAttention, "lightning": NopozenLightning}


@dataclass(frozen=True)
class NopozenMLP:
    kind: str
    ff: int
    experts: int = 0
    top: int = 0

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "NopozenMLP":
        kind = _need(d, "kind", where)
        if kind == "dense":
            return cls(kind, _positive_int(d, "ff", where))
        if kind != "moe":
            raise ConfigError(f"{where}: kind={kind!r} is not implemented (dense and moe only)")
        ro = _need(d, "router", where)
        experts, top = _positive_int(ro, "experts", where + ".router"), _positive_int(ro, "top", where + ".router")
        if top > experts:
            raise ConfigError(f"{where}.router: top={top} of {experts} experts")
        return cls(kind, _positive_int(_need(d, "expert", where), "ff", where + ".expert"), experts, top)

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class NopozenLayer:
    type: str
    mixer: Any
    mlp: NopozenMLP | None


@dataclass(frozen=True)
class NopozenConfig(ModelConfig):
    norm_eps: float = 1e-6
    layers: tuple = ()
    loop: tuple | None = None            # (start, stop, times)

    @classmethod
    def from_hf_dict(cls, cfg: dict[str, Any], architecture: str = "Nopozen") -> "NopozenConfig":
        top = "the top level"
        vocab, width = _positive_int(cfg, "vocab", top), _positive_int(cfg, "width", top)
        eps = float(_need(_need(cfg, "norm", top), "eps", "norm"))
        if not (eps > 0 and math.isfinite(eps)):
            raise ConfigError(f"norm.eps must be positive, got {eps}")
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
            layers.append(NopozenLayer(kind, _MIXERS[kind].from_dict(_need(lay, "mixer", where), where + ".mixer"),
                                       NopozenMLP.from_dict(mlp, where + ".mlp") if mlp is not None else None))
        loop = cfg.get("loop")
        if loop is not None:
            loop = tuple(int(_need(loop, k, "loop")) for k in ("start", "stop", "times"))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"loop start={loop[0]} stop={loop[1]} times={loop[2]} does not fit {len(layers)} layers")
        return cls(architecture=architecture, vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers),
                   max_position_embeddings=int(cfg.get("max_positions", 1 << 20)),
                   torch_dtype=str(cfg.get("torch_dtype") or cfg.get("dtype") or "bfloat16"),
                   norm_eps=eps, layers=tuple(layers), loop=loop)

    def to_hf_dict(self) -> dict:
        out: dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
            "layers": [{"type": lay.type, "mixer": lay.mixer.to_dict(),
                        "mlp": lay.mlp.to_dict() if lay.mlp is not None else None} for lay in self.layers],
            "torch_dtype": self.torch_dtype,
        }
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def layer_runs(self) -> list[tuple[int, bool]]:
        """(layer, whether a pass of the loop begins with it) in the order in which the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b, times = self.loop
        one_pass = [(i, i == a) for i in range(a, b)]
        return [(i, False) for i in range(a)] + one_pass * times + [(i, False) for i in range(b, n)]

    @property
    def num_parameters(self) -> int:
        from ..models.causal_lm import build_model
        from ..models.nopozen import nopozen_spec

        total = 0
        for spec in build_model(nopozen_spec(self)).tensor_specs().values():
            n = 1
            for e in spec.draw_shape or spec.shape:
                n *= e
            total += n
        return total
