"""Token embedding and the output head.

x[t] = E[ids[t]] (reference: pagedllm/model/llama.py:191, :197), times `scale` if a model gives one, plus a vector of
the position if the model names a position encoding that gives one (`SinusoidalEncoding`);
logits = h W^T in float32, where W is E itself if the head is tied
(llama.py:208-216).  A tied checkpoint may still carry the head's tensor; it is
then ignored, as tying means the embedding is used.  `softcap` c: logits become c * tanh(logits / c).
"""

from __future__ import annotations

import math

import torch

from .base import Embedding, Head, PositionEncoding, TensorSpec, register_embedding, register_head, register_position_encoding


@register_position_encoding("sinusoidal")
class SinusoidalEncoding(PositionEncoding):
    """A vector of sines and cosines per position: entry 2i is sin(p * base^(-2i / width)), entry 2i + 1 the cosine of the
    same.  Nothing is tabulated; the kernel that adds the vector forms it from `turns` (turns of the circle per position,
    double)."""

    def __init__(self, weights: dict[str, str], width: int, base: float = 10000.0):
        self.width, self.base = int(width), float(base)
        self.turns = None

    def prepare(self, max_positions, device, ops):
        i = torch.arange(0, self.width, 2, dtype=torch.float64)
        self.turns = (self.base ** (-i / self.width) / (2.0 * math.pi)).to(device)


@register_embedding("embedding")
class TokenEmbedding(Embedding):
    def __init__(self, weights: dict[str, str], vocab_size: int, hidden_size: int, scale: float = 1.0, streams: int = 1,
                 position=None):
        self.vocab_size, self.hidden_size, self.scale = vocab_size, hidden_size, float(scale)
        self.position = position
        if position is not None and (streams != 1 or position.width != hidden_size):
            raise ValueError(f"a position vector of {position.width} elements for a stream of {streams} x {hidden_size}")
        self.streams = int(streams)       # copies of the row laid side by side (a model of several residual streams)
        self.name = weights["weight"]
        self.weight = None

    def tensor_specs(self):
        return {self.name: TensorSpec((self.vocab_size, self.hidden_size))}

    def load(self, tensors):
        self.weight = tensors[self.name].contiguous()

    def forward(self, ids, ctx):
        if self.position is not None:
            return ctx.ops.embedding_sinusoid(self.weight, ids, self.scale, self.position.turns, ctx.positions)
        if self.streams > 1:
            return ctx.ops.embedding(self.weight, ids, self.scale, copies=self.streams)
        if self.scale != 1.0:
            return ctx.ops.embedding(self.weight, ids, self.scale)      # (the stream is float32: the product is too)
        return ctx.ops.embedding(self.weight, ids)


@register_head("lm_head")
class LMHead(Head):
    accepts_lazy_input = True

    def __init__(self, weights: dict[str, str], vocab_size: int, hidden_size: int, tied_to: str | None = None,
                 softcap: float | None = None):
        if softcap is not None and not softcap > 0:
            raise ValueError(f"softcap={softcap} must be positive")
        self.softcap = float(softcap) if softcap is not None else None
        self.vocab_size, self.hidden_size = vocab_size, hidden_size
        self.name = weights["weight"]
        self.tied_to = tied_to
        self.weight = None

    def tensor_specs(self):
        return {self.name: TensorSpec((self.vocab_size, self.hidden_size), optional=self.tied_to is not None,
                                      alias_of=self.tied_to)}

    def load(self, tensors):
        self.weight = (tensors[self.tied_to] if self.tied_to is not None else tensors[self.name]).contiguous()

    def bytes_read_per_step(self):
        return self.weight.numel() * self.weight.element_size()

    def forward(self, h, ctx):
        logits = ctx.ops.linear(h, self.weight, out_float32=True)
        return logits if self.softcap is None else ctx.ops.softcap(logits, self.softcap)
