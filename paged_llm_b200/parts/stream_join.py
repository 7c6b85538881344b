"""A linear join of the stream with the embedding's output: x <- W [x; x0], W [hidden, 2 hidden], x first.

W x0 is the same in every pass of a step, so it is formed once (float32); a pass then runs W's left half only, as a branch
of a stream that starts at W x0: the norm that follows adds both in its own kernel."""

from __future__ import annotations

import torch

from .base import LazyLinear, StreamJoin, TensorSpec, register_stream_join


@register_stream_join("linear_join")
class LinearJoin(StreamJoin):
    def __init__(self, weights: dict[str, str], hidden_size: int):
        self.hidden_size, self.name = hidden_size, weights["weight"]
        self.w_stream = self.w_embedding = None

    def tensor_specs(self):
        return {self.name: TensorSpec((self.hidden_size, 2 * self.hidden_size))}

    def load(self, tensors):
        w = tensors[self.name]
        self.w_stream = w[:, :self.hidden_size].contiguous()
        self.w_embedding = w[:, self.hidden_size:].contiguous()

    def bytes_read_per_step(self):
        return self.w_stream.numel() * self.w_stream.element_size()

    def start(self, x0, times, ctx):
        ops = ctx.ops
        base = ops.linear(ops.stream_copy(x0), self.w_embedding, out_float32=True)
        # (each pass sums its stream up in place)
        return [base.clone() for _ in range(times - 1)] + [base]

    def forward(self, x, pending, shared, ctx):
        ops = ctx.ops
        return shared.pop(0), LazyLinear(ops.add_copy(x, pending), self.w_stream, float32=True)
