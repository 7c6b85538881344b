"""Grouped-query attention over the paged cache behind a short convolution over time.

    q = conv(W_q h), k = conv(W_k h), v = conv(W_v h)      per channel, causal, `taps` wide, no bias, no activation:
        conv(u)_t = sum_j w[:, j] * u_(t - taps + 1 + j)   zeros before the sequence's start
    q and k rotated (`position`), k and v cached, attention, a sigmoid gate per element (or head), the output projection

The last taps - 1 projected values of a request, float32, live in a state slot beside its pages, so the cache requirement is
the pair of both and each gets its own view (`cache.parts`).  `sink_score`: the softmax counts one key more, with this score
and no value (0: 1 joins the denominator).  Projections have no biases and nothing is normed.  Everything else is
`GatedAttention`."""

from __future__ import annotations

import torch

from .attention import GatedAttention
from .base import FixedState, TensorSpec, register_mixer


@register_mixer("convolved_attention")
class ConvolvedAttention(GatedAttention):
    def __init__(self, weights: dict[str, str], hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int,
                 scale: float, eps: float, taps: int, position=None, gate: "bool | str" = True, sink_score: float | None = None,
                 window: int | None = None, chunk: int | None = None):
        # (`head_norm` keeps the norms over whole projections and their weights away; the front is this class's own)
        super().__init__(weights, hidden_size, num_heads, num_kv_heads, head_dim, value_dim, scale, eps, window=window, chunk=chunk,
                         gate=gate, position=position, head_norm=True)
        if taps < 1:
            raise ValueError(f"taps={taps}")
        self.taps = int(taps)
        self.channels = num_heads * head_dim + num_kv_heads * (head_dim + value_dim)
        self.sink_score = float(sink_score) if sink_score is not None else None
        self.conv_w = None              # [taps, channels] float32: the weights of a tap side by side

    def cache_requirement(self):
        mine = FixedState(((self.taps - 1) * self.channels,)) if self.taps > 1 else None
        return (mine, super().cache_requirement())

    def tensor_specs(self):
        out = super().tensor_specs()
        for k in ("q", "k", "v"):
            out[self.names[k + "_conv"]] = TensorSpec((out[self.names[k + "_proj"]].shape[0], self.taps), role="vector")
        return out

    def load(self, tensors):
        super().load(tensors)
        self.conv_w = torch.cat([tensors[self.names[k + "_conv"]].float() for k in ("q", "k", "v")], dim=0).t().contiguous()
        if self.sink_score is not None:
            self.sink = torch.full((self.num_heads,), self.sink_score, dtype=torch.float32, device=self.w_o.device)

    def bytes_read_per_step(self):
        return super().bytes_read_per_step() + self.conv_w.numel() * 4

    def forward(self, h, ctx, cache):
        mine, pages = cache.parts
        if mine is not None and any(slot < 0 for slot in ctx.host.state_slots):
            raise RuntimeError("a request of a model with per-request state runs without a state slot "
                               "(CacheManager.acquire_state_slot at its admission)")
        block_table = ctx.block_tables[pages.group]
        proj = ctx.ops.linear(h, self.w_in)
        q = ctx.ops.conv_qkv_write(proj, self.conv_w, self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, self.cache_dim,
                                   self.position, mine.state if mine is not None else None, ctx, pages.kv, block_table, write=pages.owner)
        return self._attend(q, proj, ctx, pages, block_table)
