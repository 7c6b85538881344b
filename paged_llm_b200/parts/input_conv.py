"""A causal convolution over time in front of any mixer: the mixer reads h + conv(h) in place of h.

    conv(h)_t = sum_j w[:, j] * h_(t - taps + 1 + j)          per channel, zeros before the start, no bias, no activation

The mixer behind it is an ordinary one, named by registry key; what it keeps per request (pages of keys and values, a
state of fixed size, nothing) is joined by the last taps - 1 inputs h, float32, in a state slot.  So the cache requirement
is the pair of both and each gets its own view (`cache.parts`).
"""

from __future__ import annotations

from .base import MIXERS, FixedState, Mixer, PartSpec, TensorSpec, make_part, register_mixer


@register_mixer("input_convolution")
class InputConvolution(Mixer):
    accepts_lazy_input = False

    def __init__(self, weights: dict[str, str], hidden_size: int, taps: int, mixer: PartSpec):
        if taps < 1:
            raise ValueError(f"taps={taps}")
        self.hidden_size, self.taps = int(hidden_size), int(taps)
        self.mixer = make_part(MIXERS, "mixer", mixer)
        self.name = weights["conv"]
        self.conv_w = None              # [taps, hidden] float32: the weights of a tap side by side

    @property
    def capturable(self):
        return self.mixer.capturable

    def cache_requirement(self):
        mine = FixedState(((self.taps - 1) * self.hidden_size,)) if self.taps > 1 else None
        return (mine, self.mixer.cache_requirement())

    def attention_plan_key(self):
        return getattr(self.mixer, "attention_plan_key", lambda: None)()

    def tensor_specs(self):
        return {self.name: TensorSpec((self.hidden_size, self.taps), role="vector"), **self.mixer.tensor_specs()}

    def load(self, tensors):
        self.conv_w = tensors[self.name].float().t().contiguous()
        self.mixer.load(tensors)

    def bytes_read_per_step(self):
        return self.conv_w.numel() * 4 + self.mixer.bytes_read_per_step()

    def forward(self, h, ctx, cache):
        mine, inner = cache.parts
        if mine is not None and any(slot < 0 for slot in ctx.host.state_slots):
            raise RuntimeError("a request of a model with per-request state runs without a state slot "
                               "(CacheManager.acquire_state_slot at its admission)")
        h = ctx.ops.residual_conv(h, self.conv_w, mine.state if mine is not None else None, ctx)
        if not self.mixer.accepts_lazy_input:
            h = ctx.ops.materialize(h)
        return self.mixer.forward(h, ctx, inner)
