"""The generalized delta rule: a matrix state per head with a decay and a removal rate per key channel, both from the
input (the state transition of RWKV-7: Peng et al., "RWKV-7 Goose with Expressive Dynamic State Evolution").

    r = W_r h,  k = W_k h,  v = W_v h                                        [heads, dim]
    w = exp(decay_scale * sigmoid(W_2 tanh(W_1 h) + w_0))                    decay per head and key channel
    a = sigmoid(W_a h + b_a)                                                 removal rate per head and key channel
    u = k / sqrt(sum(k^2) + 1e-6)                                            per head
    S <- diag(w) S - (a u)(u^T S) + k v^T,   o = S^T r                       S: [dim, dim] per head, both terms from the old S
    out = W_o (concat_heads(rms_norm(o)) * n * sigmoid(W_g h))               the norm per head, n over all heads

The rank of W_1 and W_2 is the checkpoint's.  The state per request is float32, starts at zero and is carried from token
to token, so a request's tokens may arrive in portions of any size.  Sigmoids, the decay, the unit norm, the recurrence and
the norm behind it are float32 in both precisions.
"""

from __future__ import annotations

import math

import torch

from .base import FixedState, LazyLinear, Mixer, TensorSpec, register_mixer
from .delta_rule import UNIT_NORM_EPS

# the exponent of a decay lies between this and 0: no channel loses more than about 45 % of its state per token
DECAY_SCALE = -math.exp(-0.5)


def pad8(n: int) -> int:
    return -(-n // 8) * 8


@register_mixer("general_delta")
class GeneralDeltaRule(Mixer):
    accepts_lazy_input = False

    def __init__(self, weights: dict[str, str], hidden_size: int, num_heads: int, head_dim: int, eps: float,
                 decay_scale: float = DECAY_SCALE, unit_eps: float = UNIT_NORM_EPS, decay_rank: int = 32):
        if head_dim > 256:
            raise ValueError(f"heads of {head_dim}: the recurrence's kernels take at most 256")
        self.hidden_size, self.num_heads, self.head_dim, self.eps = hidden_size, num_heads, head_dim, float(eps)
        if not -4.0 <= decay_scale <= 0.0:
            raise ValueError(f"decay_scale={decay_scale}: the kernels for prompts take -4 to 0")
        self.decay_scale, self.unit_eps = float(decay_scale), float(unit_eps)
        self.decay_rank = int(decay_rank)           # what random weights are drawn with; a checkpoint's own shape rules
        self.names = weights
        self.w_in = self.w_decay = self.decay_bias = self.removal_bias = self.norm_w = self.w_o = None

    def cache_requirement(self):
        return FixedState((self.num_heads * self.head_dim * self.head_dim,))

    def tensor_specs(self):
        n, hid, c, r = self.names, self.hidden_size, self.num_heads * self.head_dim, self.decay_rank
        return {
            **{n[k]: TensorSpec((c, hid)) for k in ("r_proj", "k_proj", "v_proj", "g_proj", "removal_proj")},
            n["removal_bias"]: TensorSpec((c,), role="vector", init="norm_zero"),
            n["decay_down"]: TensorSpec((-1, hid), draw_shape=(r, hid)),
            n["decay_up"]: TensorSpec((c, -1), draw_shape=(c, r)),
            n["decay_bias"]: TensorSpec((c,), role="vector", init="norm_zero"),
            n["norm"]: TensorSpec((c,), role="vector", init="norm"),
            n["o_proj"]: TensorSpec((hid, c)),
        }

    def load(self, tensors):
        n = self.names
        down, up = tensors[n["decay_down"]], tensors[n["decay_up"]]
        if down.shape[0] != up.shape[1]:
            raise ValueError(f"{n['decay_down']} has {down.shape[0]} rows, {n['decay_up']} {up.shape[1]} columns")
        # one product for everything that reads the input: [r | k | v | g | removal | decay], the low rank and the whole
        # filled up with zero rows to multiples of 8 (tanh(0) = 0 meets zero columns)
        self.rank = pad8(down.shape[0])
        stack = [tensors[n[k]] for k in ("r_proj", "k_proj", "v_proj", "g_proj", "removal_proj")] + [down]
        rows = sum(t.shape[0] for t in stack)
        tail = pad8(rows - down.shape[0] + self.rank) - rows
        if tail:
            stack.append(torch.zeros((tail, self.hidden_size), dtype=down.dtype, device=down.device))
        self.w_in = torch.cat(stack, dim=0).contiguous()
        self.w_decay = torch.zeros((up.shape[0], self.rank), dtype=up.dtype, device=up.device)
        self.w_decay[:, :up.shape[1]] = up
        self.decay_bias = tensors[n["decay_bias"]].float().contiguous()
        self.removal_bias = tensors[n["removal_bias"]].float().contiguous()
        self.norm_w = tensors[n["norm"]].float().contiguous()
        self.w_o = tensors[n["o_proj"]].contiguous()

    def bytes_read_per_step(self):
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_decay, self.w_o))

    def forward(self, h, ctx, cache):
        ops = ctx.ops
        if any(slot < 0 for slot in ctx.host.state_slots):
            raise RuntimeError("a request of a model with per-request state runs without a state slot "
                               "(CacheManager.acquire_state_slot at its admission)")
        proj = ops.linear(h, self.w_in)                                       # [T, r | k | v | g | removal | decay | padding]
        out = ops.general_delta_mix(proj, self.rank, self.w_decay, self.decay_bias, self.removal_bias, self.num_heads, self.head_dim,
                                    self.decay_scale, self.unit_eps, self.norm_w, self.eps, cache.state, ctx)
        return LazyLinear(out, self.w_o)
