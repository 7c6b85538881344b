"""A feed-forward of routed experts.

z = W_r h in float32; the `top_k` experts with the largest z take the token, weighted by the
softmax over those top_k logits only; y = sum of weight * expert(h), each expert a gated
feed-forward down(act(gate h) * up h) without bias.  With `shared_size`, a shared expert of the
same form runs for every token and is added times sigmoid(w_s . h), one number per token.

Options: `scoring` "sigmoid": every expert scores s = sigmoid(z) by itself, the `top_k` largest scores choose, and the
weights are those scores as they are (not renormalised).  `groups` (count, keep): the experts form `count` equal groups
of neighbours, a group scores the sum of its `group_score_top` largest scores, and only experts of the `keep` best
groups can be chosen.  `activation` "swish_clamped" with `activation_limit` L: g = min(gate, L), u = clamp(up, -L, L),
the expert's inner vector is g * sigmoid(1.702 g) * (u + 1).  `scoring` "softmax": the scores are the softmax of z over
all experts.  `correction`: one learned number per expert joins its score for the choice (and in the groups' scores), not
for the weights.  `renorm`: the chosen scores are divided by their sum (+ 1e-20); `weight_scale` multiplies the weights.
`router_bias`: one learned number per expert is added to z (tensor `router_bias`), so it takes part in the choice and in the
softmax over the chosen.  `defer_sum`: the weighted sum is left to the norm that follows (`LazyExperts`).
`gated` False: an expert, and the shared one, is down(act(up h)) with the square of relu ("relu2") as act.  `shared_gate`
False: the shared expert is added as it is.

The experts' matrices are stacked when the weights are taken ([E, 2F, D] gate over up, and
[E, D, F]), the shared gate's row rides behind the router's, and the kernel library does the
rest on the device: no count per expert ever reaches the host, so a step may be captured.
"""

from __future__ import annotations

import torch

from .base import FeedForward, TensorSpec, register_feed_forward
from .mlp import ACTIVATIONS

EXPERT_ACTIVATIONS = ACTIVATIONS + ("swish_clamped",)
UNGATED_ACTIVATIONS = ("relu2",)


@register_feed_forward("routed_mlp")
class RoutedMLP(FeedForward):
    def __init__(self, weights: dict[str, str], hidden_size: int, expert_size: int, num_experts: int, top_k: int,
                 activation: str = "silu", shared_size: int | None = None, shared_activation: str | None = None,
                 activation_limit: float | None = None, scoring: str = "softmax_top", groups=None,
                 group_score_top: int = 2, gated: bool = True, shared_gate: bool = True, correction: bool = False,
                 renorm: bool = False, weight_scale: float = 1.0, router_bias: bool = False, defer_sum: bool = False):
        if not 1 <= top_k <= num_experts:
            raise ValueError(f"top_k={top_k} of {num_experts} experts")
        for a in (activation, shared_activation or activation):
            known = EXPERT_ACTIVATIONS if gated else UNGATED_ACTIVATIONS
            if a not in known:
                raise ValueError(f"activation {a!r} is not implemented ({', '.join(known)} only)")
        if activation == "swish_clamped" and not (activation_limit is not None and activation_limit > 0):
            raise ValueError("the clamped activation needs a positive activation_limit")
        if gated and shared_size is not None and (shared_activation or activation) not in ACTIVATIONS:
            raise ValueError(f"a shared expert takes the activations {', '.join(ACTIVATIONS)} only")
        if scoring not in ("softmax_top", "sigmoid", "softmax"):
            raise ValueError(f"scoring {scoring!r} is not implemented (softmax_top, sigmoid and softmax only)")
        if scoring == "softmax_top" and (correction or renorm or weight_scale != 1.0):
            raise ValueError("a correction, renormalised weights and their scale go with sigmoid and softmax scores")
        if router_bias and scoring != "softmax_top":
            raise ValueError("a bias on the router's logits goes with the softmax over the chosen logits")
        if defer_sum and shared_size is not None:
            raise ValueError("a shared expert is added where the experts' sum is formed: the sum cannot be deferred")
        self.has_router_bias, self.defer_sum, self.router_bias = bool(router_bias), bool(defer_sum), None
        if shared_size is not None and shared_gate and scoring != "softmax_top":
            raise ValueError("a shared expert's gate rides with the softmax over the chosen experts only")
        self.gated, self.shared_gate, self.has_correction = bool(gated), bool(shared_gate), bool(correction)
        self.renorm, self.weight_scale, self.correction = bool(renorm), float(weight_scale), None
        if groups is not None:
            count, keep = (int(g) for g in groups)
            if count < 1 or num_experts % count or not 1 <= keep <= count or top_k > num_experts // count * keep:
                raise ValueError(f"{num_experts} experts in {count} groups of which {keep} are kept, top_k={top_k}")
            if scoring == "softmax_top":
                raise ValueError("groups of experts are chosen by sigmoid or softmax scores")
            groups = (count, keep, int(group_score_top))
        self.activation_limit = float(activation_limit) if activation_limit is not None else 0.0
        self.scoring, self.groups = scoring, groups
        self.hidden_size, self.expert_size, self.num_experts, self.top_k = hidden_size, expert_size, num_experts, top_k
        self.activation, self.shared_size = activation, shared_size
        self.shared_activation = shared_activation or activation
        self.names = weights
        self.w_router = None          # [E (+1) and padding, D]: the router's rows, then the shared expert's gate
        self.w_gate_up = None         # [E, 2F, D]; without a gate [E, F, D]
        self.w_down = None            # [E, D, F]
        self.shared = None            # (gate over up [2Fs, D], down [D, Fs])

    def tensor_specs(self):
        d, f = self.hidden_size, self.expert_size
        out = {self.names["router"]: TensorSpec((self.num_experts, d))}
        for e in range(self.num_experts):
            if self.gated:
                out[self.names[f"e{e}.gate"]] = TensorSpec((f, d))
            out[self.names[f"e{e}.up"]] = TensorSpec((f, d))
            out[self.names[f"e{e}.down"]] = TensorSpec((d, f))
        if self.has_correction:
            out[self.names["correction"]] = TensorSpec((self.num_experts,), role="vector", init="norm_zero")
        if self.has_router_bias:
            out[self.names["router_bias"]] = TensorSpec((self.num_experts,), role="vector", init="norm_zero")
        if self.shared_size is not None:
            s = self.shared_size
            if self.gated:
                out[self.names["shared.gate"]] = TensorSpec((s, d))
            out[self.names["shared.up"]] = TensorSpec((s, d))
            out[self.names["shared.down"]] = TensorSpec((d, s))
            if self.shared_gate:
                out[self.names["shared.sg"]] = TensorSpec((1, d))
        return out

    def load(self, tensors):
        t, n, E = tensors, self.names, self.num_experts
        def first(prefix):          # what stands in front of the activation: gate over up, or up alone
            return torch.cat([t[n[prefix + "gate"]], t[n[prefix + "up"]]], dim=0) if self.gated else t[n[prefix + "up"]]

        self.w_gate_up = torch.stack([first(f"e{e}.") for e in range(E)]).contiguous()
        self.w_down = torch.stack([t[n[f"e{e}.down"]] for e in range(E)]).contiguous()
        router = [t[n["router"]]]
        if self.shared_size is not None:
            if self.shared_gate:
                router.append(t[n["shared.sg"]])
            self.shared = (first("shared.").contiguous(), t[n["shared.down"]].contiguous())
        if self.has_router_bias:
            self.router_bias = t[n["router_bias"]].float().contiguous()
        if self.has_correction:
            self.correction = t[n["correction"]].float().contiguous()
        rows = sum(r.shape[0] for r in router)
        if rows % 8:
            # rows of zeros up to a multiple of 8: the library's product of the logits then takes an aligned form
            router.append(torch.zeros((8 - rows % 8, self.hidden_size), dtype=router[0].dtype, device=router[0].device))
        self.w_router = torch.cat(router, dim=0).contiguous()

    def bytes_read_per_step(self):
        """A step of one token: the router, its top_k experts and the shared expert."""
        per_expert = (self.w_gate_up[0].numel() + self.w_down[0].numel()) * self.w_down.element_size()
        total = self.w_router.numel() * self.w_router.element_size() + self.top_k * per_expert
        if self.shared is not None:
            total += sum(w.numel() * w.element_size() for w in self.shared)
        return total

    def forward(self, h, ctx):
        return ctx.ops.routed_experts(h, self.w_router, self.w_gate_up, self.w_down, self.top_k, self.activation,
                                      shared=self.shared, shared_activation=self.shared_activation,
                                      activation_limit=self.activation_limit, scoring=self.scoring, groups=self.groups,
                                      **self._options())

    def _options(self) -> dict:
        out = {}
        if not self.gated:
            out["gated"] = False
        if self.router_bias is not None:
            out["router_bias"] = self.router_bias
        if self.defer_sum:
            out["defer_sum"] = True
        if self.shared is not None and not self.shared_gate:
            out["shared_gate"] = False
        if self.scoring != "softmax_top" and (self.correction is not None or self.renorm or self.weight_scale != 1.0):
            out.update(correction=self.correction, renorm=self.renorm, weight_scale=self.weight_scale)
        return out
