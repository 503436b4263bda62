"""Mixture of small gated feed-forwards chosen by a softmax router, with groups of experts and a shared expert.

Router logits `z = W_router h` leave the product in float32; scores `s = softmax(z)` over all experts. The experts form
`groups` equal groups of neighbours; a group's score is its largest score, and only experts of the best `keep_groups`
groups can be chosen. Of those the `top` with the largest scores are taken (the lower index first among equals); their
weights are their scores (divided by their sum if `renormalize`). Expert e: `W_down,e (silu(W_gate,e h) * (W_up,e h))`,
no biases. A shared expert of the same form (`shared_size` > 0) runs for every token and is added times
`sigmoid(W_sg h)`, one number per token. The step sorts its (row, choice) pairs by expert on the device and runs each
expert's products over its own rows only; a row's result does not depend on the other rows. Router, softmax, weights
and the weighted sum are 32-bit; the activation is computed from unrounded 32-bit sums.

Options: `router_bias`: the logits are `W_router h + b` (tensor `<router_bias>`); `shared_gate=False`: the shared expert
is added as it is, without a gate. With one group and `renormalize`, the weights are the softmax over the chosen logits
alone (softmax over all, divided by the chosen ones' sum, is the same number). `scoring` "sigmoid": s = sigmoid(z);
`correction`: experts and groups are chosen by `s + c` (tensor `<correction>`, one number per expert) while the weights
use s; `group_score` "top2": a group's score is the sum of its two largest choice scores (of its only one, if it has
one); `sum_eps` is added to the sum that `renormalize` divides by; `weight_scale` multiplies the weights last.
`alpha`, `limit`, `up_shift`: an expert computes g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit) and
`W_down (g * sigmoid(alpha g) * (u + up_shift))`; the defaults are silu(g) * u. The part takes a block's other term and
multiplier into its last kernel: `forward(ctx, h, add=a, scale=m)` returns `m * (a + ff(h))`. `activation` "relu2": experts
without a gate, `W_down max(W_up h, 0)^2`, and a shared expert of the same form. `identity` i: the router has i more outputs
than there are experts; they are scored and chosen with the others and stand for experts that hand the input on
(`correction` then has one number per output).
"""
from __future__ import annotations
import math

import torch

from ..weights import ParamSpec
from .base import FeedForward, register_feed_forward
from .feed_forward import SwiGLU, Ungated

_NAMES = {"router": "router", "expert": "experts.{}", "gate": "gate_proj", "up": "up_proj", "down": "down_proj",
          "shared": "shared_expert", "shared_gate": "shared_gate", "router_bias": "router.bias", "correction": "correction"}
SCORINGS = ("softmax", "sigmoid")
GROUP_SCORES = {"max": 1, "top2": 2}       # how many of a group's largest choice scores are added up


@register_feed_forward("routed_moe")
class RoutedMoE(FeedForward):
    takes_sum = True      # forward(ctx, h, add=, scale=): see `ParallelSharedBlock`

    def __init__(self, hidden_size: int, intermediate_size: int, num_experts: int, top: int, groups: int = 1,
                 keep_groups: int = 1, shared_size: int = 0, renormalize: bool = False, names: dict | None = None,
                 router_bias: bool = False, shared_gate: bool = True, scoring: str = "softmax", correction: bool = False,
                 group_score: str = "max", sum_eps: float = 0.0, weight_scale: float = 1.0, alpha: float = 1.0,
                 limit: float = math.inf, up_shift: float = 0.0, activation: str = "glu", identity: int = 0):
        outputs = num_experts + identity
        if not 0 < top <= outputs or identity < 0:
            raise ValueError(f"top {top} must lie in 1..{outputs}")
        if activation not in ("glu", "relu2"):
            raise ValueError(f"activation {activation!r} is not one of 'glu', 'relu2'")
        self.activation, self.identity, self.outputs = activation, int(identity), outputs
        if groups <= 0 or outputs % groups or not 0 < keep_groups <= groups or top > keep_groups * (outputs // groups):
            raise ValueError(f"{num_experts} experts in {groups} groups of which {keep_groups} are kept cannot give {top} choices")
        self.D, self.I, self.E, self.top = hidden_size, intermediate_size, num_experts, top
        self.groups, self.keep, self.renormalize = int(groups), int(keep_groups), bool(renormalize)
        self.names = {**_NAMES, **(names or {})}
        if scoring not in SCORINGS or group_score not in GROUP_SCORES:
            raise ValueError(f"scoring {scoring!r} / group_score {group_score!r} is not one of {SCORINGS} / {sorted(GROUP_SCORES)}")
        self.scoring, self.has_correction, self.group_top = scoring, bool(correction), GROUP_SCORES[group_score]
        self.sum_eps, self.weight_scale = float(sum_eps), float(weight_scale)
        self.alpha, self.limit, self.up_shift = float(alpha), float(limit), float(up_shift)
        self.correction = None
        self.router_bias, self.shared_gate = bool(router_bias), bool(shared_gate) and shared_size > 0
        self.b_router = None
        self.shared = None
        if shared_size:
            n = self.names
            self.shared = (SwiGLU(hidden_size, shared_size, names=(n["gate"], n["up"], n["down"]), suffix="") if activation == "glu" else
                           Ungated(hidden_size, shared_size, names=(n["up"], n["down"]), suffix="", activation=activation))
        self.w_router = self.w_gate_up = self.w_down = None

    def children(self):
        return ((self.names["shared"], self.shared),) if self.shared is not None else ()

    def _expert(self, e: int, which: str) -> str:
        return f"{self.names['expert'].format(e)}.{self.names[which]}"

    def tensors(self) -> dict[str, ParamSpec]:
        n, out = self.names, {}
        for e in range(self.E):
            if self.activation == "glu":
                out[self._expert(e, "gate")] = ParamSpec((self.I, self.D))
            out[self._expert(e, "up")] = ParamSpec((self.I, self.D))
            out[self._expert(e, "down")] = ParamSpec((self.D, self.I))
        out[n["router"]] = ParamSpec((self.outputs, self.D))
        if self.router_bias:
            out[n["router_bias"]] = ParamSpec((self.outputs,), role="vector")
        if self.has_correction:
            out[n["correction"]] = ParamSpec((self.outputs,), role="vector")
        if self.shared is not None:
            out.update({f"{n['shared']}.{k}": v for k, v in self.shared.tensors().items() if v.group is None})
            if self.shared_gate:
                out[f"{n['shared']}.{n['shared_gate']}"] = ParamSpec((1, self.D))
        return out

    def bind(self, tensors, ops) -> None:
        n, E = self.names, self.E
        first = ("gate", "up") if self.activation == "glu" else ("up",)
        self.w_gate_up = torch.stack([torch.cat([tensors[self._expert(e, x)] for x in first], 0)
                                      for e in range(E)]).contiguous()                  # (E, 2 I, D); ungated experts (E, I, D)
        self.w_down = torch.stack([tensors[self._expert(e, "down")] for e in range(E)]).contiguous()      # (E, D, I)
        router = tensors[n["router"]]
        if self.shared is not None:
            pre = n["shared"] + "."
            self.shared.bind({k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre)}, ops)
            if self.shared_gate:
                router = torch.cat([router, tensors[pre + n["shared_gate"]]], 0)        # one product: [router; shared gate]
        self.w_router = router.contiguous()
        if self.router_bias:
            b = tensors[n["router_bias"]].float()
            self.b_router = torch.cat([b, b.new_zeros(router.shape[0] - self.outputs)]).contiguous()
        if self.has_correction:
            self.correction = tensors[n["correction"]].float().contiguous()

    def weight_tensors(self) -> list:
        return [self.w_router, self.w_gate_up, self.w_down]

    def forward(self, ctx, h: torch.Tensor, add: torch.Tensor | None = None, scale: float = 1.0) -> torch.Tensor:
        n, ops, ws = h.shape[0], ctx.ops, ctx.ws
        z = ws.get("router_logits", (n, self.w_router.shape[0]), torch.float32)
        ops.linear(h, self.w_router, self.b_router, z)
        weights = ws.get("router_weights", (n, self.top), torch.float32)
        rule = {}
        if (self.scoring, self.has_correction, self.group_top, self.sum_eps, self.weight_scale) != ("softmax", False, 1, 0.0, 1.0):
            rule = {"scoring": self.scoring, "correction": self.correction, "group_top": self.group_top,
                    "sum_eps": self.sum_eps, "scale": self.weight_scale}
        if self.identity:
            rule["identity"] = self.identity
        route = ops.route_by_scores(z, self.outputs, self.top, self.groups, self.keep, self.renormalize, ctx.meta, weights,
                                    math.gcd(self.D, self.I), **rule)
        y = ws.get("moe_act", (n * self.top, self.I), ops.dtype)             # rows in the sorted order of the pairs
        if self.activation == "glu":
            ops.grouped_linear_glu(h, self.w_gate_up, route, y, self.alpha, self.limit, self.up_shift)
        else:
            ops.grouped_linear_act(h, self.w_gate_up, route, y, self.activation)
        terms = ws.get("moe_terms", (n * self.top, self.D), torch.float32)   # row n * top + k: the k-th expert of row n
        ops.grouped_linear_scatter(y, self.w_down, route, terms)
        shared = self.shared.forward(ctx, h, tag="shared_") if self.shared is not None else None
        out = ws.get("moe_delta", (n, self.D), torch.float32)
        gate = z if self.shared_gate else None
        options = {} if add is None and scale == 1.0 else {"add": add, "scale": scale}
        if self.identity:
            options["handed_on"] = (route, self.E, h)
        ops.moe_combine(terms, weights, shared, gate, self.outputs, out, **options)
        return out
