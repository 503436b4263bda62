"""Gated linear attention: linear attention whose state decays per head and key channel, by a number each token computes.

`q = W_q h * query_scale`, `k = W_k h` (num_heads x key_dim), `v = W_v h` (num_heads x value_dim). The decay is
`alpha = sigmoid(z)^(1 / decay_root)` with `z = W_a2 (W_a1 h) + b`, laid out num_heads x key_dim. Per head, with S (key_dim x
value_dim, float32, zero at a request's start, one per request and layer):

    S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t          (the decay acts on the rows of S)

Each head's o is divided by its root mean square over value_dim (`eps` inside the root), times the weight `norm` (value_dim,
shared by the heads), the heads are concatenated and multiplied by `gate`(W_g h), then the output product. One product with
the rows [q; k; v; gate; a1] leaves float32 and enters the recurrence unrounded; z, the decay, the recurrence, the state and
the norm are 32-bit in both dtypes; W_a1 h is rounded once to the activation dtype as the operand of the second product.
"""
from __future__ import annotations
import torch

from ..weights import ParamSpec
from .base import LayerCache, Mixer, register_mixer

_NAMES = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "gate": "g_proj", "decay_in": "a_down", "decay_out": "a_up",
          "norm": "norm", "out": "o_proj"}


@register_mixer("gated_linear_attention")
class GatedLinearAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, key_dim: int, value_dim: int, query_scale: float = 1.0,
                 decay_root: float = 1.0, eps: float = 1e-6, gate: str = "silu", names: dict | None = None,
                 bias_suffix: str = ".bias", low_rank: int = 0):
        """low_rank: the inner size of the two-step decay projection for writers of random weights (0: a sixteenth of the
        hidden size, at least 8); a checkpoint's own size is read from its tensors."""
        if not decay_root > 0:
            raise ValueError(f"the root of the decay must be positive, got {decay_root}")
        self.D, self.H, self.dk, self.dv = hidden_size, num_heads, key_dim, value_dim
        self.query_scale, self.decay_root, self.eps, self.gate = float(query_scale), float(decay_root), float(eps), gate
        self.names = {**_NAMES, **(names or {})}
        self.bias_name = self.names["decay_out"] + bias_suffix
        self.low_rank = int(low_rank) or max(8, hidden_size // 16)
        self.rank = 0
        self.w_in = self.w_decay = self.b_decay = self.wo = self.norm_w = None

    def tensors(self) -> dict[str, ParamSpec]:
        n, H, dk, dv, D, r = self.names, self.H, self.dk, self.dv, self.D, self.low_rank
        return {n["q"]: ParamSpec((H * dk, D)), n["k"]: ParamSpec((H * dk, D)), n["v"]: ParamSpec((H * dv, D)),
                n["gate"]: ParamSpec((H * dv, D)), n["decay_in"]: ParamSpec((-1, D), open=r),
                n["decay_out"]: ParamSpec((H * dk, -1), open=r), self.bias_name: ParamSpec((H * dk,), role="vector"),
                n["norm"]: ParamSpec((dv,), role="vector", init="ones"), n["out"]: ParamSpec((D, H * dv))}

    def bind(self, tensors, ops) -> None:
        n, H, dk, dv = self.names, self.H, self.dk, self.dv
        a1, a2 = tensors[n["decay_in"]], tensors[n["decay_out"]]
        self.rank = a1.shape[0]
        if a2.shape[1] != self.rank:
            raise ValueError(f"the two steps of the decay projection do not fit: {tuple(a1.shape)} -> {tuple(a2.shape)}")
        # one product for everything that reads h: columns [q | k | v | gate | decay step one]
        self.w_in = torch.cat([tensors[n[x]] for x in ("q", "k", "v", "gate")] + [a1], 0).contiguous()
        self.off_gate = H * (2 * dk + dv)
        self.off_low = self.off_gate + H * dv
        self.w_decay = a2.contiguous()
        self.b_decay = tensors[self.bias_name].float().contiguous()
        self.norm_w = tensors[n["norm"]].float().contiguous()
        self.wo = tensors[n["out"]]
        self.state_shape = ops.recurrent_state_shape(H, dk, dv)
        ops.check_chunked_scan(H, dk, dv)

    def state_need(self) -> dict:
        return {"S": self.state_shape}

    def step_needs(self) -> tuple[str, ...]:
        return ("portions",)      # which scan runs depends on the longest portion, which is then part of a step's shape

    def forward(self, ctx, h: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        n, ops, ws = h.shape[0], ctx.ops, ctx.ws
        H, dk, dv = self.H, self.dk, self.dv
        proj = ws.get("gla_proj", (n, self.off_low + self.rank), torch.float32)
        ops.linear(h, self.w_in, None, proj)
        low = ws.get("gla_low", (n, self.rank), ops.dtype)
        ops.activate(proj, self.off_low, "identity", low)
        z = ws.get("gla_decay", (n, H * dk), torch.float32)
        ops.linear(low, self.w_decay, self.b_decay, z)
        o = ws.get("gla_o", (n, H * dv), torch.float32)
        ops.channel_decay_scan(proj, H, dk, dv, z, self.decay_root, self.query_scale, cache.state["S"], ctx.meta, o)
        y = ws.get("gla_y", (n, H * dv), ops.dtype)
        ops.head_norm_gate(o, H, dv, self.norm_w, self.eps, proj, self.off_gate, self.gate, y)
        delta = ws.get("gla_delta", (n, self.D), torch.float32)
        ops.linear(y, self.wo, None, delta)
        return delta
