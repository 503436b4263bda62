"""Selective state space mixer (the state-space duality form of Mamba-2): a matrix state per head with a decay that
depends on the token.

`W_in h` is laid out as [z: inner | x: inner | B: groups * state | C: groups * state | dt: heads], inner = heads *
value_dim. x, B and C together pass a short causal convolution per channel with a bias and then silu. Per head, with
group `g = h // (heads / groups)` and S (state x value_dim, zero at a request's start):

    dt  <- softplus(dt + dt_bias_h)
    S_t = exp(-exp(A_log_h) * dt) * S_(t-1) + dt * B_t,g x_t,h^T
    y_t = S_t^T C_t,g + D_h x_t,h

The heads' y side by side are multiplied by silu(z), then divided by their root mean square in `norm_groups` equal parts
(each part by its own, `eps` inside the root; the gate comes before the norm), times the weight `norm`, then the output
product. S (float32) and the convolution's last `taps - 1` inputs are request state. dt, its softplus, the decay and its
exponentials, the recurrence, the gate and the norm are 32-bit in both dtypes; the input product leaves float32; x, B and
C are rounded once, after their silu.
"""
from __future__ import annotations
import torch

from ..weights import ParamSpec
from .base import LayerCache, Mixer, register_mixer
from .short_conv import ShortConv

_NAMES = {"in": "in_proj", "conv": "conv", "conv_bias": "bias", "dt_bias": "dt_bias", "decay_log": "A_log", "skip": "D",
          "norm": "norm", "out": "out_proj"}


@register_mixer("mamba2")
class StateSpace(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state_dim: int, groups: int, taps: int,
                 norm_groups: int = 1, eps: float = 1e-6, names: dict | None = None):
        if num_heads % groups:
            raise ValueError(f"{num_heads} heads are not a multiple of {groups} groups")
        self.D, self.H, self.P, self.N, self.G = hidden_size, num_heads, value_dim, state_dim, groups
        self.inner = num_heads * value_dim
        if norm_groups <= 0 or self.inner % norm_groups:
            raise ValueError(f"{self.inner} channels cannot be normed in {norm_groups} equal parts")
        self.norm_groups, self.eps = int(norm_groups), float(eps)
        self.names = {**_NAMES, **(names or {})}
        self.C = self.inner + 2 * groups * state_dim                  # channels of [x | B | C]
        self.width = self.inner + self.C + num_heads
        self.conv = ShortConv(self.C, taps, name="", residual=False, activation="silu", bias=self.names["conv_bias"])
        self.w_in = self.wo = self.dt_bias = self.a_log = self.skip = self.norm_w = None

    def tensors(self) -> dict[str, ParamSpec]:
        n, H = self.names, self.H
        conv = {f"{n['conv']}.{k}" if k else n["conv"]: v for k, v in self.conv.tensors().items()}
        return {n["in"]: ParamSpec((self.width, self.D)), **conv, n["dt_bias"]: ParamSpec((H,), role="vector"),
                n["decay_log"]: ParamSpec((H,), role="vector"), n["skip"]: ParamSpec((H,), role="vector"),
                n["norm"]: ParamSpec((self.inner,), role="vector", init="ones"), n["out"]: ParamSpec((self.D, self.inner))}

    def bind(self, tensors, ops) -> None:
        n = self.names
        pre = n["conv"] + "."
        self.conv.bind({("" if k == n["conv"] else k[len(pre):]): v for k, v in tensors.items() if k == n["conv"] or k.startswith(pre)}, ops)
        self.w_in, self.wo = tensors[n["in"]], tensors[n["out"]]
        self.dt_bias, self.a_log, self.skip, self.norm_w = (tensors[n[k]].float().contiguous()
                                                            for k in ("dt_bias", "decay_log", "skip", "norm"))
        ops.check_ssd_scan(self.H, self.G, self.N, self.P)
        self.state_shape = ops.recurrent_state_shape(self.H, self.N, self.P)

    def children(self):
        return ((self.names["conv"], self.conv),)

    def step_needs(self) -> tuple[str, ...]:
        return ("portions",)      # single tokens, short and long portions take different kernels

    def state_need(self) -> dict:
        return {"S": self.state_shape, **self.conv.state_need()}

    def forward(self, ctx, h: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        n, ops, ws = h.shape[0], ctx.ops, ctx.ws
        proj = ws.get("ssm_in", (n, self.width), torch.float32)
        ops.linear(h, self.w_in, None, proj)
        xbc = self.conv.forward(ctx, proj, cache.state.get("conv"), tag="ssm_conv", offset=self.inner)
        y = ws.get("ssm_y", (n, self.inner), torch.float32)
        ops.ssd_scan(xbc, self.H, self.G, self.N, self.P, proj, self.inner + self.C, self.dt_bias, self.a_log, self.skip,
                     cache.state["S"], ctx.meta, y)
        u = ws.get("ssm_u", (n, self.inner), ops.dtype)
        ops.head_norm_gate(y, self.norm_groups, self.inner // self.norm_groups, self.norm_w, self.eps, proj, 0, "silu", u,
                           gate_first=True)
        delta = ws.get("ssm_delta", (n, self.D), torch.float32)
        ops.linear(u, self.wo, None, delta)
        return delta
