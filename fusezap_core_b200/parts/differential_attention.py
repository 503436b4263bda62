"""Differential attention over the paged cache: two softmax maps per head that read the same values.

Query head h and key head g hold two vectors of map_dim values each, [map 1 | map 2]; query head h reads key / value head
`h // (heads / kv_heads)`. Each map is causal attention of its own, `s_j = (q_i . k_j,i) * scale` for map i, over the values
of the head; with their results a1, a2 and one number lambda for the layer,

    o = a1 - lambda * a2,       o <- o / sqrt(mean(o^2) + eps) over value_dim, times (1 - start),
    lambda = exp(sum(l_q1 l_k1)) - exp(sum(l_q2 l_k2)) + start,

the heads are concatenated and the output product follows. No positions enter. `bias` names the products that have one (of
"q", "k", "v", "out"). One product with the rows [q; k; v] leaves float32; both maps' queries and keys, and the values, are
rounded once into the operands and the cache (a cached key has 2 map_dim values); scores, softmax, value sums, the
difference, its norm and lambda are 32-bit in both dtypes.
"""
from __future__ import annotations
import torch

from ..cache import KVNeed
from ..weights import ParamSpec
from .base import LayerCache, Mixer, register_mixer

_NAMES = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "out": "o_proj", "mix": ("lambda_q1", "lambda_k1", "lambda_q2", "lambda_k2")}


@register_mixer("differential_attention")
class DifferentialAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, map_dim: int, value_dim: int, scale: float,
                 start: float, eps: float = 1e-6, bias: tuple = (), bias_suffix: str = ".bias", names: dict | None = None):
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} query heads are not a multiple of {num_kv_heads} kv heads")
        if not set(bias) <= {"q", "k", "v", "out"}:
            raise ValueError(f"bias {bias!r} names something else than the q, k, v and out products")
        self.D, self.H, self.G, self.d, self.dv = hidden_size, num_heads, num_kv_heads, map_dim, value_dim
        self.scale, self.start, self.eps = float(scale), float(start), float(eps)
        self.bias, self.bias_suffix = tuple(bias), bias_suffix
        self.names = {**_NAMES, **(names or {})}
        self.wqkv = self.bqkv = self.wo = self.bo = self.lam = None

    def tensors(self) -> dict[str, ParamSpec]:
        n = self.names
        rows = {"q": self.H * 2 * self.d, "k": self.G * 2 * self.d, "v": self.G * self.dv, "out": self.D}
        out = {n["q"]: ParamSpec((rows["q"], self.D)), n["k"]: ParamSpec((rows["k"], self.D)), n["v"]: ParamSpec((rows["v"], self.D)),
               n["out"]: ParamSpec((self.D, self.H * self.dv))}
        out.update({n[x] + self.bias_suffix: ParamSpec((rows[x],), role="vector") for x in self.bias})
        out.update({name: ParamSpec((self.d,), role="vector") for name in n["mix"]})
        return out

    def bind(self, tensors, ops) -> None:
        n = self.names
        self.wqkv = torch.cat([tensors[n[x]] for x in ("q", "k", "v")], 0).contiguous()
        if set(self.bias) & {"q", "k", "v"}:
            self.bqkv = torch.cat([tensors[n[x] + self.bias_suffix].float() if x in self.bias else
                                   torch.zeros(tensors[n[x]].shape[0], dtype=torch.float32, device=self.wqkv.device)
                                   for x in ("q", "k", "v")], 0).contiguous()
        self.wo = tensors[n["out"]]
        self.bo = tensors[n["out"] + self.bias_suffix].float().contiguous() if "out" in self.bias else None
        q1, k1, q2, k2 = (tensors[name].float() for name in n["mix"])
        self.lam = (torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum()) + self.start).reshape(1).contiguous()
        ops.check_differential_attention(self.H, self.G, self.d, self.dv)

    def cache_need(self) -> KVNeed:
        # (keys and values of one size lie in halves of a page, as the paged attention's kernels want them)
        return KVNeed(self.G, 2 * self.d, 0, value_dim=0 if self.dv == 2 * self.d else self.dv)

    def step_needs(self) -> tuple[str, ...]:
        return ("portions",)      # its kernels tile the rows of portions: the longest portion is part of a step's shape

    def forward(self, ctx, h: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        n, ops, ws = h.shape[0], ctx.ops, ctx.ws
        H, G, d, dv = self.H, self.G, self.d, self.dv
        qkv = ws.get("diff_qkv", (n, self.wqkv.shape[0]), torch.float32)
        ops.linear(h, self.wqkv, self.bqkv, qkv)
        q = ws.get("diff_q", (n, H * 2 * d), ops.dtype)
        ops.rotate_kv_write(qkv, None, None, 0, 0, ctx.meta, cache, q, H, G, 2 * d, dv)
        o = ws.get("diff_out", (n, H * dv), ops.dtype)
        ops.differential_attention(q, cache, ctx.meta, o, H, G, d, dv, self.scale, self.lam, self.eps, 1.0 - self.start)
        delta = ws.get("diff_delta", (n, self.D), torch.float32)
        ops.linear(o, self.wo, self.bo, delta)
        return delta
