"""Plain, slow Gimupel: one function per mechanism, written from the design's equations in 64-bit, whole sequences,
token by token where the design is a recurrence. It shares no code with the package (only the tensor names and the keys
of config.json, which are the design's own).

A model is (config dict, {tensor name: float64 tensor}). `forward(config, tensors, tokens)` returns the logits of every
position, and with `layers=True` also the residual stream after every layer that ran. Inside `with rounded_operands():`
what a 16-bit engine hands to its matrix products, its cache and its scan is rounded to bfloat16 on the way, which shows
how far rounding alone moves the logits.
"""
from __future__ import annotations
import contextlib
import math

import torch

F = torch.float64
GATE_SHARPNESS = 1.702       # an expert's gate: g * sigmoid(1.702 g)
SUM_EPS = 1e-20              # added to the sum of the chosen scores


_rounding = False


@contextlib.contextmanager
def rounded_operands():
    global _rounding
    _rounding = True
    try:
        yield
    finally:
        _rounding = False


def R(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).to(x.dtype) if _rounding else x


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """Mean taken off, divided by the root of the mean squared deviation, times a weight; no bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


# ---- the state-space mixer
def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x: (T, C), w: (C, taps). The last column multiplies the token's own input; zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] += w[:, j] * x[src]
        y[t] += b
    return y


def ssd_recurrence(x, B, C, dt, a_log, D):
    """x: (T, H, P); B, C: (T, G, N); dt: (T, H) after the softplus. Head h reads group h // (H / G):
    S_t = exp(-exp(a_log) dt) S_(t-1) + dt B_t x_t^T (N x P), y_t = S_t^T C_t + D x_t. Returns y and the last state."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            decay = torch.exp(-torch.exp(a_log[h]) * dt[t, h])
            S[h] = decay * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def ssd_recurrence_fast(x, B, C, dt, a_log, D):
    """The same, all heads of a token at once (for the longer sequences of the tests)."""
    T, H, P = x.shape
    rep = H // B.shape[1]
    Bh, Ch = B.repeat_interleave(rep, 1), C.repeat_interleave(rep, 1)
    decay = torch.exp(-torch.exp(a_log) * dt)
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype)
    y = torch.empty_like(x)
    for t in range(T):
        S = decay[t][:, None, None] * S + (dt[t][:, None] * Bh[t])[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, Ch[t])
    return y + D[:, None] * x, S


def gated_norm(y: torch.Tensor, z: torch.Tensor, groups: int, eps: float, w: torch.Tensor) -> torch.Tensor:
    """The gate silu(z) first, then every one of `groups` equal parts by its own root mean square, then the weight."""
    u = y * silu(z)
    return rms(u.reshape(u.shape[0], groups, -1), eps).reshape(u.shape) * w


def state_space(cfg: dict, w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    T, H, P, G, N = h.shape[0], m["heads"], m["vdim"], m["groups"], m["state"]
    inner = H * P
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner: 2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = R(silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])))
    x, B, C = xbc[:, :inner], xbc[:, inner: inner + G * N], xbc[:, inner + G * N:]
    dt = softplus(dt + w[p + "dt_bias"])
    y, _ = ssd_recurrence_fast(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, w[p + "A_log"], w[p + "D"])
    return R(gated_norm(y.reshape(T, inner), z, m["norm_groups"], cfg["norm"]["eps"], w[p + "norm"])) @ w[p + "o"].T


# ---- attention
def window_mask(T: int, size: int) -> torch.Tensor:
    """mask[i, j]: position i sees key j, 0 <= i - j < size."""
    i = torch.arange(T)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size)


def masked_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, visible) -> torch.Tensor:
    """q: (T, H, d), k: (T, H, d), v: (T, H, dv), already per query head. `visible(i, j)`: does position i see key j."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(T) if visible(i, j)]
        for h in range(H):
            s = torch.stack([(q[i, h] * k[j, h]).sum() * scale for j in js])
            e = torch.exp(s - s.max())
            out[i, h] = sum(e[n] * v[j, h] for n, j in enumerate(js)) / e.sum()
    return out


def masked_attention_fast(q, k, v, scale, mask):
    """The same with the mask as a (T, T) boolean matrix, vectorised."""
    s = (torch.einsum("ihd,jhd->hij", q, k) * scale).masked_fill(~mask[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def attention(cfg: dict, w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv, eps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], cfg["norm"]["eps"]
    q = R(rms((h @ w[p + "q"].T).view(T, H, d), eps))
    k = R(rms((h @ w[p + "k"].T).view(T, G, d), eps))
    v = R((h @ w[p + "v"].T).view(T, G, dv))
    o = masked_attention_fast(q, k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1), m["scale"],
                              window_mask(T, m["mask"]["size"]))
    return R(o.reshape(T, H * dv)) @ w[p + "o"].T


# ---- feed-forward
def dense(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return R(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(w: dict, p: str, h: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return R(g * sigmoid(GATE_SHARPNESS * g) * (u + 1.0)) @ w[p + "down"].T


def route(z: torch.Tensor, correction: torch.Tensor, top: int, groups: int, keep: int, scale: float):
    """Row by row: scores sigmoid(z); choice scores with the correction; groups of neighbours by the sum of their two
    largest choice scores (a group of one: that one); the `top` largest choice scores within the kept groups; weights:
    the scores themselves, divided by their sum, times scale."""
    idx, wts = [], []
    for row in z:
        s = sigmoid(row)
        c = s + correction
        E = c.shape[0]
        per = E // groups
        value = [sum(sorted(c[g * per: (g + 1) * per].tolist(), reverse=True)[:2]) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: (-value[g], g))[:keep]
        allowed = [e for e in range(E) if e // per in kept]
        chosen = sorted(allowed, key=lambda e: (-float(c[e]), e))[:top]
        total = sum(s[e] for e in chosen) + SUM_EPS
        idx.append(chosen)
        wts.append(torch.stack([s[e] / total * scale for e in chosen]))
    return torch.tensor(idx), torch.stack(wts)


def mixture(w: dict, p: str, mlp: dict, h: torch.Tensor) -> torch.Tensor:
    r = mlp["router"]
    idx, wt = route(h @ w[p + "router"].T, w[p + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"])
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=h.dtype)
    for e in range(r["experts"]):
        rows, n = torch.nonzero(idx == e, as_tuple=True)
        if len(rows):
            out[rows] += wt[rows, n][:, None] * expert(w, f"{p}e{e}.", h[rows], mlp["expert"]["limit"])
    return out


# ---- the whole model
def order_of_layers(cfg: dict) -> list:
    """(layer, whether the embedding output is added to x right before it)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for turn in range(loop["times"]):
        out += [(i, turn > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def forward(cfg: dict, w: dict, tokens: list[int], layers: bool = False):
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = x0
    streams = []
    for n, again in order_of_layers(cfg):
        L, p = cfg["layers"][n], f"l{n}."
        if again:
            x = x + x0
        h = R(layer_norm(x, w[p + "norm1"], eps))
        mixer = attention if L["type"] == "attention" else state_space
        x = x + mixer(cfg, w, p + "mix.", L["mixer"], h)
        if L.get("mlp") is not None:
            h = R(layer_norm(x, w[p + "norm2"], eps))
            x = x + (dense(w, p + "mlp.", h) if L["mlp"]["kind"] == "dense" else mixture(w, p + "mlp.", L["mlp"], h))
        streams.append(x)
    logits = R(layer_norm(x, w["final.norm"], eps)) @ w["embed"].T
    return (logits, torch.stack(streams)) if layers else logits
