"""Plain, slow Muretar: one function per mechanism, written from the design's equations in 64-bit, whole sequences, token
by token where the design is a recurrence. It shares no code with the package (only the tensor names and the keys of
config.json, which are the design's own).

A model is (config dict, {tensor name: float64 tensor}). `forward(config, tensors, tokens)` returns the logits of every
position, and with `layers=True` also the residual stream after every layer that ran. Inside `with rounded_operands():`
what a 16-bit engine hands to its matrix products, its cache and its scans is rounded to bfloat16 on the way, which shows
how far rounding alone moves the logits.
"""
from __future__ import annotations
import contextlib
import math

import torch

UNIT_EPS = 1e-6              # inside the root of the delta rule's unit vectors
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


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    """Mean taken off, divided by the root of the mean squared deviation, times a weight, plus a bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def norm(w: dict, name: str, x: torch.Tensor, eps: float) -> torch.Tensor:
    return layer_norm(x, w[name], w[name + ".b"], eps)


def product(w: dict, name: str, h: torch.Tensor, bias: bool = False) -> torch.Tensor:
    y = h @ w[name].T
    return y + w[name + ".b"] if bias else y


# ---- attention
def rotate(x: torch.Tensor, dims: int, base: float, factor: float) -> torch.Tensor:
    """x: (T, heads, d), row t at position t. Dimensions 2i and 2i + 1 of the first `dims` are turned by the angle
    t * base^(-2i / dims) / factor."""
    out = x.clone()
    for i in range(dims // 2):
        f = base ** (-2 * i / dims) / factor
        a = torch.arange(x.shape[0], dtype=torch.float64) * f
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q: (T, H, d), k: (T, H, d), v: (T, H, dv), already per query head; position i sees j <= i."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        for h in range(H):
            s = torch.stack([(q[i, h] * k[j, h]).sum() * scale for j in range(i + 1)])
            e = torch.exp(s - s.max())
            out[i, h] = sum(e[j] * v[j, h] for j in range(i + 1)) / e.sum()
    return out


def causal_attention_fast(q, k, v, scale):
    """The same, vectorised."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1)[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def mixing_number(lq1, lk1, lq2, lk2, diff: float) -> torch.Tensor:
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def combine_maps(a1: torch.Tensor, a2: torch.Tensor, lam: torch.Tensor, diff: float, eps: float) -> torch.Tensor:
    """(T, H, dv) each: the difference, every head by its own root mean square, times what `diff` leaves of one."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(cfg: dict, w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = R(product(w, p + "q", h, True)).view(T, H, 2, d)
    k = R(product(w, p + "k", h, True)).view(T, G, 2, d).repeat_interleave(H // G, 1)
    v = R(product(w, p + "v", h, True)).view(T, G, dv).repeat_interleave(H // G, 1)
    a = [causal_attention_fast(q[:, :, i], k[:, :, i], v, m["scale"]) for i in (0, 1)]
    lam = mixing_number(*(w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    o = combine_maps(a[0], a[1], lam, m["diff"], cfg["norm"]["eps"])
    return R(o.reshape(T, H * dv)) @ w[p + "o"].T


def rotary_attention(w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    factor = rot["scaling"]["factor"] if rot.get("scaling") else 1.0
    q = R(rotate(product(w, p + "q", h, True).view(T, H, d), rot["dims"], rot["base"], factor))
    k = R(rotate(product(w, p + "k", h, True).view(T, G, d), rot["dims"], rot["base"], factor))
    v = R(product(w, p + "v", h, True).view(T, G, dv))
    o = causal_attention_fast(q, k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1), m["scale"])
    return product(w, p + "o", R(o.reshape(T, H * dv)), True)


# ---- the gated delta rule
def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x: (T, C), w: (C, taps). The last column multiplies the token's own input; zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] += w[:, j] * x[src]
    return y


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_recurrence(q, k, v, g, beta):
    """q, k: (T, H, d); v: (T, H, dv); g, beta: (T, H). Returns the read-outs (T, H, dv) and the last state (H, d, dv)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + torch.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def delta_recurrence_fast(q, k, v, g, beta):
    """The same, all heads of a token at once."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.empty_like(v)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def gated_delta(cfg: dict, w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (R(silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"]))) for n in ("q", "k", "v"))
    q = (unit(q.view(T, G, d)) * d ** -0.5).repeat_interleave(H // G, 1)
    k = unit(k.view(T, G, d)).repeat_interleave(H // G, 1)
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_recurrence_fast(q, k, v.view(T, H, dv), g, beta)
    o = rms(o, cfg["norm"]["eps"]) * w[p + "norm"]
    return R(o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(cfg: dict, w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    eps = cfg["norm"]["eps"]
    a = rms(rotary_attention(w, p + "left.", m["left"], h), eps) * w[p + "left.out"]
    b = rms(gated_delta(cfg, w, p + "right.", m["right"], h), eps) * w[p + "right.out"]
    return 0.5 * (a + b)


# ---- gated linear attention
def gla_recurrence(q, k, v, alpha):
    """q, k, alpha: (T, H, d); v: (T, H, dv): S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            S[h] = torch.diag(alpha[t, h]) @ S[h] + torch.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def gla_recurrence_fast(q, k, v, alpha):
    """The same, all heads of a token at once."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.empty_like(v)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def channel_decay(z: torch.Tensor, tau: float) -> torch.Tensor:
    return sigmoid(z) ** (1.0 / tau)


def gated_linear_attention(cfg: dict, w: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T * d ** -0.5).view(T, H, d)
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    z = product(w, p + "a2", R(h @ w[p + "a1"].T), True)
    o, _ = gla_recurrence_fast(q, k, v, channel_decay(z, m["tau"]).view(T, H, d))
    o = rms(o, cfg["norm"]["eps"]) * w[p + "norm"]
    return R(o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward
def dense(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return R(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return R(torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2) @ w[p + "down"].T


def route(z: torch.Tensor, correction: torch.Tensor, top: int):
    """Row by row: scores softmax(z); the `top` largest of score + correction; weights: the chosen ones' scores, divided
    by their sum."""
    idx, wts = [], []
    for row in z:
        e = torch.exp(row - row.max())
        s = e / e.sum()
        c = (s + correction).tolist()
        chosen = sorted(range(len(c)), key=lambda n: (-c[n], n))[:top]
        total = sum(s[n] for n in chosen) + SUM_EPS
        idx.append(chosen)
        wts.append(torch.stack([s[n] / total for n in chosen]))
    return torch.tensor(idx), torch.stack(wts)


def mixture(w: dict, p: str, mlp: dict, h: torch.Tensor) -> torch.Tensor:
    r = mlp["router"]
    idx, wt = route(h @ w[p + "router"].T, w[p + "correction"], r["top"])
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        rows, n = torch.nonzero(idx == e, as_tuple=True)
        if len(rows):
            y = expert(w, f"{p}e{e}.", h[rows]) if e < r["experts"] else h[rows]
            out[rows] += wt[rows, n][:, None] * y
    return out + expert(w, p + "shared.", h) if mlp.get("shared") else out


# ---- the whole model
MIXERS = {"attention": differential_attention, "parallel": parallel, "gla": gated_linear_attention}


def owner(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg: dict, w: dict, tokens: list[int], layers: bool = False):
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    streams = []
    for n in range(len(cfg["layers"])):
        j = owner(cfg, n)
        L, p = cfg["layers"][j], f"l{j}."
        y = MIXERS[L["type"]](cfg, w, p + "mix.", L["mixer"], R(norm(w, p + "norm1", x, eps)))
        x = x + norm(w, p + "norm1b", y, eps)
        if L.get("mlp") is not None:
            h = R(norm(w, p + "norm2", x, eps))
            y = dense(w, p + "mlp.", h) if L["mlp"]["kind"] == "dense" else mixture(w, p + "mlp.", L["mlp"], h)
            x = x + norm(w, p + "norm2b", y, eps)
        streams.append(x)
    logits = R(norm(w, "final.norm", x, eps)) @ w["head"].T
    return (logits, torch.stack(streams)) if layers else logits
