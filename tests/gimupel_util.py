"""Small Gimupel configurations shared by the CPU and GPU tests of that design.

They differ from one another in every size and constant and keep apart what a model could make equal: state, value, key
and head counts unequal, groups of B and C from one to one per head, parts of the gated norm that are one head, several
heads, or cut through heads, one to five taps, grouped and ungrouped attention heads, windows of 1 to 300 tokens (shorter
and longer than a page and than the sequence), experts in groups of one, two and more with `top` from 1 to all of the kept
ones, every order of the layer types, layers without feed-forward, loops of one to four passes at the start, in the
middle and at the end, over one layer and over all, and no loop."""
from __future__ import annotations
import copy
import os

import numpy as np
import torch


def ssm(heads, vdim, state, groups, conv, norm_groups, kind="mamba2"):
    return kind, {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def att(heads, kv, dim, vdim, scale, size):
    return "attention", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=(1, 1), scale=1.0, limit=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}, "scale": scale}}


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def model(vocab, width, eps, scale, layers, loop=None):
    out = {"architecture": "Gimupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


GIP_MIX = model(173, 64, 1e-5, 1.7, [        # the state space first; a loop over the middle, three passes
    layer(ssm(6, 12, 20, 3, 4, 2), dense(96)),
    layer(att(4, 2, 16, 8, 0.8, 9), moe(6, 2, 24, (3, 2), 1.5, 0.7)),
    layer(ssm(4, 16, 24, 1, 3, 4, "mamba2_2"), moe(8, 3, 16, (4, 2), 0.6, 2.0)),
    layer(att(3, 3, 24, 12, 0.9, 20), None),
], (1, 3, 3))
GIP_ODD = model(89, 96, 1e-6, 1.0, [         # attention first; a loop over everything, two passes; one tap; parts of a norm cut through heads
    layer(att(6, 2, 12, 20, 1.1, 300), moe(7, 3, 12, (7, 4), 1.0, 1.3)),
    layer(ssm(3, 20, 9, 1, 1, 4), None),
    layer(ssm(8, 5, 40, 4, 5, 8, "mamba2_2"), dense(40)),
    layer(att(1, 1, 40, 40, 0.6, 1), moe(4, 2, 20, (2, 1), 3.0, 0.5)),
    layer(ssm(5, 8, 130, 5, 2, 1), moe(3, 3, 8)),
], (0, 5, 2))
GIP_ONE = model(61, 32, 1e-4, 2.5, [         # single heads; the loop at the end over one layer, four passes
    layer(ssm(1, 32, 16, 1, 2, 1, "mamba2_2"), moe(1, 1, 40, (1, 1), 0.5, 1.0)),
    layer(att(2, 1, 8, 16, 1.3, 33), dense(24)),
    layer(ssm(2, 24, 8, 2, 4, 2), moe(4, 1, 16, (2, 2), 1.0, 3.0)),
], (2, 3, 4))
GIP_TC = model(96, 64, 1e-5, 1.2, [          # no loop; sizes that the tensor-core kernels of long portions take
    layer(ssm(4, 16, 32, 2, 4, 1), dense(64)),
    layer(att(2, 1, 64, 64, 0.7, 40), moe(8, 2, 32, (4, 3), 2.0, 1.0)),
    layer(ssm(2, 64, 64, 1, 4, 2, "mamba2_2"), dense(64)),
])
CONFIGS = {"mix": (GIP_MIX, 3), "odd": (GIP_ODD, 5), "one": (GIP_ONE, 9), "tc": (GIP_TC, 4)}
STD_SCALE = 5.0


def liven(w: dict, seed: int) -> None:
    """Gives the vectors that random weights leave near zero the values a model would have, so that everything they do
    shows: decays from slow to fast, step sizes from small to large, skips, convolution biases and taps of order one,
    corrections that are larger than the scores' differences and partly negative, queries and keys that matter."""
    rng = np.random.default_rng(9000 + seed)
    for k in sorted(w):
        n = tuple(w[k].shape)
        draw = lambda lo, hi: torch.from_numpy(rng.uniform(lo, hi, n).astype(np.float32))
        if k.endswith("A_log"):
            w[k] = draw(-4.0, 1.5)
        elif k.endswith("dt_bias"):
            w[k] = draw(-4.0, 1.0)
        elif k.endswith("mix.D"):
            w[k] = draw(-1.5, 1.5)
        elif k.endswith("conv"):
            w[k] = draw(-0.8, 0.8)
        elif k.endswith("conv.b"):
            w[k] = draw(-0.4, 0.4)
        elif k.endswith("correction"):
            w[k] = draw(-0.7, 0.3)
        elif k.endswith("norm1") or k.endswith("norm2") or k.endswith("norm"):
            w[k] = draw(0.6, 1.4)
        elif k.endswith("router"):
            w[k] = w[k] * 4.0


def make_dir(name: str, tmp, cfg: dict | None = None, seed: int | None = None, change=None, dtype: str = "float32") -> tuple[str, dict, dict]:
    """Writes configuration `name` with seeded random weights; `change(tensors)` may edit them before they are written.
    Returns (folder, config, weights by name)."""
    from fusezap_core_b200.weights import write_random_model
    from fusezap_core_b200.weights.safetensors_io import read_model_dir, write_file
    base, s = CONFIGS.get(name, (cfg, seed))
    cfg = copy.deepcopy(cfg if cfg is not None else base)
    seed = seed if seed is not None else s
    d = os.path.join(str(tmp), f"gimupel-{name}")
    write_random_model(cfg, d, seed, "float32", norm_noise=True, std_scale=STD_SCALE)
    w = {k: v.clone() for k, v in read_model_dir(d).items()}
    liven(w, seed)
    if change is not None:
        change(w)
    td = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    write_file(os.path.join(d, "model.safetensors"), {k: v.to(td) for k, v in w.items()})
    return d, cfg, read_model_dir(d)


def drawn_config(seed: int, small: bool = True) -> dict:
    """A configuration drawn from a seed: the layer types in any order, odd and even sizes (the tensor-core kernels' among
    them), with and without feed-forward, any loop."""
    rng = np.random.default_rng((2000 if small else 7000) + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    kinds = ["mamba2", "attention"] + [pick("mamba2", "mamba2_2", "attention") for _ in range(int(rng.integers(0, 4)))]
    rng.shuffle(kinds)
    layers = []
    for kind in kinds:
        mlp, r = None, rng.random()
        if r < 0.3:
            mlp = dense(int(pick(16, 20, 33) if small else pick(128, 200, 320)))
        elif r < 0.85:
            count, per = int(pick(1, 2, 4)), int(pick(1, 2, 3, 4))
            keep = int(rng.integers(1, count + 1))
            top = int(rng.integers(1, keep * per + 1))
            mlp = moe(count * per, top, int(pick(8, 20, 32) if small else pick(64, 96, 200)), (count, keep), float(pick(0.5, 1.0, 2.5)),
                      float(pick(0.3, 1.0, 7.0)))
        if kind == "attention":
            kv, dk = int(pick(1, 2, 3)), int(pick(8, 12, 16, 40) if small else pick(48, 64, 96, 128))
            dv = dk if rng.random() < 0.4 else int(pick(8, 12, 24) if small else pick(32, 64, 128))
            mixer = att(kv * int(pick(1, 2, 4)), kv, dk, dv, float(pick(0.4, 0.8, 1.2)), int(pick(1, 2, 7, 16, 33) if small else pick(17, 64, 100, 260)))
        else:
            g = int(pick(1, 2, 4))
            h = g * int(pick(1, 2, 3))
            p = int(pick(4, 7, 12, 16) if small else pick(16, 32, 48, 64))
            parts = [x for x in (1, 2, 3, g, h) if h * p % x == 0]
            mixer = ssm(h, p, int(pick(3, 8, 16, 20, 33) if small else pick(16, 40, 64, 128)), g, int(pick(1, 2, 3, 4)), int(pick(*parts)), kind)
        layers.append(layer(mixer, mlp))
    loop = None
    if rng.random() < 0.75:
        a = int(rng.integers(0, len(layers)))
        loop = (a, int(rng.integers(a + 1, len(layers) + 1)), int(pick(1, 2, 3)))
    return model(int(pick(37, 64, 150) if small else pick(300, 512, 777)), int(pick(24, 40, 56, 72) if small else pick(160, 200, 256, 384)),
                 float(pick(1e-6, 1e-5)), float(pick(0.5, 1.0, 3.0)), layers, loop)


def tokens_for(cfg: dict, lengths, seed: int) -> list[list[int]]:
    rng = np.random.default_rng(seed)
    return [rng.integers(0, cfg["vocab"], n).tolist() for n in lengths]


def plain_logits(cfg: dict, w: dict, toks) -> np.ndarray:
    import plain_gimupel
    return plain_gimupel.forward(cfg, {k: v.double() for k, v in w.items()}, list(toks)).numpy()


def rounded(w: dict) -> dict:
    """The weights as a bfloat16 engine holds them: matrices rounded once, vectors stored in 32-bit as they are."""
    return {k: v.to(torch.bfloat16).to(torch.float32) if v.dim() >= 2 else v for k, v in w.items()}


class Oracle:
    """What the plain model says of one request, and how far rounding alone moves it: the oracle itself computed in 32-bit, or
    with bfloat16 operands."""
    def __init__(self, cfg: dict, w: dict, toks, dtype: str):
        import plain_gimupel
        self.dtype = dtype
        w = {k: v.float() for k, v in w.items()}
        if dtype == "float32":
            self.logits = plain_logits(cfg, w, toks)
            self.noise = self.errors(plain_gimupel.forward(cfg, w, list(toks)).double().numpy())
        else:
            self.logits = plain_logits(cfg, rounded(w), toks)
            with plain_gimupel.rounded_operands():
                self.noise = self.errors(plain_logits(cfg, rounded(w), toks))

    def errors(self, got: np.ndarray) -> np.ndarray:
        """Per row: the root-mean-square difference (row mean removed), relative to the rms of the oracle's logits."""
        d = got - self.logits
        d = d - d.mean(-1, keepdims=True)
        scale = float(np.sqrt(((self.logits - self.logits.mean(-1, keepdims=True)) ** 2).mean()))
        return np.sqrt((d ** 2).mean(-1)) / scale

    def check(self, got: np.ndarray, what=None) -> None:
        check_all([(self, got)], what)


def check_all(pairs: list, what=None) -> None:
    """`pairs`: (oracle, logits) of requests of one model. Three times what rounding alone does to the oracles (at least 2e-5
    in float32, 0.02 in bfloat16), for the median row and for nine rows in ten. float32: ten times that for all. bfloat16:
    where two experts' choice scores nearly tie, rounding picks the other one, and that row and what its state feeds move
    by more, so no more than one row in fifty may be off by the scale of the logits itself (two unrelated rows differ by
    1.4 times that)."""
    dtype = pairs[0][0].dtype
    e = np.concatenate([o.errors(got) for o, got in pairs])
    noise = np.concatenate([o.noise for o, _ in pairs])
    floor = 2e-5 if dtype == "float32" else 0.02
    for q in (0.5, 0.9):
        have, lim = np.quantile(e, q), max(floor, 3 * np.quantile(noise, q))
        assert have < lim, (what, q, float(have), float(lim), float(e.max()))
    if dtype == "float32":
        assert e.max() < 10 * max(floor, 3 * noise.max()), (what, float(e.max()), float(noise.max()))
    else:
        assert (e > 1.0).mean() <= 0.02, (what, float((e > 1.0).mean()), float(e.max()))
