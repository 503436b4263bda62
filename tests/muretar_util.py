"""Small Muretar configurations shared by the CPU and GPU tests of that design.

They differ from one another in every size and constant and keep apart what a model could make equal: key and value sizes,
query, key and value head counts, the sizes of the two parallel mixers, partly and wholly rotated heads, frequencies divided
by one and by other factors, one to five taps, roots of the decay from below one to sixteen, `top` from 1 to every router
output, with and without experts that hand their input on and with and without a shared expert, layers without feed-forward,
and layers that use an earlier (or a later) layer's weights once, twice and in a row."""
from __future__ import annotations
import copy
import os

import numpy as np
import torch


def left(heads, kv, dim, vdim, scale, base, dims, factor=1.0):
    rot = {"base": base, "dims": dims}
    if factor != 1.0:
        rot["scaling"] = {"factor": factor}
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}


def right(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def par(a, b):
    return "parallel", {"left": a, "right": b}


def gla(heads, dim, vdim, tau):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def att(heads, kv, dim, vdim, scale, diff):
    return "attention", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def model(vocab, width, eps, layers):
    """`layers`: entries, or a number j: layer j's weights once more."""
    done = []
    for L in layers:
        if isinstance(L, int):
            src = layers[L]
            while isinstance(src, int):
                src = layers[src]
            L = dict(copy.deepcopy(src), weights_of=L)
        done.append(L)
    return {"architecture": "Muretar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": done}


MUR_MIX = model(173, 64, 1e-5, [
    layer(par(left(6, 2, 16, 12, 0.4, 10000.0, 12, 4.0), right(4, 2, 10, 14, 3)), moe(5, 2, 3, 24, 40)),
    layer(gla(3, 12, 20, 16.0), dense(80)),
    layer(att(4, 2, 9, 16, 0.5, 0.6), moe(6, 0, 2, 20)),
    1,
    2,
    layer(par(left(2, 2, 8, 24, 0.7, 500.0, 8), right(3, 1, 24, 8, 1)), None),
])
MUR_ODD = model(89, 96, 1e-6, [              # every layer after the third uses the weights of another one, also in a row
    layer(att(6, 3, 20, 12, 0.3, 0.2), moe(7, 3, 10, 12, 28)),
    layer(par(left(3, 1, 40, 20, 0.25, 1e6, 24, 8.0), right(6, 3, 16, 40, 5)), moe(4, 1, 1, 36)),
    layer(gla(5, 30, 6, 2.0), None),
    0,
    2,
    4,
    layer(att(1, 1, 33, 17, 0.4, 0.8), dense(44)),
])
MUR_ONE = model(61, 32, 1e-4, [              # single heads; layer 0 uses the weights of a later one
    2,
    layer(par(left(1, 1, 8, 8, 0.9, 100.0, 2, 2.0), right(1, 1, 8, 16, 2)), moe(1, 4, 2, 16, 8)),
    layer(gla(1, 40, 16, 0.5), moe(3, 1, 4, 8)),
    layer(att(2, 1, 4, 8, 1.1, 0.5), None),
])
MUR_TC = model(96, 64, 1e-5, [               # sizes that the tensor-core kernels of long portions take
    layer(par(left(4, 1, 64, 32, 0.15, 2e5, 64, 3.0), right(4, 2, 32, 32, 4)), moe(8, 2, 3, 32, 64)),
    layer(att(6, 3, 32, 64, 0.2, 0.4), moe(8, 4, 2, 64)),
    layer(gla(2, 64, 32, 12.0), dense(64)),
    layer(att(2, 2, 64, 128, 0.15, 0.7), None),
    1,
    layer(par(left(2, 1, 128, 128, 0.1, 1e4, 64), right(2, 1, 64, 64, 2)), dense(64)),
])
CONFIGS = {"mix": (MUR_MIX, 3), "odd": (MUR_ODD, 5), "one": (MUR_ONE, 9), "tc": (MUR_TC, 13)}
STD_SCALE = 5.0


def liven(w: dict, seed: int) -> None:
    """Gives the vectors that random weights leave near zero the values a model would have, so that everything they do
    shows: decays from slow to fast, taps of order one, a lambda far from its start, corrections that are larger than the
    scores' differences and partly negative, biases of the norms and projections."""
    rng = np.random.default_rng(9000 + seed)
    for k in sorted(w):
        n = tuple(w[k].shape)
        draw = lambda lo, hi: torch.from_numpy(rng.uniform(lo, hi, n).astype(np.float32))
        if k.endswith("A_log"):
            w[k] = draw(-5.0, 1.0)
        elif k.endswith("dt_bias"):
            w[k] = draw(-3.0, 1.0)
        elif k.endswith("a2.b"):
            w[k] = draw(-2.0, 5.0)
        elif k.endswith(".conv"):
            w[k] = draw(-0.8, 0.8)
        elif k.split(".")[-1] in ("lq1", "lk1", "lq2", "lk2"):
            w[k] = draw(-1.2, 1.2) / n[0] ** 0.5
        elif k.endswith("correction"):
            w[k] = draw(-0.4, 0.4)
        elif k.endswith(".b"):
            if w[k].dim() == 1:              # (the delta rule's beta projection is called b too)
                w[k] = draw(-0.4, 0.4)
        elif k.endswith(("norm1", "norm1b", "norm2", "norm2b", "norm", "left.out", "right.out")):
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
    d = os.path.join(str(tmp), f"muretar-{name}")
    write_random_model(cfg, d, seed, "float32", norm_noise=True, std_scale=STD_SCALE)
    w = {k: v.clone() for k, v in read_model_dir(d).items()}
    liven(w, seed)
    if change is not None:
        change(w)
    td = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    write_file(os.path.join(d, "model.safetensors"), {k: v.to(td) for k, v in w.items()})
    return d, cfg, read_model_dir(d)


def corrections_apart(w: dict) -> None:
    """Router corrections further apart than any two scores, so that no choice hangs on rounding."""
    for k in [k for k in w if k.endswith("correction")]:
        n = w[k].shape[0]
        w[k] = torch.randperm(n, generator=torch.Generator().manual_seed(n)).float() * 1.5 - 4.0


def other_rank(w: dict, rank: int) -> None:
    """Gives every two-step decay projection this inner size."""
    g = torch.Generator().manual_seed(rank)
    for k in [k for k in w if k.endswith("mix.a1")]:
        k2 = k[:-1] + "2"
        w[k] = torch.randn(rank, w[k].shape[1], generator=g) * 0.1
        w[k2] = torch.randn(w[k2].shape[0], rank, generator=g) * 0.5


def drawn_config(seed: int, small: bool = True) -> dict:
    """A configuration drawn from a seed: the layer types in any order, odd and even sizes (the tensor-core kernels' among
    them), with and without feed-forward, layers that share weights."""
    rng = np.random.default_rng((3000 if small else 8000) + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    kinds = ["parallel", "gla", "attention"] + [pick("parallel", "gla", "attention") for _ in range(int(rng.integers(0, 3)))]
    rng.shuffle(kinds)
    layers: list = []
    for kind in kinds:
        mlp, r = None, rng.random()
        if r < 0.25:
            mlp = dense(int(pick(16, 20, 33) if small else pick(128, 200, 320)))
        elif r < 0.85:
            e, i = int(rng.integers(1, 13)), int(pick(0, 1, 2, 5))
            mlp = moe(e, i, int(rng.integers(1, min(e + i, 9) + 1)), int(pick(8, 20, 32) if small else pick(64, 96, 200)),
                      int(pick(0, 12, 40) if small else pick(0, 96, 128)))
        if kind == "attention":
            kv, d = int(pick(1, 2, 3)), int(pick(4, 9, 16, 20) if small else pick(24, 32, 48, 64))
            dv = 2 * d if rng.random() < 0.4 else int(pick(8, 12, 24) if small else pick(32, 64, 128))
            mixer = att(kv * int(pick(1, 2, 4)), kv, d, dv, float(pick(0.3, 0.6, 1.0)) * (1.0 if small else 0.3), float(pick(0.2, 0.5, 0.8)))
        elif kind == "gla":
            mixer = gla(int(pick(1, 2, 3)), int(pick(5, 12, 16, 33) if small else pick(24, 48, 64, 96)), int(pick(4, 7, 20) if small else pick(32, 48, 64)),
                        float(pick(0.7, 4.0, 16.0)))
        else:
            kv, d = int(pick(1, 2)), int(pick(8, 12, 16, 40) if small else pick(48, 64, 128))
            dv = d if rng.random() < 0.4 else int(pick(8, 12, 24) if small else pick(32, 64, 128))
            a = left(kv * int(pick(1, 2, 3)), kv, d, dv, float(pick(0.3, 0.6)) * (1.0 if small else 0.3), float(pick(300.0, 1e4, 5e5)),
                     2 * int(rng.integers(1, d // 2 + 1)), float(pick(1.0, 2.0, 8.0)))
            hk = int(pick(1, 2, 3))
            b = right(hk * int(pick(1, 2)), hk, int(pick(5, 8, 16, 33) if small else pick(24, 32, 64)), int(pick(4, 7, 20) if small else pick(32, 64, 80)),
                      int(pick(1, 2, 3, 4)))
            mixer = par(a, b)
        layers.append(layer(mixer, mlp))
    for _ in range(int(rng.integers(0, 3))):
        layers.insert(int(rng.integers(len(layers) + 1)), None)
    own = [i for i, L in enumerate(layers) if L is not None]
    layers = [int(own[int(rng.integers(len(own)))]) if L is None else L for L in layers]
    return model(int(pick(37, 64, 150) if small else pick(300, 512, 777)), int(pick(24, 40, 56, 72) if small else pick(160, 200, 256, 384)),
                 float(pick(1e-6, 1e-5)), layers)


def tokens_for(cfg: dict, lengths, seed: int) -> list[list[int]]:
    rng = np.random.default_rng(seed)
    return [rng.integers(0, cfg["vocab"], n).tolist() for n in lengths]


def plain_logits(cfg: dict, w: dict, toks) -> np.ndarray:
    import plain_muretar
    return plain_muretar.forward(cfg, {k: v.double() for k, v in w.items()}, list(toks)).numpy()


def rounded(w: dict) -> dict:
    """The weights as a bfloat16 engine holds them: matrices rounded once, vectors stored in 32-bit as they are."""
    return {k: v.to(torch.bfloat16).to(torch.float32) if v.dim() >= 2 else v for k, v in w.items()}


class Oracle:
    """What the plain model says of one request, and how far rounding alone moves it: the oracle itself computed in 32-bit, or
    with bfloat16 operands. (`gimupel_util.check_all` holds an engine's logits to three times that.)"""
    def __init__(self, cfg: dict, w: dict, toks, dtype: str):
        import plain_muretar
        self.dtype = dtype
        w = {k: v.float() for k, v in w.items()}
        if dtype == "float32":
            self.logits = plain_logits(cfg, w, toks)
            self.noise = self.errors(plain_muretar.forward(cfg, w, list(toks)).double().numpy())
        else:
            self.logits = plain_logits(cfg, rounded(w), toks)
            with plain_muretar.rounded_operands():
                self.noise = self.errors(plain_logits(cfg, rounded(w), toks))

    def errors(self, got: np.ndarray) -> np.ndarray:
        """Per row: the root-mean-square difference (row mean removed), relative to the rms of the oracle's logits."""
        d = got - self.logits
        d = d - d.mean(-1, keepdims=True)
        scale = float(np.sqrt(((self.logits - self.logits.mean(-1, keepdims=True)) ** 2).mean()))
        return np.sqrt((d ** 2).mean(-1)) / scale

    def check(self, got: np.ndarray, what=None) -> None:
        from gimupel_util import check_all
        check_all([(self, got)], what)
