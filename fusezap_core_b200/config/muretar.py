"""Typed configuration of the Muretar decoder, read from its own config.json keys, and its model description.

config.json: `architecture` "Muretar"; `vocab`, `width`; `norm.eps`; `layers`: a list whose entries give `type` (the
mixer kind: "parallel", "gla" or "attention"), `mixer` (its sizes and constants), `mlp` (the feed-forward: `kind` "dense"
with `ff`, or "moe" with `expert.ff`, `router.experts`, `router.top`, `router.identity` and `shared.ff`, or null for none)
and optionally `weights_of` j: the entry has no tensors of its own and runs layer j once more, with a cache or state of
its own. Tensor names: `embed`, `final.norm`, `head`, and per layer i that owns tensors `l<i>.norm1`, `l<i>.norm1b`,
`l<i>.norm2`, `l<i>.norm2b` (each with a `.b`), `l<i>.mix.*`, `l<i>.mlp.*`.

What the design is made of (every piece is a part of this package that another design can name with other constants):

  layer         x <- x + norm1b(mixer(norm1(x))); x <- x + norm2b(ff(norm2(x)))       (block `sandwich_norm`, the second
                half optional; norm `layernorm` with a weight and a bias)
  parallel      mixer `parallel_mixers`: half the sum of two mixers' results, each divided by its root mean square over
                the width and multiplied by a weight
    left        mixer `sink_attention` without window and sink: causal grouped-query attention with biases, neighbours
                paired in the rotation, frequencies divided by a factor (`rope`, kind "linear", angles in 64-bit)
    right       mixer `gated_delta`: the gated delta rule with one decay per head and a silu gate of one product
  gla           mixer `gated_linear_attention`: S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with
                alpha = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau) per head and key channel
  attention     mixer `differential_attention`: two softmax maps over the same values, o = a1 - lambda a2, divided by its
                root mean square per head, times 1 - diff; no positions
  feed-forward  `swiglu` (dense) or `routed_moe` with experts W_down relu(W_up h)^2, softmax scores over all router
                outputs, chosen with a correction, weights renormalised; the last outputs are experts that hand h on; a
                shared expert of the same form without a gate
  output        the model's norm, then the output matrix `head`
"""
from __future__ import annotations
from dataclasses import dataclass
from typing import Any

from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXER_KINDS = ("parallel", "gla", "attention")
UNIT_EPS = 1e-6        # inside the root of the unit-vector norm of the delta rule's q and k: fixed by the design
SUM_EPS = 1e-20        # added to the sum of the chosen scores: fixed by the design
HALF = 0.5             # what each of two parallel mixers contributes: fixed by the design


def _need(m: dict, keys: tuple, where: str) -> None:
    missing = [k for k in keys if k not in m]
    if missing:
        raise ValueError(f"config.json: {where} lacks {missing}")


def _positive_heads(heads: int, kv_heads: int, dim: int, vdim: int, where: str) -> None:
    if min(heads, kv_heads, dim, vdim) <= 0 or heads % kv_heads:
        raise ValueError(f"config.json: {where}: heads must be a positive multiple of kv_heads, dim and vdim positive")


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    factor: float = 1.0                 # every frequency is divided by this

    @staticmethod
    def from_json(r: dict, dim: int, where: str) -> "Rotation":
        _need(r, ("base", "dims"), where + ".rot")
        sc = r.get("scaling")
        if sc is not None:
            _need(sc, ("factor",), where + ".rot.scaling")
        out = Rotation(float(r["base"]), int(r["dims"]), float(sc["factor"]) if sc is not None else 1.0)
        if out.dims % 2 or not 0 <= out.dims <= dim:
            raise ValueError(f"config.json: {where}.rot.dims {out.dims} must be even and at most dim {dim}")
        if not out.factor > 0 or not out.base > 0:
            raise ValueError(f"config.json: {where}.rot: base and scaling.factor must be positive")
        return out

    def to_json(self) -> dict:
        return {"base": self.base, "dims": self.dims, "scaling": {"factor": self.factor}}

    def name(self) -> str:
        return f"rot{self.dims}@{self.base!r}/{self.factor!r}"

    def spec(self) -> PartSpec:
        return PartSpec("rope", {"head_dim": self.dims, "theta": self.base, "precise": True, "kind": "linear", "factor": self.factor})


@dataclass(frozen=True)
class RotaryAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation

    @staticmethod
    def from_json(m: dict, where: str) -> "RotaryAttentionConfig":
        _need(m, ("heads", "kv_heads", "dim", "vdim", "scale", "rot"), where)
        out = RotaryAttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                    Rotation.from_json(m["rot"], int(m["dim"]), where))
        _positive_heads(out.heads, out.kv_heads, out.dim, out.vdim, where)
        return out

    def to_json(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "rot": self.rot.to_json(), "scale": self.scale,
                "vdim": self.vdim}


@dataclass(frozen=True)
class GatedDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @staticmethod
    def from_json(m: dict, where: str) -> "GatedDeltaConfig":
        _need(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
        out = GatedDeltaConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        _positive_heads(out.heads, out.kv_heads, out.dim, out.vdim, where)
        if out.conv < 1:
            raise ValueError(f"config.json: {where}.conv must be at least 1 tap")
        return out

    def to_json(self) -> dict:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}


@dataclass(frozen=True)
class ParallelConfig:
    left: RotaryAttentionConfig
    right: GatedDeltaConfig

    @staticmethod
    def from_json(m: dict, where: str) -> "ParallelConfig":
        _need(m, ("left", "right"), where)
        return ParallelConfig(RotaryAttentionConfig.from_json(m["left"], where + ".left"),
                              GatedDeltaConfig.from_json(m["right"], where + ".right"))

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "right": self.right.to_json()}


@dataclass(frozen=True)
class LinearAttentionConfig:
    heads: int
    dim: int
    vdim: int
    tau: float

    @staticmethod
    def from_json(m: dict, where: str) -> "LinearAttentionConfig":
        _need(m, ("heads", "dim", "vdim", "tau"), where)
        out = LinearAttentionConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]))
        _positive_heads(out.heads, out.heads, out.dim, out.vdim, where)
        if not out.tau > 0:
            raise ValueError(f"config.json: {where}.tau must be positive, got {out.tau!r}")
        return out

    def to_json(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}


@dataclass(frozen=True)
class DifferentialAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                       # of one map: a query or key head has 2 * dim values
    vdim: int
    scale: float
    diff: float

    @staticmethod
    def from_json(m: dict, where: str) -> "DifferentialAttentionConfig":
        _need(m, ("heads", "kv_heads", "dim", "vdim", "scale", "diff"), where)
        out = DifferentialAttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                          float(m["diff"]))
        _positive_heads(out.heads, out.kv_heads, out.dim, out.vdim, where)
        return out

    def to_json(self) -> dict:
        return {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                "vdim": self.vdim}


_MIXERS = {"parallel": ParallelConfig, "gla": LinearAttentionConfig, "attention": DifferentialAttentionConfig}


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                     # "dense" or "moe"
    ff: int                       # dense: the intermediate size; moe: an expert's
    experts: int = 0
    identity: int = 0             # router outputs beyond the experts that hand the input on
    top: int = 0
    shared_ff: int = 0            # 0: no shared expert

    @staticmethod
    def from_json(m: dict, where: str) -> "FeedForwardConfig":
        kind = m.get("kind")
        if kind == "dense":
            _need(m, ("ff",), where)
            out = FeedForwardConfig("dense", int(m["ff"]))
        elif kind == "moe":
            _need(m, ("router", "expert"), where)
            r = m["router"]
            _need(r, ("experts", "top"), where + ".router")
            _need(m["expert"], ("ff",), where + ".expert")
            shared = m.get("shared") or {}
            out = FeedForwardConfig("moe", int(m["expert"]["ff"]), int(r["experts"]), int(r.get("identity") or 0), int(r["top"]),
                                    int(shared.get("ff", 0)))
            if out.experts <= 0 or out.identity < 0 or not 0 < out.top <= out.experts + out.identity:
                raise ValueError(f"config.json: {where}.router: need experts > 0, identity >= 0 and 0 < top <= experts + identity, "
                                 f"got {out.experts}, {out.identity}, {out.top}")
            if out.shared_ff < 0:
                raise ValueError(f"config.json: {where}.shared.ff must not be negative")
        else:
            raise NotImplementedError(f"config.json: {where}.kind {kind!r} is not supported (have ['dense', 'moe'])")
        if out.ff <= 0:
            raise ValueError(f"config.json: {where}: ff must be positive")
        return out

    def to_json(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        out: dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe",
                               "router": {"experts": self.experts, "identity": self.identity, "top": self.top}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class MuretarLayer:
    type: str
    mixer: Any                     # ParallelConfig | LinearAttentionConfig | DifferentialAttentionConfig
    mlp: FeedForwardConfig | None
    weights_of: int | None = None  # the layer whose tensors this one uses


@dataclass(frozen=True)
class MuretarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple
    max_position: int = 1 << 17      # positions are not bounded by the design; the engine sizes its tables itself

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ValueError("config: vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ValueError(f"config: norm.eps must be positive, got {self.norm_eps!r}")
        for i in range(len(self.layers)):
            j = self.owner(i)
            a, b = self.layers[i], self.layers[j]
            if (a.type, a.mixer, a.mlp) != (b.type, b.mixer, b.mlp):
                raise ValueError(f"config.json: layers[{i}] uses the weights of layers[{j}] but differs from it")

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses (itself, unless `weights_of` names another)."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers):
                raise ValueError(f"config.json: weights_of names layer {i}, there are {len(self.layers)}")
            if i in seen:
                raise ValueError(f"config.json: weights_of goes round in a circle at layers {sorted(seen)}")
            seen.add(i)
        return i

    @staticmethod
    def from_json(c: dict) -> "MuretarConfig":
        _need(c, ("vocab", "width", "layers", "norm"), "the top level")
        _need(c["norm"], ("eps",), "norm")
        layers = []
        for i, L in enumerate(c["layers"]):
            where = f"layers[{i}]"
            kind = L.get("type")
            if kind not in MIXER_KINDS:
                raise NotImplementedError(f"config.json: {where}.type {kind!r} is not supported (have {list(MIXER_KINDS)})")
            _need(L, ("mixer",), where)
            mlp, of = L.get("mlp"), L.get("weights_of")
            layers.append(MuretarLayer(kind, _MIXERS[kind].from_json(L["mixer"], where + ".mixer"),
                                       FeedForwardConfig.from_json(mlp, where + ".mlp") if mlp is not None else None,
                                       int(of) if of is not None else None))
        return MuretarConfig(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), tuple(layers),
                             int(c.get("max_position", 1 << 17)))

    def to_json(self) -> dict:
        layers = []
        for L in self.layers:
            e: dict[str, Any] = {"mixer": L.mixer.to_json(), "mlp": L.mlp.to_json() if L.mlp else None, "type": L.type}
            if L.weights_of is not None:
                e["weights_of"] = L.weights_of
            layers.append(e)
        return {"architecture": "Muretar", "layers": layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}

    def random_optional_groups(self, expected: dict) -> set:
        return {"lm_head"}

    # ---- the model description
    def _parallel(self, m: ParallelConfig, positions: dict) -> PartSpec:
        a, d = m.left, m.right
        if a.rot.dims:
            positions.setdefault(a.rot.name(), a.rot.spec())
        left = PartSpec("sink_attention", {
            "hidden_size": self.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "key_dim": a.dim, "value_dim": a.vdim,
            "scale": a.scale, "sink": False, "rotated": a.rot.dims, "pairing": "neighbours",
            "position": a.rot.name() if a.rot.dims else None, "bias": ("q", "k", "v", "out"), "bias_suffix": ".b",
            "names": {"q": "q", "k": "k", "v": "v", "out": "o"}})
        right = PartSpec("gated_delta", {
            "hidden_size": self.width, "num_heads": d.heads, "num_key_heads": d.kv_heads, "key_dim": d.dim,
            "value_dim": d.vdim, "taps": d.conv, "unit_eps": UNIT_EPS, "query_scale": d.dim ** -0.5, "eps": self.norm_eps,
            "head_decay": True, "gate": "silu", "one_step": True,
            "names": {"q": "q", "k": "k", "v": "v", "conv": "conv", "beta": "b", "decay_log": "A_log", "decay_in": "a",
                      "decay_bias": "dt_bias", "gate_in": "g", "norm": "norm", "out": "o"}})
        return PartSpec("parallel_mixers", {"hidden_size": self.width, "norm_name": "out", "norm_eps": self.norm_eps,
                                            "mixers": (("left", left, HALF), ("right", right, HALF))})

    def _gla(self, m: LinearAttentionConfig) -> PartSpec:
        return PartSpec("gated_linear_attention", {
            "hidden_size": self.width, "num_heads": m.heads, "key_dim": m.dim, "value_dim": m.vdim,
            "query_scale": m.dim ** -0.5, "decay_root": m.tau, "eps": self.norm_eps, "gate": "silu", "bias_suffix": ".b",
            "names": {"q": "q", "k": "k", "v": "v", "gate": "g", "decay_in": "a1", "decay_out": "a2", "norm": "norm", "out": "o"}})

    def _attention(self, m: DifferentialAttentionConfig) -> PartSpec:
        return PartSpec("differential_attention", {
            "hidden_size": self.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "map_dim": m.dim, "value_dim": m.vdim,
            "scale": m.scale, "start": m.diff, "eps": self.norm_eps, "bias": ("q", "k", "v"), "bias_suffix": ".b",
            "names": {"q": "q", "k": "k", "v": "v", "out": "o", "mix": ("lq1", "lk1", "lq2", "lk2")}})

    def _ffn(self, f: FeedForwardConfig) -> PartSpec:
        if f.kind == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": f.ff,
                                       "names": ("gate", "up", "down"), "suffix": ""})
        return PartSpec("routed_moe", {
            "hidden_size": self.width, "intermediate_size": f.ff, "num_experts": f.experts, "identity": f.identity, "top": f.top,
            "shared_size": f.shared_ff, "shared_gate": False, "renormalize": True, "correction": True, "sum_eps": SUM_EPS,
            "activation": "relu2",
            "names": {"router": "router", "expert": "e{}", "up": "up", "down": "down", "shared": "shared",
                      "correction": "correction"}})

    def spec(self) -> ModelSpec:
        D = self.width
        def norm(name: str) -> PartSpec:
            return PartSpec("layernorm", {"size": D, "eps": self.norm_eps, "name": name, "bias": "b"})
        positions: dict[str, PartSpec] = {}
        layers, at = [], {}
        for i, L in enumerate(self.layers):
            if L.weights_of is not None:
                continue
            mixer = (self._parallel(L.mixer, positions) if L.type == "parallel" else
                     self._gla(L.mixer) if L.type == "gla" else self._attention(L.mixer))
            block = PartSpec("sandwich_norm", {"names": ("norm1", "mix", "norm1b", "norm2", "mlp", "norm2b"), "norms": (norm(""),) * 4})
            at[i] = len(layers)
            layers.append(LayerSpec(f"l{i}.", block, mixer, self._ffn(L.mlp) if L.mlp is not None else None))
        schedule = tuple(ScheduleEntry(at[self.owner(i)], i) for i in range(len(self.layers)))
        return ModelSpec(
            architecture="Muretar", hidden_size=D, vocab_size=self.vocab, embed_name="embed", lm_head_name="head",
            tie_embeddings=False, final_norm=norm("norm"), final_norm_name="final.norm", layers=tuple(layers),
            schedule=schedule, positions=positions, max_position=self.max_position)
