"""Typed configuration of the Gimupel decoder, read from its own config.json keys, and its model description.

config.json: `architecture` "Gimupel"; `vocab`, `width`; `norm.eps`; `embedding.scale`; `layers`: a list whose entries
give `type` (the mixer kind: "mamba2", "mamba2_2" or "attention"), `mixer` (its sizes and constants) and `mlp` (`kind`
"dense" with `ff`, or "moe" with `expert.ff`, `expert.limit`, `router.experts`, `router.top`, `router.groups` (`count`,
`keep`) and `router.scale`, or null for none); `loop` (`start`, `stop`, `times`, or null): layers start .. stop-1 run
`times` times in a row. Tensor names: `embed`, `final.norm`, and per layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`,
`l<i>.mlp.*`. The output matrix is the embedding table.

What the design is made of (every piece is a part of this package that another design can name with other constants):

  embedding      the token's row times `embedding.scale`
  order          the schedule runs the looped layers several times with the same weights and a cache or state of its own
                 per pass; before each pass but the first the embedding output is added to the stream (`add_embedding`)
  layer          block `pre_norm`: x <- x + mixer(norm1(x)); x <- x + ff(norm2(x)); norm `layernorm` (a weight, no bias)
  mamba2(_2)     mixer `mamba2`: selective state space with grouped B and C, a short convolution with a bias, a gated norm
                 in parts; the two names are the same mixer in sizes of their own
  attention      mixer `sink_attention` without rotation and sink: grouped-query attention over a sliding window, every q
                 and k head divided by its root mean square (no weight)
  feed-forward   `swiglu` (dense) or `routed_moe`: sigmoid scores, experts and groups chosen with a correction per expert,
                 a group's score the sum of its two largest, weights renormalised and scaled, clamped gated experts
"""
from __future__ import annotations
from dataclasses import dataclass
from typing import Any

from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXER_KINDS = ("mamba2", "mamba2_2", "attention")
EXPERT_ALPHA = 1.702            # an expert's gate is g * sigmoid(EXPERT_ALPHA * g): fixed by the design
EXPERT_UP_SHIFT = 1.0           # and multiplies u + EXPERT_UP_SHIFT: fixed by the design
WEIGHT_SUM_EPS = 1e-20          # added to the sum of the chosen scores: fixed by the design


def _need(m: dict, keys: tuple, where: str) -> None:
    missing = [k for k in keys if k not in m]
    if missing:
        raise ValueError(f"config.json: {where} lacks {missing}")


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @staticmethod
    def from_json(m: dict, where: str) -> "StateSpaceConfig":
        keys = ("heads", "vdim", "state", "groups", "conv", "norm_groups")
        _need(m, keys, where)
        out = StateSpaceConfig(*(int(m[k]) for k in keys))
        if min(out.heads, out.vdim, out.state, out.groups, out.conv, out.norm_groups) <= 0:
            raise ValueError(f"config.json: {where}: heads, vdim, state, groups, conv and norm_groups must be positive")
        if out.heads % out.groups:
            raise ValueError(f"config.json: {where}: heads must be a multiple of groups")
        if out.heads * out.vdim % out.norm_groups:
            raise ValueError(f"config.json: {where}: heads * vdim must be a multiple of norm_groups")
        return out

    def to_json(self) -> dict:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups,
                "state": self.state, "vdim": self.vdim}


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int

    @staticmethod
    def from_json(m: dict, where: str) -> "AttentionConfig":
        _need(m, ("heads", "kv_heads", "dim", "vdim", "scale", "mask"), where)
        _need(m["mask"], ("size",), where + ".mask")
        out = AttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                              int(m["mask"]["size"]))
        if min(out.heads, out.kv_heads, out.dim, out.vdim) <= 0 or out.heads % out.kv_heads:
            raise ValueError(f"config.json: {where}: heads must be a positive multiple of kv_heads, dim and vdim positive")
        if out.window <= 0:
            raise ValueError(f"config.json: {where}.mask.size must be positive")
        return out

    def to_json(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "mask": {"size": self.window},
                "scale": self.scale, "vdim": self.vdim}


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                     # "dense" or "moe"
    ff: int                       # dense: the intermediate size; moe: an expert's
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1
    scale: float = 1.0

    @staticmethod
    def from_json(m: dict, where: str) -> "FeedForwardConfig":
        kind = m.get("kind")
        if kind == "dense":
            _need(m, ("ff",), where)
            out = FeedForwardConfig("dense", int(m["ff"]))
        elif kind == "moe":
            _need(m, ("router", "expert"), where)
            r, e = m["router"], m["expert"]
            _need(r, ("experts", "top", "scale"), where + ".router")
            _need(e, ("ff", "limit"), where + ".expert")
            g = r.get("groups") or {"count": 1, "keep": 1}
            _need(g, ("count", "keep"), where + ".router.groups")
            out = FeedForwardConfig("moe", int(e["ff"]), float(e["limit"]), int(r["experts"]), int(r["top"]), int(g["count"]),
                                    int(g["keep"]), float(r["scale"]))
            if not 0 < out.top <= out.experts:
                raise ValueError(f"config.json: {where}.router: need 0 < top <= experts, got {out.top}, {out.experts}")
            if out.groups <= 0 or out.experts % out.groups or not 0 < out.keep <= out.groups:
                raise ValueError(f"config.json: {where}.router.groups: {out.experts} experts do not form {out.groups} "
                                 f"equal groups of which {out.keep} are kept")
            if out.top > out.keep * (out.experts // out.groups):
                raise ValueError(f"config.json: {where}.router: top {out.top} exceeds the experts of the {out.keep} kept groups")
            if not out.limit > 0:
                raise ValueError(f"config.json: {where}.expert.limit must be positive")
        else:
            raise NotImplementedError(f"config.json: {where}.kind {kind!r} is not supported (have ['dense', 'moe'])")
        if out.ff <= 0:
            raise ValueError(f"config.json: {where}: ff must be positive")
        return out

    def to_json(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        return {"expert": {"ff": self.ff, "limit": self.limit}, "kind": "moe",
                "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep}, "scale": self.scale,
                           "top": self.top}}


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int

    @staticmethod
    def from_json(m: dict, n_layers: int) -> "Loop":
        _need(m, ("start", "stop", "times"), "loop")
        out = Loop(int(m["start"]), int(m["stop"]), int(m["times"]))
        if not 0 <= out.start < out.stop <= n_layers or out.times < 1:
            raise ValueError(f"config.json: loop {m}: need 0 <= start < stop <= {n_layers} and times >= 1")
        return out

    def to_json(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


@dataclass(frozen=True)
class GimupelLayer:
    type: str
    mixer: Any                     # StateSpaceConfig | AttentionConfig
    mlp: FeedForwardConfig | None


@dataclass(frozen=True)
class GimupelConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    layers: tuple
    loop: Loop | None = None
    max_position: int = 1 << 17      # positions are not bounded by the design; the engine sizes its tables itself

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ValueError("config: vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ValueError(f"config: norm.eps must be positive, got {self.norm_eps!r}")

    @staticmethod
    def from_json(c: dict) -> "GimupelConfig":
        _need(c, ("vocab", "width", "layers", "norm", "embedding"), "the top level")
        _need(c["norm"], ("eps",), "norm")
        _need(c["embedding"], ("scale",), "embedding")
        layers = []
        for i, L in enumerate(c["layers"]):
            where = f"layers[{i}]"
            kind = L.get("type")
            if kind not in MIXER_KINDS:
                raise NotImplementedError(f"config.json: {where}.type {kind!r} is not supported (have {list(MIXER_KINDS)})")
            _need(L, ("mixer",), where)
            mixer = (AttentionConfig if kind == "attention" else StateSpaceConfig).from_json(L["mixer"], where + ".mixer")
            mlp = FeedForwardConfig.from_json(L["mlp"], where + ".mlp") if L.get("mlp") is not None else None
            layers.append(GimupelLayer(kind, mixer, mlp))
        loop = Loop.from_json(c["loop"], len(layers)) if c.get("loop") is not None else None
        return GimupelConfig(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c["embedding"]["scale"]),
                             tuple(layers), loop, int(c.get("max_position", 1 << 17)))

    def to_json(self) -> dict:
        out = {"architecture": "Gimupel", "embedding": {"scale": self.embed_scale},
               "layers": [{"mixer": L.mixer.to_json(), "mlp": L.mlp.to_json() if L.mlp is not None else None, "type": L.type}
                          for L in self.layers],
               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = self.loop.to_json()
        return out

    def random_optional_groups(self, expected: dict) -> set:
        return set()

    # ---- the model description
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("layernorm", {"size": self.width, "eps": self.norm_eps, "name": name})

    def _state_space(self, m: StateSpaceConfig) -> PartSpec:
        return PartSpec("mamba2", {
            "hidden_size": self.width, "num_heads": m.heads, "value_dim": m.vdim, "state_dim": m.state, "groups": m.groups,
            "taps": m.conv, "norm_groups": m.norm_groups, "eps": self.norm_eps,
            "names": {"in": "in", "conv": "conv", "conv_bias": "b", "dt_bias": "dt_bias", "decay_log": "A_log", "skip": "D",
                      "norm": "norm", "out": "o"}})

    def _attention(self, a: AttentionConfig) -> PartSpec:
        return PartSpec("sink_attention", {
            "hidden_size": self.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "key_dim": a.dim,
            "value_dim": a.vdim, "scale": a.scale, "window": a.window, "keep_first": 0, "sink": False, "rotated": 0,
            "qk_norm": True, "norm_weight": False, "norm_eps": self.norm_eps,
            "names": {"q": "q", "k": "k", "v": "v", "out": "o"}})

    def _ffn(self, f: FeedForwardConfig) -> PartSpec:
        if f.kind == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": f.ff,
                                       "names": ("gate", "up", "down"), "suffix": ""})
        return PartSpec("routed_moe", {
            "hidden_size": self.width, "intermediate_size": f.ff, "num_experts": f.experts, "top": f.top,
            "groups": f.groups, "keep_groups": f.keep, "renormalize": True, "scoring": "sigmoid", "correction": True,
            "group_score": "top2", "sum_eps": WEIGHT_SUM_EPS, "weight_scale": f.scale,
            "alpha": EXPERT_ALPHA, "limit": f.limit, "up_shift": EXPERT_UP_SHIFT,
            "names": {"router": "router", "correction": "correction", "expert": "e{}", "gate": "gate", "up": "up",
                      "down": "down"}})

    def _order(self) -> list[tuple[int, bool]]:
        """(layer, whether the embedding output is added right before it) of every execution."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [(i, False) for i in range(n)]
        passes = [(i, turn > 0 and i == loop.start) for turn in range(loop.times) for i in range(loop.start, loop.stop)]
        return [(i, False) for i in range(loop.start)] + passes + [(i, False) for i in range(loop.stop, n)]

    def spec(self) -> ModelSpec:
        layers = []
        for i, L in enumerate(self.layers):
            mixer = self._attention(L.mixer) if L.type == "attention" else self._state_space(L.mixer)
            block = PartSpec("pre_norm", {"names": ("norm1", "mix", "norm2", "mlp"), "norms": (self._norm(""), self._norm(""))})
            layers.append(LayerSpec(f"l{i}.", block, mixer, self._ffn(L.mlp) if L.mlp is not None else None))
        schedule = tuple(ScheduleEntry(layer, n, add_embedding=again) for n, (layer, again) in enumerate(self._order()))
        return ModelSpec(
            architecture="Gimupel", hidden_size=self.width, vocab_size=self.vocab, embed_name="embed", lm_head_name=None,
            tie_embeddings=True, final_norm=self._norm("norm"), final_norm_name="final.norm", layers=tuple(layers),
            schedule=schedule, positions={}, max_position=self.max_position, embed_scale=self.embed_scale)
