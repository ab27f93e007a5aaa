"""Typed Suvunex configuration, read from the design's own config.json keys.

A Suvunex model multiplies its embedded tokens by a constant and runs layers listed one by one in ``layers``.  A layer
norms what each sublayer reads and what it returns (RMS norms with a gain of one number), multiplies the normed result by
a learned factor per coordinate and adds it to the residual row; what the mixer reads has first passed a short causal
convolution over time that is added to itself (``canon.taps``).  Mixers: ``parallel`` (grouped-query attention with biased
projections, a halves-paired rotation whose slow pairs are slowed further, queries and keys divided by their length, a one
in the softmax's denominator; beside it gated linear attention with a decay per key channel; their results added with two
constant factors) and ``attention`` (values are the projected keys, head norms with gains, an evenly slowed rotation,
learned sinks, the heads' weights mixed across heads before they meet the values).  The feed-forward is gelu(gate) * up, or
absent.  Logits have a table of their own and a constant factor.  Every size and constant comes from the file.

    {"architecture": "Suvunex", "vocab": V, "width": W, "norm": {"eps": e}, "canon": {"taps": t},
     "embedding": {"scale": s}, "logit_scale": l,
     "layers": [{"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale",
                                    "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}},
                           "right": {"heads", "dim", "vdim", "tau"}, "left_scale", "right_scale"},
                 "mlp": {"kind": "dense", "ff"} | null},
                {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale",
                           "rot": {"base", "dims", "scaling": {"factor"}}},
                 "mlp": ...}]}
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import List, Optional

from pagedserve_b200.config.registry import ConfigError, ModelConfig

LAYER_TYPES = ("parallel", "attention")
# No position table: a request may grow until the cache is full (the engine's own setting bounds it).
UNBOUNDED = 1 << 30
# the keys that a rotation's scaling has: pairs slowed by the turns they make, or all of them evenly
SCALINGS = ({"factor", "low", "high", "original"}, {"factor"})


def _positive_int(value, what):
    if not isinstance(value, int) or isinstance(value, bool) or value <= 0:
        raise ConfigError(f"Suvunex: {what} must be a positive integer, got {value!r}")
    return value


def _any_number(value, what):
    if isinstance(value, bool) or not isinstance(value, (int, float)) or value != value or value in (float("inf"), -float("inf")):
        raise ConfigError(f"Suvunex: {what} must be a number, got {value!r}")
    return float(value)


def _number(value, what):
    if not _any_number(value, what) > 0:
        raise ConfigError(f"Suvunex: {what} must be a positive number, got {value!r}")
    return float(value)


def _object(value, what):
    if not isinstance(value, dict):
        raise ConfigError(f"Suvunex: {what} must be an object")
    return value


def _rotation(rot, dim, where):
    if rot is None:
        return None
    rot = dict(_object(rot, f"{where}.rot"))
    rot["base"] = _number(rot.get("base"), f"{where}.rot.base")
    dims = rot.get("dims")
    if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"Suvunex: {where}.rot.dims must be even and at most dim")
    if rot.get("scaling") is None:
        rot.pop("scaling", None)
        return rot
    scaling = _object(rot["scaling"], f"{where}.rot.scaling")
    if set(scaling) not in SCALINGS:
        raise ConfigError(f"Suvunex: {where}.rot.scaling has the keys factor, low, high and original, or factor alone")
    rot["scaling"] = {key: _number(value, f"{where}.rot.scaling.{key}") for key, value in scaling.items()}
    if "low" in scaling and not rot["scaling"]["low"] < rot["scaling"]["high"]:
        raise ConfigError(f"Suvunex: {where}.rot.scaling.low must lie below high")
    return rot


def _attention(mixer, where):
    """Checks what both kinds of attention share; returns a checked copy."""
    mixer = dict(_object(mixer, where))
    mixer.setdefault("kv_heads", mixer.get("heads"))              # absent: every query head has its own
    for key in ("heads", "kv_heads", "dim"):
        _positive_int(mixer.get(key), f"{where}.{key}")
    mixer["vdim"] = _positive_int(mixer.get("vdim", mixer["dim"]), f"{where}.vdim")
    if mixer["heads"] % mixer["kv_heads"]:
        raise ConfigError(f"Suvunex: {where}: heads must be a multiple of kv_heads")
    if max(mixer["dim"], mixer["vdim"]) > 256:
        raise ConfigError(f"Suvunex: {where}: head sizes above 256 are not supported")
    mixer["scale"] = _number(mixer.get("scale"), f"{where}.scale")
    mixer["rot"] = _rotation(mixer.get("rot"), mixer["dim"], where)
    return mixer


@dataclass
class SuvunexConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    canon_taps: int = 1
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    layers: List[dict] = field(default_factory=list)

    def __post_init__(self):
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        self.norm_eps = _number(self.norm_eps, "norm.eps")
        if _positive_int(self.canon_taps, "canon.taps") > 16:
            raise ConfigError("Suvunex: more than 16 taps are not supported")
        self.embedding_scale = _any_number(self.embedding_scale, "embedding.scale")
        self.logit_scale = _any_number(self.logit_scale, "logit_scale")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("Suvunex: 'layers' must be a non-empty list")
        self.layers = [self._check_layer(index, layer) for index, layer in enumerate(self.layers)]

    @staticmethod
    def _check_layer(index: int, layer) -> dict:
        where = f"layer {index}"
        if not isinstance(layer, dict) or layer.get("type") not in LAYER_TYPES:
            raise ConfigError(f"Suvunex: {where}: 'type' must be one of {LAYER_TYPES}")
        layer = copy.deepcopy(layer)
        mixer = _object(layer.get("mixer"), f"{where}: mixer")
        if layer["type"] == "parallel":
            mixer["left"] = _attention(mixer.get("left"), f"{where}: mixer.left")
            right = _object(mixer.get("right"), f"{where}: mixer.right")
            for key in ("heads", "dim", "vdim"):
                _positive_int(right.get(key), f"{where}: mixer.right.{key}")
            right["tau"] = _number(right.get("tau"), f"{where}: mixer.right.tau")
            for key in ("left_scale", "right_scale"):
                mixer[key] = _any_number(mixer.get(key), f"{where}: mixer.{key}")
        else:
            layer["mixer"] = mixer = _attention(mixer, f"{where}: mixer")
            if mixer["vdim"] != mixer["dim"]:
                raise ConfigError(f"Suvunex: {where}: the values are the keys, so vdim is dim")
        mlp = layer.get("mlp")
        if mlp is not None:
            if _object(mlp, f"{where}: mlp").get("kind") != "dense":
                raise ConfigError(f"Suvunex: {where}: mlp.kind must be 'dense' (or mlp null)")
            _positive_int(mlp.get("ff"), f"{where}: mlp.ff")
        layer["mlp"] = mlp
        return layer

    # ---- ModelConfig interface ----------------------------------------
    @property
    def architecture(self) -> str:
        return "Suvunex"

    @property
    def vocabulary_size(self) -> int:
        return self.vocab

    @property
    def max_model_len(self) -> int:
        return UNBOUNDED

    @classmethod
    def from_dict(cls, values: dict) -> "SuvunexConfig":
        inner = {}
        for name, key in (("norm", "eps"), ("canon", "taps"), ("embedding", "scale")):
            part = values.get(name)
            if not isinstance(part, dict) or key not in part:
                raise ConfigError(f"Suvunex: config.json needs {name}.{key}")
            inner[name] = part[key]
        if "logit_scale" not in values:
            raise ConfigError("Suvunex: config.json needs logit_scale")
        return cls(vocab=values.get("vocab"), width=values.get("width"), norm_eps=inner["norm"], canon_taps=inner["canon"],
                   embedding_scale=inner["embedding"], logit_scale=values["logit_scale"], layers=values.get("layers"))

    def to_dict(self) -> dict:
        layers = copy.deepcopy(self.layers)
        for layer in layers:                       # an optional key that is absent stays absent
            attention = layer["mixer"]["left"] if layer["type"] == "parallel" else layer["mixer"]
            if attention["rot"] is None:
                attention.pop("rot")
        return {"architecture": self.architecture, "canon": {"taps": self.canon_taps},
                "embedding": {"scale": self.embedding_scale}, "layers": layers, "logit_scale": self.logit_scale,
                "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}


# ---- layer entries as config.json writes them (for random models: benchmarks, the command line)
def parallel_layer(heads: int, kv_heads: int, dim: int, right_heads: int, right_dim: int, right_vdim: int,
                   ff: Optional[int], vdim: Optional[int] = None, rot_dims: Optional[int] = None, base: float = 10000.0,
                   scaling: Optional[dict] = None, tau: float = 16.0, left_scale: float = 0.75,
                   right_scale: float = 0.5) -> dict:
    rot = {"base": base, "dims": dim // 2 * 2 if rot_dims is None else rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(scaling)
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim,
                               "rot": rot, "scale": dim ** -0.5},
                      "right": {"heads": right_heads, "dim": right_dim, "vdim": right_vdim, "tau": tau},
                      "left_scale": left_scale, "right_scale": right_scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention_layer(heads: int, kv_heads: int, dim: int, ff: Optional[int], base: float = 10000.0,
                    factor: Optional[float] = None) -> dict:
    rot = {"base": base, "dims": dim // 2 * 2}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": rot, "scale": dim ** -0.5},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def repeating_config(width: int, heads: int, head_dim: int, layers: int, vocab: int, ff: int, kv_heads: int = 2,
                     right_heads: Optional[int] = None, right_dim: Optional[int] = None, taps: int = 4, eps: float = 1e-6,
                     pattern=("parallel", "attention")) -> SuvunexConfig:
    """A model for random weights: the layer kinds of ``pattern`` in turn, all with a feed-forward."""
    entries = []
    for index in range(layers):
        if pattern[index % len(pattern)] == "parallel":
            entries.append(parallel_layer(heads, kv_heads, head_dim, right_heads or heads, right_dim or head_dim,
                                          right_dim or head_dim, ff,
                                          scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1024}))
        else:
            entries.append(attention_layer(heads, kv_heads, head_dim, ff, factor=4.0))
    return SuvunexConfig(vocab=vocab, width=width, norm_eps=eps, canon_taps=taps, embedding_scale=1.0, logit_scale=0.5,
                         layers=entries)


# sizes that the command line and the benchmark know by name (random weights)
NAMED_CONFIGS = {
    "suvunex-tiny": dict(width=64, heads=4, head_dim=16, layers=3, vocab=512, ff=96),
    "suvunex-w1024": dict(width=1024, heads=16, head_dim=64, layers=8, vocab=32000, ff=2816),
    "suvunex-w2048": dict(width=2048, heads=16, head_dim=128, layers=8, vocab=32000, ff=5632,
                          right_heads=32, right_dim=64),
}


def named_config(name: str) -> SuvunexConfig:
    if name not in NAMED_CONFIGS:
        raise ConfigError(f"unknown named configuration {name!r}; known: {sorted(NAMED_CONFIGS)}")
    return repeating_config(**NAMED_CONFIGS[name])
