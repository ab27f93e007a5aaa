"""Typed Vozirax configuration, read from the design's own config.json keys.

A Vozirax model adds sines and cosines of the position to its embedded tokens and runs layers listed one by one in
``layers``.  A layer's mixer and its feed-forward read the same residual row, each through an RMS norm of its own (gains
stored as their distance from one), and both results, times a learned factor per coordinate, are added to it.  Mixers:
``mamba2`` (a state-space recurrence with one decay per head and token behind a short convolution, gated and then normed in
groups) and ``attention`` (differential attention: two normed query/key maps per head over one value, subtracted; queries
that grow warmer with the position; a gate per head; optionally over the keys and values of an earlier layer).  The
feed-forward is silu(gate) * up, routed experts (squared relu, a sigmoid router with an election correction and groups), or
absent.  Logits have a table of their own and a constant factor.  Every size and constant comes from the file.

    {"architecture": "Vozirax", "vocab": V, "width": W, "norm": {"eps": e}, "logit_scale": l,
     "layers": [{"type": "mamba2",
                 "mixer": {"heads", "vdim", "state", "groups", "norm_groups", "conv"},
                 "mlp": {"kind": "dense", "ff"} | null},
                {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "q_temp": {"coef", "every"}, "kv_from"},
                 "mlp": {"kind": "moe", "expert": {"ff"},
                         "router": {"experts", "top", "scale", "groups": {"count", "keep"}}}}]}
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import List, Optional

from pagedserve_b200.config.registry import ConfigError, ModelConfig

LAYER_TYPES = ("mamba2", "attention")
# No position table: a request may grow until the cache is full (the engine's own setting bounds it).
UNBOUNDED = 1 << 30


def _positive_int(value, what):
    if not isinstance(value, int) or isinstance(value, bool) or value <= 0:
        raise ConfigError(f"Vozirax: {what} must be a positive integer, got {value!r}")
    return value


def _any_number(value, what):
    if isinstance(value, bool) or not isinstance(value, (int, float)) or value != value or value in (float("inf"), -float("inf")):
        raise ConfigError(f"Vozirax: {what} must be a number, got {value!r}")
    return float(value)


def _number(value, what):
    if not _any_number(value, what) > 0:
        raise ConfigError(f"Vozirax: {what} must be a positive number, got {value!r}")
    return float(value)


def _object(value, what):
    if not isinstance(value, dict):
        raise ConfigError(f"Vozirax: {what} must be an object")
    return value


@dataclass
class VoziraxConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    logit_scale: float = 1.0
    layers: List[dict] = field(default_factory=list)

    def __post_init__(self):
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        self.norm_eps = _number(self.norm_eps, "norm.eps")
        self.logit_scale = _any_number(self.logit_scale, "logit_scale")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("Vozirax: 'layers' must be a non-empty list")
        checked = []
        for index, layer in enumerate(self.layers):
            checked.append(self._check_layer(index, layer, checked))
        self.layers = checked

    @classmethod
    def _check_layer(cls, index: int, layer, before) -> dict:
        where = f"layer {index}"
        if not isinstance(layer, dict) or layer.get("type") not in LAYER_TYPES:
            raise ConfigError(f"Vozirax: {where}: 'type' must be one of {LAYER_TYPES}")
        layer = copy.deepcopy(layer)
        mixer = _object(layer.get("mixer"), f"{where}: mixer")
        if layer["type"] == "mamba2":
            cls._check_mamba(mixer, where)
        else:
            cls._check_attention(mixer, where, index, before)
        if layer.get("mlp") is not None:
            cls._check_mlp(_object(layer["mlp"], f"{where}: mlp"), where)
        layer["mlp"] = layer.get("mlp")
        return layer

    @staticmethod
    def _check_mamba(mixer, where):
        for key in ("heads", "vdim", "state", "groups", "norm_groups", "conv"):
            _positive_int(mixer.get(key), f"{where}: mixer.{key}")
        if mixer["heads"] % mixer["groups"]:
            raise ConfigError(f"Vozirax: {where}: heads must be a multiple of groups")
        if (mixer["heads"] * mixer["vdim"]) % mixer["norm_groups"] or mixer["norm_groups"] > 64:
            raise ConfigError(f"Vozirax: {where}: norm_groups (at most 64) must divide heads * vdim")
        if mixer["conv"] > 16 or mixer["state"] > 512 or mixer["vdim"] > 1024:
            raise ConfigError(f"Vozirax: {where}: more than 16 taps or a state of more than 512 x 1024 is not supported")

    @staticmethod
    def _check_attention(mixer, where, index, before):
        mixer.setdefault("kv_heads", mixer.get("heads"))              # absent: every query head has its own
        for key in ("heads", "kv_heads", "dim"):
            _positive_int(mixer.get(key), f"{where}: mixer.{key}")
        mixer["vdim"] = _positive_int(mixer.get("vdim", mixer["dim"]), f"{where}: mixer.vdim")
        if mixer["heads"] % mixer["kv_heads"]:
            raise ConfigError(f"Vozirax: {where}: heads must be a multiple of kv_heads")
        if max(2 * mixer["dim"], mixer["vdim"]) > 1024:
            raise ConfigError(f"Vozirax: {where}: two keys, or a value, of more than 1024 numbers are not supported")
        mixer["scale"] = _number(mixer.get("scale"), f"{where}: mixer.scale")
        mixer["diff"] = _any_number(mixer.get("diff"), f"{where}: mixer.diff")
        if mixer.get("q_temp") is None:
            mixer.pop("q_temp", None)
        else:
            temp = _object(mixer["q_temp"], f"{where}: mixer.q_temp")
            temp["coef"] = _any_number(temp.get("coef"), f"{where}: mixer.q_temp.coef")
            if isinstance(temp.get("every"), float) and temp["every"].is_integer():
                temp["every"] = int(temp["every"])
            _positive_int(temp.get("every"), f"{where}: mixer.q_temp.every")
        if mixer.get("kv_from") is None:
            mixer.pop("kv_from", None)
            return
        lender = mixer["kv_from"]
        if not isinstance(lender, int) or isinstance(lender, bool) or not (0 <= lender < index):
            raise ConfigError(f"Vozirax: {where}: mixer.kv_from must name an earlier layer")
        other = before[lender]
        if other["type"] != "attention" or "kv_from" in other["mixer"]:
            raise ConfigError(f"Vozirax: {where}: layer {lender} has no keys and values of its own")
        if any(other["mixer"][key] != mixer[key] for key in ("kv_heads", "dim", "vdim")):
            raise ConfigError(f"Vozirax: {where}: key heads and sizes differ from those of layer {lender}")

    @staticmethod
    def _check_mlp(mlp, where):
        if mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"Vozirax: {where}: mlp.kind must be 'dense' or 'moe' (or mlp null)")
        if mlp["kind"] == "dense":
            _positive_int(mlp.get("ff"), f"{where}: mlp.ff")
            return
        router = _object(mlp.get("router"), f"{where}: mlp.router")
        _positive_int(_object(mlp.get("expert"), f"{where}: mlp.expert").get("ff"), f"{where}: mlp.expert.ff")
        _positive_int(router.get("experts"), f"{where}: mlp.router.experts")
        _positive_int(router.get("top"), f"{where}: mlp.router.top")
        router["scale"] = _any_number(router.get("scale", 1.0), f"{where}: mlp.router.scale")
        standing = router["experts"]
        if router.get("groups") is None:
            router.pop("groups", None)
        else:
            groups = _object(router["groups"], f"{where}: mlp.router.groups")
            for key in ("count", "keep"):
                _positive_int(groups.get(key), f"{where}: mlp.router.groups.{key}")
            if router["experts"] % groups["count"] or groups["keep"] > groups["count"]:
                raise ConfigError(f"Vozirax: {where}: groups.count must divide the experts, and keep <= count")
            standing = router["experts"] // groups["count"] * groups["keep"]
        if router["experts"] > 256 or router["top"] > standing:
            raise ConfigError(f"Vozirax: {where}: at most 256 experts, and top at most those that can be chosen")

    # ---- ModelConfig interface ----------------------------------------
    @property
    def architecture(self) -> str:
        return "Vozirax"

    @property
    def vocabulary_size(self) -> int:
        return self.vocab

    @property
    def max_model_len(self) -> int:
        return UNBOUNDED

    @classmethod
    def from_dict(cls, values: dict) -> "VoziraxConfig":
        norm = values.get("norm")
        if not isinstance(norm, dict) or "eps" not in norm:
            raise ConfigError("Vozirax: config.json needs norm.eps")
        if "logit_scale" not in values:
            raise ConfigError("Vozirax: config.json needs logit_scale")
        return cls(vocab=values.get("vocab"), width=values.get("width"), norm_eps=norm["eps"],
                   logit_scale=values["logit_scale"], layers=values.get("layers"))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "layers": copy.deepcopy(self.layers), "logit_scale": self.logit_scale,
                "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}


# ---- layer entries as config.json writes them (for random models: benchmarks, the command line)
def mamba_layer(heads: int, vdim: int, state: int, mlp: Optional[dict], groups: int = 1, norm_groups: int = 1,
                conv: int = 4) -> dict:
    return {"type": "mamba2", "mlp": copy.deepcopy(mlp),
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def attention_layer(heads: int, kv_heads: int, dim: int, mlp: Optional[dict], vdim: Optional[int] = None, diff: float = 0.4,
                    coef: float = 0.1, every: int = 1024, kv_from: Optional[int] = None) -> dict:
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": 2 * dim if vdim is None else vdim,
             "scale": dim ** -0.5, "diff": diff, "q_temp": {"coef": coef, "every": every}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": copy.deepcopy(mlp)}


def dense_mlp(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts: int, top: int, ff: int, groups: Optional[tuple] = None, scale: float = 1.0) -> dict:
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def repeating_config(width: int, heads: int, kv_heads: int, head_dim: int, ssm_heads: int, ssm_dim: int, ssm_state: int, ff: int,
                     layers: int, vocab: int, experts: int = 8, top: int = 2, expert_ff: Optional[int] = None,
                     eps: float = 1e-6) -> VoziraxConfig:
    """A model for random weights: spans of four layers (state space with a dense feed-forward, state space with experts,
    attention with a dense one, attention with experts over the keys and values of the layer before)."""
    experts_mlp = moe_mlp(experts, top, expert_ff or ff // 2, groups=(2, 1) if experts % 2 == 0 and experts >= 2 * top else None,
                          scale=2.0)
    entries = []
    for index in range(layers):
        place = index % 4
        mlp = dense_mlp(ff) if place % 2 == 0 else experts_mlp
        if place < 2:
            entries.append(mamba_layer(ssm_heads, ssm_dim, ssm_state, mlp))
        else:
            entries.append(attention_layer(heads, kv_heads, head_dim, mlp, kv_from=index - 1 if place == 3 else None))
    return VoziraxConfig(vocab=vocab, width=width, norm_eps=eps, logit_scale=1.0, layers=entries)


# sizes that the command line and the benchmark know by name (random weights)
NAMED_CONFIGS = {
    "vozirax-tiny": dict(width=64, heads=4, kv_heads=2, head_dim=8, ssm_heads=4, ssm_dim=16, ssm_state=16, ff=96, layers=4,
                         vocab=512, experts=4, top=2),
    "vozirax-w1024": dict(width=1024, heads=16, kv_heads=4, head_dim=32, ssm_heads=32, ssm_dim=64, ssm_state=64, ff=2816,
                          layers=8, vocab=32000, experts=8, top=2, expert_ff=1024),
    "vozirax-w2048": dict(width=2048, heads=16, kv_heads=4, head_dim=64, ssm_heads=64, ssm_dim=64, ssm_state=128, ff=5632,
                          layers=8, vocab=32000, experts=8, top=2, expert_ff=2048),
}


def named_config(name: str) -> VoziraxConfig:
    if name not in NAMED_CONFIGS:
        raise ConfigError(f"unknown named configuration {name!r}; known: {sorted(NAMED_CONFIGS)}")
    return repeating_config(**NAMED_CONFIGS[name])
