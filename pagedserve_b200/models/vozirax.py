"""Vozirax as a ModelSpec.

Token table plus sines and cosines of the position -> layers in the listed order -> the model's norm -> logits against a
table of their own, times a constant (which is folded into that norm's gain).  Every layer is
:class:`ParallelPreNormBlock`: mixer and feed-forward read the same row through a norm of their own, and a factor per
coordinate multiplies what each adds.  ``mamba2`` layers are :class:`StateSpaceMixer`, ``attention`` layers
:class:`DifferentialAttention` (a layer that borrows keys and values runs on its lender's cache layer); the feed-forward is
the gated :class:`DenseMLP`, :class:`RoutedExperts` without gate matrices, or none.

Tensor names in a checkpoint: ``embed``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.ls1``, ``l<i>.ls2``, ``l<i>.mix.*``, ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router,correction,e<j>.up,e<j>.down}``;
matrices are stored ``[out, in]``.
"""

from __future__ import annotations

import re
from typing import Optional

from pagedserve_b200.config.registry import register_architecture
from pagedserve_b200.config.vozirax import VoziraxConfig
from pagedserve_b200.models.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

POSITION_BASE = 10000.0
# parts shared with other models name their tensors "<name>.weight"; this design stores the bare name
_BARE = re.compile(r"^(embed|head|final\.norm|l\d+\.(norm1|norm2|mlp\.gate|mlp\.up|mlp\.down))$")
_SUFFIX = ".weight"


def _normalise_name(name: str) -> Optional[str]:
    return name + _SUFFIX if _BARE.match(name) else name


def _checkpoint_name(name: str) -> str:
    if name.endswith(_SUFFIX) and _BARE.match(name[:-len(_SUFFIX)]):
        return name[:-len(_SUFFIX)]
    return name


def _mixer(entry: dict, width: int, eps: float, prefix: str) -> PartSpec:
    mixer = entry["mixer"]
    common = dict(hidden_size=width, n_heads=mixer["heads"], v_dim=mixer["vdim"], eps=eps, init_std=width ** -0.5,
                  out_init_std=(mixer["heads"] * mixer["vdim"]) ** -0.5)
    if entry["type"] == "mamba2":
        return PartSpec("state_space", dict(common, state=mixer["state"], groups=mixer["groups"],
                                            norm_groups=mixer["norm_groups"], taps=mixer["conv"]), prefix)
    return PartSpec("differential_attention", dict(
        common, n_kv_heads=mixer["kv_heads"], head_dim=mixer["dim"], scale=mixer["scale"], diff=mixer["diff"],
        q_temp=mixer.get("q_temp"), kv_source=mixer.get("kv_from") is None), prefix)


def _feed_forward(mlp: dict, width: int, prefix: str) -> PartSpec:
    std = width ** -0.5
    if mlp["kind"] == "dense":
        return PartSpec("dense_mlp", dict(
            hidden_size=width, inner_size=mlp["ff"], activation="silu", has_bias=False, stored_in_out=False,
            gate_name="mlp.gate", up_name="mlp.up", down_name="mlp.down", init_std=std, out_init_std=mlp["ff"] ** -0.5), prefix)
    router, groups = mlp["router"], mlp["router"].get("groups") or {}
    return PartSpec("routed_experts", dict(
        hidden_size=width, n_experts=router["experts"], expert_ff=mlp["expert"]["ff"], top=router["top"],
        groups=groups.get("count", 0), group_keep=groups.get("keep", 0), group_mark="two_largest", shared_ff=None,
        score="sigmoid", normalize=True, weight_scale=router["scale"], correction_name="correction",
        expert_form=dict(kind="relu_squared"), init_std=std, out_init_std=mlp["expert"]["ff"] ** -0.5), prefix + "mlp.")


def build_vozirax_spec(config: VoziraxConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = dict(width=width, eps=eps, has_mean=False, has_bias=False, weight_offset=1.0, init_std=0.1)
    layers, schedule = [], []
    for index, entry in enumerate(config.layers):
        prefix = f"l{index}."
        norms = {"pre_mixer": PartSpec("layernorm", dict(norm, name="norm1"), prefix)}
        scales = {"mixer": "ls1"}
        feed_forward = PartSpec("none")
        if entry["mlp"] is not None:
            norms["pre_feed_forward"] = PartSpec("layernorm", dict(norm, name="norm2"), prefix)
            scales["feed_forward"] = "ls2"
            feed_forward = _feed_forward(entry["mlp"], width, prefix)
        layers.append(LayerSpec(PartSpec("parallel_pre_norm", dict(scales=scales), prefix),
                                _mixer(entry, width, eps, prefix + "mix."), feed_forward, norms))
        schedule.append(ScheduleEntry(index, entry["mixer"].get("kv_from", index)))
    return ModelSpec(
        architecture=config.architecture,
        hidden_size=width,
        vocab_size=config.vocab,
        max_model_len=config.max_model_len,
        embedding=PartSpec("token_embedding", dict(vocab_size=config.vocab, hidden_size=width, name="embed", init_std=1.0)),
        positions=PartSpec("sinusoidal", dict(hidden_size=width, base=POSITION_BASE)),
        layers=layers,
        schedule=schedule,
        final_norm=PartSpec("layernorm", dict(norm, name="final.norm", weight_factor=config.logit_scale)),
        head=PartSpec("lm_head", dict(vocab_size=config.vocab, hidden_size=width, tied=False, name="head",
                                      init_std=width ** -0.5)),
        normalise_name=_normalise_name,
        checkpoint_name=_checkpoint_name,
    )


register_architecture("Vozirax", VoziraxConfig, build_vozirax_spec, replace=True)
