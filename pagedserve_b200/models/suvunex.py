"""Suvunex as a ModelSpec.

Token table times a constant -> layers in the listed order -> the model's norm -> logits against a table of their own,
times a constant (which is folded into that norm's gain).  Every layer is :class:`SandwichNormBlock`: norms with a gain of
one number before and after each sublayer, a factor per coordinate on the normed results, a short convolution over time on
what the mixer reads.  ``parallel`` layers are :class:`ParallelMixers` of :class:`RotaryAttention` (biased projections,
slowed rotation, heads divided by their length, a one in the denominator) and :class:`GatedLinearAttention`;
``attention`` layers are :class:`RotaryAttention` whose values are the keys as projected, with head norms, learned sinks
and mixed heads.  The feed-forward is the gated :class:`DenseMLP` with the tanh form of gelu, or none.

Tensor names in a checkpoint: ``embed``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm1b``,
``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.ls1``, ``l<i>.ls2``, ``l<i>.canon1``, ``l<i>.mix.*`` (``l<i>.mix.left.*`` and
``l<i>.mix.right.*`` in a parallel layer), ``l<i>.mlp.{gate,up,down}``; matrices are stored ``[out, in]``.
"""

from __future__ import annotations

import re
from typing import Optional

from pagedserve_b200.config.registry import register_architecture
from pagedserve_b200.config.suvunex import SuvunexConfig
from pagedserve_b200.models.spec import LayerSpec, ModelSpec, PartSpec

# parts shared with other models name their tensors "<name>.weight"; this design stores the bare name
_BARE = re.compile(r"^(embed|head|final\.norm|l\d+\.(norm1|norm2|norm1b|norm2b|mlp\.gate|mlp\.up|mlp\.down))$")
_SUFFIX = ".weight"


def _normalise_name(name: str) -> Optional[str]:
    return name + _SUFFIX if _BARE.match(name) else name


def _checkpoint_name(name: str) -> str:
    if name.endswith(_SUFFIX) and _BARE.match(name[:-len(_SUFFIX)]):
        return name[:-len(_SUFFIX)]
    return name


def _attention(mixer: dict, width: int, eps: float, names: str, **extras) -> dict:
    """Parameters of :class:`RotaryAttention` that both kinds of layer share; ``names``: what its tensors begin with."""
    rot = mixer.get("rot")
    return dict(hidden_size=width, n_heads=mixer["heads"], n_kv_heads=mixer["kv_heads"], head_dim=mixer["dim"],
                v_dim=mixer["vdim"], scale=mixer["scale"], window=None, softcap=None,
                rotary=dict(dims=rot["dims"], base=rot["base"], interleaved=False, scaling=rot.get("scaling")) if rot else None,
                q_name=names + "q", k_name=names + "k", out_name=names + "o", bias=True, init_std=width ** -0.5,
                out_init_std=(mixer["heads"] * mixer["vdim"]) ** -0.5, **extras)


def build_suvunex_spec(config: SuvunexConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = dict(width=width, eps=eps, has_mean=False, has_bias=False, scalar=True, init_std=0.1)
    width_std = width ** -0.5
    layers = []
    for index, entry in enumerate(config.layers):
        prefix = f"l{index}."
        mixer = entry["mixer"]
        if entry["type"] == "parallel":
            right = mixer["right"]
            left = _attention(mixer["left"], width, eps, "", v_name="v", out_bias=True, unit_sink=True,
                              head_norm=dict(q_name=None, k_name=None, eps=eps))
            recurrent = dict(hidden_size=width, n_heads=right["heads"], head_dim=right["dim"], v_dim=right["vdim"],
                             tau=right["tau"], eps=eps, init_std=width_std,
                             out_init_std=(right["heads"] * right["vdim"]) ** -0.5)
            mixer_spec = PartSpec("parallel", dict(hidden_size=width, mixers=[
                ("rotary_attention", left, "left.", mixer["left_scale"]),
                ("gated_linear_attention", recurrent, "right.", mixer["right_scale"])]), prefix + "mix.")
        else:
            mixer_spec = PartSpec("rotary_attention", _attention(
                mixer, width, eps, "mix.", v_name=None, sink_name="mix.sink", talk_name="mix.talk",
                head_norm=dict(q_name="mix.q.norm", k_name="mix.k.norm", eps=eps)), prefix)
        norms = {"pre_mixer": PartSpec("layernorm", dict(norm, name="norm1"), prefix),
                 "post_mixer": PartSpec("layernorm", dict(norm, name="norm1b"), prefix)}
        scales = {"mixer": "ls1"}
        if entry["mlp"] is None:
            feed_forward = PartSpec("none")
        else:
            norms["pre_feed_forward"] = PartSpec("layernorm", dict(norm, name="norm2"), prefix)
            norms["post_feed_forward"] = PartSpec("layernorm", dict(norm, name="norm2b"), prefix)
            scales["feed_forward"] = "ls2"
            feed_forward = PartSpec("dense_mlp", dict(
                hidden_size=width, inner_size=entry["mlp"]["ff"], activation="gelu_tanh", has_bias=False,
                stored_in_out=False, gate_name="mlp.gate", up_name="mlp.up", down_name="mlp.down", init_std=width_std,
                out_init_std=entry["mlp"]["ff"] ** -0.5), prefix)
        block = PartSpec("sandwich_norm", dict(scales=scales, conv=dict(taps=config.canon_taps, name="canon1")), prefix)
        layers.append(LayerSpec(block, mixer_spec, feed_forward, norms))
    return ModelSpec(
        architecture=config.architecture,
        hidden_size=width,
        vocab_size=config.vocab,
        max_model_len=config.max_model_len,
        embedding=PartSpec("token_pair_embedding", dict(vocab_size=config.vocab, hidden_size=width, name="embed",
                                                        scale=config.embedding_scale, pair=None, init_std=1.0)),
        positions=PartSpec("none"),
        layers=layers,
        schedule=[],
        final_norm=PartSpec("layernorm", dict(norm, name="final.norm", weight_factor=config.logit_scale)),
        head=PartSpec("lm_head", dict(vocab_size=config.vocab, hidden_size=width, tied=False, name="head",
                                      init_std=width_std)),
        normalise_name=_normalise_name,
        checkpoint_name=_checkpoint_name,
    )


register_architecture("Suvunex", SuvunexConfig, build_suvunex_spec, replace=True)
