"""The Zomurax decoder as a recipe of parts.

Embedding rows as they are; layers of the arrangement ``postnorm`` — the branches read the stream itself, and an RMS norm
with one gain for all coordinates (``rms`` with ``one_gain``) stands behind each sum and replaces the stream —; a mixer per
layer: ``distance_attention`` (grouped queries, unit-size q and k heads, a temperature on the queries, a bias by distance, a
sink, values mixed with those of the first layer that mixes) or ``latent_attention`` (queries straight from the stream,
a rotation of (i, i + dims/2), a sliding window); a feed-forward per layer or none: ``routed_experts`` whose experts a table
gives each token id, with a gated ``swiglu`` beside them that every token runs; a last norm and an untied head whose logits
are capped.  Tensor names: ``embed``, ``head``, ``final.norm`` and per layer i ``l<i>.norm1`` (behind the mixer),
``l<i>.norm2`` (behind the feed-forward), ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

import re

from ..config.registry import Architecture, register_architecture
from ..config.zomurax import ARCHITECTURE, ZomuraxConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 24        # the design sets no limit: angles, biases and temperatures are computed on the fly


def _mixer(c: ZomuraxConfig, layer, value_mix, prefix: str) -> PartSpec:
    m = layer.mixer
    if layer.type == "attention":
        return PartSpec("distance_attention", {
            "width": c.width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
            "eps": c.norm_eps, "unit_qk": True, "temperature": (m.temp_coef, m.temp_every) if m.temp_every else None,
            "distance_bias": True, "sink": True, "value_mix": value_mix}, prefix)
    return PartSpec("latent_attention", {
        "width": c.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": 0,
        "scale": m.scale, "rot_base": m.rot_base, "rot_dims": m.rot_dims, "pairing": 0, "window": m.window, "eps": c.norm_eps},
        prefix)


def _ffn(c: ZomuraxConfig, mlp, prefix: str) -> PartSpec:
    beside = None
    if mlp.shared_ff:
        beside = PartSpec("swiglu", {"width": c.width, "inner": mlp.shared_ff, "activation": "silu", "names": ("gate", "up", "down")},
                          "shared.")
    return PartSpec("routed_experts", {"width": c.width, "inner": mlp.ff, "experts": mlp.experts, "top": mlp.top, "activation": "silu",
                                       "scoring": "token_table", "vocab": c.vocab, "beside": beside}, prefix)


def zomurax_model_spec(c: ZomuraxConfig) -> ModelSpec:
    def norm(name):
        return PartSpec("rms", {"width": c.width, "eps": c.norm_eps, "tensor": "", "one_gain": True}, name)
    layers, schedule, kept = [], [], False
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        value_mix = None
        if layer.type == "attention" and layer.mixer.v_mix:
            value_mix = "later" if kept else "first"
            kept = True
        layers.append(LayerSpec(
            block="postnorm", mixer_norm=norm(p + "norm1"), mixer=_mixer(c, layer, value_mix, p + "mix."),
            ffn_norm=norm(p + "norm2") if layer.mlp is not None else None,
            ffn=_ffn(c, layer.mlp, p + "mlp.") if layer.mlp is not None else None, block_params={"alpha": c.alpha}))
        schedule.append(ScheduleEntry(i))
    return ModelSpec(
        architecture=c.architecture, vocab_size=c.vocab, width=c.width, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_table", {"vocab": c.vocab, "width": c.width, "tensor": "embed"}, ""),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab": c.vocab, "width": c.width, "tied": False, "tensor": "head",
                                      "softcap": c.logit_softcap}, ""),
        stop_ids=())


# The first layer that mixes values has nothing to mix with: its mixing number is not used, nor is one of a layer that does
# not mix; a layer without a feed-forward has no second norm.  A file that carries them all the same is not refused.
_UNUSED = re.compile(r"^l\d+\.(norm2|mix\.vmix)$")

register_architecture(Architecture(ARCHITECTURE, ZomuraxConfig.from_dict, zomurax_model_spec,
                                   tolerated_extra_tensors=lambda name: bool(_UNUSED.match(name))))
