"""The Sobezen decoder as a recipe of parts.

Embedding rows times a constant; layers of the arrangement ``prenorm`` with RMS norms and a learned factor per entry on
what each sublayer adds (``vector`` parts in the slots ``mixer_scale`` and ``ffn_scale``); a mixer per layer:
``latent_attention`` (queries through a latent, a rotation of neighbouring entries with stretched frequencies, optionally
on another layer's rows), ``channel_delta`` (the gated delta rule with a decay per key channel) or ``gated_attention``
(grouped queries, biases on q and k, values that are the keys before the rotation; none of its other pieces); a feed-forward
per layer or none (``swiglu`` with the bounded gate and biases); a last RMS norm and an untied head whose logits are
multiplied by a constant.  Tensor names: ``embed``, ``head``, ``final.norm`` and per layer i ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.ls1``, ``l<i>.norm2``, ``l<i>.mlp.*``, ``l<i>.ls2``.

A layer that reads layer j's rows becomes a scheduled call with ``cache_of`` = j: it writes nothing into that cache.
"""
from __future__ import annotations

import re

from ..config.registry import Architecture, register_architecture
from ..config.sobezen import ARCHITECTURE, SobezenConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 24        # the design sets no limit: angles are computed on the fly, and a state has no length
GATE_ALPHA = 1.702             # the slope inside the gate's logistic function, fixed by the design


def _position(rot, head_dim: int):
    if not rot.dims:
        return PartSpec("none")
    s = rot.scaling
    return PartSpec("rotary_pairs", {
        "head_dim": head_dim, "rotary_dim": rot.dims, "theta": rot.base,
        "scaling": None if s is None else {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}})


def _mixer(c: SobezenConfig, layer, prefix: str) -> PartSpec:
    m = layer.mixer
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", {
            "width": c.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
            "q_rank": m.q_rank, "scale": m.scale, "position": _position(m.rot, m.rot_dim), "shares_kv": m.kv_from is not None,
            "eps": c.norm_eps}, prefix)
    if layer.type == "channel_delta":
        return PartSpec("channel_delta", {"width": c.width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
                                          "conv": m.conv, "eps": c.norm_eps}, prefix)
    return PartSpec("gated_attention", {
        "width": c.width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.dim, "scale": m.scale, "bias": True,
        "out_bias": False, "values_from_keys": True, "position": _position(m.rot, m.dim)}, prefix)


def sobezen_model_spec(c: SobezenConfig) -> ModelSpec:
    def norm(name):
        return PartSpec("rms", {"width": c.width, "eps": c.norm_eps, "tensor": ""}, name)

    def vector(name):
        return PartSpec("vector", {"width": c.width}, name)
    layers, schedule = [], []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        more = [("mixer_scale", "scale", vector(p + "ls1"))]
        ffn = None
        if layer.mlp is not None:
            more.append(("ffn_scale", "scale", vector(p + "ls2")))
            ffn = PartSpec("swiglu", {"width": c.width, "inner": layer.mlp.ff, "activation": "bounded", "alpha": GATE_ALPHA,
                                      "limit": layer.mlp.limit, "bias": True, "names": ("gate", "up", "down")}, p + "mlp.")
        layers.append(LayerSpec(
            block="prenorm", mixer_norm=norm(p + "norm1"), mixer=_mixer(c, layer, p + "mix."),
            ffn_norm=norm(p + "norm2") if ffn is not None else None, ffn=ffn, more=tuple(more)))
        schedule.append(ScheduleEntry(i, cache_of=getattr(layer.mixer, "kv_from", None)))
    return ModelSpec(
        architecture=c.architecture, vocab_size=c.vocab, width=c.width, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_table", {"vocab": c.vocab, "width": c.width, "scale": c.embedding_scale,
                                           "tensor": "embed"}, ""),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab": c.vocab, "width": c.width, "tied": False, "tensor": "head",
                                      "scale": c.logit_scale}, ""),
        stop_ids=())


# a layer without a feed-forward has no second norm and no second factor; a file that carries them all the same is not
# refused for it
_UNUSED = re.compile(r"^l\d+\.(norm2|ls2)$")

register_architecture(Architecture(ARCHITECTURE, SobezenConfig.from_dict, sobezen_model_spec,
                                   tolerated_extra_tensors=lambda name: bool(_UNUSED.match(name))))
