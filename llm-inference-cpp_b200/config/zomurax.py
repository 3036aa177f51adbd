"""Typed configuration of the Zomurax decoder.

config.json names the design with ``"architecture": "Zomurax"`` and gives every size and every constant that can
differ between models of the design:

* ``vocab``, ``width``; ``norm.eps`` (of every RMS norm); ``postln_alpha`` (what the stream is multiplied by before a
  branch joins it); ``logit_softcap`` (the cap on the logits);
* ``layers``: a list, one entry per layer, with ``type`` (``attention`` or ``latent_attention``), ``mixer`` (that mixer's
  sizes) and ``mlp`` (``null`` for a layer without a feed-forward, else ``kind`` ``moe``).

  - an ``attention`` mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``; optional ``q_temp`` with ``coef`` and
    ``every``, optional ``v_mix`` (whether the layer takes part in the mixing of values; all that do have equal
    ``kv_heads`` * ``vdim``);
  - a ``latent_attention`` mixer: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``; optional ``rot`` with
    ``base`` and ``dims``, optional ``mask.size`` (the window);
  - a ``moe`` feed-forward: ``expert.ff``, ``router`` with ``experts`` and ``top``, and an optional ``shared.ff``.

No size has a default: a missing or ill-typed key is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .garodra import _number, _obj, _uint
from .llama import MAX_LAYERS, MAX_VOCAB, ConfigError

ARCHITECTURE = "Zomurax"
MAX_EXPERTS = 256
MAX_TOP = 32
MAX_SPAN = 1 << 30


@dataclass(frozen=True)
class DistanceAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 0      # 0: no temperature
    v_mix: bool = False


@dataclass(frozen=True)
class WindowLatentSizes:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float = 1.0
    rot_dims: int = 0        # 0: no rotation
    window: int = 0          # 0: every earlier position


@dataclass(frozen=True)
class TableExpertsSizes:
    ff: int
    experts: int
    top: int
    shared_ff: int = 0       # 0: no shared expert


@dataclass(frozen=True)
class ZomuraxLayer:
    type: str                # "attention" | "latent_attention"
    mixer: Any
    mlp: Optional[TableExpertsSizes]


def _span(root: Mapping[str, Any], key: str, where: str) -> int:
    """A count of positions; a number without a fraction will do."""
    v = root.get(key)
    if isinstance(v, float) and v.is_integer():
        root = {key: int(v)}
    return _uint(root, key, where, MAX_SPAN)


def _attention(m: Mapping[str, Any], where: str) -> DistanceAttentionSizes:
    heads, kv_heads = _uint(m, "heads", where), _uint(m, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f'config: {where}"heads" is not a multiple of "kv_heads"')
    coef, every = 0.0, 0
    if m.get("q_temp") is not None:
        t = _obj(m, "q_temp", where)
        coef = _number(t, "coef", where + "q_temp.", positive=False)
        every = _span(t, "every", where + "q_temp.")
    mix = m.get("v_mix", False)
    if mix is not None and not isinstance(mix, bool):
        raise ConfigError(f'config: {where}"v_mix" must be true or false')
    return DistanceAttentionSizes(heads=heads, kv_heads=kv_heads, dim=_uint(m, "dim", where), vdim=_uint(m, "vdim", where),
                                  scale=_number(m, "scale", where), temp_coef=coef, temp_every=every, v_mix=bool(mix))


def _latent(m: Mapping[str, Any], where: str) -> WindowLatentSizes:
    rot_dim = _uint(m, "rot_dim", where, least=0)
    base, dims = 1.0, 0
    if m.get("rot") is not None:
        rot = _obj(m, "rot", where)
        dims = _uint(rot, "dims", where + "rot.", least=0)
        if dims % 2 or dims > rot_dim:
            raise ConfigError(f'config: {where}rot."dims" must be even and at most "rot_dim"')
        if dims:
            base = _number(rot, "base", where + "rot.")
    return WindowLatentSizes(
        heads=_uint(m, "heads", where), dim=_uint(m, "dim", where), rot_dim=rot_dim, vdim=_uint(m, "vdim", where),
        kv_rank=_uint(m, "kv_rank", where), scale=_number(m, "scale", where), rot_base=base, rot_dims=dims,
        window=_span(_obj(m, "mask", where), "size", where + "mask.") if m.get("mask") is not None else 0)


def _experts(mlp: Mapping[str, Any], where: str) -> TableExpertsSizes:
    if mlp.get("kind") != "moe":
        raise ConfigError(f'config: {where}"kind" must be "moe"')
    r = _obj(mlp, "router", where)
    experts = _uint(r, "experts", where + "router.", MAX_EXPERTS)
    top = _uint(r, "top", where + "router.", MAX_TOP)
    if top > experts:
        raise ConfigError(f'config: {where}router."top" is larger than "experts"')
    return TableExpertsSizes(ff=_uint(_obj(mlp, "expert", where), "ff", where + "expert."), experts=experts, top=top,
                             shared_ff=_uint(_obj(mlp, "shared", where), "ff", where + "shared.") if mlp.get("shared") is not None else 0)


@dataclass(frozen=True)
class ZomuraxConfig:
    vocab: int
    width: int
    norm_eps: float
    alpha: float
    logit_softcap: float     # 0: logits are not capped
    layers: tuple
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, root: Mapping[str, Any]) -> "ZomuraxConfig":
        vocab = _uint(root, "vocab", "", MAX_VOCAB)
        width = _uint(root, "width", "")
        eps = _number(_obj(root, "norm", ""), "eps", "norm.")
        alpha = _number(root, "postln_alpha", "", positive=False)
        cap = 0.0
        if root.get("logit_softcap") is not None:
            cap = _number(root, "logit_softcap", "", positive=False)
            if cap < 0:
                raise ConfigError('config: "logit_softcap" must not be negative')
        raw = root.get("layers")
        if not isinstance(raw, list) or not raw or len(raw) > MAX_LAYERS:
            raise ConfigError(f'config: "layers" must be a list of 1..{MAX_LAYERS} layers')
        layers, mixed = [], None
        for i, entry in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config: layers[{i}] must be an object")
            kind = entry.get("type")
            m = _obj(entry, "mixer", where)
            if kind == "attention":
                mixer = _attention(m, where + "mixer.")
                if mixer.v_mix:
                    size = mixer.kv_heads * mixer.vdim
                    if mixed is not None and size != mixed:
                        raise ConfigError(f'config: {where}mixer: layers that mix values need equal "kv_heads" * "vdim"')
                    mixed = size
            elif kind == "latent_attention":
                mixer = _latent(m, where + "mixer.")
            else:
                raise ConfigError(f'config: {where}"type" must be "attention" or "latent_attention", not {kind!r}')
            mlp = entry.get("mlp")
            if mlp is not None and not isinstance(mlp, dict):
                raise ConfigError(f'config: {where}"mlp" must be an object or null')
            layers.append(ZomuraxLayer(kind, mixer, _experts(mlp, where + "mlp.") if mlp is not None else None))
        return cls(vocab=vocab, width=width, norm_eps=eps, alpha=alpha, logit_softcap=cap, layers=tuple(layers))
