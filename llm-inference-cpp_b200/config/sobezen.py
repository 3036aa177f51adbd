"""Typed configuration of the Sobezen decoder.

config.json names the design with ``"architecture": "Sobezen"`` and gives every size and every constant that can
differ between models of the design:

* ``vocab``, ``width``; ``embedding.scale`` (what the looked-up rows are multiplied by); ``norm.eps`` (of every RMS
  norm); ``logit_scale`` (what the logits are multiplied by);
* ``layers``: a list, one entry per layer, with ``type`` (``latent_attention``, ``channel_delta`` or ``attention``),
  ``mixer`` (that mixer's sizes) and ``mlp`` (``null`` for a layer without a feed-forward, else ``kind`` ``dense`` with
  ``ff`` and ``limit``).

  - a ``latent_attention`` mixer: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``, ``scale``; ``rot`` with
    ``base``, ``dims`` and an optional ``scaling`` of ``factor``, ``original``, ``fast``, ``slow``; an optional ``kv_from``
    (the index of an earlier latent layer whose cached rows this one reads);
  - a ``channel_delta`` mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps); the inner sizes of its two
    low-rank paths are read from the file's tensors;
  - an ``attention`` mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim`` (equal to ``dim``: the values are the keys),
    ``scale``, ``rot``.

No size has a default: a missing or ill-typed key is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .garodra import _number, _obj, _uint
from .gemosun import RotationScaling
from .llama import MAX_LAYERS, MAX_VOCAB, ConfigError

ARCHITECTURE = "Sobezen"
MAX_TAPS = 16


@dataclass(frozen=True)
class Rotation:
    base: float = 1.0
    dims: int = 0                               # 0: no rotation
    scaling: Optional[RotationScaling] = None


@dataclass(frozen=True)
class SharedLatentSizes:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Rotation
    kv_from: Optional[int] = None               # the layer whose cached rows are read (None: rows of its own)


@dataclass(frozen=True)
class ChannelDeltaSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class KeyValueAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: Rotation


@dataclass(frozen=True)
class BoundedFeedForwardSizes:
    ff: int
    limit: float


@dataclass(frozen=True)
class SobezenLayer:
    type: str                                   # "latent_attention" | "channel_delta" | "attention"
    mixer: Any
    mlp: Optional[BoundedFeedForwardSizes]


def _rotation(m: Mapping[str, Any], where: str, limit: int, limit_name: str) -> Rotation:
    if m.get("rot") is None:
        return Rotation()
    rot, rw = _obj(m, "rot", where), where + "rot."
    dims = _uint(rot, "dims", rw, least=0)
    if dims % 2 or dims > limit:
        raise ConfigError(f'config: {rw}"dims" must be even and at most "{limit_name}"')
    if not dims:
        return Rotation()
    base, scaling = _number(rot, "base", rw), None
    if rot.get("scaling") is not None:
        s, sw = _obj(rot, "scaling", rw), rw + "scaling."
        scaling = RotationScaling(factor=_number(s, "factor", sw), original=_number(s, "original", sw),
                                  fast=_number(s, "fast", sw), slow=_number(s, "slow", sw))
        if base <= 1.0:
            raise ConfigError(f'config: {rw}"base" must be larger than 1 where the rotation is scaled')
    return Rotation(base=base, dims=dims, scaling=scaling)


def _latent(m: Mapping[str, Any], where: str, i: int, layers: list) -> SharedLatentSizes:
    rot_dim = _uint(m, "rot_dim", where, least=0)
    s = SharedLatentSizes(
        heads=_uint(m, "heads", where), dim=_uint(m, "dim", where), rot_dim=rot_dim, vdim=_uint(m, "vdim", where),
        kv_rank=_uint(m, "kv_rank", where), q_rank=_uint(m, "q_rank", where), scale=_number(m, "scale", where),
        rot=_rotation(m, where, rot_dim, "rot_dim"),
        kv_from=_uint(m, "kv_from", where, MAX_LAYERS, least=0) if m.get("kv_from") is not None else None)
    if s.kv_from is not None:
        src = layers[s.kv_from] if s.kv_from < i else None
        if src is None or src.type != "latent_attention" or src.mixer.kv_from is not None:
            raise ConfigError(f'config: {where}"kv_from" must name an earlier "latent_attention" layer with rows of its own')
        if (src.mixer.kv_rank, src.mixer.rot_dim, src.mixer.rot) != (s.kv_rank, s.rot_dim, s.rot):
            raise ConfigError(f'config: {where}"kv_from": layer {s.kv_from} keeps rows of another size or rotation')
    return s


def _grouped(m: Mapping[str, Any], where: str) -> tuple:
    heads, kv_heads = _uint(m, "heads", where), _uint(m, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f'config: {where}"heads" is not a multiple of "kv_heads"')
    return heads, kv_heads


def _delta(m: Mapping[str, Any], where: str) -> ChannelDeltaSizes:
    heads, kv_heads = _grouped(m, where)
    return ChannelDeltaSizes(heads=heads, kv_heads=kv_heads, dim=_uint(m, "dim", where), vdim=_uint(m, "vdim", where),
                             conv=_uint(m, "conv", where, MAX_TAPS))


def _attention(m: Mapping[str, Any], where: str) -> KeyValueAttentionSizes:
    heads, kv_heads = _grouped(m, where)
    dim = _uint(m, "dim", where)
    if _uint(m, "vdim", where) != dim:
        raise ConfigError(f'config: {where}"vdim" must equal "dim": the values are the keys as projected')
    return KeyValueAttentionSizes(heads=heads, kv_heads=kv_heads, dim=dim, scale=_number(m, "scale", where),
                                  rot=_rotation(m, where, dim, "dim"))


def _feed_forward(mlp: Mapping[str, Any], where: str) -> BoundedFeedForwardSizes:
    if mlp.get("kind") != "dense":
        raise ConfigError(f'config: {where}"kind" must be "dense", not {mlp.get("kind")!r}')
    return BoundedFeedForwardSizes(ff=_uint(mlp, "ff", where), limit=_number(mlp, "limit", where))


@dataclass(frozen=True)
class SobezenConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    logit_scale: float
    layers: tuple
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, root: Mapping[str, Any]) -> "SobezenConfig":
        vocab = _uint(root, "vocab", "", MAX_VOCAB)
        width = _uint(root, "width", "")
        scale = _number(_obj(root, "embedding", ""), "scale", "embedding.", positive=False)
        eps = _number(_obj(root, "norm", ""), "eps", "norm.")
        logit_scale = _number(root, "logit_scale", "", positive=False)
        raw = root.get("layers")
        if not isinstance(raw, list) or not raw or len(raw) > MAX_LAYERS:
            raise ConfigError(f'config: "layers" must be a list of 1..{MAX_LAYERS} layers')
        layers: list = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config: layers[{i}] must be an object")
            kind = entry.get("type")
            m, mw = _obj(entry, "mixer", where), where + "mixer."
            if kind == "latent_attention":
                mixer = _latent(m, mw, i, layers)
            elif kind == "channel_delta":
                mixer = _delta(m, mw)
            elif kind == "attention":
                mixer = _attention(m, mw)
            else:
                raise ConfigError(f'config: {where}"type" must be "latent_attention", "channel_delta" or "attention", not {kind!r}')
            mlp = entry.get("mlp")
            if mlp is not None and not isinstance(mlp, dict):
                raise ConfigError(f'config: {where}"mlp" must be an object or null')
            layers.append(SobezenLayer(kind, mixer, _feed_forward(mlp, where + "mlp.") if mlp is not None else None))
        return cls(vocab=vocab, width=width, embedding_scale=scale, norm_eps=eps, logit_scale=logit_scale, layers=tuple(layers))
