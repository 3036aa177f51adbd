"""Registries of part kinds, one per family, and the interface each family keeps.

Families and what the engine calls on their members (``rt`` is the
:class:`~..engine.runtime.Runtime`, ``ctx`` the step's
:class:`~..engine.batch.StepContext`, ``x`` the fp32 residual stream
``[tokens, width]``, ``h`` a normalised copy of it in the compute type):

``norm``       ``forward(x, rows=None) -> h``
``position``   held by another part through its params (``"position": PartSpec``), with tensors of its
               own if it declares any: by a mixer that keeps keys and values, which calls
               ``rotate_and_store(qkv, ctx, binding, n_heads, n_kv_heads, head_dim)``, or by the
               embedding, which calls ``at_embedding(x, ctx)`` after the lookup (may add to ``x``)
``mixer``      ``cache_request() -> KVRequest | StateRequest | None`` and
               ``forward(h, x, ctx, binding)``: adds its output to ``x``; optionally ``more_cache_requests() -> {name:
               request}`` for what it keeps beside that (handed to it as ``binding.more[name]``)
``ffn``        ``forward(h, x, ctx)``: adds its output to ``x``
``block``      ``forward(x, ctx, binding)``: one layer's arrangement of the above; built with one keyword argument
               per filled slot of its ``LayerSpec`` (``mixer_norm``, ``mixer``, ``ffn_norm``, ``ffn`` and whatever
               the spec adds under ``more``)
``embedding``  ``forward(token_ids, ctx) -> x`` and ``table()`` (for a tied head)
``head``       ``forward(h_rows) -> logits fp32 [rows, vocab]``
``pass_entry`` ``forward(x, x0, ctx)``: acts on the stream right before a scheduled call (``ScheduleEntry.before``); ``x0`` is
               the embedding output, kept for the step if the part sets ``needs_embedding_output``
``pass_exit``  ``forward(x, history, index, ctx)``: acts on the stream right behind scheduled call ``index``
               (``ScheduleEntry.after``); ``history`` fp32 ``[calls + 1, tokens, width]`` is the model's record of the
               step: row 0 the embedding output, row j + 1 the result of call j.  The part files the result of its call
               (``history[index + 1] = x``) and may then rewrite ``x`` from the rows so far.  Where the next block names
               the norms it applies first (``entry_norms``), the call comes with ``then=`` those norms; a part that makes
               their outputs in its own pass returns them (the block takes them as ``entry``), else None
``conv``       ``cache_request() -> StateRequest | None`` and ``forward(h, ctx, binding) -> h'``: reshapes a sublayer's input
               over time (a short causal convolution) and keeps the inputs it still needs per sequence; ``binding`` is
               its own place in the cache (``CacheBinding.more[slot]`` of the call).  Any part of a layer other than the
               mixer that has ``cache_request`` gets such a place

``scale``      ``weight``: fp32 ``[width]``, a factor per entry on what a sublayer adds; the block hands it to a mixer or
               feed-forward that sets ``scales_output`` as ``forward(..., out_scale=weight)``

Every member also has ``declare(spec) -> {local tensor name: TensorDecl}`` (a
classmethod: what it reads from the weight file under ``spec.prefix``) and is
constructed as ``cls(spec, tensors, rt, **context)`` with its declared tensors.
No part knows which model it is in.

Optional extras, for fusions that cross two parts.  A part without them works unchanged; the caller falls
back to the plain path.

``position``   ``fused_rotation() -> (inv_freq, rotary_dim) | None``: all the part does to q, k, v is the
               rotation of pairs and the append of ``rotate_and_store``, so a mixer may let its attention
               kernel do both.
``norm``       ``deferred(n_tokens, name) -> kernels.DeferredNorm | None``: the norm split over the products
               around it (the one before fills it, the one after applies the scale).
``mixer``/``ffn``  class attribute ``defers_norm = True``: ``forward`` accepts a filled ``DeferredNorm`` as
               ``h`` and a keyword ``then_norm=`` (a ``DeferredNorm`` to fill with the part's last,
               residual-adding product) and returns whether it filled it.
``block``      property ``entry_norm`` (the norm it applies first, if the block before may fill its deferred
               form) and ``forward(x, ctx, binding, entry=None, next_norm=None) -> DeferredNorm | None``.
``mixer``      ``step_plan(ctx, binding) -> hashable | None``: what the part's launches for this step depend on
               beside the step's padded shape (its attention kernel's split, which follows the live sequences).
               A recorded decode step is replayed only for a step whose mixers give the same answers.
any part       class attribute ``takes_padding_rows = True``: token rows that belong to no sequence (index -1)
               do it no harm, so its model's short prompt steps may be padded to a shape and replayed.
"""
from __future__ import annotations

from dataclasses import dataclass

FAMILIES = ("norm", "position", "mixer", "ffn", "block", "embedding", "head", "pass_entry", "conv", "pass_exit", "scale")
_PARTS: dict[str, dict[str, type]] = {f: {} for f in FAMILIES}


@dataclass(frozen=True)
class FreeDim:
    """A size that the weight file decides (an inner rank that no configuration key gives): any positive value is
    accepted, the part reads it from its tensor, and random weights are drawn with ``default``."""
    default: int


def resolved_shape(shape) -> tuple:
    """A declared shape with every free size at its default (for random weights and parameter counts)."""
    return tuple(int(d.default) if isinstance(d, FreeDim) else int(d) for d in shape)


@dataclass(frozen=True)
class TensorDecl:
    shape: tuple                    # sizes; an entry may be a FreeDim
    # "matrix" | "norm_scale" | "bias" | "table" | "mix": floating tensors (the role says how random weights draw them);
    # "int_table": the only role a file may store as integers
    role: str = "matrix"
    high: int = 0                   # of an int_table: entries are 0 .. high - 1 (random weights: the entries of a row differ)


def register_part(family: str, kind: str, cls: type, *, replace: bool = False) -> None:
    if family not in _PARTS:
        raise ValueError(f"unknown part family {family!r}; families are {FAMILIES}")
    if kind in _PARTS[family] and not replace:
        raise ValueError(f"{family} part {kind!r} is already registered")
    _PARTS[family][kind] = cls


def get_part(family: str, kind: str) -> type:
    try:
        return _PARTS[family][kind]
    except KeyError:
        known = ", ".join(sorted(_PARTS.get(family, {}))) or "none"
        raise KeyError(f"no {family} part of kind {kind!r} is registered (known: {known})") from None


def nested_declare(family: str, ps) -> dict:
    """The tensors of a part that another part holds in its params (a mixer's or an embedding's position
    part): its own declarations under its own prefix, which is relative to the holder's."""
    return {ps.prefix + name: decl for name, decl in get_part(family, ps.kind).declare(ps).items()}


def nested_build(family: str, ps, tensors: dict, rt, **context):
    """Build such a part from the holder's tensors (see :func:`nested_declare`)."""
    cls = get_part(family, ps.kind)
    return cls(ps, {name: tensors[ps.prefix + name] for name in cls.declare(ps)}, rt, **context)


def part(family: str, kind: str):
    """Class decorator: ``@part("mixer", "gqa")``."""
    def deco(cls):
        register_part(family, kind, cls)
        cls.family, cls.kind = family, kind
        return cls
    return deco
