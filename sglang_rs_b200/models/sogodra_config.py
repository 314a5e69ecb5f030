"""Validated configuration of a ``Sogodra`` checkpoint.

The document is nested: ``vocab``, ``width``, ``norm.eps`` and ``layers`` (one entry per layer: ``type`` ``delta``, ``mingru`` or
``parallel``, the mixer's sizes under ``mixer``, the feed-forward under ``mlp`` or null).  A ``delta`` mixer has ``heads``,
``kv_heads``, ``dim``, ``vdim`` and ``conv`` (taps of the short convolution); a ``mingru`` mixer a ``width``; a ``parallel`` mixer
two mixers, ``left`` (windowed attention: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, the window ``mask.size`` and the
rotation ``rot``: ``base``, ``dims`` and, optionally, ``scaling`` with ``factor``, ``low``, ``high``, ``original``) and ``right``
(sizes as a ``delta`` mixer), with the factors ``left_scale`` and ``right_scale``.  A feed-forward is ``kind`` ``dense`` with ``ff``
and ``limit``.  Every size and every constant that can differ between checkpoints is read here, layer by layer; nothing is assumed
equal between layers.  (The ranks of the thin matrix pairs are found in the checkpoint's tensors.)
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Sequence, Tuple, Union

from ..config.model_config import ConfigError, RawConfig, missing_field, required_positive_int

ARCHITECTURE = "Sogodra"
DELTA_TYPE, MINGRU_TYPE, PARALLEL_TYPE = "delta", "mingru", "parallel"
#: positions a request may reach when the document gives no limit (every position is exact in 32-bit floats)
DEFAULT_MAX_POSITIONS = 1 << 24


def _section(document: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = document.get(key)
    if not isinstance(value, dict):
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be an object")
    return value


def _number(document: Mapping[str, Any], key: str, where: str) -> float:
    value = document.get(key)
    if value is None:
        raise missing_field(ARCHITECTURE, where + key)
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be a number, found {value!r}")
    return float(value)


def _count(document: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    value = document.get(key)
    if value is None:
        raise missing_field(ARCHITECTURE, where + key)
    if isinstance(value, bool) or not isinstance(value, int) or value < least:
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be an integer of at least {least}, found {value!r}")
    return value


@dataclass(frozen=True)
class RotationSpec:
    base: float
    dims: int                                   # leading entries of every head that turn; the rest pass
    #: (factor, low, high, original) of the stretching of long wavelengths, or None
    scaling: Optional[Tuple[float, float, float, float]] = None


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    rot: Optional[RotationSpec]


@dataclass(frozen=True)
class DeltaSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class MinGruSizes:
    width: int


@dataclass(frozen=True)
class ParallelSizes:
    left: AttentionSizes
    right: DeltaSizes
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DenseSizes:
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerSpec:
    kind: str
    mixer: Union[DeltaSizes, MinGruSizes, ParallelSizes]
    mlp: Optional[DenseSizes]


@dataclass(frozen=True)
class SogodraConfig:
    ARCHITECTURE = ARCHITECTURE

    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Sequence[int] = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_raw(cls, raw: RawConfig) -> "SogodraConfig":
        doc = raw.document
        vocab = required_positive_int(ARCHITECTURE, doc, "vocab")
        width = required_positive_int(ARCHITECTURE, doc, "width")
        eps = _number(_section(doc, "norm", ""), "eps", "norm.")
        if not eps >= 0:
            raise ConfigError(ARCHITECTURE, "`norm.eps` must be non-negative")
        entries = doc.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(ARCHITECTURE, "`layers` must be a list with at least one layer")
        layers = tuple(_layer(entry, f"layers[{i}].") for i, entry in enumerate(entries))
        limit = doc.get("max_position_embeddings")
        if limit is not None:
            limit = required_positive_int(ARCHITECTURE, doc, "max_position_embeddings")
        return cls(vocab, width, eps, layers, limit or DEFAULT_MAX_POSITIONS, tuple(raw.eos_token_ids), doc)


def _heads(m: Mapping[str, Any], where: str) -> Tuple[int, int]:
    heads, kv_heads = _count(m, "heads", where), _count(m, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(ARCHITECTURE, f"`{where}heads` {heads} is not a multiple of `kv_heads` {kv_heads}")
    return heads, kv_heads


def _rotation(mixer: Mapping[str, Any], where: str, most: int) -> Optional[RotationSpec]:
    """``rot`` of a mixer; None if the document has none or it turns no entries."""
    if mixer.get("rot") is None:
        return None
    rot = _section(mixer, "rot", where)
    inside = where + "rot."
    dims = _count(rot, "dims", inside, 0)
    if dims == 0:
        return None
    base = _number(rot, "base", inside)
    if dims % 2 or dims > most or not base > 0:
        raise ConfigError(ARCHITECTURE, f"`{inside[:-1]}` must rotate an even number of at most {most} entries with a positive base")
    scaling = None
    if rot.get("scaling") is not None:
        s = _section(rot, "scaling", inside)
        scaling = tuple(_number(s, key, inside + "scaling.") for key in ("factor", "low", "high", "original"))
        if not all(value > 0 for value in scaling) or scaling[1] > scaling[2]:
            raise ConfigError(ARCHITECTURE, f"`{inside}scaling` needs positive numbers, `low` no larger than `high`")
    return RotationSpec(base, dims, scaling)


def _attention(m: Mapping[str, Any], where: str) -> AttentionSizes:
    heads, kv_heads = _heads(m, where)
    dim = _count(m, "dim", where)
    window = None
    if m.get("mask") is not None:
        window = _count(_section(m, "mask", where), "size", where + "mask.")
    return AttentionSizes(heads, kv_heads, dim, _count(m, "vdim", where), _number(m, "scale", where), window,
                          _rotation(m, where, dim))


def _delta(m: Mapping[str, Any], where: str) -> DeltaSizes:
    heads, kv_heads = _heads(m, where)
    return DeltaSizes(heads, kv_heads, _count(m, "dim", where), _count(m, "vdim", where), _count(m, "conv", where))


def _layer(entry: Any, where: str) -> LayerSpec:
    if not isinstance(entry, dict):
        raise ConfigError(ARCHITECTURE, f"`{where[:-1]}` must be an object")
    kind = entry.get("type")
    m = _section(entry, "mixer", where)
    inside = where + "mixer."
    if kind == DELTA_TYPE:
        mixer = _delta(m, inside)
    elif kind == MINGRU_TYPE:
        mixer = MinGruSizes(_count(m, "width", inside))
    elif kind == PARALLEL_TYPE:
        mixer = ParallelSizes(_attention(_section(m, "left", inside), inside + "left."),
                              _delta(_section(m, "right", inside), inside + "right."),
                              _number(m, "left_scale", inside), _number(m, "right_scale", inside))
    else:
        raise ConfigError(ARCHITECTURE, f"`{where}type` {kind!r} is not a mixer of this design ({DELTA_TYPE}, {MINGRU_TYPE}, {PARALLEL_TYPE})")
    mlp = None
    if entry.get("mlp") is not None:
        f = _section(entry, "mlp", where)
        inside = where + "mlp."
        if f.get("kind") != "dense":
            raise ConfigError(ARCHITECTURE, f"`{inside}kind` {f.get('kind')!r} is not a feed-forward of this design (dense)")
        mlp = DenseSizes(_count(f, "ff", inside), _number(f, "limit", inside))
    return LayerSpec(kind, mixer, mlp)
