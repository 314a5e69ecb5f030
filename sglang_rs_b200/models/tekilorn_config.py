"""Validated configuration of a ``Tekilorn`` checkpoint.

The document is nested: ``vocab``, ``width``, ``norm.eps``, ``layers`` (one entry per layer: ``type`` ``attention`` or
``attention_2``, the mixer's sizes under ``mixer``, the feed-forward under ``mlp`` or null) and ``loop`` (``start``, ``stop``,
``times``: layers start .. stop-1 are walked ``times`` times in a row).  The mixer ``attention`` has two maps per head of
``dim`` entries each, ``diff``, and optionally ``q_temp`` (``coef``, ``every``) and ``softcap``; ``attention_2`` has, each
optional, ``rot`` (``base``, ``dims``) and ``mask`` (``size``, ``keep_first``).  A feed-forward is ``kind`` ``dense`` (``ff``,
``limit``) or ``moe`` (``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top`` and, optionally, ``shared.ff``,
``shared.limit``).  Every size and every constant that can differ between checkpoints is read here, layer by layer; nothing is
assumed equal between layers.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Sequence, Tuple, Union

from ..config.model_config import ConfigError, RawConfig, missing_field, required_positive_int

ARCHITECTURE = "Tekilorn"
DIFFERENTIAL_TYPE, WINDOWED_TYPE = "attention", "attention_2"
#: positions a request may reach when the document gives no limit (every position is exact in 32-bit floats)
DEFAULT_MAX_POSITIONS = 1 << 24


def _section(document: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = document.get(key)
    if not isinstance(value, dict):
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be an object")
    return value


def _number(document: Mapping[str, Any], key: str, where: str, positive: bool = False) -> float:
    value = document.get(key)
    if value is None:
        raise missing_field(ARCHITECTURE, where + key)
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be a number, found {value!r}")
    if positive and not value > 0:
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be positive, found {value!r}")
    return float(value)


def _count(document: Mapping[str, Any], key: str, where: str, least: int = 1, default: Optional[int] = None) -> int:
    value = document.get(key)
    if value is None:
        if default is not None:
            return default
        raise missing_field(ARCHITECTURE, where + key)
    if isinstance(value, float) and value.is_integer():
        value = int(value)
    if isinstance(value, bool) or not isinstance(value, int) or value < least:
        raise ConfigError(ARCHITECTURE, f"`{where}{key}` must be an integer of at least {least}, found {value!r}")
    return value


@dataclass(frozen=True)
class DifferentialSizes:
    heads: int
    kv_heads: int
    dim: int                                    # query/key entries of ONE map of a head
    vdim: int
    scale: float
    diff: float
    #: (coef, every) of the query temperature, or None
    temperature: Optional[Tuple[float, int]]
    softcap: Optional[float]


@dataclass(frozen=True)
class RotationSpec:
    base: float
    dims: int                                   # leading entries of a head that turn; the rest pass


@dataclass(frozen=True)
class WindowedSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationSpec]
    window: Optional[int]
    keep_first: int


@dataclass(frozen=True)
class ClampedSizes:
    ff: int
    limit: float


@dataclass(frozen=True)
class RoutedSizes:
    experts: int
    top: int
    expert: ClampedSizes
    shared: Optional[ClampedSizes]


@dataclass(frozen=True)
class LayerSpec:
    kind: str
    mixer: Union[DifferentialSizes, WindowedSizes]
    mlp: Union[ClampedSizes, RoutedSizes, None]


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class TekilornConfig:
    ARCHITECTURE = ARCHITECTURE

    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Sequence[int] = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_raw(cls, raw: RawConfig) -> "TekilornConfig":
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
        loop = None
        if doc.get("loop") is not None:
            section = _section(doc, "loop", "")
            loop = LoopSpec(_count(section, "start", "loop.", 0), _count(section, "stop", "loop.", 0),
                            _count(section, "times", "loop."))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(ARCHITECTURE, f"`loop` must name a stretch of the {len(layers)} layers, "
                                                f"found {loop.start} .. {loop.stop}")
        limit = doc.get("max_position_embeddings")
        if limit is not None:
            limit = required_positive_int(ARCHITECTURE, doc, "max_position_embeddings")
        return cls(vocab, width, eps, layers, loop, limit or DEFAULT_MAX_POSITIONS, tuple(raw.eos_token_ids), doc)


def _rotation(mixer: Mapping[str, Any], where: str, most: int) -> Optional[RotationSpec]:
    """``rot`` of a mixer; None if the document has none or it turns no entries."""
    if mixer.get("rot") is None:
        return None
    rot = _section(mixer, "rot", where)
    inside = where + "rot."
    dims = _count(rot, "dims", inside, 0)
    if dims == 0:
        return None
    base = _number(rot, "base", inside, positive=True)
    if dims % 2 or dims > most:
        raise ConfigError(ARCHITECTURE, f"`{inside}dims` must be an even number of at most {most}, found {dims}")
    return RotationSpec(base, dims)


def _clamped(section: Mapping[str, Any], where: str) -> ClampedSizes:
    return ClampedSizes(_count(section, "ff", where), _number(section, "limit", where, positive=True))


def _mixer(kind: Any, m: Mapping[str, Any], where: str, inside: str) -> Union[DifferentialSizes, WindowedSizes]:
    if kind not in (DIFFERENTIAL_TYPE, WINDOWED_TYPE):
        raise ConfigError(ARCHITECTURE, f"`{where}type` {kind!r} is not a mixer of this design ({DIFFERENTIAL_TYPE}, {WINDOWED_TYPE})")
    heads, kv_heads = _count(m, "heads", inside), _count(m, "kv_heads", inside)
    if heads % kv_heads:
        raise ConfigError(ARCHITECTURE, f"`{inside}heads` {heads} is not a multiple of `kv_heads` {kv_heads}")
    dim, vdim, scale = _count(m, "dim", inside), _count(m, "vdim", inside), _number(m, "scale", inside)
    if kind == DIFFERENTIAL_TYPE:
        temperature = None
        if m.get("q_temp") is not None:
            section = _section(m, "q_temp", inside)
            temperature = (_number(section, "coef", inside + "q_temp."), _count(section, "every", inside + "q_temp."))
        softcap = None if m.get("softcap") is None else _number(m, "softcap", inside, positive=True)
        return DifferentialSizes(heads, kv_heads, dim, vdim, scale, _number(m, "diff", inside), temperature, softcap)
    window, keep_first = None, 0
    if m.get("mask") is not None:
        mask = _section(m, "mask", inside)
        window = _count(mask, "size", inside + "mask.")
        keep_first = _count(mask, "keep_first", inside + "mask.", 0, default=0)
    return WindowedSizes(heads, kv_heads, dim, vdim, scale, _rotation(m, inside, dim), window, keep_first)


def _layer(entry: Any, where: str) -> LayerSpec:
    if not isinstance(entry, dict):
        raise ConfigError(ARCHITECTURE, f"`{where[:-1]}` must be an object")
    kind = entry.get("type")
    mixer = _mixer(kind, _section(entry, "mixer", where), where, where + "mixer.")
    mlp = None
    if entry.get("mlp") is not None:
        f = _section(entry, "mlp", where)
        inside = where + "mlp."
        if f.get("kind") == "dense":
            mlp = _clamped(f, inside)
        elif f.get("kind") == "moe":
            router = _section(f, "router", inside)
            shared = _clamped(_section(f, "shared", inside), inside + "shared.") if f.get("shared") is not None else None
            mlp = RoutedSizes(_count(router, "experts", inside + "router."), _count(router, "top", inside + "router."),
                              _clamped(_section(f, "expert", inside), inside + "expert."), shared)
            if mlp.top > mlp.experts:
                raise ConfigError(ARCHITECTURE, f"`{inside}router.top` exceeds the number of experts")
        else:
            raise ConfigError(ARCHITECTURE, f"`{inside}kind` {f.get('kind')!r} is not a feed-forward of this design (dense, moe)")
    return LayerSpec(kind, mixer, mlp)
