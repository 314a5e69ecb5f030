"""Interfaces of the parts a model is put together from.

A model is a list of blocks; a block arranges a mixer, a feed-forward and norms; a mixer
may use a position encoding.  Each part is constructed from its sizes, its constants and
the checkpoint names of its tensors, and is chosen layer by layer by the architecture's
builder.  No part knows which model it is in.

What each kind must offer:

* every part: ``tensor_specs()`` (checkpoint name -> :class:`TensorSpec`) and
  ``load(tensors, device, dtype)``;
* :class:`Norm`: ``add_norm(residual, delta, out_dtype, row_index=None)``;
* :class:`PositionEncoding`: ``fused_rotary()``: what the fused q/k kernel rotates with: a
  frequency table, or a function from the step's positions to the angle of every (row, pair),
  which covers any encoding of the rotary family; None leaves q and k alone;
* :class:`Mixer`: ``cache_need()`` and ``forward(ctx, cache, x) -> y``;
* :class:`FeedForward`: ``forward(ctx, x) -> y``;
* a block: ``forward(ctx, cache, residual, delta) -> (residual, delta)`` where the hidden
  state is ``residual + delta`` (the sum is taken, in 32-bit, by the next norm).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Mapping, Optional, Tuple, Union

import torch


#: a dimension of a :class:`TensorSpec` whose size the checkpoint decides
FREE = -1


@dataclass(frozen=True)
class TensorSpec:
    """Shape of a checkpoint tensor and how the random-weights mode fills it:
    ``normal`` N(0, 0.02), ``scale`` 1 + U(-0.1, 0.1), ``zeros``.

    A dimension of ``FREE`` takes whatever size the checkpoint's tensor has there (a rank that no configuration names);
    the part reads it at load.  ``free_size`` is the size the random-weights mode gives it."""
    shape: Tuple[int, ...]
    init: str = "normal"
    free_size: int = 1

    @property
    def sample_shape(self) -> Tuple[int, ...]:
        """The shape with every free dimension filled in, for weights that are made up."""
        return tuple(self.free_size if size == FREE else size for size in self.shape)


@dataclass(frozen=True)
class PagedKV:
    """A mixer that keeps keys and values per token.  ``window`` None keeps all of them;
    a number keeps only what the last ``window`` positions can still see.  ``values`` False keeps one
    row per token and kv head only (a latent that serves as key and as value): no value pool is made.
    ``value_dim``: the width of a value row where it differs from the keys' ``head_dim`` (None: the same).
    ``keep_first``: with a window, how many of a sequence's first tokens every later position sees beside it (their pages
    stay)."""
    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    values: bool = True
    value_dim: Optional[int] = None
    keep_first: int = 0

    def __post_init__(self):
        if self.keep_first < 0 or (self.keep_first and self.window is None):
            raise ValueError("first tokens are kept behind a window: there is none, or their number is negative")

    @property
    def value_width(self) -> int:
        return 0 if not self.values else (self.value_dim if self.value_dim is not None else self.head_dim)


@dataclass(frozen=True)
class RequestState:
    """A mixer that keeps a fixed-size state per request (shape without the slot axis).
    ``dtype`` None means the compute dtype."""
    shape: Tuple[int, ...]
    dtype: Optional[torch.dtype] = None


@dataclass(frozen=True)
class JointNeed:
    """Several needs of one layer call: a mixer made of mixers that each keep something of their own (keys and values
    beside a state, say).  The call is handed one cache whose ``parts`` are the needs' caches in this order."""
    parts: Tuple[Union[PagedKV, RequestState, None], ...]


CacheNeed = Union[PagedKV, RequestState, JointNeed, None]


def simple_needs(needs):
    """The needs of a model with every :class:`JointNeed` replaced by its parts."""
    for need in needs:
        if isinstance(need, JointNeed):
            yield from simple_needs(need.parts)
        else:
            yield need


class Part:
    #: True if ``forward`` only launches kernels that read the step's device arrays: nothing is
    #: decided on the host from the step's values, so the call may be captured in a CUDA graph
    graph_safe = False

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {}

    def load(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype) -> None:
        pass


@dataclass
class NormedDelta:
    """A pending term of the residual sum that is normalised before it is added: the hidden state is
    ``residual + norm(values)``.  Blocks whose sublayers end in a norm hand it on like this, so that the
    norm, the sum and the next norm run in one kernel."""
    values: torch.Tensor
    norm: "Norm"


@dataclass
class PendingSum:
    """A pending term of the residual sum and one row that is added to every row beside it: the hidden state is
    ``residual + values + row`` (``values``: a tensor, a :class:`NormedDelta` or None; ``row``: float32 [width]).  The norms that
    take a :class:`NormedDelta` take this too, in the same kernel."""
    values: Union[torch.Tensor, NormedDelta, None]
    row: torch.Tensor


class Norm(Part):
    #: the kernels' name of the norm ("rms", "layer")
    kind = "rms"

    def spec(self):
        """(kind, weight, bias, eps) as :func:`ops.norm_add_norm` takes it."""
        raise NotImplementedError

    def add_norm(self, residual: torch.Tensor, delta: Optional[torch.Tensor], out_dtype: torch.dtype,
                 row_index: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError


class PositionEncoding(Part):
    #: True if the fused q/k kernel can apply it from ``fused_rotary()``
    fused = False

    def fused_rotary(self):
        raise NotImplementedError

    def apply(self, q: torch.Tensor, k: Optional[torch.Tensor], positions: torch.Tensor) -> None:
        raise NotImplementedError


class Mixer(Part):
    def cache_need(self) -> CacheNeed:
        return None

    def split_scratch(self) -> Tuple[int, int]:
        """Floats of scratch per (row, key split) that a split attention run needs:
        (partial accumulators, partial maxima and sums); (0, 0) for mixers without."""
        return (0, 0)

    def forward(self, ctx, cache, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, ctx, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


def matrix_to(tensor: torch.Tensor, device, dtype: torch.dtype) -> torch.Tensor:
    """A projection matrix in the compute dtype on the device (round to nearest even)."""
    return tensor.to(device=device, dtype=dtype).contiguous()


def scale_to(tensor: torch.Tensor, device) -> torch.Tensor:
    """A norm's scale or a bias: always used in 32-bit."""
    return tensor.to(device=device, dtype=torch.float32).contiguous()
