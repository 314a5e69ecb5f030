"""Matrices that read the same input, stacked into one product.

A mixer that can stand beside another one (:class:`Stackable`) says how wide its columns of the joint projection and of
the joint result are, gives its matrices, and computes its result from a view of the one into a view of the other.  Alone
it makes both products itself; beside another mixer (``parts/parallel.py``) one product serves both at each end.
"""
from __future__ import annotations

from typing import List, Mapping, Sequence, Tuple

import torch

from .base import Mixer

#: columns that kernels read with 16-byte loads start on multiples of this many entries
ALIGN = 8


def aligned(width: int) -> int:
    return -(-width // ALIGN) * ALIGN


def stack_rows(matrices: Sequence[torch.Tensor]) -> torch.Tensor:
    """The matrices above each other, each padded with rows of zeros to a multiple of ``ALIGN`` rows."""
    padded: List[torch.Tensor] = []
    for matrix in matrices:
        missing = aligned(matrix.shape[0]) - matrix.shape[0]
        padded.append(matrix)
        if missing:
            padded.append(torch.zeros((missing, *matrix.shape[1:]), dtype=matrix.dtype, device=matrix.device))
    return torch.cat(padded, dim=0).contiguous()


def result_columns(rows: int, width: int, dtype: torch.dtype, device) -> torch.Tensor:
    """An unwritten [rows, width] whose rows start on 16-byte borders."""
    return torch.empty((rows, aligned(width)), dtype=dtype, device=device)[:, :width]


class Stackable(Mixer):
    """A mixer whose first product is a stack of matrices over its input and whose last product is one matrix."""

    @property
    def in_width(self) -> int:
        """Columns of the joint projection that are this mixer's (a multiple of ``ALIGN``); known from :meth:`load_inner` on."""
        raise NotImplementedError

    @property
    def out_width(self) -> int:
        """Columns of the result that the last product reads."""
        raise NotImplementedError

    def load_inner(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype) -> Tuple[torch.Tensor, torch.Tensor]:
        """Loads everything but the first and the last matrix; returns those two, the first with ``in_width`` rows."""
        raise NotImplementedError

    def mix(self, ctx, cache, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        """``out`` [rows, out_width] = ``scale`` times the mixer's result from ``proj`` [rows, in_width]; both may be
        columns of wider matrices."""
        raise NotImplementedError
