"""Two mixers side by side: left_scale * left(h) + right_scale * right(h), both reading the same h.

Each keeps what it keeps (:class:`JointNeed`).  Both are :class:`Stackable`, so there is one product over h for the two
together and one output product whose inner side is the two results beside each other, [W_left | W_right]; each mixer writes
its columns, multiplied in 32-bit by its scale before they are rounded.
"""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from .. import ops
from .base import JointNeed, Mixer, TensorSpec, matrix_to
from .stacking import Stackable, result_columns


class ParallelMixer(Mixer):
    def __init__(self, left: Stackable, right: Stackable, left_scale: float = 1.0, right_scale: float = 1.0):
        self.left, self.right = left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        self.w_in = self.w_o = None

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def cache_need(self) -> JointNeed:
        return JointNeed((self.left.cache_need(), self.right.cache_need()))

    def split_scratch(self):
        pairs = (self.left.split_scratch(), self.right.split_scratch())
        return (max(p[0] for p in pairs), max(p[1] for p in pairs))

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {**self.left.tensor_specs(), **self.right.tensor_specs()}

    def load(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype) -> None:
        left_in, left_out = self.left.load_inner(tensors, device, dtype)
        right_in, right_out = self.right.load_inner(tensors, device, dtype)
        self.w_in = matrix_to(torch.cat([left_in, right_in], dim=0), device, dtype)
        self.w_o = matrix_to(torch.cat([left_out, right_out], dim=1), device, dtype)

    def forward(self, ctx, cache, x: torch.Tensor) -> torch.Tensor:
        left_cache, right_cache = cache.parts
        proj = ops.linear(x, self.w_in, error_word=ctx.error_word)
        split, at = self.left.out_width, self.left.in_width
        out = result_columns(x.shape[0], split + self.right.out_width, x.dtype, x.device)
        self.left.mix(ctx, left_cache, proj[:, :at], out[:, :split], self.left_scale)
        self.right.mix(ctx, right_cache, proj[:, at:], out[:, split:], self.right_scale)
        return ops.linear(out, self.w_o, error_word=ctx.error_word, partial_ok=True)
