"""minGRU: a recurrence per channel whose gate and candidate read the current token only.

z = sigmoid(W_z h + b_z), u = W_x h + b_x, the candidate is u + 1/2 where u >= 0 and sigmoid(u) where u < 0; channel by channel
S_t = (1 - z) S_(t-1) + z * candidate, and the result is W_o (S_t * silu(W_g h)).  The state starts at zero and is kept in
32-bit floats per request (``RequestState``); gates, candidates and the state are 32-bit in both dtypes.  W_z, W_x and W_g read
the same input and are one product.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Mapping

import torch

from .. import ops
from .base import RequestState, TensorSpec, matrix_to, scale_to
from .stacking import Stackable, aligned, result_columns, stack_rows


@dataclass(frozen=True)
class MinGruNames:
    z: str
    z_bias: str
    x: str
    x_bias: str
    gate: str
    o: str


class MinGru(Stackable):
    graph_safe = True

    def __init__(self, hidden: int, width: int, names: MinGruNames):
        if width <= 0:
            raise ValueError(f"minGRU: the width must be positive, found {width}")
        self.hidden, self.width, self.names = int(hidden), int(width), names
        self.w_in = self.w_o = self.z_bias = self.x_bias = None

    @property
    def in_width(self) -> int:
        return 3 * aligned(self.width)

    @property
    def out_width(self) -> int:
        return self.width

    def cache_need(self) -> RequestState:
        return RequestState((self.width,), torch.float32)

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        n, shape = self.names, (self.width, self.hidden)
        return {n.z: TensorSpec(shape), n.z_bias: TensorSpec((self.width,)), n.x: TensorSpec(shape),
                n.x_bias: TensorSpec((self.width,)), n.gate: TensorSpec(shape), n.o: TensorSpec((self.hidden, self.width))}

    def load_inner(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype):
        n = self.names
        self.z_bias, self.x_bias = scale_to(tensors[n.z_bias], device), scale_to(tensors[n.x_bias], device)
        return stack_rows([tensors[n.z], tensors[n.x], tensors[n.gate]]), tensors[n.o]

    def load(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype) -> None:
        first, last = self.load_inner(tensors, device, dtype)
        self.w_in, self.w_o = matrix_to(first, device, dtype), matrix_to(last, device, dtype)

    def forward(self, ctx, cache, x: torch.Tensor) -> torch.Tensor:
        proj = ops.linear(x, self.w_in, error_word=ctx.error_word)
        out = result_columns(x.shape[0], self.width, x.dtype, x.device)
        self.mix(ctx, cache, proj, out)
        return ops.linear(out, self.w_o, error_word=ctx.error_word, partial_ok=True)

    def mix(self, ctx, cache, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        counts = [b - a for a, b in zip(ctx.host_cu_rows, ctx.host_cu_rows[1:])]
        single = len(counts) == ctx.num_requests and all(count == 1 for count in counts)
        # (without the step's shape on the host: as many chunks as there can be)
        chunks = sum(-(-count // ops.MINGRU_CHUNK_TOKENS) for count in counts) if len(counts) == ctx.num_requests else proj.shape[0]
        step = aligned(self.width)
        ops.mingru(proj, 0, step, 2 * step, self.z_bias, self.x_bias, ctx.positions, ctx.cu_rows, ctx.state_slots, cache.state, out,
                   ctx.num_requests, chunks, scale=scale, single_rows=single, read_only=not cache.writable)
