"""The gated delta rule: linear attention whose state decays and corrects itself, over a state of fixed size per request.

q = W_q h and k = W_k h (kv_heads x dim), v = W_v h (heads x vdim) pass a short causal convolution per channel over the last
``taps`` tokens (no bias, zeros before the sequence starts) and SiLU; value head h uses q/k head h // (heads / kv_heads).
q and k are made unit vectors per head (x / sqrt(sum x^2 + 1e-6)), q is multiplied by dim^-1/2, beta = sigmoid(W_b h), and per
head, S being [dim, vdim]:

    S <- g S        u = beta (v - S^T k)        S <- S + k u^T        o = S^T q

``channel_decay`` False: one decay per head and token, g = exp(-exp(A_log) softplus(W_a h + dt_bias)).  True: one per head,
token and row of S, from W_a2 (W_a1 h) in place of W_a h.  Each head's o is RMS-normed over vdim with a weight that the heads
share, multiplied by a gate (``gate`` ``silu``: silu(W_g h); ``sigmoid_low_rank``: sigmoid(W_g2 (W_g1 h))) and projected by
W_o.  The ranks of the thin pairs are the checkpoint's (no configuration names them).

Per request the part keeps, in 32-bit floats whatever the compute dtype, the convolution's last ``taps`` - 1 inputs and S
(``RequestState``; a request that starts at position 0 starts from zeros).  Unit vectors, step sizes, decays, the state, its
sums, the norm and the gate are 32-bit; the products run in the compute dtype.  All matrices over h are one product, the second
halves of the two thin pairs another (block by block over the columns of the first halves).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Mapping, Optional

import torch

from .. import ops
from .base import FREE, RequestState, TensorSpec, matrix_to, scale_to
from .stacking import Stackable, aligned, result_columns, stack_rows

#: inside the root of the unit vectors' length
UNIT_EPS = 1e-6


@dataclass(frozen=True)
class DeltaNames:
    q: str
    k: str
    v: str
    q_conv: str
    k_conv: str
    v_conv: str
    beta: str
    a_log: str
    dt_bias: str
    norm: str
    o: str
    decay: Optional[str] = None              # one decay per head
    decay_down: Optional[str] = None         # one per row of the state, through a thin pair
    decay_up: Optional[str] = None
    gate: Optional[str] = None
    gate_down: Optional[str] = None
    gate_up: Optional[str] = None


class GatedDeltaRule(Stackable):
    graph_safe = True
    GATES = ("silu", "sigmoid_low_rank")
    #: a step in which some request brings more rows than this runs the chunk kernels (bfloat16, sizes they take); other
    #: steps walk each request's rows token by token from its state
    CHUNKED_FROM = 8

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, eps: float, names: DeltaNames, *,
                 channel_decay: bool = False, gate: str = "silu"):
        for name, value in (("heads", heads), ("kv_heads", kv_heads), ("dim", dim), ("vdim", vdim), ("conv", taps)):
            if value <= 0:
                raise ValueError(f"gated delta rule: {name} must be positive, found {value}")
        if heads % kv_heads:
            raise ValueError(f"gated delta rule: {heads} heads are not a multiple of {kv_heads} q/k heads")
        if taps > 16 or dim > 512:
            raise ValueError(f"gated delta rule: the kernels take at most 16 taps and q/k heads of 512 entries, not {taps} and {dim}")
        if gate not in self.GATES:
            raise ValueError(f"gated delta rule: unknown gate {gate!r}; available: {self.GATES}")
        thin_gate = gate == "sigmoid_low_rank"
        if channel_decay != thin_gate:
            raise ValueError("gated delta rule: a decay per row of the state comes with a low-rank gate (their thin pairs share a product)")
        wanted = (("decay_down", "decay_up", "gate_down", "gate_up") if thin_gate else ("decay", "gate"))
        for name in wanted:
            if getattr(names, name) is None:
                raise ValueError(f"gated delta rule: the name of {name} is missing")
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = int(hidden), int(heads), int(kv_heads), int(dim), int(vdim)
        self.taps, self.eps, self.names, self.channel_decay, self.gate = int(taps), float(eps), names, bool(channel_decay), gate
        self.w_in = self.w_o = self.w_thin = self.conv = self.a_log = self.dt_bias = self.norm = None
        self._ranks = (0, 0)

    # ------------------------------------------------------------------ sizes
    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def sizes(self) -> Dict[str, int]:
        return dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, taps=self.taps)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def _tail_width(self) -> int:
        """Columns behind the convolution's channels: the gate's logits, or the thin pairs' first halves."""
        if self.channel_decay:
            return aligned(self._ranks[0]) + aligned(self._ranks[1])
        return aligned(self.heads * self.vdim)

    @property
    def in_width(self) -> int:
        return aligned(self.channels) + self._tail_width + aligned(self.heads if self.channel_decay else 2 * self.heads)

    def cache_need(self) -> RequestState:
        return RequestState((ops.delta_slot_floats(**self.sizes),), torch.float32)

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        n, qk, vv = self.names, self.kv_heads * self.dim, self.heads * self.vdim
        specs = {n.q: TensorSpec((qk, self.hidden)), n.k: TensorSpec((qk, self.hidden)), n.v: TensorSpec((vv, self.hidden)),
                 n.q_conv: TensorSpec((qk, self.taps)), n.k_conv: TensorSpec((qk, self.taps)), n.v_conv: TensorSpec((vv, self.taps)),
                 n.beta: TensorSpec((self.heads, self.hidden)), n.a_log: TensorSpec((self.heads,)),
                 n.norm: TensorSpec((self.vdim,), "scale"), n.o: TensorSpec((self.hidden, vv))}
        if self.channel_decay:
            rows = self.heads * self.dim
            specs.update({n.decay_down: TensorSpec((FREE, self.hidden), free_size=self.dim),
                          n.decay_up: TensorSpec((rows, FREE), free_size=self.dim), n.dt_bias: TensorSpec((rows,)),
                          n.gate_down: TensorSpec((FREE, self.hidden), free_size=self.dim),
                          n.gate_up: TensorSpec((vv, FREE), free_size=self.dim)})
        else:
            specs.update({n.decay: TensorSpec((self.heads, self.hidden)), n.dt_bias: TensorSpec((self.heads,)),
                          n.gate: TensorSpec((vv, self.hidden))})
        return specs

    # ------------------------------------------------------------------ weights
    def load_inner(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype):
        n = self.names
        first = [torch.cat([tensors[n.q], tensors[n.k], tensors[n.v]], dim=0)]
        if self.channel_decay:
            for down, up in ((n.decay_down, n.decay_up), (n.gate_down, n.gate_up)):
                if tensors[down].shape[0] != tensors[up].shape[1]:
                    raise ValueError(f"{down} has {tensors[down].shape[0]} rows, {up} {tensors[up].shape[1]} columns")
            self._ranks = (tensors[n.decay_down].shape[0], tensors[n.gate_down].shape[0])
            first += [tensors[n.decay_down], tensors[n.gate_down], tensors[n.beta]]
            # the second halves side by side: rows of the decay read the first block of columns, rows of the gate the second
            rows, ra, rg = self.heads * self.dim, aligned(self._ranks[0]), aligned(self._ranks[1])
            up, gate_up = tensors[n.decay_up], tensors[n.gate_up]
            thin = torch.zeros((aligned(rows) + gate_up.shape[0], ra + rg), dtype=up.dtype, device=up.device)
            thin[:rows, :self._ranks[0]] = up
            thin[aligned(rows):, ra:ra + self._ranks[1]] = gate_up
            self.w_thin = matrix_to(thin, device, dtype)
        else:
            first += [tensors[n.gate], torch.cat([tensors[n.decay], tensors[n.beta]], dim=0)]
        self.conv = scale_to(torch.cat([tensors[n.q_conv], tensors[n.k_conv], tensors[n.v_conv]], dim=0), device)
        self.a_log, self.dt_bias, self.norm = (scale_to(tensors[name], device) for name in (n.a_log, n.dt_bias, n.norm))
        return stack_rows(first), tensors[n.o]

    def load(self, tensors: Mapping[str, torch.Tensor], device, dtype: torch.dtype) -> None:
        first, last = self.load_inner(tensors, device, dtype)
        self.w_in, self.w_o = matrix_to(first, device, dtype), matrix_to(last, device, dtype)

    # ------------------------------------------------------------------ the step
    def forward(self, ctx, cache, x: torch.Tensor) -> torch.Tensor:
        proj = ops.linear(x, self.w_in, error_word=ctx.error_word)
        out = result_columns(x.shape[0], self.out_width, x.dtype, x.device)
        self.mix(ctx, cache, proj, out)
        return ops.linear(out, self.w_o, error_word=ctx.error_word, partial_ok=True)

    def mix(self, ctx, cache, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        rows, vv = proj.shape[0], self.heads * self.vdim
        tail = aligned(self.channels)
        behind = tail + self._tail_width
        if self.channel_decay:
            thin = ops.linear(proj[:, tail:behind], self.w_thin, error_word=ctx.error_word)
            at = aligned(self.heads * self.dim)
            decay, gate = thin[:, :self.heads * self.dim], thin[:, at:at + vv]
            beta = proj[:, behind:behind + self.heads]
        else:
            gate = proj[:, tail:tail + vv]
            decay, beta = proj[:, behind:behind + self.heads], proj[:, behind + self.heads:behind + 2 * self.heads]
        counts = [b - a for a, b in zip(ctx.host_cu_rows, ctx.host_cu_rows[1:])]
        known = len(counts) == ctx.num_requests
        chunked = known and max(counts, default=0) > self.CHUNKED_FROM and ops.delta_chunks_takes(proj.dtype, self.dim, self.vdim)
        qkv = torch.empty((rows, self.channels), dtype=proj.dtype if chunked else torch.float32, device=proj.device)
        single = known and all(count == 1 for count in counts)
        ops.short_conv(proj[:, :self.channels], self.conv, None, ctx.positions, ctx.row_request, ctx.cu_rows, ctx.state_slots,
                       cache.state, qkv, ctx.num_requests, read_only=not cache.writable,
                       single_rows=single)
        o = torch.empty((rows, vv), dtype=torch.float32, device=proj.device)
        args = (qkv, beta, decay, self.a_log, self.dt_bias, ctx.positions, ctx.cu_rows, ctx.state_slots, cache.state, o,
                ctx.num_requests)
        options = dict(channel_decay=self.channel_decay, unit_eps=UNIT_EPS, read_only=not cache.writable, **self.sizes)
        if chunked:
            ops.delta_chunks(*args, sum(-(-count // ops.DELTA_CHUNK_TOKENS) for count in counts), **options)
        else:
            ops.delta_scan(*args, single_rows=single, **options)
        ops.delta_gate_norm(o, gate, self.norm, self.eps, out, silu=self.gate == "silu", scale=scale, heads=self.heads)
