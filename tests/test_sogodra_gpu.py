"""Sogodra on the GPU against the plain implementation: each mechanism alone (the short convolution, the gated delta rule token by
token and in chunks, minGRU, attention with norms per head and a learned sink written into columns of a wider result, the
clamped feed-forward, norms on outputs only), whole prompts, prompts with a tail decoded token by token, portions down to two
tokens, mixed batches over a small pool (pages and state slots are used again), keys just inside and just outside a window,
states that must survive hundreds of tokens, long decoding from captured graphs, and greedy generation through the entry point,
the command line and the trace program."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_sogodra as ps
import replay_helpers as rh
import sogodra_helpers as sh

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [("float32", torch.float32, 1e-4), ("bfloat16", torch.bfloat16, 4e-2)]
BOTH = [torch.float32, torch.bfloat16]


def seen(tensor, dtype):
    """What the kernel sees of a tensor: rounded to the storage type, as float64."""
    return tensor.to(dtype).to(torch.float64)


def close(got, want, dtype, what, fraction=None):
    tolerance = fraction if fraction is not None else (2e-5 if dtype == torch.float32 else 2e-2)
    scale = float(want.abs().max()) or 1.0
    error = float((got.detach().cpu().to(torch.float64) - want).abs().max()) / scale
    assert error <= tolerance, (what, error)


def dev(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def whole_model_close(rows, expected, dtype_name, what=""):
    if dtype_name == "float32":
        sh.assert_rows_close(rows, expected, 1e-4, what)
    else:
        sh.assert_rows_close(rows, expected, 0.1, what, median=0.025)


def step_arrays(counts, starts):
    cu = np.cumsum([0] + counts).tolist()
    positions = [s + i for s, c in zip(starts, counts) for i in range(c)]
    row_request = [r for r, c in enumerate(counts) for _ in range(c)]
    return cu, dev(positions), dev(row_request), dev(cu)


# ------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_short_convolution_over_inputs_in_slots(dtype, taps):
    """Columns of a wider projection, no bias: a prompt in a slot that holds rubbish, a later portion shorter than the filter, one
    decoded token at position 1; then a step of single rows (one launch); the slots keep the last inputs."""
    from sglang_rs_b200 import ops
    g = torch.Generator().manual_seed(taps)
    channels, pitch, at = 70, 90, 11
    w = torch.randn(channels, taps, generator=g)
    state = torch.randn(5, (taps - 1) * channels + 6, generator=g).to(DEV)
    sequences = {2: torch.randn(600, channels, generator=g), 0: torch.randn(9, channels, generator=g), 3: torch.randn(3, channels, generator=g)}
    slots = [2, 0, 3]
    want = {s: ps.silu(ps.causal_conv(seen(x, dtype), w.double())) for s, x in sequences.items()}
    keep = taps - 1
    for s, start in ((0, 6), (3, 1)):
        for k in range(keep):
            place = start - keep + k
            state[s, k * channels:(k + 1) * channels] = (seen(sequences[s][place], dtype).float() if place >= 0 else torch.full((channels,), 9.0)).to(DEV)
    before = state.clone()
    for starts, counts, single in (([0, 6, 1], [598, 2, 1], False), ([598, 8, 2], [1, 1, 1], True)):
        cu, positions, row_request, cu_d = step_arrays(counts, starts)
        proj = torch.zeros(cu[-1], pitch)
        for i, s in enumerate(slots):
            proj[cu[i]:cu[i + 1], at:at + channels] = sequences[s][starts[i]:starts[i] + counts[i]]
        on = proj.to(DEV, dtype)
        for out_dtype in [torch.float32] + [dtype] * (dtype != torch.float32):      # (the one that keeps the inputs last)
            for read_only in (True, False):
                if not read_only and out_dtype != dtype:
                    continue
                now = state.clone()
                out = torch.full((cu[-1], channels), float("nan"), dtype=out_dtype, device=DEV)
                ops.short_conv(on[:, at:at + channels], w.to(DEV), None, positions, row_request, cu_d, dev(slots), state, out, 3,
                               read_only=read_only, single_rows=single)
                if read_only:
                    assert torch.equal(now, state)
                for i, s in enumerate(slots):
                    close(out[cu[i]:cu[i + 1]], want[s][starts[i]:starts[i] + counts[i]], out_dtype, f"slot {s}", 2e-6 if out_dtype == torch.float32 else None)
        for i, s in enumerate(slots):
            for k in range(keep):
                place = starts[i] + counts[i] - keep + k
                kept = state[s, k * channels:(k + 1) * channels].cpu().double()
                close(kept, seen(sequences[s][place], dtype) if place >= 0 else torch.zeros(channels).double(), torch.float32, "kept", 0.0 if place >= 0 else 1e-9)
    assert torch.equal(state[1], before[1]) and torch.equal(state[:, keep * channels:], before[:, keep * channels:])


DELTA_CASES = [(4, 2, 12, 20, 3), (2, 2, 64, 48, 4), (3, 1, 7, 11, 2), (1, 1, 200, 9, 1), (2, 1, 260, 8, 4), (2, 1, 100, 40, 2)]
CHUNK_CASES = [(2, 1, 64, 64, 4), (2, 2, 128, 128, 2), (3, 1, 64, 32, 3), (2, 1, 72, 24, 2), (1, 1, 8, 8, 4), (2, 2, 128, 48, 3), (1, 1, 40, 200, 2)]


def delta_inputs(heads, kv_heads, dim, vdim, rows, channels, seed, rate):
    g = torch.Generator().manual_seed(seed)
    columns = heads * dim if channels else heads
    return {"x": torch.randn(rows, 2 * kv_heads * dim + heads * vdim, generator=g), "beta": torch.randn(rows, heads + 3, generator=g) * 2,
            "decay": torch.randn(rows, columns + 5, generator=g), "a_log": torch.rand(heads, generator=g) * 6 - 5 + rate,
            "dt_bias": torch.rand(columns, generator=g) * 4 - 3}


def plain_delta(w, rows, heads, kv_heads, dim, vdim, channels, dtype, x_dtype, begin):
    T = rows.stop - rows.start
    x = seen(w["x"][rows], x_dtype)
    per = heads // kv_heads
    q = ps.unit(x[:, :kv_heads * dim].reshape(T, kv_heads, dim)).repeat_interleave(per, 1) * dim ** -0.5
    k = ps.unit(x[:, kv_heads * dim:2 * kv_heads * dim].reshape(T, kv_heads, dim)).repeat_interleave(per, 1)
    v = x[:, 2 * kv_heads * dim:].reshape(T, heads, vdim)
    beta = torch.sigmoid(seen(w["beta"][rows, :heads], dtype))
    columns = heads * dim if channels else heads
    z = ps.softplus(seen(w["decay"][rows, :columns], dtype) + w["dt_bias"].double())
    rates = torch.exp(w["a_log"].double())
    if channels:
        decay = torch.exp(-rates[None, :, None] * z.reshape(T, heads, dim))
    else:
        decay = torch.exp(-rates[None, :] * z)[:, :, None].expand(T, heads, dim)
    o, last = ps.delta_recurrence(q, k, v, beta, decay, begin)
    return o.reshape(T, heads * vdim), last


def run_delta(kernel, w, rows, counts, starts, slots, state, sizes, channels, dtype, x_dtype, read_only=False):
    from sglang_rs_b200 import ops
    heads, dim, vdim = sizes["heads"], sizes["dim"], sizes["vdim"]
    cu, positions, _, cu_d = step_arrays(counts, starts)
    columns = heads * dim if channels else heads
    out = torch.full((cu[-1], heads * vdim), float("nan"), device=DEV)
    beta, decay = w["beta"][rows].to(DEV, dtype), w["decay"][rows].to(DEV, dtype)      # columns of wider matrices
    args = [w["x"][rows].to(DEV, x_dtype), beta[:, :heads], decay[:, :columns], w["a_log"].to(DEV), w["dt_bias"].to(DEV), positions, cu_d,
            dev(slots), state, out, len(counts)]
    if kernel is ops.delta_chunks:
        args.append(sum(-(-c // ops.DELTA_CHUNK_TOKENS) for c in counts))
    options = dict(channel_decay=channels, unit_eps=1e-6, **sizes)
    if kernel is ops.delta_scan and max(counts) == 1:
        options["single_rows"] = True
    kernel(*args, read_only=read_only, **options)
    return cu, out


def delta_over_two_steps(kernel, heads, kv_heads, dim, vdim, taps, channels, dtype, x_dtype, counts, counts2, tolerance, rate=0.0):
    """Four requests in one step (a prompt from position 0 in a slot that holds rubbish, a one-token prompt, a later portion from a
    given state, another), then a second step that continues them from what the first left; a read-only run changes nothing."""
    from sglang_rs_b200 import ops
    sizes = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, taps=taps)
    starts, slots = [0, 0, 70, 9], [2, 5, 0, 3]
    order2, slots2 = [0, 2, 3, 1], [2, 0, 3, 5]
    total, total2 = sum(counts), sum(counts2)
    w = delta_inputs(heads, kv_heads, dim, vdim, total + total2, channels, dim + vdim, rate)
    state = torch.randn(6, ops.delta_slot_floats(**sizes), device=DEV)
    given = state.cpu().double()
    conv = -(-(taps - 1) * (2 * kv_heads * dim + heads * vdim) // 4) * 4

    def unpack(slot_row):
        return slot_row[conv:conv + heads * dim * vdim].reshape(heads, vdim, dim).transpose(1, 2)
    plain = lambda rows, begin: plain_delta(w, rows, heads, kv_heads, dim, vdim, channels, dtype, x_dtype, begin)
    cu, out = run_delta(kernel, w, slice(0, total), counts, starts, slots, state, sizes, channels, dtype, x_dtype)
    after = {}
    for r in range(4):
        begin = unpack(given[slots[r]])
        want, after[r] = plain(slice(cu[r], cu[r + 1]), torch.zeros_like(begin) if starts[r] == 0 else begin)
        close(out[cu[r]:cu[r + 1]], want, torch.float32, f"request {r}", tolerance)
        close(unpack(state[slots[r]].cpu().double()), after[r], torch.float32, f"state of request {r}", tolerance)
    assert torch.equal(state[1].cpu().double(), given[1]) and torch.equal(state[:, :conv].cpu().double(), given[:, :conv])
    starts2 = [starts[r] + counts[r] for r in order2]
    before = state.clone()
    for read_only in (True, False):
        cu2, out2 = run_delta(kernel, w, slice(total, total + total2), counts2, starts2, slots2, state, sizes, channels, dtype, x_dtype, read_only)
        if read_only:
            assert torch.equal(state, before)
        for i, r in enumerate(order2):
            want, last = plain(slice(total + cu2[i], total + cu2[i + 1]), after[r])
            close(out2[cu2[i]:cu2[i + 1]], want, torch.float32, f"second step, request {r}", tolerance)
            if not read_only:
                close(unpack(state[slots2[i]].cpu().double()), last, torch.float32, f"second step, state of request {r}", tolerance)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("channels", [False, True])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", DELTA_CASES)
def test_gated_delta_rule_token_by_token(heads, kv_heads, dim, vdim, taps, channels, dtype):
    from sglang_rs_b200 import ops
    delta_over_two_steps(ops.delta_scan, heads, kv_heads, dim, vdim, taps, channels, dtype, torch.float32, [45, 1, 33, 1], [2, 38, 1, 50], 3e-5)
    delta_over_two_steps(ops.delta_scan, heads, kv_heads, dim, vdim, taps, channels, dtype, torch.float32, [1, 1, 33, 2], [1, 1, 1, 1], 3e-5)


@pytest.mark.parametrize("channels", [False, True])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", CHUNK_CASES)
def test_gated_delta_rule_in_chunks_on_the_tensor_cores(heads, kv_heads, dim, vdim, taps, channels):
    """Portions of exactly one chunk of 64 tokens, of one chunk and one token, of more than two chunks, of two tokens and of one;
    what is left against the plain recurrence over the same rounded inputs is the error of operands in two roundings."""
    from sglang_rs_b200 import ops
    assert ops.DELTA_CHUNK_TOKENS == 64 and ops.delta_chunks_takes(torch.bfloat16, dim, vdim)
    delta_over_two_steps(ops.delta_chunks, heads, kv_heads, dim, vdim, taps, channels, torch.bfloat16, torch.bfloat16, [150, 1, 65, 64],
                         [2, 67, 1, 128], 2e-4)


@pytest.mark.parametrize("channels", [False, True])
@pytest.mark.parametrize("rate", [-6.0, 6.0])
def test_chunks_with_decays_near_one_and_near_zero(channels, rate):
    """Rates from 2e-5 to 0.007 (a state that keeps everything for thousands of tokens) and from 2.7 to 1,100 (exponents far
    below what a 32-bit number holds: quotients of such decays would be infinite)."""
    from sglang_rs_b200 import ops
    delta_over_two_steps(ops.delta_chunks, 3, 1, 64, 32, 2, channels, torch.bfloat16, torch.bfloat16, [200, 1, 65, 30], [2, 67, 1, 128], 3e-4, rate)


def test_chunks_and_single_tokens_continue_each_other():
    """A prompt in chunks, then tokens one by one, then a portion in chunks: the state goes through both kernels."""
    from sglang_rs_b200 import ops
    sizes = dict(heads=2, kv_heads=1, dim=64, vdim=32, taps=2)
    dtype = torch.bfloat16
    w = delta_inputs(2, 1, 64, 32, 160, True, 5, 0.0)
    state = torch.randn(2, ops.delta_slot_floats(**sizes), device=DEV)
    want, _ = plain_delta(w, slice(0, 160), 2, 1, 64, 32, True, dtype, dtype, None)
    w = dict(w, x=w["x"].to(dtype).float())                       # the token-by-token kernel reads 32-bit inputs
    at = 0
    for count in (70, 1, 1, 1, 66, 2, 19):
        kernel, kind = (ops.delta_chunks, dtype) if count > 8 else (ops.delta_scan, torch.float32)
        _, out = run_delta(kernel, w, slice(at, at + count), [count], [at], [1], state, sizes, True, dtype, kind)
        close(out, want[at:at + count], torch.float32, f"tokens from {at}", 3e-4 * float(want.abs().max()) / float(want[at:at + count].abs().max()))
        at += count
    assert at == 160


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("silu", [False, True])
@pytest.mark.parametrize("heads,vdim", [(3, 11), (2, 64), (4, 130), (1, 300)])
def test_norm_and_gate_per_head_into_columns_of_a_wider_matrix(heads, vdim, silu, dtype):
    from sglang_rs_b200 import ops
    g = torch.Generator().manual_seed(vdim)
    rows, width, eps = 9, heads * vdim, 1e-3
    o, gate, weight = torch.randn(rows, width, generator=g) * 0.1, torch.randn(rows, width + 7, generator=g) * 2, torch.rand(vdim, generator=g) + 0.5
    wide = torch.full((rows, width + 13), 7.0, dtype=dtype, device=DEV)
    ops.delta_gate_norm(o.to(DEV), gate.to(DEV, dtype)[:, 2:2 + width], weight.to(DEV), eps, wide[:, 5:5 + width], heads=heads, silu=silu, scale=0.6)
    z = seen(gate, dtype)[:, 2:2 + width]
    want = 0.6 * (ps.rms(o.double().reshape(rows, heads, vdim), eps) * weight.double()).reshape(rows, width) * (ps.silu(z) if silu else torch.sigmoid(z))
    close(wide[:, 5:5 + width], want, dtype, "norm and gate")
    assert float(wide[:, :5].min()) == 7.0 and float(wide[:, 5 + width:].max()) == 7.0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("width", [21, 128, 300])
def test_mingru_over_states_in_slots(width, dtype):
    """A prompt of several chunks in a slot that holds rubbish, one token, a later portion of one chunk and one token; then a step of
    single rows; gates near zero (a state that lasts) and near one beside each other, candidates on both branches."""
    from sglang_rs_b200 import ops
    g = torch.Generator().manual_seed(width)
    step = -(-width // 8) * 8
    zb, xb = torch.randn(width, generator=g) * 3 - 1, torch.randn(width, generator=g)
    state = torch.randn(5, width, generator=g).to(DEV)
    slots, memory = [2, 0, 3], {}
    start_state = state.cpu().double()
    for starts, counts, single in (([0, 4, 30], [140, 1, 65], False), ([140, 5, 95], [1, 1, 1], True), ([141, 6, 96], [2, 66, 1], False)):
        cu, positions, _, cu_d = step_arrays(counts, starts)
        proj = torch.randn(cu[-1], 3 * step + 5, generator=g) * 1.5
        for read_only in (True, False):
            before = state.clone()
            wide = torch.full((cu[-1], width + 9), 7.0, dtype=dtype, device=DEV)
            chunks = sum(-(-c // ops.MINGRU_CHUNK_TOKENS) for c in counts)
            ops.mingru(proj.to(DEV, dtype), 0, step, 2 * step, zb.to(DEV), xb.to(DEV), positions, cu_d, dev(slots), state, wide[:, 4:4 + width], 3,
                       chunks, scale=0.9, single_rows=single, read_only=read_only)
            assert not read_only or torch.equal(before, state)
        p = seen(proj, dtype)
        for i, s in enumerate(slots):
            S = memory.get(s, torch.zeros(width).double() if starts[i] == 0 else start_state[s])
            z, u, gate = (p[cu[i]:cu[i + 1], k * step:k * step + width] for k in range(3))
            z, u = torch.sigmoid(z + zb.double()), u + xb.double()
            candidate = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
            assert (u >= 0).any() and (u < 0).any()
            rows = []
            for t in range(counts[i]):
                S = (1 - z[t]) * S + z[t] * candidate[t]
                rows.append(0.9 * S * ps.silu(gate[t]))
            memory[s] = S
            close(wide[cu[i]:cu[i + 1], 4:4 + width], torch.stack(rows), dtype, f"slot {s} from {starts[i]}")
            close(state[s], S, torch.float32, f"state of slot {s}", 3e-6)
        assert float(wide[:, :4].min()) == 7.0 and float(wide[:, 4 + width:].max()) == 7.0
    assert torch.equal(state[1].cpu().double(), start_state[1])


ATTENTION_CASES = [(4, 2, 16, 12, 24, 12, sh.RAMP), (3, 3, 10, 6, 1, 6, None), (2, 1, 64, 64, 40, 32, sh.RAMP), (6, 2, 128, 128, 96, 128, None),
                   (2, 2, 8, 24, None, 0, None)]


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,rot_dims,scaling", ATTENTION_CASES)
def test_windowed_attention_with_norms_per_head_and_learned_sinks(heads, kv_heads, dim, vdim, window, rot_dims, scaling, dtype_name, stored, tolerance):
    """The mixer alone, its result scaled and written into columns of a wider matrix: a prompt whose last 30 tokens are decoded one
    by one and one cut into portions (the three tensor-core kernels at heads of 64 and 128, the generic one elsewhere)."""
    from sglang_rs_b200 import ops
    from sglang_rs_b200.cache import CacheManager
    from sglang_rs_b200.engine.runner import StepEntry, StepPlanner
    from sglang_rs_b200.parts import AttentionNames, GroupedQueryAttention, NoPositionEncoding, RampScaling, RotaryEncoding
    width, eps = 40, 1e-4
    m = sh.attention(heads, kv_heads, dim, vdim, window, rot_dims, base=500.0, scaling=scaling)
    names = AttentionNames(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm", sink="sink")
    rotary = RotaryEncoding(dim, 500.0, rotary_dim=rot_dims, scaling=RampScaling(**scaling) if scaling else None) if rot_dims else NoPositionEncoding()
    part = GroupedQueryAttention(width, heads, kv_heads, dim, m["scale"], rotary, names, qk_norm_eps=eps, window=window, value_dim=vdim)
    g = torch.Generator().manual_seed(dim)
    w = {n: (torch.randn(s.shape, generator=g) / (s.shape[-1] ** 0.5 if len(s.shape) > 1 else 1)).to(stored) for n, s in part.tensor_specs().items()}
    w["q.norm"], w["sink"] = (w["q.norm"].float() * 2 + 1).to(stored), (w["sink"].float() * 2).to(stored)
    first, last = part.load_inner(w, DEV, stored)
    h = torch.randn(230, width, generator=g).to(stored)
    # the projection as the mixer sees it, so that the comparison is about the mechanism alone
    proj = (h.double() @ first.double().cpu().T).to(stored)
    w64 = {k: v.double() for k, v in w.items()}
    sizes = [heads * dim, kv_heads * dim, kv_heads * vdim]
    q, k, v = proj[:, :sum(sizes)].double().split(sizes, dim=1)

    assert torch.equal(last, w["o"])

    def plain():
        T = 230
        qn = ps.rms(q.reshape(T, heads, dim), eps) * w64["q.norm"]
        kn = ps.rms(k.reshape(T, kv_heads, dim), eps) * w64["k.norm"]
        if rot_dims:
            qn = torch.stack([ps.rotate(qn[t], t, m["rot"]) for t in range(T)])
            kn = torch.stack([ps.rotate(kn[t], t, m["rot"]) for t in range(T)])
        out = torch.zeros(T, heads, vdim).double()
        for i in range(T):
            lo = 0 if window is None else max(0, i - window + 1)
            for head in range(heads):
                s = kn[lo:i + 1, head // (heads // kv_heads)] @ qn[i, head] * m["scale"]
                e = torch.exp(s)
                out[i, head] = e @ v[lo:i + 1].reshape(-1, kv_heads, vdim)[:, head // (heads // kv_heads)] / (e.sum() + torch.exp(w64["sink"][head]))
        return 0.7 * out.reshape(T, heads * vdim)
    want = plain()
    for cuts in ([200] + [1] * 30, [17, 2, 130, 1, 64, 16]):
        cache = CacheManager([part.cache_need()], page_size=16, max_tokens=256, max_requests=1, device=DEV, dtype=stored)
        planner = StepPlanner(cache, DEV, stored, [part.split_scratch()])
        handle, at = cache.open("a"), 0
        for count in cuts:
            cache.reserve(handle, count)
            ctx, _ = planner.flatten([StepEntry(handle, [0] * count)])
            wide = torch.full((count, heads * vdim + 16), 7.0, dtype=stored, device=DEV)
            part.mix(ctx, cache.layer_caches[0], proj[at:at + count].to(DEV), wide[:, 8:8 + heads * vdim], 0.7)
            cache.commit(handle, count)
            close(wide[:, 8:8 + heads * vdim], want[at:at + count], stored, f"rows from {at}")
            assert float(wide[:, :8].min()) == 7.0 and float(wide[:, 8 + heads * vdim:].max()) == 7.0
            at += count
        assert at == 230
        ops.raise_on_error_word(planner.error_word)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows", [3, 100, 1400])
def test_clamped_feed_forward_through_every_product_kernel(rows, dtype):
    from sglang_rs_b200 import ops
    from sglang_rs_b200.parts import GatedMlp, GatedMlpNames
    g = torch.Generator().manual_seed(rows)
    width, ff, limit = 64, 136, 0.8
    part = GatedMlp(width, ff, "swiglu_clamp", GatedMlpNames(gate="gate", up="up", down="down"), activation_param=limit, partial_sums=False)
    w = {n: (torch.randn(s.shape, generator=g) / s.shape[1] ** 0.5).to(dtype) for n, s in part.tensor_specs().items()}
    part.load(w, DEV, dtype)
    h = torch.randn(rows, width, generator=g)

    class Ctx:
        error_word = ops.new_error_word(DEV)
    want = ps.feed_forward(seen(h, dtype), {k: v.double() for k, v in w.items()}, {"limit": limit})
    assert float((seen(h, dtype) @ w["gate"].double().T).max()) > limit
    close(part.forward(Ctx, h.to(DEV, dtype)), want, dtype, "clamped feed-forward")
    ops.raise_on_error_word(Ctx.error_word)
    with pytest.raises(ValueError, match="parameter"):
        GatedMlp(width, ff, "swiglu_clamp", GatedMlpNames(gate="gate", up="up", down="down"))


@pytest.mark.parametrize("dtype", BOTH)
def test_the_stream_with_a_normed_term_added_is_handed_on_rounded(dtype):
    """residual += norm(delta), and the sum rounded to the compute type: what a sublayer without a norm ahead of it reads."""
    from sglang_rs_b200.parts import GroupedRmsNorm, NormedDelta
    from sglang_rs_b200.parts.norm import rounded_sum
    g = torch.Generator().manual_seed(1)
    x, delta, weight = torch.randn(7, 50, generator=g) * 3, torch.randn(7, 50, generator=g), torch.rand(50, generator=g) + 0.5
    norm = GroupedRmsNorm(50, 1e-3, "n")
    norm.load({"n": weight}, DEV, dtype)
    residual = x.to(DEV)
    out = rounded_sum(residual, NormedDelta(delta.to(DEV, dtype), norm), dtype)
    want = x.double() + ps.rms(seen(delta, dtype), 1e-3) * weight.double()
    close(residual, want, torch.float32, "the sum", 1e-6)
    assert out.dtype == dtype and torch.equal(out, residual.to(dtype))
    assert torch.equal(rounded_sum(residual, None, dtype), residual.to(dtype))


# ------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("doc", [sh.SMALL_A, sh.SMALL_B, sh.SMALL_C, sh.SMALL_D, sh.SMALL_E, sh.SMALL_F], ids="abcdef")
def test_prompts_tails_portions_and_mixed_batches(tmp_path, doc, dtype_name, stored, tolerance):
    folder = sh.make_folder(tmp_path, "m", doc, seed=5, dtype=stored)
    requests = sh.random_requests(doc, (1, 2, 23, 64, 65, 150, 131), seed=3)
    expected = sh.oracle(folder, requests)
    worst = {}
    for name, trace, page in (("whole", rh.trace_whole(requests), 16), ("tail", rh.trace_tail_by_one(requests, tail=45), 16),
                              ("portions", rh.trace_portions(requests), 8), ("mixed", rh.trace_mixed(requests, seed=9), 16)):
        # the pool holds what is live at any time and no more, so pages and state slots go from one request to the next
        rows, session = rh.run_in_process(folder, dtype_name, trace, page_size=page)
        assert all(len(rows[rid]) == len(tokens) for rid, tokens in requests.items())
        worst[name] = rh.worst_error(rows, expected)
        whole_model_close(rows, expected, dtype_name, name)
        if name == "mixed":
            paged = any(entry["type"] == "parallel" for entry in doc["layers"])
            assert any(len(owners) > 1 for owners in session.page_owners.values()) == paged, "no page was used again"
            assert len(requests) > session.cache.max_requests, "no state slot was used again"
    print(doc["width"], dtype_name, worst)


def test_layers_one_by_one_against_the_plain_stream(tmp_path):
    """The residual stream after every layer, 32-bit, for a prompt in one step."""
    from sglang_rs_b200.engine.replay import ReplaySession
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_A, seed=2, dtype=torch.float32)
    doc, tensors = sh.load_folder(folder)
    tokens = sh.random_requests(doc, (50,), seed=6)["r0"]
    logits, after = ps.forward(doc, tensors, tokens, return_layers=True)
    session = ReplaySession(folder, "float32", 64, 16, use_cuda_graphs=False)
    streams = []
    for block in session.model.layers:
        def forward(ctx, cache, residual, delta, inner=block.forward):
            residual, delta = inner(ctx, cache, residual, delta)
            _, weight, _, eps = delta.norm.spec()[:4]              # the normed term that the next kernel will add
            streams.append(residual.double().cpu() + ps.rms(delta.values.double().cpu(), eps) * weight.double().cpu())
            return residual, delta
        block.forward = forward
    out = session.run({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": list(range(len(tokens)))}], "end": ["a"]})
    assert len(streams) == len(doc["layers"])
    for index, (got, want) in enumerate(zip(streams, after)):
        close(got, want, torch.float32, f"stream after layer {index}")
    close(torch.from_numpy(out), logits, torch.float32, "logits")


def test_the_cut_and_the_batch_change_nothing_beyond_rounding(tmp_path):
    """In 32-bit the logits of a position agree to rounding whatever the portions, the pages, the slots and the requests
    beside it."""
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_A, seed=6, dtype=torch.float32)
    requests = sh.random_requests(sh.SMALL_A, (40, 97, 130, 5, 61), seed=4)
    whole, _ = rh.run_in_process(folder, "float32", rh.trace_whole(requests), page_size=16)
    for trace, page in ((rh.trace_portions(requests, sizes=(2, 2, 3, 33, 2, 15)), 4), (rh.trace_mixed(requests, seed=2, max_live=3), 32)):
        rows, _ = rh.run_in_process(folder, "float32", trace, page_size=page)
        for rid in requests:
            for pos, row in rows[rid].items():
                assert float(np.abs(row - whole[rid][pos]).max()) <= 5e-5 * float(np.abs(whole[rid][pos]).max()), (rid, pos)


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("window", [16, 33, 96])
def test_a_marked_key_just_inside_and_just_outside_the_window(tmp_path, window, dtype_name, stored, tolerance):
    """The row that is window - 1 positions behind the mark still sees it, the next one does not: in a whole prompt, decoded token by
    token (pages behind the window go back to the pool), and in portions cut at the edge."""
    folder = sh.marked_folder(tmp_path, stored, "window", window)
    doc, tensors = sh.load_folder(folder)
    for mark in (0, 7, 31):
        tokens = sh.with_mark(doc, mark + window + 12, mark, seed=mark)
        requests = {"r0": tokens}
        expected = sh.oracle(folder, requests)
        plain = ps.forward(doc, tensors, tokens[:mark] + [sh.FILL] + tokens[mark + 1:]).numpy()
        inside, outside = mark + window - 1, mark + window
        assert np.abs(plain[inside] - expected["r0"][inside]).max() > 0.2 * np.abs(expected["r0"]).max(), "the marked key decides nothing"
        assert np.abs(plain[outside] - expected["r0"][outside]).max() == 0.0
        traces = (rh.trace_whole(requests), rh.trace_tail_by_one(requests, tail=window + 11),
                  rh.trace_portions(requests, sizes=(inside, 1, 1, 2)), rh.trace_portions(requests, sizes=(mark + 1, 2, window - 4, 2, 2, 3)))
        for trace in traces:
            rows, _ = rh.run_in_process(folder, dtype_name, trace, page_size=16)
            sh.assert_rows_close(rows, expected, tolerance, (window, mark))


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("kind,wide", [("delta", False), ("delta", True), ("channel", False), ("channel", True), ("mingru", False)])
def test_a_state_keeps_a_token_from_hundreds_of_positions_back(tmp_path, kind, wide, dtype_name, stored, tolerance):
    """The mark at position 3 of 420 tokens: the last logits hang on it.  A state that is lost between steps, zeroed with a slot,
    mixed up in a batch or not handed from chunk to chunk shows."""
    folder = sh.marked_folder(tmp_path, stored, kind, wide=wide)
    doc, tensors = sh.load_folder(folder)
    tokens = sh.with_mark(doc, 420, 3, seed=1)
    requests = {"r0": tokens, "r1": sh.with_mark(doc, 90, 50, seed=2), "r2": tokens[:200]}
    expected = sh.oracle(folder, requests)
    without = ps.forward(doc, tensors, tokens[:3] + [sh.FILL] + tokens[4:]).numpy()
    assert np.abs(without[-1] - expected["r0"][-1]).max() > 0.2 * np.abs(expected["r0"]).max(), "the far token decides nothing"
    for trace in (rh.trace_whole(requests), rh.trace_tail_by_one(requests, tail=40), rh.trace_portions(requests, sizes=(17, 2, 30, 64, 3)),
                  rh.trace_mixed(requests, seed=4, max_live=2)):
        rows, _ = rh.run_in_process(folder, dtype_name, trace, page_size=16)
        sh.assert_rows_close(rows, expected, tolerance, kind)


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
def test_long_decoding_from_the_first_token(tmp_path, dtype_name, stored, tolerance):
    """Two tokens of prompt, then 300 decoded one by one (windows pass over decoded tokens, pages go back); beside it a request that
    is fed token by token from position 0.  The decode steps replay captured graphs."""
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_D, seed=8, dtype=stored)
    requests = sh.random_requests(sh.SMALL_D, (302, 9), seed=5)
    expected = sh.oracle(folder, requests)
    long, short = requests["r0"], requests["r1"]
    trace = [{"entries": [{"id": "r0", "tokens": long[:2], "want": [0, 1]}], "end": []}]
    for p in range(2, len(long)):
        entries = [{"id": "r0", "tokens": [long[p]], "want": [0]}]
        if p - 2 < len(short):
            entries.append({"id": "r1", "tokens": [short[p - 2]], "want": [0]})
        trace.append({"entries": entries, "end": ["r1"] if p - 2 == len(short) - 1 else []})
    trace[-1]["end"] = ["r0"]
    for i, step in enumerate(trace):
        step["step"] = i
    rows, session = rh.run_in_process(folder, dtype_name, trace)
    whole_model_close(rows, expected, dtype_name)
    assert len(rows["r0"]) == 302 and len(rows["r1"]) == 9
    assert session.runner.graphs is not None and session.runner.graphs.replays > 200


@pytest.mark.parametrize("dtype_name,stored", [("float32", torch.float32), ("bfloat16", torch.bfloat16)])
def test_greedy_generation_through_the_entry_point(tmp_path, dtype_name, stored):
    from sglang_rs_b200 import Engine
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_A, seed=11, dtype=stored)
    doc, tensors = sh.load_folder(folder)
    prompts = list(sh.random_requests(sh.SMALL_A, (5, 17, 33, 70), seed=8).values())
    engine = Engine(model_path=folder, dtype=dtype_name, page_size=16, max_total_tokens=400, max_running_requests=3,
                    chunked_prefill_size=16)
    results = engine.generate(prompts, {"max_new_tokens": 12})
    for prompt, result in zip(prompts, results):
        assert result["finished"] and len(result["output_ids"]) == 12
        tokens = list(prompt)
        for token in result["output_ids"]:
            logits = ps.forward(doc, tensors, tokens)[-1]
            best = int(torch.argmax(logits))
            limit = 1e-4 if dtype_name == "float32" else 4e-2
            assert float(logits[best] - logits[token]) <= limit * float(logits.abs().max()), (prompt[:4], token, best)
            tokens.append(token)
    again = Engine(model_path=folder, dtype=dtype_name, page_size=8, max_total_tokens=400, max_running_requests=1,
                   chunked_prefill_size=7, disable_cuda_graph=True)
    if dtype_name == "float32":
        assert [again.generate(p, {"max_new_tokens": 12})["output_ids"] for p in prompts] == [r["output_ids"] for r in results]
    engine.cache.check_invariants()
    assert engine.flush_cache()
    assert all(a.free_count == a.num_pages for a in engine.cache.allocators.values())
    assert engine.cache.state_pool.free_count == engine.cache.max_requests


def test_preemption_on_a_small_pool_gives_the_same_tokens(tmp_path):
    """Three requests on a pool that cannot hold them: a request is preempted, gives its pages and its state slot back and is
    computed again from its first token, in other portions and another slot; every token stays what the plain implementation
    gives (32-bit)."""
    from sglang_rs_b200 import Engine
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_B, seed=4, dtype=torch.float32)
    doc, tensors = sh.load_folder(folder)
    prompts = list(sh.random_requests(sh.SMALL_B, (40, 35, 50), seed=2).values())
    engine = Engine(model_path=folder, dtype="float32", page_size=16, max_total_tokens=160, max_running_requests=3,
                    chunked_prefill_size=64)
    results = engine.generate(prompts, {"max_new_tokens": 40})
    assert engine.scheduler.stats["preemptions"] >= 1
    assert [r["output_ids"] for r in results] == [sh.plain_greedy(doc, tensors, p, 40) for p in prompts]
    assert engine.cache.state_pool.free_count == engine.cache.max_requests


def test_the_command_line_and_the_trace_program_take_the_design(tmp_path):
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    config_path = tmp_path / "config.json"
    config_path.write_text(json.dumps(sh.SMALL_C))
    folder = str(tmp_path / "written")
    made = subprocess.run([sys.executable, os.path.join(root, "bin", "sglang-rs"), "random-model", "--config", str(config_path),
                           "--out", folder, "--seed", "4", "--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert made.returncode == 0, made.stderr[-2000:]
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_C, seed=4, dtype=torch.float32)     # (ranks that no configuration names)
    doc, tensors = sh.load_folder(folder)
    command = [sys.executable, os.path.join(root, "bin", "sglang-rs"), "generate", f"--model-path={folder}", "--device", "cuda",
               "--dtype", "float32", "--input-ids", "5,17,3", "--input-ids", "9 8 7 6", "--max-new-tokens", "5",
               "--max-total-tokens", "256"]
    process = subprocess.run(command, capture_output=True, text=True, timeout=600)
    assert process.returncode == 0, process.stderr[-2000:]
    lines = [json.loads(line) for line in process.stdout.strip().splitlines()]
    assert [l["output_ids"] for l in lines] == [sh.plain_greedy(doc, tensors, p, 5) for p in ([5, 17, 3], [9, 8, 7, 6])]
    tokens = sh.random_requests(doc, (37,), seed=1)["r0"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[30:], "want": [6]}], "end": ["a"]}]
    out = tmp_path / "out"
    replay = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                             "--out", str(out), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                            capture_output=True, text=True, timeout=600)
    assert replay.returncode == 0 and replay.stdout.split() == ["done", "0", "done", "1"], replay.stderr[-2000:]
    want = ps.forward(doc, tensors, tokens).numpy()
    first = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    last = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    for got, pos in ((first[0], 0), (first[1], 29), (last[0], 36)):
        assert float(np.abs(got - want[pos]).max()) <= 5e-5 * float(np.abs(want).max())
