"""Tekilorn on the GPU against the plain implementation: each mechanism alone, whole prompts, prompts with a tail decoded
token by token, portions down to two tokens, mixed batches over a small pool (pages are used again), keys just inside and
just outside a window, the kept first tokens and the next ones, keys far away at page borders, long decoding, and greedy
generation through the entry point."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tekilorn as pt
import replay_helpers as rh
import tekilorn_helpers as th

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [("float32", torch.float32, 2e-5), ("bfloat16", torch.bfloat16, 6e-2)]
ALL = [th.SMALL_A, th.SMALL_B, th.SMALL_C, th.SMALL_D, th.SMALL_E]


def seen(tensor, dtype):
    """What the kernel sees of a tensor: rounded to the storage type, as a float64 array."""
    return tensor.to(dtype).to(torch.float64).numpy()


def close(got, want, dtype, what, fraction=None):
    tolerance = fraction if fraction is not None else (2e-5 if dtype == torch.float32 else 2e-2)
    want = np.asarray(want, dtype=np.float64)
    scale = float(np.abs(want).max()) or 1.0
    error = float(np.abs(got.detach().double().cpu().numpy() - want).max()) / scale
    assert error <= tolerance, (what, error)


# ------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [44, 45, 2048])
def test_the_vector_of_a_pass_rides_in_the_next_norm(dtype, width):
    from sglang_rs_b200.parts import GroupedRmsNorm, PassStep
    g = torch.Generator().manual_seed(1)
    rows, eps = 9, 1e-5
    stored = {"n": torch.rand(width, generator=g) + 0.5, "loop.step": torch.randn(3, width, generator=g)}
    norm, entry = GroupedRmsNorm(width, eps, "n"), PassStep(width, 3, "loop.step")
    norm.load(stored, DEV, dtype)
    entry.load(stored, DEV, dtype)
    x, y = torch.randn(rows, width, generator=g) * 2, torch.randn(rows, width, generator=g)
    pieces = torch.randn(3, rows, width, generator=g)
    for pending, exact in ((None, 0.0), (y.to(dtype), seen(y, dtype)), (y, y.double().numpy()), (pieces, pieces.double().sum(0).numpy())):
        for t in (0, 2):
            residual = x.to(DEV)
            stream, delta = entry.forward(None, residual, None if pending is None else pending.to(DEV), None, t)
            assert stream is residual
            out = norm.add_norm(stream, delta, dtype)
            total = x.double().numpy() + exact + stored["loop.step"][t].double().numpy()
            close(residual, total, torch.float32, "stream + pending + step", 1e-6)
            close(out, pt.norm(total, stored["n"].double().numpy(), eps), dtype, "norm of the sum")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n_q,n_kv,d,vd,rot,temp,parts", [(4, 2, 16, 8, 8, None, 0), (3, 3, 10, 14, 6, (0.5, 7), 3),
                                                          (2, 1, 64, 64, 0, (0.35, 63), 0), (5, 1, 12, 4, 12, (0.2, 1), 2)])
def test_interleaved_rotation_query_temperature_pages_and_gates(dtype, n_q, n_kv, d, vd, rot, temp, parts):
    from sglang_rs_b200 import ops
    g = torch.Generator().manual_seed(n_q * 100 + d)
    page, pages = 4, 9
    positions = torch.tensor([0, 1, 5, 6, 7, 62, 63, 64, 65, 500, 4097], dtype=torch.int32)
    rows = len(positions)
    width = (n_q + n_kv) * d + n_kv * vd + n_q
    proj = torch.randn(rows, width + 3, generator=g) * 2
    slots = torch.randperm(pages * page, generator=g)[:rows].int()
    inv_freq = torch.tensor([50.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float32) if rot else None
    if parts and dtype == torch.bfloat16:
        pieces = torch.randn(parts, rows, width + 3, generator=g)
        given, exact = pieces.to(DEV), pieces.double().sum(0).numpy()
    else:
        given, exact = proj.to(dtype).to(DEV), seen(proj, dtype)
    q_out = torch.zeros(rows, n_q, d, dtype=dtype, device=DEV)
    k_pool = torch.zeros(pages, n_kv, page, d, dtype=dtype, device=DEV)
    v_pool = torch.zeros(pages, n_kv, page, vd, dtype=dtype, device=DEV)
    gates = torch.zeros(rows, n_q, dtype=torch.float32, device=DEV)
    word = ops.new_error_word(DEV)
    ops.proj_norm_rope_kv(given, q_out, k_pool, v_pool, positions.to(DEV), slots.to(DEV), None, None, 0.0,
                          inv_freq.to(DEV) if rot else None, rot, True, n_q, n_kv, d, vd, word, gate_out=gates, per_head=True,
                          temperature=temp)
    ops.raise_on_error_word(word)
    turn = {"base": 50.0, "dims": rot} if rot else None
    q = pt.rotate_pairs(exact[:, :n_q * d].reshape(rows, n_q, d), positions.numpy(), turn)
    k = pt.rotate_pairs(exact[:, n_q * d:(n_q + n_kv) * d].reshape(rows, n_kv, d), positions.numpy(), turn)
    factor = pt.query_temperature(positions.numpy(), {"coef": temp[0], "every": temp[1]} if temp else None)
    # (angles are 32-bit: position 4,097 leaves them off by 2e-4 of a turn's radian)
    close(q_out, q * factor[:, None, None], dtype, "q", 5e-4 if dtype == torch.float32 else None)
    page_of, inside = (slots // page).long().to(DEV), (slots % page).long().to(DEV)
    close(k_pool[page_of, :, inside], k, dtype, "keys in their slots", 5e-4 if dtype == torch.float32 else None)
    close(v_pool[page_of, :, inside], exact[:, (n_q + n_kv) * d:(n_q + n_kv) * d + n_kv * vd].reshape(rows, n_kv, vd), dtype, "values")
    close(gates, pt.sigmoid(exact[:, width - n_q:width]), torch.float32, "gates", 1e-5)


def paged(keys, values, page, dtype, seed):
    """Keys [T, G, d] and values [T, G, dv] of one request laid into shuffled pages; (k_pool, v_pool, block table)."""
    tokens = keys.shape[0]
    count = -(-tokens // page)
    order = torch.randperm(count + 3, generator=torch.Generator().manual_seed(seed))[:count]
    k_pool = torch.zeros(count + 3, keys.shape[1], page, keys.shape[2], dtype=dtype)
    v_pool = torch.zeros(count + 3, values.shape[1], page, values.shape[2], dtype=dtype)
    for t in range(tokens):
        k_pool[order[t // page], :, t % page] = keys[t].to(dtype)
        v_pool[order[t // page], :, t % page] = values[t].to(dtype)
    return k_pool.to(DEV), v_pool.to(DEV), order.int().view(1, -1).to(DEV)


def without_passed_pages(table, page, length, window, keep):
    """The block table of a request of ``length`` tokens whose passed pages were given back."""
    table = table.clone()
    for logical in range(table.shape[1]):
        if window and (logical + 1) * page <= length - window and logical * page >= keep:
            table[0, logical] = -1
    return table


def loud_edges(v, window, keep, rows):
    """Values of the keys at the edges of the kept first tokens and of the rows' windows, made large."""
    tokens = v.shape[0]
    for j in {keep - 1, keep, keep + 1}:
        if 0 <= j < tokens:
            v[j] *= 5.0
    for r in rows:
        for j in (int(r) - window, int(r) - window + 1):
            if window and 0 <= j < tokens:
                v[j] *= 3.0
    return v


def expected_attention(q, k, v, per, scale, window, keep, softcap, dtype):
    return pt.attend(seen(q, dtype), np.repeat(seen(k, dtype), per, 1), np.repeat(seen(v, dtype), per, 1), scale, window or None,
                     keep, softcap)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,d,vd,window,keep,softcap,split", [
    (4, 2, 16, 8, 24, 5, None, 0), (3, 1, 10, 14, 40, 33, 4.0, 32), (34, 1, 8, 12, 70, 64, None, 64), (2, 2, 20, 20, 1, 3, 1.5, 0),
    (2, 1, 16, 16, 20, 90, None, 48), (2, 1, 16, 16, 0, 0, 2.5, 32), (2, 1, 12, 8, 7, 1, None, 128)])
def test_the_generic_kernel_keeps_first_tokens_and_caps_scores(dtype, heads, kv, d, vd, window, keep, softcap, split):
    """Rows anywhere in a sequence of 150 keys, with and without key splits; the pages that lie between the kept tokens and the
    last row's window are gone from the block table for a row at the end."""
    from sglang_rs_b200 import ops
    g = torch.Generator().manual_seed(heads + d)
    tokens, page, scale = 150, 8, 0.9
    q, k, v = torch.randn(tokens, heads, d, generator=g), torch.randn(tokens, kv, d, generator=g), torch.randn(tokens, kv, vd, generator=g)
    rows = torch.tensor([0, 1, keep, keep + 1, 23, 24, 25, 63, 64, 100, 149])
    v = loud_edges(v, window, keep, (64, 100, 149))
    gates = torch.rand(tokens, heads, generator=g)
    k_pool, v_pool, table = paged(k, v, page, dtype, 3)
    want = expected_attention(q, k, v, heads // kv, scale, window, keep, softcap, dtype) * gates.double().numpy()[:, :, None]
    word = ops.new_error_word(DEV)
    for batch, pages in ((rows, table), (rows[-1:], without_passed_pages(table, page, tokens - 1, window, keep))):
        out = torch.zeros(len(batch), heads, vd, dtype=dtype, device=DEV)
        splits = -(-tokens // split) + 1 if split else 1
        acc = torch.zeros(len(batch) * heads * splits * vd, device=DEV) if split else None
        ml = torch.zeros(len(batch) * heads * splits * 2, device=DEV) if split else None
        ops.paged_attention(q[batch].to(dtype).to(DEV), k_pool, v_pool, out, batch.int().to(DEV),
                            torch.zeros(len(batch), dtype=torch.int32, device=DEV), pages, scale=scale, window=window,
                            split_size=split, max_splits=splits, scratch_acc=acc, scratch_ml=ml, error_word=word,
                            gates=gates[batch].contiguous().to(DEV), keep_first=keep, softcap=softcap)
        ops.raise_on_error_word(word)
        close(out, want[batch.numpy()], dtype, "attention")


def split_maps(q, k, heads, kv, d):
    """[T, heads, 2 d] and [T, kv, 2 d] as the two maps' queries and keys."""
    return [(q[..., t * d:(t + 1) * d], k[..., t * d:(t + 1) * d]) for t in range(2)]


def expected_maps(q, k, v, per, d, scale, softcap, join, dtype, window=0, keep=0):
    a = [expected_attention(qm, km, v, per, scale, window, keep, softcap, dtype) for qm, km in split_maps(q, k, 0, 0, d)]
    return pt.rms(a[0] - join.subtract * a[1], join.eps) * join.scale


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,d,vd,softcap,split,window,keep", [
    (4, 2, 12, 20, 3.0, 0, 0, 0), (3, 3, 5, 14, None, 32, 0, 0), (18, 1, 8, 8, 2.0, 64, 0, 0), (2, 1, 32, 64, None, 128, 20, 6)])
def test_two_maps_through_the_generic_kernel(dtype, heads, kv, d, vd, softcap, split, window, keep):
    from sglang_rs_b200 import ops
    g = torch.Generator().manual_seed(heads + d)
    tokens, page, scale, join = 140, 8, 0.8, ops.MapJoin(0.63, 0.45, 1e-5)
    q, k, v = torch.randn(tokens, heads, 2 * d, generator=g), torch.randn(tokens, kv, 2 * d, generator=g), torch.randn(tokens, kv, vd, generator=g)
    rows = torch.tensor([0, 1, 7, 31, 32, 63, 64, 100, 139])
    k_pool, v_pool, table = paged(k, v, page, dtype, 3)
    wide = torch.zeros(len(rows), heads * vd + 8, dtype=dtype, device=DEV)              # rows of the result inside wider ones
    out = wide[:, :heads * vd].as_strided((len(rows), heads, vd), (wide.stride(0), vd, 1))
    splits = -(-tokens // split) + 1 if split else 1
    acc = torch.zeros(len(rows) * heads * 2 * splits * vd, device=DEV) if split else None
    ml = torch.zeros(len(rows) * heads * 2 * splits * 2, device=DEV) if split else None
    word = ops.new_error_word(DEV)
    ops.paged_attention(q[rows].to(dtype).to(DEV), k_pool, v_pool, out, rows.int().to(DEV),
                        torch.zeros(len(rows), dtype=torch.int32, device=DEV), table, scale=scale, window=window, split_size=split,
                        max_splits=splits, scratch_acc=acc, scratch_ml=ml, error_word=word, softcap=softcap, join=join,
                        keep_first=keep)
    ops.raise_on_error_word(word)
    want = expected_maps(q, k, v, heads // kv, d, scale, softcap, join, dtype, window, keep)
    close(out, want[rows.numpy()], dtype, "joined maps")
    assert float(wide[:, heads * vd:].abs().max()) == 0.0


def portion_tiles(first, tokens, size):
    return torch.tensor([[b - first, min(size, tokens - b), 0, b] for b in range(first, tokens, size)], dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("d,heads,kv,window,keep,softcap", [(64, 4, 2, 48, 6, None), (128, 2, 1, 100, 70, None), (64, 3, 3, 1, 64, 3.0),
                                                            (128, 3, 1, 33, 1, 2.0), (64, 2, 1, 0, 0, 1.5), (64, 2, 1, 260, 65, None),
                                                            (64, 4, 2, 0, 0, 30.0), (128, 4, 2, 90, 4, 80.0)])
def test_the_tensor_core_kernels_keep_first_tokens_and_cap_scores(d, heads, kv, window, keep, softcap):
    """tcgen05 tiles and mma.sync tiles for prompt portions, split keys for decoded rows, in bfloat16; the portions start
    inside a page; pages between the kept tokens and the first row's window are gone from the block table."""
    from sglang_rs_b200 import ops
    dtype = torch.bfloat16
    g = torch.Generator().manual_seed(d + heads)
    tokens, page, scale = 420, 16, d ** -0.5 * 1.5
    q, k, v = (torch.randn(tokens, n, d, generator=g) for n in (heads, kv, kv))
    v = loud_edges(v, window, keep, (200, 300, 419))
    gates = torch.rand(tokens, heads, generator=g)
    k_pool, v_pool, table = paged(k, v, page, dtype, 5)
    want = expected_attention(q, k, v, heads // kv, scale, window, keep, softcap, dtype) * gates.double().numpy()[:, :, None]
    word = ops.new_error_word(DEV)
    qd, gd = q.to(dtype).to(DEV), gates.to(DEV)
    terms = dict(keep_first=keep, softcap=softcap)
    for name, size, run in (("tcgen05 tiles", ops.TC_TILE_ROWS, ops.tiled_attention_tc), ("mma tiles", 64, ops.tiled_attention)):
        for first in (0, 37, 292):                           # 292: one whole tile of 128 rows behind a long prefix
            out = torch.zeros(tokens - first, heads, d, dtype=dtype, device=DEV)
            run(qd[first:].contiguous(), k_pool, v_pool, out, portion_tiles(first, tokens, size),
                without_passed_pages(table, page, first, window, keep), scale=scale, window=window, error_word=word,
                gates=gd[first:].contiguous(), **terms)
            close(out, want[first:], dtype, (name, first))
    rows = torch.tensor([0, 1, 15, 16, 63, 64, 65, 127, 200, 300, 419])
    for batch, pages in ((rows, table), (rows[-2:], table), (rows[-1:], without_passed_pages(table, page, tokens - 1, window, keep))):
        out = torch.zeros(len(batch), heads, d, dtype=dtype, device=DEV)
        ops.decode_attention(qd[batch.to(DEV)].contiguous(), k_pool, v_pool, out, batch.int().to(DEV),
                             torch.zeros(len(batch), dtype=torch.int32, device=DEV), pages, scale=scale, window=window,
                             scratch_acc=torch.zeros(1 << 20, device=DEV), scratch_ml=torch.zeros(1 << 16, device=DEV),
                             counters=torch.zeros(256, dtype=torch.int32, device=DEV), error_word=word,
                             gates=gd[batch.to(DEV)].contiguous(), max_keys=420 if len(batch) == 2 else None, **terms)
        close(out, want[batch.numpy()], dtype, f"split keys, {len(batch)} rows")
    ops.raise_on_error_word(word)


@pytest.mark.parametrize("d,heads,kv,softcap,window,keep", [(32, 4, 2, 4.0, 0, 0), (64, 3, 1, None, 0, 0), (64, 8, 1, 2.0, 90, 20),
                                                            (32, 1, 1, None, 48, 5), (64, 2, 2, 40.0, 0, 0), (32, 2, 1, 70.0, 0, 0)])
def test_two_maps_through_the_tensor_core_kernels(d, heads, kv, softcap, window, keep):
    """(Caps: some scores beyond them, all within them, and a cap so large that the running maximum is kept.)
    Both maps of a head in one block, joined in tensor memory (tcgen05 tiles) or where the splits meet (decoded rows)."""
    from sglang_rs_b200 import ops
    dtype = torch.bfloat16
    g = torch.Generator().manual_seed(d + heads)
    tokens, page, scale, join = 420, 16, d ** -0.5 * 2.0, ops.MapJoin(0.57, 0.35, 1e-5)
    q, k, v = torch.randn(tokens, heads, 2 * d, generator=g), torch.randn(tokens, kv, 2 * d, generator=g), torch.randn(tokens, kv, 2 * d, generator=g)
    k_pool, v_pool, table = paged(k, v, page, dtype, 5)
    want = expected_maps(q, k, v, heads // kv, d, scale, softcap, join, dtype, window, keep)
    word = ops.new_error_word(DEV)
    qd = q.to(dtype).to(DEV)
    terms = dict(keep_first=keep, softcap=softcap, join=join)
    for first in (0, 37, 292):
        out = torch.zeros(tokens - first, heads, 2 * d, dtype=dtype, device=DEV)
        ops.tiled_attention_tc(qd[first:].contiguous(), k_pool, v_pool, out, portion_tiles(first, tokens, ops.TC_TILE_ROWS), table,
                               scale=scale, window=window, error_word=word, **terms)
        close(out, want[first:], dtype, ("tcgen05 tiles", first))
    rows = torch.tensor([0, 1, 15, 16, 63, 64, 65, 127, 200, 300, 419])
    # many rows and a long bound: splits through memory; few rows: a cluster merges; one split: no merge at all
    for batch, bound in ((rows, None), (rows[-2:], 420), (rows[:3], 64), (rows.repeat(40), 420)):
        out = torch.zeros(len(batch), heads, 2 * d, dtype=dtype, device=DEV)
        ops.decode_attention(qd[batch.to(DEV)].contiguous(), k_pool, v_pool, out, batch.int().to(DEV),
                             torch.zeros(len(batch), dtype=torch.int32, device=DEV), table, scale=scale, window=window,
                             scratch_acc=torch.zeros(1 << 22, device=DEV), scratch_ml=torch.zeros(1 << 17, device=DEV),
                             counters=torch.zeros(1024, dtype=torch.int32, device=DEV), error_word=word, max_keys=bound, **terms)
        close(out, want[batch.numpy()], dtype, f"split keys, {len(batch)} rows")
    ops.raise_on_error_word(word)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,rows,width,ff,shared", [(5, 2, 9, 40, 24, True), (2, 2, 200, 40, 24, False), (4, 1, 33, 40, 24, True),
                                                              (3, 3, 300, 40, 24, True), (6, 2, 130, 36, 10, True)])
def test_experts_weighed_on_their_input_and_a_gated_shared_one(dtype, experts, top, rows, width, ff, shared):
    """Sigmoid scores, unnormalised, on the experts' inputs; clamped activations whose limits bite (so that a weight on the
    result instead would show); a shared expert of another limit behind a sigmoid per token; few rows and many, sizes that the
    grouped tcgen05 products take and sizes they do not."""
    from sglang_rs_b200 import ops
    from sglang_rs_b200.parts import GatedMlp, GatedMlpNames, RoutedExperts
    g = torch.Generator().manual_seed(experts * 10 + top)
    limit, shared_limit = 1.1, 0.6
    names = lambda e: GatedMlpNames(gate=f"p.e{e}.gate", up=f"p.e{e}.up", down=f"p.e{e}.down")
    part = RoutedExperts(width, ff, experts, top, "swiglu_clamp", "p.router", names, scoring="sigmoid", activation_param=limit,
                         weigh_inputs=True, shared_gate_name="p.shared.sg" if shared else None,
                         shared=GatedMlp(width, 16, "swiglu_clamp", GatedMlpNames("p.shared.gate", "p.shared.up", "p.shared.down"),
                                         float_result=True, activation_param=shared_limit) if shared else None)
    specs = part.tensor_specs()
    stored = {name: (torch.randn(specs[name].shape, generator=g) * 0.4).to(dtype) for name in sorted(specs)}
    part.load(stored, DEV, dtype)
    h = torch.randn(rows, width, generator=g)

    class Ctx:
        error_word = ops.new_error_word(DEV)
    out = part.forward(Ctx, h.to(dtype).to(DEV))
    ops.raise_on_error_word(Ctx.error_word)
    w = {k: v.double().numpy() for k, v in stored.items()}
    f = {"router": {"experts": experts, "top": top}, "expert": {"limit": limit}, "shared": {"limit": shared_limit} if shared else None}
    want = pt.routed(seen(h, dtype), w, "p.", f)
    assert out.dtype == torch.float32
    errors = np.abs(out.double().cpu().numpy() - want).max(axis=1) / np.abs(want).max()
    limit = 2e-5 if dtype == torch.float32 else 3e-2
    assert (errors > limit).sum() <= (0 if dtype == torch.float32 else 0.03 * rows), float(errors.max())


# ------------------------------------------------------------------------------ whole models, every way of cutting
@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("doc", ALL, ids="abcde")
def test_prompts_tails_portions_and_mixed_batches(tmp_path, doc, dtype_name, stored, tolerance):
    folder = th.make_folder(tmp_path, "m", doc, seed=5, dtype=stored)
    requests = th.random_requests(doc, (1, 2, 23, 64, 65, 150, 131), seed=3)
    expected = th.oracle(folder, requests)
    worst = {}
    for name, trace, page in (("whole", rh.trace_whole(requests), 16), ("tail", rh.trace_tail_by_one(requests, tail=45), 16),
                              ("portions", rh.trace_portions(requests), 8), ("mixed", rh.trace_mixed(requests, seed=9), 16)):
        # the pool holds what is live at any time and no more, so pages go from one request to the next
        rows, session = rh.run_in_process(folder, dtype_name, trace, page_size=page)
        assert all(len(rows[rid]) == len(tokens) for rid, tokens in requests.items())
        worst[name] = rh.worst_error(rows, expected)
        print(doc["width"], dtype_name, name, worst[name])
        th.assert_rows_close(rows, expected, tolerance, dtype_name, name)
        if name == "mixed":
            assert any(len(owners) > 1 for owners in session.page_owners.values()), "no page was used again"


def test_layers_one_by_one_against_the_plain_stream(tmp_path):
    """The residual stream after every layer run (a layer of the stretch counts each time), 32-bit, a prompt in one step."""
    from sglang_rs_b200.engine.replay import ReplaySession
    folder = th.make_folder(tmp_path, "m", th.SMALL_A, seed=2, dtype=torch.float32)
    doc, w = th.load_folder(folder)
    tokens = th.random_requests(doc, (50,), seed=6)["r0"]
    after = []
    logits = pt.forward(doc, w, tokens, after)
    session = ReplaySession(folder, "float32", 64, 16, use_cuda_graphs=False)
    streams = []
    for block in session.model.layers:
        def forward(ctx, cache, residual, delta, inner=block.forward):
            residual, delta = inner(ctx, cache, residual, delta)
            streams.append(residual.double().cpu().numpy() + delta.double().cpu().numpy())     # what the next kernel will sum
            return residual, delta
        block.forward = forward
    out = session.run({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": list(range(len(tokens)))}], "end": ["a"]})
    assert len(streams) == len(after) == 8
    for index, (got, want) in enumerate(zip(streams, after)):
        assert np.abs(got - want).max() <= 2e-5 * np.abs(want).max(), f"stream after layer run {index}"
    assert np.abs(out - logits).max() <= 2e-5 * np.abs(logits).max()


@pytest.mark.parametrize("doc", [th.SMALL_A, th.SMALL_D], ids="ad")
def test_the_cut_and_the_batch_change_nothing_beyond_rounding(tmp_path, doc):
    """In 32-bit the logits of a position agree to rounding whatever the portions, the pages and the requests beside it."""
    folder = th.make_folder(tmp_path, "m", doc, seed=6, dtype=torch.float32)
    requests = th.random_requests(doc, (40, 97, 130), seed=4)
    whole, _ = rh.run_in_process(folder, "float32", rh.trace_whole(requests), page_size=16)
    for trace, page in ((rh.trace_portions(requests, sizes=(2, 2, 3, 33, 2, 15)), 4), (rh.trace_mixed(requests, seed=2, max_live=3), 32)):
        rows, _ = rh.run_in_process(folder, "float32", trace, page_size=page)
        for rid in requests:
            for pos, row in rows[rid].items():
                assert float(np.abs(row - whole[rid][pos]).max()) <= 5e-5 * float(np.abs(whole[rid][pos]).max()), (rid, pos)


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("window,keep,wide", [(16, 3, False), (33, 16, False), (96, 0, False), (40, 17, True), (70, 64, True)])
def test_a_marked_key_at_the_edges_of_the_window_and_of_the_kept_tokens(tmp_path, window, keep, wide, dtype_name, stored, tolerance):
    """A model made so that head 0 looks at the marked token only (``tekilorn_helpers.marked_folder``).  The row that is
    window - 1 positions behind it still sees it, the next one does not, unless it is one of the kept first tokens, which every
    row sees: in a whole prompt, decoded token by token (the window passes over decoded tokens, pages behind it go back to the
    pool, those of the kept tokens stay), and in portions cut at the edge."""
    folder = th.marked_folder(tmp_path, stored, "attention_2", window, keep, wide)
    doc, w = th.load_folder(folder)
    for mark in sorted({0, max(keep - 1, 0), keep, keep + 6, 31}):
        tokens, without = th.with_mark(doc, mark + window + 40, mark, seed=mark)
        requests = {"r0": tokens}
        expected = th.oracle(folder, requests)
        plain = pt.forward(doc, w, without)
        inside, outside = mark + window - 1, mark + window
        size = np.abs(expected["r0"]).max()
        assert np.abs(plain[inside] - expected["r0"][inside]).max() > 0.15 * size, "the marked key decides nothing"
        moved = np.abs(plain[outside:] - expected["r0"][outside:]).max(axis=1)
        assert (moved > 0.15 * size).all() if mark < keep else (moved == 0.0).all()
        traces = (rh.trace_whole(requests), rh.trace_tail_by_one(requests, tail=window + 39),
                  rh.trace_portions(requests, sizes=(inside, 1, 1, 2)), rh.trace_portions(requests, sizes=(mark + 1, 2, window - 4, 2, 2, 3)))
        for trace in traces:
            rows, _ = rh.run_in_process(folder, dtype_name, trace, page_size=16)
            th.assert_rows_close(rows, expected, tolerance, dtype_name, (window, keep, mark))


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
@pytest.mark.parametrize("wide", [False, True])
def test_a_far_key_at_a_page_border_decides_the_logits(tmp_path, wide, dtype_name, stored, tolerance):
    """The differential attention has no window: the logits of late positions hang on a key 280 tokens back, the last one of a
    page or the first one of the next, in whole prompts, in decoded tokens and in portions."""
    folder = th.marked_folder(tmp_path, stored, "attention", wide=wide)
    doc, w = th.load_folder(folder)
    for mark in (15, 16):
        tokens, without = th.with_mark(doc, 300, mark, seed=mark)
        requests = {"r0": tokens}
        expected = th.oracle(folder, requests)
        plain = pt.forward(doc, w, without)
        assert np.abs(plain[-1] - expected["r0"][-1]).max() > 0.15 * np.abs(expected["r0"]).max(), "the far key decides nothing"
        for trace in (rh.trace_whole(requests), rh.trace_tail_by_one(requests, tail=40), rh.trace_portions(requests, sizes=(17, 2, 30))):
            rows, _ = rh.run_in_process(folder, dtype_name, trace, page_size=16)
            th.assert_rows_close(rows, expected, tolerance, dtype_name, mark)


@pytest.mark.parametrize("dtype_name,stored,tolerance", DTYPES)
def test_long_decoding_from_the_first_token(tmp_path, dtype_name, stored, tolerance):
    """Two tokens of prompt, then 300 decoded one by one (windows pass, pages go back, several key splits); beside it a
    request that is fed token by token from position 0.  The decode steps replay captured graphs."""
    folder = th.make_folder(tmp_path, "m", th.SMALL_D, seed=8, dtype=stored)
    requests = th.random_requests(th.SMALL_D, (302, 9), seed=5)
    expected = th.oracle(folder, requests)
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
    th.assert_rows_close(rows, expected, tolerance, dtype_name)
    assert len(rows["r0"]) == 302 and len(rows["r1"]) == 9
    assert session.runner.graphs is not None and session.runner.graphs.replays > 200


@pytest.mark.parametrize("dtype_name,stored", [("float32", torch.float32), ("bfloat16", torch.bfloat16)])
def test_greedy_generation_through_the_entry_point(tmp_path, dtype_name, stored):
    from sglang_rs_b200 import Engine
    folder = th.make_folder(tmp_path, "m", th.SMALL_A, seed=11, dtype=stored)
    doc, w = th.load_folder(folder)
    prompts = list(th.random_requests(th.SMALL_A, (5, 17, 33, 70), seed=8).values())
    engine = Engine(model_path=folder, dtype=dtype_name, page_size=16, max_total_tokens=400, max_running_requests=3,
                    chunked_prefill_size=16)
    results = engine.generate(prompts, {"max_new_tokens": 12})
    for prompt, result in zip(prompts, results):
        assert result["finished"] and len(result["output_ids"]) == 12
        tokens = list(prompt)
        for token in result["output_ids"]:
            logits = pt.forward(doc, w, tokens)[-1]
            best = int(np.argmax(logits))
            limit = 0.0 if dtype_name == "float32" else 6e-2
            assert float(logits[best] - logits[token]) <= limit * float(np.abs(logits).max()), (prompt[:4], token, best)
            tokens.append(token)
    again = Engine(model_path=folder, dtype=dtype_name, page_size=8, max_total_tokens=400, max_running_requests=1,
                   chunked_prefill_size=7, disable_cuda_graph=True)
    if dtype_name == "float32":
        assert [again.generate(p, {"max_new_tokens": 12})["output_ids"] for p in prompts] == [r["output_ids"] for r in results]
    # a pool too small for what runs at once: requests are preempted and start again; nothing else changes
    tight = Engine(model_path=folder, dtype=dtype_name, page_size=8, max_total_tokens=128, max_running_requests=3, chunked_prefill_size=16)
    if dtype_name == "float32":
        assert [r["output_ids"] for r in tight.generate(prompts, {"max_new_tokens": 12})] == [r["output_ids"] for r in results]
    engine.cache.check_invariants()
    assert engine.flush_cache()
    assert all(a.free_count == a.num_pages for a in engine.cache.allocators.values())


def test_the_command_line_and_the_trace_program_take_the_design(tmp_path):
    """`sglang-rs random-model` writes a folder from a configuration, `sglang-rs generate` decodes from it, and `trace_run`
    replays steps on it: the same programs as for every model."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    config_path = tmp_path / "config.json"
    config_path.write_text(json.dumps(th.SMALL_C))
    folder = str(tmp_path / "written")
    made = subprocess.run([sys.executable, os.path.join(root, "bin", "sglang-rs"), "random-model", "--config", str(config_path),
                           "--out", folder, "--seed", "4", "--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert made.returncode == 0, made.stderr[-2000:]
    doc, w = th.load_folder(folder)
    command = [sys.executable, os.path.join(root, "bin", "sglang-rs"), "generate", f"--model-path={folder}", "--device", "cuda",
               "--dtype", "float32", "--input-ids", "5,17,3", "--input-ids", "9 8 7 6", "--max-new-tokens", "5",
               "--max-total-tokens", "256"]
    process = subprocess.run(command, capture_output=True, text=True, timeout=600)
    assert process.returncode == 0, process.stderr[-2000:]
    lines = [json.loads(line) for line in process.stdout.strip().splitlines()]
    assert [l["output_ids"] for l in lines] == [th.plain_greedy(doc, w, p, 5) for p in ([5, 17, 3], [9, 8, 7, 6])]
    tokens = th.random_requests(doc, (37,), seed=1)["r0"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[30:], "want": [6]}], "end": ["a"]}]
    out = tmp_path / "out"
    replay = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                             "--out", str(out), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                            capture_output=True, text=True, timeout=600)
    assert replay.returncode == 0 and replay.stdout.split() == ["done", "0", "done", "1"], replay.stderr[-2000:]
    want = pt.forward(doc, w, tokens)
    first = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    last = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    for got, pos in ((first[0], 0), (first[1], 29), (last[0], 36)):
        assert float(np.abs(got - want[pos]).max()) <= 2e-5 * float(np.abs(want).max())
