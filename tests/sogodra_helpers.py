"""Small Sogodra configurations and model folders for the tests.  None has the sizes of a real checkpoint; each makes unequal
what a convenient configuration would make equal or 1 (key and value widths, head counts, the two mixers of a parallel layer
and their factors, the ranks of the thin pairs, filters, windows, limits)."""
from __future__ import annotations

import json
import os
import random
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

import plain_sogodra as ps


def delta_sizes(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def delta(*sizes):
    return {"type": "delta", "mixer": delta_sizes(*sizes)}


def mingru(width):
    return {"type": "mingru", "mixer": {"width": width}}


def attention(heads, kv_heads, dim, vdim, window=None, rot_dims=None, base=10000.0, scaling=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if window is not None:
        m["mask"] = {"size": window}
    if rot_dims != 0:
        m["rot"] = {"base": base, "dims": dim if rot_dims is None else rot_dims}
        if scaling:
            m["rot"]["scaling"] = scaling
    return m


def parallel(left, right, left_scale, right_scale):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def layer(mixer, ff=None, limit=1.0):
    return dict(mixer, mlp={"kind": "dense", "ff": ff, "limit": limit} if ff else None)


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Sogodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


#: with these every branch of the ramp is met by some pair of a small head
RAMP = {"factor": 6.0, "low": 1.0, "high": 5.0, "original": 100}

#: every mixer; two parallel layers with windows of two lengths (two page groups); a filter of one tap; a layer without
#: feed-forward; q/k heads shared by value heads
SMALL_A = config(48, 90, [
    layer(delta(4, 2, 12, 20, 4), 72, 0.7),
    layer(parallel(attention(4, 2, 16, 12, window=24, rot_dims=12, base=500.0, scaling=RAMP), delta_sizes(6, 3, 8, 10, 3), 0.6, 1.3), 56, 2.0),
    layer(mingru(40)),
    layer(delta(3, 3, 16, 8, 1), 40, 1.2),
    layer(parallel(attention(3, 3, 8, 24, window=37, rot_dims=8), delta_sizes(2, 1, 24, 16, 5), 1.7, 0.4), 64, 0.9),
])
#: no window, no rotation in one parallel layer and no stretching in the other, one head on one head, a recurrence narrower
#: and one wider than the stream
SMALL_B = config(40, 70, [
    layer(mingru(24), 32, 0.5),
    layer(parallel(attention(2, 1, 24, 8, rot_dims=0), delta_sizes(1, 1, 16, 24, 2), 1.0, 1.0)),
    layer(parallel(attention(6, 2, 8, 8, window=9), delta_sizes(4, 1, 8, 8, 4), -0.5, 0.9), 48, 3.0),
    layer(mingru(88)),
    layer(delta(1, 1, 32, 8, 2), 24, 1.0),
], eps=1e-6)
#: no size is a multiple of eight (columns off 16-byte borders everywhere); a window of one (a row sees itself only)
SMALL_C = config(36, 50, [
    layer(parallel(attention(3, 1, 10, 6, window=1, rot_dims=6), delta_sizes(2, 2, 7, 11, 3), 0.85, 1.15), 30, 1.4),
    layer(delta(3, 1, 9, 5, 4), 20, 0.6),
    layer(mingru(21), 18, 1.0),
    layer(parallel(attention(2, 2, 6, 10, window=33, rot_dims=2, scaling=RAMP), delta_sizes(5, 5, 6, 3, 2), 1.2, 0.7)),
])
#: sizes that the tensor-core kernels of the bfloat16 path take: attention heads of 64, delta heads of 64, of 128 and of sizes
#: that are padded to those, value columns in one and in two tiles of sixteen per block
SMALL_D = config(64, 100, [
    layer(delta(2, 1, 128, 64, 4), 96, 1.0),
    layer(parallel(attention(4, 2, 64, 64, window=48, rot_dims=32, scaling=RAMP), delta_sizes(2, 2, 64, 40, 3), 0.7, 1.2), 80, 0.8),
    layer(mingru(72), 64, 2.5),
    layer(delta(3, 1, 40, 16, 3), 64, 1.3),
    layer(parallel(attention(2, 1, 64, 64, window=150), delta_sizes(1, 1, 104, 128, 2), 1.4, 0.6)),
])
#: layers over a state only: no pages at all
SMALL_E = config(32, 60, [layer(delta(6, 2, 8, 8, 2), 40, 1.0), layer(mingru(16), 24, 1.4), layer(delta(2, 1, 24, 40, 4))])
#: more query heads on one kv head than a block has warps, one layer
SMALL_F = config(56, 40, [layer(parallel(attention(34, 1, 8, 12, window=20, rot_dims=4), delta_sizes(3, 1, 16, 8, 4), 0.9, 0.8), 40, 1.0)])
#: per configuration the ranks of the decays' and the gates' thin pairs
RANKS = {48: (7, 13), 40: (8, 3), 36: (5, 1), 64: (24, 16)}


def make_tensors(doc: dict, seed: int, sharpen: float = 2.0) -> Dict[str, torch.Tensor]:
    """Weights of order one, made so that faults show: peaked attention, sinks that matter, decays from nearly none to fast, step
    sizes spread over (0, 1), gates away from one half, feed-forwards whose clamps act, thin pairs of other ranks than the
    random-weights mode gives."""
    from sglang_rs_b200.weights import build_model
    model, _ = build_model(doc)
    g = torch.Generator().manual_seed(seed)
    rank_a, rank_g = RANKS.get(doc["width"], (6, 9))
    out = {}
    for name, spec in model.tensor_specs().items():
        rank = rank_g if name.endswith((".g1", ".g2")) else rank_a
        shape = tuple(rank if size < 0 else size for size in spec.shape)
        normal = torch.randn(shape, generator=g)
        if name.endswith("A_log"):
            v = torch.rand(shape, generator=g) * 6 - 5            # rates exp(A_log) from 0.007 to 2.7
        elif name.endswith("dt_bias"):
            v = torch.rand(shape, generator=g) * 4 - 3
        elif name.endswith(".conv"):
            v = normal * 0.5
            v[:, -1] += 0.7
        elif name.endswith(".sink"):
            v = normal * 1.5
        elif name.endswith("z.b"):
            v = normal - 2.0                                      # most channels remember
        elif name.endswith("x.b"):
            v = normal * 0.5
        elif name.endswith(("q.norm", "k.norm")):
            v = (1.0 + 0.3 * normal) * (sharpen if name.endswith("q.norm") else 1.0)
        elif "norm" in name:
            v = 1.0 + 0.2 * normal
        elif name == "embed":
            v = normal
        elif name.endswith((".mlp.gate", ".mlp.up")):
            v = normal * 1.2 / shape[1] ** 0.5
        elif name.endswith((".a", ".a2", ".b", ".g", ".g2")):
            v = normal * 1.5 / shape[1] ** 0.5
        else:
            v = normal / shape[1] ** 0.5
        out[name] = v
    return out


def write_folder(folder: str, doc: dict, tensors: Dict[str, torch.Tensor], dtype: torch.dtype) -> str:
    from sglang_rs_b200.weights import write_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(doc, handle)
    write_file(os.path.join(folder, "model.safetensors"), {k: v.to(dtype) for k, v in tensors.items()})
    return folder


def make_folder(tmp_path, name: str, doc: dict, seed: int, dtype: torch.dtype, **factors) -> str:
    return write_folder(str(tmp_path / name), doc, make_tensors(doc, seed, **factors), dtype)


def load_folder(folder: str):
    from sglang_rs_b200.weights import read_model_dir
    with open(os.path.join(folder, "config.json")) as handle:
        doc = json.load(handle)
    return doc, {k: v.to(torch.float64) for k, v in read_model_dir(folder).items()}


def random_requests(doc: dict, lengths: Sequence[int], seed: int) -> Dict[str, List[int]]:
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(doc["vocab"]) for _ in range(n)] for i, n in enumerate(lengths)}


def oracle(folder: str, requests: Dict[str, List[int]]) -> Dict[str, np.ndarray]:
    doc, tensors = load_folder(folder)
    return {rid: ps.forward(doc, tensors, tokens).numpy() for rid, tokens in requests.items()}


def plain_greedy(doc, tensors, prompt, count):
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(torch.argmax(ps.forward(doc, tensors, tokens)[-1])))
    return tokens[len(prompt):]


MARK, FILL = 41, 40


def marked_folder(tmp_path, dtype: torch.dtype, kind: str, window: Optional[int] = None, wide: bool = False) -> str:
    """One layer that hangs on the one position that holds ``MARK``: only that token's embedding has an entry in channel 0, every
    embedding has the same entry in channel 1.  ``window``: head 0 of the attention looks for the mark (its key entry reads channel
    0, its query channel 1) and the mixer beside it counts nothing.  ``delta`` / ``channel``: head 0 writes the mark's value under a
    key of its own, forgets nearly nothing, and reads that key at every token.  ``mingru``: every channel takes the mark in and then
    keeps it.  ``wide``: at sizes whose prompts run in chunks on the tensor cores."""
    d, v = (64, 32) if wide else (8, 12)
    if kind == "window":
        mixer = parallel(attention(2, 1, 16, 8, window=window, rot_dims=8, scale=0.5), delta_sizes(2, 2, 8, 8, 2), 0.7, 0.0)
    elif kind == "delta":
        mixer = delta(2, 2, d, v, 3)
    elif kind == "channel":
        mixer = parallel(attention(2, 1, 16, 8, window=4), delta_sizes(2, 2, d, v, 3), 0.0, 0.8)
    else:
        mixer = mingru(40)
    doc = config(48, 60, [layer(mixer, 32, 1.0)])
    t = make_tensors(doc, seed=7)
    t["embed"][:, :2] = 0
    t["embed"][MARK, 0] = 3.0
    t["embed"][:, 1] = 1.0
    if kind == "window":
        p, dim, entry = "l0.mix.left.", 16, 15                    # an unrotated entry
        t[p + "k"] *= 0.01
        t[p + "k"][:, 0] = 0
        t[p + "k"][entry] = 0
        t[p + "k"][entry, 0] = 4.0
        t[p + "q"][:dim] = 0
        t[p + "q"][entry, 1] = 5.0
        t[p + "q.norm"][:], t[p + "k.norm"][:], t[p + "sink"][:] = 2.0, 1.0, 0.5
        t[p + "v"][:, 0] = 2.0
    elif kind in ("delta", "channel"):
        p = "l0.mix." if kind == "delta" else "l0.mix.right."
        for name, width in (("q", d), ("k", d), ("v", v)):
            t[p + name][:width] = 0                               # head 0
            t[p + name + ".conv"][:width] = 0
            t[p + name + ".conv"][:width, -1] = 1.0
        t[p + "q"][0, 1] = 3.0                                    # every token asks for entry 0
        t[p + "k"][0, 0] = 4.0                                    # the mark's key; every other token's is entry 1
        t[p + "k"][1, 1] = 1.0
        t[p + "v"][:v, 0] = torch.linspace(0.5, 2.0, v)
        t[p + "b"][0] = 0
        t[p + "A_log"][0] = -9.0
        if kind == "delta":
            t[p + "a"][0], t[p + "dt_bias"][0] = 0, 0
        else:
            t[p + "a2"][:d], t[p + "dt_bias"][:d] = 0, 0
        t[p + "norm"][:] = 1.0
        t[p + "o"][:, v:] *= 0.1
    else:
        t["l0.mix.z"][:], t["l0.mix.z.b"][:] = 0, -8.0
        t["l0.mix.z"][:, 0] = 5.0
        t["l0.mix.x"][:, 0] = torch.linspace(-3.0, 3.0, 40)
    return write_folder(str(tmp_path / f"marked_{kind}_{window}_{wide}"), doc, t, dtype)


def with_mark(doc, length, place, seed):
    tokens = [FILL if t == MARK else t for t in random_requests(doc, (length,), seed=seed)["r0"]]
    tokens[place] = MARK
    return tokens


def assert_rows_close(rows, expected, tolerance, what="", median=None):
    """Every row within ``tolerance`` (largest difference over the largest |logit| of its request).  With ``median`` the rule is on
    the set of rows: at least 97 in 100 within ``tolerance`` and the median within ``median``.  A sublayer's result is normed behind
    it and a head's result before its gate, so where either is small (a read-out that finds nothing under its key, two terms that
    cancel) the rounding of its inputs to bfloat16 is blown up with it: the plain implementation, given products rounded to bfloat16,
    strays by as much at the same positions.  A fault of a mechanism moves most rows and fails both rules."""
    errors, where = [], []
    for rid, by_pos in rows.items():
        scale = float(np.abs(expected[rid]).max())
        for pos, row in sorted(by_pos.items()):
            error = float(np.abs(row.astype(np.float64) - expected[rid][pos]).max()) / scale
            errors.append(error if np.isfinite(error) else float("inf"))
            where.append((rid, pos))
    errors = np.asarray(errors)
    worst = int(np.argmax(errors))
    over = int((errors > tolerance).sum())
    if median is None:
        assert over == 0, (what, where[worst], float(errors[worst]))
    else:
        assert over <= 0.03 * len(errors) and float(np.median(errors)) <= median, \
            (what, over, len(errors), float(np.median(errors)), where[worst], float(errors[worst]))
