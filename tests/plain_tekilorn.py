"""A plain, slow implementation of the Tekilorn design: float64, one function per mechanism, token lists in, logits out.
It shares no code with the package; the tests compare the package with it.

Notation: x is the residual stream [tokens, width]; h a sublayer's input; W matrices are [out, in] and applied as W h;
positions count from 0.  Weights come in as a dict name -> float64 array, the configuration as the nested document of
config.json.
"""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate_pairs(v, positions, rot):
    """v [tokens, heads, n]: entries (2i, 2i + 1) of the first rot.dims entries turn by p * base^(-2i / dims)."""
    if not rot or not int(rot["dims"]):
        return v
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    angle = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    out = v.copy()
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def query_temperature(positions, temp):
    """The factor on q at every position: 1 + coef ln(floor((p + 1) / every) + 1)."""
    if not temp:
        return np.ones(len(positions))
    return np.array([1.0 + temp["coef"] * math.log((int(p) + 1) // temp["every"] + 1) for p in positions])


def visible(i, j, size, keep_first):
    """Whether position i sees key j: not later, and inside the window or among the kept first tokens."""
    return j <= i and (size is None or i - j < size or j < keep_first)


def attend(q, k, v, scale, size=None, keep_first=0, softcap=None):
    """q [T, H, d], k [T, H, d], v [T, H, dv] of one sequence (keys already per query head)."""
    tokens, heads = q.shape[0], q.shape[1]
    out = np.zeros((tokens, heads, v.shape[2]))
    for i in range(tokens):
        seen = np.array([j for j in range(i + 1) if visible(i, j, size, keep_first)])
        for h in range(heads):
            s = (k[seen, h] @ q[i, h]) * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            e = np.exp(s - s.max())
            out[i, h] = (e @ v[seen, h]) / e.sum()
    return out


def differential_lambda(w, p, diff):
    return float(np.exp(np.sum(w[p + "lq1"] * w[p + "lk1"])) - np.exp(np.sum(w[p + "lq2"] * w[p + "lk2"])) + diff)


def combine_maps(a1, a2, lam, diff, eps):
    """o = a1 - lambda a2, each head's o divided by its root mean square, times 1 - diff."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, positions, w, p, m, eps):
    """The mixer 'attention': two maps per head over the same values."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, per = h.shape[0], m["heads"] // m["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, 2, d) * query_temperature(positions, m.get("q_temp"))[:, None, None, None]
    k = np.repeat((h @ w[p + "k"].T).reshape(T, G, 2, d), per, axis=1)
    v = np.repeat((h @ w[p + "v"].T).reshape(T, G, dv), per, axis=1)
    maps = [attend(q[:, :, i], k[:, :, i], v, m["scale"], softcap=m.get("softcap")) for i in range(2)]
    o = combine_maps(maps[0], maps[1], differential_lambda(w, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def windowed_attention(h, positions, w, p, m, eps):
    """The mixer 'attention_2': a window that keeps the first tokens, rotation in interleaved pairs, a gate per head."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, per = h.shape[0], m["heads"] // m["kv_heads"]
    q = rotate_pairs((h @ w[p + "q"].T).reshape(T, H, d), positions, m.get("rot"))
    k = rotate_pairs((h @ w[p + "k"].T).reshape(T, G, d), positions, m.get("rot"))
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    mask = m.get("mask") or {}
    o = attend(q, np.repeat(k, per, axis=1), np.repeat(v, per, axis=1), m["scale"], mask.get("size"), mask.get("keep_first", 0))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def clamped(h, w, p, limit):
    """W_down (g sigmoid(1.702 g) (u + 1)) with g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit)."""
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def routed(h, w, p, f):
    """Sigmoid scores, the largest chosen, each multiplying its expert's input; a shared expert behind a gate per token."""
    r, e = f["router"], f["expert"]
    s = sigmoid(h @ w[p + "router"].T)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for i in sorted(range(r["experts"]), key=lambda i: (-s[t, i], i))[:r["top"]]:
            out[t] += clamped(s[t, i] * h[t:t + 1], w, f"{p}e{i}.", e["limit"])[0]
    if f.get("shared"):
        out += sigmoid(h @ w[p + "shared.sg"].T) * clamped(h, w, p + "shared.", f["shared"]["limit"])
    return out


def layer_runs(cfg):
    """The order in which layers run: (layer, number of the pass it opens or None)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, collect=None):
    """Logits [tokens, vocab] of one sequence fed whole; ``collect`` (a list) receives the stream after each layer run."""
    eps = cfg["norm"]["eps"]
    positions = np.arange(len(tokens))
    x = w["embed"][np.asarray(tokens)].copy()
    for index, opened in layer_runs(cfg):
        spec, p = cfg["layers"][index], f"l{index}."
        if opened is not None:
            x = x + w["loop.step"][opened]
        mixer = differential_attention if spec["type"] == "attention" else windowed_attention
        x = x + mixer(norm(x, w[p + "norm1"], eps), positions, w, p + "mix.", spec["mixer"], eps)
        f = spec.get("mlp")
        if f:
            h = norm(x, w[p + "norm2"], eps)
            x = x + (clamped(h, w, p + "mlp.", f["limit"]) if f["kind"] == "dense" else routed(h, w, p + "mlp.", f))
        if collect is not None:
            collect.append(x.copy())
    return norm(x, w["final.norm"], eps) @ w["head"].T
