"""A plain, slow implementation of the Sogodra design in float64, one function per mechanism.

It shares no code with the package: tensors come in as a dict of name -> torch tensor, the configuration as the plain
document, and every function walks tokens and heads in Python loops where that is the clearest form.  A whole sequence
is computed at once (no cache, no portions); the package must give the same logits however the sequence is cut.
"""
from __future__ import annotations

import math

import torch

F = torch.float64
UNIT_EPS = 1e-6


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    # log(1 + exp(z)) without overflow
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def causal_conv(u, weight):
    """u [T, channels]; weight [channels, taps] whose last column multiplies the current token; zeros before the start."""
    T = u.shape[0]
    taps = weight.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] = out[t] + weight[:, j] * u[s]
    return out


def frequencies(rot):
    """The turning rate of every pair: base^(-2i/dims), and with ``scaling`` long wavelengths stretched by ``factor``:
    those above original / low wholly, those below original / high not at all, a straight ramp between."""
    dims, base = rot["dims"], float(rot["base"])
    rates = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        s = rot.get("scaling")
        if s is not None:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                ramp = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - ramp) * f / s["factor"] + ramp * f
        rates.append(f)
    return torch.tensor(rates, dtype=F)


def rotate(x, position, rot):
    """The leading rot.dims entries of x [heads, dim] turned by the position's angles, entry i with entry i + dims/2."""
    half = rot["dims"] // 2
    angle = position * frequencies(rot)
    out = x.clone()
    u, v = x[:, :half], x[:, half:2 * half]
    out[:, :half] = u * torch.cos(angle) - v * torch.sin(angle)
    out[:, half:2 * half] = v * torch.cos(angle) + u * torch.sin(angle)
    return out


def windowed_attention(h, w, m, eps):
    """Softmax attention with grouped heads, a norm per q and k head, a rotation, a window and a learned sink per head."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rms((h @ w["q"].T).reshape(T, H, D), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).reshape(T, G, D), eps) * w["k.norm"]
    v = (h @ w["v"].T).reshape(T, G, V)
    if m.get("rot") is not None:
        q = torch.stack([rotate(q[t], t, m["rot"]) for t in range(T)])
        k = torch.stack([rotate(k[t], t, m["rot"]) for t in range(T)])
    window = m["mask"]["size"] if m.get("mask") else None
    out = torch.zeros(T, H, V, dtype=F)
    for i in range(T):
        first = 0 if window is None else max(0, i - window + 1)
        for head in range(H):
            g = head // (H // G)
            scores = (k[first:i + 1, g] @ q[i, head]) * m["scale"]
            top = torch.maximum(scores.max(), w["sink"][head])
            e = torch.exp(scores - top)
            out[i, head] = (e / (e.sum() + torch.exp(w["sink"][head] - top))) @ v[first:i + 1, g]
    return out.reshape(T, H * V) @ w["o"].T


def delta_recurrence(q, k, v, beta, decay, begin=None):
    """q, k [T, heads, D] (already unit vectors, q scaled), v [T, heads, V], beta [T, heads], decay [T, heads, D]:
    per head S <- decay S (row by row), u = beta (v - S^T k), S <- S + k u^T, o = S^T q, from the states ``begin``
    [heads, D, V] (zeros without).  Returns (o [T, heads, V], the last states)."""
    T, heads, D = q.shape
    V = v.shape[2]
    o = torch.zeros(T, heads, V, dtype=F)
    last = torch.zeros(heads, D, V, dtype=F)
    for head in range(heads):
        S = torch.zeros(D, V, dtype=F) if begin is None else begin[head].clone()
        for t in range(T):
            S = decay[t, head][:, None] * S
            u = beta[t, head] * (v[t, head] - S.T @ k[t, head])
            S = S + torch.outer(k[t, head], u)
            o[t, head] = S.T @ q[t, head]
        last[head] = S
    return o, last


def head_decay(h, w, T, H, D):
    """One decay per head and token, the same for all rows of the state."""
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    return g[:, :, None].expand(T, H, D)


def channel_decay(h, w, T, H, D):
    """One decay per head, token and row of the state, through a product of two thin matrices."""
    z = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).reshape(T, H, D)
    return torch.exp(-torch.exp(w["A_log"])[None, :, None] * z)


def gated_delta(h, w, m, eps, channels):
    """The gated delta rule with a decay per head and a SiLU gate, or (``channels``) a decay per head and row of the
    state and a sigmoid gate through thin matrices."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    def conv(name, heads, dim):
        return silu(causal_conv(h @ w[name].T, w[name + ".conv"])).reshape(T, heads, dim)
    per = H // G
    q = unit(conv("q", G, D)).repeat_interleave(per, dim=1) * D ** -0.5
    k = unit(conv("k", G, D)).repeat_interleave(per, dim=1)
    v = conv("v", H, V)
    beta = torch.sigmoid(h @ w["b"].T)
    decay = (channel_decay if channels else head_decay)(h, w, T, H, D)
    o, _ = delta_recurrence(q, k, v, beta, decay)
    gate = torch.sigmoid((h @ w["g1"].T) @ w["g2"].T) if channels else silu(h @ w["g"].T)
    y = (rms(o, eps) * w["norm"]).reshape(T, H * V) * gate
    return y @ w["o"].T


def min_gru(h, w):
    z = torch.sigmoid(h @ w["z"].T + w["z.b"])
    u = h @ w["x"].T + w["x.b"]
    candidate = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros(z.shape[1], dtype=F)
    states = []
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * candidate[t]
        states.append(S)
    return (torch.stack(states) * silu(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, m, eps):
    def part(name):
        return {key[len(name) + 1:]: value for key, value in w.items() if key.startswith(name + ".")}
    left = windowed_attention(h, part("left"), m["left"], eps)
    right = gated_delta(h, part("right"), m["right"], eps, channels=True)
    return m["left_scale"] * left + m["right_scale"] * right


def feed_forward(h, w, f):
    limit = f["limit"]
    g = torch.clamp(h @ w["gate"].T, max=limit)
    u = torch.clamp(h @ w["up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def mix(kind, h, w, m, eps):
    if kind == "parallel":
        return parallel(h, w, m, eps)
    if kind == "mingru":
        return min_gru(h, w)
    if kind == "delta":
        return gated_delta(h, w, m, eps, channels=False)
    raise ValueError(kind)


def short_names(tensors, prefix):
    return {name[len(prefix):]: value.to(F) for name, value in tensors.items() if name.startswith(prefix)}


def forward(config, tensors, tokens, return_layers=False):
    """Logits [T, vocab] of a whole sequence; with ``return_layers`` also the stream after every layer."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = tensors["embed"].to(F)[tokens]
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = mix(layer["type"], x, short_names(tensors, p + "mix."), layer["mixer"], eps)
        x = x + rms(y, eps) * tensors[p + "norm1"].to(F)
        if layer.get("mlp") is not None:
            y = feed_forward(x, short_names(tensors, p + "mlp."), layer["mlp"])
            x = x + rms(y, eps) * tensors[p + "norm2"].to(F)
        after.append(x)
    logits = rms(x, eps) * tensors["final.norm"].to(F) @ tensors["head"].to(F).T
    return (logits, torch.stack(after)) if return_layers else logits
