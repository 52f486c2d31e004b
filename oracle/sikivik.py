"""A plain, slow Sikivik in numpy float64: one function per mechanism, token by token where the mechanism is a recurrence.

Used by tests only; shares nothing with the product path.  Weights are a dict name -> array (any float dtype); `cfg` is the
model's config.json as a dict.
"""
from __future__ import annotations

import numpy as np

F = np.float64


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x over the last axis, divided by its root mean square (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def causal_conv(x, taps):
    """Per channel: y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c], zeros before the start."""
    n = taps.shape[1]
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def rotate_half(x, dims, base, start=0):
    """x [T, heads, D]: at position p = start + t, dimension i < dims / 2 and its partner i + dims / 2 turn by the angle
    p * base^(-2 i / dims); the dimensions from `dims` on stay as they are."""
    half = dims // 2
    out = x.copy()
    for t in range(x.shape[0]):
        for i in range(half):
            a = (start + t) * base ** (-2.0 * i / dims)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * np.cos(a) - v * np.sin(a)
            out[t, :, i + half] = v * np.cos(a) + u * np.sin(a)
    return out


def decayed_write(q, k, v, g):
    """q, k, g [T, H, D], v [T, H, V].  Per head S [D, V]: S <- diag(g) S + k v^T; o = S^T q, the current token's write included."""
    T, H, D = q.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        S = np.zeros((D, v.shape[2]), F)
        for t in range(T):
            S = g[t, h][:, None] * S + np.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def channel_decay(z, tau):
    """sigmoid(z)^(1 / tau), through the logarithm so that it neither over- nor underflows."""
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def window_attention(q, k, v, scale, size):
    """q [T, H, D], k [T, G, D], v [T, G, V]: softmax over the positions i - size < j <= i, G key heads shared by consecutive
    query heads."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        kh, vh = k[:, h // (H // G)], v[:, h // (H // G)]
        for i in range(T):
            lo = max(0, i - size + 1)
            s = kh[lo:i + 1] @ q[i, h] * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ vh[lo:i + 1]
    return out


def mix_values(v, first, share):
    return (1.0 - share) * v + share * first


def gla(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ w["k"].T).reshape(T, H, D)
    v = (h @ w["v"].T).reshape(T, H, V)
    alpha = channel_decay(h @ w["a1"].T @ w["a2"].T + w["a2.b"], m["tau"]).reshape(T, H, D)
    o = rms(decayed_write(q, k, v, alpha), eps) * w["norm"]
    return (o.reshape(T, H * V) * silu(h @ w["g"].T)) @ w["o"].T


def retention(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    turn = lambda x: rotate_half(x.reshape(T, H, D), m["rot"]["dims"], m["rot"]["base"])
    q, k = turn(h @ w["q"].T), turn(h @ w["k"].T) * D ** -0.5
    v = (h @ w["v"].T).reshape(T, H, V)
    decay = np.broadcast_to(np.asarray(m["decay"], F)[None, :, None], (T, H, D))
    o = rms(decayed_write(q, k, v, decay), eps)
    return (o.reshape(T, H * V) * silu(h @ w["g"].T)) @ w["o"].T


def attention(h, w, m, first):
    """(the mixer's output, its values [T, G, V] as cached); `first`: the values of the first layer that shares them, or None."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ w[n].T + w[n + ".b"], w[n + ".conv"]) for n in "qkv")
    turn = lambda x, heads: rotate_half(x.reshape(T, heads, D), m["rot"]["dims"], m["rot"]["base"])
    q, k, v = turn(q, H), turn(k, G), v.reshape(T, G, V)
    if first is not None:
        v = mix_values(v, first, w["vmix"])
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"])
    return (o.reshape(T, H * V) * sigmoid(h @ w["g"].T)) @ w["o"].T + w["o.b"], v


def feed_forward(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def forward(cfg, weights, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) in float64."""
    w = {n: np.asarray(t, F) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    after, first = [], None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mix = {n[len(p) + 4:]: t for n, t in w.items() if n.startswith(p + "mix.")}
        h = rms(x, eps) * w[p + "norm1"]
        if layer["type"] == "attention":
            shares = bool(m.get("v_mix"))
            y, values = attention(h, mix, m, first if shares else None)
            if shares and first is None:
                first = values
        else:
            y = {"gla": gla, "retention": retention}[layer["type"]](h, mix, m, eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
        x = x + y
        after.append(x)
    return rms(x, eps) * w["final.norm"] @ w["head"].T, np.stack(after)
