"""Plain implementation of the Nipizen design: NumPy, float64, whole sequences, no cache, one function per mechanism,
loops over tokens and heads.  Shares nothing with the library; slow on purpose.

Notation: n tokens, D width, H heads, G key/value heads, d head width, e value width.  A weight W [out, in] is applied
as W x.  `W` of a mixer is a dictionary of its tensors by the part of the name behind '<layer>.mix.' (or behind
'<layer>.mix.left.' and '<layer>.mix.right.')."""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return -(np.maximum(-z, 0.0) + np.log1p(np.exp(-np.abs(z))))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rotation(rot):
    """-> (frequencies of the pairs, factor on cosines and sines) of {base, dims, scaling {factor, original, fast, slow}}."""
    n, base = rot["dims"], rot["base"]
    freq = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    s = rot.get("scaling")
    if not s:
        return freq, 1.0

    def turns(t):              # the (fractional) pair whose angle goes round t times in the original length
        return n * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), n - 1)
    out = np.empty_like(freq)
    for i in range(n // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = freq[i] / s["factor"] * ramp + freq[i] * (1.0 - ramp)
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, freq, amp):
    """x [n, heads, d]: pairs (i, i + half) of the first 2 * half entries turn by position * freq[i]."""
    y = x.copy()
    half = len(freq)
    for p in range(x.shape[0]):
        c, s = np.cos(p * freq) * amp, np.sin(p * freq) * amp
        u, v = x[p, :, :half], x[p, :, half:2 * half]
        y[p, :, :half], y[p, :, half:2 * half] = u * c - v * s, v * c + u * s
    return y


def attention(h, W, m, eps):
    n = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ W["q"].T + W["q.b"], eps) * W["q.norm"]
    k = rms(h @ W["k"].T + W["k.b"], eps) * W["k.norm"]
    v = (h @ W["v"].T + W["v.b"]).reshape(n, G, e)
    q, k = q.reshape(n, H, d), k.reshape(n, G, d)
    if m.get("rot"):
        freq, amp = rotation(m["rot"])
        q, k = rotate(q, freq, amp), rotate(k, freq, amp)
    out = np.zeros((n, H, e))
    for i in range(n):
        for a in range(H):
            g = a // (H // G)
            sc = (k[:i + 1, g] @ q[i, a]) * m["scale"]
            w = np.exp(sc - sc.max())
            out[i, a] = (w / w.sum()) @ v[:i + 1, g]
    return (out.reshape(n, H * e) * sigmoid(h @ W["g"].T)) @ W["o"].T


def short_conv_silu(x, w):
    """Causal convolution per channel (the last tap belongs to the current token, zeros before the start), then silu."""
    n, taps = x.shape[0], w.shape[1]
    y = np.zeros((n, x.shape[1]))
    for t in range(n):
        for j in range(taps):
            if t - (taps - 1) + j >= 0:
                y[t] += w[:, j] * x[t - (taps - 1) + j]
    return y * sigmoid(y)


def delta_scan(q, k, v, g, beta):
    """q, k [n, G, d]; v [n, H, e]; g [n, H, d] decays; beta [n, H] -> o [n, H, e]: decay, write what the key does not yet
    read, read."""
    n, H, e = v.shape
    G, d = q.shape[1:]
    o = np.zeros((n, H, e))
    for a in range(H):
        s = a // (H // G)
        S = np.zeros((d, e))
        for t in range(n):
            S = g[t, a][:, None] * S
            u = beta[t, a] * (v[t, a] - S.T @ k[t, s])
            S = S + np.outer(k[t, s], u)
            o[t, a] = S.T @ q[t, s]
    return o


def delta_mixer(h, W, m, eps):
    n = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv_silu(h @ W["q"].T, W["q.conv"]).reshape(n, G, d)
    k = short_conv_silu(h @ W["k"].T, W["k.conv"]).reshape(n, G, d)
    v = short_conv_silu(h @ W["v"].T, W["v.conv"]).reshape(n, H, e)
    q = q / np.sqrt(np.sum(q * q, axis=-1, keepdims=True) + 1e-6) * d ** -0.5
    k = k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)
    rate = softplus((h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]).reshape(n, H, d)
    g = np.exp(-np.exp(W["A_log"])[None, :, None] * rate)
    o = delta_scan(q, k, v, g, sigmoid(h @ W["b"].T))
    gate = sigmoid((h @ W["g1"].T) @ W["g2"].T).reshape(n, H, e)
    return (rms(o, eps) * W["norm"] * gate).reshape(n, H * e) @ W["o"].T


def pair(h, W, m, eps):
    def side(name):
        return {t[len(name) + 1:]: w for t, w in W.items() if t.startswith(name + ".")}

    return (m["left_scale"] * attention(h, side("left"), m["left"], eps)
            + m["right_scale"] * delta_mixer(h, side("right"), m["right"], eps))


def mlstm_scan(q, k, v, i, f):
    """q, k [n, H, d]; v [n, H, e]; i, f [n, H] logarithms of the gates -> o [n, H, e]."""
    n, H, e = v.shape
    o = np.zeros((n, H, e))
    for a in range(H):
        S, z, m = np.zeros((q.shape[2], e)), np.zeros(q.shape[2]), 0.0
        for t in range(n):
            before, m = m, max(f[t, a] + m, i[t, a])
            keep, write = math.exp(f[t, a] + before - m), math.exp(i[t, a] - m)
            S = keep * S + write * np.outer(k[t, a], v[t, a])
            z = keep * z + write * k[t, a]
            o[t, a] = S.T @ q[t, a] / (max(abs(z @ q[t, a]), math.exp(-m)) + 1e-6)
    return o


def mlstm(h, W, m, eps):
    n = h.shape[0]
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W["q"].T).reshape(n, H, d) * d ** -0.5
    k = (h @ W["k"].T).reshape(n, H, d)
    v = (h @ W["v"].T).reshape(n, H, e)
    i = cap * np.tanh((h @ W["i"].T + W["i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((h @ W["f"].T + W["f.b"]) / cap))
    o = rms(mlstm_scan(q, k, v, i, f), eps).reshape(n, H * e) * W["norm"]
    return (o * sigmoid(h @ W["g"].T)) @ W["o"].T


def expert(x, W, e):
    return np.maximum(W[f"e{e}.up"] @ x, 0.0) ** 2 @ W[f"e{e}.down"].T


def moe(h, W, router, margins=None):
    """Sigmoid scores, the `top` largest, not renormalised; the weight multiplies what the expert reads.  `margins`: per
    token the smallest gap (in score) between a chosen and a left-out expert seen so far."""
    E, top = router["experts"], router["top"]
    s = sigmoid(h @ W["router"].T)
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(E), key=lambda e: (-s[t, e], e))
        for e in order[:top]:
            y[t] += expert(s[t, e] * h[t], W, e)
        if margins is not None and top < E:
            margins[t] = min(margins[t], s[t, order[top - 1]] - s[t, order[top]])
    return y


def forward(cfg, W, tokens, margins=None, residuals=None):
    """float64 logits [n, vocab] of a whole sequence; `residuals`: a list that gets the rows after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    for i, L in enumerate(cfg["layers"]):
        mix = {n[len(f"l{i}.mix."):]: w for n, w in W.items() if n.startswith(f"l{i}.mix.")}
        h = layer_norm(x, W[f"l{i}.norm1"], eps)
        x = x + (pair if L["type"] == "parallel" else mlstm)(h, mix, L["mixer"], eps)
        if L.get("mlp") is not None:
            ff = {n[len(f"l{i}.mlp."):]: w for n, w in W.items() if n.startswith(f"l{i}.mlp.")}
            x = x + moe(layer_norm(x, W[f"l{i}.norm2"], eps), ff, L["mlp"]["router"], margins)
        if residuals is not None:
            residuals.append(x.copy())
    return layer_norm(x, W["final.norm"], eps) @ W["embed"].T
