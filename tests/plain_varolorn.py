"""Plain implementation of the Varolorn design: NumPy, float64, whole sequences, no cache, one function per mechanism,
loops over tokens and heads.  Shares nothing with the library; slow on purpose.

Notation: n tokens, D width, s streams, H heads, G key/value heads (attention) or groups (recurrence), d head width,
e value width, N state channels.  A weight W [out, in] is applied as W x.  `W` of a mixer is a dictionary of its tensors
by the part of the name behind '<layer>.mix.'."""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def embed_rows(tokens, table, scale, bigram=None):
    """Token rows times `scale`; with bigram = (table [buckets + 1, D], buckets, mul_prev, mul_cur) the row of the pair
    (token before, token) is added, the last row for the first token."""
    x = table[np.asarray(tokens)] * scale
    if bigram is not None:
        rows, buckets, mul_prev, mul_cur = bigram
        for t, tok in enumerate(tokens):
            x[t] += rows[buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tok) * mul_cur) % buckets]
    return x


def distance_bucket(n, rows, most):
    """Which of `rows` table rows the distance n falls into: one row per distance below rows/2, then rows whose edges
    grow geometrically up to the distance `most`, and the last row from there on."""
    half = rows // 2
    if n < half:
        return n
    k = 0                                     # the largest k with (n / half) >= (most / half)^(k / (rows - half))
    while k < rows and n ** (rows - half) * half ** k >= most ** k * half ** (rows - half):
        k += 1
    return min(rows - 1, half + k - 1)


def visible(i, j, size):
    """Whether position i sees position j: not later, and (size > 0) in the same stretch of `size` positions."""
    return j <= i and (size <= 0 or i // size == j // size)


def attention(h, W, m, eps, v_first=None):
    """-> (output rows, the values before any mixing).  Per-head normed queries and keys, scores scaled and then moved by
    a number per (distance bucket, head), chunks, softmax, a gate per head.  With v_first the values are
    (1 - vmix) v + vmix v_first."""
    n = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    size = (m.get("mask") or {}).get("size", 0)
    q = rms((h @ W["q"].T + W["q.b"]).reshape(n, H, d), eps) * W["q.norm"]
    k = rms((h @ W["k"].T + W["k.b"]).reshape(n, G, d), eps) * W["k.norm"]
    v = own = (h @ W["v"].T + W["v.b"]).reshape(n, G, e)
    if v_first is not None:
        lam = float(W["vmix"])
        v = (1.0 - lam) * own + lam * v_first
    rows = W["rel"].shape[0]
    bucket = [distance_bucket(t, rows, m["bias_max"]) for t in range(n)]
    gate = sigmoid(h @ W["g"].T)
    out = np.zeros((n, H, e))
    for i in range(n):
        js = [j for j in range(i + 1) if visible(i, j, size)]
        far = np.array([bucket[i - j] for j in js])
        for a in range(H):
            g = a // (H // G)
            sc = (k[js, g] @ q[i, a]) * m["scale"] + W["rel"][far, a]
            w = np.exp(sc - sc.max())
            out[i, a] = (w / w.sum()) @ v[js, g] * gate[i, a]
    return out.reshape(n, H * e) @ W["o"].T + W["o.b"], own


def short_conv(x, w, b):
    """Causal convolution per channel: the last tap belongs to the current token, zeros before the start."""
    n, taps = x.shape[0], w.shape[1]
    y = np.tile(b, (n, 1)).astype(np.float64)
    for t in range(n):
        for j in range(taps):
            if t - (taps - 1) + j >= 0:
                y[t] += w[:, j] * x[t - (taps - 1) + j]
    return y


def ssd_scan(x, B, C, dt, A_log, D):
    """x [n, H, e], B and C [n, G, N], dt [n, H] (already positive) -> y [n, H, e]."""
    n, H, e = x.shape
    G, N = B.shape[1:]
    y = np.zeros((n, H, e))
    for a in range(H):
        g = a // (H // G)
        S = np.zeros((N, e))
        for t in range(n):
            S = math.exp(-math.exp(A_log[a]) * dt[t, a]) * S + dt[t, a] * np.outer(B[t, g], x[t, a])
            y[t, a] = C[t, g] @ S + D[a] * x[t, a]
    return y


def gated_group_norm(y, z, w, parts, eps):
    """(y * silu(z)), every one of `parts` equal stretches divided by its own root mean square, times w."""
    u = y * silu(z)
    return rms(u.reshape(u.shape[0], parts, -1), eps).reshape(u.shape) * w


def mamba2(h, W, m, eps):
    n = h.shape[0]
    H, e, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    p = h @ W["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, W["conv"], W["conv.b"]))
    x = xbc[:, :inner].reshape(n, H, e)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)
    C = xbc[:, inner + G * N:].reshape(n, G, N)
    y = ssd_scan(x, B, C, softplus(dt + W["dt_bias"]), W["A_log"], W["D"])
    return gated_group_norm(y.reshape(n, inner), z, W["norm"], m["norm_groups"], eps) @ W["o"].T


def gated_relu(h, gate, up, down):
    return (np.maximum(h @ gate.T, 0.0) * (h @ up.T)) @ down.T


def plus_one_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def stream_read(X, a):
    """X [s, n, D] -> sum_s a[s] X_s."""
    return np.einsum("s,snd->nd", a, X)


def stream_write(X, mix, out, y):
    """X_t <- sum_s mix[s, t] X_s + out[t] y."""
    return np.einsum("st,snd->tnd", mix, X) + out[:, None, None] * y


def sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, W, tokens, taps=None):
    """Logits [n, vocab].  taps: a list that receives the rows after every layer (the sum of the streams)."""
    eps, bg = cfg["norm"]["eps"], (cfg.get("embedding") or {}).get("bigram")
    scale = (cfg.get("embedding") or {}).get("scale", 1.0)
    e = embed_rows(tokens, W["embed"], scale,
                   (W["bigram"], bg["buckets"], bg["mul_prev"], bg["mul_cur"]) if bg else None)
    s = cfg.get("streams")
    X = np.stack([e] * (s or 1))
    v_first = None

    def sublayer(X, p, q, f):
        if s:
            y = f(plus_one_norm(stream_read(X, W[f"{p}hc{q}.in"]), W[f"{p}norm{q}"], eps))
            return stream_write(X, W[f"{p}hc{q}.mix"], W[f"{p}hc{q}.out"], y)
        return X + f(plus_one_norm(X[0], W[f"{p}norm{q}"], eps))

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mw = sub(W, p + "mix.")

        def mixer(h):
            nonlocal v_first
            if L["type"] == "mamba2":
                return mamba2(h, mw, m, eps)
            y, own = attention(h, mw, m, eps, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = own
            return y

        X = sublayer(X, p, 1, mixer)
        if L["mlp"] is not None:
            X = sublayer(X, p, 2, lambda h: gated_relu(h, W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"]))
        if taps is not None:
            taps.append(X.sum(0))
    return plus_one_norm(X.sum(0), W["final.norm"], eps) @ W["embed"].T
