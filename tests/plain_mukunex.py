"""A plain, slow implementation of the Mukunex design: numpy, one function a mechanism, whole
sequences at once (no cache, no batch), in the precision of the arrays it is given (tests pass
float64). It shares nothing with the package: the tests compare the engine with it.

A model is (config, tensors): config.json's dict and {name: array}. Notation: T tokens, W the
model's width, H heads, G key/value heads, d the query/key size of a head, e its value size.
"""
from __future__ import annotations

import math

import numpy as np


# ---------------------------------------------------------------------------------------- small pieces
def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def short_conv(x, w):
    """x [T, C], w [C, taps]: y[t] = sum_j w[:, j] x[t - taps + 1 + j], zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += x[: T - back] * w[:, j]
    return y


def frequencies(rot):
    """Turning rates of the pairs. With `scaling`, by wavelength: short waves keep their rate, long ones
    turn `factor` times slower, those between blend the two."""
    dims = int(rot["dims"])
    f = np.array([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if sc is None:
        return f
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = np.empty_like(f)
    for i, rate in enumerate(f):
        wave = 2.0 * math.pi / rate
        if wave < original / high:
            out[i] = rate
        elif wave > original / low:
            out[i] = rate / factor
        else:
            s = (original / wave - low) / (high - low)
            out[i] = (1.0 - s) * rate / factor + s * rate
    return out


def rotate_halves(x, positions, rot):
    """x [T, n, d]: the first rot["dims"] components of every vector are turned, i with i + dims/2, by
    the angle position * rate_i; the rest pass."""
    half = int(rot["dims"]) // 2
    a = np.asarray(positions, dtype=np.float64)[:, None] * frequencies(rot)[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half:]], axis=-1)


def causal_softmax(scores, sink):
    """scores [T, T]: weights of row i over the columns j <= i; e^sink joins the denominator."""
    out = np.zeros_like(scores)
    for i in range(scores.shape[0]):
        row = scores[i, : i + 1]
        top = max(row.max(), sink)
        p = np.exp(row - top)
        out[i, : i + 1] = p / (p.sum() + math.exp(sink - top))
    return out


# ---------------------------------------------------------------------------------------- mixers
def sink_attention(h, t, p, m):
    """Grouped queries, partly rotated, a sink in the denominator, one gate a head."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = np.arange(T)
    q = rotate_halves((h @ t[f"{p}.q"].T).reshape(T, H, d), pos, m["rot"])
    k = rotate_halves((h @ t[f"{p}.k"].T).reshape(T, G, d), pos, m["rot"])
    v = (h @ t[f"{p}.v"].T).reshape(T, G, e)
    gate = sigmoid(h @ t[f"{p}.g"].T)
    out = np.zeros((T, H, e), dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        w = causal_softmax((q[:, a] @ k[:, g].T) * m["scale"], float(t[f"{p}.sink"][a]))
        out[:, a] = (w @ v[:, g]) * gate[:, a, None]
    return out.reshape(T, H * e) @ t[f"{p}.o"].T


def retention_recurrence(q, k, v, decay):
    """One head. q, k [T, d], v [T, e]: S <- decay S + k v^T; o = S^T q."""
    S = np.zeros((k.shape[1], v.shape[1]), dtype=v.dtype)
    out = np.zeros_like(v)
    for i in range(k.shape[0]):
        S = decay * S + np.outer(k[i], v[i])
        out[i] = S.T @ q[i]
    return out


def retention(h, t, p, m, eps):
    H, d, e = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = np.arange(T)
    q = rotate_halves((h @ t[f"{p}.q"].T).reshape(T, H, d), pos, m["rot"])
    k = rotate_halves((h @ t[f"{p}.k"].T).reshape(T, H, d), pos, m["rot"]) * d ** -0.5
    v = (h @ t[f"{p}.v"].T).reshape(T, H, e)
    o = np.stack([retention_recurrence(q[:, i], k[:, i], v[:, i], float(m["decay"][i])) for i in range(H)], axis=1)
    return (rms_unit(o, eps).reshape(T, H * e) * silu(h @ t[f"{p}.g"].T)) @ t[f"{p}.o"].T


def parallel_mixer(h, t, p, m, eps):
    return m["left_scale"] * sink_attention(h, t, f"{p}.left", m["left"]) + m["right_scale"] * retention(h, t, f"{p}.right", m["right"], eps)


def lru_gates(u, ra, ra_b, ri, ri_b):
    """u [T, W] in equal parts, one square matrix a part: the recurrence gate and the input gate."""
    T, B = u.shape[0], ra.shape[0]
    parts = u.reshape(T, B, -1)
    r = sigmoid(np.einsum("boi,tbi->tbo", ra, parts) + ra_b)
    i = sigmoid(np.einsum("boi,tbi->tbo", ri, parts) + ri_b)
    return r.reshape(T, -1), i.reshape(T, -1)


def lru_recurrence(u, r, i, lam):
    """S <- a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), channel by channel, from zero."""
    a = np.exp(-8.0 * r * softplus(lam))
    push = np.sqrt(-np.expm1(2.0 * np.log(a))) * i * u
    S = np.zeros_like(u[0])
    out = np.zeros_like(u)
    for n in range(u.shape[0]):
        S = a[n] * S + push[n]
        out[n] = S
    return out


def rglru_mixer(h, t, p, m, eps):
    y = gelu_tanh(h @ t[f"{p}.y"].T + t[f"{p}.y.b"])
    u = short_conv(h @ t[f"{p}.x"].T + t[f"{p}.x.b"], t[f"{p}.conv"]) + t[f"{p}.conv.b"]
    r, i = lru_gates(u, t[f"{p}.ra"], t[f"{p}.ra.b"], t[f"{p}.ri"], t[f"{p}.ri.b"])
    return (lru_recurrence(u, r, i, t[f"{p}.lam"]) * y) @ t[f"{p}.o"].T


def channel_delta_recurrence(q, k, v, g, beta):
    """One head. q, k, g [T, d], v [T, e], beta [T]: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    S = np.zeros((k.shape[1], v.shape[1]), dtype=v.dtype)
    out = np.zeros_like(v)
    for i in range(k.shape[0]):
        S = g[i][:, None] * S
        u = beta[i] * (v[i] - S.T @ k[i])
        S = S + np.outer(k[i], u)
        out[i] = S.T @ q[i]
    return out


def unit_vectors(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def channel_delta_mixer(h, t, p, m, eps):
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    run = lambda n: silu(short_conv(h @ t[f"{p}.{n}"].T, t[f"{p}.{n}.conv"]))
    q = unit_vectors(run("q").reshape(T, G, d)) * d ** -0.5
    k = unit_vectors(run("k").reshape(T, G, d))
    v = run("v").reshape(T, H, e)
    beta = sigmoid(h @ t[f"{p}.b"].T)
    z = (h @ t[f"{p}.a1"].T) @ t[f"{p}.a2"].T + t[f"{p}.dt_bias"]
    g = np.exp(-np.exp(t[f"{p}.A_log"])[None, :, None] * softplus(z).reshape(T, H, d))
    per = H // G
    o = np.stack([channel_delta_recurrence(q[:, i // per], k[:, i // per], v[:, i], g[:, i], beta[:, i]) for i in range(H)], axis=1)
    o = rms_unit(o, eps) * t[f"{p}.norm"]
    gate = sigmoid((h @ t[f"{p}.g1"].T) @ t[f"{p}.g2"].T)
    return (o.reshape(T, H * e) * gate) @ t[f"{p}.o"].T


MIXERS = {"parallel": parallel_mixer, "rglru": rglru_mixer, "channel_delta": channel_delta_mixer}


# ---------------------------------------------------------------------------------------- the model
def feed_forward(h, t, p):
    return (gelu_tanh(h @ t[f"{p}.gate"].T) * (h @ t[f"{p}.up"].T)) @ t[f"{p}.down"].T


def forward(config, t, tokens, residuals=None):
    """Logits [T, vocab] of a whole sequence; `residuals`, a list, receives the stream after every layer."""
    eps = float(config["norm"]["eps"])
    x = t["embed"][np.asarray(tokens)]
    for i, rec in enumerate(config["layers"]):
        p = f"l{i}"
        x = x + MIXERS[rec["type"]](rms_unit(x, eps) * t[f"{p}.norm1"], t, f"{p}.mix", rec["mixer"], eps)
        if rec.get("mlp") is not None:
            x = x + feed_forward(rms_unit(x, eps) * t[f"{p}.norm2"], t, f"{p}.mlp")
        if residuals is not None:
            residuals.append(x)
    return (rms_unit(x, eps) * t["final.norm"]) @ t["head"].T
