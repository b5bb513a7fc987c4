"""A plain, slow implementation of the Sopalorn design: numpy, one function a mechanism, whole
sequences at once (no cache, no batch), in the precision of the arrays it is given (tests pass
float64). It shares nothing with the package: the tests compare the engine with it.

A model is (config, tensors): config.json's dict and {name: array}. Notation: T tokens, W the
model's width, H heads, G key/value heads, d the query/key size of a head, e its value size, S streams.
"""
from __future__ import annotations

import math

import numpy as np


# ---------------------------------------------------------------------------------------- small pieces
def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def short_conv(x, w):
    """x [T, C], w [C, taps]: y[t] = sum_j w[:, j] x[t - taps + 1 + j], zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += x[: T - back] * w[:, j]
    return y


def unit_vectors(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def frequencies(rot):
    """(turning rates of the pairs, the factor on cos and sin). With `scaling`, pairs that turn often over
    `original` positions keep their rate, pairs that turn seldom are slowed `factor` times, the ones between blend."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])
    pair = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair(float(sc["fast"]))), 0), min(math.ceil(pair(float(sc["slow"]))), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, positions, rot):
    """x [T, n, d]: of the first rot["dims"] components 2i turns with 2i + 1 by the angle position * rate_i; the rest pass."""
    dims = int(rot["dims"])
    f, magnitude = frequencies(rot)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = magnitude * np.cos(a)[:, None, :], magnitude * np.sin(a)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = np.array(x)
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def masked_softmax(scores, window, sink):
    """scores [T, T]: weights of row i over the columns j <= i (with a window: i - j < window); e^sink joins the denominator."""
    out = np.zeros_like(scores)
    for i in range(scores.shape[0]):
        first = max(0, i - window + 1) if window else 0
        row = scores[i, first : i + 1]
        top = max(row.max(), sink)
        p = np.exp(row - top)
        out[i, first : i + 1] = p / (p.sum() + math.exp(sink - top))
    return out


def attend(q, k, v, scale, window, sinks):
    """q [T, H, d], k [T, G, d], v [T, G, e]: [T, H e]."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        out[:, h] = masked_softmax((q[:, h] @ k[:, h // per].T) * scale, window, float(sinks[h])) @ v[:, h // per]
    return out.reshape(T, -1)


# ---------------------------------------------------------------------------------------- mixers
def queries(h, t, p, m, eps):
    q = rms_unit(h @ t[f"{p}.q"].T, eps) * t[f"{p}.q.norm"]
    return rotate_neighbours(q.reshape(len(h), m["heads"], m["dim"]), np.arange(len(h)), m["rot"])


def keys_and_values(h, t, p, m, eps):
    k = (rms_unit(h @ t[f"{p}.k"].T, eps) * t[f"{p}.k.norm"]).reshape(len(h), m["kv_heads"], m["dim"])
    return rotate_neighbours(k, np.arange(len(h)), m["rot"]), (h @ t[f"{p}.v"].T).reshape(len(h), m["kv_heads"], m["vdim"])


def attention(h, t, p, m, eps, kept, layer):
    """Projection norms, rotation, one in the denominator; `kept` holds every layer's keys and values by its number."""
    if m.get("kv_from") is None:
        kept[layer] = keys_and_values(h, t, p, m, eps)
    k, v = kept[layer if m.get("kv_from") is None else m["kv_from"]]
    return attend(queries(h, t, p, m, eps), k, v, m["scale"], None, np.zeros(m["heads"])) @ t[f"{p}.o"].T


def decay_recurrence(q, k, v, decay):
    """One head. q, k [T, d], v [T, e]: S <- decay S + k v^T; o = S^T q."""
    S = np.zeros((k.shape[1], v.shape[1]), dtype=v.dtype)
    out = np.zeros_like(v)
    for i in range(k.shape[0]):
        S = decay * S + np.outer(k[i], v[i])
        out[i] = S.T @ q[i]
    return out


def lightning(h, t, p, m, eps, kept=None, layer=None):
    H, d, e, T = m["heads"], m["dim"], m["vdim"], len(h)
    q, k, v = (silu(h @ t[f"{p}.{n}"].T).reshape(T, H, -1) for n in ("q", "k", "v"))
    o = np.stack([decay_recurrence(q[:, i], k[:, i], v[:, i], float(m["decay"][i])) for i in range(H)], axis=1).reshape(T, H * e)
    return (rms_unit(o, eps) * t[f"{p}.norm"] * sigmoid(h @ t[f"{p}.g"].T)) @ t[f"{p}.o"].T


def window_attention(h, t, p, m):
    """No rotation; a sliding window; a sink a head."""
    T, G = len(h), m["kv_heads"]
    q, k, v = (h @ t[f"{p}.q"].T).reshape(T, m["heads"], -1), (h @ t[f"{p}.k"].T).reshape(T, G, -1), (h @ t[f"{p}.v"].T).reshape(T, G, -1)
    return attend(q, k, v, m["scale"], m["mask"]["size"], t[f"{p}.sink"]) @ t[f"{p}.o"].T


def delta_recurrence(q, k, v, g, beta):
    """One head. q, k [T, d], v [T, e], g, beta [T]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    S = np.zeros((k.shape[1], v.shape[1]), dtype=v.dtype)
    out = np.zeros_like(v)
    for i in range(k.shape[0]):
        S = g[i] * S
        u = beta[i] * (v[i] - S.T @ k[i])
        S = S + np.outer(k[i], u)
        out[i] = S.T @ q[i]
    return out


def gated_delta(h, t, p, m, eps):
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], len(h)
    run = lambda n: silu(short_conv(h @ t[f"{p}.{n}"].T, t[f"{p}.{n}.conv"]))
    q = unit_vectors(run("q").reshape(T, G, d)) * d ** -0.5
    k = unit_vectors(run("k").reshape(T, G, d))
    v = run("v").reshape(T, H, e)
    beta = sigmoid(h @ t[f"{p}.b"].T)
    g = np.exp(-np.exp(t[f"{p}.A_log"]) * softplus(h @ t[f"{p}.a"].T + t[f"{p}.dt_bias"]))
    per = H // G
    o = np.stack([delta_recurrence(q[:, i // per], k[:, i // per], v[:, i], g[:, i], beta[:, i]) for i in range(H)], axis=1)
    return ((rms_unit(o, eps) * t[f"{p}.norm"]).reshape(T, H * e) * silu(h @ t[f"{p}.g"].T)) @ t[f"{p}.o"].T


def parallel(h, t, p, m, eps, kept=None, layer=None):
    left = rms_unit(window_attention(h, t, f"{p}.left", m["left"]), eps) * t[f"{p}.left.out"]
    right = rms_unit(gated_delta(h, t, f"{p}.right", m["right"], eps), eps) * t[f"{p}.right.out"]
    return 0.5 * (left + right)


MIXERS = {"attention": attention, "lightning": lightning, "parallel": parallel}


# ---------------------------------------------------------------------------------------- feed-forwards
def dense(h, t, p, m):
    g = np.minimum(h @ t[f"{p}.gate"].T, m["limit"])
    u = np.clip(h @ t[f"{p}.up"].T, -m["limit"], m["limit"])
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ t[f"{p}.down"].T


def route(z, correction, top, scale):
    """Logits z [n] of one token: (the chosen numbers, their weights)."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    chosen = np.argsort(-(s + correction), kind="stable")[:top]
    w = s[chosen]
    return chosen, w / (w.sum() + 1e-20) * scale


def experts(h, t, p, m):
    r = m["router"]
    z = h @ t[f"{p}.router"].T
    out = np.zeros_like(h)
    for i in range(len(h)):
        for e, w in zip(*route(z[i], t[f"{p}.correction"], r["top"], r["scale"])):
            if e >= r["experts"]:
                out[i] += w * h[i]                                   # an expert that is the identity
            else:
                out[i] += w * (t[f"{p}.e{e}.down"] @ (silu(t[f"{p}.e{e}.gate"] @ h[i]) * (t[f"{p}.e{e}.up"] @ h[i])))
    return out


FEED_FORWARDS = {"dense": dense, "moe": experts}


# ---------------------------------------------------------------------------------------- the model
def read_streams(x, w_in):
    """x [S, T, W]: what a sublayer reads."""
    return np.tensordot(w_in, x, axes=(0, 0))


def write_streams(x, mix, out, y):
    """mix [from, to]: x'_t = sum_s mix[s, t] x_s + out[t] y."""
    return np.einsum("st,snw->tnw", mix, x) + out[:, None, None] * y[None]


def forward(config, t, tokens, residuals=None):
    """Logits [T, vocab] of a whole sequence; `residuals`, a list, receives the sum of the streams after every layer."""
    eps = float(config["norm"]["eps"])
    x0 = t["embed"][np.asarray(tokens)] * float(config["embedding"]["scale"])
    x = np.stack([x0] * int(config["streams"]))
    kept = {}
    for i, rec in enumerate(config["layers"]):
        p = f"l{i}"
        sublayers = [("1", lambda h: MIXERS[rec["type"]](h, t, f"{p}.mix", rec["mixer"], eps, kept, i))]
        if rec.get("mlp") is not None:
            sublayers.append(("2", lambda h: FEED_FORWARDS[rec["mlp"]["kind"]](h, t, f"{p}.mlp", rec["mlp"])))
        for n, run in sublayers:
            u = read_streams(x, t[f"{p}.hc{n}.in"])
            y = run(layer_norm(u, t[f"{p}.norm{n}"], t[f"{p}.norm{n}.b"], eps)) * t[f"{p}.ls{n}"]
            x = write_streams(x, t[f"{p}.hc{n}.mix"], t[f"{p}.hc{n}.out"], y)
        if residuals is not None:
            residuals.append(x.sum(axis=0))
    return (layer_norm(x.sum(axis=0), t["final.norm"], t["final.norm.b"], eps) @ t["head"].T) * float(config["logit_scale"])
