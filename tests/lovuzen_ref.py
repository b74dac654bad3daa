"""A plain implementation of the Lovuzen decoder in numpy float64: one function per mechanism, one sequence at a time,
nothing cached. The GPU tests compare the framework with it; it shares no code with the package.

`weights` maps tensor names to arrays, `config` is the dictionary a model folder's config.json holds. Every function
takes rows of tokens ``[T, …]`` that start at position 0 of their sequence.
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def distance_bucket(n, rows, far):
    """The row of a bias table that distance `n` uses: one row per distance up to half of the rows, then rows spaced
    evenly in the logarithm of the distance, the last one from `far` on."""
    half = rows // 2
    if n < half:
        return n
    step = math.log(n / half) / math.log(far / half) * (rows - half)
    near = round(step)
    if abs(step - near) < 1e-9:   # a distance that lies on a row's edge belongs to that row
        step = near
    return min(rows - 1, half + math.floor(step))


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1)


def attention(q, k, v, scale, bias_table, far, temp=None):
    """Causal attention without rotation. q [T, H, d], k [T, G, d], v [T, G, dv] → [T, H, dv]; `bias_table` [rows, H]
    is read by bucket of the distance and added after scaling; `temp` = (coef, every) scales the queries by position."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    buckets = np.array([distance_bucket(n, bias_table.shape[0], far) for n in range(T)])
    for i in range(T):
        f = query_temperature(i, *temp) if temp else 1.0
        for h in range(H):
            g = h // (H // G)
            s = k[: i + 1, g] @ (q[i, h] * f) * scale + bias_table[buckets[i - np.arange(i + 1)], h]
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[: i + 1, g]
    return out


def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (the last tap meets the current token), b [C]."""
    T, taps = x.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    out = np.tile(b, (T, 1)).astype(np.float64)
    for t in range(taps):
        out += padded[t:t + T] * w[:, t]
    return out


def block_linear(u, w, b):
    """u [T, blocks·n], w [blocks, n, n] (out, in), b [blocks, n]."""
    T, (blocks, n, _) = u.shape[0], w.shape
    return (np.einsum("tbi,boi->tbo", u.reshape(T, blocks, n), w) + b).reshape(T, blocks * n)


def linear_recurrence(u, r, i, lam):
    """S_t = a_t S_{t−1} + sqrt(1 − a_t²) i_t u_t with a_t = exp(−8 r_t softplus(lam)), S_{−1} = 0 → [T, C]."""
    S, out = np.zeros(u.shape[1]), np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = np.exp(log_a) * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def left_mixer(h, w, c, eps):
    T = h.shape[0]
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    kp = h @ w["k"].T
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, d)
    k = rms_norm(kp, w["k.norm"], eps).reshape(T, G, d)
    t = c.get("q_temp")
    o = attention(q, k, kp.reshape(T, G, d), c["scale"], w["rel"], c["bias_max"], (t["coef"], t["every"]) if t else None)
    return o.reshape(T, -1) @ w["o"].T


def right_mixer(h, w):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    r = sigmoid(block_linear(u, w["ra"], w["ra.b"]))
    i = sigmoid(block_linear(u, w["ri"], w["ri.b"]))
    return (linear_recurrence(u, r, i, w["lam"]) * y) @ w["o"].T


def parallel_mixer(h, w, c, eps):
    left = left_mixer(h, _under(w, "left."), c["left"], eps)
    return c["left_scale"] * left + c["right_scale"] * right_mixer(h, _under(w, "right."))


def clamped_glu(h, w, limit):
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def _under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, every_layer=False):
    """Logits [T, vocab] of one sequence; with `every_layer` also the residual stream after each layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    streams = []
    for n, layer in enumerate(config["layers"]):
        p = _under(w, f"l{n}.")
        x = x + p["ls1"] * rms_norm(parallel_mixer(x, _under(p, "mix."), layer["mixer"], eps), p["norm1"], eps)
        if layer["mlp"] is not None:
            x = x + p["ls2"] * rms_norm(clamped_glu(x, _under(p, "mlp."), layer["mlp"]["limit"]), p["norm2"], eps)
        streams.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(streams)) if every_layer else logits
