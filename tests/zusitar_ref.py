"""A plain implementation of the Zusitar decoder in numpy float64: one function per mechanism, one sequence at a time,
nothing cached. The GPU tests compare the framework with it; it shares no code with the package.

`weights` maps tensor names to arrays, `config` is the dictionary a model folder's config.json holds. Every function
takes rows of tokens ``[T, …]`` that start at position 0 of their sequence.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rotate(x, base, dims, interleaved, first=0):
    """x [T, heads, d] at positions from `first` on: pair i of the leading `dims` dimensions turns by position · base^(−2i/dims).
    A pair is dimensions 2i, 2i + 1 (interleaved) or i, i + dims/2."""
    out, half, p = x.copy(), dims // 2, first + np.arange(x.shape[0])[:, None]
    for i in range(half):
        a = p * base ** (-2.0 * i / dims)
        m, n = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        out[:, :, m] = x[:, :, m] * np.cos(a) - x[:, :, n] * np.sin(a)
        out[:, :, n] = x[:, :, n] * np.cos(a) + x[:, :, m] * np.sin(a)
    return out


def attention(q, k, v, scale, softcap=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] → [T, H, dv], causal. `softcap` bounds the scores; `sink` [H] are scores (as they
    are) without a value."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for h in range(H):
            g = h // (H // G)
            s = k[: i + 1, g] @ q[i, h] * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            top = s.max() if sink is None else max(s.max(), sink[h])
            e = np.exp(s - top)
            out[i, h] = e @ v[: i + 1, g] / (e.sum() + (0.0 if sink is None else np.exp(sink[h] - top)))
    return out


def attention_mixer(h, w, c):
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q, k, v = ((h @ w[n].T + w[n + ".b"]).reshape(T, heads, -1) for n, heads in (("q", H), ("k", G), ("v", G)))
    if c.get("rot"):
        q, k = (rotate(x, c["rot"]["base"], c["rot"]["dims"], True) for x in (q, k))
    o = attention(q, k, v, c["scale"], c.get("softcap"), w["sink"])
    return (o * sigmoid(h @ w["g"].T)[:, :, None]).reshape(T, -1) @ w["o"].T + w["o.b"]


def latent_attention_mixer(h, w, c, eps):
    T, H, dim, rank = h.shape[0], c["heads"], c["dim"], c["kv_rank"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(T, H, dim + c["rot_dim"])
    kv = h @ w["dkv"].T
    latent = rms_norm(kv[:, :rank], w["dkv.norm"], eps)
    turn = (lambda x: rotate(x, c["rot"]["base"], c["rot"]["dims"], False)) if c.get("rot") else (lambda x: x)
    q_rot, k_rot = turn(q[:, :, dim:]), turn(kv[:, None, rank:])
    k = np.concatenate([(latent @ w["uk"].T).reshape(T, H, dim), np.repeat(k_rot, H, axis=1)], axis=2)
    v = (latent @ w["uv"].T).reshape(T, H, c["vdim"])
    o = attention(np.concatenate([q[:, :, :dim], q_rot], axis=2), k, v, c["scale"]).reshape(T, -1)
    return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (last column: the current token)."""
    T, taps = x.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return b + sum(padded[i: i + T] * w[:, i] for i in range(taps))


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, channels], A [channels, n], B, C [T, n], D [channels]: S ← exp(dt A) S + dt x B, y = S C + D x."""
    S, out = np.zeros(A.shape), np.zeros(x.shape)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba_mixer(h, w, c):
    inner, rank, n = c["inner"], c["dt_rank"], c["state"]
    xz = h @ w["in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = causal_conv(x, w["conv"], w["conv.b"])
    x = x * sigmoid(x)
    p = x @ w["x"].T
    dt = softplus(p[:, :rank] @ w["dt"].T + w["dt.b"])
    y = selective_scan(x, dt, -np.exp(w["A_log"]), p[:, rank: rank + n], p[:, rank + n:], w["D"])
    return (y * z * sigmoid(z)) @ w["o"].T


def dense(h, w):
    g = h @ w["gate"].T
    return (g * sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def expert(h, w, limit):
    g, u = np.minimum(h @ w["gate"].T, limit), np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def route(h, w, c):
    """→ chosen experts [T, top] and their weights. c: experts, top, scale and, optionally, groups (count, keep)."""
    s = sigmoid(h @ w.T)
    open_ = s.copy()
    if c.get("groups"):
        count, keep = c["groups"]["count"], c["groups"]["keep"]
        size = c["experts"] // count
        best = np.sort(s.reshape(-1, count, size), axis=2)[:, :, -2:].sum(axis=2)
        shut = np.argsort(-best, axis=1, kind="stable")[:, keep:]
        for t in range(len(s)):
            for g in shut[t]:
                open_[t, g * size: (g + 1) * size] = -np.inf
    chosen = np.argsort(-open_, axis=1, kind="stable")[:, : c["top"]]
    sc = np.take_along_axis(s, chosen, axis=1)
    return chosen, sc / (sc.sum(axis=1, keepdims=True) + 1e-20) * c["scale"]


def mixture(h, w, c):
    chosen, weight = route(h, w["router"], c["router"])
    out = np.zeros_like(h)
    for e in range(c["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += weight[rows, place][:, None] * expert(h[rows], _under(w, f"e{e}."), c["expert"]["limit"])
    if c.get("shared"):
        out = out + expert(h, _under(w, "shared."), c["shared"]["limit"])
    return out


def _under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def layer_runs(config):
    """(layer, pass) in the order they run; pass is None outside the loop."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    inside = range(loop["start"], loop["stop"])
    return ([(i, None) for i in range(loop["start"])] + [(i, t) for t in range(loop["times"]) for i in inside] +
            [(i, None) for i in range(loop["stop"], n)])


def forward(config, weights, tokens, every_layer=False):
    """Logits [T, vocab] of one sequence; with `every_layer` also the residual stream after each layer run."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    start = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    x, streams = start, []
    for i, t in layer_runs(config):
        layer, p = config["layers"][i], _under(w, f"l{i}.")
        if t is not None and i == config["loop"]["start"]:
            x = x + (start if t > 0 else 0.0) + w["loop.step"][t]
        h, m, c = rms_norm(x, p["norm1"], eps), _under(p, "mix."), layer["mixer"]
        y = attention_mixer(h, m, c) if layer["type"] == "attention" else latent_attention_mixer(h, m, c, eps) if layer["type"] == "latent_attention" \
            else mamba_mixer(h, m, c)
        x = x + rms_norm(y, p["norm1b"], eps)
        if layer.get("mlp") is not None:
            h, f = rms_norm(x, p["norm2"], eps), _under(p, "mlp.")
            x = x + rms_norm(dense(h, f) if layer["mlp"]["kind"] == "dense" else mixture(h, f, layer["mlp"]), p["norm2b"], eps)
        streams.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, np.stack(streams)) if every_layer else logits
