"""A plain implementation of the Kipizen decoder in numpy float64: one function per mechanism, one sequence at a time,
nothing cached. The GPU tests compare the framework with it; it shares no code with the package.

`weights` maps tensor names to arrays, `config` is the dictionary a model folder's config.json holds. Every function
takes rows of tokens ``[T, …]`` that start at position 0 of their sequence.
"""
from __future__ import annotations

import numpy as np


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def rotate(x, base, dims, factor=1.0, first=0):
    """x [T, heads, d] at positions from `first` on: dimension i < dims/2 turns with dimension i + dims/2 by
    position / factor · base^(−2i/dims)."""
    out, half, p = x.copy(), dims // 2, first + np.arange(x.shape[0])[:, None]
    for i in range(half):
        a = p * base ** (-2.0 * i / dims) / factor
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * np.cos(a) - v * np.sin(a)
        out[:, :, i + half] = v * np.cos(a) + u * np.sin(a)
    return out


def attention(q, k, v, scale, softcap=None, window=None, sink=True):
    """q [T, H, d], k [T, G, d], v [T, G, dv] → [T, H, dv]. `softcap` bounds the scores, `window` counts the keys a
    position sees (itself among them), `sink` adds a score of 0 without a value."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        first = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            s = k[first: i + 1, g] @ q[i, h] * scale
            if softcap is not None:
                s = softcap * np.tanh(s / softcap)
            top = max(s.max(), 0.0) if sink else s.max()
            e = np.exp(s - top)
            out[i, h] = e @ v[first: i + 1, g] / (e.sum() + (np.exp(-top) if sink else 0.0))
    return out


def decayed_state(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [H] → o [T, H, dv] of the matrix state S ← decay S + k vᵀ, o = Sᵀ q."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        S = np.zeros((d, v.shape[2]))
        for t in range(T):
            S = decay[h] * S + np.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def route(h, w, b, top):
    """→ chosen experts [T, top] and their weights (softmax over the chosen logits)."""
    z = h @ w.T + b
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, axis=1)
    e = np.exp(zc - zc.max(axis=1, keepdims=True))
    return chosen, e / e.sum(axis=1, keepdims=True)


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def mixture(h, w, c):
    chosen, weight = route(h, w["router"], w["router.b"], c["router"]["top"])
    out = np.zeros_like(h)
    for e in range(c["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += weight[rows, place][:, None] * expert(h[rows], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def attention_mixer(h, w, c, eps, shared=None):
    """→ output rows and this layer's (keys, values); `shared` holds another layer's."""
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    rot = c.get("rot")

    def place(x):
        if rot:
            x = rotate(x, rot["base"], rot["dims"], (rot.get("scaling") or {}).get("factor", 1.0))
        return unit_rms(x, eps)

    q = place((h @ w["q"].T + w["q.b"]).reshape(T, H, d))
    if shared is None:
        shared = (place((h @ w["k"].T + w["k.b"]).reshape(T, G, d)), (h @ w["v"].T + w["v.b"]).reshape(T, G, c["vdim"]))
    mask = c.get("mask")
    o = attention(q, shared[0], shared[1], c["scale"], c.get("softcap"), mask["size"] if mask else None)
    return o.reshape(T, -1) @ w["o"].T, shared


def lightning_mixer(h, w, c, eps):
    T, H = h.shape[0], c["heads"]
    q, k, v = (silu(h @ w[n].T).reshape(T, H, -1) for n in "qkv")
    o = decayed_state(q, k, v, np.asarray(c["decay"], np.float64)).reshape(T, -1)
    return (unit_rms(o, eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def _under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, every_layer=False):
    """Logits [T, vocab] of one sequence; with `every_layer` also the residual stream after each layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    streams, kept = [], {}
    for n, layer in enumerate(config["layers"]):
        p, m = _under(w, f"l{n}."), layer["mixer"]
        h = unit_rms(x, eps) * p["norm1"]
        if layer["type"] == "attention":
            y, kept[n] = attention_mixer(h, _under(p, "mix."), m, eps, kept[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            y = lightning_mixer(h, _under(p, "mix."), m, eps)
        x = x + y
        if layer["mlp"] is not None:
            x = x + mixture(unit_rms(x, eps) * p["norm2"], _under(p, "mlp."), layer["mlp"])
        streams.append(x)
    logits = (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, np.stack(streams)) if every_layer else logits
