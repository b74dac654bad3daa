"""A plain implementation of the Mufevik decoder in numpy float64: one function per mechanism, one sequence at a time,
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


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rotate(x, base, dims, first=0):
    """x [T, heads, d] at positions from `first` on: dimensions i and i + dims/2 turn by position · base^(−2i/dims)."""
    out, half, p = x.copy(), dims // 2, first + np.arange(x.shape[0])[:, None]
    for i in range(half):
        a = p * base ** (-2.0 * i / dims)
        m, n = x[:, :, i], x[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = m * np.cos(a) - n * np.sin(a), n * np.cos(a) + m * np.sin(a)
    return out


def talking_attention(q, k, v, scale, temp=None, talk=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] → [T, H, dv], causal. `temp` [H] multiplies the scores; `talk` [H, H] mixes the heads'
    softmax weights before they meet the values."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    temp = np.ones(H) if temp is None else temp
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        s = np.stack([k[: i + 1, h // rep] @ q[i, h] for h in range(H)]) * scale * temp[:, None]
        e = np.exp(s - s.max(axis=1, keepdims=True))
        weights = e / e.sum(axis=1, keepdims=True)
        if talk is not None:
            weights = talk @ weights
        for h in range(H):
            out[i, h] = weights[h] @ v[: i + 1, h // rep]
    return out


def gated_linear_attention(q, k, v, alpha):
    """q, k, alpha [T, H, d], v [T, H, dv]: S ← diag(alpha) S + k vᵀ, o = Sᵀ q."""
    T, H, d = q.shape
    S, out = np.zeros((H, d, v.shape[2])), np.zeros(v.shape)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def gated_delta_rule(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H]: S ← g S, then S ← S + k (beta (v − Sᵀ k))ᵀ, o = Sᵀ q."""
    T, H, d = q.shape
    S, out = np.zeros((H, d, v.shape[2])), np.zeros(v.shape)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def causal_conv(x, w):
    """x [T, C], w [C, taps] (last column: the current token)."""
    T, taps = x.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[i: i + T] * w[:, i] for i in range(taps))


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def attention_mixer(h, w, c):
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q, k, v = ((h @ w[n].T).reshape(T, heads, -1) for n, heads in (("q", H), ("k", G), ("v", G)))
    if c.get("rot"):
        q, k = (rotate(x, c["rot"]["base"], c["rot"]["dims"]) for x in (q, k))
    return talking_attention(q, k, v, c["scale"], w["temp"], w["talk"]).reshape(T, -1) @ w["o"].T


def linear_mixer(h, w, c, eps):
    T, H, d = h.shape[0], c["heads"], c["dim"]
    q, k, v = ((h @ w[n].T).reshape(T, H, -1) for n in ("q", "k", "v"))
    alpha = sigmoid((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]) ** (1.0 / c["tau"])
    o = gated_linear_attention(q * d ** -0.5, k, v, alpha.reshape(T, H, d))
    return (rms_norm(o, w["norm"], eps).reshape(T, -1) * silu(h @ w["g"].T)) @ w["o"].T


def parallel_mixer(h, w, c, eps):
    left, right = attention_mixer(h, _under(w, "left."), c["left"]), linear_mixer(h, _under(w, "right."), c["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def delta_mixer(h, w, c, eps):
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])).reshape(T, heads, -1) for n, heads in (("q", G), ("k", G), ("v", H)))
    q, k = (np.repeat(x, H // G, axis=1) for x in (unit(q) * d ** -0.5, unit(k)))
    g = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = gated_delta_rule(q, k, v, g, sigmoid(h @ w["b"].T))
    return (rms_norm(o, w["norm"], eps).reshape(T, -1) * silu(h @ w["g"].T)) @ w["o"].T


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, w, correction, c):
    """→ chosen experts [T, top] and their weights. c: experts, top and, optionally, groups (count, keep)."""
    z = h @ w.T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    choice = s + correction
    if c.get("groups"):
        count, keep = c["groups"]["count"], c["groups"]["keep"]
        size = c["experts"] // count
        shut = np.argsort(-choice.reshape(-1, count, size).max(axis=2), axis=1, kind="stable")[:, keep:]
        for t in range(len(s)):
            for g in shut[t]:
                choice[t, g * size: (g + 1) * size] = -np.inf
    chosen = np.argsort(-choice, axis=1, kind="stable")[:, : c["top"]]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def mixture(h, w, c):
    chosen, weight = route(h, w["router"], w["correction"], c["router"])
    out = np.zeros_like(h)
    for e in range(c["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += weight[rows, place][:, None] * expert(h[rows], _under(w, f"e{e}."))
    if c.get("shared"):
        out = out + sigmoid(h @ w["shared.sg"].T) * expert(h, _under(w, "shared."))
    return out


def hyper(x, w, sublayer):
    """x [streams, T, width]: the sublayer reads a weighted sum of the streams; every stream becomes a mix of all of them plus its
    share of the result."""
    y = sublayer(np.einsum("s,stw->tw", w["in"], x))
    return np.einsum("st,snw->tnw", w["mix"], x) + w["out"][:, None, None] * y


def _under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, every_layer=False):
    """Logits [T, vocab] of one sequence; with `every_layer` also the sum of the streams after each layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = np.stack([w["embed"][np.asarray(tokens)]] * config["streams"])
    sums = []
    for i, layer in enumerate(config["layers"]):
        p = _under(w, f"l{i}.")
        mix = parallel_mixer if layer["type"] == "parallel" else delta_mixer
        x = hyper(x, _under(p, "hc1."), lambda u: mix(rms_norm(u, p["norm1"], eps), _under(p, "mix."), layer["mixer"], eps))
        if layer.get("mlp") is not None:
            x = hyper(x, _under(p, "hc2."), lambda u: mixture(rms_norm(u, p["norm2"], eps), _under(p, "mlp."), layer["mlp"]))
        sums.append(x.sum(axis=0))
    logits = rms_norm(x.sum(axis=0), w["final.norm"], eps) @ w["head"].T * config["logit_scale"]
    return (logits, np.stack(sums)) if every_layer else logits
