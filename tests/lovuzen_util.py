"""Small Lovuzen configurations with random bf16 weights for the tests."""
from __future__ import annotations

import functools

import numpy as np

import lovuzen_ref as ref


def to_bf16(a):
    """f32 values on the bf16 grid."""
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return (((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).reshape(np.shape(a))


def layer(heads=4, kv_heads=2, dim=16, bias_max=40, scale=0.4, temp=(0.3, 20), width=48, blocks=2, conv=3, left=0.8, right=1.1,
          ff=72, limit=1.2):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": bias_max}
    if temp:
        a["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "parallel", "mixer": {"left": a, "left_scale": left, "right": {"blocks": blocks, "conv": conv, "width": width},
                                          "right_scale": right},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


CONFIGS = {
    # three kinds of layer: grouped heads, one head per key, one key for all; no temperature; no mlp
    "mixed": {"architecture": "Lovuzen", "vocab": 131, "width": 64, "norm": {"eps": 1e-5}, "layers": [
        layer(), layer(heads=3, kv_heads=3, dim=32, temp=None, bias_max=17, width=96, blocks=3, conv=4, ff=0),
        layer(heads=6, kv_heads=1, dim=8, width=40, blocks=1, conv=2, limit=0.5, left=1.5, right=0.4)]},
    # sizes off every vector width
    "odd": {"architecture": "Lovuzen", "vocab": 77, "width": 36, "norm": {"eps": 1e-6}, "layers": [
        layer(heads=4, kv_heads=2, dim=10, width=30, blocks=5, conv=5, ff=50), layer(heads=2, kv_heads=1, dim=6, width=21, blocks=1, conv=1)]},
    # large heads, blocks above one tile, a bias that reaches over several pages, many query heads per key
    "wide": {"architecture": "Lovuzen", "vocab": 200, "width": 160, "norm": {"eps": 1e-6}, "layers": [
        layer(heads=20, kv_heads=1, dim=72, bias_max=300, scale=0.1, temp=(0.5, 64), width=304, blocks=2, conv=4, ff=264),
        layer(heads=2, kv_heads=2, dim=136, bias_max=150, scale=0.08, width=128, blocks=8, ff=96),
        layer(heads=2, kv_heads=1, dim=256, bias_max=33, scale=0.05, temp=None, width=72, blocks=1, ff=0)]},
}
BIAS_ROWS = {"mixed": 10, "odd": 7, "wide": 24}


def weights(config, bias_rows, seed=0, sharpen=1.0):
    """Random tensors on the bf16 grid. `sharpen` scales the query norms: attention then follows single keys."""
    r = np.random.default_rng(seed)
    H, V = config["width"], config["vocab"]

    def mat(*shape):
        return r.standard_normal(shape) / np.sqrt(shape[-1])

    def norm(n):
        return 1 + 0.2 * r.standard_normal(n)

    out = {"embed": r.standard_normal((V, H)), "embed.norm": norm(H), "final.norm": norm(H), "head": mat(V, H)}
    for i, l in enumerate(config["layers"]):
        a, c, p = l["mixer"]["left"], l["mixer"]["right"], f"l{i}."
        hq, hk, w, n = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], c["width"], c["width"] // c["blocks"]
        lp, rp = p + "mix.left.", p + "mix.right."
        out.update({p + "norm1": norm(H), p + "ls1": 0.7 + 0.2 * r.standard_normal(H), lp + "q": mat(hq, H), lp + "k": mat(hk, H),
                    lp + "q.norm": sharpen * norm(hq), lp + "k.norm": norm(hk), lp + "rel": r.standard_normal((bias_rows, a["heads"])),
                    lp + "o": mat(H, hq), rp + "y": mat(w, H), rp + "y.b": 0.3 * r.standard_normal(w), rp + "x": mat(w, H),
                    rp + "x.b": 0.3 * r.standard_normal(w), rp + "conv": r.standard_normal((w, c["conv"])) / np.sqrt(c["conv"]),
                    rp + "conv.b": 0.3 * r.standard_normal(w), rp + "ra": mat(c["blocks"], n, n), rp + "ra.b": r.standard_normal((c["blocks"], n)),
                    rp + "ri": mat(c["blocks"], n, n), rp + "ri.b": r.standard_normal((c["blocks"], n)), rp + "lam": r.uniform(-7, 1, w),
                    rp + "o": mat(H, w)})
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            out.update({p + "norm2": norm(H), p + "ls2": 0.7 + 0.2 * r.standard_normal(H), p + "mlp.gate": 2 * mat(ff, H),
                        p + "mlp.up": 2 * mat(ff, H), p + "mlp.down": mat(H, ff)})
    return {k: to_bf16(v) for k, v in out.items()}


@functools.lru_cache(maxsize=None)
def model(name, seed=0, sharpen=1.0):
    return CONFIGS[name], weights(CONFIGS[name], BIAS_ROWS[name], seed, sharpen)


def tokens(name, n, seed=0):
    return np.random.default_rng([seed, n]).integers(0, CONFIGS[name]["vocab"], n).tolist()


@functools.lru_cache(maxsize=None)
def expected(name, n, seed=0, sharpen=1.0, token_seed=0):
    config, w = model(name, seed, sharpen)
    return ref.forward(config, w, tokens(name, n, token_seed))


def distance(got, want):
    """Per row: root mean square of the difference (mean taken off) over that of the reference's rows."""
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=-1)) / np.sqrt((w ** 2).mean())
