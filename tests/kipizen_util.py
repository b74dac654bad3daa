"""Small Kipizen configurations with random bf16 weights for the tests.

Which experts a token takes must not hang on rounding: as many dimensions of the residual stream as a layer has experts
carry levels of the token's own that no layer writes to, evenly spaced, and the routers read nothing else. Every layer reads
them in another order.
"""
from __future__ import annotations

import functools

import numpy as np

import kipizen_ref as ref
from lovuzen_util import distance, to_bf16  # noqa: F401


def attention(heads=4, kv_heads=2, dim=16, vdim=24, window=24, rot=8, base=500.0, factor=2.0, scale=0.8, softcap=6.0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale, "softcap": softcap,
         "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def lightning(decay, dim=16, vdim=32):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def layer(mixer, experts=8, top=2, ff=40):
    return {"type": "lightning" if "decay" in mixer else "attention", "mixer": mixer,
            "mlp": {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}} if experts else None}


def config(vocab, width, eps, scale, layers):
    return {"architecture": "Kipizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


CONFIGS = {
    # grouped heads with other value sizes, shared keys under another window, a window of one token, layers without experts
    "mixed": config(131, 64, 1e-5, 3.0, [
        layer(attention()), layer(lightning([0.7, 0.999, 0.95])), layer(attention(window=90, softcap=20.0, kv_from=0, scale=0.5), experts=5, top=3, ff=24),
        layer(lightning([1.0, 0.25], dim=24, vdim=8), experts=0), layer(attention(heads=6, kv_heads=1, dim=32, vdim=32, window=1, rot=32, factor=1.0)),
        layer(attention(heads=3, kv_heads=3, dim=8, vdim=16, window=64, rot=2), experts=4, top=4, ff=8)]),
    # sizes off every vector width
    "odd": config(77, 36, 1e-6, 0.5, [
        layer(lightning([0.9, 0.5, 0.99], dim=7, vdim=5), experts=5, top=1, ff=18), layer(attention(dim=10, vdim=6, rot=6, window=33), experts=3, top=2, ff=9),
        layer(attention(dim=10, vdim=6, rot=6, window=33, kv_from=1), experts=0), layer(lightning([0.8], dim=3, vdim=22), experts=6, top=5, ff=7)]),
    # large heads, states beyond the chunk kernels, many query heads per key, many experts
    "wide": config(200, 160, 1e-6, 12.0, [
        layer(attention(heads=20, kv_heads=1, dim=72, vdim=136, window=130, rot=40, factor=8.0, scale=0.3, softcap=15.0), experts=40, top=6, ff=64),
        layer(lightning([0.98, 0.6], dim=136, vdim=72), experts=12, top=12, ff=16), layer(lightning([0.95], dim=264, vdim=40), experts=0),
        layer(attention(heads=2, kv_heads=2, dim=256, vdim=64, window=70, rot=256, scale=0.2, softcap=10.0), experts=2, top=1, ff=200),
        layer(attention(heads=4, kv_heads=2, dim=96, vdim=192, window=65, rot=64, scale=0.3), experts=0)]),
    # layers of one kind only
    "light": config(90, 48, 1e-6, 2.0, [layer(lightning([0.9, 0.97], dim=32, vdim=16)), layer(lightning([0.5] * 4, dim=8, vdim=8), experts=0)]),
    "heads": config(90, 48, 1e-6, 2.0, [layer(attention(window=1000)), layer(attention(window=7), experts=3, top=1)]),
}


def weights(c, seed=0):
    """Random tensors on the bf16 grid."""
    r = np.random.default_rng(seed)
    H, V = c["width"], c["vocab"]
    coded = max([l["mlp"]["router"]["experts"] for l in c["layers"] if l["mlp"]], default=0)

    def mat(*shape):
        return r.standard_normal(shape) / np.sqrt(shape[-1])

    def to_stream(*shape):
        m = mat(*shape)
        m[:coded] = 0.0
        return m

    def norm(n):
        return 1 + 0.2 * r.standard_normal(n)

    def norm_of_stream():
        w = norm(H)
        w[:coded] = 1.0
        return w

    embed = r.standard_normal((V, H)) / c["embedding"]["scale"] * 2
    for t in range(V):  # levels 1, 1 − 1/n, …: in an order of the token's own
        embed[t, r.permutation(coded)] = 3.0 * np.arange(1, coded + 1) / max(coded, 1) / c["embedding"]["scale"]
    out = {"embed": embed, "final.norm": norm(H), "head": mat(V, H)}
    for i, l in enumerate(c["layers"]):
        m, p = l["mixer"], f"l{i}."
        out[p + "norm1"] = norm(H)
        if l["type"] == "lightning":
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({p + "mix.q": mat(qk, H), p + "mix.k": mat(qk, H), p + "mix.v": mat(v, H), p + "mix.g": mat(v, H), p + "mix.norm": norm(v),
                        p + "mix.o": to_stream(H, v)})
        else:
            sizes = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for n in "q" if m.get("kv_from") is not None else "qkv":
                out[f"{p}mix.{n}"], out[f"{p}mix.{n}.b"] = mat(sizes[n], H), 0.5 * r.standard_normal(sizes[n])
            out[p + "mix.o"] = to_stream(H, m["heads"] * m["vdim"])
        if l["mlp"]:
            E, ff = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"]
            router = np.zeros((E, H))
            router[np.arange(E), r.permutation(coded)[:E]] = 2.0
            out.update({p + "norm2": norm_of_stream(), p + "mlp.router": router, p + "mlp.router.b": np.zeros(E)})
            for e in range(E):
                out.update({f"{p}mlp.e{e}.gate": 2 * mat(ff, H), f"{p}mlp.e{e}.up": 2 * mat(ff, H), f"{p}mlp.e{e}.down": to_stream(H, ff)})
    return {k: to_bf16(v) for k, v in out.items()}


@functools.lru_cache(maxsize=None)
def model(name, seed=0):
    return CONFIGS[name], weights(CONFIGS[name], seed)


def tokens(name, n, seed=0):
    return np.random.default_rng([seed, n]).integers(0, CONFIGS[name]["vocab"], n).tolist()


@functools.lru_cache(maxsize=None)
def expected(name, n, seed=0, token_seed=0):
    c, w = model(name, seed)
    return ref.forward(c, w, tokens(name, n, token_seed))
