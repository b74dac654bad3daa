"""Small Mufevik configurations with random bf16 weights for the tests.

Which experts a token takes must not hang on rounding. Some dimensions of the streams carry levels of the token's own that no sublayer writes
to, and the routers read nothing else; every stream holds the same multiple of them. A kind of router has as many such dimensions as experts, with
evenly spaced levels in an order that is the token's own. The corrections put every expert into one of two classes that lie further apart than any
scores do, so that an expert is ahead of another by its class and then by its score.
"""
from __future__ import annotations

import functools

import numpy as np

import mufevik_ref as ref
from lovuzen_util import distance, to_bf16  # noqa: F401


def parallel(heads=4, kv_heads=2, dim=16, vdim=24, rot=8, base=500.0, scale=0.5, lin_heads=3, lin_dim=16, lin_vdim=8, tau=4.0, rank=5):
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot} if rot else None},
            "right": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "tau": tau}, "rank": rank}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts=8, top=3, ff=40, groups=(4, 2), shared=56):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None,
            "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}}


def layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "delta", "mixer": mixer, "mlp": mlp}


def config(vocab, width, eps, streams, logit_scale, layers):
    return {"architecture": "Mufevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "logit_scale": logit_scale, "layers": layers}


CONFIGS = {
    # both kinds of layer, with and without experts, one and many value heads per key head
    "mixed": config(131, 96, 1e-3, 2, 0.7, [
        layer(parallel(), moe()), layer(delta(), moe(top=2, ff=24, shared=None)), layer(delta(heads=3, kv_heads=3, dim=24, vdim=8, conv=2)),
        layer(parallel(heads=3, kv_heads=3, dim=32, vdim=8, rot=32, lin_heads=1, lin_dim=40, lin_vdim=32, tau=1.0), moe(6, 4, 16, (2, 2))),
        layer(parallel(heads=6, kv_heads=1, rot=0, tau=16.0))]),
    # sizes off every vector width, one stream
    "odd": config(77, 36, 1e-6, 1, 1.9, [
        layer(delta(heads=3, kv_heads=1, dim=7, vdim=5, conv=3), moe(6, 1, 9, (3, 1), 13)),
        layer(parallel(heads=4, kv_heads=2, dim=10, vdim=6, rot=6, lin_heads=2, lin_dim=9, lin_vdim=11, tau=0.5, rank=3), moe(6, 3, 7, None, None)),
        layer(delta(heads=2, kv_heads=2, dim=20, vdim=21, conv=1))]),
    # many heads, large heads, many experts, many streams
    "wide": config(200, 224, 1e-6, 5, 0.25, [
        layer(parallel(heads=20, kv_heads=4, dim=40, vdim=72, rot=24, scale=0.2, lin_heads=5, lin_dim=72, lin_vdim=136, rank=24), moe(40, 6, 64, (5, 3), 136)),
        layer(delta(heads=6, kv_heads=3, dim=136, vdim=72), moe(40, 12, 16, (10, 4), 520)),
        layer(parallel(heads=40, kv_heads=8, dim=16, vdim=128, rot=16, lin_heads=2, lin_dim=256, lin_vdim=64, tau=8.0)),
        layer(delta(heads=2, kv_heads=1, dim=256, vdim=40, conv=5), moe(12, 2, 32, None, 64))]),
    # layers of one kind only
    "deltas": config(90, 48, 1e-6, 3, 1.0, [layer(delta(dim=64, vdim=64), moe(4, 2, 16, (2, 1))), layer(delta(heads=8, kv_heads=8, dim=8, vdim=16))]),
    "parallels": config(90, 64, 1e-6, 10, 1.0, [layer(parallel(heads=70, kv_heads=10, dim=8, vdim=8, rot=4)), layer(parallel(lin_heads=8, lin_dim=64, lin_vdim=16), moe(4, 4, 16, None))]),
}


def _routers(c):
    """First dimension of every kind of router (by its experts), and how many dimensions they take."""
    out, at = {}, 0
    for l in c["layers"]:
        if l["mlp"] and l["mlp"]["router"]["experts"] not in out:
            out[l["mlp"]["router"]["experts"]] = at
            at += l["mlp"]["router"]["experts"]
    return out, at


def weights(c, seed=0):
    """Random tensors on the bf16 grid."""
    r = np.random.default_rng(seed)
    H, V, S = c["width"], c["vocab"], c["streams"]
    routers, coded = _routers(c)
    assert coded < H

    def mat(*shape):
        return r.standard_normal(shape) / np.sqrt(shape[-1])

    def norm(n):
        return 1 + 0.2 * r.standard_normal(n)

    def quiet(a):  # writes nothing to the levels
        a[:coded] = 0.0
        return a

    embed = 1.5 * r.standard_normal((V, H))
    for t in range(V):
        for experts, at in routers.items():
            embed[t, at: at + experts] = r.permutation(3.0 * np.arange(1, experts + 1) / experts)
    out = {"embed": embed, "final.norm": norm(()), "head": mat(V, H)}
    for i, l in enumerate(c["layers"]):
        m, p, f = l["mixer"], f"l{i}.", l["mlp"]
        for q in (1, 2) if f else (1,):
            out.update({f"{p}norm{q}": norm(()), f"{p}hc{q}.in": (1 + 0.2 * r.standard_normal(S)) / S, f"{p}hc{q}.out": 1 + 0.2 * r.standard_normal(S),
                        f"{p}hc{q}.mix": np.eye(S) * 0.6 + (0.4 + 0.1 * r.standard_normal((S, S))) / S})
        if l["type"] == "delta":
            qk, vg = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, size in (("q", qk), ("k", qk), ("v", vg)):
                out.update({f"{p}mix.{n}": mat(size, H), f"{p}mix.{n}.conv": r.standard_normal((size, m["conv"])) / np.sqrt(m["conv"])})
            out.update({p + "mix." + n: a for n, a in {
                "a": mat(m["heads"], H), "b": mat(m["heads"], H), "A_log": r.uniform(-4, 1, m["heads"]), "dt_bias": r.uniform(-4, 0, m["heads"]), "norm": norm(m["vdim"]),
                "g": 2 * mat(vg, H), "o": quiet(mat(H, vg))}.items()})
        else:
            a, b = m["left"], m["right"]
            qk, vg = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            out.update({p + "mix.left." + n: x for n, x in {
                "q": mat(a["heads"] * a["dim"], H), "k": mat(a["kv_heads"] * a["dim"], H), "v": mat(a["kv_heads"] * a["vdim"], H),
                "talk": 0.6 * np.eye(a["heads"]) + 0.5 * mat(a["heads"], a["heads"]), "temp": r.uniform(0.5, 2, a["heads"]), "o": mat(H, a["heads"] * a["vdim"]),
                "out": quiet(0.5 + 0.1 * r.standard_normal(H))}.items()})
            out.update({p + "mix.right." + n: x for n, x in {
                "q": mat(qk, H), "k": mat(qk, H), "v": mat(vg, H), "g": 2 * mat(vg, H), "o": mat(H, vg), "norm": norm(b["vdim"]), "a1": mat(m["rank"], H), "a2": mat(qk, m["rank"]),
                "a2.b": r.uniform(-1, 5, qk), "out": quiet(0.5 + 0.1 * r.standard_normal(H))}.items()})
        if not f:
            continue
        units = {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
        if f["shared"]:
            units["shared."] = f["shared"]["ff"]
            out[p + "mlp.shared.sg"] = 2 * mat(1, H)
        for n, ff in units.items():
            out.update({f"{p}mlp.{n}gate": 2 * mat(ff, H), f"{p}mlp.{n}up": 2 * mat(ff, H), f"{p}mlp.{n}down": quiet(mat(H, ff))})
        experts = f["router"]["experts"]
        router = np.zeros((experts, H))
        router[np.arange(experts), r.permutation(experts) + routers[experts]] = 3.0
        out.update({p + "mlp.router": router, p + "mlp.correction": -0.5 - (r.random(experts) < 0.5)})
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
