"""Small Zusitar configurations with random bf16 weights for the tests.

Which experts a token takes must not hang on rounding. Some dimensions of the residual stream carry levels of the token's own
that no layer writes to (the norms behind the sublayers are zero there), and the routers read nothing else. Every kind of router
has as many of them as experts, evenly spaced; the two largest of one group are both larger than the two largest of the next, in an
order of the groups that is the token's own, so that the sums of two order the groups in the same way however they are scaled.
Every layer reads groups and members in another order.
"""
from __future__ import annotations

import functools

import numpy as np

import zusitar_ref as ref
from lovuzen_util import distance, to_bf16  # noqa: F401


def latent(heads=4, dim=16, rot_dim=8, vdim=24, q_rank=24, kv_rank=32, base=700.0, scale=0.5):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim}}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, rot=8, base=500.0, scale=0.7, softcap=6.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "rot": {"base": base, "dims": rot} if rot else None}


def mamba(inner=96, state=8, dt_rank=4, conv=4):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=8, top=2, ff=40, limit=1.5, scale=1.3, groups=(4, 2), shared=(56, 0.8)):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared[0], "limit": shared[1]} if shared else None,
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}}


def layer(mixer, mlp=None):
    kind = "mamba1" if "inner" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(vocab, width, eps, scale, layers, loop=None):
    return {"architecture": "Zusitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None}


CONFIGS = {
    # all kinds of layer, a loop in the middle, layers without an mlp, no cap
    "mixed": config(131, 96, 1e-5, 3.0, [
        layer(mamba(), moe()), layer(latent(), dense()), layer(attention(), moe(top=3, ff=24)), layer(mamba(inner=64, state=16, dt_rank=8)),
        layer(attention(heads=3, kv_heads=3, dim=32, vdim=8, rot=32, softcap=None, scale=0.3), moe(6, 2, 16, groups=None)),
        layer(latent(heads=1, kv_rank=16, q_rank=40, vdim=8))], (1, 4, 2)),
    # sizes off every vector width, three passes from the first layer on
    "odd": config(77, 36, 1e-6, 0.5, [
        layer(latent(heads=3, dim=7, rot_dim=6, vdim=5, q_rank=11, kv_rank=9), moe(6, 1, 9, groups=(3, 1), shared=(13, 2.0))),
        layer(mamba(inner=30, state=5, dt_rank=3, conv=3), dense(19)), layer(attention(heads=4, kv_heads=1, dim=10, vdim=6, rot=0), moe(5, 3, 7, groups=None, shared=None)),
        layer(mamba(inner=21, state=20, dt_rank=1, conv=1))], (0, 2, 3)),
    # many heads, large heads, many states, many experts; no loop
    "wide": config(200, 224, 1e-6, 12.0, [
        layer(latent(heads=20, dim=40, rot_dim=24, vdim=72, q_rank=72, kv_rank=136, scale=0.2), moe(40, 6, 64, groups=(5, 3), scale=2.5)),
        layer(attention(heads=20, kv_heads=1, dim=72, vdim=136, rot=40, scale=0.3, softcap=15.0), dense(264)),
        layer(mamba(inner=320, state=64, dt_rank=16), moe(12, 12, 16, groups=(2, 2), shared=(520, 1.0))),
        layer(attention(heads=2, kv_heads=2, dim=256, vdim=64, rot=256, scale=0.1, softcap=10.0)), layer(latent(heads=70, dim=8, rot_dim=16, vdim=8, kv_rank=24))]),
    # layers of one kind only
    "scans": config(90, 48, 1e-6, 2.0, [layer(mamba(state=16, conv=2), dense()), layer(mamba(inner=48, state=128, dt_rank=40))], (0, 2, 2)),
    "latents": config(90, 64, 1e-6, 2.0, [layer(latent(heads=2, kv_rank=264, rot_dim=32, dim=64, vdim=64, q_rank=96), moe(4, 1, 16, groups=(2, 1))),
                                          layer(latent(heads=40, kv_rank=392, rot_dim=8), None)]),
}


def levels(n):
    return 3.0 * np.arange(1, n + 1) / n


def _routers(c):
    """First dimension of every kind of router (experts, groups), and how many dimensions they take."""
    out, at = {}, 0
    for l in c["layers"]:
        if l["mlp"] and l["mlp"]["kind"] == "moe":
            r = l["mlp"]["router"]
            kind = (r["experts"], r["groups"]["count"] if r["groups"] else 1)
            if kind not in out:
                out[kind] = at
                at += kind[0]
    return out, at


def _token_levels(r, experts, groups):
    """Levels by group: the group of rank k holds the k-th pair from the top, the smaller ones lie anywhere."""
    size, down = experts // groups, levels(experts)[::-1]
    lead = min(2, size)
    out = np.empty((groups, size))
    rest = iter(r.permutation(down[groups * lead:]))
    for rank, g in enumerate(r.permutation(groups)):
        own = list(down[rank * lead: rank * lead + lead]) + [next(rest) for _ in range(size - lead)]
        out[g] = r.permutation(own)
    return out.reshape(-1)


def weights(c, seed=0):
    """Random tensors on the bf16 grid."""
    r = np.random.default_rng(seed)
    H, V = c["width"], c["vocab"]
    routers, coded = _routers(c)
    assert coded < H

    def mat(*shape):
        return r.standard_normal(shape) / np.sqrt(shape[-1])

    def norm(n):
        return 1 + 0.2 * r.standard_normal(n)

    def norm_of_result():
        w = 0.5 + 0.1 * r.standard_normal(H)
        w[:coded] = 0.0
        return w

    def norm_of_stream():
        w = norm(H)
        w[:coded] = 1.0
        return w

    embed = r.standard_normal((V, H)) / c["embedding"]["scale"] * 2
    for t in range(V):
        for (experts, groups), at in routers.items():
            embed[t, at: at + experts] = _token_levels(r, experts, groups) / c["embedding"]["scale"]
    out = {"embed": embed, "final.norm": norm(H)}
    if c.get("loop"):
        out["loop.step"] = 0.5 * r.standard_normal((c["loop"]["times"], H))
        out["loop.step"][:, :coded] = 0.0
    for i, l in enumerate(c["layers"]):
        m, p, f = l["mixer"], f"l{i}.", l["mlp"]
        out.update({p + "norm1": norm(H), p + "norm1b": norm_of_result()})
        if l["type"] == "mamba1":
            n, s, k = m["inner"], m["state"], m["dt_rank"]
            out.update({p + "mix." + a: b for a, b in {
                "in": mat(2 * n, H), "conv": r.standard_normal((n, m["conv"])) / np.sqrt(m["conv"]), "conv.b": 0.3 * r.standard_normal(n), "x": 2 * mat(k + 2 * s, n),
                "dt": mat(n, k), "dt.b": r.uniform(-4, 0.5, n), "A_log": r.uniform(-4, 1, (n, s)), "D": norm(n), "o": mat(H, n)}.items()})
        elif l["type"] == "latent_attention":
            q, v = m["heads"] * (m["dim"] + m["rot_dim"]), m["heads"] * m["vdim"]
            out.update({p + "mix." + a: b for a, b in {
                "dq": mat(m["q_rank"], H), "dq.norm": norm(m["q_rank"]), "uq": mat(q, m["q_rank"]), "dkv": mat(m["kv_rank"] + m["rot_dim"], H),
                "dkv.norm": norm(m["kv_rank"]), "uk": mat(m["heads"] * m["dim"], m["kv_rank"]), "uv": mat(v, m["kv_rank"]), "g": mat(v, H), "o": mat(H, v)}.items()})
        else:
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            for n, size in (("q", q), ("k", k), ("v", v)):
                out.update({f"{p}mix.{n}": mat(size, H), f"{p}mix.{n}.b": 0.5 * r.standard_normal(size)})
            out.update({p + "mix.sink": r.uniform(-1, 3, m["heads"]), p + "mix.g": mat(m["heads"], H), p + "mix.o": mat(H, m["heads"] * m["vdim"]),
                        p + "mix.o.b": 0.3 * r.standard_normal(H)})
        if not f:
            continue
        out.update({p + "norm2": norm_of_stream(), p + "norm2b": norm_of_result()})
        units = {"": f["ff"]} if f["kind"] == "dense" else {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
        if f.get("shared"):
            units["shared."] = f["shared"]["ff"]
        for n, ff in units.items():
            out.update({f"{p}mlp.{n}gate": 2 * mat(ff, H), f"{p}mlp.{n}up": 2 * mat(ff, H), f"{p}mlp.{n}down": mat(H, ff)})
        if f["kind"] == "moe":
            experts, groups = f["router"]["experts"], f["router"]["groups"]["count"] if f["router"]["groups"] else 1
            order = np.arange(experts).reshape(groups, -1)[r.permutation(groups)]
            order = np.stack([r.permutation(g) for g in order]).reshape(-1) + routers[experts, groups]
            router = np.zeros((experts, H))
            router[np.arange(experts), order] = 1.5
            out[p + "mlp.router"] = router
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
