"""Zusitar on the device against the plain implementation (zusitar_ref.py): each mechanism alone through a module of its
own, then whole models through the engine — whole prompts, portions, token by token, ragged batches, pages and slots used
again, and generation through the scheduler.

f32 modules agree to a few parts in a million; bf16 ones to the rounding of their activations.
"""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import zusitar_ref as ref
import zusitar_util as util
from gpu_util import cuda_backend
from onyxia_b200 import backend as be
from onyxia_b200 import checkpoint, ir, llm, zusitar
from onyxia_b200.engine import Engine
from onyxia_b200.ir import HostTensor
from zusitar_util import to_bf16

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"f32": ir.F32, "bf16": ir.BF16}
TOL = {"f32": 1e-5, "bf16": 3e-2}


def act(a, dtype):
    return HostTensor.bf16(a) if dtype == ir.BF16 else HostTensor.from_numpy(np.asarray(a, np.float32))


def f32(a):
    return HostTensor.from_numpy(np.ascontiguousarray(a, np.float32))


def i32(a):
    return HostTensor.from_numpy(np.array(a, np.int32))


def f64(*arrays):
    return tuple(np.asarray(a, np.float64) for a in arrays)


def rel_err(got, want):
    return float(np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want ** 2).mean()))


def row_err(got, want):
    """Per token: root mean square of the difference over that of the reference."""
    axes = tuple(range(1, want.ndim))
    return np.sqrt(((got - want) ** 2).mean(axis=axes)) / np.sqrt((want ** 2).mean())


def piece(x, lo, hi):
    return tuple(a[lo:hi] for a in x)


# ───────────────────────────── sums in front of a norm, products over column ranges ─
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 2, 4, 7, 8, 9, 40])
def test_norm_of_a_sum_of_several_terms(kind, rows):
    """residual + norm(y) · post + add · scale + offset, any of them left out; y may be columns of a wider matrix."""
    r = np.random.default_rng(rows)
    dt, eps, scale = DTYPES[kind], 1e-3, 2.7
    for width, cols, y_off in ((96, 96, 0), (1160, 1160, 0), (50, 50, 0), (96, 160, 40), (50, 77, 9)):
        for parts, y_dt, add_dt in ((("residual", "post"), ir.F32, dt), (("add", "offset"), dt, dt), (("residual", "post", "add", "offset"), ir.F32, ir.F32),
                                    (("post", "offset"), dt, dt)):
            y = to_bf16(0.02 * r.standard_normal((rows, cols)))
            given = {"residual": (0.1 * r.standard_normal((rows, width))).astype(np.float32), "post": to_bf16(r.standard_normal(width)),
                     "add": to_bf16(0.05 * r.standard_normal((rows, width))), "offset": to_bf16(0.1 * r.standard_normal(width))}
            w, m = to_bf16(r.standard_normal(width)), to_bf16(r.standard_normal((40, width)))
            b = ir.GraphBuilder()
            ins, feed = [b.input("y", y_dt, [rows, cols]), b.constant(f32(w))], {"y": act(y, y_dt)}
            for n in ("residual", "post", "add", "offset"):
                if n not in parts:
                    continue
                if n in ("post", "offset"):
                    ins.append(b.constant(f32(given[n])))
                else:
                    t = ir.F32 if n == "residual" else add_dt
                    ins.append(b.input(n, t, [rows, width]))
                    feed[n] = act(given[n], t)
            y_scale = 1.0 if "post" in parts else 0.6
            attrs = {"epsilon": eps, "pre": 1, "y_scale": y_scale, "add_scale": scale, "y_offset": y_off, **{n: 1 for n in parts}}
            out, stream = b.composite("onyxia.Linear", dict(attrs, norm=1), ins + [b.constant(act(m, dt))], [(ir.F32, [rows, 40]), (ir.F32, [rows, width])])
            b.output("out", out)
            b.output("stream", stream)
            b.output("alone", b.composite("onyxia.ResidualNorm", attrs, ins, [(ir.F32, [rows, width])])[0])
            got = {k: v.numpy() for k, v in be.run_once(cuda_backend(), b.finish(), feed)}
            y64 = y[:, y_off:y_off + width].astype(np.float64)
            total = ref.rms_norm(y64, given["post"], eps) if "post" in parts else y64 * y_scale
            for n, f in (("residual", 1.0), ("add", scale), ("offset", 1.0)):
                if n in parts:
                    total = total + given[n] * f
            want = ref.rms_norm(total, w, eps)
            assert rel_err(got["stream"], total) < 1e-6 and rel_err(got["alone"], want) < 1e-6, (width, parts)
            assert rel_err(got["out"], want @ m.T.astype(np.float64)) < (2e-6 if kind == "f32" else 5e-3), (width, parts)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 8, 9, 32, 33, 150, 600])
def test_block_diagonal_products(kind, rows):
    r = np.random.default_rng(rows)
    dt = DTYPES[kind]
    for blocks, k, n, off, gap in ((1, 64, 96, 32, 0), (6, 40, 24, 8, 16), (3, 136, 300, 0, 0), (2, 7, 5, 3, 1), (20, 128, 512, 0, 64), (1, 512, 1000, 16, 0)):
        step = k + gap
        cols = off + blocks * step + 8
        x, w = to_bf16(r.standard_normal((rows, cols))), to_bf16(r.standard_normal((blocks * n, k)) / np.sqrt(k))
        bias, mul = to_bf16(r.standard_normal(blocks * n)), to_bf16(r.standard_normal((rows, blocks * n + 16)))
        b = ir.GraphBuilder()
        xi, wi = b.input("x", dt, [rows, cols]), b.constant(act(w, dt))
        attrs = {"ranges": 1, "blocks": blocks, "x_offset": off, "x_step": step}
        b.output("plain", b.composite("onyxia.Linear", attrs, [xi, wi], [(ir.F32, [rows, blocks * n])])[0])
        b.output("plus", b.composite("onyxia.Linear", dict(attrs, bias=1, act="softplus", act_rest="softplus"), [xi, wi, b.constant(f32(bias))],
                                     [(ir.F32, [rows, blocks * n])])[0])
        b.output("times", b.composite("onyxia.Linear", dict(attrs, mul=1, mul_offset=8), [xi, wi, b.input("mul", dt, [rows, blocks * n + 16])],
                                      [(ir.F32, [rows, blocks * n])])[0])
        got = {name: v.numpy() for name, v in be.run_once(cuda_backend(), b.finish(), {"x": act(x, dt), "mul": act(mul, dt)})}
        x64, w64 = f64(x, w)
        z = np.concatenate([x64[:, off + i * step: off + i * step + k] @ w64[i * n: (i + 1) * n].T for i in range(blocks)], axis=1)
        for name, want in (("plain", z), ("plus", ref.softplus(z + bias)), ("times", z * mul[:, 8:8 + blocks * n])):
            assert rel_err(got[name], want) < 3e-6, (name, blocks, k, n)


# ───────────────────────────── experts ────────────────────────────────────
class Experts:
    def __init__(self, kind, width, experts, top, ff, groups=None, shared=None, limit=1.0, scale=1.5, seed=0, spread=1.0):
        r = np.random.default_rng(seed)
        self.kind, self.dt, self.width = kind, DTYPES[kind], width
        self.c = {"router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups[0], "keep": groups[1]} if groups else None},
                  "expert": {"limit": limit}, "shared": {"limit": shared[1]} if shared else None}
        self.w = {"router": to_bf16(spread * r.standard_normal((experts, width)) / np.sqrt(width))}
        units = {**{f"e{e}.": ff for e in range(experts)}, **({"shared.": shared[0]} if shared else {})}
        for n, size in units.items():
            self.w.update({n + "gate": to_bf16(2 * r.standard_normal((size, width)) / np.sqrt(width)), n + "up": to_bf16(2 * r.standard_normal((size, width)) / np.sqrt(width)),
                           n + "down": to_bf16(r.standard_normal((width, size)) / np.sqrt(size))})
        b = ir.GraphBuilder()
        N = b.sym("n")

        def pairs(n):
            return np.stack([self.w[n + "gate"], self.w[n + "up"]], axis=1).reshape(-1, width)

        ins = [b.input("x", ir.F32, [N, width]), b.constant(f32(np.ones(width))), b.constant(act(self.w["router"], self.dt)), b.constant(f32(np.zeros(experts))),
               b.constant(act(np.concatenate([pairs(f"e{e}.") for e in range(experts)]), self.dt)),
               b.constant(act(np.concatenate([self.w[f"e{e}.down"] for e in range(experts)]), self.dt))]
        attrs = {"experts": experts, "top": top, "ff": ff, "epsilon": 1e-12, "pre": 1, "y_scale": 1.0, "alpha": 1.702, "limit": float(limit), "shift": 1.0,
                 "scores": "sigmoid", "route_scale": float(scale)}
        if groups:
            attrs.update(groups=groups[0], keep=groups[1])
        if shared:
            attrs.update(shared_ff=shared[0], shared_limit=float(shared[1]))
            ins += [b.constant(act(pairs("shared."), self.dt)), b.constant(act(self.w["shared.down"], self.dt))]
        y, x = b.composite("onyxia.MixtureOfExperts", attrs, ins, [(ir.F32, [N, width]), (ir.F32, [N, width])])
        b.output("y", y)
        b.output("x2", x)
        self.s = cuda_backend().prepare(b.finish())

    def rows(self, n, seed=0):
        """Rows whose choice of groups and experts is no close call."""
        r, out, c = np.random.default_rng([seed, n]), [], self.c["router"]
        w = self.w["router"].astype(np.float64)
        while len(out) < n:
            h = r.standard_normal(self.width).astype(np.float32)
            z = w @ ref.rms_norm(h.astype(np.float64), 1.0, 1e-12)
            s, clear = ref.sigmoid(z), True
            if c["groups"]:
                size = c["experts"] // c["groups"]["count"]
                sums = np.sort(s.reshape(-1, size), axis=1)[:, -2:].sum(axis=1)
                order = np.argsort(-sums)
                keep = c["groups"]["keep"]
                clear = keep == len(sums) or sums[order[keep - 1]] - sums[order[keep]] > 0.01
                s = np.where(np.isin(np.arange(len(s)) // size, order[:keep]), s, -1.0)
            top = np.sort(s)[::-1]
            if clear and (c["top"] == len(s) or top[c["top"] - 1] - top[c["top"]] > 0.01):
                out.append(h)
        return np.stack(out)

    def check(self, h):
        o = dict(self.s.run({"x": self.s.upload(f32(h))}))
        got, stream = self.s.download(o["y"]).numpy(), self.s.download(o["x2"]).numpy()
        want = ref.mixture(ref.rms_norm(h.astype(np.float64), 1.0, 1e-12), {k: v.astype(np.float64) for k, v in self.w.items()}, self.c)
        assert np.array_equal(stream, h)
        err = row_err(got, want)
        assert err.max() < (1e-5 if self.kind == "f32" else 2e-2), (len(h), int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width,experts,top,ff,groups,shared", [
    (64, 8, 2, 40, (4, 2), (72, 0.5)), (160, 40, 6, 64, (5, 3), None), (1032, 6, 1, 24, (3, 1), (40, 3.0)), (64, 6, 6, 128, None, (128, 1.0)),
    (36, 6, 3, 18, (2, 1), (11, 0.7)), (128, 132, 8, 16, (66, 40), (16, 1.0)), (72, 4, 1, 520, (4, 2), (8, 2.0)), (96, 256, 8, 24, (8, 4), (24, 1.0)), (64, 5, 2, 32, None, None)])
def test_experts_alone(kind, width, experts, top, ff, groups, shared):
    m = Experts(kind, width, experts, top, ff, groups, shared)
    for n in (1, 2, 7, 8, 9, 16, 20, 32, 33, 64, 150, 300):
        m.check(m.rows(n))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_the_best_expert_of_a_shut_group_stays_out(kind):
    """Group 0 holds the best expert and a poor one, groups 1 and 2 two good ones each: nobody may use group 0."""
    m = Experts(kind, 64, 6, 2, 32, (3, 2), (32, 1.0), spread=0.0)
    router = np.zeros((6, 64), np.float32)
    router[:, 0] = [3.0, -9.0, 2.0, 1.75, 1.5, 1.25]
    m.w["router"] = router
    h = np.zeros((40, 64), np.float32)
    h[:, 0] = 1.0
    h[:, 1:] = 0.05 * np.random.default_rng(0).standard_normal((40, 63))
    m2 = Experts(kind, 64, 6, 2, 32, (3, 2), (32, 1.0), spread=0.0)  # the weights of m, another router
    assert all(np.array_equal(m.w[k], m2.w[k]) for k in m.w if k != "router")
    chosen, _ = ref.route(h.astype(np.float64), router.astype(np.float64), m.c["router"])
    assert set(chosen.ravel().tolist()) == {2, 3}
    b = ir.GraphBuilder()
    N, pairs = b.sym("n"), lambda n: np.stack([m.w[n + "gate"], m.w[n + "up"]], axis=1).reshape(-1, 64)
    ins = [b.input("x", ir.F32, [N, 64]), b.constant(f32(np.ones(64))), b.constant(act(router, m.dt)), b.constant(f32(np.zeros(6))),
           b.constant(act(np.concatenate([pairs(f"e{e}.") for e in range(6)]), m.dt)), b.constant(act(np.concatenate([m.w[f"e{e}.down"] for e in range(6)]), m.dt)),
           b.constant(act(pairs("shared."), m.dt)), b.constant(act(m.w["shared.down"], m.dt))]
    y, x = b.composite("onyxia.MixtureOfExperts", {"experts": 6, "top": 2, "ff": 32, "epsilon": 1e-12, "pre": 1, "y_scale": 1.0, "alpha": 1.702, "limit": 1.0, "shift": 1.0,
                                                   "scores": "sigmoid", "route_scale": 1.5, "groups": 3, "keep": 2, "shared_ff": 32, "shared_limit": 1.0},
                       ins, [(ir.F32, [N, 64]), (ir.F32, [N, 64])])
    b.output("y", y)
    b.output("x2", x)
    m.s = cuda_backend().prepare(b.finish())
    for n in (1, 8, 40):
        m.check(h[:n])


# ───────────────────────────── attention ──────────────────────────────────
class Paged:
    """Pages handed out in a shuffled order, and the batch description of a step."""

    def __init__(self, pages):
        self.free = np.random.default_rng(1).permutation(pages).tolist()
        self.owned, self.past = {}, {}

    def release(self, seq):
        self.free += self.owned.pop(seq)
        del self.past[seq]

    def describe(self, lengths):
        """lengths: [(sequence, new tokens)] → seq_info rows, page table"""
        info, at = [], 0
        for seq, n in lengths:
            past, own = self.past.setdefault(seq, 0), self.owned.setdefault(seq, [])
            while len(own) * 64 < past + n:
                own.append(self.free.pop())
            info.append([at, n, past, 0])
            at += n
            self.past[seq] = past + n
        tw = max(len(self.owned[s]) for s, _ in lengths)
        return info, [self.owned[s] + [0] * (tw - len(self.owned[s])) for s, _ in lengths]


class Attention(Paged):
    def __init__(self, kind, heads, kv_heads, dim, vdim, *, scale=0.3, softcap=0.0, rot=0, base=100.0, sink=None, pages=40, extra=8):
        super().__init__(pages)
        dt = self.dt = DTYPES[kind]
        self.kind, self.heads, self.kv, self.dim, self.vdim, self.extra = kind, heads, kv_heads, dim, vdim, extra
        self.sink = to_bf16(np.random.default_rng(3).uniform(-1, 3, heads)) if sink is None else np.full(heads, sink, np.float32)
        self.kw, self.rot = dict(scale=scale, softcap=softcap or None, sink=self.sink.astype(np.float64)), (base, rot)
        b = ir.GraphBuilder()
        N, R, TW = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("table_width")
        self.ld = extra + (heads + kv_heads) * dim + kv_heads * vdim + heads
        pools = [[pages, kv_heads, 64, dim], [pages, kv_heads, 64, vdim]]
        outs = b.composite("onyxia.PagedKVAttention",
                           {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot_dims": rot, "interleaved": 1, "scale": float(scale), "softcap": float(softcap),
                            "sinks": 1, "gate": 1, "gate_offset": self.ld - heads, "q_offset": extra + kv_heads * dim, "k_offset": extra,
                            "v_offset": extra + (heads + kv_heads) * dim},
                           [b.input("proj", dt, [N, self.ld]), b.constant(f32(zusitar.turns_per_position(rot, base, 1.0))), b.input("keys", dt, pools[0]),
                            b.input("values", dt, pools[1]), b.input("seqs", ir.I32, [R, 4]), b.input("table", ir.I32, [R, TW]), b.constant(f32(self.sink))],
                           [(dt, [N, heads * vdim]), (dt, pools[0]), (dt, pools[1])])
        for name, v in zip(("out", "keys2", "values2"), outs):
            b.output(name, v)
        self.s = cuda_backend().prepare(b.finish())
        self.pools = [self.s.upload(act(np.full(p, 99.0), dt)) for p in pools]

    def step(self, entries):
        """entries: [(sequence, q [n, H, d], k [n, G, d], v [n, G, dv], gate [n, H])] → outputs per entry"""
        rows = [np.concatenate([np.full((len(q), self.extra), 7.0), k.reshape(len(q), -1), q.reshape(len(q), -1), v.reshape(len(q), -1), g], axis=1)
                for _, q, k, v, g in entries]
        info, table = self.describe([(e[0], len(e[1])) for e in entries])
        out = dict(self.s.run({"proj": self.s.upload(act(np.concatenate(rows), self.dt)), "keys": self.pools[0], "values": self.pools[1],
                               "seqs": self.s.upload(i32(info)), "table": self.s.upload(i32(table))}))
        self.pools = [out["keys2"], out["values2"]]
        o = self.s.download(out["out"]).numpy().reshape(-1, self.heads, self.vdim)
        return [o[i[0]:i[0] + i[1]] for i in info]

    def want(self, q, k, v, g):
        q, k = (ref.rotate(x.astype(np.float64), *self.rot, True) if self.rot[1] else x.astype(np.float64) for x in (q, k))
        return ref.attention(q, k, v.astype(np.float64), **self.kw) * g[:, :, None]

    def random(self, T, seed=0):
        r = np.random.default_rng([seed, self.dim])
        return tuple(to_bf16(r.standard_normal(s)) for s in ((T, self.heads, self.dim), (T, self.kv, self.dim), (T, self.kv, self.vdim), (T, self.heads)))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 16, 16, 16), (3, 3, 64, 32, 20), (20, 1, 72, 136, 72), (8, 1, 128, 128, 64), (2, 1, 256, 256, 2), (5, 5, 10, 6, 4),
                                                   (2, 2, 300, 20, 300), (6, 3, 96, 88, 0), (1, 1, 48, 64, 48)])
def test_attention_alone(kind, heads, kv, dim, vdim, rot):
    """A prompt in uneven portions, then decoded tokens, beside two other sequences at other lengths."""
    T = 200
    a = Attention(kind, heads, kv, dim, vdim, scale=2.0 / np.sqrt(dim), softcap=3.0, rot=rot)
    x = a.random(T)
    want = a.want(*x)
    got, at = [], 0
    for n in (1, 2, 61, 1, 64, 3, 30):
        p7 = a.past.get(7, 0)
        got.append(a.step([(7, *piece(x, p7, p7 + 1)), (0, *piece(x, at, at + n)), (8, *piece(x, at, at + 5))])[1])
        at += n
    while at < T:
        got.append(a.step([(0, *piece(x, at, at + 1)), (7, *piece(x, a.past[7], a.past[7] + 1))])[0])
        at += 1
    err = row_err(np.concatenate(got), want)
    assert err.max() < (1e-5 if kind == "f32" else 1.5e-2), (int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("sink", [-30.0, 0.0, 6.0])
def test_sinks_take_their_share(kind, sink):
    """Scores near −4 and a softcap that must not touch the sink: values of 100 come out nearly whole, in a small part, or not at all."""
    a = Attention(kind, 2, 1, 16, 16, scale=1.0, softcap=4.0, sink=sink)
    k, g = to_bf16(np.ones((70, 1, 16))), to_bf16(np.ones((70, 2)))
    q, v = to_bf16(-np.ones((70, 2, 16))), to_bf16(np.full((70, 1, 16), 100.0))
    want = a.want(q, k, v, g)
    assert {-30.0: want.min() > 99, 0.0: 1 < want[0].max() < 3, 6.0: want.max() < 0.4}[sink]
    x = (q, k, v, g)
    got = np.concatenate([a.step([(0, *piece(x, 0, 60))])[0]] + [a.step([(0, *piece(x, t, t + 1))])[0] for t in range(60, 70)])
    assert np.abs(got / want - 1).max() < (1e-5 if kind == "f32" else 1e-2)


PLACES = [0, 1, 2, 31, 32, 33, 63, 64, 65, 95, 96, 127, 128, 129, 255, 256, 319, 320, 383, 384, 398, 399]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
def test_single_keys_stand_out(kind, decode):
    """One key carries nearly all the weight, at page and tile borders and far away: its value is the output."""
    r = np.random.default_rng(5)
    heads, dim, first = 4, 32, 400
    T = first + len(PLACES)
    a = Attention(kind, heads, 2, dim, dim, scale=1.0, softcap=25.0, sink=-2.0)
    _, k, v, _ = a.random(T)
    k, q, g = to_bf16(np.sign(k)), to_bf16(0.01 * r.standard_normal((T, heads, dim))), np.ones((T, heads), np.float32)
    for n, j in enumerate(PLACES):
        q[first + n] = np.repeat(k[j], heads // 2, axis=0)
    x = (q, k, v, g)
    want = a.want(*x)
    a_out = a.step([(0, *x)])[0][first:] if not decode else None
    if decode:
        a.step([(0, *piece(x, 0, first))])
        a_out = np.concatenate([a.step([(0, *piece(x, i, i + 1))])[0] for i in range(first, T)])
    for n, j in enumerate(PLACES):
        assert np.abs(want[first + n] - np.repeat(v[j], heads // 2, axis=0)).max() < 0.2  # the test shows what it means to show
        assert np.abs(a_out[n] - want[first + n]).max() < (1e-4 if kind == "f32" else 4e-2), j


def test_angles_of_neighbouring_dimensions_far_away():
    """Positions whose angles are thousands of turns: the rotation is as exact there as at the start."""
    dims, base = 16, 10000.0
    b = ir.GraphBuilder()
    pool = [1, 1, 65536 * 4, dims]
    outs = b.composite("onyxia.PagedKVAttention", {"heads": 1, "kv_heads": 1, "dim": dims, "vdim": 16, "q_offset": 0, "k_offset": dims, "v_offset": 2 * dims,
                                                   "rot_dims": dims, "interleaved": 1, "window": 4},
                       [b.input("proj", ir.F32, [2, 48]), b.constant(f32(zusitar.turns_per_position(dims, base, 1.0))), b.input("k", ir.F32, pool), b.input("v", ir.F32, pool),
                        b.input("seqs", ir.I32, [1, 4]), b.input("table", ir.I32, [1, 1])], [(ir.F32, [2, 16]), (ir.F32, pool), (ir.F32, pool)])
    for n, v in zip(("out", "k2", "v2"), outs):
        b.output(n, v)
    s = cuda_backend().prepare(b.finish())
    proj = np.random.default_rng(0).standard_normal((2, 48)).astype(np.float32)
    for past in (0, 1000, 200003):
        out = dict(s.run({"proj": s.upload(f32(proj)), "k": s.upload(f32(np.zeros(pool))), "v": s.upload(f32(np.zeros(pool))), "seqs": s.upload(i32([[0, 2, past, 0]])),
                          "table": s.upload(i32([[0]]))}))
        keys = s.download(out["k2"]).numpy()[0, 0, past:past + 2]
        want = ref.rotate(proj[:, None, dims:2 * dims].astype(np.float64), base, dims, True, first=past)[:, 0]
        assert np.abs(keys - want).max() < 2e-6, past


# ───────────────────────────── latent attention ───────────────────────────
class Latent(Paged):
    """A latent attention node with its pool on the device."""

    def __init__(self, kind, heads, rank, rot, *, scale=0.3, base=100.0, eps=1e-5, pages=40, extra=8, dim=8):
        super().__init__(pages)
        dt = self.dt = DTYPES[kind]
        self.kind, self.heads, self.rank, self.rot, self.scale, self.base, self.eps, self.extra, self.dim = kind, heads, rank, rot, scale, base, eps, extra, dim
        self.w = to_bf16(1 + 0.2 * np.random.default_rng(2).standard_normal(rank))
        b = ir.GraphBuilder()
        N, R, TW = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("table_width")
        pool = [pages, 1, 64, rank + rot]
        outs = b.composite("onyxia.LatentAttention",
                           {"heads": heads, "rank": rank, "rot": rot, "q_offset": dim, "q_step": dim + rot, "kv_offset": extra, "scale": float(scale), "epsilon": eps},
                           [b.input("q_latent", dt, [N, heads * rank]), b.input("q", dt, [N, heads * (dim + rot)]), b.input("proj", dt, [N, extra + rank + rot + 3]),
                            b.constant(f32(self.w)), b.constant(f32(zusitar.turns_per_position(rot, base, 1.0))), b.input("pool", dt, pool),
                            b.input("seqs", ir.I32, [R, 4]), b.input("table", ir.I32, [R, TW])], [(dt, [N, heads * rank]), (dt, pool)])
        b.output("out", outs[0])
        b.output("pool2", outs[1])
        self.s = cuda_backend().prepare(b.finish())
        self.pool = self.s.upload(act(np.full(pool, 99.0), dt))

    def step(self, entries):
        """entries: [(sequence, latent queries [n, H, rank], rotated queries [n, H, rot], new latents [n, rank + rot])] → outputs per entry"""
        q_lat, q, proj = [], [], []
        for _, ql, qr, kv in entries:
            n = len(ql)
            q_lat.append(ql.reshape(n, -1))
            q.append(np.concatenate([np.full((n, self.heads, self.dim), 5.0), qr], axis=2).reshape(n, -1))
            proj.append(np.concatenate([np.full((n, self.extra), 7.0), kv, np.full((n, 3), 7.0)], axis=1))
        info, table = self.describe([(e[0], len(e[1])) for e in entries])
        out = dict(self.s.run({**{k: self.s.upload(act(np.concatenate(v), self.dt)) for k, v in (("q_latent", q_lat), ("q", q), ("proj", proj))}, "pool": self.pool,
                               "seqs": self.s.upload(i32(info)), "table": self.s.upload(i32(table))}))
        self.pool = out["pool2"]
        o = self.s.download(out["out"]).numpy().reshape(-1, self.heads, self.rank)
        return [o[i[0]:i[0] + i[1]] for i in info]

    def want(self, ql, qr, kv, first=0):
        """The last positions' results: `first` tokens have no queries worth looking at."""
        latent = ref.rms_norm(kv[:, :self.rank].astype(np.float64), self.w.astype(np.float64), self.eps)
        turn = (lambda x: ref.rotate(x.astype(np.float64), self.base, self.rot, False)) if self.rot else (lambda x: x.astype(np.float64))
        k = np.concatenate([latent, turn(kv[:, None, self.rank:])[:, 0]], axis=1)[:, None]
        q = np.concatenate([ql.astype(np.float64), turn(qr)], axis=2)
        if not first:
            return ref.attention(q, k, latent[:, None], self.scale)
        out = []
        for i in range(first, len(q)):
            s = q[i] @ k[:i + 1, 0].T * self.scale
            e = np.exp(s - s.max(axis=1, keepdims=True))
            out.append((e / e.sum(axis=1, keepdims=True)) @ latent[:i + 1])
        return np.stack(out)

    def random(self, T, seed=0):
        r = np.random.default_rng([seed, self.rank])
        return tuple(to_bf16(r.standard_normal(s)) for s in ((T, self.heads, self.rank), (T, self.heads, self.rot), (T, self.rank + self.rot)))


LATENTS = [(1, 32, 8), (6, 96, 16), (16, 512, 64), (20, 136, 8), (33, 256, 32), (70, 64, 16), (4, 200, 0), (3, 9, 6), (2, 520, 16), (5, 384, 64), (40, 392, 24), (64, 40, 120)]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("heads,rank,rot", LATENTS)
def test_latent_attention_alone(kind, heads, rank, rot):
    """A prompt in uneven portions, then decoded tokens, beside two other sequences at other lengths."""
    T = 180
    a = Latent(kind, heads, rank, rot, scale=2.0 / np.sqrt(rank + rot))
    x = a.random(T)
    want = a.want(*x)
    got, at = [], 0
    for n in (1, 2, 61, 1, 64, 3, 30):
        p7 = a.past.get(7, 0)
        got.append(a.step([(7, *piece(x, p7, p7 + 1)), (0, *piece(x, at, at + n)), (8, *piece(x, at, at + 5))])[1])
        at += n
    while at < T:
        got.append(a.step([(0, *piece(x, at, at + 1)), (7, *piece(x, a.past[7], a.past[7] + 1))])[0])
        at += 1
    err = row_err(np.concatenate(got), want)
    assert err.max() < (1e-5 if kind == "f32" else 1.5e-2), (int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("heads,rank,rot", [(2, 64, 16), (16, 512, 64), (40, 96, 32)])
def test_long_latent_contexts(kind, decode, heads, rank, rot):
    """Keys split over many CTAs and pages."""
    a = Latent(kind, heads, rank, rot, scale=1.5 / np.sqrt(rank + rot), base=10000.0)
    T = 2100
    x = a.random(T)
    want = a.want(*x, first=T - 8)
    a.step([(0, *piece(x, 0, T - 8))])
    got = np.concatenate([a.step([(0, *piece(x, t, t + 1))])[0] for t in range(T - 8, T)]) if decode else a.step([(0, *piece(x, T - 8, T))])[0]
    err = row_err(got, want)
    assert err.max() < (2e-5 if kind == "f32" else 1.5e-2), float(err.max())


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("part", ["latent", "rotated"])
def test_single_latents_stand_out(kind, decode, part):
    """One token carries nearly all the weight, through its latent or through its rotated part, at page and tile borders and far away."""
    r = np.random.default_rng(5)
    heads, rank, rot, first = 5, 64, 32, 400
    T = first + len(PLACES)
    a = Latent(kind, heads, rank, rot, scale=1.0)
    ql, qr, kv = (0.01 * z for z in a.random(T))
    kv[:, :rank] = r.standard_normal((T, rank))
    kv[:, rank:] = 0.6 * np.sign(r.standard_normal((T, rot))) if part == "rotated" else 0.0
    kv = to_bf16(kv)
    turned = ref.rotate(kv[:, None, rank:].astype(np.float64), a.base, rot, False)
    for n, j in enumerate(PLACES):
        if part == "latent":
            ql[first + n] = 0.7 * ref.rms_norm(kv[j, :rank].astype(np.float64), 1.0, 1e-5)
        else:  # the query that, rotated at its own place, meets the key rotated at place j
            half = rot // 2
            angle = (first + n) * a.base ** (-2.0 * np.arange(half) / rot)
            u, v = 4.0 * turned[j, 0, :half], 4.0 * turned[j, 0, half:]
            qr[first + n] = np.concatenate([u * np.cos(angle) + v * np.sin(angle), v * np.cos(angle) - u * np.sin(angle)])
    x = (to_bf16(ql), to_bf16(qr), kv)
    want = a.want(*x, first=first)
    if decode:
        a.step([(0, *piece(x, 0, first))])
        got = np.concatenate([a.step([(0, *piece(x, i, i + 1))])[0] for i in range(first, T)])
    else:
        got = a.step([(0, *x)])[0][first:]
    latent = ref.rms_norm(kv[:, :rank].astype(np.float64), a.w.astype(np.float64), a.eps)
    for n, j in enumerate(PLACES):
        assert np.abs(want[n] - latent[j]).max() < 0.2  # the test shows what it means to show
        assert np.abs(got[n] - want[n]).max() < (1e-4 if kind == "f32" else 6e-2), j


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_used_pages_hold_nothing_of_their_last_owner(kind):
    a = Latent(kind, 3, 48, 16, pages=3)
    for seq in range(4):
        x = a.random(130, seed=seq)
        got = np.concatenate(a.step([(seq, *piece(x, 0, 100))]) + [a.step([(seq, *piece(x, t, t + 1))])[0] for t in range(100, 130)])
        assert row_err(got, a.want(*x)).max() < (1e-5 if kind == "f32" else 1.5e-2)
        a.release(seq)


def test_bad_page_tables_are_reported():
    a = Latent("bf16", 2, 16, 16, pages=3)
    a.free = [5]
    with pytest.raises(Exception, match="out of range"):
        a.step([(0, *a.random(2))])


# ───────────────────────────── selective scan ─────────────────────────────
class Scan:
    """A selective scan node with its state on the device. The projections inside are chosen by the caller."""

    def __init__(self, kind, inner, state, rank, taps, slots=4, extra=8, seed=0):
        dt = self.dt = DTYPES[kind]
        self.kind, self.inner, self.extra = kind, inner, extra
        r = np.random.default_rng(seed)
        self.w = {"conv": to_bf16(r.standard_normal((inner, taps)) / np.sqrt(taps)), "conv.b": to_bf16(0.3 * r.standard_normal(inner)),
                  "x": to_bf16(2 * r.standard_normal((rank + 2 * state, inner)) / np.sqrt(inner)), "dt": to_bf16(r.standard_normal((inner, rank)) / np.sqrt(rank)),
                  "dt.b": to_bf16(r.uniform(-5, 0.5, inner)), "A_log": to_bf16(r.uniform(-5, 1, (inner, state))), "D": to_bf16(1 + 0.2 * r.standard_normal(inner))}
        b = ir.GraphBuilder()
        N, R = b.sym("num_tokens"), b.sym("num_seqs")
        A = -np.exp(self.w["A_log"].astype(np.float64))
        shapes = ([slots, taps, inner], [slots, inner, state])
        outs = b.composite("onyxia.SelectiveScan", {"width": inner, "state": state, "rank": rank, "taps": taps, "x_offset": extra + inner, "z_offset": extra},
                           [b.input("proj", dt, [N, extra + 2 * inner]), b.constant(f32(self.w["conv"])), b.constant(f32(self.w["conv.b"])), b.constant(act(self.w["x"], dt)),
                            b.constant(act(self.w["dt"], dt)), b.constant(f32(self.w["dt.b"])), b.constant(f32(A)), b.constant(f32(self.w["D"])),
                            b.input("ring", dt, shapes[0]), b.input("state", ir.F32, shapes[1]), b.input("seqs", ir.I32, [R, 4])],
                           [(dt, [N, inner]), (dt, shapes[0]), (ir.F32, shapes[1])])
        for n, v in zip(("out", "ring2", "state2"), outs):
            b.output(n, v)
        self.s = cuda_backend().prepare(b.finish())
        self.state = [self.s.upload(act(np.full(shapes[0], 50.0), dt)), self.s.upload(f32(np.full(shapes[1], 50.0)))]

    def step(self, entries):
        """entries: [((x, z), past, slot)]"""
        rows, info, at = [], [], 0
        for (x, z), past, slot in entries:
            rows.append(np.concatenate([np.full((len(x), self.extra), 9.0), z, x], axis=1))
            info.append([at, len(x), past, slot])
            at += len(x)
        out = dict(self.s.run({"proj": self.s.upload(act(np.concatenate(rows), self.dt)), "seqs": self.s.upload(i32(info)), "ring": self.state[0], "state": self.state[1]}))
        self.state = [out["ring2"], out["state2"]]
        o = self.s.download(out["out"]).numpy()
        return [o[i[0]:i[0] + i[1]] for i in info]

    def random(self, T, seed=0):
        r = np.random.default_rng([seed, self.inner])
        return tuple(to_bf16(r.standard_normal((T, self.inner))) for _ in range(2))

    def want(self, x, z):
        w = {k: v.astype(np.float64) for k, v in self.w.items()}
        u = ref.causal_conv(x.astype(np.float64), w["conv"], w["conv.b"])
        u = u * ref.sigmoid(u)
        if self.kind == "bf16":  # what the products read, and what they hand on
            u = to_bf16(u).astype(np.float64)
        p, rank = u @ w["x"].T, w["dt"].shape[1]
        if self.kind == "bf16":
            p = to_bf16(p).astype(np.float64)
        n = w["A_log"].shape[1]
        dt = ref.softplus(p[:, :rank] @ w["dt"].T + w["dt.b"])
        return ref.selective_scan(u, dt, -np.exp(w["A_log"]), p[:, rank:rank + n], p[:, rank + n:], w["D"]) * z

    def check(self, x, got):
        got, want = np.concatenate(got), self.want(*x)
        rms = lambda a: np.sqrt((a ** 2).mean(axis=1))
        err = rms(got - want) / np.maximum(rms(want), np.sqrt((want ** 2).mean()))  # results grow with the state
        assert err.max() < (1e-5 if self.kind == "f32" else 1e-2), (int(err.argmax()), float(err.max()))


SCANS = [(64, 8, 4, 4), (96, 16, 8, 4), (320, 64, 16, 4), (30, 5, 3, 3), (21, 20, 1, 1), (48, 128, 40, 2), (40, 256, 8, 4), (2560, 16, 32, 4), (72, 1, 2, 5), (24, 33, 7, 8)]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("inner,state,rank,taps", SCANS)
def test_scan_alone(kind, inner, state, rank, taps):
    """Portions of all sizes and decoded tokens, beside another sequence; slots are dirty and used again."""
    a = Scan(kind, inner, state, rank, taps)
    T = 330 if inner < 1000 else 150
    x, y = a.random(T), a.random(T, seed=1)
    a.check(x, a.step([(x, 0, 2)]))  # slot 2 is dirty afterwards
    got, got2, at, at2 = [], [], 0, 0
    for n in (1, 1, 2, 3, 63, 1, 64, 2, 1, 65, 5, 1, 100):
        n = min(n, T - at)
        if not n:
            break
        m = 1 if at2 % 3 else 2
        o = a.step([(piece(x, at, at + n), at, 2), (piece(y, at2, at2 + m), at2, 0)])
        got.append(o[0])
        got2.append(o[1])
        at, at2 = at + n, at2 + m
    while at < T:
        o = a.step([(piece(x, at, at + 1), at, 2), (piece(y, at2, at2 + 1), at2, 0)])
        got.append(o[0])
        got2.append(o[1])
        at, at2 = at + 1, at2 + 1
    a.check(x, got)
    a.check(piece(y, 0, at2), got2)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("portions", [[400], [64, 1, 200, 135], [33, 1, 1, 300], [7]])
def test_a_single_token_stays_in_the_state(kind, portions):
    """One token far above the others in channels that hardly forget: it shows at every distance, across tile edges and portions."""
    a = Scan(kind, 64, 16, 4, 4)
    for place in (0, 31, 32, 33, 63, 64, 127):
        x, z = a.random(400)
        x = to_bf16(0.01 * x)
        x[place] = 8.0
        z = to_bf16(np.sign(z))
        want = a.want(x, z)
        quiet = a.want(np.where(np.arange(400)[:, None] == place, to_bf16(np.float32(0.01)), x), z)
        assert np.abs(want[place + 200] - quiet[place + 200]).max() > 0.1  # the test shows what it means to show
        got, at = [], 0
        while at < 400:
            n = min(portions[min(len(got), len(portions) - 1)], 400 - at)
            got.append(a.step([(piece((x, z), at, at + n), at, 1)])[0])
            at += n
        got = np.concatenate(got)
        for t in (place, place + 1, place + 3, place + 4, place + 64, place + 200):
            assert rel_err(got[t], want[t]) < (1e-5 if kind == "f32" else 1e-2), (place, t)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_many_portions_in_one_batch(kind):
    a = Scan(kind, 64, 16, 8, 4, slots=40)
    xs = [a.random(n, seed=n) for n in range(1, 36)] + [a.random(300, seed=99)]
    first = a.step([(piece(x, 0, (len(x[0]) + 1) // 2), 0, i) for i, x in enumerate(xs)])
    rest = [(i, x) for i, x in enumerate(xs) if len(x[0]) > 1]
    second = a.step([(piece(x, (len(x[0]) + 1) // 2, len(x[0])), (len(x[0]) + 1) // 2, i) for i, x in rest])
    for (i, x), o in zip(rest, second):
        a.check(x, [first[i], o])


@pytest.mark.parametrize("count", [1, 3, 8, 9, 33])
def test_decode_batches_of_the_scan(count):
    a = Scan("bf16", 96, 16, 8, 4, slots=40)
    xs = [a.random(12, seed=n) for n in range(count)]
    got = [[o] for o in a.step([(piece(x, 0, 5), 0, 39 - i) for i, x in enumerate(xs)])]
    for t in range(5, 12):
        for g, o in zip(got, a.step([(piece(x, t, t + 1), t, 39 - i) for i, x in enumerate(xs)])):
            g.append(o)
    for x, g in zip(xs, got):
        a.check(x, g)


# ───────────────────────────── whole models ───────────────────────────────
@functools.lru_cache(maxsize=None)
def session(name, kind):
    c, w = util.model(name)
    return cuda_backend().prepare(zusitar.build(zusitar.ZusitarConfig.from_dict(c), checkpoint.Weights.from_f32(w), DTYPES[kind]))


def engine(name, kind, max_tokens=2048, max_seqs=4):
    return Engine(session(name, kind), max_tokens, max_seqs)


def feed(e, seq, toks, portions):
    """All logits of `toks`, in portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(portions[min(i, len(portions) - 1)], len(toks) - at)
        out.append(e.forward([(seq, toks[at:at + n], range(n))]))
        at, i = at + n, i + 1
    return np.concatenate(out)


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("portions", [[150], [1], [2], [3, 1, 1, 70, 2, 1], [64, 63, 5], [65, 1], [40, 9]])
def test_prompts_and_portions(name, kind, portions):
    toks = util.tokens(name, 150)
    err = util.distance(feed(engine(name, kind), 0, toks, portions), util.expected(name, 150))
    assert err.max() < TOL[kind], (float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_long_decoding(kind):
    toks = util.tokens("mixed", 420)
    err = util.distance(feed(engine("mixed", kind), 0, toks, [90, 1]), util.expected("mixed", 420))
    assert err.max() < TOL[kind], (float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_ragged_batches_and_reuse(name, kind):
    """Up to four of nine sequences live at once in a pool that is just large enough; each must match itself alone."""
    r = np.random.default_rng(4)
    lengths = [1, 23, 150, 64, 2, 97, 130, 65, 150]
    seqs = {i: util.tokens(name, n, seed=i) for i, n in enumerate(lengths)}
    got = {i: [] for i in seqs}
    e = engine(name, kind, max_tokens=64 * 9, max_seqs=4)
    waiting, live, fed = list(seqs), [], {i: 0 for i in seqs}
    total = e.stats()["free_pages"]
    pages = lambda i: -(-len(seqs[i]) // 64)
    while waiting or live:
        while waiting and len(live) < 4 and sum(map(pages, live)) + pages(waiting[0]) <= total:
            live.append(waiting.pop(0))
        entries = []
        for i in live:
            if len(live) > 1 and r.random() < 0.2:
                continue  # left out of this step
            n = min(int(r.choice([1, 1, 1, 2, 3, 29, 64])), len(seqs[i]) - fed[i])
            entries.append((i, seqs[i][fed[i]:fed[i] + n], range(n)))
        if not entries:
            continue
        out, at = e.forward(entries), 0
        for i, t, _ in entries:
            got[i].append(out[at:at + len(t)])
            at += len(t)
            fed[i] += len(t)
        for i in [i for i in live if fed[i] == len(seqs[i])]:
            e.release(i)
            live.remove(i)
    assert e.stats()["free_pages"] == total and e.stats()["free_slots"] == 4
    for i, n in enumerate(lengths):
        err = util.distance(np.concatenate(got[i]), util.expected(name, n, token_seed=i))
        assert err.max() < TOL[kind] * (2 if n < 3 else 1), (i, n, float(err.max()), int(err.argmax()))


def test_wide_decode_batches():
    """Twelve to forty sequences decoding together: the other products."""
    for count in (12, 20, 40):
        e = engine("mixed", "bf16", max_tokens=64 * count, max_seqs=count)
        seqs = [util.tokens("mixed", 12, seed=i) for i in range(count)]
        e.forward([(i, s[:4 + i % 3], []) for i, s in enumerate(seqs)])
        at = [4 + i % 3 for i in range(count)]
        for _ in range(5):
            out = e.forward([(i, [s[at[i]]], [0]) for i, s in enumerate(seqs)])
            for i, s in enumerate(seqs):
                err = util.distance(out[i][None], util.expected("mixed", 12, token_seed=i)[at[i]][None])
                assert err[0] < TOL["bf16"] * 2
                at[i] += 1


# ───────────────────────────── generation ─────────────────────────────────
def greedy_plain(name, prompt, n):
    c, w = util.model(name)
    toks = list(prompt)
    for _ in range(n):
        logits = ref.forward(c, w, toks)[-1]
        top = np.sort(logits)[-2:]
        assert top[1] - top[0] > 1e-3, "an argmax this close proves nothing"
        toks.append(int(np.argmax(logits)))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    prompts = [util.tokens("mixed", n, seed=20 + n) for n in (5, 70, 33, 1, 18)]
    want = [greedy_plain("mixed", p, 6) for p in prompts]
    for budget in (7, 2048):  # portions of seven tokens; everything at once
        e = engine("mixed", "f32", max_tokens=320, max_seqs=3)
        assert e.generate(prompts, 6, token_budget=budget) == want
        assert e.stats()["free_pages"] == 5 and e.stats()["free_slots"] == 3


def test_the_single_sequence_loop_serves_it_too():
    c, w = util.model("mixed")
    prompt = util.tokens("mixed", 30, seed=9)
    want = greedy_plain("mixed", prompt, 5)
    s = llm.NativeLlmSession(cuda_backend(), zusitar.build(zusitar.ZusitarConfig.from_dict(c), checkpoint.Weights.from_f32(w), ir.F32), 128)
    assert s.generate(prompt, 5) == want
    s.reset()
    got = [s.step_greedy(prompt)]
    for _ in range(4):
        got.append(s.step_greedy([got[-1]]))
    assert got == want and s.sequence_length() == 34


def test_command_line(tmp_path):
    c, w = util.model("mixed")
    with open(tmp_path / "config.json", "w") as f:
        json.dump(c, f)
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), checkpoint.Weights.from_bf16(
        {k: checkpoint.Weights.from_f32({k: v}).bf16_bits(k) for k, v in w.items()}))
    prompt = util.tokens("mixed", 12, seed=2)
    r = subprocess.run([sys.executable, "-m", "onyxia_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                        ",".join(map(str, prompt)), "-n", "4", "--max-tokens", "256", "--max-seqs", "2"],
                       cwd=ROOT, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(v) for v in r.stdout.split()] == greedy_plain("mixed", prompt, 4)
    # the same prompt replayed as a trace
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompt[:7], "want": []}, {"id": "b", "tokens": prompt, "want": [11]}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": prompt[7:], "want": [0, 4]}], "end": ["a"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), cwd=str(tmp_path), stdout=subprocess.PIPE, stderr=subprocess.PIPE,
                       text=True, timeout=300)
    assert r.returncode == 0 and r.stdout.split("\n")[:2] == ["done 0", "done 1"], r.stderr[-2000:]
    want = ref.forward(c, w, prompt)
    for step, places in ((0, [11]), (1, [7, 11])):
        got = np.fromfile(tmp_path / f"{step}.f32", np.float32).reshape(len(places), -1)
        assert util.distance(got, want[places]).max() < TOL["f32"]
