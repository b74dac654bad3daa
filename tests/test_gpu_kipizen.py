"""Kipizen on the device against the plain implementation (kipizen_ref.py): each mechanism alone through a module of its
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

import kipizen_ref as ref
import kipizen_util as util
from gpu_util import cuda_backend
from kipizen_util import to_bf16
from onyxia_b200 import backend as be
from onyxia_b200 import checkpoint, ir, kipizen, llm
from onyxia_b200.engine import Engine
from onyxia_b200.ir import HostTensor

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"f32": ir.F32, "bf16": ir.BF16}
TOL = {"f32": 1e-5, "bf16": 3e-2}


def act(a, dtype):
    return HostTensor.bf16(a) if dtype == ir.BF16 else HostTensor.from_numpy(np.asarray(a, np.float32))


def f32(a):
    return HostTensor.from_numpy(np.ascontiguousarray(a, np.float32))


def rel_err(got, want):
    return float(np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want ** 2).mean()))


def row_err(got, want):
    """Per token: root mean square of the difference over that of the reference."""
    axes = tuple(range(1, want.ndim))
    return np.sqrt(((got - want) ** 2).mean(axis=axes)) / np.sqrt((want ** 2).mean())


# ───────────────────────────── products with functions, norms of sums, gates ─
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 8, 9, 32, 33, 150])
def test_functions_of_column_ranges(kind, rows):
    r = np.random.default_rng(rows)
    dt = DTYPES[kind]
    for k, n, split in ((64, 96, 40), (520, 131, 100), (18, 12, 5)):
        x, w, bias = to_bf16(r.standard_normal((rows, k))), to_bf16(r.standard_normal((n, k)) / np.sqrt(k)), to_bf16(r.standard_normal(n))
        b = ir.GraphBuilder()
        for name, first, rest in (("a", "silu", "sigmoid"), ("b", "none", "silu"), ("c", "sigmoid", "none")):
            b.output(name, b.composite("onyxia.Linear", {"bias": 1, "act": first, "act_rest": rest, "act_split": split},
                                       [b.input("x" + name, dt, [rows, k]), b.constant(act(w, dt)), b.constant(f32(bias))], [(ir.F32, [rows, n])])[0])
        got = {name: v.numpy() for name, v in be.run_once(cuda_backend(), b.finish(), {"x" + n2: act(x, dt) for n2 in "abc"})}
        z = x.astype(np.float64) @ w.T.astype(np.float64) + bias
        fs = {"none": lambda v: v, "silu": ref.silu, "sigmoid": ref.sigmoid}
        for name, first, rest in (("a", "silu", "sigmoid"), ("b", "none", "silu"), ("c", "sigmoid", "none")):
            want = np.concatenate([fs[first](z[:, :split]), fs[rest](z[:, split:])], axis=1)
            assert rel_err(got[name], want) < 3e-6, (k, name)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 2, 4, 7, 8, 9, 40])
def test_norm_of_a_sum_in_front_of_a_product(kind, rows):
    r = np.random.default_rng(rows)
    dt, eps, scale = DTYPES[kind], 1e-3, 2.7
    for width, n in ((96, 64), (1160, 40), (50, 30)):
        for has_res, y_dt in ((1, ir.F32), (0, dt)):
            y, res = to_bf16(0.02 * r.standard_normal((rows, width))), (0.02 * r.standard_normal((rows, width))).astype(np.float32)
            w, m = to_bf16(r.standard_normal(width)), to_bf16(r.standard_normal((n, width)))
            b = ir.GraphBuilder()
            ins = [b.input("y", y_dt, [rows, width]), b.constant(f32(w))]
            feed = {"y": act(y, y_dt)}
            if has_res:
                ins.append(b.input("res", ir.F32, [rows, width]))
                feed["res"] = f32(res)
            attrs = {"epsilon": eps, "residual": has_res, "pre": 1, "y_scale": scale}
            b.output("alone", b.composite("onyxia.ResidualNorm", attrs, ins, [(ir.F32, [rows, width])])[0])
            out, stream = b.composite("onyxia.Linear", dict(attrs, norm=1), ins + [b.constant(act(m, dt))], [(ir.F32, [rows, n]), (ir.F32, [rows, width])])
            b.output("out", out)
            b.output("stream", stream)
            got = {k: v.numpy() for k, v in be.run_once(cuda_backend(), b.finish(), feed)}
            total = y.astype(np.float64) * scale + (res if has_res else 0.0)
            want = ref.unit_rms(total, eps) * w
            assert rel_err(got["alone"], want) < 1e-6 and rel_err(got["stream"], total) < 1e-6
            assert rel_err(got["out"], want @ m.T.astype(np.float64)) < (2e-6 if kind == "f32" else 5e-3)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 70])
@pytest.mark.parametrize("width,offset,cols", [(96, 40, 160), (50, 7, 61), (264, 264, 528)])
def test_gated_norm_in_front_of_a_product(kind, rows, width, offset, cols):
    r = np.random.default_rng(rows)
    dt = DTYPES[kind]
    y, w, m = r.standard_normal((rows, width)).astype(np.float32), to_bf16(r.standard_normal(width)), to_bf16(r.standard_normal((24, width)))
    gate = to_bf16(r.standard_normal((rows, cols)))
    b = ir.GraphBuilder()
    b.output("out", b.composite("onyxia.Linear", {"norm": 1, "stream": 0, "epsilon": 1e-5, "gate": 1, "gate_offset": offset},
                                [b.input("y", ir.F32, [rows, width]), b.constant(f32(w)), b.input("gate", dt, [rows, cols]), b.constant(act(m, dt))],
                                [(ir.F32, [rows, 24])])[0])
    got = be.run_once(cuda_backend(), b.finish(), {"y": f32(y), "gate": act(gate, dt)})[0][1].numpy()
    want = (ref.unit_rms(y.astype(np.float64), 1e-5) * w * gate[:, offset:offset + width]) @ m.T.astype(np.float64)
    assert rel_err(got, want) < (2e-6 if kind == "f32" else 5e-3)


# ───────────────────────────── experts ────────────────────────────────────
class Experts:
    def __init__(self, kind, width, experts, top, ff, seed=0, bias=None):
        r = np.random.default_rng(seed)
        self.kind, self.dt, self.width, self.c = kind, DTYPES[kind], width, {"router": {"experts": experts, "top": top}}
        self.w = {"router": to_bf16(r.standard_normal((experts, width)) / np.sqrt(width)),
                  "router.b": to_bf16(r.standard_normal(experts) if bias is None else bias)}
        for e in range(experts):
            self.w.update({f"e{e}.gate": to_bf16(2 * r.standard_normal((ff, width)) / np.sqrt(width)), f"e{e}.up": to_bf16(2 * r.standard_normal((ff, width)) / np.sqrt(width)),
                           f"e{e}.down": to_bf16(r.standard_normal((width, ff)) / np.sqrt(ff))})
        up = np.stack([np.stack([self.w[f"e{e}.gate"], self.w[f"e{e}.up"]], axis=1) for e in range(experts)]).reshape(-1, width)
        down = np.concatenate([self.w[f"e{e}.down"] for e in range(experts)])
        b = ir.GraphBuilder()
        N = b.sym("n")
        y, x = b.composite("onyxia.MixtureOfExperts", {"experts": experts, "top": top, "ff": ff, "epsilon": 1e-12, "pre": 1, "y_scale": 1.0},
                           [b.input("x", ir.F32, [N, width]), b.constant(f32(np.ones(width))), b.constant(act(self.w["router"], self.dt)),
                            b.constant(f32(self.w["router.b"])), b.constant(act(up, self.dt)), b.constant(act(down, self.dt))],
                           [(ir.F32, [N, width]), (ir.F32, [N, width])])
        b.output("y", y)
        b.output("x2", x)
        self.s = cuda_backend().prepare(b.finish())

    def rows(self, n, seed=0):
        """Rows whose choice of experts is no close call."""
        r, out = np.random.default_rng([seed, n]), []
        while len(out) < n:
            h = r.standard_normal(self.width).astype(np.float32)
            z = np.sort(self.w["router"].astype(np.float64) @ ref.unit_rms(h, 1e-12) + self.w["router.b"])[::-1]
            top = self.c["router"]["top"]
            if top == len(z) or z[top - 1] - z[top] > 0.02:
                out.append(h)
        return np.stack(out)

    def check(self, h):
        o = dict(self.s.run({"x": self.s.upload(f32(h))}))
        got, stream = self.s.download(o["y"]).numpy(), self.s.download(o["x2"]).numpy()
        want = ref.mixture(ref.unit_rms(h.astype(np.float64), 1e-12), {k: v.astype(np.float64) for k, v in self.w.items()}, self.c)
        assert np.array_equal(stream, h)
        err = row_err(got, want)
        assert err.max() < (1e-5 if self.kind == "f32" else 2e-2), (len(h), int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width,experts,top,ff", [(64, 8, 2, 40), (160, 40, 6, 64), (1032, 5, 1, 24), (64, 6, 6, 128), (36, 5, 3, 18), (128, 130, 8, 16), (72, 2, 1, 520)])
def test_experts_alone(kind, width, experts, top, ff):
    m = Experts(kind, width, experts, top, ff)
    for n in (1, 2, 7, 8, 9, 16, 20, 32, 33, 64, 150, 300):
        m.check(m.rows(n))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_experts_that_nobody_or_everybody_chooses(kind):
    for bias in ([30.0] + [0.0] * 7, [0.0] * 7 + [30.0], [30.0, 0, 0, 0, 0, 0, 0, 30.0], [-30.0, 0, 0, -30.0, 0, 0, -30.0, -30.0]):
        m = Experts(kind, 64, 8, 2, 48, bias=np.array(bias))
        for n in (1, 5, 32, 140):
            m.check(m.rows(n))


# ───────────────────────────── attention ──────────────────────────────────
class Attention:
    """An attention node with its pools on the device, and optionally a second one that reads the same pools with queries of
    its own; pages are handed out in a shuffled order."""

    def __init__(self, kind, heads, kv_heads, dim, vdim, *, scale=0.3, softcap=0.0, window=0, rot=0, base=100.0, factor=1.0, eps=1e-5, norm=1, sink=1,
                 shared=None, pages=40, extra=8):
        dt = self.dt = DTYPES[kind]
        self.kind, self.heads, self.kv, self.dim, self.vdim, self.extra, self.eps = kind, heads, kv_heads, dim, vdim, extra, eps
        self.kw = dict(scale=scale, softcap=softcap or None, window=window or None, sink=bool(sink))
        self.rot, self.norm, self.shared = (base, rot, factor), norm, shared
        b = ir.GraphBuilder()
        N, R, TW = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("table_width")
        self.ld = extra + (heads + kv_heads) * dim + kv_heads * vdim + heads * dim
        pools = [[pages, kv_heads, 64, dim], [pages, kv_heads, 64, vdim]]
        proj, turns = b.input("proj", dt, [N, self.ld]), b.constant(f32(kipizen.turns_per_position(rot, base, factor)))
        where = [b.input("seqs", ir.I32, [R, 4]), b.input("table", ir.I32, [R, TW])]
        attrs = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot_dims": rot, "window": window, "scale": float(scale),
                 "softcap": float(softcap), "epsilon": eps, "norm": norm, "sink": sink}
        outs = b.composite("onyxia.PagedKVAttention",
                           dict(attrs, q_offset=extra + kv_heads * dim, k_offset=extra, v_offset=extra + (heads + kv_heads) * dim),
                           [proj, turns, b.input("keys", dt, pools[0]), b.input("values", dt, pools[1])] + where,
                           [(dt, [N, heads * vdim]), (dt, pools[0]), (dt, pools[1])])
        names = ["out", "keys2", "values2"]
        if shared:
            attrs.update({"scale": float(shared["scale"]), "window": shared["window"]})
            outs += b.composite("onyxia.SharedKVAttention", dict(attrs, q_offset=self.ld - heads * dim), [proj, turns, outs[1], outs[2]] + where,
                                [(dt, [N, heads * vdim])])
            names.append("other")
        for name, v in zip(names, outs):
            b.output(name, v)
        self.s = cuda_backend().prepare(b.finish())
        self.pools = [self.s.upload(act(np.full(p, 99.0), dt)) for p in pools]
        self.free = np.random.default_rng(1).permutation(pages).tolist()
        self.owned, self.past = {}, {}

    def release(self, seq):
        self.free += self.owned.pop(seq)
        del self.past[seq]

    def step(self, entries, output="out"):
        """entries: [(sequence, q [n, H, d], k [n, G, d], v [n, G, dv])] → outputs per entry. The second node's queries are −q."""
        rows, info, at = [], [], 0
        for seq, q, k, v in entries:
            n, past = len(q), self.past.setdefault(seq, 0)
            own = self.owned.setdefault(seq, [])
            while len(own) * 64 < past + n:
                own.append(self.free.pop())
            info.append([at, n, past, 0])
            rows.append(np.concatenate([np.full((n, self.extra), 7.0), k.reshape(n, -1), q.reshape(n, -1), v.reshape(n, -1), -q.reshape(n, -1)], axis=1))
            at += n
            self.past[seq] = past + n
        tw = max(len(self.owned[e[0]]) for e in entries)
        table = [self.owned[e[0]] + [0] * (tw - len(self.owned[e[0]])) for e in entries]
        out = dict(self.s.run({"proj": self.s.upload(act(np.concatenate(rows), self.dt)), "keys": self.pools[0], "values": self.pools[1],
                               "seqs": self.s.upload(HostTensor.from_numpy(np.array(info, np.int32))),
                               "table": self.s.upload(HostTensor.from_numpy(np.array(table, np.int32)))}))
        self.pools = [out["keys2"], out["values2"]]
        o = self.s.download(out[output]).numpy().reshape(-1, self.heads, self.vdim)
        return [o[i[0]:i[0] + i[1]] for i in info]

    def want(self, q, k, v, **kw):
        def place(x):
            x = ref.rotate(x.astype(np.float64), self.rot[0], self.rot[1], self.rot[2])
            return ref.unit_rms(x, self.eps) if self.norm else x
        return ref.attention(place(q), place(k), v.astype(np.float64), **dict(self.kw, **kw))

    def random(self, T, seed=0):
        r = np.random.default_rng([seed, self.dim])
        return tuple(to_bf16(r.standard_normal((T, n, d))) for n, d in ((self.heads, self.dim), (self.kv, self.dim), (self.kv, self.vdim)))


def piece(x, lo, hi):
    return tuple(a[lo:hi] for a in x)


SHAPES = [  # heads, kv heads, dim, vdim, rotating dims, window
    (4, 2, 16, 16, 16, 40), (3, 3, 64, 32, 20, 64), (20, 1, 72, 136, 72, 100), (8, 1, 128, 128, 64, 0), (2, 1, 256, 256, 2, 65), (5, 5, 10, 6, 4, 33),
    (2, 2, 300, 20, 300, 90), (6, 3, 96, 88, 0, 1), (12, 1, 48, 64, 48, 2)]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,window", SHAPES)
def test_attention_alone(kind, heads, kv, dim, vdim, rot, window):
    """A prompt in uneven portions, then decoded tokens, beside two other sequences at other lengths."""
    T = 200
    a = Attention(kind, heads, kv, dim, vdim, scale=2.0 / np.sqrt(dim), softcap=3.0, window=window, rot=rot, factor=4.0)
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
@pytest.mark.parametrize("sink,norm,softcap", [(0, 1, 5.0), (1, 0, 0.0), (0, 0, 0.0)])
def test_attention_parts_left_out(kind, sink, norm, softcap):
    a = Attention(kind, 4, 2, 32, 32, scale=0.3, softcap=softcap, window=50, rot=16, sink=sink, norm=norm)
    x = a.random(150)
    want = a.want(*x)
    got = a.step([(0, *piece(x, 0, 130))]) + [a.step([(0, *piece(x, t, t + 1))])[0] for t in range(130, 150)]
    err = row_err(np.concatenate(got), want)
    assert err.max() < (1e-5 if kind == "f32" else 1.5e-2), (int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
def test_long_contexts(kind, decode):
    """Keys split over many CTAs and pages; the window reaches over some of them or over all."""
    for window in (0, 1500):
        a = Attention(kind, 2, 1, 64, 64, scale=0.5, softcap=10.0, window=window, rot=64, base=10000.0)
        T = 2100
        x = a.random(T)
        x = (x[0] * np.where(np.arange(T) < T - 8, 0, 1)[:, None, None], x[1], x[2])  # only the last queries matter
        low = 0 if not window else T - 8 - window
        q, k, v = x
        kk = ref.unit_rms(ref.rotate(k[low:].astype(np.float64), 10000.0, 64, first=low), a.eps)
        qq = ref.unit_rms(ref.rotate(q[T - 8:].astype(np.float64), 10000.0, 64, first=T - 8), a.eps)
        want = ref.attention(np.concatenate([np.zeros((len(kk) - 8, 2, 64)), qq]), kk, v[low:].astype(np.float64), **a.kw)[-8:]
        a.step([(0, *piece(x, 0, T - 8))])
        got = np.concatenate([a.step([(0, *piece(x, t, t + 1))])[0] for t in range(T - 8, T)]) if decode else a.step([(0, *piece(x, T - 8, T))])[0]
        err = row_err(got, want)
        assert err.max() < (2e-5 if kind == "f32" else 1.5e-2), (window, float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [0, 63, 64, 65, 130])
def test_single_keys_stand_out(kind, decode, window):
    """One key carries nearly all the weight, just inside or just outside a query's window: its value is the output, or none of it."""
    r = np.random.default_rng(5)
    heads, kv, dim, T, first = 4, 2, 32, 420, 400
    a = Attention(kind, heads, kv, dim, dim, scale=1.0, softcap=25.0, window=window, rot=0)
    _, k, v = a.random(T)
    k, q = to_bf16(np.sign(k)), to_bf16(0.01 * r.standard_normal((T, heads, dim)))
    reach = window or T
    places = {}
    for n, i in enumerate(range(first, T)):
        j = [i, i - reach + 1, i - reach, i - reach - 1, i - 1, i - reach // 2, 0, 1, 63, 64, 65, 127, 128, 255, 256, 319, 320, 383, 384, 399][n]
        places[i] = j = min(max(j, 0), i)
        q[i] = np.repeat(k[j], heads // kv, axis=0)
    want = a.want(q, k, v)
    for i, j in places.items():
        inside = not window or i - j < window
        near = np.abs(want[i] - np.repeat(v[j], heads // kv, axis=0)).max() < 0.2
        assert near == inside, (i, j)  # the test shows what it means to show
    if decode:
        a.step([(0, *piece((q, k, v), 0, first))])
        got = {i: a.step([(0, *piece((q, k, v), i, i + 1))])[0][0] for i in places}
    else:
        out = a.step([(0, q, k, v)])[0]
        got = {i: out[i] for i in places}
    for i, j in places.items():
        assert np.abs(got[i] - want[i]).max() < (1e-4 if kind == "f32" else 4e-2), (i, j)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_the_sink_takes_its_share(kind):
    """Few keys with scores far below zero: without the sink their values would come out in full."""
    a = Attention(kind, 2, 1, 16, 16, scale=1.0, softcap=4.0, window=3)
    k = to_bf16(np.ones((70, 1, 16)))
    q, v = to_bf16(-np.ones((70, 2, 16))), to_bf16(np.full((70, 1, 16), 100.0))
    want = a.want(q, k, v)
    assert 0 < want.min() and want.max() < 6.0
    got = np.concatenate([a.step([(0, *piece((q, k, v), 0, 60))])[0]] + [a.step([(0, *piece((q, k, v), t, t + 1))])[0] for t in range(60, 70)])
    assert np.abs(got / want - 1).max() < (1e-5 if kind == "f32" else 1e-2)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_two_layers_over_the_same_pools(kind):
    """The second node attends to what the first one stores in the same step, with other queries, scale and window."""
    a = Attention(kind, 4, 2, 32, 48, scale=0.4, softcap=5.0, window=20, rot=16, shared={"scale": 0.9, "window": 75})
    x = a.random(160)
    want = a.want(-x[0], x[1], x[2], scale=0.9, window=75)
    got, at = [], 0
    for n in (70, 2, 1, 1, 40, 1):
        got.append(a.step([(5, *piece(x, a.past.get(5, 0), a.past.get(5, 0) + 1)), (0, *piece(x, at, at + n))], "other")[1])
        at += n
    while at < 160:
        got.append(a.step([(0, *piece(x, at, at + 1))], "other")[0])
        at += 1
    err = row_err(np.concatenate(got), want)
    assert err.max() < (1e-5 if kind == "f32" else 1.5e-2), (int(err.argmax()), float(err.max()))


def test_used_pages_hold_nothing_of_their_last_owner():
    a = Attention("f32", 2, 1, 16, 16, window=100, rot=8, pages=3)
    for seq in range(4):
        x = a.random(130, seed=seq)
        got = np.concatenate(a.step([(seq, *piece(x, 0, 100))]) + [a.step([(seq, *piece(x, t, t + 1))])[0] for t in range(100, 130)])
        assert row_err(got, a.want(*x)).max() < 1e-5
        a.release(seq)


def test_bad_page_tables_are_reported():
    a = Attention("bf16", 2, 2, 16, 16, pages=3)
    a.free = [5]
    with pytest.raises(Exception, match="out of range"):
        a.step([(0, *a.random(2))])


def test_angles_far_away():
    """Positions whose angles are thousands of turns: the rotation is as exact there as at the start."""
    dims, base = 16, 10000.0
    turns = kipizen.turns_per_position(dims, base, 3.0)
    b = ir.GraphBuilder()
    outs = b.composite("onyxia.PagedKVAttention",
                       {"heads": 1, "kv_heads": 1, "dim": dims, "vdim": 16, "q_offset": 0, "k_offset": dims, "v_offset": 2 * dims, "rot_dims": dims, "norm": 0,
                        "window": 4},
                       [b.input("proj", ir.F32, [2, 48]), b.constant(f32(turns)), b.input("k", ir.F32, [1, 1, 65536 * 4, dims]),
                        b.input("v", ir.F32, [1, 1, 65536 * 4, 16]), b.input("seqs", ir.I32, [1, 4]), b.input("table", ir.I32, [1, 1])],
                       [(ir.F32, [2, 16]), (ir.F32, [1, 1, 65536 * 4, dims]), (ir.F32, [1, 1, 65536 * 4, 16])])
    for n, v in zip(("out", "k2", "v2"), outs):
        b.output(n, v)
    s = cuda_backend().prepare(b.finish())
    proj = np.random.default_rng(0).standard_normal((2, 48)).astype(np.float32)
    for past in (0, 1000, 200003):
        out = dict(s.run({"proj": s.upload(f32(proj)), "k": s.upload(f32(np.zeros((1, 1, 65536 * 4, dims)))),
                          "v": s.upload(f32(np.zeros((1, 1, 65536 * 4, 16)))), "seqs": s.upload(HostTensor.from_numpy(np.array([[0, 2, past, 0]], np.int32))),
                          "table": s.upload(HostTensor.from_numpy(np.zeros((1, 1), np.int32)))}))
        keys = s.download(out["k2"]).numpy()[0, 0, past:past + 2]
        for i in range(2):
            a = (past + i) * base ** (-2.0 * np.arange(8) / dims) / 3.0
            u, v = proj[i, dims:dims + 8].astype(np.float64), proj[i, dims + 8:2 * dims].astype(np.float64)
            want = np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)])
            assert np.abs(keys[i] - want).max() < 2e-6, past


# ───────────────────────────── lightning attention ────────────────────────
class Lightning:
    def __init__(self, kind, decay, dim, vdim, slots=4, extra=8):
        dt = self.dt = DTYPES[kind]
        self.kind, self.heads, self.dim, self.vdim, self.decay, self.extra = kind, len(decay), dim, vdim, np.asarray(decay), extra
        H = self.heads
        b = ir.GraphBuilder()
        N, R = b.sym("num_tokens"), b.sym("num_seqs")
        shape = [slots, H, dim, vdim]
        outs = b.composite("onyxia.LightningAttention",
                           {"heads": H, "dim": dim, "vdim": vdim, "v_offset": extra, "q_offset": extra + H * vdim, "k_offset": extra + H * (vdim + dim)},
                           [b.input("proj", dt, [N, extra + H * (2 * dim + vdim)]), b.constant(f32(kipizen.decay_table(decay))), b.input("state", ir.F32, shape),
                            b.input("seqs", ir.I32, [R, 4])], [(ir.F32, [N, H * vdim]), (ir.F32, shape)])
        b.output("out", outs[0])
        b.output("state2", outs[1])
        self.s = cuda_backend().prepare(b.finish())
        self.state = self.s.upload(f32(np.full(shape, 50.0)))

    def step(self, entries):
        """entries: [((q, k, v), past, slot)]"""
        rows, info, at = [], [], 0
        for (q, k, v), past, slot in entries:
            n = len(q)
            rows.append(np.concatenate([np.full((n, self.extra), 9.0), v.reshape(n, -1), q.reshape(n, -1), k.reshape(n, -1)], axis=1))
            info.append([at, n, past, slot])
            at += n
        out = dict(self.s.run({"proj": self.s.upload(act(np.concatenate(rows), self.dt)), "seqs": self.s.upload(HostTensor.from_numpy(np.array(info, np.int32))),
                               "state": self.state}))
        self.state = out["state2"]
        o = self.s.download(out["out"]).numpy().reshape(-1, self.heads, self.vdim)
        return [o[i[0]:i[0] + i[1]] for i in info]

    def random(self, T, seed=0):
        r = np.random.default_rng([seed, self.dim])
        return tuple(to_bf16(r.standard_normal((T, self.heads, d))) for d in (self.dim, self.dim, self.vdim))

    def want(self, q, k, v):
        return ref.decayed_state(q.astype(np.float64), k.astype(np.float64), v.astype(np.float64), self.decay)

    def check(self, x, got):
        err = row_err(np.concatenate(got), self.want(*x))
        # chunks keep 16 bits of what is not bf16 already
        assert err.max() < (2e-6 if self.kind == "f32" else 3e-5), (int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decay,dim,vdim", [([0.6, 0.95, 0.999], 32, 32), ([1.0, 0.0], 16, 48), ([0.99], 128, 128), ([0.9, 0.8], 7, 5), ([0.97], 264, 40),
                                            ([0.97, 0.3], 256, 72), ([0.5], 24, 200), ([0.9], 40, 6), ([0.98], 400, 24)])
def test_lightning_alone(kind, decay, dim, vdim):
    """Portions of all sizes and decoded tokens, beside another sequence; slots are dirty and used again."""
    a = Lightning(kind, decay, dim, vdim)
    x, y = a.random(330), a.random(330, seed=1)
    a.check(x, a.step([(x, 0, 2)]))  # slot 2 is dirty afterwards
    got, got2, at, at2 = [], [], 0, 0
    for n in (1, 1, 2, 3, 63, 1, 64, 65, 5, 1, 100):
        m = 1 if at2 % 3 else 2
        o = a.step([(piece(x, at, at + n), at, 2), (piece(y, at2, at2 + m), at2, 0)])
        got.append(o[0])
        got2.append(o[1])
        at, at2 = at + n, at2 + m
    while at < 330:
        o = a.step([(piece(x, at, at + 1), at, 2), (piece(y, at2, at2 + 1), at2, 0)])
        got.append(o[0])
        got2.append(o[1])
        at, at2 = at + 1, at2 + 1
    a.check(x, got)
    a.check(piece(y, 0, at2), got2)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_a_single_token_stays_in_the_state(kind):
    """One key and value far above the others: what is left of them shows at every distance, in both directions across chunk edges."""
    a = Lightning(kind, [0.999, 0.97], 16, 16)
    for place in (0, 63, 64, 65, 127):
        q, k, v = (0.01 * z for z in a.random(400))
        q, k, v = to_bf16(np.ones_like(q)), to_bf16(k), to_bf16(v)
        k[place], v[place] = 8.0, 8.0
        want = a.want(q, k, v)
        assert abs(want[place + 200, 0].mean() / want[place, 0].mean() - 0.999 ** 200) < 0.01
        for portions in ([400], [64, 1, 200, 135], [place + 1, 1, 1, 300]):
            got, at = [], 0
            while at < 400:
                n = min(portions[min(len(got), len(portions) - 1)], 400 - at)
                got.append(a.step([(piece((q, k, v), at, at + n), at, 1)])[0])
                at += n
            got = np.concatenate(got)
            for t in (place, place + 1, place + 64, place + 128, place + 200):
                assert np.abs(got[t] / want[t] - 1).max() < (1e-5 if kind == "f32" else 1e-4), (place, portions, t)


def test_many_portions_in_one_batch():
    a = Lightning("bf16", [0.9, 0.99], 32, 64, slots=40)
    xs = [a.random(n, seed=n) for n in range(1, 36)] + [a.random(140, seed=99)]
    first = a.step([(piece(x, 0, (len(x[0]) + 1) // 2), 0, i) for i, x in enumerate(xs)])
    rest = [(i, x) for i, x in enumerate(xs) if len(x[0]) > 1]
    second = a.step([(piece(x, (len(x[0]) + 1) // 2, len(x[0])), (len(x[0]) + 1) // 2, i) for i, x in rest])
    for (i, x), o in zip(rest, second):
        err = row_err(np.concatenate([first[i], o]), a.want(*x))
        assert err.max() < 3e-5, (i, float(err.max()))


# ───────────────────────────── whole models ───────────────────────────────
@functools.lru_cache(maxsize=None)
def session(name, kind):
    c, w = util.model(name)
    return cuda_backend().prepare(kipizen.build(kipizen.KipizenConfig.from_dict(c), checkpoint.Weights.from_f32(w), DTYPES[kind]))


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
    s = llm.NativeLlmSession(cuda_backend(), kipizen.build(kipizen.KipizenConfig.from_dict(c), checkpoint.Weights.from_f32(w), ir.F32), 128)
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
