"""Lovuzen on the device against the plain implementation (lovuzen_ref.py): each mechanism alone through a module of its
own, then whole models through the engine — whole prompts, portions, token by token, ragged batches, pages and slots used
again, and generation through the scheduler.

f32 modules agree to a few parts in a million; bf16 ones to the rounding of their activations.
"""
import functools
import os
import subprocess
import sys
import json

import numpy as np
import pytest

import lovuzen_ref as ref
import lovuzen_util as util
from gpu_util import cuda_backend, differential
from lovuzen_util import to_bf16
from onyxia_b200 import backend as be
from onyxia_b200 import checkpoint, ir, llm, lovuzen
from onyxia_b200.engine import Engine
from onyxia_b200.ir import HostTensor

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"f32": ir.F32, "bf16": ir.BF16}
TOL = {"f32": 1e-5, "bf16": 3e-2}


def act(a, dtype):
    return HostTensor.bf16(a) if dtype == ir.BF16 else HostTensor.from_numpy(np.asarray(a, np.float32))


def rel_err(got, want):
    return float(np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want ** 2).mean()))


# ───────────────────────────── bf16 storage ───────────────────────────────
def bf16_storage_module():
    r = np.random.default_rng(2)
    b = ir.GraphBuilder()
    x, t, i = b.input("x", ir.F32, [5, 7]), b.input("t", ir.BF16, [9, 4]), b.input("i", ir.I64, [3])
    b.output("narrow", b.cast(x, ir.BF16))
    b.output("wide", b.cast(t, ir.F32))
    b.output("half", b.cast(t, ir.F16))
    b.output("rows", b.gather(t, i, 0))
    b.output("turned", b.transpose(t, [1, 0]))
    feed = {"x": HostTensor.from_numpy(r.standard_normal((5, 7)).astype(np.float32)), "t": HostTensor.bf16(r.standard_normal((9, 4))),
            "i": HostTensor.from_numpy(np.array([8, 0, 3], np.int64))}
    return b.finish(), feed


def test_bf16_tensors_are_cast_and_moved_like_the_oracle_does():
    module, feed = bf16_storage_module()
    got, want = differential(module, feed, atol=0.0, rtol=0.0)
    for (name, g), (_, w) in zip(got, want):
        assert g.dtype == w.dtype and np.array_equal(g.data, w.data), name
    assert np.array_equal(dict(got)["narrow"].numpy(), to_bf16(feed["x"].numpy()))


# ───────────────────────────── dense products ─────────────────────────────
def run_linear(dtype, x, w, *, x1=None, w1=None, bias=None, glu=None, out_dtype=None):
    b = ir.GraphBuilder()
    ins = [b.input("x", dtype, list(x.shape))]
    feed = {"x": act(x, dtype)}
    if x1 is not None:
        ins.append(b.input("x1", dtype, list(x1.shape)))
        feed["x1"] = act(x1, dtype)
    ins += [b.constant(act(a, dtype)) for a in (w, w1) if a is not None]
    if bias is not None:
        ins.append(b.constant(HostTensor.from_numpy(bias.astype(np.float32))))
    attrs = {"pair": int(x1 is not None), "bias": int(bias is not None)}
    if glu:
        attrs.update(glu=1, alpha=glu[0], limit=glu[1], shift=glu[2])
    out = ir.F32 if out_dtype is None else out_dtype
    b.output("y", b.composite("onyxia.Linear", attrs, ins, [(out, [x.shape[0], w.shape[0] // (2 if glu else 1)])])[0])
    return be.run_once(cuda_backend(), b.finish(), feed)[0][1].numpy()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 17, 32, 33, 100, 129, 300])
def test_linear(kind, rows):
    r = np.random.default_rng(rows)
    for k, n in ((64, 48), (200, 331), (1096, 272), (36, 50), (8, 16), (30, 20)):
        x, w = to_bf16(r.standard_normal((rows, k))), to_bf16(r.standard_normal((n, k)))
        assert rel_err(run_linear(DTYPES[kind], x, w), x.astype(np.float64) @ w.T.astype(np.float64)) < 2e-6, (k, n)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [2, 20, 70, 260])
def test_linear_pair_bias_gate(kind, rows):
    r = np.random.default_rng(rows)
    for k, k1, n in ((64, 136, 80), (520, 24, 258), (18, 7, 12)):
        x, x1 = to_bf16(r.standard_normal((rows, k))), to_bf16(r.standard_normal((rows, k1)))
        w, w1, bias = to_bf16(r.standard_normal((n, k))), to_bf16(r.standard_normal((n, k1))), to_bf16(r.standard_normal(n))
        x64, w64 = x.astype(np.float64), w.astype(np.float64)
        want = x64 @ w64.T + x1.astype(np.float64) @ w1.T.astype(np.float64) + bias
        assert rel_err(run_linear(DTYPES[kind], x, w, x1=x1, w1=w1, bias=bias), want) < 2e-6
        alpha, limit, shift = 1.3, 4.0, 0.5
        z = x64 @ w64.T + bias
        g, u = np.minimum(z[:, ::2], limit), np.clip(z[:, 1::2], -limit, limit)
        want = g * ref.sigmoid(alpha * g) * (u + shift)
        assert rel_err(run_linear(DTYPES[kind], x, w, bias=bias, glu=(alpha, limit, shift)), want) < 3e-6
        if kind == "bf16":
            assert rel_err(run_linear(ir.BF16, x, w, out_dtype=ir.BF16), x64 @ w64.T) < 4e-3


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 2, 4, 7, 8, 9, 40])
def test_residual_norm_in_front_of_a_product(kind, rows):
    r = np.random.default_rng(rows)
    eps = 1e-3
    for width, n in ((96, 64), (1160, 40), (50, 30)):
        for has_res, has_gain, y_dt in ((1, 1, ir.F32), (0, 0, DTYPES[kind]), (1, 0, ir.F32)):
            y, res = to_bf16(0.02 * r.standard_normal((rows, width))), r.standard_normal((rows, width)).astype(np.float32)
            w, gain, m = to_bf16(r.standard_normal(width)), to_bf16(r.standard_normal(width)), to_bf16(r.standard_normal((n, width)))
            b = ir.GraphBuilder()
            ins = [b.input("y", y_dt, [rows, width]), b.constant(HostTensor.from_numpy(w))]
            feed = {"y": act(y, y_dt)}
            if has_res:
                ins.append(b.input("res", ir.F32, [rows, width]))
                feed["res"] = HostTensor.from_numpy(res)
            if has_gain:
                ins.append(b.constant(HostTensor.from_numpy(gain)))
            attrs = {"epsilon": eps, "residual": has_res, "gain": has_gain}
            alone = b.composite("onyxia.ResidualNorm", attrs, ins, [(ir.F32, [rows, width])])[0]
            out, stream = b.composite("onyxia.Linear", dict(attrs, norm=1), ins + [b.constant(act(m, DTYPES[kind]))],
                                      [(ir.F32, [rows, n]), (ir.F32, [rows, width])])
            for name, v in (("alone", alone), ("out", out), ("stream", stream)):
                b.output(name, v)
            got = {k: v.numpy() for k, v in be.run_once(cuda_backend(), b.finish(), feed)}
            want = ref.rms_norm(y.astype(np.float64), w.astype(np.float64), eps) * (gain if has_gain else 1.0) + (res if has_res else 0.0)
            assert rel_err(got["alone"], want) < 1e-6 and rel_err(got["stream"], want) < 1e-6
            assert rel_err(got["out"], want @ m.T.astype(np.float64)) < (2e-6 if kind == "f32" else 5e-3)


# ───────────────────────────── attention ──────────────────────────────────
class Attention:
    """One attention node with its pools on the device; pages are handed out in a shuffled order."""

    def __init__(self, kind, heads, kv_heads, dim, bias, q_w, k_w, *, scale=0.3, temp=None, eps=1e-5, out_scale=1.0, pages=40, extra=3):
        dt = self.dt = DTYPES[kind]
        self.kind, self.heads, self.kv, self.dim, self.extra = kind, heads, kv_heads, dim, extra
        b = ir.GraphBuilder()
        N, R, TW = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("table_width")
        width = extra + (heads + kv_heads) * dim + 2
        ins = [b.input("proj", dt, [N, width]), b.constant(HostTensor.from_numpy(q_w)), b.constant(HostTensor.from_numpy(k_w)),
               b.constant(HostTensor.from_numpy(bias.astype(np.float32))), b.input("pool", dt, [pages, kv_heads, 64, dim]),
               b.input("scales", ir.F32, [pages, 64]), b.input("seqs", ir.I32, [R, 4]), b.input("table", ir.I32, [R, TW])]
        t = temp or (0.0, 0.0)
        outs = b.composite("onyxia.PagedAttention",
                           {"heads": heads, "kv_heads": kv_heads, "dim": dim, "k_offset": extra, "q_offset": extra + kv_heads * dim,
                            "scale": scale, "epsilon": eps, "temp_coef": float(t[0]), "temp_every": float(t[1]), "out_scale": out_scale},
                           ins, [(dt, [N, heads * dim]), (dt, [pages, kv_heads, 64, dim]), (ir.F32, [pages, 64])])
        for name, v in zip(("out", "pool2", "scales2"), outs):
            b.output(name, v)
        self.s = cuda_backend().prepare(b.finish())
        self.pool = self.s.upload(act(np.full((pages, kv_heads, 64, dim), 99.0), dt))
        self.scales = self.s.upload(HostTensor.from_numpy(np.full((pages, 64), 99.0, np.float32)))
        self.free = np.random.default_rng(1).permutation(pages).tolist()
        self.owned, self.past = {}, {}

    def step(self, entries):
        """entries: [(sequence, q [n, H, d], k [n, G, d])] → outputs per entry."""
        rows, info, at = [], [], 0
        for seq, q, k in entries:
            n, past = len(q), self.past.setdefault(seq, 0)
            own = self.owned.setdefault(seq, [])
            while len(own) * 64 < past + n:
                own.append(self.free.pop())
            info.append([at, n, past, 0])
            rows.append(np.concatenate([np.full((n, self.extra), 7.0), k.reshape(n, -1), q.reshape(n, -1), np.full((n, 2), -7.0)], axis=1))
            at += n
            self.past[seq] = past + n
        tw = max(len(self.owned[e[0]]) for e in entries)
        table = [self.owned[e[0]] + [0] * (tw - len(self.owned[e[0]])) for e in entries]
        feed = {"proj": self.s.upload(act(np.concatenate(rows), self.dt)), "pool": self.pool, "scales": self.scales,
                "seqs": self.s.upload(HostTensor.from_numpy(np.array(info, np.int32))),
                "table": self.s.upload(HostTensor.from_numpy(np.array(table, np.int32)))}
        out = dict(self.s.run(feed))
        self.pool, self.scales = out["pool2"], out["scales2"]
        o = self.s.download(out["out"]).numpy().reshape(-1, self.heads, self.dim)
        return [o[i[0]:i[0] + i[1]] for i in info]


def attention_want(q, k, bias_rows, far, q_w, k_w, *, scale=0.3, temp=None, eps=1e-5):
    T = len(q)
    qn = ref.rms_norm(q.reshape(T, -1).astype(np.float64), q_w, eps).reshape(q.shape)
    kn = ref.rms_norm(k.reshape(T, -1).astype(np.float64), k_w, eps).reshape(k.shape)
    return ref.attention(qn, kn, k.astype(np.float64), scale, bias_rows, far, temp)


SHAPES = [(4, 2, 16), (3, 3, 64), (20, 1, 72), (8, 1, 128), (2, 1, 256), (5, 5, 10), (2, 2, 300)]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("heads,kv,dim", SHAPES)
def test_attention_alone(kind, heads, kv, dim):
    """A prompt in uneven portions, then decoded tokens, beside two other sequences at other lengths."""
    r = np.random.default_rng(dim)
    T, rows, far = 200, 12, 90
    q, k = to_bf16(r.standard_normal((T, heads, dim))), to_bf16(r.standard_normal((T, kv, dim)))
    q_w, k_w = to_bf16(1 + 0.3 * r.standard_normal(heads * dim)), to_bf16(1 + 0.3 * r.standard_normal(kv * dim))
    bias = r.standard_normal((rows, heads))
    kw = dict(scale=2.0 / np.sqrt(dim), temp=(0.4, 30))
    want = attention_want(q, k, bias, far, q_w, k_w, **kw)
    a = Attention(kind, heads, kv, dim, lovuzen.distance_bias(bias, far), q_w, k_w, **kw)
    got, at = [], 0
    for n in (1, 2, 61, 1, 64, 3, 30):
        others = [(7, q[a.past.get(7, 0)][None], k[a.past.get(7, 0)][None]), (8, q[at:at + 5], k[at:at + 5])]
        got.append(a.step([others[0], (0, q[at:at + n], k[at:at + n]), others[1]])[1])
        at += n
    while at < T:
        got.append(a.step([(0, q[at:at + 1], k[at:at + 1]), (7, q[a.past[7]][None], k[a.past[7]][None])])[0])
        at += 1
    got = np.concatenate(got)
    tol = 1e-5 if kind == "f32" else 1e-2
    err = np.sqrt(((got - want) ** 2).mean(axis=(1, 2))) / np.sqrt((want ** 2).mean())
    assert err.max() < tol, (int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
def test_single_keys_stand_out(kind, decode):
    """One key carries nearly all the weight: its value is the output, wherever the key lies."""
    r = np.random.default_rng(5)
    heads, kv, dim, T = 4, 2, 32, 700
    ones = np.ones(heads * dim, np.float32)
    a = Attention(kind, heads, kv, dim, np.zeros((heads, 50), np.float32), 4 * ones, np.ones(kv * dim, np.float32), scale=1.0)
    places = (0, 1, 62, 63, 64, 65, 127, 128, 255, 256, 511, 512, 513, 640)
    k = to_bf16(0.2 * r.standard_normal((T, kv, dim)))
    for j in places:
        k[j] = to_bf16(r.standard_normal((kv, dim)))
    q = to_bf16(r.standard_normal((T, heads, dim)))
    look = {699 - i: j for i, j in enumerate(places)}  # query position → the key it looks for
    for i, j in look.items():
        q[i] = np.repeat(k[j], heads // kv, axis=0)
    want = attention_want(q, k, np.zeros((4, heads)), 50, 4.0 * ones, np.ones(kv * dim), scale=1.0)
    for i, j in look.items():
        assert np.abs(want[i] - np.repeat(k[j], heads // kv, axis=0)).max() < 0.05  # it does stand out
    if decode:
        a.step([(0, q[:680], k[:680])])
        got = {i: a.step([(0, q[i:i + 1], k[i:i + 1])])[0][0] for i in range(680, T)}
    else:
        out = a.step([(0, q, k)])[0]
        got = {i: out[i] for i in range(680, T)}
    for i in look:
        assert np.abs(got[i] - want[i]).max() < (1e-4 if kind == "f32" else 3e-2), (i, look[i])


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
def test_every_distance_row_decides(kind, decode):
    """One bias row is far above the others: the output is the mean of the values at that row's distances, so a distance
    that read its neighbour's row would show."""
    r = np.random.default_rng(9)
    heads, kv, dim, T, rows, far = 2, 1, 16, 160, 8, 70
    k = to_bf16(r.standard_normal((T, kv, dim)))
    q = to_bf16(r.standard_normal((T, heads, dim)))
    w1, w2 = np.full(heads * dim, 0.01, np.float32), np.ones(kv * dim, np.float32)
    for row in range(rows):
        bias = np.zeros((rows, heads))
        bias[row, 0], bias[row, 1] = 25.0, 20.0
        want = attention_want(q, k, bias, far, w1, w2)
        a = Attention(kind, heads, kv, dim, lovuzen.distance_bias(bias, far), w1, w2)
        if decode:
            a.step([(0, q[:150], k[:150])])
            got = np.concatenate([a.step([(0, q[i:i + 1], k[i:i + 1])])[0] for i in range(150, T)])
            want = want[150:]
        else:
            got = a.step([(0, q, k)])[0]
        assert np.abs(got - want).max() < (1e-4 if kind == "f32" else 3e-2), row


def test_bad_page_tables_are_reported():
    one = np.ones(32, np.float32)
    a = Attention("bf16", 2, 2, 16, np.zeros((2, 4), np.float32), one, one, pages=3)
    x = to_bf16(np.random.default_rng(0).standard_normal((2, 2, 16)))
    a.free = [5]
    with pytest.raises(Exception, match="out of range"):
        a.step([(0, x, x)])


# ───────────────────────────── recurrence ─────────────────────────────────
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width,blocks,taps", [(48, 2, 3), (40, 1, 4), (160, 1, 2), (21, 3, 5), (64, 8, 1), (304, 2, 6), (600, 1, 4)])
def test_recurrence_alone(kind, width, blocks, taps):
    """Portions down to one token, three sequences in turn over two slots' neighbours, slots used again."""
    r = np.random.default_rng(width)
    dt, T, n = DTYPES[kind], 330, width // blocks
    conv, cb = to_bf16(r.standard_normal((width, taps)) / np.sqrt(taps)), to_bf16(0.3 * r.standard_normal(width))
    ra, ri = (to_bf16(r.standard_normal((blocks, n, n)) / np.sqrt(n)) for _ in range(2))
    rab, rib = (to_bf16(r.standard_normal((blocks, n))) for _ in range(2))
    lam = to_bf16(r.uniform(-7, 1, width))
    b = ir.GraphBuilder()
    N, R = b.sym("num_tokens"), b.sym("num_seqs")
    c = lambda a: b.constant(HostTensor.from_numpy(np.asarray(a, np.float32)))
    ins = [b.input("proj", dt, [N, 2 * width + 5]), c(conv), c(cb), b.constant(act(ra, dt)), c(rab.reshape(-1)), b.constant(act(ri, dt)),
           c(rib.reshape(-1)), c(lam), b.input("ring", dt, [4, taps, width]), b.input("state", ir.F32, [4, width]), b.input("seqs", ir.I32, [R, 4])]
    outs = b.composite("onyxia.GatedRecurrence", {"width": width, "blocks": blocks, "taps": taps, "x_offset": 2, "y_offset": width + 5, "decay": 8.0,
                                                  "out_scale": 0.5}, ins, [(dt, [N, width]), (dt, [4, taps, width]), (ir.F32, [4, width])])
    for name, v in zip(("out", "ring2", "state2"), outs):
        b.output(name, v)
    s = cuda_backend().prepare(b.finish())
    state = {"ring": s.upload(act(np.full((4, taps, width), 50.0), dt)), "state": s.upload(HostTensor.from_numpy(np.full((4, width), 50.0, np.float32)))}

    def step(parts):  # (x, y, past, slot)
        info, rows, at = [], [], 0
        for x, y, past, slot in parts:
            rows.append(np.concatenate([np.full((len(x), 2), 3.0), x, np.full((len(x), 3), 3.0), y], axis=1))
            info.append([at, len(x), past, slot])
            at += len(x)
        out = dict(s.run({"proj": s.upload(act(np.concatenate(rows), dt)), "seqs": s.upload(HostTensor.from_numpy(np.array(info, np.int32))), **state}))
        state.update(ring=out["ring2"], state=out["state2"])
        o = s.download(out["out"]).numpy()
        return [o[i[0]:i[0] + i[1]] for i in info]

    def want(x, y):
        u = ref.causal_conv(x.astype(np.float64), conv.astype(np.float64), cb)
        rr, ii = (ref.sigmoid(ref.block_linear(u, w.astype(np.float64), bb)) for w, bb in ((ra, rab), (ri, rib)))
        return ref.linear_recurrence(u, rr, ii, lam.astype(np.float64)) * ref.gelu_tanh(y.astype(np.float64)) * 0.5

    def check(x, y, got):
        w = want(x, y)
        err = np.sqrt(((got - w) ** 2).mean(axis=1)) / np.sqrt((w ** 2).mean())
        assert err.max() < (1e-5 if kind == "f32" else 2e-2), (int(err.argmax()), float(err.max()))

    x, y = to_bf16(r.standard_normal((T, width))), to_bf16(r.standard_normal((T, width)))
    x2, y2 = x[::-1].copy(), y[::-1].copy()
    check(x, y, step([(x, y, 0, 2)])[0])                     # one long prompt; slot 2 is dirty afterwards
    got, got2, at = [], [], 0
    for n_new in (1, 1, 2, 3, 17, 1, 40, 5, 1, 130):
        a, c2 = step([(x[at:at + n_new], y[at:at + n_new], at, 2), (x2[len(got2)][None], y2[len(got2)][None], len(got2), 0)])
        got.append(a)
        got2.append(c2)
        at += n_new
    while at < 260:
        a, c2 = step([(x[at:at + 1], y[at:at + 1], at, 2), (x2[len(got2)][None], y2[len(got2)][None], len(got2), 0)])
        got.append(a)
        got2.append(c2)
        at += 1
    check(x[:at], y[:at], np.concatenate(got))
    check(x2[:len(got2)], y2[:len(got2)], np.concatenate(got2))
    # many sequences at once, one token each (their slots collide only with themselves)
    outs2 = [step([(x[t:t + 1], y[t:t + 1], t, 1), (x2[t:t + 1], y2[t:t + 1], t, 3)]) for t in range(20)]
    check(x[:20], y[:20], np.concatenate([o[0] for o in outs2]))
    check(x2[:20], y2[:20], np.concatenate([o[1] for o in outs2]))


# ───────────────────────────── whole models ───────────────────────────────
@functools.lru_cache(maxsize=None)
def session(name, kind, seed=0, sharpen=1.0):
    config, w = util.model(name, seed, sharpen)
    return cuda_backend().prepare(lovuzen.build(lovuzen.LovuzenConfig.from_dict(config), checkpoint.Weights.from_f32(w), DTYPES[kind]))


def engine(name, kind, max_tokens=2048, max_seqs=4, **kw):
    return Engine(session(name, kind, **kw), max_tokens, max_seqs)


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
def test_whole_prompt_against_the_plain_model(name, kind):
    toks = util.tokens(name, 150)
    for sharpen in (1.0, 4.0):
        e = engine(name, kind, sharpen=sharpen)
        err = util.distance(feed(e, 0, toks, [150]), util.expected(name, 150, sharpen=sharpen))
        assert err.max() < TOL[kind] * sharpen ** 0.5, (sharpen, float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("portions", [[1], [2], [3, 1, 1, 70, 2, 1], [64, 63, 5], [65, 1]])
def test_portions_do_not_matter(name, kind, portions):
    toks = util.tokens(name, 150)
    err = util.distance(feed(engine(name, kind), 0, toks, portions), util.expected(name, 150))
    assert err.max() < TOL[kind], (float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_long_decoding(kind):
    toks = util.tokens("mixed", 420)
    err = util.distance(feed(engine("mixed", kind), 0, toks, [90, 1]), util.expected("mixed", 420))
    assert err.max() < TOL[kind] and err[-50:].max() < TOL[kind]


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
    """Twenty and forty sequences decoding together: the other products and recurrence tilings."""
    for count in (20, 40):
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


def test_wanted_places_only():
    toks = util.tokens("mixed", 40)
    e = engine("mixed", "f32")
    out = e.forward([(3, toks, [39, 0, 17])])
    assert util.distance(out, util.expected("mixed", 40)[[39, 0, 17]]).max() < TOL["f32"]
    assert e.forward([(3, [1, 2], [])]).shape == (0, 131)


def test_engine_refuses_what_does_not_fit():
    e = engine("mixed", "bf16", max_tokens=128, max_seqs=2)
    with pytest.raises(Exception, match="out of cache pages"):
        e.forward([(0, util.tokens("mixed", 129), [])])
    assert e.stats()["free_pages"] == 2 and e.stats()["free_slots"] == 2
    e.forward([(0, [1], []), (1, [2], [])])
    with pytest.raises(Exception, match="no free slot"):
        e.forward([(2, [1], [])])
    with pytest.raises(Exception, match="twice"):
        e.forward([(0, [1], []), (0, [2], [])])
    with pytest.raises(Exception, match="outside"):
        e.forward([(0, [1], [1])])
    with pytest.raises(Exception, match="no live sequence"):
        e.release(9)
    with pytest.raises(Exception, match="pages"):
        e.submit([1] * 100, 100)


# ───────────────────────────── generation ─────────────────────────────────
def greedy_plain(name, prompt, n):
    config, w = util.model(name)
    toks = list(prompt)
    for _ in range(n):
        logits = ref.forward(config, w, toks)[-1]
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
    # an end token cuts a request short
    e = engine("mixed", "f32", max_tokens=320, max_seqs=3)
    eos = want[1][2]
    got = e.generate([prompts[1]], 6, eos=eos)[0]
    assert got == want[1][:want[1].index(eos) + 1]


def test_the_single_sequence_loop_serves_it_too():
    config, w = util.model("mixed")
    prompt = util.tokens("mixed", 30, seed=9)
    want = greedy_plain("mixed", prompt, 5)
    module = lovuzen.build(lovuzen.LovuzenConfig.from_dict(config), checkpoint.Weights.from_f32(w), ir.F32)
    s = llm.NativeLlmSession(cuda_backend(), module, 128)
    assert s.generate(prompt, 5) == want
    s.reset()
    got = [s.step_greedy(prompt)]
    for _ in range(4):
        got.append(s.step_greedy([got[-1]]))
    assert got == want and s.sequence_length() == 34
    s.reset()
    logits = s.step_logits(prompt)
    assert util.distance(logits[None], ref.forward(config, w, prompt)[-1:]).max() < TOL["f32"]
    assert s.step_sampled([want[0]], 0.7, 1, 1.0, 0.5) == want[1]  # the one most likely token


def test_sampled_generation_is_reproducible():
    prompts = [util.tokens("mixed", 9, seed=i) for i in range(4)]
    e = engine("mixed", "f32")
    kw = dict(temperature=1.0, top_k=20, seed=5)
    a, b = e.generate(prompts, 8, **kw), e.generate(prompts, 8, **kw)
    assert a == b and all(0 <= t < 131 for row in a for t in row)
    assert e.generate(prompts, 8, temperature=1.0, top_k=20, seed=6) != a
    assert e.generate(prompts, 8, temperature=1.0, top_k=1, seed=6) == e.generate(prompts, 8)


def test_command_line(tmp_path):
    config, w = util.model("mixed")
    with open(tmp_path / "config.json", "w") as f:
        json.dump(config, f)
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
    want = ref.forward(config, w, prompt)
    for step, places in ((0, [11]), (1, [7, 11])):
        got = np.fromfile(tmp_path / f"{step}.f32", np.float32).reshape(len(places), -1)
        assert util.distance(got, want[places]).max() < TOL["f32"]
