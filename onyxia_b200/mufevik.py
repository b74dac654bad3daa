"""Mufevik: a decoder over several residual streams. Each layer mixes tokens by attention whose heads share their softmax weights beside
gated linear attention, or by a gated delta rule, in any order; a mixture of experts or nothing follows.

    x_s = embed[token]                                       for every stream s
    every sublayer:  y = sublayer(norm(Σ_s in[s] x_s))
                     x_t ← Σ_s mix[s, t] x_s + out[t] y      for all streams at once
    logits = scale · head · norm(Σ_s x_s)

parallel  ½ norm(attention(h)) + ½ norm(linear attention(h)):
          attention         grouped queries, rotation of the leading dimensions of a head in two halves, a factor of the scores per head, softmax
                            weights mixed over heads before they meet the values
          linear attention  a matrix state per head whose rows decay by sigmoid(z)^(1 / tau), z of low rank; norm per head, gate
delta     a gated delta rule behind short convolutions, queries and keys as unit vectors; norm per head, gate
experts   softmax scores, compared with a correction, the best experts of the groups with the best expert; weights as scored; a shared expert
          with a factor per token
norms     divide by the root mean square; those of the stream multiply by one number

The module runs ragged batches over paged pools and state slots (csrc/backend/engine.hpp). Projections that read the same norm are one product
with it as the prologue; that norm also forms the new streams from the old ones and the sublayer's result or results.
"""
from __future__ import annotations

import dataclasses
import math

import numpy as np

from . import ir
from .checkpoint import Weights, host_tensor
from .ir import HostTensor
from .kipizen import turns_per_position

PAGE = 64            # tokens per cache page
UNIT_EPS = 1e-6      # of the delta rule's unit vectors


@dataclasses.dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0
    rot_base: float = 10000.0


@dataclasses.dataclass
class LinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclasses.dataclass
class ParallelConfig:
    left: AttentionConfig
    right: LinearConfig


@dataclasses.dataclass
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclasses.dataclass
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    groups: int = 0           # 0: all experts compete
    keep: int = 0
    shared_ff: int = 0        # 0: no shared expert


@dataclasses.dataclass
class LayerConfig:
    mixer: ParallelConfig | DeltaConfig
    experts: ExpertsConfig | None


def _grouped(i: int, m: dict) -> tuple:
    if m["heads"] % m["kv_heads"]:
        raise ValueError(f"layer {i}: {m['heads']} heads over {m['kv_heads']} key heads")
    return m["heads"], m["kv_heads"], m["dim"], m["vdim"]


def _parallel(i: int, m: dict) -> ParallelConfig:
    left, right = m["left"], m["right"]
    a = AttentionConfig(*_grouped(i, left), float(left["scale"]))
    if left.get("rot"):
        a.rot_dims, a.rot_base = left["rot"]["dims"], float(left["rot"]["base"])
    if a.rot_dims % 2 or a.rot_dims > a.dim:
        raise ValueError(f"layer {i}: {a.rot_dims} of {a.dim} dimensions cannot rotate in pairs")
    if not right["tau"] > 0:
        raise ValueError(f"layer {i}: decays to the power of 1 / {right['tau']}")
    return ParallelConfig(a, LinearConfig(right["heads"], right["dim"], right["vdim"], float(right["tau"])))


def _experts(i: int, m: dict | None) -> ExpertsConfig | None:
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {m['kind']!r}")
    r, groups = m["router"], m["router"].get("groups")
    e = ExpertsConfig(r["experts"], r["top"], m["expert"]["ff"])
    if groups:
        e.groups, e.keep = groups["count"], groups["keep"]
        if e.groups < 1 or e.experts % e.groups or not 1 <= e.keep <= e.groups:
            raise ValueError(f"layer {i}: {e.keep} of {e.groups} groups of {e.experts} experts")
    if m.get("shared"):
        e.shared_ff = m["shared"]["ff"]
    if not 1 <= e.top <= (e.experts // e.groups * e.keep if e.groups else e.experts):
        raise ValueError(f"layer {i}: {e.top} of {e.experts} experts")
    return e


@dataclasses.dataclass
class MufevikConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    logit_scale: float
    layers: list

    @staticmethod
    def from_dict(c: dict) -> "MufevikConfig":
        layers = []
        for i, l in enumerate(c["layers"]):
            if l["type"] == "parallel":
                mixer = _parallel(i, l["mixer"])
            elif l["type"] == "delta":
                mixer = DeltaConfig(*_grouped(i, l["mixer"]), l["mixer"]["conv"])
            else:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            layers.append(LayerConfig(mixer, _experts(i, l.get("mlp"))))
        if c["streams"] < 1:
            raise ValueError(f"{c['streams']} streams")
        return MufevikConfig(c["vocab"], c["width"], float(c["norm"]["eps"]), c["streams"], float(c.get("logit_scale", 1.0)), layers)


def build(cfg: MufevikConfig, w: Weights, dtype: int = ir.BF16) -> ir.Module:
    """The module in activation type `dtype`: BF16, or F32 for true 32-bit arithmetic."""
    if dtype not in (ir.BF16, ir.F32):
        raise ValueError(f"Mufevik modules run in bf16 or f32, not {ir.DTYPE_NAMES[dtype]}")
    b = ir.GraphBuilder()
    N, R, W = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("num_logits")
    NP, NS, TW = b.sym("num_pages"), b.sym("num_slots"), b.sym("table_width")
    H, S, eps = cfg.width, cfg.streams, float(cfg.eps)
    storage = np.uint16 if dtype == ir.BF16 else np.float32  # bf16 travels as bit patterns

    def const(a, dt=ir.F32):
        return b.constant(host_tensor(np.ascontiguousarray(a), dt))

    def plain(name, *shape):
        a = w.f32(name)
        if a.shape != shape:
            raise ValueError(f"tensor '{name}' has shape {list(a.shape)}, expected {list(shape)}")
        return a

    def stored(name, *shape):
        if w.shape(name) != shape:
            raise ValueError(f"tensor '{name}' has shape {list(w.shape(name))}, expected {list(shape)}")
        return w.stored(name, dtype)

    def matrix(name, rows, cols):
        return const(stored(name, rows, cols), dtype)

    def gain(name, factor=1.0):
        return const(np.full(H, plain(name) * np.float32(factor), np.float32))

    ids = b.input("input_ids", ir.I64, [N])
    seqs = b.input("seq_info", ir.I32, [R, 4])
    table = b.input("page_table", ir.I32, [R, TW]) if any(isinstance(l.mixer, ParallelConfig) for l in cfg.layers) else None
    rows = b.input("logit_rows", ir.I64, [W])
    state = []
    for i, l in enumerate(cfg.layers):
        m = l.mixer
        if isinstance(m, DeltaConfig):
            state.append((b.input(f"slots.{i}.conv", dtype, [NS, m.taps, 2 * m.kv_heads * m.dim + m.heads * m.vdim]),
                          b.input(f"slots.{i}.state", ir.F32, [NS, m.heads, m.dim, m.vdim])))
        else:
            a, r = m.left, m.right
            state.append((b.input(f"pages.{i}.keys", dtype, [NP, a.kv_heads, PAGE, a.dim]), b.input(f"pages.{i}.values", dtype, [NP, a.kv_heads, PAGE, a.vdim]),
                          b.input(f"slots.{i}.state", ir.F32, [NS, r.heads, r.dim, r.vdim])))

    # Streams that have not been formed yet: the old ones, the result or results that join them and how. The norm that reads the next
    # sublayer's share of them forms them.
    def norm_inputs(pend, weight, take):
        res, twin = pend.get("residual"), pend.get("twin")
        attrs = {"epsilon": eps, "pre": 1, "streams": S, "residual": int(res is not None), "post": int(twin is not None), "twin": int(twin is not None)}
        ins = [pend["y"], weight] + ([res] if res is not None else []) + ([pend["post"]] if twin is not None else [])
        return attrs, ins + [const(np.concatenate([pend["mix"].reshape(-1), pend["out"], take]))] + (list(twin) if twin is not None else [])

    def linear(name, attrs, ins, out, dt=ir.F32):
        b.set_loc(name, "Linear")
        return b.composite("onyxia.Linear", attrs, ins, [(dt, [N, out])])[0]

    def norm_linear(name, pend, norm, take, weight, out, dt, count=N, **extra):
        attrs, ins = norm_inputs(pend, norm, take)
        b.set_loc(name, "Linear")
        return b.composite("onyxia.Linear", {**attrs, "norm": 1, **extra}, ins + [weight], [(dt, [count, out]), (ir.F32, [count, S * H])])

    def stacked(p, parts):  # one matrix, its rows padded to a multiple of 8, and where each part starts
        at = np.cumsum([0] + [size for _, size in parts]).tolist()
        a = np.concatenate([stored(f"{p}.{n}", size, H) for n, size in parts] + [np.zeros((-at[-1] % 8, H), storage)])
        return const(a, dtype), len(a), dict(zip([n for n, _ in parts], at))

    def head_norm(name, o, norm, heads, vdim, gates, gate_at, out):  # norm per head, gate, product
        return linear(name, {"norm": 1, "stream": 0, "epsilon": eps, "norm_groups": heads, "gate": 1, "gate_offset": gate_at},
                      [o, const(np.tile(plain(norm, vdim), heads)), gates, matrix(out, H, heads * vdim)], H)

    def parallel(i, m, p, pend, norm, take):
        a, r = m.left, m.right
        q, k, v = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        qk, vg, rank = r.heads * r.dim, r.heads * r.vdim, w.shape(f"{p}.right.a1")[0]
        parts = [("left.q", q), ("left.k", k), ("left.v", v), ("right.q", qk), ("right.k", qk), ("right.v", vg), ("right.g", vg), ("right.a1", rank)]
        weight, columns, at = stacked(p, parts)
        proj, x = norm_linear(f"{p}.in", pend, norm, take, weight, columns, dtype, act_rest="silu", act_split=at["right.g"], act_end=at["right.a1"])
        z = linear(f"{p}.right.a2", {"ranges": 1, "bias": 1, "x_offset": at["right.a1"]},
                   [proj, matrix(f"{p}.right.a2", qk, rank), const(plain(f"{p}.right.a2.b", qk))], qk)
        b.set_loc(f"{p}.left", "PagedKVAttention")
        o, keys, values = b.composite(
            "onyxia.PagedKVAttention",
            {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "q_offset": 0, "k_offset": at["left.k"], "v_offset": at["left.v"],
             "rot_dims": a.rot_dims, "scale": a.scale, "epsilon": eps, "temps": 1, "talk": 1},
            [proj, const(turns_per_position(a.rot_dims, a.rot_base, 1.0)), state[i][0], state[i][1], seqs, table, const(plain(f"{p}.left.temp", a.heads)),
             const(plain(f"{p}.left.talk", a.heads, a.heads))],
            [(dtype, [N, a.heads * a.vdim]), (dtype, [NP, a.kv_heads, PAGE, a.dim]), (dtype, [NP, a.kv_heads, PAGE, a.vdim])])
        left = linear(f"{p}.left.out", {}, [o, matrix(f"{p}.left.o", H, a.heads * a.vdim)], H)
        b.set_loc(f"{p}.right", "GatedLinearAttention")
        o, new_state = b.composite(
            "onyxia.GatedLinearAttention", {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "q_offset": at["right.q"], "k_offset": at["right.k"],
                                            "v_offset": at["right.v"], "tau": r.tau, "q_scale": r.dim ** -0.5},
            [proj, z, state[i][2], seqs], [(ir.F32, [N, vg]), (ir.F32, [NS, r.heads, r.dim, r.vdim])])
        right = head_norm(f"{p}.right.out", o, f"{p}.right.norm", r.heads, r.vdim, proj, at["right.g"], f"{p}.right.o")
        updated.extend([(f"pages.{i}.keys", keys), (f"pages.{i}.values", values), (f"slots.{i}.state", new_state)])
        half = lambda n: const(0.5 * plain(f"{p}.{n}", H))
        return {"residual": x, "y": left, "post": half("left.out"), "twin": (right, half("right.out"))}

    def delta(i, m, p, pend, norm, take):
        qk, vg = m.kv_heads * m.dim, m.heads * m.vdim
        parts = [("q", qk), ("k", qk), ("v", vg), ("g", vg), ("a", m.heads), ("b", m.heads)]
        weight, columns, at = stacked(p, parts)
        proj, x = norm_linear(f"{p}.in", pend, norm, take, weight, columns, dtype, act_rest="silu", act_split=at["g"], act_end=at["a"])
        conv = np.concatenate([plain(f"{p}.{n}.conv", size, m.taps) for n, size in (("q", qk), ("k", qk), ("v", vg))])
        decay = np.exp(plain(f"{p}.A_log", m.heads).astype(np.float64)).astype(np.float32)
        b.set_loc(p, "GatedDeltaRule")
        o, conv_state, new_state = b.composite(
            "onyxia.GatedDeltaRule", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "taps": m.taps, "q_offset": 0, "a_offset": at["a"],
                                      "b_offset": at["b"], "q_scale": m.dim ** -0.5, "unit_epsilon": UNIT_EPS},
            [proj, const(conv), const(decay), const(plain(f"{p}.dt_bias", m.heads)), *state[i], seqs],
            [(ir.F32, [N, vg]), (dtype, [NS, m.taps, 2 * qk + vg]), (ir.F32, [NS, m.heads, m.dim, m.vdim])])
        updated.extend([(f"slots.{i}.conv", conv_state), (f"slots.{i}.state", new_state)])
        return {"residual": x, "y": head_norm(f"{p}.out", o, f"{p}.norm", m.heads, m.vdim, proj, at["g"], f"{p}.o")}

    def gated_pairs(p, ff):  # gate and up rows, interleaved
        return np.stack([stored(f"{p}.gate", ff, H), stored(f"{p}.up", ff, H)], axis=1).reshape(2 * ff, H)

    def experts(m, p, pend, norm, take):
        up, down = np.empty((m.experts, 2 * m.ff, H), storage), np.empty((m.experts, H, m.ff), storage)
        for e in range(m.experts):
            up[e], down[e] = gated_pairs(f"{p}.e{e}", m.ff), stored(f"{p}.e{e}.down", H, m.ff)
        router = [stored(f"{p}.router", m.experts, H)]
        if m.shared_ff:
            router.append(stored(f"{p}.shared.sg", 1, H))
        router = np.concatenate(router)
        consts = [const(router, dtype), const(np.zeros(len(router), np.float32)), const(up.reshape(-1, H), dtype), const(down.reshape(-1, m.ff), dtype)]
        extra = {"experts": m.experts, "top": m.top, "ff": m.ff, "scores": "softmax_all", "renorm": 0, "group_max": 1, "groups": m.groups, "keep": m.keep, "correction": 1}
        if m.shared_ff:
            consts += [const(gated_pairs(f"{p}.shared", m.shared_ff), dtype), matrix(f"{p}.shared.down", H, m.shared_ff)]
            extra.update(shared_ff=m.shared_ff, shared_gate=1)
        attrs, ins = norm_inputs(pend, norm, take)
        b.set_loc(p, "MixtureOfExperts")
        y, x = b.composite("onyxia.MixtureOfExperts", {**attrs, **extra}, ins + consts + [const(plain(f"{p}.correction", m.experts))],
                           [(ir.F32, [N, H]), (ir.F32, [N, S * H])])
        return {"residual": x, "y": y}

    b.set_loc("embed", "Gather")
    start = b.gather(b.constant(host_tensor(stored("embed", cfg.vocab, H), dtype), borrow=True), ids, 0)
    updated, pend = [], {"y": start, "mix": np.zeros((S, S), np.float32), "out": np.ones(S, np.float32)}
    for i, l in enumerate(cfg.layers):
        for q, sub in ((1, l.mixer), (2, l.experts)):
            if sub is None:
                continue
            norm, take = gain(f"l{i}.norm{q}"), plain(f"l{i}.hc{q}.in", S)
            if q == 2:
                pend = experts(sub, f"l{i}.mlp", pend, norm, take)
            else:
                pend = (delta if isinstance(sub, DeltaConfig) else parallel)(i, sub, f"l{i}.mix", pend, norm, take)
            pend.update(mix=plain(f"l{i}.hc{q}.mix", S, S), out=plain(f"l{i}.hc{q}.out", S))

    # only the rows whose logits are wanted go on
    b.set_loc("logit_rows", "Gather")
    pend.update({k: b.gather(pend[k], rows, 0) for k in ("y", "residual") if k in pend})
    if "twin" in pend:
        pend["twin"] = (b.gather(pend["twin"][0], rows, 0), pend["twin"][1])
    logits, _ = norm_linear("head", pend, gain("final.norm", cfg.logit_scale), np.ones(S, np.float32), matrix("head", cfg.vocab, H), cfg.vocab, ir.F32, count=W)
    b.set_loc(None)
    b.output("logits", logits)
    for name, v in updated:
        b.output("updated." + name, v)
    return b.finish()


def tensor_shapes(cfg: MufevikConfig, rank: int = 16) -> dict:
    """Names and shapes of a checkpoint of this configuration; `rank` is that of the decays' map."""
    H, S = cfg.width, cfg.streams
    out = {"embed": (cfg.vocab, H), "final.norm": (), "head": (cfg.vocab, H)}
    for i, l in enumerate(cfg.layers):
        p, m, f = f"l{i}.mix.", l.mixer, l.experts
        for q in (1, 2) if f else (1,):
            out.update({f"l{i}.norm{q}": (), f"l{i}.hc{q}.in": (S,), f"l{i}.hc{q}.out": (S,), f"l{i}.hc{q}.mix": (S, S)})
        if isinstance(m, DeltaConfig):
            for n, size in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                out.update({p + n: (size, H), f"{p}{n}.conv": (size, m.taps)})
            out.update({p + "b": (m.heads, H), p + "A_log": (m.heads,), p + "norm": (m.vdim,), p + "a": (m.heads, H), p + "dt_bias": (m.heads,),
                        p + "g": (m.heads * m.vdim, H), p + "o": (H, m.heads * m.vdim)})
        else:
            a, r = m.left, m.right
            qk, vg = r.heads * r.dim, r.heads * r.vdim
            out.update({p + "left." + n: s for n, s in {
                "q": (a.heads * a.dim, H), "k": (a.kv_heads * a.dim, H), "v": (a.kv_heads * a.vdim, H), "talk": (a.heads, a.heads), "temp": (a.heads,),
                "o": (H, a.heads * a.vdim), "out": (H,)}.items()})
            out.update({p + "right." + n: s for n, s in {
                "q": (qk, H), "k": (qk, H), "v": (vg, H), "g": (vg, H), "o": (H, vg), "norm": (r.vdim,), "a1": (rank, H), "a2": (qk, rank), "a2.b": (qk,),
                "out": (H,)}.items()})
        if f is None:
            continue
        for n, ff in {**{f"e{e}.": f.ff for e in range(f.experts)}, **({"shared.": f.shared_ff} if f.shared_ff else {})}.items():
            out.update({f"l{i}.mlp.{n}gate": (ff, H), f"l{i}.mlp.{n}up": (ff, H), f"l{i}.mlp.{n}down": (H, ff)})
        out.update({f"l{i}.mlp.router": (f.experts, H), f"l{i}.mlp.correction": (f.experts,)})
        if f.shared_ff:
            out[f"l{i}.mlp.shared.sg"] = (1, H)
    return out


def random_weights(cfg: MufevikConfig, seed: int = 0) -> Weights:
    """bf16 weights of a plausible scale (benchmarks, smoke runs). Large matrices repeat one random block."""
    rng = np.random.default_rng(seed)
    block = rng.standard_normal(1 << 20, dtype=np.float32)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last, n = name.rsplit(".", 1)[-1], int(np.prod(shape))
        if last in ("norm", "norm1", "norm2", "temp") or name.endswith((".left.out", ".right.out")):
            a = 1.0 + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif last in ("in", "out") or last == "mix":  # of the streams
            a = (np.eye(cfg.streams).reshape(-1) if last == "mix" else np.full(n, 1.0 if last == "out" else 1.0 / n)) + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif last == "talk":
            a = np.eye(shape[0]).reshape(-1) + 0.2 / math.sqrt(shape[0]) * rng.standard_normal(n, dtype=np.float32)
        elif last == "b" and name.endswith("a2.b"):
            a = rng.uniform(-1.0, 5.0, n).astype(np.float32)
        elif last in ("A_log", "dt_bias"):
            a = rng.uniform(-4.0, -1.0, n).astype(np.float32)
        elif last == "correction":
            a = 0.02 * rng.standard_normal(n, dtype=np.float32)
        else:
            at = int(rng.integers(0, 1 << 19))
            a = np.resize(block[at:], n) / (1.0 if name == "embed" else math.sqrt(shape[-1]))
        out[name] = HostTensor.bf16(np.asarray(a, np.float32).reshape(shape)).data.view(np.uint16).reshape(shape)
    return Weights.from_bf16(out)
