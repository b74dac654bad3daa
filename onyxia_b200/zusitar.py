"""Zusitar: a decoder whose layers mix tokens by grouped-query attention, attention over a latent, or a selective scan, in any
order; a run of them can be gone through several times with the same weights.

    x = e = scale · embed[token]
    every layer:              x += norm1b(mixer(norm1(x)))
                              x += norm2b(mlp(norm2(x)))                    (layers may have no mlp)
    before pass t of a loop:  x += step[t], and from the second pass on  x += e
    logits = embed · norm(x)

attention         rotation of neighbouring dimensions, capped scores, a learned sink per head, a gate per head
latent_attention  queries through a latent of their own, keys and values from one latent per token that is all the cache holds
                  beside a rotated key part; a gate per output. The maps from the latent to keys and values are moved to the
                  queries and results: attention runs in the latent space
mamba1            a selective scan behind a short convolution
mlp               a gated unit, or a mixture of experts: sigmoid scores, the best experts of the best groups, a shared expert

The module runs ragged batches over paged pools and state slots (csrc/backend/engine.hpp); every pass of a looped layer has pools
and slots of its own. Projections that read the same norm are one product with it as the prologue; that norm also forms the residual
sum from the sublayer's result, its second norm and what a loop adds.
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
GLU_ALPHA = 1.702    # the experts' gated unit
GLU_SHIFT = 1.0


@dataclasses.dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0
    rot_base: float = 10000.0
    softcap: float = 0.0      # 0: none


@dataclasses.dataclass
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclasses.dataclass
class MambaConfig:
    inner: int
    state: int
    dt_rank: int
    taps: int


@dataclasses.dataclass
class DenseConfig:
    ff: int


@dataclasses.dataclass
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    limit: float
    scale: float
    groups: int = 0           # 0: all experts compete
    keep: int = 0
    shared_ff: int = 0        # 0: no shared expert
    shared_limit: float = math.inf


@dataclasses.dataclass
class LayerConfig:
    mixer: AttentionConfig | LatentConfig | MambaConfig
    mlp: DenseConfig | ExpertsConfig | None


def _rotation(i: int, rot: dict | None, dim: int) -> tuple:
    dims, base = (rot["dims"], float(rot["base"])) if rot else (0, 10000.0)
    if dims % 2 or dims > dim:
        raise ValueError(f"layer {i}: {dims} of {dim} dimensions cannot rotate in pairs")
    return dims, base


def _attention(i: int, m: dict) -> AttentionConfig:
    if m["heads"] % m["kv_heads"]:
        raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key heads")
    dims, base = _rotation(i, m.get("rot"), m["dim"])
    return AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), dims, base, float(m.get("softcap") or 0.0))


def _latent(i: int, m: dict) -> LatentConfig:
    dims, base = _rotation(i, m.get("rot"), m["rot_dim"])
    if dims != m["rot_dim"]:
        raise ValueError(f"layer {i}: {dims} of the {m['rot_dim']} shared dimensions rotate")
    return LatentConfig(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]), base)


def _mlp(i: int, m: dict | None):
    if m is None:
        return None
    if m["kind"] == "dense":
        return DenseConfig(m["ff"])
    if m["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {m['kind']!r}")

    def limit(c):
        return math.inf if c.get("limit") is None else float(c["limit"])

    r, groups, shared = m["router"], m["router"].get("groups"), m.get("shared")
    e = ExpertsConfig(r["experts"], r["top"], m["expert"]["ff"], limit(m["expert"]), float(r["scale"]))
    if groups:
        e.groups, e.keep = groups["count"], groups["keep"]
        if e.groups < 1 or e.experts % e.groups or not 1 <= e.keep <= e.groups:
            raise ValueError(f"layer {i}: {e.keep} of {e.groups} groups of {e.experts} experts")
    if shared:
        e.shared_ff, e.shared_limit = shared["ff"], limit(shared)
    if not 1 <= e.top <= (e.experts // e.groups * e.keep if e.groups else e.experts):
        raise ValueError(f"layer {i}: {e.top} of {e.experts} experts")
    return e


@dataclasses.dataclass
class ZusitarConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: list
    loop: tuple = (0, 0, 1)   # layers start … stop − 1 run `times` times; an empty range: no loop

    @staticmethod
    def from_dict(c: dict) -> "ZusitarConfig":
        layers = []
        for i, l in enumerate(c["layers"]):
            m = l["mixer"]
            if l["type"] == "attention":
                mixer = _attention(i, m)
            elif l["type"] == "latent_attention":
                mixer = _latent(i, m)
            elif l["type"] == "mamba1":
                mixer = MambaConfig(m["inner"], m["state"], m["dt_rank"], m["conv"])
            else:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            layers.append(LayerConfig(mixer, _mlp(i, l.get("mlp"))))
        out = ZusitarConfig(c["vocab"], c["width"], float(c["norm"]["eps"]), float(c["embedding"]["scale"]), layers)
        if c.get("loop"):
            out.loop = (c["loop"]["start"], c["loop"]["stop"], c["loop"]["times"])
            if not 0 <= out.loop[0] < out.loop[1] <= len(layers) or out.loop[2] < 1:
                raise ValueError(f"a loop of layers {out.loop[0]} … {out.loop[1] - 1} of {len(layers)}, {out.loop[2]} times")
        return out

    def runs(self) -> list:
        """(layer, number of the pass that starts in front of it or None) in the order they run."""
        start, stop, times = self.loop
        n = len(self.layers)
        if start == stop:
            return [(i, None) for i in range(n)]
        return ([(i, None) for i in range(start)] + [(i, t if i == start else None) for t in range(times) for i in range(start, stop)] +
                [(i, None) for i in range(stop, n)])


def build(cfg: ZusitarConfig, w: Weights, dtype: int = ir.BF16) -> ir.Module:
    """The module in activation type `dtype`: BF16, or F32 for true 32-bit arithmetic."""
    if dtype not in (ir.BF16, ir.F32):
        raise ValueError(f"Zusitar modules run in bf16 or f32, not {ir.DTYPE_NAMES[dtype]}")
    b = ir.GraphBuilder()
    N, R, W = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("num_logits")
    NP, NS, TW = b.sym("num_pages"), b.sym("num_slots"), b.sym("table_width")
    H, eps = cfg.width, float(cfg.eps)
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

    runs = cfg.runs()
    ids = b.input("input_ids", ir.I64, [N])
    seqs = b.input("seq_info", ir.I32, [R, 4])
    table = b.input("page_table", ir.I32, [R, TW]) if any(not isinstance(cfg.layers[i].mixer, MambaConfig) for i, _ in runs) else None
    rows = b.input("logit_rows", ir.I64, [W])
    state = []  # per run
    for n, (i, _) in enumerate(runs):
        m = cfg.layers[i].mixer
        if isinstance(m, MambaConfig):
            state.append((b.input(f"slots.{n}.conv", dtype, [NS, m.taps, m.inner]), b.input(f"slots.{n}.state", ir.F32, [NS, m.inner, m.state])))
        elif isinstance(m, LatentConfig):
            state.append((b.input(f"pages.{n}.latents", dtype, [NP, 1, PAGE, m.kv_rank + m.rot_dim]),))
        else:
            state.append((b.input(f"pages.{n}.keys", dtype, [NP, m.kv_heads, PAGE, m.dim]), b.input(f"pages.{n}.values", dtype, [NP, m.kv_heads, PAGE, m.vdim])))

    # A sum that has not been formed yet. The norm that reads it forms it and leaves the new residual.
    def norm_inputs(pend, weight):
        parts = [("residual", pend.get("residual")), ("post", pend.get("post")), ("add", pend.get("add")), ("offset", pend.get("offset"))]
        attrs = {"epsilon": eps, "pre": 1, "y_scale": float(pend.get("scale", 1.0)), **{n: int(v is not None) for n, v in parts}}
        if pend.get("add") is not None:
            attrs["add_scale"] = float(cfg.embed_scale)
        return attrs, [pend["y"], weight] + [v for _, v in parts if v is not None]

    def linear(name, attrs, ins, out, dt=ir.F32):
        b.set_loc(name, "Linear")
        return b.composite("onyxia.Linear", attrs, ins, [(dt, [N, out])])[0]

    def norm_linear(name, pend, norm, weight, out, dt, count=N, bias=None, **extra):
        attrs, ins = norm_inputs(pend, norm)
        attrs.update({"norm": 1, "bias": int(bias is not None)}, **extra)
        b.set_loc(name, "Linear")
        return b.composite("onyxia.Linear", attrs, ins + [weight] + ([bias] if bias is not None else []),
                           [(dt, [count, out]), (ir.F32, [count, H])])

    # Constants of a layer, shared by its passes. Each returns a function of (run, sum) → new residual, sublayer's result.
    def attention(p, m):
        q_n, k_n, v_n = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        own, gate = q_n + k_n + v_n, q_n + k_n + v_n + m.heads
        weight = const(np.concatenate([stored(f"{p}.{n}", size, H) for n, size in (("q", q_n), ("k", k_n), ("v", v_n), ("g", m.heads))]), dtype)
        bias = const(np.concatenate([plain(f"{p}.{n}.b", size) for n, size in (("q", q_n), ("k", k_n), ("v", v_n))] + [np.zeros(m.heads, np.float32)]))
        norm, out, out_b = const(plain(f"{p[:-4]}.norm1", H)), matrix(f"{p}.o", H, m.heads * m.vdim), const(plain(f"{p}.o.b", H))
        turns, sinks = const(turns_per_position(m.rot_dims, m.rot_base, 1.0)), const(plain(f"{p}.sink", m.heads))

        def run(n, pend):
            proj, x = norm_linear(f"{p}.in", pend, norm, weight, gate, dtype, bias=bias, act_rest="sigmoid", act_split=own)
            b.set_loc(p, "PagedKVAttention")
            o, keys, values = b.composite(
                "onyxia.PagedKVAttention",
                {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "q_offset": 0, "k_offset": q_n, "v_offset": q_n + k_n,
                 "rot_dims": m.rot_dims, "interleaved": 1, "scale": m.scale, "softcap": m.softcap, "epsilon": eps, "sinks": 1, "gate": 1, "gate_offset": own},
                [proj, turns, *state[n], seqs, table, sinks],
                [(dtype, [N, m.heads * m.vdim]), (dtype, [NP, m.kv_heads, PAGE, m.dim]), (dtype, [NP, m.kv_heads, PAGE, m.vdim])])
            updated.extend([(f"pages.{n}.keys", keys), (f"pages.{n}.values", values)])
            return x, linear(f"{p}.out", {"bias": 1}, [o, out, out_b], H)
        return run

    def latent(p, m):
        q_n, kv_n, v_n = m.heads * (m.dim + m.rot_dim), m.kv_rank + m.rot_dim, m.heads * m.vdim
        own = m.q_rank + kv_n
        weight = const(np.concatenate([stored(f"{p}.{n}", size, H) for n, size in (("dq", m.q_rank), ("dkv", kv_n), ("g", v_n))]), dtype)
        norm, q_norm, kv_norm = (const(plain(n, size)) for n, size in ((f"{p[:-4]}.norm1", H), (f"{p}.dq.norm", m.q_rank), (f"{p}.dkv.norm", m.kv_rank)))
        uq, uv, out = matrix(f"{p}.uq", q_n, m.q_rank), matrix(f"{p}.uv", v_n, m.kv_rank), matrix(f"{p}.o", H, v_n)
        # keys of a head = uk · latent: a query meets the latent as ukᵀ · query
        uk = const(stored(f"{p}.uk", m.heads * m.dim, m.kv_rank).reshape(m.heads, m.dim, m.kv_rank).transpose(0, 2, 1).reshape(m.heads * m.kv_rank, m.dim), dtype)
        turns = const(turns_per_position(m.rot_dim, m.rot_base, 1.0))

        def run(n, pend):
            proj, x = norm_linear(f"{p}.in", pend, norm, weight, own + v_n, dtype, act_rest="sigmoid", act_split=own)
            q = linear(f"{p}.uq", {"norm": 1, "stream": 0, "epsilon": eps}, [proj, q_norm, uq], q_n, dtype)
            q_latent = linear(f"{p}.uk", {"ranges": 1, "blocks": m.heads, "x_step": m.dim + m.rot_dim}, [q, uk], m.heads * m.kv_rank, dtype)
            b.set_loc(p, "LatentAttention")
            o, pool = b.composite(
                "onyxia.LatentAttention", {"heads": m.heads, "rank": m.kv_rank, "rot": m.rot_dim, "q_offset": m.dim, "q_step": m.dim + m.rot_dim,
                                           "kv_offset": m.q_rank, "scale": m.scale, "epsilon": eps},
                [q_latent, q, proj, kv_norm, turns, *state[n], seqs, table], [(dtype, [N, m.heads * m.kv_rank]), (dtype, [NP, 1, PAGE, kv_n])])
            updated.append((f"pages.{n}.latents", pool))
            o = linear(f"{p}.uv", {"ranges": 1, "blocks": m.heads, "x_step": m.kv_rank, "mul": 1, "mul_offset": own}, [o, uv, proj], v_n, dtype)
            return x, linear(f"{p}.out", {}, [o, out], H)
        return run

    def mamba(p, m):
        cols = m.dt_rank + 2 * m.state
        norm, weight, out = const(plain(f"{p[:-4]}.norm1", H)), matrix(f"{p}.in", 2 * m.inner, H), matrix(f"{p}.o", H, m.inner)
        consts = [const(plain(f"{p}.conv", m.inner, m.taps)), const(plain(f"{p}.conv.b", m.inner)), matrix(f"{p}.x", cols, m.inner),
                  matrix(f"{p}.dt", m.inner, m.dt_rank), const(plain(f"{p}.dt.b", m.inner)),
                  const(-np.exp(plain(f"{p}.A_log", m.inner, m.state).astype(np.float64)).astype(np.float32)), const(plain(f"{p}.D", m.inner))]

        def run(n, pend):
            proj, x = norm_linear(f"{p}.in", pend, norm, weight, 2 * m.inner, dtype, act_rest="silu", act_split=m.inner)
            b.set_loc(p, "SelectiveScan")
            o, conv_state, new_state = b.composite(
                "onyxia.SelectiveScan", {"width": m.inner, "state": m.state, "rank": m.dt_rank, "taps": m.taps, "x_offset": 0, "z_offset": m.inner},
                [proj, *consts, *state[n], seqs], [(dtype, [N, m.inner]), (dtype, [NS, m.taps, m.inner]), (ir.F32, [NS, m.inner, m.state])])
            updated.extend([(f"slots.{n}.conv", conv_state), (f"slots.{n}.state", new_state)])
            return x, linear(f"{p}.out", {}, [o, out], H)
        return run

    def gated_pairs(p, ff):  # gate and up rows, interleaved
        return np.stack([stored(f"{p}.gate", ff, H), stored(f"{p}.up", ff, H)], axis=1).reshape(2 * ff, H)

    def dense(p, m):
        norm, up, down = const(plain(f"{p[:-4]}.norm2", H)), const(gated_pairs(p, m.ff), dtype), matrix(f"{p}.down", H, m.ff)

        def run(pend):
            act, x = norm_linear(f"{p}.in", pend, norm, up, m.ff, dtype, glu=1)
            return x, linear(f"{p}.down", {}, [act, down], H)
        return run

    def experts(p, m):
        up, down = np.empty((m.experts, 2 * m.ff, H), storage), np.empty((m.experts, H, m.ff), storage)
        for e in range(m.experts):
            up[e], down[e] = gated_pairs(f"{p}.e{e}", m.ff), stored(f"{p}.e{e}.down", H, m.ff)
        norm = const(plain(f"{p[:-4]}.norm2", H))
        consts = [matrix(f"{p}.router", m.experts, H), const(np.zeros(m.experts, np.float32)), const(up.reshape(-1, H), dtype), const(down.reshape(-1, m.ff), dtype)]
        extra = {"experts": m.experts, "top": m.top, "ff": m.ff, "alpha": GLU_ALPHA, "limit": m.limit, "shift": GLU_SHIFT, "scores": "sigmoid",
                 "route_scale": m.scale, "groups": m.groups, "keep": m.keep}
        if m.shared_ff:
            consts += [const(gated_pairs(f"{p}.shared", m.shared_ff), dtype), matrix(f"{p}.shared.down", H, m.shared_ff)]
            extra.update(shared_ff=m.shared_ff, shared_limit=m.shared_limit)

        def run(pend):
            attrs, ins = norm_inputs(pend, norm)
            b.set_loc(p, "MixtureOfExperts")
            y, x = b.composite("onyxia.MixtureOfExperts", {**attrs, **extra}, ins + consts, [(ir.F32, [N, H]), (ir.F32, [N, H])])
            return x, y
        return run

    b.set_loc("embed", "Gather")
    embed = b.constant(host_tensor(stored("embed", cfg.vocab, H), dtype), borrow=True)
    start = b.gather(embed, ids, 0)
    updated, made = [], {}
    for i in sorted({i for i, _ in runs}):
        m, f, p = cfg.layers[i].mixer, cfg.layers[i].mlp, f"l{i}"
        mixer = (mamba if isinstance(m, MambaConfig) else latent if isinstance(m, LatentConfig) else attention)(f"{p}.mix", m)
        mlp = None if f is None else (dense if isinstance(f, DenseConfig) else experts)(f"{p}.mlp", f)
        made[i] = (mixer, const(plain(f"{p}.norm1b", H)), mlp, None if f is None else const(plain(f"{p}.norm2b", H)))
    steps = plain("loop.step", cfg.loop[2], H) if cfg.loop[0] < cfg.loop[1] else None
    pend = {"y": start, "scale": cfg.embed_scale}
    for n, (i, t) in enumerate(runs):
        mixer, norm1b, mlp, norm2b = made[i]
        if t is not None:
            pend["offset"] = const(steps[t])
            if t > 0:
                pend["add"] = start
        x, y = mixer(n, pend)
        pend = {"residual": x, "y": y, "post": norm1b}
        if mlp is not None:
            x, y = mlp(pend)
            pend = {"residual": x, "y": y, "post": norm2b}

    # only the rows whose logits are wanted go on
    b.set_loc("logit_rows", "Gather")
    pend = {k: b.gather(v, rows, 0) if k in ("y", "residual") else v for k, v in pend.items()}
    logits, _ = norm_linear("head", pend, const(plain("final.norm", H)), embed, cfg.vocab, ir.F32, count=W)
    b.set_loc(None)
    b.output("logits", logits)
    for name, v in updated:
        b.output("updated." + name, v)
    return b.finish()


def tensor_shapes(cfg: ZusitarConfig) -> dict:
    """Names and shapes of a checkpoint of this configuration."""
    H = cfg.width
    out = {"embed": (cfg.vocab, H), "final.norm": (H,)}
    if cfg.loop[0] < cfg.loop[1]:
        out["loop.step"] = (cfg.loop[2], H)
    for i, l in enumerate(cfg.layers):
        p, m, f = f"l{i}.mix.", l.mixer, l.mlp
        out.update({f"l{i}.norm1": (H,), f"l{i}.norm1b": (H,)})
        if isinstance(m, MambaConfig):
            out.update({p + "in": (2 * m.inner, H), p + "conv": (m.inner, m.taps), p + "conv.b": (m.inner,), p + "x": (m.dt_rank + 2 * m.state, m.inner),
                        p + "dt": (m.inner, m.dt_rank), p + "dt.b": (m.inner,), p + "A_log": (m.inner, m.state), p + "D": (m.inner,), p + "o": (H, m.inner)})
        elif isinstance(m, LatentConfig):
            out.update({p + "dq": (m.q_rank, H), p + "dq.norm": (m.q_rank,), p + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                        p + "dkv": (m.kv_rank + m.rot_dim, H), p + "dkv.norm": (m.kv_rank,), p + "uk": (m.heads * m.dim, m.kv_rank),
                        p + "uv": (m.heads * m.vdim, m.kv_rank), p + "g": (m.heads * m.vdim, H), p + "o": (H, m.heads * m.vdim)})
        else:
            for n, size in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                out.update({p + n: (size, H), f"{p}{n}.b": (size,)})
            out.update({p + "sink": (m.heads,), p + "g": (m.heads, H), p + "o": (H, m.heads * m.vdim), p + "o.b": (H,)})
        if f is None:
            continue
        out.update({f"l{i}.norm2": (H,), f"l{i}.norm2b": (H,)})
        units = {"": f.ff} if isinstance(f, DenseConfig) else {**{f"e{e}.": f.ff for e in range(f.experts)}, **({"shared.": f.shared_ff} if f.shared_ff else {})}
        for n, ff in units.items():
            out.update({f"l{i}.mlp.{n}gate": (ff, H), f"l{i}.mlp.{n}up": (ff, H), f"l{i}.mlp.{n}down": (H, ff)})
        if not isinstance(f, DenseConfig):
            out[f"l{i}.mlp.router"] = (f.experts, H)
    return out


def random_weights(cfg: ZusitarConfig, seed: int = 0) -> Weights:
    """bf16 weights of a plausible scale (benchmarks, smoke runs). Large matrices repeat one random block."""
    rng = np.random.default_rng(seed)
    block = rng.standard_normal(1 << 20, dtype=np.float32)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last, n = name.rsplit(".", 1)[-1], int(np.prod(shape))
        if last in ("norm", "norm1", "norm2", "D"):
            a = 1.0 + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif last in ("norm1b", "norm2b"):
            a = 0.3 + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif name.endswith("dt.b"):
            a = rng.uniform(-6.0, -2.0, n).astype(np.float32)
        elif last in ("b", "sink", "step"):
            a = 0.1 * rng.standard_normal(n, dtype=np.float32)
        elif last == "A_log":
            a = np.log(np.arange(1, shape[1] + 1, dtype=np.float32))[None, :].repeat(shape[0], axis=0)
        else:
            at = int(rng.integers(0, 1 << 19))
            a = np.resize(block[at:], n) / (cfg.embed_scale if name == "embed" else math.sqrt(shape[-1]))
        out[name] = HostTensor.bf16(a.reshape(shape)).data.view(np.uint16).reshape(shape)
    return Weights.from_bf16(out)
