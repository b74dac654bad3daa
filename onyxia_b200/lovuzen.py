"""Lovuzen: a decoder whose layers run grouped-query attention and a gated linear recurrence side by side.

    x = norm(embed[token])
    every layer:  x += ls1 · norm1(left_scale · left(x) + right_scale · right(x))
                  x += ls2 · norm2(mlp(x))                        (layers may have no mlp)
    logits = head · norm(x)

left   grouped-query attention without rotation: queries and keys are RMS-normed over their whole projection, the values
       are the keys as projected, queries are scaled by a factor that grows with the logarithm of the position, and a learned
       bias per head and distance bucket is added to the scaled scores
right  a causal convolution and a real-gated linear recurrence, multiplied by the gelu of a second branch (the
       recurrent block of "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient Language Models", De et al.)
mlp    gated unit with clamped branches

The module runs ragged batches over paged key pools and state slots (csrc/backend/engine.hpp). All four projections that
read x are one product; left and right leave through one product over two operands; the norm of a sublayer's result,
its gain and the residual sum are the prologue of the next product.
"""
from __future__ import annotations

import dataclasses
import math

import numpy as np

from . import ir
from .checkpoint import Weights, host_tensor
from .ir import HostTensor

PAGE = 64            # tokens per cache page
DECAY = 8.0          # exponent of the recurrence's decay
GLU_ALPHA = 1.702
GLU_SHIFT = 1.0


@dataclasses.dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    bias_max: int
    temp_coef: float = 0.0
    temp_every: float = 0.0   # 0: no temperature


@dataclasses.dataclass
class RecurrenceConfig:
    width: int
    blocks: int
    taps: int


@dataclasses.dataclass
class MlpConfig:
    ff: int
    limit: float


@dataclasses.dataclass
class LayerConfig:
    left: AttentionConfig
    right: RecurrenceConfig
    left_scale: float
    right_scale: float
    mlp: MlpConfig | None


@dataclasses.dataclass
class LovuzenConfig:
    vocab: int
    width: int
    eps: float
    layers: list

    @staticmethod
    def from_dict(c: dict) -> "LovuzenConfig":
        layers = []
        for i, l in enumerate(c["layers"]):
            if l["type"] != "parallel":
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            m = l["mixer"]
            a, r, t = m["left"], m["right"], m["left"].get("q_temp")
            if a["heads"] % a["kv_heads"]:
                raise ValueError(f"layer {i}: {a['heads']} query heads over {a['kv_heads']} key heads")
            if a.get("vdim", a["dim"]) != a["dim"]:
                raise ValueError(f"layer {i}: the values are the keys, yet their sizes differ")
            if r["width"] % r["blocks"]:
                raise ValueError(f"layer {i}: width {r['width']} does not divide into {r['blocks']} blocks")
            mlp = l.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerConfig(
                AttentionConfig(a["heads"], a["kv_heads"], a["dim"], float(a["scale"]), a["bias_max"],
                                float(t["coef"]) if t else 0.0, float(t["every"]) if t else 0.0),
                RecurrenceConfig(r["width"], r["blocks"], r["conv"]),
                float(m["left_scale"]), float(m["right_scale"]),
                MlpConfig(mlp["ff"], float(mlp["limit"])) if mlp is not None else None))
        return LovuzenConfig(c["vocab"], c["width"], float(c["norm"]["eps"]), layers)

    def weight_bytes_per_token(self, element: int = 2) -> int:
        """Weight matrices one decode step reads."""
        n = self.vocab * self.width
        for l in self.layers:
            a, r = l.left, l.right
            n += self.width * ((a.heads + a.kv_heads) * a.dim + 2 * r.width) + self.width * (a.heads * a.dim + r.width)
            n += 2 * r.width * r.width // r.blocks
            n += 3 * self.width * l.mlp.ff if l.mlp else 0
        return n * element

    def cache_bytes_per_token(self, context: int, element: int = 2) -> int:
        """Cached keys one decode step of one sequence reads at a context length."""
        return sum((context + 1) * (l.left.kv_heads * l.left.dim * element + 4) for l in self.layers)


def distance_rows(rows: int, far: int) -> np.ndarray:
    """For every distance 0 … far the row of a `rows`-row bias table it reads: exact up to rows // 2, then rows spaced
    evenly in the logarithm of the distance, the last one from `far` on."""
    half = rows // 2
    if half < 1 or far <= half:
        raise ValueError(f"a bias table of {rows} rows cannot reach distance {far}")
    out = np.arange(far + 1)
    for n in range(half, far + 1):
        step = math.log(n / half) / math.log(far / half) * (rows - half)
        if abs(step - round(step)) < 1e-9:  # on a row's edge: the logarithms' rounding must not decide
            step = round(step)
        out[n] = min(rows - 1, half + math.floor(step))
    return out


def distance_bias(table: np.ndarray, far: int) -> np.ndarray:
    """[rows, heads] → [heads, far + 1]: the bias of every distance, the last column for all distances beyond."""
    return np.ascontiguousarray(table[distance_rows(table.shape[0], far)].T, dtype=np.float32)


def build(cfg: LovuzenConfig, w: Weights, dtype: int = ir.BF16) -> ir.Module:
    """The module in activation type `dtype`: BF16, or F32 for true 32-bit arithmetic."""
    if dtype not in (ir.BF16, ir.F32):
        raise ValueError(f"Lovuzen modules run in bf16 or f32, not {ir.DTYPE_NAMES[dtype]}")
    b = ir.GraphBuilder()
    N, R, W = b.sym("num_tokens"), b.sym("num_seqs"), b.sym("num_logits")
    NP, NS, TW = b.sym("num_pages"), b.sym("num_slots"), b.sym("table_width")
    H = cfg.width

    def const(a, dt=ir.F32):
        return b.constant(host_tensor(np.ascontiguousarray(a), dt))

    def vec(name, n):
        a = w.f32(name)
        if a.shape != (n,):
            raise ValueError(f"tensor '{name}' has shape {list(a.shape)}, expected [{n}]")
        return const(a)

    def stored(name, *shape):
        if w.shape(name) != shape:
            raise ValueError(f"tensor '{name}' has shape {list(w.shape(name))}, expected {list(shape)}")
        return w.stored(name, dtype)

    def matrix(name, rows, cols):
        return const(stored(name, rows, cols), dtype)

    ids = b.input("input_ids", ir.I64, [N])
    seqs = b.input("seq_info", ir.I32, [R, 4])
    table = b.input("page_table", ir.I32, [R, TW])
    rows = b.input("logit_rows", ir.I64, [W])
    state = []
    for i, l in enumerate(cfg.layers):
        a, r = l.left, l.right
        state.append((b.input(f"pages.{i}.keys", dtype, [NP, a.kv_heads, PAGE, a.dim]),
                      b.input(f"pages.{i}.key_scale", ir.F32, [NP, PAGE]),
                      b.input(f"slots.{i}.conv", dtype, [NS, r.taps, r.width]),
                      b.input(f"slots.{i}.recurrence", ir.F32, [NS, r.width])))

    # A residual norm that has not run yet: (residual or None, sublayer result, weight, gain or None). It becomes
    # the prologue of the next product.
    def norm_inputs(pend):
        res, y, weight, gain = pend
        attrs = {"epsilon": float(cfg.eps), "residual": int(res is not None), "gain": int(gain is not None)}
        return attrs, [y, weight] + ([res] if res is not None else []) + ([gain] if gain is not None else [])

    def norm_linear(name, pend, weight, out, dt, count=N, bias=None, glu=None):
        attrs, ins = norm_inputs(pend)
        attrs.update({"norm": 1, "bias": int(bias is not None)})
        if glu is not None:
            attrs.update({"glu": 1, "alpha": GLU_ALPHA, "limit": float(glu), "shift": GLU_SHIFT})
        b.set_loc(name, "Linear")
        return b.composite("onyxia.Linear", attrs, ins + [weight] + ([bias] if bias is not None else []),
                           [(dt, [count, out]), (ir.F32, [count, H])])

    b.set_loc("embed", "Gather")
    x = b.gather(b.constant(host_tensor(stored("embed", cfg.vocab, H), dtype), borrow=True), ids, 0)
    pend = (None, x, vec("embed.norm", H), None)
    updated = []
    for i, l in enumerate(cfg.layers):
        p, a, r = f"l{i}", l.left, l.right
        q_n, k_n = a.heads * a.dim, a.kv_heads * a.dim
        lp, rp = f"{p}.mix.left", f"{p}.mix.right"
        weight = np.concatenate([stored(f"{lp}.q", q_n, H), stored(f"{lp}.k", k_n, H), stored(f"{rp}.y", r.width, H),
                                 stored(f"{rp}.x", r.width, H)])
        bias = np.concatenate([np.zeros(q_n + k_n, np.float32), w.f32(f"{rp}.y.b"), w.f32(f"{rp}.x.b")])
        proj, x = norm_linear(f"{p}.mix.in", pend, const(weight, dtype), weight.shape[0], dtype, bias=const(bias))
        rel = w.f32(f"{lp}.rel")
        if rel.shape[1:] != (a.heads,):
            raise ValueError(f"tensor '{lp}.rel' has shape {list(rel.shape)}, expected [rows, {a.heads}]")
        b.set_loc(lp, "PagedAttention")
        left, keys, key_scale = b.composite(
            "onyxia.PagedAttention",
            {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "q_offset": 0, "k_offset": q_n, "scale": float(a.scale),
             "epsilon": float(cfg.eps), "temp_coef": float(a.temp_coef), "temp_every": float(a.temp_every), "out_scale": float(l.left_scale)},
            [proj, vec(f"{lp}.q.norm", q_n), vec(f"{lp}.k.norm", k_n), const(distance_bias(rel, a.bias_max)),
             state[i][0], state[i][1], seqs, table],
            [(dtype, [N, q_n]), (dtype, [NP, a.kv_heads, PAGE, a.dim]), (ir.F32, [NP, PAGE])])
        n = r.width // r.blocks
        b.set_loc(rp, "GatedRecurrence")
        conv = w.f32(f"{rp}.conv")
        if conv.shape != (r.width, r.taps):
            raise ValueError(f"tensor '{rp}.conv' has shape {list(conv.shape)}, expected [{r.width}, {r.taps}]")
        right, conv_state, recurrence = b.composite(
            "onyxia.GatedRecurrence",
            {"width": r.width, "blocks": r.blocks, "taps": r.taps, "y_offset": q_n + k_n, "x_offset": q_n + k_n + r.width,
             "decay": DECAY, "out_scale": float(l.right_scale)},
            [proj, const(conv), vec(f"{rp}.conv.b", r.width),
             const(stored(f"{rp}.ra", r.blocks, n, n), dtype), const(w.f32(f"{rp}.ra.b").reshape(-1)),
             const(stored(f"{rp}.ri", r.blocks, n, n), dtype), const(w.f32(f"{rp}.ri.b").reshape(-1)),
             vec(f"{rp}.lam", r.width), state[i][2], state[i][3], seqs],
            [(dtype, [N, r.width]), (dtype, [NS, r.taps, r.width]), (ir.F32, [NS, r.width])])
        updated += [(f"pages.{i}.keys", keys), (f"pages.{i}.key_scale", key_scale),
                    (f"slots.{i}.conv", conv_state), (f"slots.{i}.recurrence", recurrence)]
        b.set_loc(f"{p}.mix.out", "Linear")
        mixed = b.composite("onyxia.Linear", {"pair": 1},
                            [left, right, matrix(f"{lp}.o", H, q_n), matrix(f"{rp}.o", H, r.width)], [(ir.F32, [N, H])])[0]
        pend = (x, mixed, vec(f"{p}.norm1", H), vec(f"{p}.ls1", H))
        if l.mlp is not None:
            ff = l.mlp.ff
            pairs = np.stack([stored(f"{p}.mlp.gate", ff, H), stored(f"{p}.mlp.up", ff, H)], axis=1).reshape(2 * ff, H)
            act, x = norm_linear(f"{p}.mlp.in", pend, const(pairs, dtype), ff, dtype, glu=l.mlp.limit)
            b.set_loc(f"{p}.mlp.down", "Linear")
            down = b.composite("onyxia.Linear", {}, [act, matrix(f"{p}.mlp.down", H, ff)], [(ir.F32, [N, H])])[0]
            pend = (x, down, vec(f"{p}.norm2", H), vec(f"{p}.ls2", H))

    # only the rows whose logits are wanted go on
    res, y, weight, gain = pend
    b.set_loc("logit_rows", "Gather")
    y = b.gather(y, rows, 0)
    res = b.gather(res, rows, 0) if res is not None else None
    attrs, ins = norm_inputs((res, y, weight, gain))
    b.set_loc("final.residual", "ResidualNorm")
    x = b.composite("onyxia.ResidualNorm", attrs, ins, [(ir.F32, [W, H])])[0]
    logits, _ = norm_linear("head", (None, x, vec("final.norm", H), None), matrix("head", cfg.vocab, H), cfg.vocab, ir.F32, count=W)
    b.set_loc(None)
    b.output("logits", logits)
    for name, v in updated:
        b.output("updated." + name, v)
    return b.finish()


def tensor_shapes(cfg: LovuzenConfig, bias_rows: int = 32) -> dict:
    """Names and shapes of a checkpoint of this configuration."""
    H = cfg.width
    out = {"embed": (cfg.vocab, H), "embed.norm": (H,), "final.norm": (H,), "head": (cfg.vocab, H)}
    for i, l in enumerate(cfg.layers):
        p, a, r = f"l{i}", l.left, l.right
        lp, rp, n = f"{p}.mix.left", f"{p}.mix.right", r.width // r.blocks
        out.update({f"{p}.norm1": (H,), f"{p}.ls1": (H,), f"{lp}.q": (a.heads * a.dim, H), f"{lp}.k": (a.kv_heads * a.dim, H),
                    f"{lp}.q.norm": (a.heads * a.dim,), f"{lp}.k.norm": (a.kv_heads * a.dim,), f"{lp}.rel": (bias_rows, a.heads),
                    f"{lp}.o": (H, a.heads * a.dim), f"{rp}.y": (r.width, H), f"{rp}.y.b": (r.width,), f"{rp}.x": (r.width, H),
                    f"{rp}.x.b": (r.width,), f"{rp}.conv": (r.width, r.taps), f"{rp}.conv.b": (r.width,),
                    f"{rp}.ra": (r.blocks, n, n), f"{rp}.ra.b": (r.blocks, n), f"{rp}.ri": (r.blocks, n, n),
                    f"{rp}.ri.b": (r.blocks, n), f"{rp}.lam": (r.width,), f"{rp}.o": (H, r.width)})
        if l.mlp is not None:
            out.update({f"{p}.norm2": (H,), f"{p}.ls2": (H,), f"{p}.mlp.gate": (l.mlp.ff, H), f"{p}.mlp.up": (l.mlp.ff, H),
                        f"{p}.mlp.down": (H, l.mlp.ff)})
    return out


def random_weights(cfg: LovuzenConfig, seed: int = 0, bias_rows: int = 32) -> Weights:
    """bf16 weights of a plausible scale (benchmarks, smoke runs). Large matrices repeat one random block."""
    rng = np.random.default_rng(seed)
    block = rng.standard_normal(1 << 20, dtype=np.float32)
    out = {}
    for name, shape in tensor_shapes(cfg, bias_rows).items():
        last, n = name.rsplit(".", 1)[-1], int(np.prod(shape))
        if last in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif last in ("ls1", "ls2"):
            a = 0.5 + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif last == "lam":
            a = rng.uniform(-6.0, -1.0, n).astype(np.float32)
        elif last in ("b", "rel"):
            a = 0.1 * rng.standard_normal(n, dtype=np.float32)
        elif last == "conv":
            a = rng.standard_normal(n, dtype=np.float32) / math.sqrt(shape[1])
        else:
            at = int(rng.integers(0, 1 << 19))
            a = np.resize(block[at:], n) * (1.0 if name == "embed" else 1.0 / math.sqrt(shape[-1]))
        out[name] = HostTensor.bf16(a.reshape(shape)).data.view(np.uint16).reshape(shape)
    return Weights.from_bf16(out)
