"""Kipizen: a decoder whose layers are either softmax attention in a window or lightning attention, in any order, each
followed by a mixture of experts.

    x = scale · embed[token]
    every layer:  x += mixer(norm1(x))
                  x += experts(norm2(x))                          (layers may have none)
    logits = head · norm(x)

attention  grouped-query attention with biased projections: rotation of the leading dimensions of a head with all frequencies
           divided by a factor, queries and keys divided by their root mean square after it, capped scores, a window, a
           sink of score 0 in the softmax. A layer may read the keys and values of an earlier one
lightning  linear attention with a matrix state per head that decays by a constant; the heads' results are normed
           together, gated and projected
experts    the router's best few, weighted by the softmax over their logits; gated units with silu

The module runs ragged batches over paged pools and state slots (csrc/backend/engine.hpp). The projections of a mixer are
one product with the norm in front of it as its prologue; norm and gate behind lightning attention are the prologue of its
output product; norm and router run in front of the experts.
"""
from __future__ import annotations

import dataclasses
import math

import numpy as np

from . import ir
from .checkpoint import Weights, host_tensor
from .ir import HostTensor

PAGE = 64    # tokens per cache page
CHUNK = 64   # tokens per chunk of lightning attention (csrc/kernels/kernels.hpp)


@dataclasses.dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_factor: float = 1.0
    softcap: float = 0.0      # 0: none
    window: int = 0           # 0: all keys
    kv_from: int | None = None


@dataclasses.dataclass
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: list


@dataclasses.dataclass
class ExpertsConfig:
    experts: int
    top: int
    ff: int


@dataclasses.dataclass
class LayerConfig:
    mixer: AttentionConfig | LightningConfig
    experts: ExpertsConfig | None


def _attention(i: int, m: dict, layers: list) -> AttentionConfig:
    rot, mask = m.get("rot"), m.get("mask")
    a = AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                        window=int(mask["size"]) if mask else 0, kv_from=m.get("kv_from"))
    if rot:
        a.rot_dims, a.rot_base = rot["dims"], float(rot["base"])
        a.rot_factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    if a.heads % a.kv_heads:
        raise ValueError(f"layer {i}: {a.heads} query heads over {a.kv_heads} key heads")
    if a.rot_dims % 2 or a.rot_dims > a.dim:
        raise ValueError(f"layer {i}: {a.rot_dims} of {a.dim} dimensions cannot rotate in pairs")
    if mask and a.window < 1:
        raise ValueError(f"layer {i}: a window of {a.window} tokens")
    if a.kv_from is not None:
        source = layers[a.kv_from].mixer if 0 <= a.kv_from < i else None
        if not isinstance(source, AttentionConfig) or source.kv_from is not None:
            raise ValueError(f"layer {i}: layer {a.kv_from} has no keys of its own before it")
        if (source.kv_heads, source.dim, source.vdim) != (a.kv_heads, a.dim, a.vdim):
            raise ValueError(f"layer {i}: its keys and values differ in size from those of layer {a.kv_from}")
    return a


def _lightning(i: int, m: dict) -> LightningConfig:
    decay = [float(v) for v in m["decay"]]
    if len(decay) != m["heads"]:
        raise ValueError(f"layer {i}: {len(decay)} decays for {m['heads']} heads")
    return LightningConfig(m["heads"], m["dim"], m["vdim"], decay)


@dataclasses.dataclass
class KipizenConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: list

    @staticmethod
    def from_dict(c: dict) -> "KipizenConfig":
        layers = []
        for i, l in enumerate(c["layers"]):
            if l["type"] == "attention":
                mixer = _attention(i, l["mixer"], layers)
            elif l["type"] == "lightning":
                mixer = _lightning(i, l["mixer"])
            else:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            mlp, experts = l.get("mlp"), None
            if mlp is not None:
                if mlp["kind"] != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
                experts = ExpertsConfig(mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"])
                if not 1 <= experts.top <= experts.experts:
                    raise ValueError(f"layer {i}: {experts.top} of {experts.experts} experts")
            layers.append(LayerConfig(mixer, experts))
        return KipizenConfig(c["vocab"], c["width"], float(c["norm"]["eps"]), float(c["embedding"]["scale"]), layers)


def turns_per_position(dims: int, base: float, factor: float) -> np.ndarray:
    """[2, dims / 2] f32: how many turns each pair of dimensions makes per position, as the sum of two f32."""
    if not dims:
        return np.zeros((2, 1), np.float32)
    turns = np.array([base ** (-2.0 * i / dims) / factor / (2.0 * math.pi) for i in range(dims // 2)])
    high = turns.astype(np.float32)
    return np.stack([high, (turns - high).astype(np.float32)])


def decay_table(decay) -> np.ndarray:
    """[heads, CHUNK + 2] f32: powers 0 … CHUNK of every decay, then the decay minus one."""
    d = np.asarray(decay, np.float64)[:, None]
    return np.concatenate([d ** np.arange(CHUNK + 1), d - 1.0], axis=1).astype(np.float32)


def build(cfg: KipizenConfig, w: Weights, dtype: int = ir.BF16) -> ir.Module:
    """The module in activation type `dtype`: BF16, or F32 for true 32-bit arithmetic."""
    if dtype not in (ir.BF16, ir.F32):
        raise ValueError(f"Kipizen modules run in bf16 or f32, not {ir.DTYPE_NAMES[dtype]}")
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

    own_kv = [isinstance(l.mixer, AttentionConfig) and l.mixer.kv_from is None for l in cfg.layers]
    ids = b.input("input_ids", ir.I64, [N])
    seqs = b.input("seq_info", ir.I32, [R, 4])
    table = b.input("page_table", ir.I32, [R, TW]) if any(own_kv) else None
    rows = b.input("logit_rows", ir.I64, [W])
    state = {}
    for i, l in enumerate(cfg.layers):
        m = l.mixer
        if isinstance(m, LightningConfig):
            state[i] = (b.input(f"slots.{i}.state", ir.F32, [NS, m.heads, m.dim, m.vdim]),)
        elif own_kv[i]:
            state[i] = (b.input(f"pages.{i}.keys", dtype, [NP, m.kv_heads, PAGE, m.dim]),
                        b.input(f"pages.{i}.values", dtype, [NP, m.kv_heads, PAGE, m.vdim]))

    # A sum that has not been formed yet: (residual or None, sublayer result, its factor). The norm that reads it forms it
    # and leaves the new residual.
    def norm_inputs(pend, weight):
        res, y, scale = pend
        return ({"epsilon": float(cfg.eps), "residual": int(res is not None), "pre": 1, "y_scale": float(scale)},
                [y, weight] + ([res] if res is not None else []))

    def norm_linear(name, pend, norm, weight, out, dt, count=N, bias=None, **extra):
        attrs, ins = norm_inputs(pend, norm)
        attrs.update({"norm": 1, "bias": int(bias is not None)}, **extra)
        b.set_loc(name, "Linear")
        return b.composite("onyxia.Linear", attrs, ins + [weight] + ([bias] if bias is not None else []),
                           [(dt, [count, out]), (ir.F32, [count, H])])

    def attention(i, m, p, pend, norm):
        q_n, k_n, v_n = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        parts = [("q", q_n)] + ([("k", k_n), ("v", v_n)] if own_kv[i] else [])
        weight = np.concatenate([stored(f"{p}.mix.{n}", size, H) for n, size in parts])
        bias = np.concatenate([w.f32(f"{p}.mix.{n}.b") for n, _ in parts])
        if bias.shape != (weight.shape[0],):
            raise ValueError(f"layer {i}: {bias.size} biases for {weight.shape[0]} projected dimensions")
        proj, x = norm_linear(f"{p}.mix.in", pend, norm, const(weight, dtype), weight.shape[0], dtype, bias=const(bias))
        attrs = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "q_offset": 0, "rot_dims": m.rot_dims,
                 "window": m.window, "scale": float(m.scale), "softcap": float(m.softcap), "epsilon": float(cfg.eps), "norm": 1, "sink": 1}
        turns, out = const(turns_per_position(m.rot_dims, m.rot_base, m.rot_factor)), (dtype, [N, m.heads * m.vdim])
        if own_kv[i]:
            b.set_loc(f"{p}.mix", "PagedKVAttention")
            o, keys, values = b.composite(
                "onyxia.PagedKVAttention", dict(attrs, k_offset=q_n, v_offset=q_n + k_n), [proj, turns, *state[i], seqs, table],
                [out, (dtype, [NP, m.kv_heads, PAGE, m.dim]), (dtype, [NP, m.kv_heads, PAGE, m.vdim])])
            pools[i] = (keys, values)
            updated.extend([(f"pages.{i}.keys", keys), (f"pages.{i}.values", values)])
        else:
            b.set_loc(f"{p}.mix", "SharedKVAttention")
            o = b.composite("onyxia.SharedKVAttention", attrs, [proj, turns, *pools[m.kv_from], seqs, table], [out])[0]
        b.set_loc(f"{p}.mix.out", "Linear")
        return x, b.composite("onyxia.Linear", {}, [o, matrix(f"{p}.mix.o", H, m.heads * m.vdim)], [(ir.F32, [N, H])])[0]

    def lightning(i, m, p, pend, norm):
        qk, vg = m.heads * m.dim, m.heads * m.vdim
        weight = np.concatenate([stored(f"{p}.mix.{n}", size, H) for n, size in (("q", qk), ("k", qk), ("v", vg), ("g", vg))])
        proj, x = norm_linear(f"{p}.mix.in", pend, norm, const(weight, dtype), weight.shape[0], dtype, act="silu", act_rest="sigmoid",
                              act_split=2 * qk + vg)
        b.set_loc(f"{p}.mix", "LightningAttention")
        o, new_state = b.composite("onyxia.LightningAttention", {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_offset": 0, "k_offset": qk,
                                                                 "v_offset": 2 * qk},
                                   [proj, const(decay_table(m.decay)), *state[i], seqs],
                                   [(ir.F32, [N, vg]), (ir.F32, [NS, m.heads, m.dim, m.vdim])])
        updated.append((f"slots.{i}.state", new_state))
        b.set_loc(f"{p}.mix.out", "Linear")
        y = b.composite("onyxia.Linear", {"norm": 1, "stream": 0, "epsilon": float(cfg.eps), "gate": 1, "gate_offset": 2 * qk + vg},
                        [o, vec(f"{p}.mix.norm", vg), proj, matrix(f"{p}.mix.o", H, vg)], [(ir.F32, [N, H])])[0]
        return x, y

    def experts(m, p, pend, norm):
        E, F = m.experts, m.ff
        up, down = np.empty((E, F, 2, H), _storage(dtype)), np.empty((E, H, F), _storage(dtype))
        for e in range(E):
            up[e, :, 0], up[e, :, 1] = stored(f"{p}.mlp.e{e}.gate", F, H), stored(f"{p}.mlp.e{e}.up", F, H)
            down[e] = stored(f"{p}.mlp.e{e}.down", H, F)
        attrs, ins = norm_inputs(pend, norm)
        attrs.update({"experts": E, "top": m.top, "ff": F})
        b.set_loc(f"{p}.mlp", "MixtureOfExperts")
        y, x = b.composite("onyxia.MixtureOfExperts", attrs,
                           ins + [matrix(f"{p}.mlp.router", E, H), vec(f"{p}.mlp.router.b", E), const(up.reshape(2 * E * F, H), dtype),
                                  const(down.reshape(E * H, F), dtype)],
                           [(ir.F32, [N, H]), (ir.F32, [N, H])])
        return x, y

    b.set_loc("embed", "Gather")
    x = b.gather(b.constant(host_tensor(stored("embed", cfg.vocab, H), dtype), borrow=True), ids, 0)
    pend = (None, x, cfg.embed_scale)
    pools, updated = {}, []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}"
        mixer = lightning if isinstance(l.mixer, LightningConfig) else attention
        pend = (*mixer(i, l.mixer, p, pend, vec(f"{p}.norm1", H)), 1.0)
        if l.experts is not None:
            pend = (*experts(l.experts, p, pend, vec(f"{p}.norm2", H)), 1.0)

    # only the rows whose logits are wanted go on
    res, y, scale = pend
    b.set_loc("logit_rows", "Gather")
    pend = (b.gather(res, rows, 0) if res is not None else None, b.gather(y, rows, 0), scale)
    logits, _ = norm_linear("head", pend, vec("final.norm", H), matrix("head", cfg.vocab, H), cfg.vocab, ir.F32, count=W)
    b.set_loc(None)
    b.output("logits", logits)
    for name, v in updated:
        b.output("updated." + name, v)
    return b.finish()


def _storage(dtype: int):
    return np.uint16 if dtype == ir.BF16 else np.float32  # bf16 travels as bit patterns


def tensor_shapes(cfg: KipizenConfig) -> dict:
    """Names and shapes of a checkpoint of this configuration."""
    H = cfg.width
    out = {"embed": (cfg.vocab, H), "final.norm": (H,), "head": (cfg.vocab, H)}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        out[p + "norm1"] = (H,)
        if isinstance(m, LightningConfig):
            qk, vg = m.heads * m.dim, m.heads * m.vdim
            out.update({p + "mix.q": (qk, H), p + "mix.k": (qk, H), p + "mix.v": (vg, H), p + "mix.g": (vg, H), p + "mix.norm": (vg,),
                        p + "mix.o": (H, vg)})
        else:
            sizes = [("q", m.heads * m.dim)]
            if m.kv_from is None:
                sizes += [("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)]
            for n, size in sizes:
                out.update({f"{p}mix.{n}": (size, H), f"{p}mix.{n}.b": (size,)})
            out[p + "mix.o"] = (H, m.heads * m.vdim)
        if l.experts is not None:
            out.update({p + "norm2": (H,), p + "mlp.router": (l.experts.experts, H), p + "mlp.router.b": (l.experts.experts,)})
            for e in range(l.experts.experts):
                out.update({f"{p}mlp.e{e}.gate": (l.experts.ff, H), f"{p}mlp.e{e}.up": (l.experts.ff, H), f"{p}mlp.e{e}.down": (H, l.experts.ff)})
    return out


def random_weights(cfg: KipizenConfig, seed: int = 0) -> Weights:
    """bf16 weights of a plausible scale (benchmarks, smoke runs). Large matrices repeat one random block."""
    rng = np.random.default_rng(seed)
    block = rng.standard_normal(1 << 20, dtype=np.float32)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last, n = name.rsplit(".", 1)[-1], int(np.prod(shape))
        if last in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.05 * rng.standard_normal(n, dtype=np.float32)
        elif last == "b":
            a = 0.1 * rng.standard_normal(n, dtype=np.float32)
        else:
            at = int(rng.integers(0, 1 << 19))
            a = np.resize(block[at:], n) / (cfg.embed_scale if name == "embed" else math.sqrt(shape[-1]))
        out[name] = HostTensor.bf16(a.reshape(shape)).data.view(np.uint16).reshape(shape)
    return Weights.from_bf16(out)
