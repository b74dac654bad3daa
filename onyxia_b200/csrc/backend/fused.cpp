// Fused-composite registry (≙ standard_kernels,
// crates/onyxia-backend-wgpu/src/fused.rs:71-86). Registry membership is what
// `Backend::supports` reports; `accepts` narrows a kernel to the operand types
// it implements, every other instance of the composite is legalised through
// its decomposition.
#include <cmath>

#include "../kernels/common.cuh"
#include "runtime.hpp"

namespace oxrt {

using namespace ox;
using oxk::TRef;

namespace {

const TensorType& ty(const Module& m, ValueId v) { return m.values[v].ty; }
bool is_float(DType d) { return d == DType::F32 || d == DType::F16; }

// ── Softmax ──
bool softmax_accepts(const Module& m, const Node& n) {
    if (n.inputs.size() != 1) return false;
    const TensorType& x = ty(m, n.inputs[0]);
    if (!is_float(x.dtype) || x.shape.empty()) return false;
    auto* a = n.composite.attrs.get("axis");
    return a && a->kind == AttrValue::Int && (size_t)a->i == x.shape.size() - 1;
}
void softmax_lower(FusedCtx& c) { oxk::emit_softmax(c.em, c.ins[0], c.outs[0]); }

// ── SimplifiedLayerNormalization ──
bool rmsnorm_accepts(const Module& m, const Node& n) {
    if (n.inputs.size() != 2) return false;
    const TensorType &x = ty(m, n.inputs[0]), &w = ty(m, n.inputs[1]);
    if (!is_float(x.dtype) || w.dtype != x.dtype || x.shape.empty()) return false;
    return w.shape.size() == 1 && w.shape[0] == x.shape.back();
}
void rmsnorm_lower(FusedCtx& c) {
    double eps = c.node.composite.attrs.float_or("epsilon", 1e-5);
    oxk::emit_rmsnorm(c.em, c.ins[0], c.ins[1], c.outs[0], eps, nullptr, nullptr);
}

// ── Gelu ──
bool gelu_accepts(const Module& m, const Node& n) { return n.inputs.size() == 1 && is_float(ty(m, n.inputs[0]).dtype); }
void gelu_lower(FusedCtx& c) {
    bool tanh = c.node.composite.attrs.str_or("approximate", "none") == "tanh";
    oxk::emit_gelu(c.em, c.ins[0], c.outs[0], tanh, nullptr);
}

// ── RotaryEmbedding ──
// Head count and rotary width are resolved exactly like the decomposition
// (crates/onyxia-ir/src/decomp.rs:283-311).
bool rotary_geometry(const Module& m, const Node& n, int64_t* heads, int64_t* half) {
    const TensorType &x = ty(m, n.inputs[0]), &cosc = ty(m, n.inputs[2]);
    auto hidden = x.shape[2].as_const();
    auto cache_half = cosc.shape[1].as_const();
    if (!hidden || !cache_half) return false;
    int64_t nh = n.composite.attrs.int_or("num_heads", 0);
    int64_t h;
    if (nh > 0) h = nh;
    else {
        int64_t r = (int64_t)*cache_half * 2;
        h = (r > 0 && (int64_t)*hidden % r == 0) ? (int64_t)*hidden / r : 1;
    }
    if ((int64_t)*hidden % h != 0) return false;
    int64_t rdim = n.composite.attrs.int_or("rotary_embedding_dim", 0);
    int64_t hf = rdim == 0 ? (int64_t)*cache_half : rdim / 2;
    int64_t d = (int64_t)*hidden / h;
    if (hf <= 0 || 2 * hf > d || hf > (int64_t)*cache_half) return false;
    // the decomposition reshapes the gathered cache row to `half` columns
    if (hf != (int64_t)*cache_half) return false;
    *heads = h;
    *half = hf;
    return true;
}
bool rotary_accepts(const Module& m, const Node& n) {
    if (n.inputs.size() != 4) return false;
    if (n.composite.attrs.int_or("interleaved", 0) != 0) return false;
    const TensorType &x = ty(m, n.inputs[0]), &pos = ty(m, n.inputs[1]), &cosc = ty(m, n.inputs[2]), &sinc = ty(m, n.inputs[3]);
    if (!is_float(x.dtype) || x.shape.size() != 3 || pos.dtype != DType::I64 || pos.shape.size() != 2) return false;
    if (cosc.dtype != x.dtype || sinc.dtype != x.dtype || cosc.shape.size() != 2 || sinc.shape != cosc.shape) return false;
    int64_t h, hf;
    return rotary_geometry(m, n, &h, &hf);
}
// geometry is recomputed from concrete shapes at lowering time
void rotary_lower(FusedCtx& c) {
    int64_t hidden = c.ins[0].shape[2], cache_half = c.ins[2].shape[1];
    int64_t nh = c.node.composite.attrs.int_or("num_heads", 0);
    int64_t heads = nh > 0 ? nh : ((cache_half > 0 && hidden % (2 * cache_half) == 0) ? hidden / (2 * cache_half) : 1);
    oxk::emit_rotary(c.em, c.ins[0], c.ins[1], c.ins[2], c.ins[3], c.outs[0], heads, cache_half);
}

// ── GroupQueryAttention ──
bool gqa_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() < 6) return false;
    int64_t heads = a.int_or("num_heads", 0), kv = a.int_or("kv_num_heads", 0);
    if (heads <= 0 || kv <= 0 || heads % kv != 0) return false;
    bool rot = a.int_or("do_rotary", 0) != 0, bias = a.int_or("has_attention_bias", 0) != 0;
    if (n.inputs.size() != (size_t)(6 + (rot ? 2 : 0) + (bias ? 1 : 0))) return false;
    if (rot && a.int_or("rotary_interleaved", 0) != 0) return false;
    const TensorType &q = ty(m, n.inputs[0]), &k = ty(m, n.inputs[1]), &v = ty(m, n.inputs[2]);
    const TensorType &pk = ty(m, n.inputs[3]), &pv = ty(m, n.inputs[4]), &sl = ty(m, n.inputs[5]);
    if (!is_float(q.dtype) || k.dtype != q.dtype || v.dtype != q.dtype || pk.dtype != q.dtype || pv.dtype != q.dtype) return false;
    if (sl.dtype != DType::I32) return false;
    if (q.shape.size() != 3 || k.shape.size() != 3 || v.shape.size() != 3 || pk.shape.size() != 4 || pv.shape.size() != 4) return false;
    auto hidden = q.shape[2].as_const();
    if (!hidden || *hidden % (uint64_t)heads != 0) return false;
    uint64_t d = *hidden / (uint64_t)heads;
    if (d != 32 && d != 64 && d != 128 && d != 256) return false;
    if (pk.shape[3].as_const() != std::optional<uint64_t>(d) || pk.shape[1].as_const() != std::optional<uint64_t>((uint64_t)kv)) return false;
    if (pv.shape != pk.shape) return false;
    if (rot) {
        const TensorType &cosc = ty(m, n.inputs[6]), &sinc = ty(m, n.inputs[7]);
        if (cosc.dtype != q.dtype || sinc.dtype != q.dtype || cosc.shape.size() != 2 || sinc.shape != cosc.shape) return false;
        auto half = cosc.shape[1].as_const();
        if (!half || *half == 0 || 2 * *half > d) return false;
    }
    if (bias) {
        const TensorType& bt = ty(m, n.inputs.back());
        if (bt.dtype != q.dtype || bt.shape.size() != 4) return false;
    }
    if (a.float_or("scale", 0.0) == 0.0 && !q.shape[2].as_const()) return false;
    return true;
}
void gqa_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::GqaDesc d{};
    d.batch = c.ins[0].shape[0];
    d.seq = c.ins[0].shape[1];
    d.heads = a.int_("num_heads");
    d.kv_heads = a.int_("kv_num_heads");
    d.head_dim = c.ins[0].shape[2] / d.heads;
    d.past = c.ins[3].shape[2];
    double sc = a.float_or("scale", 0.0);
    d.scale = sc == 0.0 ? 1.0 / std::sqrt((double)d.head_dim) : sc;
    d.window = a.int_or("local_window_size", -1);
    bool rot = a.int_or("do_rotary", 0) != 0;
    d.has_bias = a.int_or("has_attention_bias", 0) != 0;
    const TRef *cosr = nullptr, *sinr = nullptr, *biasr = nullptr;
    if (rot) {
        cosr = &c.ins[6];
        sinr = &c.ins[7];
        d.rot_half = cosr->shape[1];
        d.cache_rows = cosr->shape[0];
        // ≙ the rope-cache bound of the reference kernel (fused.rs:417-422)
        if (d.past + d.seq > d.cache_rows)
            fail(ErrKind::Shape, "GQA rope cache has " + std::to_string(d.cache_rows) + " positions but the sequence reaches " +
                                     std::to_string(d.past + d.seq));
    }
    if (c.ins[5].numel() != d.batch)
        fail(ErrKind::Shape, "GQA seqlens_k has " + std::to_string(c.ins[5].numel()) + " elements for batch size " + std::to_string(d.batch));
    if (d.has_bias) {
        biasr = &c.ins.back();
        const auto& bs = biasr->shape;
        int64_t T = d.past + d.seq;
        bool ok = (bs[0] == d.batch || bs[0] == 1) && (bs[1] == d.heads || bs[1] == 1) && bs[2] == d.seq && bs[3] == T;
        if (!ok) fail(ErrKind::Shape, "GQA attention_bias does not broadcast over the scores");
        d.bias_b = bs[0];
        d.bias_h = bs[1];
    }
    d.in_place = c.kv_in_place;
    // A decode step on a cache that is appended to in place: size the launch for
    // the next multiple of 256 rows and pass the true length as a per-run scalar.
    if (d.in_place && d.seq == 1 && !d.has_bias) {
        d.t_bucket = (d.past + d.seq + 255) / 256 * 256;
        c.bucket = d.t_bucket;
        c.bucket_step = 256;
    }
    oxk::emit_gqa(c.em, d, c.ins[0], c.ins[1], c.ins[2], c.ins[3], c.ins[4], c.ins[5], cosr, sinr, biasr, c.outs[0], c.outs[1], c.outs[2]);
}

// ── MatMulNBits ──
bool nbits_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() < 3 || n.inputs.size() > 4) return false;
    if (a.int_or("bits", 4) != 4 || a.int_or("block_size", 0) != 32) return false;
    const TensorType &x = ty(m, n.inputs[0]), &w = ty(m, n.inputs[1]), &s = ty(m, n.inputs[2]);
    if (!is_float(x.dtype) || !is_float(s.dtype) || w.dtype != DType::U4 || x.shape.empty()) return false;
    int64_t K = a.int_or("K", 0), N = a.int_or("N", 0);
    if (K <= 0 || N <= 0) return false;
    auto wd = shape_as_static(w.shape);
    if (!wd || wd->size() != 3 || (*wd)[0] != (uint64_t)N || (*wd)[2] != 32 || (*wd)[1] != (uint64_t)((K + 31) / 32)) return false;
    if (x.shape.back().as_const() != std::optional<uint64_t>((uint64_t)K)) return false;
    auto sd = shape_as_static(s.shape);
    if (!sd) return false;
    uint64_t sn = 1;
    for (auto d : *sd) sn *= d;
    if (sn != (uint64_t)N * (*wd)[1]) return false;
    if (n.inputs.size() == 4) {
        const TensorType& z = ty(m, n.inputs[3]);
        auto zd = shape_as_static(z.shape);
        if (z.dtype != DType::U4 || !zd) return false;
        uint64_t zn = 1;
        for (auto d : *zd) zn *= d;
        if (zn != sn) return false;
    }
    // weights must be constants: their device copy is 16-byte aligned and immutable
    return m.values[n.inputs[1]].origin.kind == Origin::Const;
}
void nbits_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::NBitsDesc d{};
    d.k = a.int_("K");
    d.n = a.int_("N");
    d.block_size = 32;
    d.n_blocks = (d.k + 31) / 32;
    d.m = c.ins[0].numel() / d.k;
    d.act_dtype = c.ins[0].dtype;
    d.scale_dtype = c.ins[2].dtype;
    d.has_zp = c.ins.size() > 3;
    d.interleaved = c.weights_layout == 1;
    d.tiled = c.weights_layout == 2;
    oxk::emit_matmul_nbits(c.em, d, c.ins[0], c.ins[1], c.ins[2], d.has_zp ? &c.ins[3] : nullptr, c.outs[0]);
}

// ── onyxia.ResidualNorm / onyxia.Linear ──
// Operands of a residual norm, in front of whatever else a node takes: y (its columns from "y_offset" on), weight, residual
// (attribute "residual"), gain (attribute "gain"), gate matrix (attribute "gate", its columns from "gate_offset" on). With "pre"
// the norm is taken of the sum and the new residual is the sum; "y_scale" multiplies y there. What else a sum may have: the
// weight of a norm of y in front of it ("post"), another matrix times "add_scale" ("add"), a vector ("offset").
// "streams" = S: the residual is S streams side by side; the last operands are what connects them (mix by origin, out, in as one vector) and,
// with "twin", a second result with the weight of its norm. "norm_groups" = n: the norm is taken of n runs of columns, each for itself.
size_t norm_operands(const Attrs& a) {
    size_t n = 2;
    for (const char* part : {"residual", "gain", "gate", "post", "add", "offset"}) n += a.int_or(part, 0) != 0;
    n += a.int_or("streams", 0) != 0;
    n += a.int_or("twin", 0) != 0 ? 2 : 0;
    return n;
}
bool is_act(DType d) { return d == DType::F32 || d == DType::BF16; }
bool is_const(const DimExpr& d, int64_t v) { return d.as_const() == std::optional<uint64_t>((uint64_t)v); }
bool is_f32_vector(const Module& m, ValueId v, uint64_t n) {
    const TensorType& t = ty(m, v);
    return t.dtype == DType::F32 && t.shape.size() == 1 && t.shape[0].as_const() == std::optional<uint64_t>(n);
}
bool norm_accepts(const Module& m, const Node& n, const ValueId* stream) {
    const Attrs& a = n.composite.attrs;
    const TensorType &y = ty(m, n.inputs[0]), &w = ty(m, n.inputs[1]);
    if (!is_act(y.dtype) || y.shape.size() != 2 || w.shape.size() != 1 || !w.shape[0].as_const() || !y.shape[1].as_const()) return false;
    const uint64_t width = *w.shape[0].as_const();
    const int64_t y_off = a.int_or("y_offset", 0);
    if (!is_f32_vector(m, n.inputs[1], width) || y_off < 0 || y_off + (int64_t)width > (int64_t)*y.shape[1].as_const()) return false;
    const bool pre = a.int_or("pre", 0) != 0, post = a.int_or("post", 0) != 0;
    if ((!pre || post) && a.float_or("y_scale", 1.0) != 1.0) return false;
    if (!pre && (post || a.int_or("add", 0) != 0 || a.int_or("offset", 0) != 0)) return false;
    const int64_t streams = a.int_or("streams", 0), groups = a.int_or("norm_groups", 1);
    const bool twin = a.int_or("twin", 0) != 0;
    if (streams < 0 || streams > oxk::kMaxStreams || groups < 1 || width % (uint64_t)groups != 0) return false;
    auto has = [&](const char* part) { return a.int_or(part, 0) != 0; };
    if (streams > 0 && (!pre || groups > 1 || width > 50000 || has("gain") || has("gate") || has("add") || has("offset"))) return false;
    if (groups > 1 && (pre || has("residual") || has("gain"))) return false;
    if (twin && (streams == 0 || !post)) return false;
    auto rows_of = [&](const TensorType& t, int64_t times = 1) { return t.shape.size() == 2 && t.shape[0] == y.shape[0] && is_const(t.shape[1], (int64_t)width * times); };
    const int64_t times = std::max<int64_t>(streams, 1);
    if (stream && (ty(m, *stream).dtype != DType::F32 || !rows_of(ty(m, *stream), times))) return false;
    size_t i = 2;
    if (a.int_or("residual", 0) != 0) {
        const TensorType& r = ty(m, n.inputs[i++]);
        if (r.dtype != DType::F32 || !rows_of(r, times)) return false;
    }
    if (a.int_or("gain", 0) != 0 && !is_f32_vector(m, n.inputs[i++], width)) return false;
    if (a.int_or("gate", 0) != 0) {
        const TensorType& g = ty(m, n.inputs[i++]);
        const int64_t off = a.int_or("gate_offset", 0);
        if (!is_act(g.dtype) || g.shape.size() != 2 || g.shape[0] != y.shape[0] || !g.shape[1].as_const()) return false;
        if (off < 0 || off + (int64_t)width > (int64_t)*g.shape[1].as_const()) return false;
    }
    if (post && !is_f32_vector(m, n.inputs[i++], width)) return false;
    if (a.int_or("add", 0) != 0) {
        const TensorType& t = ty(m, n.inputs[i++]);
        if (!is_act(t.dtype) || !rows_of(t)) return false;
    }
    if (a.int_or("offset", 0) != 0 && !is_f32_vector(m, n.inputs[i++], width)) return false;
    if (streams > 0 && !is_f32_vector(m, n.inputs[i++], (uint64_t)(streams * (streams + 2)))) return false;
    if (twin) {
        const TensorType& t = ty(m, n.inputs[i++]);
        if (t.dtype != y.dtype || !rows_of(t) || !is_f32_vector(m, n.inputs[i++], width)) return false;
    }
    return true;
}
oxk::ResidualNormDesc norm_desc(FusedCtx& c, const TRef* stream) {
    const Attrs& a = c.node.composite.attrs;
    oxk::ResidualNormDesc d;
    size_t i = 2;
    d.y = &c.ins[0];
    d.w = &c.ins[1];
    if (a.int_or("residual", 0) != 0) d.res = &c.ins[i++];
    if (a.int_or("gain", 0) != 0) d.gain = &c.ins[i++];
    if (a.int_or("gate", 0) != 0) d.gate = &c.ins[i++];
    if (a.int_or("post", 0) != 0) d.post = &c.ins[i++];
    if (a.int_or("add", 0) != 0) d.add = &c.ins[i++];
    if (a.int_or("offset", 0) != 0) d.offset = &c.ins[i++];
    d.streams = a.int_or("streams", 0);
    d.groups = a.int_or("norm_groups", 1);
    if (d.streams > 0) d.connect = &c.ins[i++];
    if (a.int_or("twin", 0) != 0) {
        d.y2 = &c.ins[i++];
        d.post2 = &c.ins[i++];
    }
    d.y_off = a.int_or("y_offset", 0);
    d.gate_off = a.int_or("gate_offset", 0);
    d.add_scale = a.float_or("add_scale", 1.0);
    d.stream = stream;
    d.eps = a.float_or("epsilon", 1e-6);
    d.y_scale = a.float_or("y_scale", 1.0);
    d.pre = a.int_or("pre", 0) != 0;
    return d;
}
bool residual_norm_accepts(const Module& m, const Node& n) {
    return n.inputs.size() == norm_operands(n.composite.attrs) && n.outputs.size() == 1 && norm_accepts(m, n, &n.outputs[0]);
}
void residual_norm_lower(FusedCtx& c) {
    const bool pre = c.node.composite.attrs.int_or("pre", 0) != 0;  // the result is the normed sum, not the sum
    oxk::emit_residual_norm(c.em, norm_desc(c, pre ? nullptr : &c.outs[0]), pre ? &c.outs[0] : nullptr);
}

int activation(const Attrs& a, const char* name) {
    const std::string f = a.str_or(name, "none");
    return f == "none" ? oxk::ACT_NONE : f == "silu" ? oxk::ACT_SILU : f == "sigmoid" ? oxk::ACT_SIGMOID : f == "softplus" ? oxk::ACT_SOFTPLUS : -1;
}
// "stream" = 0: a node with a norm in front has no second result. "act" and "act_rest": functions of the result's columns before
// and from "act_split" on, to "act_end" (when given) at most. "ranges": x, weight, [bias,] [a matrix that multiplies the result ("mul"), its columns from "mul_offset"
// on] of "blocks" block-diagonal products, block b over the columns of x from "x_offset" + b · "x_step" on.
bool ranges_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    const bool bias = a.int_or("bias", 0) != 0, mul = a.int_or("mul", 0) != 0;
    const int64_t blocks = a.int_or("blocks", 1), off = a.int_or("x_offset", 0), step = a.int_or("x_step", 0), mul_off = a.int_or("mul_offset", 0);
    if (n.inputs.size() != 2u + bias + mul || n.outputs.size() != 1 || blocks < 1 || off < 0 || step < 0) return false;
    const TensorType &x = ty(m, n.inputs[0]), &w = ty(m, n.inputs[1]), &y = ty(m, n.outputs[0]);
    if (!is_act(w.dtype) || x.dtype != w.dtype || !is_act(y.dtype) || (w.dtype == DType::F32 && y.dtype != DType::F32)) return false;
    if (x.shape.size() != 2 || w.shape.size() != 2 || y.shape.size() != 2 || m.values[n.inputs[1]].origin.kind != Origin::Const) return false;
    auto cols = x.shape[1].as_const(), out = w.shape[0].as_const(), k = w.shape[1].as_const();
    if (!cols || !out || !k || *out % (uint64_t)blocks != 0 || off + (blocks - 1) * step + (int64_t)*k > (int64_t)*cols) return false;
    if (bias && !is_f32_vector(m, n.inputs[2], *out)) return false;
    if (mul) {
        const TensorType& t = ty(m, n.inputs.back());
        if (t.dtype != w.dtype || t.shape.size() != 2 || t.shape[0] != x.shape[0] || !t.shape[1].as_const()) return false;
        if (mul_off < 0 || mul_off + (int64_t)*out > (int64_t)*t.shape[1].as_const()) return false;
    }
    return y.shape[0] == x.shape[0] && y.shape[1].as_const() == out;
}
bool linear_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    const bool norm = a.int_or("norm", 0) != 0, pair = a.int_or("pair", 0) != 0, bias = a.int_or("bias", 0) != 0, glu = a.int_or("glu", 0) != 0;
    const bool stream = norm && a.int_or("stream", 1) != 0, ranges = a.int_or("ranges", 0) != 0;
    const size_t nx = norm ? norm_operands(a) : (pair ? 2 : 1), nw = pair ? 2 : 1;
    if ((norm && pair) || (!ranges && n.inputs.size() != nx + nw + bias) || n.outputs.size() != (stream ? 2u : 1u)) return false;
    if (norm && !norm_accepts(m, n, stream ? &n.outputs[1] : nullptr)) return false;
    if (activation(a, "act") < 0 || activation(a, "act_rest") < 0 || (glu && (activation(a, "act") || activation(a, "act_rest")))) return false;
    if (a.int_or("ranges", 0) != 0) return !norm && !pair && !glu && ranges_accepts(m, n);
    const TensorType& y = ty(m, n.outputs[0]);
    if (y.shape.size() != 2 || !is_act(y.dtype)) return false;
    std::optional<uint64_t> out;
    const DType wt = ty(m, n.inputs[nx]).dtype;
    if (!is_act(wt) || (wt == DType::F32 && y.dtype != DType::F32)) return false;
    if (norm && a.int_or("gate", 0) != 0 && ty(m, n.inputs[nx - 1]).dtype != wt) return false;
    for (size_t i = 0; i < nw; i++) {
        const ValueId wv = n.inputs[nx + i];
        const TensorType &x = ty(m, n.inputs[norm ? 0 : i]), &w = ty(m, wv);
        if (x.shape.size() != 2 || w.shape.size() != 2 || w.dtype != wt || (!norm && x.dtype != wt)) return false;
        if (m.values[wv].origin.kind != Origin::Const) return false;
        if ((norm ? ty(m, n.inputs[1]).shape[0] : x.shape[1]) != w.shape[1] || x.shape[0] != y.shape[0] || (i > 0 && w.shape[0].as_const() != out)) return false;
        out = w.shape[0].as_const();
    }
    if (!out || (glu && *out % 2 != 0)) return false;
    if (bias && !is_f32_vector(m, n.inputs.back(), *out)) return false;
    return y.shape[1].as_const() == std::optional<uint64_t>(glu ? *out / 2 : *out);
}
void linear_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    const bool norm = a.int_or("norm", 0) != 0, pair = a.int_or("pair", 0) != 0, bias = a.int_or("bias", 0) != 0;
    const size_t nx = norm ? norm_operands(a) : (pair ? 2 : 1);
    oxk::LinearDesc d;
    d.rows = c.outs[0].shape[0];
    d.out = c.ins[nx].shape[0];
    d.k[0] = c.ins[nx].shape[1];
    d.k[1] = pair ? c.ins[nx + 1].shape[1] : 0;
    d.glu = a.int_or("glu", 0) != 0;
    d.alpha = (float)a.float_or("alpha", 1.0);
    d.limit = (float)a.float_or("limit", INFINITY);
    d.shift = (float)a.float_or("shift", 0.0);
    d.act[0] = activation(a, "act");
    d.act[1] = activation(a, "act_rest");
    d.act_split = a.int_or("act_split", 0);
    d.act_end = a.int_or("act_end", 0);
    oxk::ResidualNormDesc nd;
    if (norm) nd = norm_desc(c, c.outs.size() > 1 ? &c.outs[1] : nullptr);
    if (a.int_or("ranges", 0) != 0) {
        d.blocks = a.int_or("blocks", 1);
        d.out /= d.blocks;
        d.x_off = a.int_or("x_offset", 0);
        d.x_step = a.int_or("x_step", 0);
        if (a.int_or("mul", 0) != 0) d.mul = &c.ins.back();
        d.mul_off = a.int_or("mul_offset", 0);
        oxk::emit_linear(c.em, d, &c.ins[0], nullptr, c.ins[1], nullptr, bias ? &c.ins[2] : nullptr, c.outs[0], nullptr);
        return;
    }
    oxk::emit_linear(c.em, d, norm ? nullptr : &c.ins[0], pair ? &c.ins[1] : nullptr, c.ins[nx], pair ? &c.ins[nx + 1] : nullptr,
                     bias ? &c.ins.back() : nullptr, c.outs[0], norm ? &nd : nullptr);
}

// ── onyxia.MixtureOfExperts ──
// residual norm operands, router, router bias, up (gate and up rows interleaved), down [, shared up, shared down ("shared_ff")]
// [, correction of the scores ("correction")] → y, new residual. "scores": softmax (over the chosen ones), sigmoid or softmax_all; "renorm" = 0: the
// weights are the scores themselves; "groups" and "keep": only experts of the best groups, judged by their two largest scores or, with "group_max",
// by the largest. "shared_gate": the router has one more row, whose sigmoid multiplies the shared expert.
bool moe_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    const int64_t E = a.int_or("experts", 0), top = a.int_or("top", 0), F = a.int_or("ff", 0);
    const size_t nx = norm_operands(a);
    if (E <= 0 || E > 2048 || top <= 0 || top > 32 || top > E || F <= 0 || n.outputs.size() != 2) return false;
    const int64_t groups = a.int_or("groups", 0), keep = a.int_or("keep", 0), SF = a.int_or("shared_ff", 0);
    const std::string scores = a.str_or("scores", "softmax");
    if (scores != "softmax" && scores != "sigmoid" && scores != "softmax_all") return false;
    const bool correction = a.int_or("correction", 0) != 0, shared_gate = a.int_or("shared_gate", 0) != 0;
    if (scores == "softmax" && (correction || a.int_or("renorm", 1) == 0)) return false;
    if (shared_gate && SF <= 0) return false;
    if (groups != 0 && (scores == "softmax" || groups < 0 || groups > oxk::kMoeMaxGroups || E % groups != 0 || keep < 1 || keep > groups || top > keep * (E / groups))) return false;
    if (SF < 0 || n.inputs.size() != nx + (SF ? 6 : 4) + correction || !norm_accepts(m, n, &n.outputs[1])) return false;
    const TensorType &x = ty(m, n.inputs[0]), &router = ty(m, n.inputs[nx]), &up = ty(m, n.inputs[nx + 2]), &down = ty(m, n.inputs[nx + 3]), &y = ty(m, n.outputs[0]);
    const int64_t H = (int64_t)*x.shape[1].as_const(), RR = E + shared_gate;
    if (correction && !is_f32_vector(m, n.inputs.back(), (uint64_t)E)) return false;
    if (!is_act(up.dtype) || router.dtype != up.dtype || down.dtype != up.dtype || y.dtype != DType::F32 || y.shape != x.shape) return false;
    if (router.shape.size() != 2 || !is_const(router.shape[0], RR) || !is_const(router.shape[1], H) || !is_f32_vector(m, n.inputs[nx + 1], (uint64_t)RR)) return false;
    if (up.shape.size() != 2 || !is_const(up.shape[0], E * 2 * F) || !is_const(up.shape[1], H)) return false;
    if (down.shape.size() != 2 || !is_const(down.shape[0], E * H) || !is_const(down.shape[1], F)) return false;
    for (size_t i : {nx, nx + 2, nx + 3})
        if (m.values[n.inputs[i]].origin.kind != Origin::Const) return false;
    if (SF) {
        const TensorType &su = ty(m, n.inputs[nx + 4]), &sd = ty(m, n.inputs[nx + 5]);
        if (su.dtype != up.dtype || su.shape.size() != 2 || !is_const(su.shape[0], 2 * SF) || !is_const(su.shape[1], H)) return false;
        if (sd.dtype != up.dtype || sd.shape.size() != 2 || !is_const(sd.shape[0], H) || !is_const(sd.shape[1], SF)) return false;
        for (size_t i : {nx + 4, nx + 5})
            if (m.values[n.inputs[i]].origin.kind != Origin::Const) return false;
    }
    return true;
}
void moe_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    const size_t nx = norm_operands(a);
    oxk::MoeDesc d{};
    d.rows = c.outs[0].shape[0];
    d.width = c.outs[0].shape[1];
    d.experts = a.int_("experts");
    d.top = a.int_("top");
    d.ff = a.int_("ff");
    d.alpha = (float)a.float_or("alpha", 1.0);
    d.limit = (float)a.float_or("limit", INFINITY);
    d.shift = (float)a.float_or("shift", 0.0);
    const std::string scores = a.str_or("scores", "softmax");
    d.scores = scores == "sigmoid" ? oxk::MOE_SIGMOID : scores == "softmax_all" ? oxk::MOE_SOFTMAX : oxk::MOE_CHOSEN;
    d.renorm = a.int_or("renorm", 1) != 0;
    d.group_max = a.int_or("group_max", 0) != 0;
    d.shared_gate = a.int_or("shared_gate", 0) != 0;
    if (a.int_or("correction", 0) != 0) d.correction = &c.ins.back();
    d.groups = a.int_or("groups", 0);
    d.keep = a.int_or("keep", 0);
    d.route_scale = (float)a.float_or("route_scale", 1.0);
    d.shared_ff = a.int_or("shared_ff", 0);
    d.shared_limit = (float)a.float_or("shared_limit", INFINITY);
    oxk::emit_moe(c.em, d, norm_desc(c, &c.outs[1]), c.ins[nx], c.ins[nx + 1], c.ins[nx + 2], c.ins[nx + 3], d.shared_ff ? &c.ins[nx + 4] : nullptr,
                  d.shared_ff ? &c.ins[nx + 5] : nullptr, c.outs[0]);
}

// ── onyxia.PagedAttention ──
// proj, q_norm, k_norm, distance bias, key pool, key scales, seqs, pages → out, key pool, key scales
bool paged_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 8 || n.outputs.size() != 3) return false;
    const int64_t H = a.int_or("heads", 0), G = a.int_or("kv_heads", 0), D = a.int_or("dim", 0);
    if (H <= 0 || G <= 0 || D <= 0 || H % G != 0) return false;
    const TensorType &x = ty(m, n.inputs[0]), &bias = ty(m, n.inputs[3]), &pool = ty(m, n.inputs[4]), &ks = ty(m, n.inputs[5]);
    const TensorType &seqs = ty(m, n.inputs[6]), &pages = ty(m, n.inputs[7]), &out = ty(m, n.outputs[0]);
    auto is = [](const DimExpr& d, int64_t v) { return d.as_const() == std::optional<uint64_t>((uint64_t)v); };
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    const int64_t qo = a.int_or("q_offset", 0), ko = a.int_or("k_offset", 0);
    if (!is_act(x.dtype) || !width || qo < 0 || ko < 0 || qo + H * D > (int64_t)*width || ko + G * D > (int64_t)*width) return false;
    if (!is_f32_vector(m, n.inputs[1], (uint64_t)(H * D)) || !is_f32_vector(m, n.inputs[2], (uint64_t)(G * D))) return false;
    if (bias.dtype != DType::F32 || bias.shape.size() != 2 || !is(bias.shape[0], H) || !bias.shape[1].as_const()) return false;
    if (pool.dtype != x.dtype || pool.shape.size() != 4 || !is(pool.shape[1], G) || !pool.shape[2].as_const() || !is(pool.shape[3], D)) return false;
    const uint64_t page = *pool.shape[2].as_const();
    if (page == 0 || (page & (page - 1)) != 0) return false;  // pages are found by shifting
    if (ks.dtype != DType::F32 || ks.shape.size() != 2 || ks.shape[0] != pool.shape[0] || ks.shape[1] != pool.shape[2]) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is(seqs.shape[1], 4)) return false;
    if (pages.dtype != DType::I32 || pages.shape.size() != 2 || pages.shape[0] != seqs.shape[0]) return false;
    return out.dtype == x.dtype && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is(out.shape[1], H * D);
}
void paged_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::PagedAttnDesc d{};
    d.heads = a.int_("heads");
    d.kv_heads = a.int_("kv_heads");
    d.dim = a.int_("dim");
    d.page = c.ins[4].shape[2];
    d.q_off = a.int_or("q_offset", 0);
    d.k_off = a.int_or("k_offset", 0);
    d.scale = a.float_or("scale", 1.0);
    d.eps = a.float_or("epsilon", 1e-6);
    d.out_scale = a.float_or("out_scale", 1.0);
    d.temp_coef = a.float_or("temp_coef", 0.0);
    d.temp_every = a.float_or("temp_every", 0.0);
    oxk::emit_paged_attention(c.em, d, c.ins[0], c.ins[1], c.ins[2], &c.ins[3], c.outs[1], c.outs[2], c.ins[6], c.ins[7], c.outs[0]);
}

// ── onyxia.GatedRecurrence ──
// proj, conv weight, conv bias, ra, ra bias, ri, ri bias, lam, conv state, state, seqs → out, conv state, state
bool recurrence_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 11 || n.outputs.size() != 3) return false;
    const int64_t C = a.int_or("width", 0), B = a.int_or("blocks", 0), K = a.int_or("taps", 0);
    if (C <= 0 || B <= 0 || K <= 0 || C % B != 0) return false;
    const uint64_t nb = (uint64_t)(C / B);
    const TensorType &x = ty(m, n.inputs[0]), &cs = ty(m, n.inputs[8]), &st = ty(m, n.inputs[9]), &seqs = ty(m, n.inputs[10]), &out = ty(m, n.outputs[0]);
    auto is = [](const DimExpr& d, int64_t v) { return d.as_const() == std::optional<uint64_t>((uint64_t)v); };
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    const int64_t xo = a.int_or("x_offset", 0), yo = a.int_or("y_offset", 0);
    if (!is_act(x.dtype) || !width || xo < 0 || yo < 0 || xo + C > (int64_t)*width || yo + C > (int64_t)*width) return false;
    const TensorType& cw = ty(m, n.inputs[1]);
    if (cw.dtype != DType::F32 || cw.shape.size() != 2 || !is(cw.shape[0], C) || !is(cw.shape[1], K)) return false;
    for (int i : {2, 4, 6, 7})
        if (!is_f32_vector(m, n.inputs[i], (uint64_t)C)) return false;
    for (int i : {3, 5}) {
        const TensorType& w = ty(m, n.inputs[i]);
        if (w.dtype != x.dtype || w.shape.size() != 3 || !is(w.shape[0], B) || !is(w.shape[1], (int64_t)nb) || !is(w.shape[2], (int64_t)nb)) return false;
        if (m.values[n.inputs[i]].origin.kind != Origin::Const) return false;
    }
    if (cs.dtype != x.dtype || cs.shape.size() != 3 || !is(cs.shape[1], K) || !is(cs.shape[2], C)) return false;
    if (st.dtype != DType::F32 || st.shape.size() != 2 || st.shape[0] != cs.shape[0] || !is(st.shape[1], C)) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is(seqs.shape[1], 4)) return false;
    return out.dtype == x.dtype && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is(out.shape[1], C);
}
void recurrence_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::GatedRecurrenceDesc d{};
    d.width = a.int_("width");
    d.blocks = a.int_("blocks");
    d.taps = a.int_("taps");
    d.x_off = a.int_or("x_offset", 0);
    d.y_off = a.int_or("y_offset", 0);
    d.decay = a.float_or("decay", 8.0);
    d.out_scale = a.float_or("out_scale", 1.0);
    oxk::emit_gated_recurrence(c.em, d, c.ins[0], c.ins[1], c.ins[2], c.ins[3], c.ins[4], c.ins[5], c.ins[6], c.ins[7], c.outs[1], c.outs[2], c.ins[10],
                               c.outs[0]);
}

// ── onyxia.PagedKVAttention / onyxia.SharedKVAttention ──
// proj, turns per position, keys, values, seqs, pages [, sinks] [, temps] [, talk] → out [, keys, values]; the shared form attends to what
// another node has put into the pools and appends nothing. "sinks": a score per head without a value; "gate": heads are multiplied by columns
// of proj from "gate_offset" on; "temps": a factor per head of the scores; "talk": a matrix that mixes the heads' softmax weights.
bool paged_kv_fits(const Module& m, const Node& n, bool append) {
    const Attrs& a = n.composite.attrs;
    const bool sinks = a.int_or("sinks", 0) != 0, temps = a.int_or("temps", 0) != 0, talk = a.int_or("talk", 0) != 0;
    if (n.inputs.size() != 6u + sinks + temps + talk || n.outputs.size() != (append ? 3u : 1u)) return false;
    const int64_t H = a.int_or("heads", 0), G = a.int_or("kv_heads", 0), D = a.int_or("dim", 0), V = a.int_or("vdim", 0), R = a.int_or("rot_dims", 0);
    if (H <= 0 || G <= 0 || D <= 0 || V <= 0 || H % G != 0 || R < 0 || R > D || R % 2 != 0 || a.int_or("window", 0) < 0) return false;
    const TensorType &x = ty(m, n.inputs[0]), &turns = ty(m, n.inputs[1]), &keys = ty(m, n.inputs[2]), &values = ty(m, n.inputs[3]);
    const TensorType &seqs = ty(m, n.inputs[4]), &pages = ty(m, n.inputs[5]), &out = ty(m, n.outputs[0]);
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    if (!is_act(x.dtype) || !width) return false;
    auto inside = [&](const char* name, int64_t cols) {
        const int64_t off = a.int_or(name, 0);
        return off >= 0 && off + cols <= (int64_t)*width;
    };
    if (!inside("q_offset", H * D) || (append && (!inside("k_offset", G * D) || !inside("v_offset", G * V)))) return false;
    if (a.int_or("gate", 0) != 0 && !inside("gate_offset", H)) return false;
    if (sinks && (a.int_or("sink", 0) != 0 || !is_f32_vector(m, n.inputs[6], (uint64_t)H))) return false;
    if (temps && !is_f32_vector(m, n.inputs[6u + sinks], (uint64_t)H)) return false;
    if (talk) {
        const TensorType& t = ty(m, n.inputs.back());
        if (t.dtype != DType::F32 || t.shape.size() != 2 || !is_const(t.shape[0], H) || !is_const(t.shape[1], H) || H * (D + V + 64) > 50000) return false;
        for (const char* other : {"sinks", "sink", "window", "gate"})
            if (a.int_or(other, 0) != 0) return false;
        if (a.float_or("softcap", 0.0) != 0.0) return false;
    }
    if (turns.dtype != DType::F32 || turns.shape.size() != 2 || !is_const(turns.shape[0], 2)) return false;
    if (R > 0 && !is_const(turns.shape[1], R / 2)) return false;
    for (auto [t, d] : {std::pair<const TensorType*, int64_t>{&keys, D}, {&values, V}})
        if (t->dtype != x.dtype || t->shape.size() != 4 || !is_const(t->shape[1], G) || !t->shape[2].as_const() || !is_const(t->shape[3], d)) return false;
    const uint64_t page = *keys.shape[2].as_const();
    if (page == 0 || (page & (page - 1)) != 0 || values.shape[0] != keys.shape[0] || values.shape[2] != keys.shape[2]) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is_const(seqs.shape[1], 4)) return false;
    if (pages.dtype != DType::I32 || pages.shape.size() != 2 || pages.shape[0] != seqs.shape[0]) return false;
    return out.dtype == x.dtype && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is_const(out.shape[1], H * V);
}
bool paged_kv_accepts(const Module& m, const Node& n) { return paged_kv_fits(m, n, true); }
bool shared_kv_accepts(const Module& m, const Node& n) { return paged_kv_fits(m, n, false); }
void paged_kv_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::PagedKvDesc d{};
    d.heads = a.int_("heads");
    d.kv_heads = a.int_("kv_heads");
    d.dim = a.int_("dim");
    d.vdim = a.int_("vdim");
    d.page = c.ins[2].shape[2];
    d.q_off = a.int_or("q_offset", 0);
    d.k_off = a.int_or("k_offset", 0);
    d.v_off = a.int_or("v_offset", 0);
    d.rot_dims = a.int_or("rot_dims", 0);
    d.window = a.int_or("window", 0);
    d.scale = a.float_or("scale", 1.0);
    d.softcap = a.float_or("softcap", 0.0);
    d.eps = a.float_or("epsilon", 1e-6);
    d.norm = a.int_or("norm", 0) != 0;
    if (a.int_or("sinks", 0) != 0) d.sinks = &c.ins[6];
    d.sink = d.sinks || a.int_or("sink", 0) != 0;
    if (a.int_or("temps", 0) != 0) d.temps = &c.ins[d.sinks ? 7 : 6];
    if (a.int_or("talk", 0) != 0) d.talk = &c.ins.back();
    d.interleaved = a.int_or("interleaved", 0) != 0;
    if (a.int_or("gate", 0) != 0) d.gate_off = a.int_or("gate_offset", 0);
    d.append = c.outs.size() > 1;
    oxk::emit_paged_kv_attention(c.em, d, c.ins[0], c.ins[1], d.append ? c.outs[1] : c.ins[2], d.append ? c.outs[2] : c.ins[3], c.ins[4], c.ins[5], c.outs[0]);
}

// ── onyxia.LatentAttention ──
// queries in the latent space, queries, proj, norm weight, turns per position, pool, seqs, pages → out, pool
bool latent_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 8 || n.outputs.size() != 2) return false;
    const int64_t H = a.int_or("heads", 0), K = a.int_or("rank", 0), R = a.int_or("rot", 0), kv = a.int_or("kv_offset", 0), qo = a.int_or("q_offset", 0);
    const int64_t step = a.int_or("q_step", 0);
    if (H <= 0 || K <= 0 || R < 0 || R % 2 != 0 || kv < 0 || qo < 0 || step < 0) return false;
    const TensorType &lat = ty(m, n.inputs[0]), &q = ty(m, n.inputs[1]), &x = ty(m, n.inputs[2]), &turns = ty(m, n.inputs[4]), &pool = ty(m, n.inputs[5]);
    const TensorType &seqs = ty(m, n.inputs[6]), &pages = ty(m, n.inputs[7]), &out = ty(m, n.outputs[0]);
    for (const TensorType* t : {&lat, &q, &x, &out})
        if (!is_act(t->dtype) || t->dtype != x.dtype || t->shape.size() != 2 || t->shape[0] != x.shape[0] || !t->shape[1].as_const()) return false;
    if (!is_const(lat.shape[1], H * K) || !is_const(out.shape[1], H * K) || kv + K + R > (int64_t)*x.shape[1].as_const()) return false;
    if (R > 0 && qo + (H - 1) * step + R > (int64_t)*q.shape[1].as_const()) return false;
    if (!is_f32_vector(m, n.inputs[3], (uint64_t)K) || turns.dtype != DType::F32 || turns.shape.size() != 2 || !is_const(turns.shape[0], 2)) return false;
    if (R > 0 && !is_const(turns.shape[1], R / 2)) return false;
    if (pool.dtype != x.dtype || pool.shape.size() != 4 || !is_const(pool.shape[1], 1) || !pool.shape[2].as_const() || !is_const(pool.shape[3], K + R)) return false;
    const uint64_t page = *pool.shape[2].as_const();
    if (page == 0 || (page & (page - 1)) != 0) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is_const(seqs.shape[1], 4)) return false;
    return pages.dtype == DType::I32 && pages.shape.size() == 2 && pages.shape[0] == seqs.shape[0];
}
void latent_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::LatentAttnDesc d{};
    d.heads = a.int_("heads");
    d.rank = a.int_("rank");
    d.rot = a.int_or("rot", 0);
    d.page = c.ins[5].shape[2];
    d.q_off = a.int_or("q_offset", 0);
    d.q_step = a.int_or("q_step", 0);
    d.kv_off = a.int_or("kv_offset", 0);
    d.scale = a.float_or("scale", 1.0);
    d.eps = a.float_or("epsilon", 1e-6);
    oxk::emit_latent_attention(c.em, d, c.ins[0], c.ins[1], c.ins[2], c.ins[3], c.ins[4], c.outs[1], c.ins[6], c.ins[7], c.outs[0]);
}

// ── onyxia.SelectiveScan ──
// proj, conv weight, conv bias, W_x, W_dt, dt bias, A, D, conv state, state, seqs → out, conv state, state
bool selective_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 11 || n.outputs.size() != 3) return false;
    const int64_t C = a.int_or("width", 0), S = a.int_or("state", 0), R = a.int_or("rank", 0), K = a.int_or("taps", 0);
    if (C <= 0 || S <= 0 || S > 256 || R <= 0 || K <= 0) return false;
    const TensorType &x = ty(m, n.inputs[0]), &cs = ty(m, n.inputs[8]), &st = ty(m, n.inputs[9]), &seqs = ty(m, n.inputs[10]), &out = ty(m, n.outputs[0]);
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    const int64_t xo = a.int_or("x_offset", 0), zo = a.int_or("z_offset", 0);
    if (!is_act(x.dtype) || !width || xo < 0 || zo < 0 || xo + C > (int64_t)*width || zo + C > (int64_t)*width) return false;
    auto matrix = [&](size_t i, DType d, int64_t rows, int64_t cols) {
        const TensorType& t = ty(m, n.inputs[i]);
        return t.dtype == d && t.shape.size() == 2 && is_const(t.shape[0], rows) && is_const(t.shape[1], cols) && m.values[n.inputs[i]].origin.kind == Origin::Const;
    };
    if (!matrix(1, DType::F32, C, K) || !matrix(3, x.dtype, R + 2 * S, C) || !matrix(4, x.dtype, C, R) || !matrix(6, DType::F32, C, S)) return false;
    for (int i : {2, 5, 7})
        if (!is_f32_vector(m, n.inputs[i], (uint64_t)C)) return false;
    if (cs.dtype != x.dtype || cs.shape.size() != 3 || !is_const(cs.shape[1], K) || !is_const(cs.shape[2], C)) return false;
    if (st.dtype != DType::F32 || st.shape.size() != 3 || st.shape[0] != cs.shape[0] || !is_const(st.shape[1], C) || !is_const(st.shape[2], S)) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is_const(seqs.shape[1], 4)) return false;
    return out.dtype == x.dtype && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is_const(out.shape[1], C);
}
void selective_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::SelectiveScanDesc d{};
    d.width = a.int_("width");
    d.state = a.int_("state");
    d.rank = a.int_("rank");
    d.taps = a.int_("taps");
    d.x_off = a.int_or("x_offset", 0);
    d.z_off = a.int_or("z_offset", 0);
    oxk::emit_selective_scan(c.em, d, c.ins[0], c.ins[1], c.ins[2], c.ins[3], c.ins[4], c.ins[5], c.ins[6], c.ins[7], c.outs[1], c.outs[2], c.ins[10],
                             c.outs[0]);
}

// ── onyxia.GatedLinearAttention ──
// proj, z, state, seqs → out, state
bool gated_linear_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 4 || n.outputs.size() != 2) return false;
    const int64_t H = a.int_or("heads", 0), D = a.int_or("dim", 0), V = a.int_or("vdim", 0);
    if (H <= 0 || D <= 0 || D > 512 || V <= 0 || !(a.float_or("tau", 1.0) > 0.0)) return false;
    const TensorType &x = ty(m, n.inputs[0]), &z = ty(m, n.inputs[1]), &st = ty(m, n.inputs[2]), &seqs = ty(m, n.inputs[3]), &out = ty(m, n.outputs[0]);
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    if (!is_act(x.dtype) || !width) return false;
    auto inside = [&](const char* name, int64_t cols) {
        const int64_t off = a.int_or(name, 0);
        return off >= 0 && off + cols <= (int64_t)*width;
    };
    if (!inside("q_offset", H * D) || !inside("k_offset", H * D) || !inside("v_offset", H * V)) return false;
    if (z.dtype != DType::F32 || z.shape.size() != 2 || z.shape[0] != x.shape[0] || !is_const(z.shape[1], H * D)) return false;
    if (st.dtype != DType::F32 || st.shape.size() != 4 || !is_const(st.shape[1], H) || !is_const(st.shape[2], D) || !is_const(st.shape[3], V)) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is_const(seqs.shape[1], 4)) return false;
    return out.dtype == DType::F32 && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is_const(out.shape[1], H * V);
}
void gated_linear_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::GatedLinearDesc d{};
    d.heads = a.int_("heads");
    d.dim = a.int_("dim");
    d.vdim = a.int_("vdim");
    d.q_off = a.int_or("q_offset", 0);
    d.k_off = a.int_or("k_offset", 0);
    d.v_off = a.int_or("v_offset", 0);
    d.tau = a.float_or("tau", 1.0);
    d.q_scale = a.float_or("q_scale", 1.0);
    oxk::emit_gated_linear(c.em, d, c.ins[0], c.ins[1], c.outs[1], c.ins[3], c.outs[0]);
}

// ── onyxia.GatedDeltaRule ──
// proj, conv weight, decay, dt bias, conv state, state, seqs → out, conv state, state
bool delta_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 7 || n.outputs.size() != 3) return false;
    const int64_t H = a.int_or("heads", 0), G = a.int_or("kv_heads", 0), D = a.int_or("dim", 0), V = a.int_or("vdim", 0), K = a.int_or("taps", 0);
    if (H <= 0 || G <= 0 || H % G != 0 || D <= 0 || D > 512 || V <= 0 || K <= 0) return false;
    const int64_t C = 2 * G * D + H * V;
    const TensorType &x = ty(m, n.inputs[0]), &cw = ty(m, n.inputs[1]), &cs = ty(m, n.inputs[4]), &st = ty(m, n.inputs[5]), &seqs = ty(m, n.inputs[6]), &out = ty(m, n.outputs[0]);
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    if (!is_act(x.dtype) || !width) return false;
    auto inside = [&](const char* name, int64_t cols) {
        const int64_t off = a.int_or(name, 0);
        return off >= 0 && off + cols <= (int64_t)*width;
    };
    if (!inside("q_offset", C) || !inside("a_offset", H) || !inside("b_offset", H)) return false;
    if (cw.dtype != DType::F32 || cw.shape.size() != 2 || !is_const(cw.shape[0], C) || !is_const(cw.shape[1], K)) return false;
    if (!is_f32_vector(m, n.inputs[2], (uint64_t)H) || !is_f32_vector(m, n.inputs[3], (uint64_t)H)) return false;
    if (cs.dtype != x.dtype || cs.shape.size() != 3 || !is_const(cs.shape[1], K) || !is_const(cs.shape[2], C)) return false;
    if (st.dtype != DType::F32 || st.shape.size() != 4 || st.shape[0] != cs.shape[0] || !is_const(st.shape[1], H) || !is_const(st.shape[2], D) || !is_const(st.shape[3], V)) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is_const(seqs.shape[1], 4)) return false;
    return out.dtype == DType::F32 && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is_const(out.shape[1], H * V);
}
void delta_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::DeltaRuleDesc d{};
    d.heads = a.int_("heads");
    d.kv_heads = a.int_("kv_heads");
    d.dim = a.int_("dim");
    d.vdim = a.int_("vdim");
    d.taps = a.int_("taps");
    d.q_off = a.int_or("q_offset", 0);
    d.a_off = a.int_or("a_offset", 0);
    d.b_off = a.int_or("b_offset", 0);
    d.q_scale = a.float_or("q_scale", 1.0);
    d.unit_eps = a.float_or("unit_epsilon", 1e-6);
    oxk::emit_delta_rule(c.em, d, c.ins[0], c.ins[1], c.ins[2], c.ins[3], c.outs[1], c.outs[2], c.ins[6], c.outs[0]);
}

// ── onyxia.LightningAttention ──
// proj, decay table, state, seqs → out, state
bool lightning_accepts(const Module& m, const Node& n) {
    const Attrs& a = n.composite.attrs;
    if (n.inputs.size() != 4 || n.outputs.size() != 2) return false;
    const int64_t H = a.int_or("heads", 0), D = a.int_or("dim", 0), V = a.int_or("vdim", 0);
    if (H <= 0 || D <= 0 || D > 512 || V <= 0) return false;
    const TensorType &x = ty(m, n.inputs[0]), &decay = ty(m, n.inputs[1]), &st = ty(m, n.inputs[2]), &seqs = ty(m, n.inputs[3]), &out = ty(m, n.outputs[0]);
    auto width = x.shape.size() == 2 ? x.shape[1].as_const() : std::nullopt;
    if (!is_act(x.dtype) || !width) return false;
    auto inside = [&](const char* name, int64_t cols) {
        const int64_t off = a.int_or(name, 0);
        return off >= 0 && off + cols <= (int64_t)*width;
    };
    if (!inside("q_offset", H * D) || !inside("k_offset", H * D) || !inside("v_offset", H * V)) return false;
    if (decay.dtype != DType::F32 || decay.shape.size() != 2 || !is_const(decay.shape[0], H) || !is_const(decay.shape[1], oxk::kLightningChunk + 2)) return false;
    if (st.dtype != DType::F32 || st.shape.size() != 4 || !is_const(st.shape[1], H) || !is_const(st.shape[2], D) || !is_const(st.shape[3], V)) return false;
    if (seqs.dtype != DType::I32 || seqs.shape.size() != 2 || !is_const(seqs.shape[1], 4)) return false;
    return out.dtype == DType::F32 && out.shape.size() == 2 && out.shape[0] == x.shape[0] && is_const(out.shape[1], H * V);
}
void lightning_lower(FusedCtx& c) {
    const Attrs& a = c.node.composite.attrs;
    oxk::LightningDesc d{};
    d.heads = a.int_("heads");
    d.dim = a.int_("dim");
    d.vdim = a.int_("vdim");
    d.q_off = a.int_or("q_offset", 0);
    d.k_off = a.int_or("k_offset", 0);
    d.v_off = a.int_or("v_offset", 0);
    oxk::emit_lightning(c.em, d, c.ins[0], c.ins[1], c.outs[1], c.ins[3], c.outs[0]);
}

// ── onyxia.AllReduce (tensor parallelism) ──
bool allreduce_accepts(const Module& m, const Node& n) {
    if (n.inputs.size() != 1 || n.outputs.size() != 1) return false;
    const TensorType& t = ty(m, n.inputs[0]);
    return (t.dtype == DType::F16 || t.dtype == DType::F32) && t == ty(m, n.outputs[0]);
}
void allreduce_lower(FusedCtx& c) { oxk::emit_allreduce(c.em, c.ins[0], c.outs[0]); }

}  // namespace

}  // namespace oxrt

namespace oxk {
void emit_allreduce(Emitter& em, const TRef& x, const TRef& y) {
    if (x.numel() == 0) return;
    CollP p{};
    p.count = (unsigned long long)x.numel();
    p.dtype = x.dtype;
    LaunchRec r;
    r.coll = 1;
    r.params.resize(sizeof(CollP));
    std::memcpy(r.params.data(), &p, sizeof(CollP));
    r.relocs.push_back(Reloc{(uint32_t)offsetof(CollP, send), x.buf});
    r.relocs.push_back(Reloc{(uint32_t)offsetof(CollP, recv), y.buf});
    r.label = "allreduce";
    r.node = em.node;
    em.recs.push_back(std::move(r));
}
}  // namespace oxk

namespace oxrt {

const KernelRegistry& standard_kernels() {
    static const KernelRegistry reg = [] {
        KernelRegistry r;
        r.add({"Softmax", softmax_accepts, softmax_lower});
        r.add({"SimplifiedLayerNormalization", rmsnorm_accepts, rmsnorm_lower});
        r.add({"Gelu", gelu_accepts, gelu_lower});
        r.add({"com.microsoft.RotaryEmbedding", rotary_accepts, rotary_lower});
        r.add({"com.microsoft.GemmaRotaryEmbedding", rotary_accepts, rotary_lower});
        r.add({"com.microsoft.GroupQueryAttention", gqa_accepts, gqa_lower});
        r.add({"com.microsoft.MatMulNBits", nbits_accepts, nbits_lower});
        r.add({"onyxia.AllReduce", allreduce_accepts, allreduce_lower});
        r.add({"onyxia.ResidualNorm", residual_norm_accepts, residual_norm_lower});
        r.add({"onyxia.Linear", linear_accepts, linear_lower});
        r.add({"onyxia.PagedAttention", paged_accepts, paged_lower, {{1, 4}, {2, 5}}});
        r.add({"onyxia.GatedRecurrence", recurrence_accepts, recurrence_lower, {{1, 8}, {2, 9}}});
        r.add({"onyxia.PagedKVAttention", paged_kv_accepts, paged_kv_lower, {{1, 2}, {2, 3}}});
        r.add({"onyxia.SharedKVAttention", shared_kv_accepts, paged_kv_lower});
        r.add({"onyxia.LightningAttention", lightning_accepts, lightning_lower, {{1, 2}}});
        r.add({"onyxia.GatedLinearAttention", gated_linear_accepts, gated_linear_lower, {{1, 2}}});
        r.add({"onyxia.GatedDeltaRule", delta_accepts, delta_lower, {{1, 4}, {2, 5}}});
        r.add({"onyxia.MixtureOfExperts", moe_accepts, moe_lower});
        r.add({"onyxia.LatentAttention", latent_accepts, latent_lower, {{1, 5}}});
        r.add({"onyxia.SelectiveScan", selective_accepts, selective_lower, {{1, 8}, {2, 9}}});
        return r;
    }();
    return reg;
}

}  // namespace oxrt
