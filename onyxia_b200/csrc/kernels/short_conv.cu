// Causal convolution over time per channel with silu, over a ragged batch: u = silu(Σ_k w[c, taps − 1 − k] x_(t − k)[c] + b[c]).
//
// Inputs of earlier steps come from a ring per slot (row = position modulo taps); inputs in front of a sequence's start are zero. Where every
// sequence has one new token it can go to its ring at once (`keep`), in place of the oldest one, which nobody reads any more; in a longer portion a
// token may still need what a later one replaces.
//
// Bytes per token and channel: 4.
#include "tc_util.cuh"

namespace oxk {

namespace {

struct ConvP {
    const void* proj;             // [rows, ld], from the first channel's column on
    const float *cw, *cb;         // [width, taps], [width] or null
    void* u;                      // [rows, width]
    void* ring;                   // [slots, taps, width]
    const int* seqs;
    ErrWord* err;
    long long rows, ld;
    int n_seqs, n_slots, width, taps, keep, node;
};

__device__ __forceinline__ int slot_of(const ConvP& p, int slot) {
    if ((unsigned)slot >= (unsigned)p.n_slots) {
        report(p.err, ERR_GATHER_OOB, p.node, slot, p.n_slots);
        return 0;
    }
    return slot;
}

// V consecutive channels of one row
template <typename T, int V> struct Chan {
    float v[V];
    __device__ __forceinline__ void load(const T* from) {
        if constexpr (V == 8) {
            const uint4 x = *reinterpret_cast<const uint4*>(from);
            const unsigned w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
            for (int e = 0; e < 4; e++) {
                v[2 * e] = __uint_as_float(w[e] << 16);
                v[2 * e + 1] = __uint_as_float(w[e] & 0xFFFF0000u);
            }
        } else {
            v[0] = to_f(from[0]);
        }
    }
    __device__ __forceinline__ void store(T* to) const {
        if constexpr (V == 8) *reinterpret_cast<uint4*>(to) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
        else to[0] = from_f<T>(v[0]);
    }
};
// Thread: V channels of ROWS consecutive batch rows, the inputs of the last taps in registers where TAPS is known.
template <typename T, int V, int TAPS, int ROWS> __global__ void __launch_bounds__(128) short_conv(const ConvP p) {
    pdl_enter();
    const int c = (blockIdx.x * 128 + threadIdx.x) * V;
    const long long row0 = (long long)blockIdx.y * ROWS;
    if (c >= p.width) return;
    const int taps = TAPS ? TAPS : p.taps;
    const T* x = (const T*)p.proj + c;
    const T* ring = (const T*)p.ring + c;
    Chan<T, V> now[ROWS], w[TAPS ? TAPS : 1], bias;
#pragma unroll
    for (int j = 0; j < ROWS; j++)
        if (row0 + j < p.rows) now[j].load(x + (row0 + j) * p.ld);
#pragma unroll
    for (int e = 0; e < V; e++) {
        bias.v[e] = p.cb ? p.cb[c + e] : 0.f;
        if constexpr (TAPS > 0)
#pragma unroll
            for (int k = 0; k < TAPS; k++) {
                if constexpr (TAPS == 4) {
                    if (k == 0) {
                        const float4 all = *reinterpret_cast<const float4*>(p.cw + (long long)(c + e) * 4);
                        w[0].v[e] = all.w;
                        w[1].v[e] = all.z;
                        w[2].v[e] = all.y;
                        w[3].v[e] = all.x;
                    }
                } else {
                    w[k].v[e] = p.cw[(long long)(c + e) * TAPS + TAPS - 1 - k];
                }
            }
    }
    int s = find_seq(p.seqs, p.n_seqs, (int)row0);
    SeqRow sq = load_seq(p.seqs, s);
    int slot = slot_of(p, sq.slot);
    // the input `back` tokens before row `row`
    auto input = [&](long long row, int back) {
        Chan<T, V> in;
        const int pos = sq.past + (int)(row - sq.start) - back;
        if (pos < 0) {
#pragma unroll
            for (int e = 0; e < V; e++) in.v[e] = 0.f;
        } else if (row - back >= sq.start) {
            in.load(x + (row - back) * p.ld);
        } else {
            in.load(ring + ((long long)slot * taps + pos % taps) * p.width);
        }
        return in;
    };
    Chan<T, V> before[TAPS > 1 ? TAPS - 1 : 1];  // the inputs 1, 2, … tokens before
    bool known = false;
#pragma unroll
    for (int j = 0; j < ROWS; j++) {
        const long long row = row0 + j;
        if (row >= p.rows) break;
        if (row >= sq.start + sq.len && s + 1 < p.n_seqs) {
            while (s + 1 < p.n_seqs && row >= sq.start + sq.len) sq = load_seq(p.seqs, ++s);
            slot = slot_of(p, sq.slot);
            known = false;
        }
        Chan<T, V> acc = bias;
        if constexpr (TAPS > 0) {
            if (!known)
#pragma unroll
                for (int k = 1; k < TAPS; k++) before[k - 1] = input(row, k);
            known = true;
#pragma unroll
            for (int e = 0; e < V; e++) {
                acc.v[e] = fmaf(now[j].v[e], w[0].v[e], acc.v[e]);
#pragma unroll
                for (int k = 1; k < TAPS; k++) acc.v[e] = fmaf(before[k - 1].v[e], w[k].v[e], acc.v[e]);
            }
#pragma unroll
            for (int k = TAPS - 1; k > 1; k--) before[k - 1] = before[k - 2];
            if constexpr (TAPS > 1) before[0] = now[j];
        } else {
            for (int k = 0; k < taps; k++) {
                const Chan<T, V> in = input(row, k);
#pragma unroll
                for (int e = 0; e < V; e++) acc.v[e] = fmaf(in.v[e], p.cw[(long long)(c + e) * taps + taps - 1 - k], acc.v[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < V; e++) acc.v[e] *= sizeof(T) == 2 ? sigmoid_fast(acc.v[e]) : sigmoid_f(acc.v[e]);
        acc.store((T*)p.u + row * p.width + c);
        if (ROWS == 1 && p.keep) now[0].store((T*)p.ring + ((long long)slot * taps + sq.past % taps) * p.width + c);
    }
}

}  // namespace

void emit_short_conv(Emitter& em, const ShortConvDesc& d, const TRef& proj, const TRef& w, const TRef* bias, const TRef& ring, const TRef& seqs, const TRef& u) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    const bool bf = proj.dtype == DT_BF16;
    ConvP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.n_seqs = (int)n_seqs;
    p.n_slots = (int)ring.shape[0];
    p.width = (int)d.width;
    p.taps = (int)d.taps;
    p.keep = d.keep;
    p.node = em.node;
    const bool decode = rows == n_seqs, vec = bf && d.width % 8 == 0 && p.ld % 8 == 0 && d.x_off % 8 == 0 && d.taps == 4;
    const int per_thread = decode ? 1 : 8;
    void (*k)(const ConvP);
    if (vec) k = decode ? short_conv<bf16, 8, 4, 1> : short_conv<bf16, 8, 4, 8>;
    else if (bf) k = decode ? short_conv<bf16, 1, 0, 1> : short_conv<bf16, 1, 0, 8>;
    else k = decode ? short_conv<float, 1, 0, 1> : short_conv<float, 1, 0, 8>;
    const int64_t per_cta = 128 * (vec ? 8 : 1);
    em.launch(k, dim3((unsigned)((d.width + per_cta - 1) / per_cta), (unsigned)((rows + per_thread - 1) / per_thread)), dim3(128), 0, p,
              {{&p.proj, proj.buf.at(d.x_off * (bf ? 2 : 4))}, {&p.cw, w.buf}, {&p.cb, bias ? bias->buf : Buf{kSlotNull, 0}}, {&p.u, u.buf}, {&p.ring, ring.buf},
               {&p.seqs, seqs.buf}, {&p.err, Buf{kSlotErr, 0}}},
              "short_conv", /*pdl=*/true);
}

}  // namespace oxk
