// Gated delta rule ("Gated Delta Networks: Improving Mamba2 with Delta Rule", Yang, Kautz and Hatamizadeh) over a ragged batch with per-slot
// state, behind a short convolution.
//
//   S ← g S,  u = beta (v − Sᵀ k),  S ← S + k uᵀ,  o = Sᵀ q             (S: dim × vdim in f32; q, k unit vectors)
//
// q, k and v are the convolution's results (short_conv.cu) in the activation type; unit norms, decays and step sizes are formed from them and
// from the projection in f32.
//
//   delta_step     one new token per sequence: 32 columns of one head's state per CTA, read, updated, multiplied and written once. Also runs
//                  whole portions token by token (f32, and shapes that the chunk kernels do not take)
//
// Bytes: step 8 · dim · vdim per head and sequence.
#include "paged_util.cuh"

namespace oxk {

namespace {

struct DeltaP {
    const void* proj;            // [rows, ld]
    const void* u;               // [rows, channels]: q, k, v behind the convolution
    const float *decay, *dt_b;   // [heads]
    void* ring;                  // [slots, taps, channels]
    float* state;                // [slots, heads, dim, vdim]
    const int* seqs;
    float* out;                  // [rows, heads · vdim]
    ErrWord* err;
    long long rows, ld, x_off, a_off, b_off;
    int n_seqs, n_slots, heads, kv_heads, dim, vdim, taps, channels, node;
    int singles_only;            // step: leave longer portions to the chunk kernels
    float q_scale, eps;
};

__device__ __forceinline__ int slot_of(const DeltaP& p, int slot) {
    if ((unsigned)slot >= (unsigned)p.n_slots) {
        report(p.err, ERR_GATHER_OOB, p.node, slot, p.n_slots);
        return 0;
    }
    return slot;
}
// A token's logarithm of the decay, and its step size.
template <typename T> __device__ __forceinline__ float log_decay(const DeltaP& p, long long row, int h) {
    return -p.decay[h] * softplus_f(to_f(((const T*)p.proj)[row * p.ld + p.a_off + h]) + p.dt_b[h]);
}
template <typename T> __device__ __forceinline__ float step_size(const DeltaP& p, long long row, int h) {
    return sigmoid_f(to_f(((const T*)p.proj)[row * p.ld + p.b_off + h]));
}

// ───────────────────────────── token by token ───────────────────────────
// Grid: (32-column slices, heads, sequences). Thread: four columns, every 32nd row of the state. V4: vdim is a multiple of 4.
constexpr int kStepThreads = 256;
template <typename T, int DI, bool V4> __global__ void __launch_bounds__(kStepThreads) delta_step(const DeltaP p) {
    __shared__ float red[8][32], norms[8][2];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d0 = tid >> 3, c0 = blockIdx.x * 32 + (tid & 7) * 4, h = blockIdx.y, g = h / (p.heads / p.kv_heads);
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);  // no launch of a step writes the batch description
    const bool mine = sq.len == 1 || !p.singles_only;
    const int slot = slot_of(p, sq.slot);
    float* state = p.state + ((long long)slot * p.heads + h) * p.dim * p.vdim;
    float S[DI][4];
#pragma unroll
    for (int i = 0; i < DI; i++) {  // this layer's state is written by no launch before this one
        const int d = d0 + 32 * i;
        const bool live = mine && sq.past > 0 && d < p.dim;
        if constexpr (V4) {
            const float4 v = live && c0 < p.vdim ? *reinterpret_cast<const float4*>(state + (long long)d * p.vdim + c0) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[i][0] = v.x;
            S[i][1] = v.y;
            S[i][2] = v.z;
            S[i][3] = v.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++) S[i][e] = live && c0 + e < p.vdim ? state[(long long)d * p.vdim + c0 + e] : 0.f;
        }
    }
    pdl_wait();
    if (!mine) return;
    // sums over the state's rows: per column, in every thread of it
    auto over_rows = [&](float (&o)[4]) {
#pragma unroll
        for (int e = 0; e < 4; e++) {
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
            if (lane < 8) red[warp][lane * 4 + e] = o[e];
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 4; e++) {
            o[e] = 0.f;
#pragma unroll
            for (int w = 0; w < 8; w++) o[e] += red[w][(tid & 7) * 4 + e];
        }
        __syncthreads();
    };
    for (int t = 0; t < sq.len; t++) {
        const long long row = sq.start + t;
        const T *x = (const T*)p.u + row * p.channels, *q = x + (long long)g * p.dim, *k = q + (long long)p.kv_heads * p.dim;
        const T* v = x + 2ll * p.kv_heads * p.dim + (long long)h * p.vdim;
        float kd[DI], qd[DI], vv[4], qq = 0.f, kk = 0.f;
#pragma unroll
        for (int i = 0; i < DI; i++) {
            const int d = d0 + 32 * i;
            kd[i] = d < p.dim ? to_f(k[d]) : 0.f;
            qd[i] = d < p.dim ? to_f(q[d]) : 0.f;
            kk = fmaf(kd[i], kd[i], kk);
            qq = fmaf(qd[i], qd[i], qq);
        }
#pragma unroll
        for (int e = 0; e < 4; e++) vv[e] = c0 + e < p.vdim ? to_f(v[c0 + e]) : 0.f;
        // eight threads hold the same rows
        for (int o = 8; o < 32; o <<= 1) {
            kk += __shfl_xor_sync(0xffffffffu, kk, o);
            qq += __shfl_xor_sync(0xffffffffu, qq, o);
        }
        if (lane == 0) {
            norms[warp][0] = kk;
            norms[warp][1] = qq;
        }
        const float less = expm1f(log_decay<T>(p, row, h)), beta = step_size<T>(p, row, h);
        float got[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < DI; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                S[i][e] = fmaf(less, S[i][e], S[i][e]);
                got[e] = fmaf(kd[i], S[i][e], got[e]);
            }
        over_rows(got);
        kk = qq = 0.f;
#pragma unroll
        for (int w = 0; w < 8; w++) {
            kk += norms[w][0];
            qq += norms[w][1];
        }
        const float kf = 1.f / sqrtf(kk + p.eps), qf = p.q_scale / sqrtf(qq + p.eps);
        float o[4] = {0.f, 0.f, 0.f, 0.f}, add[4];
#pragma unroll
        for (int e = 0; e < 4; e++) add[e] = beta * (vv[e] - got[e] * kf) * kf;
#pragma unroll
        for (int i = 0; i < DI; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                S[i][e] = fmaf(kd[i], add[e], S[i][e]);
                o[e] = fmaf(qd[i], S[i][e], o[e]);
            }
        over_rows(o);
        if (d0 == 0)
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (c0 + e < p.vdim) p.out[(row * p.heads + h) * p.vdim + c0 + e] = o[e] * qf;
    }
#pragma unroll
    for (int i = 0; i < DI; i++) {
        const int d = d0 + 32 * i;
        if (d >= p.dim) continue;
        if constexpr (V4) {
            if (c0 < p.vdim) *reinterpret_cast<float4*>(state + (long long)d * p.vdim + c0) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (c0 + e < p.vdim) state[(long long)d * p.vdim + c0 + e] = S[i][e];
        }
    }
}

// A sequence's last inputs go to its ring. Grid: (channel blocks, taps, sequences).
template <typename T> __global__ void __launch_bounds__(256) delta_keep(const DeltaP p) {
    pdl_enter();
    const int c = blockIdx.x * 256 + threadIdx.x;
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int t = sq.len - 1 - (int)blockIdx.y;
    if (c >= p.channels || t < 0) return;
    ((T*)p.ring)[((long long)slot_of(p, sq.slot) * p.taps + (sq.past + t) % p.taps) * p.channels + c] = ((const T*)p.proj)[(sq.start + t) * p.ld + p.x_off + c];
}

using DeltaKernel = void (*)(const DeltaP);
template <typename T, bool V4> DeltaKernel step_kernel(int64_t dim) {
    return dim <= 32 ? delta_step<T, 1, V4> : dim <= 64 ? delta_step<T, 2, V4> : dim <= 128 ? delta_step<T, 4, V4> : dim <= 256 ? delta_step<T, 8, V4> : delta_step<T, 16, V4>;
}

}  // namespace

void emit_delta_rule(Emitter& em, const DeltaRuleDesc& d, const TRef& proj, const TRef& conv_w, const TRef& decay, const TRef& dt_bias, const TRef& conv_state,
                     const TRef& state, const TRef& seqs, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    const bool bf = proj.dtype == DT_BF16, v4 = d.vdim % 4 == 0;
    DeltaP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.x_off = d.q_off;
    p.a_off = d.a_off;
    p.b_off = d.b_off;
    p.n_seqs = (int)n_seqs;
    p.n_slots = (int)state.shape[0];
    p.heads = (int)d.heads;
    p.kv_heads = (int)d.kv_heads;
    p.dim = (int)d.dim;
    p.vdim = (int)d.vdim;
    p.taps = (int)d.taps;
    p.channels = (int)(2 * d.kv_heads * d.dim + d.heads * d.vdim);
    p.q_scale = (float)d.q_scale;
    p.eps = (float)d.unit_eps;
    p.node = em.node;
    TRef u;
    u.dtype = proj.dtype;
    u.shape = {rows, p.channels};
    u.buf = em.scratch((size_t)(rows * p.channels * (bf ? 2 : 4)));
    ShortConvDesc cd;
    cd.width = p.channels;
    cd.taps = d.taps;
    cd.x_off = d.q_off;
    emit_short_conv(em, cd, proj, conv_w, nullptr, conv_state, seqs, u);
    auto launch = [&](DeltaKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.u, u.buf}, {&p.decay, decay.buf}, {&p.dt_b, dt_bias.buf}, {&p.ring, conv_state.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf},
                   {&p.out, out.buf}, {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    launch(bf ? delta_keep<bf16> : delta_keep<float>, dim3((unsigned)((p.channels + 255) / 256), (unsigned)d.taps, (unsigned)n_seqs), 256, 0, "delta_keep");
    const DeltaKernel k = bf ? (v4 ? step_kernel<bf16, true>(d.dim) : step_kernel<bf16, false>(d.dim)) : (v4 ? step_kernel<float, true>(d.dim) : step_kernel<float, false>(d.dim));
    launch(k, dim3((unsigned)((d.vdim + 31) / 32), (unsigned)d.heads, (unsigned)n_seqs), kStepThreads, 0, "delta_step");
}

}  // namespace oxk
