// Linear attention with a matrix state per head whose rows decay by a factor of their own, over a ragged batch with per-slot state.
//
//   S_t = diag(α_t) S_{t−1} + k_t v_tᵀ,  o_t = S_tᵀ (c q_t),  α_t = sigmoid(z_t)^(1 / tau)       (S: dim × vdim in f32)
//
//   gated_linear_step    one new token per sequence: 32 columns of one head's state per CTA, read, updated, multiplied and written once.
//                        Also runs whole portions token by token (f32, and shapes that the chunk kernels do not take)
//
// A step multiplies by α as S + (α − 1) S, since α itself next to 1 would be rounded too coarsely.
//
// Bytes: step 8 · dim · vdim per head and sequence.
#include "paged_util.cuh"

namespace oxk {

namespace {

struct GatedP {
    const void* proj;      // [rows, ld]
    const float* z;        // [rows, heads · dim]
    float* state;          // [slots, heads, dim, vdim]
    const int* seqs;
    float* out;            // [rows, heads · vdim]
    ErrWord* err;
    long long rows, ld, q_off, k_off, v_off;
    int n_seqs, n_slots, heads, dim, vdim, node;
    int singles_only;      // step: leave longer portions to the chunk kernels
    float rate, q_scale;   // rate = 1 / tau
};

__device__ __forceinline__ int slot_of(const GatedP& p, int slot) {
    if ((unsigned)slot >= (unsigned)p.n_slots) {
        report(p.err, ERR_GATHER_OOB, p.node, slot, p.n_slots);
        return 0;
    }
    return slot;
}

// ───────────────────────────── token by token ───────────────────────────
// Grid: (32-column slices, heads, sequences). Thread: four columns, every 32nd row of the state. V4: vdim is a multiple of 4.
constexpr int kStepThreads = 256;
template <typename T, int DI, bool V4> __global__ void __launch_bounds__(kStepThreads) gated_linear_step(const GatedP p) {
    __shared__ float red[8][32];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d0 = tid >> 3, c0 = blockIdx.x * 32 + (tid & 7) * 4, h = blockIdx.y;
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);  // no launch of a step writes the batch description
    const bool mine = sq.len == 1 || !p.singles_only;
    float* state = p.state + ((long long)slot_of(p, sq.slot) * p.heads + h) * p.dim * p.vdim;
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
    for (int t = 0; t < sq.len; t++) {
        const T* x = (const T*)p.proj + (sq.start + t) * p.ld;
        const T *q = x + p.q_off + (long long)h * p.dim, *k = x + p.k_off + (long long)h * p.dim, *v = x + p.v_off + (long long)h * p.vdim;
        const float* z = p.z + ((sq.start + t) * (long long)p.heads + h) * p.dim;
        float vv[4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int e = 0; e < 4; e++) vv[e] = c0 + e < p.vdim ? to_f(v[c0 + e]) : 0.f;
#pragma unroll
        for (int i = 0; i < DI; i++) {
            const int d = d0 + 32 * i;
            const bool live = d < p.dim;
            const float kd = live ? to_f(k[d]) : 0.f, qd = live ? to_f(q[d]) * p.q_scale : 0.f, less = live ? expm1f(-softplus_f(-z[d]) * p.rate) : 0.f;
#pragma unroll
            for (int e = 0; e < 4; e++) {
                S[i][e] = fmaf(kd, vv[e], fmaf(less, S[i][e], S[i][e]));
                o[e] = fmaf(qd, S[i][e], o[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < 4; e++) {
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
            if (lane < 8) red[warp][lane * 4 + e] = o[e];
        }
        __syncthreads();
        if (tid < 32 && blockIdx.x * 32 + tid < p.vdim) {
            float s = 0.f;
#pragma unroll
            for (int w = 0; w < 8; w++) s += red[w][tid];
            p.out[((sq.start + t) * (long long)p.heads + h) * p.vdim + blockIdx.x * 32 + tid] = s;
        }
        __syncthreads();
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

using GatedKernel = void (*)(const GatedP);
template <typename T, bool V4> GatedKernel step_kernel(int64_t dim) {
    return dim <= 32 ? gated_linear_step<T, 1, V4> : dim <= 64 ? gated_linear_step<T, 2, V4> : dim <= 128 ? gated_linear_step<T, 4, V4>
           : dim <= 256 ? gated_linear_step<T, 8, V4> : gated_linear_step<T, 16, V4>;
}

}  // namespace

void emit_gated_linear(Emitter& em, const GatedLinearDesc& d, const TRef& proj, const TRef& z, const TRef& state, const TRef& seqs, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    GatedP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.q_off = d.q_off;
    p.k_off = d.k_off;
    p.v_off = d.v_off;
    p.n_seqs = (int)n_seqs;
    p.n_slots = (int)state.shape[0];
    p.heads = (int)d.heads;
    p.dim = (int)d.dim;
    p.vdim = (int)d.vdim;
    p.rate = (float)(1.0 / d.tau);
    p.q_scale = (float)d.q_scale;
    p.node = em.node;
    const bool bf = proj.dtype == DT_BF16, v4 = d.vdim % 4 == 0;
    auto launch = [&](GatedKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.z, z.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf}, {&p.out, out.buf}, {&p.err, Buf{kSlotErr, 0}}}, label, /*pdl=*/true);
    };
    const GatedKernel k = bf ? (v4 ? step_kernel<bf16, true>(d.dim) : step_kernel<bf16, false>(d.dim)) : (v4 ? step_kernel<float, true>(d.dim) : step_kernel<float, false>(d.dim));
    launch(k, dim3((unsigned)((d.vdim + 31) / 32), (unsigned)d.heads, (unsigned)n_seqs), kStepThreads, 0, "gated_linear_step");
}

}  // namespace oxk
