// Linear attention with a matrix state per head that decays by a constant, over a ragged batch with per-slot state.
//
//   S_t = γ S_{t−1} + k_t v_tᵀ,  o_t = S_tᵀ q_t       (S: dim × vdim in f32, γ per head)
//
//   lightning_step    one new token per sequence: 32 columns of one head's state per CTA, read, updated, multiplied and written
//                     once. Also runs whole portions token by token (f32, and shapes the chunk kernels do not take)
//   lightning_chunk   sequences with several new tokens, cut into chunks of C = 64: Σ_t γ^(n−1−t) k_t v_tᵀ of every chunk
//   lightning_scan    per state element: the state that enters every chunk, and the one that the portion leaves
//   lightning_out     per chunk: o_i = γ^(i+1) Sᵀ q_i + Σ_{j ≤ i} γ^(i−j) (q_i · k_j) v_j
//
// The chunk kernels multiply on `mma.sync`. q, k and v are bf16 as projected; what is f32 there (the state, the decayed
// scores, the decayed values) enters as the sum of two bf16, which keeps 16 bits of it. Powers of γ are f32 roundings
// of 64-bit ones; a step multiplies by γ as S + (γ − 1) S, since γ itself next to 1 would be rounded too coarsely.
//
// Bytes: step 8 · dim · vdim per head and sequence. FLOPs of a portion: 2 · (C (dim + 2 vdim) + 4 dim · vdim) per token and head.
#include "chunk_util.cuh"

namespace oxk {

namespace {

constexpr int kC = kLightningChunk;

struct LightP {
    const void* proj;      // [rows, ld]
    const float* decay;    // [heads, kC + 2]
    float* state;          // [slots, heads, dim, vdim]
    const int* seqs;
    float* chunk;          // [chunks, heads, dim, vdim]: contributions, then entering states (4 elements: 4 high, 4 low bf16)
    float* out;            // [rows, heads · vdim]
    ErrWord* err;
    long long rows, ld, q_off, k_off, v_off;
    int n_seqs, n_slots, heads, dim, vdim, node;
    int singles_only;      // step: leave longer portions to the chunk kernels
};

__device__ __forceinline__ int slot_of(const LightP& p, int slot) {
    if ((unsigned)slot >= (unsigned)p.n_slots) {
        report(p.err, ERR_GATHER_OOB, p.node, slot, p.n_slots);
        return 0;
    }
    return slot;
}

// ───────────────────────────── token by token ───────────────────────────
// Grid: (32-column slices, heads, sequences). Thread: four columns, every 32nd row of the state. V4: vdim is a multiple of 4.
constexpr int kStepThreads = 256;
template <typename T, int DI, bool V4> __global__ void __launch_bounds__(kStepThreads) lightning_step(const LightP p) {
    __shared__ float red[8][32];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d0 = tid >> 3, c0 = blockIdx.x * 32 + (tid & 7) * 4, h = blockIdx.y;
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);  // no launch of a step writes the batch description
    const bool mine = sq.len == 1 || !p.singles_only;
    const float less = p.decay[h * (kC + 2) + kC + 1];
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
        float vv[4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int e = 0; e < 4; e++) vv[e] = c0 + e < p.vdim ? to_f(v[c0 + e]) : 0.f;
#pragma unroll
        for (int i = 0; i < DI; i++) {
            const int d = d0 + 32 * i;
            const float kd = d < p.dim ? to_f(k[d]) : 0.f, qd = d < p.dim ? to_f(q[d]) : 0.f;
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

// ───────────────────────────── chunks ───────────────────────────────────
// Grid: (chunks, heads, 64-column slices); eight warps, 16 rows of the state each in turn.
__global__ void __launch_bounds__(256) lightning_chunk(const LightP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // k [kC][row_stride], v high, v low [kC][kColStride]
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, v0 = blockIdx.z * kCols;
    const int n_tok = min(kC, sq.len - first), stride = row_stride(p.dim), n_cols = min(kCols, p.vdim - v0);
    const bf16* x = (const bf16*)p.proj + (long long)(sq.start + first) * p.ld;
    const unsigned ks = smem_u32(smem), vh = ks + kC * stride, vl = vh + kC * kColStride;
    load_rows(ks, stride, x + p.k_off + (long long)h * p.dim, p.ld, n_tok, p.dim, padded(p.dim), tid, 256);
    cp_async_commit();
    unsigned char *vh_p = smem + kC * stride, *vl_p = vh_p + kC * kColStride;
    for (int i = tid; i < kC * (kCols / 8); i += 256) {
        const int r = i / (kCols / 8), c = i % (kCols / 8) * 8;
        uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
        if (r < n_tok && c < n_cols) {
            const uint4 v = *reinterpret_cast<const uint4*>(x + r * p.ld + p.v_off + (long long)h * p.vdim + v0 + c);
            const float f = p.decay[h * (kC + 2) + n_tok - 1 - r];
            const unsigned w[4] = {v.x, v.y, v.z, v.w};
            unsigned oh[4], ol[4];
#pragma unroll
            for (int e = 0; e < 4; e++) split2(__uint_as_float(w[e] << 16) * f, __uint_as_float(w[e] & 0xFFFF0000u) * f, oh + e, ol + e);
            hi = make_uint4(oh[0], oh[1], oh[2], oh[3]);
            lo = make_uint4(ol[0], ol[1], ol[2], ol[3]);
        }
        *reinterpret_cast<uint4*>(vh_p + r * kColStride + c * 2) = hi;
        *reinterpret_cast<uint4*>(vl_p + r * kColStride + c * 2) = lo;
    }
    cp_async_wait<0>();
    __syncthreads();
    float* dst = p.chunk + ((long long)blockIdx.x * p.heads + h) * p.dim * p.vdim;
    for (int m0 = warp * 16; m0 < p.dim; m0 += 128) {
        float acc[kCols / 8][4];
#pragma unroll
        for (int n = 0; n < kCols / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[n][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < kC / 16; kk++) {
            unsigned a[4];
            ldmatrix_x4_trans(a, ks + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * stride + m0 * 2 + ((lane >> 3) & 1) * 16);
#pragma unroll
            for (int n = 0; n < kCols / 8; n += 2) {
                const unsigned at = (kk * 16 + (lane & 15)) * kColStride + n * 16 + (lane >> 4) * 16;
                unsigned b[4];
                ldmatrix_x4_trans(b, vh + at);
                mma_bf16(acc[n], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(acc[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                ldmatrix_x4_trans(b, vl + at);
                mma_bf16(acc[n], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(acc[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < kCols / 8; n++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int d = m0 + g8 + 8 * r, c = n * 8 + t4 * 2;
                if (d < p.dim && c < n_cols) *reinterpret_cast<float2*>(dst + (long long)d * p.vdim + v0 + c) = make_float2(acc[n][2 * r], acc[n][2 * r + 1]);
            }
    }
}

// Grid: (1024-element pieces of a head's state, heads, sequences); four elements per thread.
__global__ void __launch_bounds__(256) lightning_scan(const LightP p) {
    constexpr int kAhead = 8;
    pdl_trigger();
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int h = blockIdx.y, at = (blockIdx.x * 256 + threadIdx.x) * 4, size = p.dim * p.vdim;
    const int chunk0 = chunks_before(p.seqs, blockIdx.z);
    pdl_wait();
    if (sq.len == 1 || at >= size) return;
    const float* decay = p.decay + h * (kC + 2);
    float4* state = reinterpret_cast<float4*>(p.state + ((long long)slot_of(p, sq.slot) * p.heads + h) * size + at);
    float4* chunk = reinterpret_cast<float4*>(p.chunk + ((long long)chunk0 * p.heads + h) * size + at);
    const long long next = (long long)p.heads * size / 4;
    const int n = (sq.len + kC - 1) / kC;
    float4 S = sq.past > 0 ? *state : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c0 = 0; c0 < n; c0 += kAhead) {
        float4 x[kAhead];
#pragma unroll
        for (int j = 0; j < kAhead; j++) x[j] = c0 + j < n ? chunk[(c0 + j) * next] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < kAhead; j++) {
            if (c0 + j >= n) break;
            uint4 w;
            split2(S.x, S.y, &w.x, &w.z);
            split2(S.z, S.w, &w.y, &w.w);
            *reinterpret_cast<uint4*>(chunk + (c0 + j) * next) = w;
            const float f = decay[min(kC, sq.len - (c0 + j) * kC)];
            S = make_float4(fmaf(S.x, f, x[j].x), fmaf(S.y, f, x[j].y), fmaf(S.z, f, x[j].z), fmaf(S.w, f, x[j].w));
        }
    }
    *state = S;
}

// Grid: (chunks, heads, 64-column slices); four warps of 16 tokens.
__global__ void __launch_bounds__(128) lightning_out(const LightP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // q, k [kC][row_stride], v [kC], state high, low [dim][kColStride]
    __shared__ float power[kC + 1];
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, v0 = blockIdx.z * kCols;
    const int n_tok = min(kC, sq.len - first), stride = row_stride(p.dim), dp = padded(p.dim), n_cols = min(kCols, p.vdim - v0);
    const bf16* x = (const bf16*)p.proj + (long long)(sq.start + first) * p.ld;
    const unsigned qs = smem_u32(smem), ks = qs + kC * stride, vs = ks + kC * stride, sh = vs + kC * kColStride, sl = sh + dp * kColStride;
    load_rows(qs, stride, x + p.q_off + (long long)h * p.dim, p.ld, n_tok, p.dim, dp, tid, 128);
    load_rows(ks, stride, x + p.k_off + (long long)h * p.dim, p.ld, n_tok, p.dim, dp, tid, 128);
    load_rows(vs, kColStride, x + p.v_off + (long long)h * p.vdim + v0, p.ld, n_tok, n_cols, kCols, tid, 128);
    cp_async_commit();
    for (int i = tid; i <= kC; i += 128) power[i] = p.decay[h * (kC + 2) + i];
    const bool carried = sq.past > 0 || first > 0;  // a state enters the chunk
    if (carried) {
        unsigned char* s_p = smem + (size_t)2 * kC * stride + kC * kColStride;
        const uint4* src = reinterpret_cast<const uint4*>(p.chunk + ((long long)blockIdx.x * p.heads + h) * p.dim * p.vdim + v0);
        for (int i = tid; i < dp * (kCols / 4); i += 128) {
            const int d = i / (kCols / 4), c = i % (kCols / 4);
            const uint4 w = d < p.dim && c * 4 < n_cols ? src[(long long)d * (p.vdim / 4) + c] : make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint2*>(s_p + d * kColStride + c * 8) = make_uint2(w.x, w.y);
            *reinterpret_cast<uint2*>(s_p + (dp + d) * kColStride + c * 8) = make_uint2(w.z, w.w);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    const int r0 = warp * 16;
    if (r0 >= n_tok) return;
    float s[kC / 8][4], o[kCols / 8][4];
#pragma unroll
    for (int n = 0; n < kC / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) s[n][e] = o[n][e] = 0.f;
    for (int kk = 0; kk < dp / 16; kk++) {
        unsigned a[4];
        ldmatrix_x4(a, qs + (r0 + (lane & 15)) * stride + kk * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int n = 0; n < kC / 8; n += 2) {
            if (n * 8 > r0 + 15) continue;  // keys behind every row of the warp
            unsigned b[4];
            ldmatrix_x4(b, ks + (n * 8 + (lane & 7) + (lane >> 4) * 8) * stride + kk * 32 + ((lane >> 3) & 1) * 16);
            mma_bf16(s[n], a[0], a[1], a[2], a[3], b[0], b[1]);
            mma_bf16(s[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
        }
        if (!carried) continue;
#pragma unroll
        for (int n = 0; n < kCols / 8; n += 2) {
            const unsigned at = (kk * 16 + (lane & 15)) * kColStride + n * 16 + (lane >> 4) * 16;
            unsigned b[4];
            ldmatrix_x4_trans(b, sh + at);
            mma_bf16(o[n], a[0], a[1], a[2], a[3], b[0], b[1]);
            mma_bf16(o[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            ldmatrix_x4_trans(b, sl + at);
            mma_bf16(o[n], a[0], a[1], a[2], a[3], b[0], b[1]);
            mma_bf16(o[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
        }
    }
    const int i0 = r0 + g8;  // this lane's rows: i0, i0 + 8
    const float in0 = power[i0 + 1], in1 = power[i0 + 9];
#pragma unroll
    for (int n = 0; n < kCols / 8; n++) {
        o[n][0] *= in0;
        o[n][1] *= in0;
        o[n][2] *= in1;
        o[n][3] *= in1;
    }
#pragma unroll
    for (int n = 0; n < kC / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int back = i0 + 8 * (e >> 1) - (n * 8 + t4 * 2 + (e & 1));
            s[n][e] = back >= 0 ? s[n][e] * power[back] : 0.f;
        }
#pragma unroll
    for (int kk = 0; kk < kC / 16; kk++) {
        if (kk * 16 > r0 + 15) continue;
        unsigned ah[4], al[4];
        split2(s[2 * kk][0], s[2 * kk][1], ah, al);
        split2(s[2 * kk][2], s[2 * kk][3], ah + 1, al + 1);
        split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ah + 2, al + 2);
        split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ah + 3, al + 3);
#pragma unroll
        for (int n = 0; n < kCols / 8; n += 2) {
            unsigned b[4];
            ldmatrix_x4_trans(b, vs + (kk * 16 + (lane & 15)) * kColStride + n * 16 + (lane >> 4) * 16);
            mma_bf16(o[n], ah[0], ah[1], ah[2], ah[3], b[0], b[1]);
            mma_bf16(o[n + 1], ah[0], ah[1], ah[2], ah[3], b[2], b[3]);
            mma_bf16(o[n], al[0], al[1], al[2], al[3], b[0], b[1]);
            mma_bf16(o[n + 1], al[0], al[1], al[2], al[3], b[2], b[3]);
        }
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int i = i0 + 8 * r;
        if (i >= n_tok) continue;
        float* out = p.out + ((sq.start + first + i) * (long long)p.heads + h) * p.vdim + v0;
#pragma unroll
        for (int n = 0; n < kCols / 8; n++) {
            const int c = n * 8 + t4 * 2;
            if (c < n_cols) *reinterpret_cast<float2*>(out + c) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
        }
    }
}

using LightKernel = void (*)(const LightP);
template <typename T, bool V4> LightKernel step_kernel(int64_t dim) {
    return dim <= 32 ? lightning_step<T, 1, V4> : dim <= 64 ? lightning_step<T, 2, V4> : dim <= 128 ? lightning_step<T, 4, V4>
           : dim <= 256 ? lightning_step<T, 8, V4> : lightning_step<T, 16, V4>;
}

}  // namespace

void emit_lightning(Emitter& em, const LightningDesc& d, const TRef& proj, const TRef& decay, const TRef& state, const TRef& seqs, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    LightP p{};
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
    p.node = em.node;
    const bool bf = proj.dtype == DT_BF16, v4 = d.vdim % 4 == 0;
    const bool chunks = bf && rows > n_seqs && d.dim % 8 == 0 && d.vdim % 8 == 0 && d.dim <= 256 && p.ld % 8 == 0 && d.q_off % 8 == 0 && d.k_off % 8 == 0 &&
                        d.v_off % 8 == 0 && proj.buf.off % 16 == 0;
    const int64_t tiles = rows / kC + n_seqs;
    const Buf chunk = chunks ? em.scratch((size_t)(tiles * d.heads * d.dim * d.vdim) * 4) : Buf{kSlotNull, 0};
    auto launch = [&](LightKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.decay, decay.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf}, {&p.chunk, chunk}, {&p.out, out.buf},
                   {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    p.singles_only = chunks;
    if (!chunks || n_seqs > 1) {
        const LightKernel k = bf ? (v4 ? step_kernel<bf16, true>(d.dim) : step_kernel<bf16, false>(d.dim))
                                 : (v4 ? step_kernel<float, true>(d.dim) : step_kernel<float, false>(d.dim));
        launch(k, dim3((unsigned)((d.vdim + 31) / 32), (unsigned)d.heads, (unsigned)n_seqs), kStepThreads, 0, "lightning_step");
    }
    if (!chunks) return;
    const unsigned slices = (unsigned)((d.vdim + kCols - 1) / kCols), stride = (unsigned)row_stride((int)d.dim);
    const unsigned chunk_smem = kC * stride + 2 * kC * kColStride, out_smem = 2 * kC * stride + kC * kColStride + 2 * (unsigned)padded((int)d.dim) * kColStride;
    ensure_max_dynamic_smem((const void*)lightning_chunk, 200 * 1024);
    ensure_max_dynamic_smem((const void*)lightning_out, 200 * 1024);
    launch(lightning_chunk, dim3((unsigned)tiles, (unsigned)d.heads, slices), 256, chunk_smem, "lightning_chunk");
    launch(lightning_scan, dim3((unsigned)((d.dim * d.vdim + 1023) / 1024), (unsigned)d.heads, (unsigned)n_seqs), 256, 0, "lightning_scan");
    launch(lightning_out, dim3((unsigned)tiles, (unsigned)d.heads, slices), 128, out_smem, "lightning_out");
}

}  // namespace oxk
