// Linear attention with a matrix state per head whose rows decay by a factor of their own, over a ragged batch with per-slot state.
//
//   S_t = diag(α_t) S_{t−1} + k_t v_tᵀ,  o_t = S_tᵀ (c q_t),  α_t = sigmoid(z_t)^(1 / tau)       (S: dim × vdim in f32)
//
//   gated_linear_step    one new token per sequence: 32 columns of one head's state per CTA, read, updated, multiplied and written once.
//                        Also runs whole portions token by token (f32, and shapes that the chunk kernels do not take)
//   gated_linear_decay   sequences with several new tokens, cut into chunks of 64: b_i, the sum of log2 α from the chunk's first token on
//   gated_linear_chunk   per chunk: what it adds to the state, Σ_j (2^(b_last − b_j) k_j) v_jᵀ; and its scores
//                        A_ij = Σ_d q_id k_jd 2^(b_id − b_jd) for j ≤ i, in blocks of 16 × 16
//   gated_linear_scan    per state element: the state that enters every chunk, and the one that the portion leaves
//   gated_linear_out     per chunk: o_i = Sᵀ (2^(b_i) q_i) + Σ_{j ≤ i} A_ij v_j
//
// A step multiplies by α as S + (α − 1) S, since α itself next to 1 would be rounded too coarsely. The chunk kernels multiply on `mma.sync`; what is
// f32 there enters as the sum of two bf16, which keeps 16 bits of it. The powers of a block of scores are taken relative to the token in front of
// its rows, so that none of another block's keys is above 1; in a block on the diagonal keys may be, and where one would leave the range of the
// format the block is formed without factors.
//
// Bytes: step 8 · dim · vdim per head and sequence. FLOPs of a portion: 2 · (64 (dim + vdim) + 4 dim · vdim) per token and head.
#include "chunk_util.cuh"

namespace oxk {

namespace {

struct GatedP {
    const void* proj;      // [rows, ld]
    const float* z;        // [rows, heads · dim]
    float* state;          // [slots, heads, dim, vdim]
    const int* seqs;
    float* out;            // [rows, heads · vdim]
    float* sums;           // [rows, heads · dim]: b
    float* chunk;          // [chunks, heads, dim, vdim]: contributions, then entering states (4 elements: 4 high, 4 low bf16)
    float* scores;         // [chunks, heads, 64, 64], times q_scale
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

// ───────────────────────────── chunks ───────────────────────────────────
constexpr int kC = kLightningChunk, kScoreBlocks = 10;  // blocks of 16 × 16 scores on and below the diagonal

// Grid: (chunks, blocks of 32 channels of all heads); a quarter of the tokens per warp.
__global__ void __launch_bounds__(128) gated_linear_decay(const GatedP p) {
    constexpr int kMine = kC / 4;
    __shared__ float part[4][32];
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int lane = threadIdx.x & 31, quarter = threadIdx.x >> 5, n_tok = min(kC, sq.len - first) - quarter * kMine, c = blockIdx.y * 32 + lane;
    const long long width = (long long)p.heads * p.dim, at = (sq.start + first + quarter * kMine) * width + c;
    const float rate = -p.rate * kLog2e;
    float b[kMine], sum = 0.f;
#pragma unroll
    for (int i = 0; i < kMine; i++) b[i] = i < n_tok && c < width ? p.z[at + i * width] : 0.f;
#pragma unroll
    for (int i = 0; i < kMine; i++) b[i] = sum = fmaf(softplus_f(-b[i]), rate, sum);
    part[quarter][lane] = sum;
    __syncthreads();
    float before = 0.f;
    for (int i = 0; i < quarter; i++) before += part[i][lane];
#pragma unroll
    for (int i = 0; i < kMine; i++)
        if (i < n_tok && c < width) p.sums[at + i * width] = before + b[i];
}

// Eight consecutive elements of a row times 2^(their sums' difference), as high and low parts.
struct Eight {
    unsigned hi[4], lo[4];
};
__device__ __forceinline__ Eight weighed(uint4 x, const float (&power)[8]) {
    const unsigned w[4] = {x.x, x.y, x.z, x.w};
    Eight o;
#pragma unroll
    for (int e = 0; e < 4; e++) split2(__uint_as_float(w[e] << 16) * power[2 * e], __uint_as_float(w[e] & 0xFFFF0000u) * power[2 * e + 1], o.hi + e, o.lo + e);
    return o;
}
__device__ __forceinline__ void load8(float (&v)[8], const float* from, bool live) {
    const float4 a = live ? *reinterpret_cast<const float4*>(from) : make_float4(0.f, 0.f, 0.f, 0.f), b = live ? *reinterpret_cast<const float4*>(from + 4) : a;
    v[0] = a.x;
    v[1] = a.y;
    v[2] = a.z;
    v[3] = a.w;
    v[4] = b.x;
    v[5] = b.y;
    v[6] = b.z;
    v[7] = b.w;
}

// Scores of 16 queries and 16 keys of a chunk, by one warp. q, k, b: the chunk's first token.
__device__ __forceinline__ void score_block(const GatedP& p, const bf16* q, const bf16* k, const float* b, int n_tok, int rows, int cols, float* out) {
    const int lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
    const long long width = (long long)p.heads * p.dim;
    const bool diagonal = rows == cols;
    float s[2][4];
#pragma unroll
    for (int n = 0; n < 2; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) s[n][e] = 0.f;
    bool wild = false;
#pragma unroll 1
    for (int d0 = 0; d0 < p.dim; d0 += 32) {  // (a dot product does not care in which order its dimensions come)
        const int d = d0 + t4 * 8;
        const bool live = d < p.dim;
        float ref[8], sum[8];
        load8(ref, b + (rows - 1) * width + d, live && rows > 0);
        Eight qs[2], ks[2];
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = min(rows + g8 + 8 * r, n_tok - 1), j = min(cols + g8 + 8 * r, n_tok - 1);
            load8(sum, b + i * width + d, live);
#pragma unroll
            for (int e = 0; e < 8; e++) sum[e] = power2(sum[e] - ref[e]);
            qs[r] = weighed(live ? *reinterpret_cast<const uint4*>(q + i * p.ld + d) : make_uint4(0, 0, 0, 0), sum);
            load8(sum, b + j * width + d, live);
#pragma unroll
            for (int e = 0; e < 8; e++) {
                wild = wild || ref[e] - sum[e] > 100.f;
                sum[e] = power2(ref[e] - sum[e]);
            }
            ks[r] = weighed(live ? *reinterpret_cast<const uint4*>(k + j * p.ld + d) : make_uint4(0, 0, 0, 0), sum);
        }
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int x = 2 * half, y = x + 1;
                mma_bf16(s[n], qs[0].hi[x], qs[1].hi[x], qs[0].hi[y], qs[1].hi[y], ks[n].hi[x], ks[n].hi[y]);
                mma_bf16(s[n], qs[0].hi[x], qs[1].hi[x], qs[0].hi[y], qs[1].hi[y], ks[n].lo[x], ks[n].lo[y]);
                mma_bf16(s[n], qs[0].lo[x], qs[1].lo[x], qs[0].lo[y], qs[1].lo[y], ks[n].hi[x], ks[n].hi[y]);
            }
    }
    const bool direct = diagonal && __any_sync(0xffffffffu, wild);
#pragma unroll
    for (int n = 0; n < 2; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = rows + g8 + 8 * (e >> 1), j = cols + n * 8 + t4 * 2 + (e & 1);
            float v = s[n][e];
            if (direct && j <= i && i < n_tok) {
                v = 0.f;
                for (int d = 0; d < p.dim; d++) v = fmaf(to_f(q[i * p.ld + d]) * to_f(k[j * p.ld + d]), exp2f(b[i * width + d] - b[j * width + d]), v);
            }
            s[n][e] = j <= i ? v * p.q_scale : 0.f;
        }
#pragma unroll
    for (int n = 0; n < 2; n++)
#pragma unroll
        for (int r = 0; r < 2; r++)
            *reinterpret_cast<float2*>(out + (rows + g8 + 8 * r) * kC + cols + n * 8 + t4 * 2) = make_float2(s[n][2 * r], s[n][2 * r + 1]);
}

// Grid: (chunks, heads, 64-column slices and one more for the scores).
constexpr int kChunkThreads = kScoreBlocks * 32;
__global__ void __launch_bounds__(kChunkThreads, 2) gated_linear_chunk(const GatedP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // k high, low [kC][row_stride], v [kC][kColStride]
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, v0 = blockIdx.z * kCols;
    const int n_tok = min(kC, sq.len - first), stride = row_stride(p.dim), n_cols = min(kCols, p.vdim - v0), dp = padded(p.dim);
    const bf16* x = (const bf16*)p.proj + (long long)(sq.start + first) * p.ld;
    const long long width = (long long)p.heads * p.dim;
    const bf16 *q = x + p.q_off + (long long)h * p.dim, *k = x + p.k_off + (long long)h * p.dim;
    const float* b = p.sums + (long long)(sq.start + first) * width + (long long)h * p.dim;
    if (blockIdx.z == gridDim.z - 1) {
        int row = 0;
        while ((row + 1) * (row + 2) / 2 <= warp) row++;
        const int col = warp - row * (row + 1) / 2;
        if (row * 16 < n_tok) score_block(p, q, k, b, n_tok, row * 16, col * 16, p.scores + ((long long)blockIdx.x * p.heads + h) * kC * kC);
        return;
    }
    const unsigned kh = smem_u32(smem), kl = kh + kC * stride, vs = kl + kC * stride;
    load_rows(vs, kColStride, x + p.v_off + (long long)h * p.vdim + v0, p.ld, n_tok, n_cols, kCols, tid, kChunkThreads);
    cp_async_commit();
    for (int i = tid; i < kC * (dp / 8); i += kChunkThreads) {
        const int r = i / (dp / 8), d = i % (dp / 8) * 8;
        Eight o{};
        if (r < n_tok && d < p.dim) {
            float last[8], sum[8];
            load8(last, b + (n_tok - 1) * width + d, true);
            load8(sum, b + r * width + d, true);
#pragma unroll
            for (int e = 0; e < 8; e++) sum[e] = power2(last[e] - sum[e]);
            o = weighed(*reinterpret_cast<const uint4*>(k + r * p.ld + d), sum);
        }
        *reinterpret_cast<uint4*>(smem + r * stride + d * 2) = make_uint4(o.hi[0], o.hi[1], o.hi[2], o.hi[3]);
        *reinterpret_cast<uint4*>(smem + (kC + r) * stride + d * 2) = make_uint4(o.lo[0], o.lo[1], o.lo[2], o.lo[3]);
    }
    cp_async_wait<0>();
    __syncthreads();
    float* dst = p.chunk + ((long long)blockIdx.x * p.heads + h) * p.dim * p.vdim;
    for (int m0 = warp * 16; m0 < p.dim; m0 += kScoreBlocks * 16) {
        float acc[kCols / 8][4];
#pragma unroll
        for (int n = 0; n < kCols / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[n][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < kC / 16; kk++) {
            const unsigned at = (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * stride + m0 * 2 + ((lane >> 3) & 1) * 16;
            unsigned ah[4], al[4];
            ldmatrix_x4_trans(ah, kh + at);
            ldmatrix_x4_trans(al, kl + at);
#pragma unroll
            for (int n = 0; n < kCols / 8; n += 2) {
                unsigned v[4];
                ldmatrix_x4_trans(v, vs + (kk * 16 + (lane & 15)) * kColStride + n * 16 + (lane >> 4) * 16);
                mma_bf16(acc[n], ah[0], ah[1], ah[2], ah[3], v[0], v[1]);
                mma_bf16(acc[n + 1], ah[0], ah[1], ah[2], ah[3], v[2], v[3]);
                mma_bf16(acc[n], al[0], al[1], al[2], al[3], v[0], v[1]);
                mma_bf16(acc[n + 1], al[0], al[1], al[2], al[3], v[2], v[3]);
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

// Grid: (1024-element pieces of a head's state, heads, sequences); four elements of a row per thread.
__global__ void __launch_bounds__(256) gated_linear_scan(const GatedP p) {
    constexpr int kAhead = 8;
    pdl_trigger();
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int h = blockIdx.y, at = (blockIdx.x * 256 + threadIdx.x) * 4, size = p.dim * p.vdim;
    const int chunk0 = chunks_before(p.seqs, blockIdx.z);
    pdl_wait();
    if (sq.len == 1 || at >= size) return;
    const long long width = (long long)p.heads * p.dim;
    const float* b = p.sums + sq.start * width + (long long)h * p.dim + at / p.vdim;
    float4* state = reinterpret_cast<float4*>(p.state + ((long long)slot_of(p, sq.slot) * p.heads + h) * size + at);
    float4* chunk = reinterpret_cast<float4*>(p.chunk + ((long long)chunk0 * p.heads + h) * size + at);
    const long long next = (long long)p.heads * size / 4;
    const int n = (sq.len + kC - 1) / kC;
    float4 S = sq.past > 0 ? *state : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c0 = 0; c0 < n; c0 += kAhead) {
        float4 x[kAhead];
        float f[kAhead];
#pragma unroll
        for (int j = 0; j < kAhead; j++) {
            x[j] = c0 + j < n ? chunk[(c0 + j) * next] : make_float4(0.f, 0.f, 0.f, 0.f);
            f[j] = c0 + j < n ? b[(long long)(min((c0 + j + 1) * kC, sq.len) - 1) * width] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < kAhead; j++) {
            if (c0 + j >= n) break;
            uint4 w;
            split2(S.x, S.y, &w.x, &w.z);
            split2(S.z, S.w, &w.y, &w.w);
            *reinterpret_cast<uint4*>(chunk + (c0 + j) * next) = w;
            const float g = exp2f(f[j]);
            S = make_float4(fmaf(S.x, g, x[j].x), fmaf(S.y, g, x[j].y), fmaf(S.z, g, x[j].z), fmaf(S.w, g, x[j].w));
        }
    }
    *state = S;
}

// Grid: (chunks, heads, 64-column slices); four warps of 16 tokens.
__global__ void __launch_bounds__(128) gated_linear_out(const GatedP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // v [kC][kColStride], state high, low [dim][kColStride]
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, v0 = blockIdx.z * kCols;
    const int n_tok = min(kC, sq.len - first), dp = padded(p.dim), n_cols = min(kCols, p.vdim - v0);
    const long long width = (long long)p.heads * p.dim;
    const bf16* x = (const bf16*)p.proj + (long long)(sq.start + first) * p.ld;
    const unsigned vs = smem_u32(smem), sh = vs + kC * kColStride, sl = sh + dp * kColStride;
    load_rows(vs, kColStride, x + p.v_off + (long long)h * p.vdim + v0, p.ld, n_tok, n_cols, kCols, tid, 128);
    cp_async_commit();
    const bool carried = sq.past > 0 || first > 0;  // a state enters the chunk
    if (carried) {
        unsigned char* s_p = smem + kC * kColStride;
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
    float o[kCols / 8][4];
#pragma unroll
    for (int n = 0; n < kCols / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    if (carried) {
        const bf16* q[2];
        const float* b[2];
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = min(r0 + g8 + 8 * r, n_tok - 1);
            q[r] = x + i * p.ld + p.q_off + (long long)h * p.dim;
            b[r] = p.sums + (sq.start + first + i) * width + (long long)h * p.dim;
        }
        for (int kk = 0; kk < dp / 16; kk++) {
            unsigned ah[4], al[4];
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = e & 1, d = kk * 16 + t4 * 2 + (e >> 1) * 8;
                const bool live = d < p.dim;
                const unsigned w = live ? *reinterpret_cast<const unsigned*>(q[r] + d) : 0u;
                const float2 s = live ? *reinterpret_cast<const float2*>(b[r] + d) : make_float2(0.f, 0.f);
                split2(__uint_as_float(w << 16) * (power2(s.x) * p.q_scale), __uint_as_float(w & 0xFFFF0000u) * (power2(s.y) * p.q_scale), ah + e, al + e);
            }
#pragma unroll
            for (int n = 0; n < kCols / 8; n += 2) {
                const unsigned at = (kk * 16 + (lane & 15)) * kColStride + n * 16 + (lane >> 4) * 16;
                unsigned s[4];
                ldmatrix_x4_trans(s, sh + at);
                mma_bf16(o[n], ah[0], ah[1], ah[2], ah[3], s[0], s[1]);
                mma_bf16(o[n + 1], ah[0], ah[1], ah[2], ah[3], s[2], s[3]);
                mma_bf16(o[n], al[0], al[1], al[2], al[3], s[0], s[1]);
                mma_bf16(o[n + 1], al[0], al[1], al[2], al[3], s[2], s[3]);
                ldmatrix_x4_trans(s, sl + at);
                mma_bf16(o[n], ah[0], ah[1], ah[2], ah[3], s[0], s[1]);
                mma_bf16(o[n + 1], ah[0], ah[1], ah[2], ah[3], s[2], s[3]);
            }
        }
    }
    const float* scores = p.scores + ((long long)blockIdx.x * p.heads + h) * kC * kC + (r0 + g8) * kC;
#pragma unroll
    for (int kk = 0; kk < kC / 16; kk++) {
        if (kk * 16 > r0 + 15) continue;
        unsigned ah[4], al[4];
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const float2 s = *reinterpret_cast<const float2*>(scores + (e & 1) * 8 * kC + kk * 16 + (e >> 1) * 8 + t4 * 2);
            split2(s.x, s.y, ah + e, al + e);
        }
#pragma unroll
        for (int n = 0; n < kCols / 8; n += 2) {
            unsigned v[4];
            ldmatrix_x4_trans(v, vs + (kk * 16 + (lane & 15)) * kColStride + n * 16 + (lane >> 4) * 16);
            mma_bf16(o[n], ah[0], ah[1], ah[2], ah[3], v[0], v[1]);
            mma_bf16(o[n + 1], ah[0], ah[1], ah[2], ah[3], v[2], v[3]);
            mma_bf16(o[n], al[0], al[1], al[2], al[3], v[0], v[1]);
            mma_bf16(o[n + 1], al[0], al[1], al[2], al[3], v[2], v[3]);
        }
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int i = r0 + g8 + 8 * r;
        if (i >= n_tok) continue;
        float* out = p.out + ((sq.start + first + i) * (long long)p.heads + h) * p.vdim + v0;
#pragma unroll
        for (int n = 0; n < kCols / 8; n++) {
            const int c = n * 8 + t4 * 2;
            if (c < n_cols) *reinterpret_cast<float2*>(out + c) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
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
    const bool chunks = bf && rows > n_seqs && d.dim % 8 == 0 && d.vdim % 8 == 0 && d.dim <= 256 && p.ld % 8 == 0 && d.q_off % 8 == 0 && d.k_off % 8 == 0 &&
                        d.v_off % 8 == 0 && proj.buf.off % 16 == 0 && z.buf.off % 16 == 0;
    const int64_t tiles = std::min(rows, rows / kC + n_seqs);
    const Buf none{kSlotNull, 0}, sums = chunks ? em.scratch((size_t)(rows * d.heads * d.dim) * 4) : none;
    const Buf chunk = chunks ? em.scratch((size_t)(tiles * d.heads * d.dim * d.vdim) * 4) : none, scores = chunks ? em.scratch((size_t)(tiles * d.heads * kC * kC) * 4) : none;
    p.singles_only = chunks;
    auto launch = [&](GatedKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.z, z.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf}, {&p.out, out.buf}, {&p.sums, sums}, {&p.chunk, chunk}, {&p.scores, scores},
                   {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    if (chunks) {
        const unsigned slices = (unsigned)((d.vdim + kCols - 1) / kCols), stride = (unsigned)row_stride((int)d.dim);
        const unsigned chunk_smem = 2 * kC * stride + kC * kColStride, out_smem = kC * kColStride + 2 * (unsigned)padded((int)d.dim) * kColStride;
        ensure_max_dynamic_smem((const void*)gated_linear_chunk, 200 * 1024);
        ensure_max_dynamic_smem((const void*)gated_linear_out, 200 * 1024);
        launch(gated_linear_decay, dim3((unsigned)tiles, (unsigned)((d.heads * d.dim + 31) / 32)), 128, 0, "gated_linear_decay");
        launch(gated_linear_chunk, dim3((unsigned)tiles, (unsigned)d.heads, slices + 1), kChunkThreads, chunk_smem, "gated_linear_chunk");
        launch(gated_linear_scan, dim3((unsigned)((d.dim * d.vdim + 1023) / 1024), (unsigned)d.heads, (unsigned)n_seqs), 256, 0, "gated_linear_scan");
        launch(gated_linear_out, dim3((unsigned)tiles, (unsigned)d.heads, slices), 128, out_smem, "gated_linear_out");
        if (n_seqs == 1) return;
    }
    const GatedKernel k = bf ? (v4 ? step_kernel<bf16, true>(d.dim) : step_kernel<bf16, false>(d.dim)) : (v4 ? step_kernel<float, true>(d.dim) : step_kernel<float, false>(d.dim));
    launch(k, dim3((unsigned)((d.vdim + 31) / 32), (unsigned)d.heads, (unsigned)n_seqs), kStepThreads, 0, "gated_linear_step");
}

}  // namespace oxk
