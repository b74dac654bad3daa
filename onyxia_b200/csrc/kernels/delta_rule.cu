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
//   delta_chunk    sequences with several new tokens, cut into chunks of 64. With b_i the sum of log2 g from the chunk's first token on, and S what
//                  enters the chunk, u_i = beta_i (v_i − 2^(b_i) Sᵀ k_i − Σ_{j < i} 2^(b_i − b_j) (k_i · k_j) u_j): a triangular system, whose inverse T
//                  is formed in f32 (blocks of 16, then the blocks below them). U = T diag(beta) V and W = T diag(beta 2^b) K leave u = U − W S
//   delta_scan     chunk after chunk, 16 or 32 columns of the state per CTA, the state in registers: u = U − W S,
//                  S ← 2^(b_last) S + Σ_j 2^(b_last − b_j) k_j u_jᵀ; a chunk's W and k lie together and arrive as bulk copies, W one chunk ahead. It
//                  leaves u and the entering states
//   delta_out      per chunk: o_i = 2^(b_i) Sᵀ q_i + Σ_{j ≤ i} 2^(b_i − b_j) (q_i · k_j) u_j
//   delta_keep     the last inputs of the convolution
//
// The chunk kernels multiply on `mma.sync`. Convolved q and k are exact operands, their unit factors join the f32 results; what is f32 enters as
// the sum of two bf16, which keeps 16 bits of it.
//
// Bytes: step 8 · dim · vdim per head and sequence. FLOPs of a portion: 2 · (64 (3 dim + 2 vdim) + 6 dim · vdim) per token and head.
#include "chunk_util.cuh"

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
    float *sums, *unit;          // [rows, heads]: b, the unit factor of k
    float *factor, *whole;       // [rows, heads]: 2^(b_last − b) · unit; [chunks, heads]: 2^(b_last)
    unsigned char* tiles;        // [chunks, heads]: W's high and low part and k, [3][64][row_stride(dim)], as delta_scan keeps them
    float* uv;                   // [rows, heads, vdim]: U
    bf16* us;                    // [2][rows, heads, vdim]: u, high and low part
    bf16* chunk;                 // [2][chunks, heads, dim, vdim]: entering states, high and low part
    ErrWord* err;
    long long rows, ld, x_off, a_off, b_off;
    int n_seqs, n_slots, heads, kv_heads, dim, vdim, taps, channels, node;
    int singles_only;            // step: leave longer portions to the chunk kernels
    int chunks;                  // most chunks of a batch
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

// ───────────────────────────── chunks ───────────────────────────────────
constexpr int kC = kLightningChunk, kTStride = kC + 4;  // floats per row of a 64 × 64 matrix
// 1 / length of the rows of a chunk in shared memory; eight warps. Rows beyond the tokens are zero.
__device__ __forceinline__ void unit_factors(const unsigned char* rows, int stride, int dim, float eps, float scale, float* to, int warp, int warps) {
    const int lane = threadIdx.x & 31;
    for (int r = warp; r < kC; r += warps) {
        float ss = 0.f;
        for (int d = lane * 2; d < dim; d += 64) {
            const unsigned w = *reinterpret_cast<const unsigned*>(rows + r * stride + d * 2);
            const float a = __uint_as_float(w << 16), b = __uint_as_float(w & 0xFFFF0000u);
            ss = fmaf(a, a, fmaf(b, b, ss));
        }
        ss = warp_sum(ss);
        if (lane == 0) to[r] = scale / sqrtf(ss + eps);
    }
}

// Grid: (chunks, heads); eight warps.
__global__ void __launch_bounds__(256) delta_chunk(const DeltaP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // A, then T [64][kTStride], k [kC][row_stride(dim)], v [kC][row_stride(vdim)]
    __shared__ float b[kC], beta[kC], unit[kC], part[3][16][17];
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, g = h / (p.heads / p.kv_heads);
    const int n_tok = min(kC, sq.len - first), ks = row_stride(p.dim), vst = row_stride(p.vdim), dp = padded(p.dim), vp = padded(p.vdim);
    const long long row0 = sq.start + first;
    float* T = reinterpret_cast<float*>(smem);
    unsigned char* k_p = smem + kC * kTStride * 4;
    const unsigned k_s = smem_u32(k_p), v_s = k_s + kC * ks;
    const bf16 *k = (const bf16*)p.u + row0 * p.channels + (long long)(p.kv_heads + g) * p.dim, *v = (const bf16*)p.u + row0 * p.channels + 2ll * p.kv_heads * p.dim + (long long)h * p.vdim;
    load_rows(k_s, ks, k, p.channels, n_tok, p.dim, dp, tid, 256);
    load_rows(v_s, vst, v, p.channels, n_tok, p.vdim, vp, tid, 256);
    cp_async_commit();
    if (warp == 0) {  // sums of the decays' logarithms, two tokens per lane
        const int i = lane * 2;
        const float x = i < n_tok ? log_decay<bf16>(p, row0 + i, h) * kLog2e : 0.f, y = i + 1 < n_tok ? log_decay<bf16>(p, row0 + i + 1, h) * kLog2e : 0.f;
        float s = x + y;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float t = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += t;
        }
        b[i] = s - y;
        b[i + 1] = s;
    } else if (warp < 3) {
        const int i = (warp - 1) * 32 + lane;
        beta[i] = i < n_tok ? step_size<bf16>(p, row0 + i, h) : 0.f;
    }
    for (int i = tid; i < kC * kTStride; i += 256) T[i] = 0.f;
    cp_async_wait<0>();
    __syncthreads();
    unit_factors(k_p, ks, p.dim, p.eps, 1.f, unit, warp, 8);
    __syncthreads();
    if (tid < n_tok) {
        p.sums[(row0 + tid) * p.heads + h] = b[tid];
        p.unit[(row0 + tid) * p.heads + h] = unit[tid];
        p.factor[(row0 + tid) * p.heads + h] = exp2f(b[n_tok - 1] - b[tid]) * unit[tid];
        if (tid == 0) p.whole[(long long)blockIdx.x * p.heads + h] = exp2f(b[n_tok - 1]);
    }
    unsigned char* tile = p.tiles + ((long long)blockIdx.x * p.heads + h) * 3 * kC * ks;
    for (int i = tid; i < kC * ks / 16; i += 256) reinterpret_cast<uint4*>(tile + 2 * kC * ks)[i] = reinterpret_cast<const uint4*>(k_p)[i];
    // A_ij = beta_i 2^(b_i − b_j) (k_i · k_j) for j < i, in blocks of 16 × 16
    for (int block = warp; block < 10; block += 8) {
        int row = 0;
        while ((row + 1) * (row + 2) / 2 <= block) row++;
        const int r0 = row * 16, c0 = (block - row * (row + 1) / 2) * 16;
        float s[2][4];
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[n][e] = 0.f;
        for (int kk = 0; kk < dp / 16; kk++) {
            unsigned a[4], c[4];
            ldmatrix_x4(a, k_s + (r0 + (lane & 15)) * ks + kk * 32 + (lane >> 4) * 16);
            ldmatrix_x4(c, k_s + (c0 + (lane & 7) + (lane >> 4) * 8) * ks + kk * 32 + ((lane >> 3) & 1) * 16);
            mma_bf16(s[0], a[0], a[1], a[2], a[3], c[0], c[1]);
            mma_bf16(s[1], a[0], a[1], a[2], a[3], c[2], c[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = r0 + g8 + 8 * (e >> 1), j = c0 + n * 8 + t4 * 2 + (e & 1);
                T[i * kTStride + j] = j < i ? s[n][e] * beta[i] * unit[i] * unit[j] * exp2f(b[i] - b[j]) : 0.f;
            }
    }
    __syncthreads();
    // (I + A)^−1: blocks on the diagonal by substitution, a column per lane
    if (warp < 4) {
        float* D = T + warp * 16 * (kTStride + 1);
        float x[16];
#pragma unroll
        for (int r = 0; r < 16; r++) {
            float s = lane == r ? 1.f : 0.f;
#pragma unroll
            for (int c = 0; c < 16; c++)
                if (c < r) s = fmaf(-D[r * kTStride + c], x[c], s);
            x[r] = s;
        }
        __syncwarp();
        if (lane < 16)
#pragma unroll
            for (int r = 0; r < 16; r++) D[r * kTStride + lane] = r >= lane ? x[r] : 0.f;
    }
    __syncthreads();
    // blocks below, a row of blocks after the other: T_IJ = −T_II Σ_{J ≤ K < I} A_IK T_KJ; an element per thread and block
    const int er = tid >> 4, ec = tid & 15;
    for (int I = 1; I < 4; I++) {
        // the sums of all J before any A_IK is replaced
        for (int J = 0; J < I; J++) {
            float s = 0.f;
            for (int c = J * 16; c < I * 16; c++) s = fmaf(T[(I * 16 + er) * kTStride + c], T[c * kTStride + J * 16 + ec], s);
            part[J][er][ec] = s;
        }
        __syncthreads();
        for (int J = 0; J < I; J++) {
            float s = 0.f;
#pragma unroll
            for (int c = 0; c < 16; c++) s = fmaf(-T[(I * 16 + er) * kTStride + I * 16 + c], part[J][c][ec], s);
            T[(I * 16 + er) * kTStride + J * 16 + ec] = s;
        }
        __syncthreads();
    }
    // U = T diag(beta) V, W = T diag(beta 2^b unit) K: 16 tokens per warp and half of the columns
    const int m = warp & 3, side = warp >> 2, r0 = m * 16;
    float* uv = p.uv + (row0 * p.heads + h) * (long long)p.vdim;
#pragma unroll
    for (int which = 0; which < 2; which++) {
        unsigned ah[4][4], al[4][4];
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            if (kk > m) break;
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = r0 + g8 + 8 * (e & 1), j = kk * 16 + (e >> 1) * 8 + t4 * 2;
                const float2 t = *reinterpret_cast<const float2*>(T + i * kTStride + j);
                float f0 = beta[j], f1 = beta[j + 1];
                if (which) {
                    f0 *= exp2f(b[j]) * unit[j];
                    f1 *= exp2f(b[j + 1]) * unit[j + 1];
                }
                split2(t.x * f0, t.y * f1, &ah[kk][e], &al[kk][e]);
            }
        }
        const int cols = which ? dp : vp, st = which ? ks : vst;
        const unsigned from = which ? k_s : v_s;
        for (int c0 = side * 16; c0 < cols; c0 += 32) {
            float acc[2][4];
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[n][e] = 0.f;
#pragma unroll
            for (int kk = 0; kk < 4; kk++) {
                if (kk > m) break;
                unsigned x[4];
                ldmatrix_x4_trans(x, from + (kk * 16 + (lane & 15)) * st + c0 * 2 + (lane >> 4) * 16);
                mma_bf16(acc[0], ah[kk][0], ah[kk][1], ah[kk][2], ah[kk][3], x[0], x[1]);
                mma_bf16(acc[1], ah[kk][0], ah[kk][1], ah[kk][2], ah[kk][3], x[2], x[3]);
                mma_bf16(acc[0], al[kk][0], al[kk][1], al[kk][2], al[kk][3], x[0], x[1]);
                mma_bf16(acc[1], al[kk][0], al[kk][1], al[kk][2], al[kk][3], x[2], x[3]);
            }
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int i = r0 + g8 + 8 * r, c = c0 + n * 8 + t4 * 2;
                    if (which) {  // (rows without a token are zero)
                        unsigned hi, lo;
                        split2(acc[n][2 * r], acc[n][2 * r + 1], &hi, &lo);
                        *reinterpret_cast<unsigned*>(tile + i * ks + c * 2) = hi;
                        *reinterpret_cast<unsigned*>(tile + (kC + i) * ks + c * 2) = lo;
                    } else if (i < n_tok && c < p.vdim) {
                        *reinterpret_cast<float2*>(uv + (long long)i * p.heads * p.vdim + c) = make_float2(acc[n][2 * r], acc[n][2 * r + 1]);
                    }
                }
        }
    }
}

// Shared memory of the scan for 16 · NS columns: two stages of W's high and low part, k, then the state and the scaled u, high and low.
__host__ __device__ constexpr int slice_stride(int ns) { return ns * 32 + 16; }  // bytes per row
struct ScanSmem {
    int rows, k, state, u, total;
};
__host__ __device__ constexpr ScanSmem scan_smem(int dim, int ns) {
    const int rows = kC * row_stride(dim), state = 5 * rows, u = state + 2 * padded(dim) * slice_stride(ns);
    return {rows, 4 * rows, state, u, u + 2 * kC * slice_stride(ns)};
}
__device__ __forceinline__ void bulk_load(unsigned dst, const void* src, int bytes, unsigned bar) {
    mbar_expect_tx(bar, (unsigned)bytes);
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
// Grid: (slices of 16 · NS columns, heads, sequences); eight warps. MT: 16-row tiles of the state per warp.
template <int MT, int NS> __global__ void __launch_bounds__(256) delta_scan(const DeltaP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float factor[kC];
    __shared__ __align__(8) unsigned long long bars[3];  // W's stages, k
    constexpr int kSlice = 16 * NS, kStride = slice_stride(NS);
    pdl_trigger();
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, v0 = blockIdx.x * kSlice;
    const int dp = padded(p.dim), st = row_stride(p.dim), n_cols = min(kSlice, p.vdim - v0), n = (sq.len + kC - 1) / kC;
    const ScanSmem L = scan_smem(p.dim, NS);
    const int chunk0 = chunks_before(p.seqs, blockIdx.z);
    float* state = p.state + ((long long)slot_of(p, sq.slot) * p.heads + h) * p.dim * p.vdim + v0;
    if (tid == 0) {
        for (int i = 0; i < 3; i++) mbar_init(smem_u32(bars + i), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    if (sq.len == 1) return;
    const unsigned sm0 = smem_u32(smem), ks = sm0 + L.k, sh = sm0 + L.state, sl = sh + dp * kStride, uh = sm0 + L.u, ul = uh + kC * kStride;
    const unsigned char* tiles = p.tiles + ((long long)chunk0 * p.heads + h) * 3 * L.rows;
    const long long next = (long long)p.heads * 3 * L.rows;
    auto tokens = [&](int c) { return min(kC, sq.len - c * kC); };
    auto load_w = [&](int c) {
        if (tid == 0 && c < n) bulk_load(sm0 + (c & 1) * 2 * L.rows, tiles + c * next, 2 * L.rows, smem_u32(bars + (c & 1)));
    };
    auto load_k = [&](int c) {
        if (tid == 0 && c < n) bulk_load(ks, tiles + c * next + 2 * L.rows, L.rows, smem_u32(bars + 2));
    };
    // u of this warp: tokens m · 16 …, columns side · 8 NS …; U and the factors come one chunk ahead
    const int m = warp & 3, side = warp >> 2, col = side * 8 * NS + t4 * 2;
    float2 U[NS][2];
    float f_mine = 0.f, f_whole = 0.f;
    auto ask = [&](int c) {
        if (c >= n) return;
        const long long row0 = sq.start + (long long)c * kC;
        const int n_tok = tokens(c);
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = m * 16 + g8 + 8 * r;
            const float* from = p.uv + ((row0 + i) * p.heads + h) * p.vdim + v0 + col;
#pragma unroll
            for (int x = 0; x < NS; x++) U[x][r] = i < n_tok && col + x * 8 < n_cols ? *reinterpret_cast<const float2*>(from + x * 8) : make_float2(0.f, 0.f);
        }
        f_whole = p.whole[(long long)(chunk0 + c) * p.heads + h];
        if (tid < kC) f_mine = tid < n_tok ? p.factor[(row0 + tid) * p.heads + h] : 0.f;
    };
    load_w(0);
    load_k(0);
    ask(0);
    float S[MT][2 * NS][4];  // rows (warp + 8 i) · 16 + g8 (+ 8), columns x · 8 + 2 t4 (+ 1)
    auto each = [&](auto&& f) {
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int x = 0; x < 2 * NS; x++)
#pragma unroll
                for (int r = 0; r < 2; r++) f(S[i][x][2 * r], S[i][x][2 * r + 1], (warp + 8 * i) * 16 + g8 + 8 * r, x * 8 + t4 * 2);
    };
    each([&](float& x, float& y, int d, int c) {
        const float2 s = sq.past > 0 && d < p.dim && c < n_cols ? *reinterpret_cast<const float2*>(state + (long long)d * p.vdim + c) : make_float2(0.f, 0.f);
        x = s.x;
        y = s.y;
    });
    const long long plane = (long long)p.chunks * p.heads * p.dim * p.vdim, u_plane = p.rows * p.heads * (long long)p.vdim;
    bool ok = true;
    for (int c = 0; c < n; c++) {
        const long long row0 = sq.start + (long long)c * kC;
        const int n_tok = tokens(c);
        load_w(c + 1);  // (the stage was read before the last barriers)
        const bool carried = sq.past > 0 || c > 0;
        if (carried)
            each([&](float& x, float& y, int d, int cc) {
                unsigned hi, lo;
                split2(x, y, &hi, &lo);
                if (d >= dp) return;
                *reinterpret_cast<unsigned*>(smem + L.state + d * kStride + cc * 2) = hi;
                *reinterpret_cast<unsigned*>(smem + L.state + (dp + d) * kStride + cc * 2) = lo;
            });
        if (tid < kC) factor[tid] = f_mine;
        const float whole = f_whole;
        float2 u[NS][2];
#pragma unroll
        for (int x = 0; x < NS; x++)
#pragma unroll
            for (int r = 0; r < 2; r++) u[x][r] = U[x][r];
        if (ok) ok = mbar_wait(smem_u32(bars + (c & 1)), c >> 1 & 1);
        __syncthreads();
        ask(c + 1);
        if (carried) {
            bf16* to = p.chunk + ((long long)(chunk0 + c) * p.heads + h) * p.dim * p.vdim + v0;
            for (int i = tid; i < 4 * NS * p.dim; i += 256) {  // 16 bytes: eight columns of a row, high or low part
                const int d = i / (4 * NS), cc = i % (2 * NS) * 8, low = i / (2 * NS) & 1;
                if (cc < n_cols) *reinterpret_cast<uint4*>(to + low * plane + (long long)d * p.vdim + cc) = *reinterpret_cast<const uint4*>(smem + L.state + (low * dp + d) * kStride + cc * 2);
            }
        }
        float acc[NS][3][4];
#pragma unroll
        for (int x = 0; x < NS; x++)
#pragma unroll
            for (int y = 0; y < 3; y++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[x][y][e] = 0.f;
        if (carried) {
            const unsigned wh = sm0 + (c & 1) * 2 * L.rows + (m * 16 + (lane & 15)) * st + (lane >> 4) * 16, wl = wh + L.rows;
            const unsigned from = (lane < 16 ? sh : sl) + (lane & 15) * kStride + side * 16 * NS;  // high parts of the state's 16 rows, then the low ones
#pragma unroll 4
            for (int kk = 0; kk < dp / 16; kk++) {
                unsigned ah[4], al[4], s[4];
                ldmatrix_x4(ah, wh + kk * 32);
                ldmatrix_x4(al, wl + kk * 32);
#pragma unroll
                for (int x = 0; x < NS; x++) {
                    ldmatrix_x4_trans(s, from + kk * 16 * kStride + x * 16);
                    mma_bf16(acc[x][0], ah[0], ah[1], ah[2], ah[3], s[0], s[1]);
                    mma_bf16(acc[x][1], ah[0], ah[1], ah[2], ah[3], s[2], s[3]);
                    mma_bf16(acc[x][2], al[0], al[1], al[2], al[3], s[0], s[1]);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = m * 16 + g8 + 8 * r;
            const float f = factor[i];
            bf16* to = p.us + ((row0 + i) * p.heads + h) * p.vdim + v0 + col;
#pragma unroll
            for (int w = 0; w < NS; w++) {
                const float x = u[w][r].x - (acc[w][0][2 * r] + (acc[w][1][2 * r] + acc[w][2][2 * r]));
                const float y = u[w][r].y - (acc[w][0][2 * r + 1] + (acc[w][1][2 * r + 1] + acc[w][2][2 * r + 1]));
                unsigned hi, lo;
                split2(x * f, y * f, &hi, &lo);
                *reinterpret_cast<unsigned*>(smem + L.u + i * kStride + (col + w * 8) * 2) = hi;
                *reinterpret_cast<unsigned*>(smem + L.u + (kC + i) * kStride + (col + w * 8) * 2) = lo;
                if (i < n_tok && col + w * 8 < n_cols) {
                    split2(x, y, &hi, &lo);
                    *reinterpret_cast<unsigned*>(to + w * 8) = hi;
                    *reinterpret_cast<unsigned*>(to + w * 8 + u_plane) = lo;
                }
            }
        }
        if (ok) ok = mbar_wait(smem_u32(bars + 2), c & 1);
        __syncthreads();
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int d0 = (warp + 8 * i) * 16;
            if (d0 >= dp) break;
#pragma unroll
            for (int x = 0; x < 2 * NS; x++)
#pragma unroll
                for (int e = 0; e < 4; e++) S[i][x][e] *= whole;
#pragma unroll
            for (int kk = 0; kk < kC / 16; kk++) {
                unsigned a[4], x[4];
                ldmatrix_x4_trans(a, ks + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * st + d0 * 2 + ((lane >> 3) & 1) * 16);
#pragma unroll
                for (int w = 0; w < NS; w++) {
                    const unsigned at = (kk * 16 + (lane & 15)) * kStride + (lane >> 4) * 16 + w * 32;
                    ldmatrix_x4_trans(x, uh + at);
                    mma_bf16(S[i][2 * w], a[0], a[1], a[2], a[3], x[0], x[1]);
                    mma_bf16(S[i][2 * w + 1], a[0], a[1], a[2], a[3], x[2], x[3]);
                    ldmatrix_x4_trans(x, ul + at);
                    mma_bf16(S[i][2 * w], a[0], a[1], a[2], a[3], x[0], x[1]);
                    mma_bf16(S[i][2 * w + 1], a[0], a[1], a[2], a[3], x[2], x[3]);
                }
            }
        }
        __syncthreads();  // k, u and the factors are free again
        load_k(c + 1);
    }
    if (!ok && lane == 0) report(p.err, ERR_WAIT_TIMEOUT, p.node, blockIdx.x, warp);
    each([&](float& x, float& y, int d, int c) {
        if (d < p.dim && c < n_cols) *reinterpret_cast<float2*>(state + (long long)d * p.vdim + c) = make_float2(x, y);
    });
}

// Grid: (chunks, heads, 64-column slices); eight warps of 16 tokens and half of the columns.
__global__ void __launch_bounds__(256) delta_out(const DeltaP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // q, k [kC][row_stride], u high, low [kC][kColStride], state high, low [dim][kColStride]
    __shared__ float b[kC], unit[kC], q_unit[kC];
    pdl_enter();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.x, kC, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, h = blockIdx.y, g = h / (p.heads / p.kv_heads), v0 = blockIdx.z * kCols;
    const int n_tok = min(kC, sq.len - first), stride = row_stride(p.dim), dp = padded(p.dim), n_cols = min(kCols, p.vdim - v0);
    const long long row0 = sq.start + first;
    const bf16* x = (const bf16*)p.u + row0 * p.channels + (long long)g * p.dim;
    const unsigned qs = smem_u32(smem), ks = qs + kC * stride, uh = ks + kC * stride, ul = uh + kC * kColStride, sh = ul + kC * kColStride, sl = sh + dp * kColStride;
    load_rows(qs, stride, x, p.channels, n_tok, p.dim, dp, tid, 256);
    load_rows(ks, stride, x + (long long)p.kv_heads * p.dim, p.channels, n_tok, p.dim, dp, tid, 256);
    cp_async_commit();
    const bf16* u = p.us + (row0 * p.heads + h) * p.vdim + v0;
    load_rows(uh, kColStride, u, (long long)p.heads * p.vdim, n_tok, n_cols, kCols, tid, 256);
    load_rows(ul, kColStride, u + p.rows * p.heads * (long long)p.vdim, (long long)p.heads * p.vdim, n_tok, n_cols, kCols, tid, 256);
    if (tid < kC) {
        b[tid] = tid < n_tok ? p.sums[(row0 + tid) * p.heads + h] : 0.f;
        unit[tid] = tid < n_tok ? p.unit[(row0 + tid) * p.heads + h] : 0.f;
    }
    const bool carried = sq.past > 0 || first > 0;  // a state enters the chunk
    if (carried) {
        const bf16* src = p.chunk + ((long long)blockIdx.x * p.heads + h) * p.dim * p.vdim + v0;
        const long long plane = (long long)p.chunks * p.heads * p.dim * p.vdim;
        for (int i = tid; i < dp * (kCols / 8) * 2; i += 256) {
            const int c = i % (kCols / 8) * 8, d = i / (kCols / 8) % dp, low = i >= dp * (kCols / 8);
            const bool live = d < p.dim && c < n_cols;
            cp_async16((low ? sl : sh) + d * kColStride + c * 2, live ? src + low * plane + (long long)d * p.vdim + c : src, live);
        }
    }
    cp_async_commit();
    cp_async_wait<1>();  // queries and keys
    __syncthreads();
    unit_factors(smem, stride, p.dim, p.eps, p.q_scale, q_unit, warp, 8);
    cp_async_wait<0>();
    __syncthreads();
    constexpr int kHalf = kCols / 2;
    const int r0 = (warp & 3) * 16, half = (warp >> 2) * kHalf;
    if (r0 >= n_tok || half >= n_cols) return;
    float s[kC / 8][4], o[kHalf / 8][4];
#pragma unroll
    for (int n = 0; n < kC / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) s[n][e] = 0.f;
#pragma unroll
    for (int n = 0; n < kHalf / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    for (int kk = 0; kk < dp / 16; kk++) {
        unsigned a[4];
        ldmatrix_x4(a, qs + (r0 + (lane & 15)) * stride + kk * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int n = 0; n < kC / 8; n += 2) {
            if (n * 8 > r0 + 15) continue;  // keys behind every row of the warp
            unsigned c[4];
            ldmatrix_x4(c, ks + (n * 8 + (lane & 7) + (lane >> 4) * 8) * stride + kk * 32 + ((lane >> 3) & 1) * 16);
            mma_bf16(s[n], a[0], a[1], a[2], a[3], c[0], c[1]);
            mma_bf16(s[n + 1], a[0], a[1], a[2], a[3], c[2], c[3]);
        }
        if (!carried) continue;
#pragma unroll
        for (int n = 0; n < kHalf / 8; n += 2) {
            const unsigned at = (kk * 16 + (lane & 15)) * kColStride + half * 2 + n * 16 + (lane >> 4) * 16;
            unsigned c[4];
            ldmatrix_x4_trans(c, sh + at);
            mma_bf16(o[n], a[0], a[1], a[2], a[3], c[0], c[1]);
            mma_bf16(o[n + 1], a[0], a[1], a[2], a[3], c[2], c[3]);
            ldmatrix_x4_trans(c, sl + at);
            mma_bf16(o[n], a[0], a[1], a[2], a[3], c[0], c[1]);
            mma_bf16(o[n + 1], a[0], a[1], a[2], a[3], c[2], c[3]);
        }
    }
    const int i0 = r0 + g8;  // this lane's rows: i0, i0 + 8
    const float qf[2] = {q_unit[i0], q_unit[i0 + 8]}, bi[2] = {b[i0], b[i0 + 8]}, in[2] = {qf[0] * exp2f(bi[0]), qf[1] * exp2f(bi[1])};
#pragma unroll
    for (int n = 0; n < kHalf / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] *= in[e >> 1];
#pragma unroll
    for (int n = 0; n < kC / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = e >> 1, j = n * 8 + t4 * 2 + (e & 1);
            s[n][e] = j <= i0 + 8 * r ? s[n][e] * qf[r] * unit[j] * exp2f(bi[r] - b[j]) : 0.f;
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
        for (int n = 0; n < kHalf / 8; n += 2) {
            const unsigned at = (kk * 16 + (lane & 15)) * kColStride + half * 2 + n * 16 + (lane >> 4) * 16;
            unsigned c[4];
            ldmatrix_x4_trans(c, uh + at);
            mma_bf16(o[n], ah[0], ah[1], ah[2], ah[3], c[0], c[1]);
            mma_bf16(o[n + 1], ah[0], ah[1], ah[2], ah[3], c[2], c[3]);
            mma_bf16(o[n], al[0], al[1], al[2], al[3], c[0], c[1]);
            mma_bf16(o[n + 1], al[0], al[1], al[2], al[3], c[2], c[3]);
            ldmatrix_x4_trans(c, ul + at);
            mma_bf16(o[n], ah[0], ah[1], ah[2], ah[3], c[0], c[1]);
            mma_bf16(o[n + 1], ah[0], ah[1], ah[2], ah[3], c[2], c[3]);
        }
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int i = i0 + 8 * r;
        if (i >= n_tok) continue;
        float* out = p.out + ((row0 + i) * p.heads + h) * p.vdim + v0;
#pragma unroll
        for (int n = 0; n < kHalf / 8; n++) {
            const int c = half + n * 8 + t4 * 2;
            if (c < n_cols) *reinterpret_cast<float2*>(out + c) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
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
    cd.keep = rows == n_seqs;
    emit_short_conv(em, cd, proj, conv_w, nullptr, conv_state, seqs, u);
    const bool chunks = bf && rows > n_seqs && d.dim % 8 == 0 && d.vdim % 8 == 0 && d.dim <= 256 && d.vdim <= 512;
    const int64_t tiles = std::min(rows, rows / kC + n_seqs);
    auto room = [&](int64_t bytes) { return chunks ? em.scratch((size_t)bytes) : Buf{kSlotNull, 0}; };
    const Buf sums = room(rows * d.heads * 4), unit = room(rows * d.heads * 4), uv = room(rows * d.heads * d.vdim * 4);
    const Buf factor = room(rows * d.heads * 4), whole = room(tiles * d.heads * 4), blocks = room(tiles * d.heads * 3 * kC * row_stride((int)d.dim));
    const Buf us = room(rows * d.heads * d.vdim * 4), chunk = room(tiles * d.heads * d.dim * d.vdim * 4);
    p.chunks = (int)tiles;
    p.singles_only = chunks;
    auto launch = [&](DeltaKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.u, u.buf}, {&p.decay, decay.buf}, {&p.dt_b, dt_bias.buf}, {&p.ring, conv_state.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf},
                   {&p.out, out.buf}, {&p.sums, sums}, {&p.unit, unit}, {&p.factor, factor}, {&p.whole, whole}, {&p.tiles, blocks}, {&p.uv, uv}, {&p.us, us}, {&p.chunk, chunk}, {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    if (!cd.keep) launch(bf ? delta_keep<bf16> : delta_keep<float>, dim3((unsigned)((p.channels + 255) / 256), (unsigned)d.taps, (unsigned)n_seqs), 256, 0, "delta_keep");
    if (chunks) {
        const unsigned stride = (unsigned)row_stride((int)d.dim);
        const unsigned chunk_smem = kC * kTStride * 4 + kC * (stride + (unsigned)row_stride((int)d.vdim));
        const unsigned out_smem = 2 * kC * stride + 2 * kC * kColStride + 2 * (unsigned)padded((int)d.dim) * kColStride;
        // 16 columns per CTA where that leaves a multiprocessor to each
        const int ns = (d.vdim + 15) / 16 * d.heads * n_seqs <= sm_count() || scan_smem((int)d.dim, 2).total > 220 * 1024 ? 1 : 2;
        const DeltaKernel scan = ns == 1 ? (d.dim <= 128 ? delta_scan<1, 1> : delta_scan<2, 1>) : d.dim <= 128 ? delta_scan<1, 2> : delta_scan<2, 2>;
        for (const void* f : {(const void*)delta_chunk, (const void*)scan, (const void*)delta_out}) ensure_max_dynamic_smem(f, 220 * 1024);
        launch(delta_chunk, dim3((unsigned)tiles, (unsigned)d.heads), 256, chunk_smem, "delta_chunk");
        launch(scan, dim3((unsigned)((d.vdim + 16 * ns - 1) / (16 * ns)), (unsigned)d.heads, (unsigned)n_seqs), 256, (unsigned)scan_smem((int)d.dim, ns).total, "delta_scan");
        launch(delta_out, dim3((unsigned)tiles, (unsigned)d.heads, (unsigned)((d.vdim + kCols - 1) / kCols)), 256, out_smem, "delta_out");
        if (n_seqs == 1) return;
    }
    const DeltaKernel k = bf ? (v4 ? step_kernel<bf16, true>(d.dim) : step_kernel<bf16, false>(d.dim)) : (v4 ? step_kernel<float, true>(d.dim) : step_kernel<float, false>(d.dim));
    launch(k, dim3((unsigned)((d.vdim + 31) / 32), (unsigned)d.heads, (unsigned)n_seqs), kStepThreads, 0, "delta_step");
}

}  // namespace oxk
