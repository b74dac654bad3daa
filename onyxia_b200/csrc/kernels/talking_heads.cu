// Causal attention over paged pools whose heads' softmax weights are mixed before they meet the values ("Talking-Heads Attention", Shazeer, Lan,
// Cheng, Ding and Hou, with the mixing behind the softmax):
//
//   w_g(i, j) = softmax_j(temp_g · scale · q_g,i · k_j),   out_h,i = Σ_j (Σ_g talk[h, g] w_g(i, j)) v_j      (v of head h's own value head)
//
// A mixed weight needs the finished softmax of all heads, so the softmax's sums come first:
//
//   paged_kv_prepare   (paged_kv_attention.cu) rotated queries; the new keys and values go to the pools
//   talk_lse           (paged_kv_attention.cu, the prefill kernel without values) log of the sums of sequences with several new tokens
//   talk_prefill       their results, 16 tokens and up to 16 heads per CTA: a warp keeps a head's queries in registers and forms its weights for tiles
//                      of keys. Weights (as two bf16, 16 bits of them) meet in shared memory as [head][token, key], with more than 16 heads in that
//                      of both CTAs of a cluster; the mix is a matrix product over heads, and its bf16 result the operand of the one over values.
//                      Long ranges of keys are cut between CTAs: finished weights need no rescaling, talk_merge adds the parts
//   talk_prefill_any   the same with all heads' scores in one CTA and keys straight from memory: sizes that the other does not take
//   talk_scores        sequences with one new token: scores and sums of a range of keys, which stream through registers; rotation and append
//   talk_values        weights of a range of keys, their mix, and the values, which stream through registers; the last CTA adds the ranges
//   talk_simt_lse, talk_simt   f32, and shapes the tensor-core kernels do not take
//
// Decode reads past · kv_heads · (dim + vdim) · 2 bytes per sequence (and 8 per head and key for scores); prefill
// 2 · S · T · heads · (dim + vdim + heads) FLOPs.
#include <cooperative_groups.h>

#include "chunk_util.cuh"
#include "paged_kv.cuh"

namespace oxk {

namespace cg = cooperative_groups;

namespace {

struct TalkP {
    KvP kv;
    const float* talk;  // [heads, heads]
    float* scores;      // decode [R, heads, span]: base-2 scores
    float* stats;       // decode [R, splits, heads, 2]: maximum, sum
    float* parts;       // decode [R, slices, value splits, slice_heads · vdim]; prefill [splits, rows, heads · vdim]
    int span, slices, slice_heads, value_splits, pre_splits;
};

// ───────────────────────────── any shape ────────────────────────────────
constexpr int kSimtThreads = 256, kSimtKeys = 32;
template <typename T> __device__ __forceinline__ float dot_key(const KvP& p, const float* q, int seq, int g, int j) {
    const T* k = (const T*)p.keys + key_row(p, page_of(p, seq, j), g, j) * p.dim;
    float d = 0.f;
    for (int i = 0; i < p.dim; i++) d = fmaf(q[i], to_f(k[i]), d);
    return d;
}
// One CTA per (row, head): the natural logarithm of the softmax's sum.
template <typename T> __global__ void __launch_bounds__(kSimtThreads) talk_simt_lse(const TalkP tp) {
    const KvP& p = tp.kv;
    extern __shared__ float q[];
    __shared__ float red[32];
    pdl_enter();
    const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, s = find_seq(p.seqs, p.n_seqs, row);
    const SeqRow sq = load_seq(p.seqs, s);
    if (row >= sq.start + sq.len) return;
    const int pos = sq.past + row - sq.start, g = h / (p.heads / p.kv_heads);
    for (int i = tid; i < p.dim; i += kSimtThreads) q[i] = to_f(((const T*)p.q)[((long long)row * p.heads + h) * p.dim + i]);
    __syncthreads();
    const float f = p.scale * temp_of(p, h);
    float m = -INFINITY, l = 0.f;
    for (int j = tid; j <= pos; j += kSimtThreads) {
        const float sc = dot_key<T>(p, q, s, g, j) * f, m2 = fmaxf(m, sc);
        l = l * expf(m - m2) + expf(sc - m2);
        m = m2;
    }
    const float top = block_max(m, red);
    const float sum = block_sum(m == -INFINITY ? 0.f : l * expf(m - top), red);
    if (tid == 0) p.lse[(long long)row * p.heads + h] = top + logf(sum);
}
// One CTA per row, key chunks of 32.
template <typename T> __global__ void __launch_bounds__(kSimtThreads) talk_simt(const TalkP tp) {
    const KvP& p = tp.kv;
    extern __shared__ float sm[];  // q [heads][dim], weights [heads][32], mixed [heads][32], result [heads][vdim]
    pdl_enter();
    const int row = blockIdx.x, tid = threadIdx.x, s = find_seq(p.seqs, p.n_seqs, row), H = p.heads, rep = H / p.kv_heads;
    const SeqRow sq = load_seq(p.seqs, s);
    if (row >= sq.start + sq.len) return;
    const int pos = sq.past + row - sq.start;
    float *q = sm, *w = q + H * p.dim, *mixed = w + H * kSimtKeys, *acc = mixed + H * kSimtKeys;
    for (int i = tid; i < H * p.dim; i += kSimtThreads) q[i] = to_f(((const T*)p.q)[(long long)row * H * p.dim + i]);
    for (int i = tid; i < H * p.vdim; i += kSimtThreads) acc[i] = 0.f;
    const float* lse = p.lse + (long long)row * H;
    __syncthreads();
    for (int j0 = 0; j0 <= pos; j0 += kSimtKeys) {
        for (int i = tid; i < H * kSimtKeys; i += kSimtThreads) {
            const int h = i / kSimtKeys, j = j0 + i % kSimtKeys;
            w[i] = j <= pos ? expf(dot_key<T>(p, q + h * p.dim, s, h / rep, j) * (p.scale * temp_of(p, h)) - lse[h]) : 0.f;
        }
        __syncthreads();
        for (int i = tid; i < H * kSimtKeys; i += kSimtThreads) {
            const int h = i / kSimtKeys;
            float a = 0.f;
            for (int g = 0; g < H; g++) a = fmaf(tp.talk[h * H + g], w[g * kSimtKeys + i % kSimtKeys], a);
            mixed[i] = a;
        }
        __syncthreads();
        const int live = min(kSimtKeys, pos + 1 - j0);
        for (int i = tid; i < H * p.vdim; i += kSimtThreads) {
            const int h = i / p.vdim;
            float a = acc[i];
            long long pg = 0;
            for (int jj = 0; jj < live; jj++) {
                if (jj == 0 || ((j0 + jj) & ((1 << p.shift) - 1)) == 0) pg = page_of(p, s, j0 + jj);
                a = fmaf(mixed[h * kSimtKeys + jj], to_f(((const T*)p.values)[key_row(p, pg, h / rep, j0 + jj) * p.ldv + i % p.vdim]), a);
            }
            acc[i] = a;
        }
        __syncthreads();
    }
    for (int i = tid; i < H * p.vdim; i += kSimtThreads) ((T*)p.out)[(long long)row * H * p.vdim + i] = from_f<T>(acc[i]);
}

// ───────────────────────────── shared pieces ────────────────────────────
__device__ __forceinline__ uint4 ld16(const bf16* p, bool live) { return live ? *reinterpret_cast<const uint4*>(p) : make_uint4(0, 0, 0, 0); }
// The mixing matrix in bf16, padded with zeros: rows h_lo …, KS · 16 rows and columns, `KS · 32 + 16` bytes per row.
template <int KS> __device__ __forceinline__ void stage_talk(unsigned char* dst, const float* talk, int heads, int h_lo, int tid, int threads) {
    constexpr int n = KS * 16, stride = n * 2 + 16;
    for (int i = tid; i < n * n; i += threads) {
        const int h = h_lo + i / n, g = i % n;
        *reinterpret_cast<bf16*>(dst + i / n * stride + g * 2) = __float2bfloat16_rn(h < heads && g < heads ? talk[h * heads + g] : 0.f);
    }
}
// Sixteen columns of the mix: B fragments of all heads' weights, high and low part; `at` the columns' bytes in head 0's row.
template <int KS> __device__ __forceinline__ void load_weights(unsigned (&b)[KS][2][4], unsigned hi, unsigned lo, int head_bytes, int at) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int k = 0; k < KS; k++) {
        const unsigned off = (unsigned)((k * 16 + (lane & 15)) * head_bytes + at + (lane >> 4) * 16);
        ldmatrix_x4_trans(b[k][0], hi + off);
        ldmatrix_x4_trans(b[k][1], lo + off);
    }
}
// … times 16 rows of the matrix: mixed[0], mixed[1] are the C fragments of eight columns each.
template <int KS> __device__ __forceinline__ void mix(float (&mixed)[2][4], const unsigned (&b)[KS][2][4], unsigned talk, int m_tile) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int e = 0; e < 4; e++) mixed[0][e] = mixed[1][e] = 0.f;
#pragma unroll
    for (int k = 0; k < KS; k++) {
        unsigned a[4];
        ldmatrix_x4(a, talk + (m_tile * 16 + (lane & 15)) * (KS * 32 + 16) + k * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int part = 0; part < 2; part++) {
            mma_bf16(mixed[0], a[0], a[1], a[2], a[3], b[k][part][0], b[k][part][1]);
            mma_bf16(mixed[1], a[0], a[1], a[2], a[3], b[k][part][2], b[k][part][3]);
        }
    }
}

// The same of one step after the other, where the matrix has 16 rows.
template <int KS> __device__ __forceinline__ void mix_columns(float (&mixed)[2][4], unsigned hi, unsigned lo, int head_bytes, int at, unsigned talk) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int e = 0; e < 4; e++) mixed[0][e] = mixed[1][e] = 0.f;
#pragma unroll
    for (int k = 0; k < KS; k++) {
        unsigned a[4], b[4];
        const unsigned off = (unsigned)((k * 16 + (lane & 15)) * head_bytes + at + (lane >> 4) * 16);
        ldmatrix_x4(a, talk + (lane & 15) * (KS * 32 + 16) + k * 32 + (lane >> 4) * 16);
        ldmatrix_x4_trans(b, hi + off);
        mma_bf16(mixed[0], a[0], a[1], a[2], a[3], b[0], b[1]);
        mma_bf16(mixed[1], a[0], a[1], a[2], a[3], b[2], b[3]);
        ldmatrix_x4_trans(b, lo + off);
        mma_bf16(mixed[0], a[0], a[1], a[2], a[3], b[0], b[1]);
        mma_bf16(mixed[1], a[0], a[1], a[2], a[3], b[2], b[3]);
    }
}

// ───────────────────────────── prefill ──────────────────────────────────
constexpr int kTalkSmem = 224 * 1024;
constexpr int kTalkThreads = 512, kTalkWarps = 16, kTalkTokens = 16, kTalkUnits = 2;  // units: (head, 64 value columns) of a warp

// TK keys per tile, KS · 16 ≥ heads
template <int TK, int KS> struct TalkSmem {
    static constexpr int row = (TK + 8) * 2;                         // bytes of a token's weights: conflict-free ldmatrix
    static constexpr int head = kTalkTokens * row + 16;
    static constexpr int talk = 0;
    static constexpr int hi = KS * 16 * (KS * 32 + 16);
    static constexpr int lo = hi + KS * 16 * head;
    static constexpr int values = lo + KS * 16 * head;               // [value heads of the slice][TK][value_row]
};
__host__ __device__ constexpr int value_row(int vdim) { return (vdim + 15) / 16 * 32 + 16; }

// Grid: (tiles of 16 tokens, slices of the result's heads).
template <int TK, int KS> __global__ void __launch_bounds__(kTalkThreads, 1) talk_prefill_any(const __grid_constant__ TalkP tp) {
    extern __shared__ __align__(16) unsigned char smem[];
    using L = TalkSmem<TK, KS>;
    const KvP& p = tp.kv;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    const int H = p.heads, rep = H / p.kv_heads, dim = p.dim, vdim = p.vdim, h_lo = blockIdx.y * tp.slice_heads, n_heads = min(tp.slice_heads, H - h_lo);
    pdl_trigger();
    stage_talk<KS>(smem + L::talk, tp.talk, H, h_lo, tid, kTalkThreads);
    for (int i = tid; i < (L::values - L::hi) / 4; i += kTalkThreads) reinterpret_cast<unsigned*>(smem + L::hi)[i] = 0;  // heads beyond the last
    pdl_wait();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)gridDim.x - 1 - (int)blockIdx.x, kTalkTokens, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int n_tok = min(kTalkTokens, sq.len - first), pos0 = sq.past + first, last = pos0 + n_tok - 1;
    const bf16 *q = (const bf16*)p.q + (long long)(sq.start + first) * H * dim, *keys = (const bf16*)p.keys, *values = (const bf16*)p.values;
    const float* lse = p.lse + (long long)(sq.start + first) * H;
    const unsigned sm0 = smem_u32(smem);
    const int g_lo = h_lo / rep, g_n = (h_lo + n_heads - 1) / rep - g_lo + 1, vrow = value_row(vdim), vcols = (vrow - 16) / 16;
    const int blocks = (vdim + 63) / 64, units = n_heads * blocks;
    const int tok[2] = {min(g8, n_tok - 1), min(g8 + 8, n_tok - 1)};
    float o[kTalkUnits][8][4];
#pragma unroll
    for (int k = 0; k < kTalkUnits; k++)
#pragma unroll
        for (int n = 0; n < 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[k][n][e] = 0.f;
    __syncthreads();
    for (int j0 = 0; j0 <= last; j0 += TK) {
        for (int i = tid; i < g_n * TK * vcols; i += kTalkThreads) {
            const int c = i % vcols, key = i / vcols % TK, g = i / (vcols * TK), j = j0 + key;
            const bool live = j <= last && c * 8 < vdim;
            const bf16* src = live ? values + key_row(p, page_of(p, seq, j), g_lo + g, j) * p.ldv + c * 8 : values;
            cp_async16(sm0 + L::values + (g * TK + key) * vrow + c * 16, src, live);
        }
        cp_async_commit();
        // weights of all heads: a unit is 16 keys of a head
        for (int u = warp; u < H * (TK / 16); u += kTalkWarps) {
            const int h = u / (TK / 16), k0 = u % (TK / 16) * 16, g = h / rep;
            const bf16* key[2];
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const int j = min(j0 + k0 + n * 8 + g8, last);
                key[n] = keys + key_row(p, page_of(p, seq, j), g, j) * dim;
            }
            const bf16 *q0 = q + ((long long)tok[0] * H + h) * dim, *q1 = q + ((long long)tok[1] * H + h) * dim;
            float s[2][4];
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) s[n][e] = 0.f;
#pragma unroll 4
            for (int d = t4 * 8; d < (dim + 31) / 32 * 32; d += 32) {  // (a dot product does not care in which order its dimensions come)
                const bool live = d < dim;
                const uint4 a = ld16(q0 + d, live), b = ld16(q1 + d, live);
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    const uint4 k = ld16(key[n] + d, live);
                    mma_bf16(s[n], a.x, b.x, a.y, b.y, k.x, k.y);
                    mma_bf16(s[n], a.z, b.z, a.w, b.w, k.z, k.w);
                }
            }
            const float f = p.mul2 * temp_of(p, h), less[2] = {lse[tok[0] * H + h], lse[tok[1] * H + h]};
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int i = g8 + 8 * r, c = k0 + n * 8 + t4 * 2, seen = i < n_tok ? pos0 + i - j0 : -1;  // the last key that the token sees
                    unsigned hi, lo;
                    split2(c <= seen ? exp2f(s[n][2 * r] * f - less[r]) : 0.f, c < seen ? exp2f(s[n][2 * r + 1] * f - less[r]) : 0.f, &hi, &lo);
                    const int at = h * L::head + i * L::row + c * 2;
                    *reinterpret_cast<unsigned*>(smem + L::hi + at) = hi;
                    *reinterpret_cast<unsigned*>(smem + L::lo + at) = lo;
                }
        }
        __syncthreads();
        // the mix, 16 columns (of a token) at a time; it takes the place of the weights' high parts
        for (int c = warp; c < kTalkTokens * (TK / 16); c += kTalkWarps) {
            const int at = c / (TK / 16) * L::row + c % (TK / 16) * 32;
            unsigned b[KS][2][4];
            load_weights<KS>(b, sm0 + L::hi, sm0 + L::lo, L::head, at);
            __syncwarp();
#pragma unroll
            for (int m = 0; m < KS; m++) {
                if (m * 16 >= n_heads) break;
                float mixed[2][4];
                mix<KS>(mixed, b, sm0 + L::talk, m);
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int r = 0; r < 2; r++)
                        *reinterpret_cast<unsigned*>(smem + L::hi + (m * 16 + g8 + 8 * r) * L::head + at + n * 16 + t4 * 4) = pack_bf16(mixed[n][2 * r], mixed[n][2 * r + 1]);
            }
        }
        cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kTalkUnits; k++) {
            const int u = warp + k * kTalkWarps;
            if (u >= units) break;
            const int h = u / blocks, block = u % blocks, cols = min(vcols * 8 - block * 64, 64);
            const unsigned ps = sm0 + L::hi + h * L::head, vs = sm0 + L::values + ((h_lo + h) / rep - g_lo) * TK * vrow + block * 128;
#pragma unroll
            for (int kk = 0; kk < TK / 16; kk++) {
                unsigned a[4];
                ldmatrix_x4(a, ps + (lane & 15) * L::row + kk * 32 + (lane >> 4) * 16);
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    if (n * 8 >= cols) break;
                    unsigned b[4];
                    ldmatrix_x4_trans(b, vs + (kk * 16 + (lane & 15)) * vrow + n * 16 + (lane >> 4) * 16);
                    mma_bf16(o[k][n], a[0], a[1], a[2], a[3], b[0], b[1]);
                    mma_bf16(o[k][n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int k = 0; k < kTalkUnits; k++) {
        const int u = warp + k * kTalkWarps;
        if (u >= units) break;
        const int h = h_lo + u / blocks, c0 = u % blocks * 64;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = g8 + 8 * r;
            if (i >= n_tok) continue;
            bf16* out = (bf16*)p.out + ((long long)(sq.start + first + i) * H + h) * vdim;
#pragma unroll
            for (int n = 0; n < 8; n++) {
                const int c = c0 + n * 8 + t4 * 2;
                if (c < vdim) *reinterpret_cast<unsigned*>(out + c) = pack_bf16(o[k][n][2 * r], o[k][n][2 * r + 1]);
            }
        }
    }
}

// False when the phase did not complete within about a second; orders what other CTAs of the cluster did before they arrived.
__device__ __forceinline__ bool mbar_wait_cluster(unsigned bar, unsigned parity) {
    const long long t0 = clock64();
    do {
        unsigned done;
        asm volatile("{\n .reg .pred p;\n mbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}\n" : "=r"(done) : "r"(bar), "r"(parity) : "memory");
        if (done) return true;
    } while (clock64() - t0 < 2000000000LL);
    return false;
}
// CL CTAs of a cluster, each with the scores, keys, values and results of heads / CL heads; QS · 16 ≥ dim; UN units per warp.
template <int TK, int CL> struct StagedSmem {
    static constexpr int row = (TK + 8) * 2, head = kTalkTokens * row + 16;
    static constexpr int talk = 0, hi = 16 * (CL * 32 + 16), lo = hi + CL * 16 * head;
    static constexpr int keys = lo + CL * 16 * head;                 // [key heads of the CTA][TK][value_row(dim)], then the values
};
// FULL: dim and vdim are QS · 16.
template <int TK, int CL, int QS, int UN, bool FULL> __global__ void __launch_bounds__(kTalkThreads, 1) talk_prefill(const __grid_constant__ TalkP tp) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(8) unsigned long long bars[2];  // CL > 1: the other CTA's weights are here; ours may be written there
    using L = StagedSmem<TK, CL>;
    const KvP& p = tp.kv;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    const int H = p.heads, rep = H / p.kv_heads, dim = FULL ? QS * 16 : p.dim, vdim = FULL ? QS * 16 : p.vdim, rank = (int)blockIdx.x % CL, each = tp.slice_heads, h_lo = rank * each, n_heads = min(each, H - h_lo);
    pdl_trigger();
    if (CL > 1 && tid == 0) {
        mbar_init(smem_u32(bars), 1);
        mbar_init(smem_u32(bars + 1), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    for (int i = tid; i < 16 * CL * 16; i += kTalkThreads) {
        const int h = i / (CL * 16), g = i % (CL * 16);
        *reinterpret_cast<bf16*>(smem + L::talk + h * (CL * 32 + 16) + g * 2) = __float2bfloat16_rn(h < n_heads && g < H ? tp.talk[(h_lo + h) * H + g] : 0.f);
    }
    for (int i = tid; i < (L::keys - L::hi) / 4; i += kTalkThreads) reinterpret_cast<unsigned*>(smem + L::hi)[i] = 0;  // heads beyond the last
    pdl_wait();
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, ((int)gridDim.x - 1 - (int)blockIdx.x) / CL, kTalkTokens, &seq, &first)) return;  // (the whole cluster)
    const SeqRow sq = load_seq(p.seqs, seq);
    const int n_tok = min(kTalkTokens, sq.len - first), pos0 = sq.past + first, last = pos0 + n_tok - 1;
    const long long token0 = sq.start + first;
    const unsigned sm0 = smem_u32(smem);
    const int g_lo = h_lo / rep, g_n = (h_lo + n_heads - 1) / rep - g_lo + 1, krow = value_row(dim), vrow = value_row(vdim), vs0 = L::keys + g_n * TK * krow;
    const int tiles = last / TK + 1, t0 = (int)((long long)tiles * blockIdx.y / tp.pre_splits), t1 = (int)((long long)tiles * (blockIdx.y + 1) / tp.pre_splits);

    // A tile of keys or values: a row per power of two of lanes. The page of a tile that lies in one is looked up a tile ahead.
    const bool whole = (1 << p.shift) >= TK;
    auto page_at = [&](int t) { return whole && t < t1 ? (int)page_of(p, seq, t * TK) : 0; };
    auto load = [&](const bf16* pool, const int width, int t, int at, const int stride, int page) {
        if (t < t1) {
            const int chunks = (stride - 16) / 16, shift = chunks <= 2 ? 1 : chunks <= 4 ? 2 : chunks <= 8 ? 3 : chunks <= 16 ? 4 : 5;
            const int c = lane & ((1 << shift) - 1), per = kTalkThreads >> shift, r0 = tid >> shift, j0 = t * TK, key0 = r0 & (TK - 1);
            const bool cut = j0 + TK - 1 > last || (!FULL && c * 8 >= width);
            if (c < chunks) {
                int g = r0 / TK;
                const int step = per > TK ? per / TK : 1;
                const long long pitch = ((long long)step << p.shift) * width;
                const bf16* head = pool + key_row(p, page, g_lo + g, j0) * width + c * 8;
                unsigned to = sm0 + at + g * TK * stride + c * 16;
                for (; g < g_n; g += step, head += pitch, to += step * TK * stride)
#pragma unroll 2
                    for (int key = key0; key < TK; key += per) {
                        const int j = j0 + key;
                        if (whole && !cut) {
                            cp_async16(to + key * stride, head + key * width);
                            continue;
                        }
                        const bool live = j <= last && c * 8 < width;
                        const bf16* from = whole ? head + key * width : live ? pool + key_row(p, page_of(p, seq, j), g_lo + g, j) * width + c * 8 : pool;
                        cp_async16(to + key * stride, live ? from : pool, live);
                    }
            }
        }
        cp_async_commit();
    };
    int page = page_at(t0), page_next = page_at(t0 + 1);  // of the tile in work and of the one behind it
    auto load_keys = [&](int t, int pg) { load((const bf16*)p.keys, dim, t, L::keys, krow, pg); };
    auto load_values = [&](int t, int pg) { load((const bf16*)p.values, vdim, t, vs0, vrow, pg); };
    load_keys(t0, page);
    load_values(t0, page);

    // this warp's head and share of a tile's keys
    int pow = 1;
    while (pow < n_heads) pow *= 2;
    const int mine = warp % pow, share = warp / pow, shares = kTalkWarps / pow, h = h_lo + min(mine, n_heads - 1);
    const bool scores = mine < n_heads;
    const int tok[2] = {min(g8, n_tok - 1), min(g8 + 8, n_tok - 1)};
    unsigned qa[QS][4];
#pragma unroll
    for (int kk = 0; kk < QS; kk++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int d = kk * 16 + t4 * 2 + (e >> 1) * 8;
            qa[kk][e] = d < dim ? *reinterpret_cast<const unsigned*>((const bf16*)p.q + ((token0 + tok[e & 1]) * H + h) * dim + d) : 0u;
        }
    const float f = p.mul2 * temp_of(p, h), less[2] = {p.lse[(token0 + tok[0]) * H + h], p.lse[(token0 + tok[1]) * H + h]};
    const unsigned ks = sm0 + L::keys + (h / rep - g_lo) * TK * krow + ((lane & 7) + (lane >> 4) * 8) * krow + ((lane >> 3) & 1) * 16;
    unsigned char* dst = smem + L::hi + h * L::head + g8 * L::row + t4 * 4;  // this head's weights
    const int blocks = (vdim + 63) / 64, units = n_heads * blocks;
    float o[UN][8][4];
#pragma unroll
    for (int k = 0; k < UN; k++)
#pragma unroll
        for (int n = 0; n < 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[k][n][e] = 0.f;
    // The other CTA's addresses, and what goes there: this CTA's heads, high and low parts.
    const int mixed_at = L::hi + (CL > 1 && rank == 0 ? each * L::head : 0), own = n_heads * L::head, theirs = (H - n_heads) * L::head;
    unsigned there = 0, there_bars = 0;
    if constexpr (CL > 1) {
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(there) : "r"(sm0), "r"(rank ^ 1));
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(there_bars) : "r"(smem_u32(bars)), "r"(rank ^ 1));
    }
    bool ok = true;
    cp_async_wait<1>();
    if constexpr (CL > 1) cg::this_cluster().sync();
    else __syncthreads();  // keys are here, and every CTA's weights are cleared
    for (int t = t0; t < t1; t++) {
        const int j0 = t * TK;
        const bool edge = j0 + TK - 1 > pos0 || n_tok < kTalkTokens;  // not every token sees every key
        // the other CTA has used what this one sent it, which is therefore read to the end, and its place is free
        if (CL > 1 && t > t0 && ok) ok = mbar_wait_cluster(smem_u32(bars + 1), (t - t0 - 1) & 1);
        if (scores)
            for (int c = share; c < TK / 16; c += shares) {
                float s[2][4];
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[n][e] = 0.f;
#pragma unroll
                for (int kk = 0; kk < QS; kk++) {
                    if (!FULL && kk * 16 >= dim) break;
                    unsigned b[4];
                    ldmatrix_x4(b, ks + c * 16 * krow + kk * 32);
                    mma_bf16(s[0], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b[0], b[1]);
                    mma_bf16(s[1], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b[2], b[3]);
                }
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[n][e] = power2(fmaf(s[n][e], f, -less[e >> 1]));
                if (edge)
#pragma unroll
                    for (int n = 0; n < 2; n++)
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const int i = g8 + 8 * (e >> 1);
                            if (i >= n_tok || j0 + c * 16 + n * 8 + t4 * 2 + (e & 1) > pos0 + i) s[n][e] = 0.f;
                        }
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int r = 0; r < 2; r++) {
                        unsigned hi, lo;
                        split2(s[n][2 * r], s[n][2 * r + 1], &hi, &lo);
                        *reinterpret_cast<unsigned*>(dst + 8 * r * L::row + (c * 16 + n * 8) * 2) = hi;
                        *reinterpret_cast<unsigned*>(dst + 8 * r * L::row + (c * 16 + n * 8) * 2 + (L::lo - L::hi)) = lo;
                    }
            }
        if constexpr (CL > 1) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // the weights are read by a bulk copy
        __syncthreads();
        if constexpr (CL > 1) {
            if (tid == 0 && ok) {
                mbar_expect_tx(smem_u32(bars), (unsigned)(2 * theirs));
#pragma unroll
                for (int part = 0; part < 2; part++) {
                    const unsigned at = (part ? L::lo : L::hi) + h_lo * L::head;
                    asm volatile("cp.async.bulk.shared::cluster.shared::cta.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(there + at), "r"(sm0 + at), "r"(own), "r"(there_bars)
                                 : "memory");
                }
            }
        }
        load_keys(t + 1, page_next);
        if (CL > 1 && ok) ok = mbar_wait(smem_u32(bars), (t - t0) & 1);
        // 16 columns of a token at a time; the mix takes the place of the weights' high parts, in a cluster of those that came from the other CTA
        for (int c = warp; c < TK; c += kTalkWarps) {
            const int at = c / (TK / 16) * L::row + c % (TK / 16) * 32;
            float mixed[2][4];
            mix_columns<CL>(mixed, sm0 + L::hi, sm0 + L::lo, L::head, at, sm0 + L::talk);
            __syncwarp();
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int r = 0; r < 2; r++)
                    if (CL == 1 || g8 + 8 * r < n_heads)
                        *reinterpret_cast<unsigned*>(smem + mixed_at + (g8 + 8 * r) * L::head + at + n * 16 + t4 * 4) = pack_bf16(mixed[n][2 * r], mixed[n][2 * r + 1]);
        }
        cp_async_wait<1>();  // this tile's values
        __syncthreads();
#pragma unroll
        for (int k = 0; k < UN; k++) {
            const int u = warp + k * kTalkWarps;
            if (u >= units) break;
            const int hl = u / blocks, block = u % blocks, cols = min((vrow - 16) / 2 - block * 64, 64);
            const unsigned ps = sm0 + mixed_at + hl * L::head + (lane & 15) * L::row + (lane >> 4) * 16;
            const unsigned vs = sm0 + vs0 + ((h_lo + hl) / rep - g_lo) * TK * vrow + block * 128 + (lane & 15) * vrow + (lane >> 4) * 16;
#pragma unroll
            for (int kk = 0; kk < TK / 16; kk++) {
                unsigned a[4];
                ldmatrix_x4(a, ps + kk * 32);
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    if (!FULL && n * 8 >= cols) break;
                    unsigned b[4];
                    ldmatrix_x4_trans(b, vs + kk * 16 * vrow + n * 16);
                    mma_bf16(o[k][n], a[0], a[1], a[2], a[3], b[0], b[1]);
                    mma_bf16(o[k][n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                }
            }
        }
        cp_async_wait<0>();  // the next tile's keys
        __syncthreads();
        if (CL > 1 && tid == 0) asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];" ::"r"(there_bars + 8) : "memory");
        load_values(t + 1, page_next);
        page_next = page_at(t + 2);
    }
    cp_async_wait<0>();
    if constexpr (CL > 1) {
        if (!ok && lane == 0) report(p.err, ERR_WAIT_TIMEOUT, p.node, blockIdx.x, warp);
        cg::this_cluster().sync();  // neither CTA's memory is needed by the other any more
    }
#pragma unroll
    for (int k = 0; k < UN; k++) {
        const int u = warp + k * kTalkWarps;
        if (u >= units) break;
        const int head = h_lo + u / blocks, c0 = u % blocks * 64;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = g8 + 8 * r;
            if (i >= n_tok) continue;
            const long long at = ((token0 + i) * H + head) * vdim;
#pragma unroll
            for (int n = 0; n < 8; n++) {
                const int c = c0 + n * 8 + t4 * 2;
                if (c >= vdim) continue;
                if (tp.pre_splits == 1) *reinterpret_cast<unsigned*>((bf16*)p.out + at + c) = pack_bf16(o[k][n][2 * r], o[k][n][2 * r + 1]);
                else *reinterpret_cast<float2*>(tp.parts + (long long)blockIdx.y * p.rows * H * vdim + at + c) = make_float2(o[k][n][2 * r], o[k][n][2 * r + 1]);
            }
        }
    }
}

// Adds the parts of sequences with several new tokens. Grid: (1024-element pieces of a row, rows).
__global__ void __launch_bounds__(256) talk_merge(const __grid_constant__ TalkP tp) {
    const KvP& p = tp.kv;
    pdl_enter();
    const int row = blockIdx.y, width = p.heads * p.vdim, i = (blockIdx.x * 256 + threadIdx.x) * 4;  // vdim is a multiple of 8
    const SeqRow sq = load_seq(p.seqs, find_seq(p.seqs, p.n_seqs, row));
    if (i >= width || sq.len == 1) return;
    const float* from = tp.parts + (long long)row * width + i;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < tp.pre_splits; k++) {
        const float4 v = *reinterpret_cast<const float4*>(from + (long long)k * p.rows * width);
        s = make_float4(s.x + v.x, s.y + v.y, s.z + v.z, s.w + v.w);
    }
    *reinterpret_cast<uint2*>((bf16*)p.out + (long long)row * width + i) = make_uint2(pack_bf16(s.x, s.y), pack_bf16(s.z, s.w));
}

// ───────────────────────────── decode ───────────────────────────────────
constexpr int kScoreWarps = 4, kScoreThreads = kScoreWarps * 32, kScoreKeys = kScoreWarps * 16;

__host__ __device__ constexpr int query_row(int dim) { return (dim + 63) / 64 * 128 + 64; }  // bytes: conflict-free fragment loads
// Grid: (splits, kv_heads · groups of 8 · NH query heads, sequences). Keys are the rows of the product, straight from memory.
template <int NH> __global__ void __launch_bounds__(kScoreThreads) talk_scores(const __grid_constant__ TalkP tp) {
    extern __shared__ __align__(16) unsigned char smem[];  // queries [8 · NH][stride], cos, sin [half]
    __shared__ float merge[kScoreWarps][8 * NH][2];
    const KvP& p = tp.kv;
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, H = p.heads, rep = H / p.kv_heads, dim = p.dim;
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    constexpr int kRows = 8 * NH;
    const int groups = (rep + kRows - 1) / kRows, g = blockIdx.y / groups, h0 = g * rep + (blockIdx.y % groups) * kRows, n_heads = min(kRows, (g + 1) * rep - h0);
    const int seq = blockIdx.z, pos = sq.past, dp = (dim + 31) / 32 * 32, stride = query_row(dim);
    float *cs = reinterpret_cast<float*>(smem + kRows * stride), *sn = cs + p.half;
    bf16 *keys = (bf16*)p.keys, *values = (bf16*)p.values;
    const int blocks = sq.len == 1 ? pos / kScoreKeys + 1 : 0;
    const int lo = (int)((long long)blocks * blockIdx.x / p.splits) * kScoreKeys, hi = min((int)((long long)blocks * (blockIdx.x + 1) / p.splits) * kScoreKeys, pos + 1);
    angles(p.turns, p.half, pos, cs, sn, tid, kScoreThreads);
    pdl_wait();
    if (sq.len != 1) return;
    __syncthreads();
    const bf16* x = (const bf16*)p.proj + (long long)sq.start * p.ld;
    if (hi == pos + 1 && lo < hi && h0 == g * rep && p.append) {  // the new key and value
        const long long row = key_row(p, page_of(p, seq, pos), g, pos);
        const bf16* k = x + p.k_off + g * dim;
        const float f = head_factor(p, k);
        for (int i = tid; i < dim; i += kScoreThreads) keys[row * dim + i] = __float2bfloat16_rn(rotated(p.half, p.interleaved, k, cs, sn, i) * f);
        for (int i = tid; i < p.vdim; i += kScoreThreads) values[row * p.ldv + i] = x[p.v_off + g * p.vdim + i];
    }
    for (int r = warp; r < kRows; r += kScoreWarps) {
        const bool live = r < n_heads;
        const bf16* q = x + p.q_off + (long long)(live ? h0 + r : h0) * dim;
        const float f = head_factor(p, q);
        for (int i = lane; i < dp; i += 32)
            *reinterpret_cast<bf16*>(smem + r * stride + i * 2) = __float2bfloat16_rn(live && i < dim ? rotated(p.half, p.interleaved, q, cs, sn, i) * f : 0.f);
    }
    __syncthreads();
    float m[NH][2], l[NH][2], mul2[NH][2];
#pragma unroll
    for (int n = 0; n < NH; n++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            m[n][e] = kNoScore;
            l[n][e] = 0.f;
            mul2[n][e] = p.mul2 * temp_of(p, h0 + min(n * 8 + t4 * 2 + e, n_heads - 1));
        }
    float* scores = tp.scores + ((long long)seq * H + h0) * tp.span;
    // a key head with more query heads than a CTA takes: the other CTAs take the new key from the projection
    const bool fresh = p.append && h0 != g * rep;
    const float fresh_factor = fresh ? head_factor(p, x + p.k_off + g * dim) : 0.f;
    for (int j0 = lo + warp * 16; j0 < hi; j0 += kScoreKeys) {
        const bf16* key[2];
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int j = min(j0 + g8 + 8 * r, pos);
            key[r] = keys + key_row(p, page_of(p, seq, j), g, j) * dim;
        }
        float s[NH][4];
#pragma unroll
        for (int n = 0; n < NH; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[n][e] = 0.f;
#pragma unroll 4
        for (int d = t4 * 8; d < dp; d += 32) {
            const uint4 a = ld16(key[0] + d, d < dim), b = ld16(key[1] + d, d < dim);
#pragma unroll
            for (int n = 0; n < NH; n++) {
                const uint4 k = *reinterpret_cast<const uint4*>(smem + (n * 8 + g8) * stride + d * 2);
                mma_bf16(s[n], a.x, b.x, a.y, b.y, k.x, k.y);
                mma_bf16(s[n], a.z, b.z, a.w, b.w, k.z, k.w);
            }
        }
#pragma unroll
        for (int n = 0; n < NH; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int j = j0 + g8 + 8 * (e >> 1), h = n * 8 + t4 * 2 + (e & 1);
                float v = s[n][e] * mul2[n][e & 1];
                if (fresh && j == pos) {
                    const bf16* k = x + p.k_off + g * dim;
                    const bf16* q = reinterpret_cast<const bf16*>(smem + h * stride);
                    float d = 0.f;
                    for (int i = 0; i < dim; i++) d = fmaf(to_f(q[i]), to_f(__float2bfloat16_rn(rotated(p.half, p.interleaved, k, cs, sn, i) * fresh_factor)), d);
                    v = d * mul2[n][e & 1];
                }
                if (j >= hi || h >= n_heads) continue;
                scores[(long long)h * tp.span + j] = v;
                const float top = fmaxf(m[n][e & 1], v);
                l[n][e & 1] = fmaf(l[n][e & 1], exp2f(m[n][e & 1] - top), exp2f(v - top));
                m[n][e & 1] = top;
            }
    }
#pragma unroll
    for (int n = 0; n < NH; n++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
#pragma unroll
            for (int d = 4; d < 32; d <<= 1) {
                const float om = __shfl_xor_sync(0xffffffffu, m[n][e], d), ol = __shfl_xor_sync(0xffffffffu, l[n][e], d), top = fmaxf(m[n][e], om);
                l[n][e] = l[n][e] * exp2f(m[n][e] - top) + ol * exp2f(om - top);
                m[n][e] = top;
            }
            if (g8 == 0) {
                merge[warp][n * 8 + t4 * 2 + e][0] = m[n][e];
                merge[warp][n * 8 + t4 * 2 + e][1] = l[n][e];
            }
        }
    __syncthreads();
    if (tid < n_heads) {
        float top = kNoScore, sum = 0.f;
#pragma unroll
        for (int w = 0; w < kScoreWarps; w++) top = fmaxf(top, merge[w][tid][0]);
#pragma unroll
        for (int w = 0; w < kScoreWarps; w++) sum = fmaf(merge[w][tid][1], exp2f(merge[w][tid][0] - top), sum);
        float* to = tp.stats + (((long long)seq * p.splits + blockIdx.x) * H + h0 + tid) * 2;
        to[0] = top;
        to[1] = sum;
    }
}

constexpr int kValueWarps = 8, kValueThreads = kValueWarps * 32, kValueKeys = 64, kValueUnits = 8;  // units: (key head, 32 columns, 8 heads), most of a warp
template <int KS> struct ValueSmem {
    static constexpr int row = kValueKeys * 2 + 16;
    static constexpr int talk = 0;
    static constexpr int hi = KS * 16 * (KS * 32 + 16);
    static constexpr int lo = hi + KS * 16 * row;
    static constexpr int mixed = lo + KS * 16 * row;
    static constexpr int total = mixed + KS * 16 * row;
};
// Grid: (value splits, slices of the result's heads, sequences). Values are the rows of the product as well (out^T = v^T w^T): a lane loads eight columns
// of a key, and transposing 8 × 8 blocks in registers makes them its fragments.
template <int KS, int UN> __global__ void __launch_bounds__(kValueThreads, 2) talk_values(const __grid_constant__ TalkP tp) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float lse[KS * 16];
    __shared__ unsigned arrived;
    using L = ValueSmem<KS>;
    const KvP& p = tp.kv;
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3, H = p.heads, rep = H / p.kv_heads, vdim = p.vdim;
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int seq = blockIdx.z, pos = sq.past, h_lo = blockIdx.y * tp.slice_heads, n_heads = min(tp.slice_heads, H - h_lo);
    stage_talk<KS>(smem + L::talk, tp.talk, H, h_lo, tid, kValueThreads);
    for (int i = tid; i < (L::total - L::hi) / 4; i += kValueThreads) reinterpret_cast<unsigned*>(smem + L::hi)[i] = 0;
    pdl_wait();
    if (sq.len != 1) return;
    const int tiles = pos / kValueKeys + 1, first = (int)((long long)tiles * blockIdx.x / tp.value_splits), end = (int)((long long)tiles * (blockIdx.x + 1) / tp.value_splits);
    // units of this slice: its heads of one key head, eight at a time, by 32 columns
    const int g_lo = h_lo / rep, g_n = n_heads / rep, eights = (rep + 7) / 8, blocks = (vdim + 31) / 32, units = g_n * eights * blocks;
    const bf16* values = (const bf16*)p.values;
    const bool whole = (1 << p.shift) >= kValueKeys;  // a tile lies in one page
    struct Tile {
        uint4 v[kValueKeys / 16][2];
    };
    auto load = [&](Tile& to, int k, int t, long long page) {
        const int u = warp + k * kValueWarps;
        if (u >= units || t >= end) return;
        const int g = g_lo + u / (blocks * eights), col = u % blocks * 32 + t4 * 8;
#pragma unroll
        for (int kk = 0; kk < kValueKeys / 16; kk++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int j = min(t * kValueKeys + kk * 16 + g8 + 8 * r, pos);
                to.v[kk][r] = ld16(values + key_row(p, whole ? page : page_of(p, seq, j), g, j) * p.ldv + col, col < vdim);
            }
    };
    auto page_at = [&](int t) { return whole && t < end ? page_of(p, seq, t * kValueKeys) : 0ll; };
    constexpr int kBuffers = UN > 1 ? 2 : 1, kScores = KS * 16 * (kValueKeys / 2) / kValueThreads;
    Tile v[kBuffers];
    long long page = page_at(first);
#pragma unroll
    for (int k = 0; k < kBuffers; k++) load(v[k], k, first, page);
    const float* scores = tp.scores + (long long)seq * H * tp.span;
    float2 sc[kScores];
    auto ask = [&](int t) {
        if (t >= end) return;
#pragma unroll
        for (int i = 0; i < kScores; i++) {
            const int at = tid + i * kValueThreads, h = at / (kValueKeys / 2);
            if (h < H) sc[i] = *reinterpret_cast<const float2*>(scores + (long long)h * tp.span + t * kValueKeys + at % (kValueKeys / 2) * 2);
        }
    };
    ask(first);
    for (int h = warp; h < H; h += kValueWarps) {  // a lane takes splits lane and lane + 32
        const float2* from = reinterpret_cast<const float2*>(tp.stats) + (long long)seq * p.splits * H + h;
        const float2 none = make_float2(kNoScore, 0.f), a = lane < p.splits ? from[(long long)lane * H] : none, b = lane + 32 < p.splits ? from[(long long)(lane + 32) * H] : none;
        const float top = warp_max(fmaxf(a.x, b.x)), sum = warp_sum(fmaf(a.y, exp2f(a.x - top), b.y * exp2f(b.x - top)));
        if (lane == 0) lse[h] = top + log2f(sum);
    }
    __syncthreads();
    const unsigned sm0 = smem_u32(smem);
    float o[UN][2][4];
#pragma unroll
    for (int k = 0; k < UN; k++)
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[k][m][e] = 0.f;
    for (int t = first; t < end; t++) {
        const int j0 = t * kValueKeys;
#pragma unroll
        for (int i = 0; i < kScores; i++) {
            const int at = tid + i * kValueThreads, h = at / (kValueKeys / 2), c = at % (kValueKeys / 2) * 2;
            if (h >= H) break;
            unsigned hi, lo;
            split2(j0 + c <= pos ? exp2f(sc[i].x - lse[h]) : 0.f, j0 + c < pos ? exp2f(sc[i].y - lse[h]) : 0.f, &hi, &lo);
            *reinterpret_cast<unsigned*>(smem + L::hi + h * L::row + c * 2) = hi;
            *reinterpret_cast<unsigned*>(smem + L::lo + h * L::row + c * 2) = lo;
        }
        ask(t + 1);
        const long long next_page = page_at(t + 1);
        __syncthreads();
        for (int x = warp; x < kValueKeys / 16 * KS; x += kValueWarps) {
            const int c = x % (kValueKeys / 16), m = x / (kValueKeys / 16);
            if (m * 16 >= n_heads) break;
            unsigned b[KS][2][4];
            float mixed[2][4];
            load_weights<KS>(b, sm0 + L::hi, sm0 + L::lo, L::row, c * 32);
            mix<KS>(mixed, b, sm0 + L::talk, m);
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int r = 0; r < 2; r++)
                    *reinterpret_cast<unsigned*>(smem + L::mixed + (m * 16 + g8 + 8 * r) * L::row + c * 32 + n * 16 + t4 * 4) = pack_bf16(mixed[n][2 * r], mixed[n][2 * r + 1]);
        }
        __syncthreads();  // (the next tile's weights are written before it, its mix behind the next one)
#pragma unroll
        for (int k = 0; k < UN; k++) {
            const int u = warp + k * kValueWarps;
            if (u >= units) break;
            const int eight = u / blocks % eights, g = g_lo + u / (blocks * eights);
            const int ha = g * rep + eight * 8 + g8;  // this lane's head
            const bool has = ha < (g + 1) * rep;
            const Tile& x = v[k % kBuffers];
#pragma unroll
            for (int kk = 0; kk < kValueKeys / 16; kk++) {
                const unsigned char* w = smem + L::mixed + (has ? ha - h_lo : 0) * L::row + kk * 32 + t4 * 4;
                const unsigned b0 = has ? *reinterpret_cast<const unsigned*>(w) : 0u, b1 = has ? *reinterpret_cast<const unsigned*>(w + 16) : 0u;
                mma_bf16(o[k][0], transpose8x8(x.v[kk][0].x), transpose8x8(x.v[kk][0].y), transpose8x8(x.v[kk][1].x), transpose8x8(x.v[kk][1].y), b0, b1);
                mma_bf16(o[k][1], transpose8x8(x.v[kk][0].z), transpose8x8(x.v[kk][0].w), transpose8x8(x.v[kk][1].z), transpose8x8(x.v[kk][1].w), b0, b1);
            }
            // this buffer's next unit: of this tile, or the first ones of the next
            if (k + kBuffers < UN && warp + (k + kBuffers) * kValueWarps < units) load(v[k % kBuffers], k + kBuffers, t, page);
            else load(v[k % kBuffers], k % kBuffers, t + 1, next_page);
        }
        page = next_page;
    }
    // fragment word m, row r of a unit is column (r / 2) · 8 + 2 m + r % 2 of its 32
    const long long cell = ((long long)seq * gridDim.y + blockIdx.y) * tp.value_splits, part = (long long)tp.slice_heads * vdim;
    bf16* out = (bf16*)p.out + ((long long)sq.start * H + h_lo) * vdim;
    float* mine = tp.parts + (cell + blockIdx.x) * part;
#pragma unroll
    for (int k = 0; k < UN; k++) {
        const int u = warp + k * kValueWarps;
        if (u >= units) break;
        const int block = u % blocks, eight = u / blocks % eights, g = g_lo + u / (blocks * eights);
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int c = block * 32 + g8 / 2 * 8 + 2 * (2 * m + (e >> 1)) + g8 % 2, h = g * rep + eight * 8 + t4 * 2 + (e & 1);
                if (c >= vdim || h >= (g + 1) * rep) continue;
                if (tp.value_splits == 1) out[(h - h_lo) * vdim + c] = __float2bfloat16_rn(o[k][m][e]);
                else mine[(h - h_lo) * vdim + c] = o[k][m][e];
            }
    }
    if (tp.value_splits == 1) return;
    __threadfence();
    __syncthreads();
    unsigned* counter = p.counters + (long long)seq * gridDim.y + blockIdx.y;
    if (tid == 0) arrived = atomicAdd(counter, 1u);
    __syncthreads();
    if (arrived != (unsigned)tp.value_splits - 1) return;
    __threadfence();
    if (tid == 0) *counter = 0;
    for (int i = tid; i < n_heads * vdim; i += kValueThreads) {
        float s = 0.f;
#pragma unroll 8
        for (int k = 0; k < tp.value_splits; k++) s += __ldcg(tp.parts + (cell + k) * part + i);
        out[i] = __float2bfloat16_rn(s);
    }
}

using TalkKernel = void (*)(const TalkP);
template <int KS> TalkKernel any_of(int tk) { return tk == 64 ? talk_prefill_any<64, KS> : talk_prefill_any<32, KS>; }
template <int KS> int any_smem(int tk) { return tk == 64 ? TalkSmem<64, KS>::values : TalkSmem<32, KS>::values; }
template <int KS> TalkKernel values_of(int64_t units) { return units == 1 ? talk_values<KS, 1> : units == 2 ? talk_values<KS, 2> : units <= 4 ? talk_values<KS, 4> : talk_values<KS, 8>; }
template <int TK, int CL, bool FULL> TalkKernel staged_of(int64_t dim, int units) {
    if (units == 1) return dim <= 64 ? talk_prefill<TK, CL, 4, 1, FULL> : dim <= 128 ? talk_prefill<TK, CL, 8, 1, FULL> : talk_prefill<TK, CL, 16, 1, FULL>;
    return dim <= 64 ? talk_prefill<TK, CL, 4, 2, FULL> : talk_prefill<TK, CL, 8, 2, FULL>;
}
template <int CL> TalkKernel staged_of(int tk, int64_t dim, int64_t vdim, int units) {
    const bool full = vdim == dim && (dim == 64 || dim == 128 || dim == 256);
    if (tk == 64) return full ? staged_of<64, CL, true>(dim, units) : staged_of<64, CL, false>(dim, units);
    if (tk == 32) return full ? staged_of<32, CL, true>(dim, units) : staged_of<32, CL, false>(dim, units);
    return staged_of<16, CL, false>(dim, units);
}

}  // namespace

void emit_talking_heads(Emitter& em, const PagedKvDesc& d, KvP p, const TRef& proj, const TRef& turns, Buf q, const TRef& keys, const TRef& values,
                        const TRef& seqs, const TRef& pages, const TRef& out) {
    const Buf none{kSlotNull, 0}, temps = d.temps ? d.temps->buf : none;
    const bool bf = proj.dtype == DT_BF16;
    const int64_t rows = p.rows, n_seqs = p.n_seqs, rep = d.heads / d.kv_heads, H = d.heads;
    const bool tc = !p.singles, decode_only = tc && rows == n_seqs;
    TalkP tp{};
    const Buf lse = decode_only ? none : em.scratch((size_t)(rows * H) * 4);
    Buf scores = none, stats = none, parts = none;
    auto launch = [&](TalkKernel k, dim3 grid, unsigned block, unsigned smem, const char* label, unsigned cluster = 1) {
        ensure_max_dynamic_smem((const void*)k, kTalkSmem);
        tp.kv = p;
        LaunchRec& rec = em.launch(k, grid, dim3(block), smem, tp,
                  {{&tp.kv.proj, proj.buf}, {&tp.kv.turns, turns.buf}, {&tp.kv.keys, keys.buf}, {&tp.kv.values, values.buf}, {&tp.kv.q, q}, {&tp.kv.temps, temps}, {&tp.kv.lse, lse},
                   {&tp.kv.out, out.buf}, {&tp.kv.seqs, seqs.buf}, {&tp.kv.table, pages.buf}, {&tp.kv.counters, Buf{kSlotCounters, 0}}, {&tp.kv.err, Buf{kSlotErr, 0}},
                   {&tp.talk, d.talk->buf}, {&tp.scores, scores}, {&tp.stats, stats}, {&tp.parts, parts}},
                  label, /*pdl=*/true);
        if (cluster > 1) rec.cluster = dim3(cluster, 1, 1);
    };
    if (!tc) {
        launch(bf ? talk_simt_lse<bf16> : talk_simt_lse<float>, dim3((unsigned)rows, (unsigned)H), kSimtThreads, (unsigned)(d.dim * 4), "talk_simt_lse");
        launch(bf ? talk_simt<bf16> : talk_simt<float>, dim3((unsigned)rows), kSimtThreads, (unsigned)(H * (d.dim + d.vdim + 2 * kSimtKeys) * 4), "talk_simt");
        return;
    }
    const int ks = (int)(H + 15) / 16;
    if (!decode_only) {
        emit_kv_lse(em, d, p, q, lse, keys, seqs, pages);
        const int cl = ks;
        const int64_t blocks = (d.vdim + 63) / 64, each = (H + cl - 1) / cl, own_g = std::min(d.kv_heads, (each + rep - 1) / rep + (each % rep != 0)), units = (each * blocks + kTalkWarps - 1) / kTalkWarps;
        auto staged_smem = [&](int tk) {
            const int fixed = cl == 1 ? (tk == 64 ? StagedSmem<64, 1>::keys : tk == 32 ? StagedSmem<32, 1>::keys : StagedSmem<16, 1>::keys)
                                      : (tk == 64 ? StagedSmem<64, 2>::keys : tk == 32 ? StagedSmem<32, 2>::keys : StagedSmem<16, 2>::keys);
            return fixed + (int)own_g * tk * (value_row((int)d.dim) + value_row((int)d.vdim));
        };
        int tk = cl > 2 || units > 2 || (units == 2 && d.dim > 128) ? 0 : 64;
        while (tk >= 16 && staged_smem(tk) > kTalkSmem) tk /= 2;
        if (tk >= 16) {
            const int64_t tiles = (rows + kTalkTokens - 1) / kTalkTokens + n_seqs, seen = (int64_t)p.width * d.page;
            // the longest range of keys or all of them on average, whichever takes longer, and the trip of the parts
            double best = 1e300;
            for (int sp = 1; sp <= 8 && sp * 2 * tk <= std::max<int64_t>(seen, 2 * tk); sp++) {
                const double per_tile = 0.8 + 0.03 * tk, longest = (double)seen / tk, all = (double)tiles * cl * std::max<double>((double)seen - 0.5 * (double)rows / n_seqs, tk) / tk / sm_count();
                const double us = per_tile * std::max(longest / sp, all + 0.5 * longest / sp) + (sp > 1 ? 4.0 + (double)(2 * sp) * rows * H * d.vdim * 4.0 / 4e6 : 0.0);
                if (us < best * 0.97) {
                    best = us;
                    tp.pre_splits = sp;
                }
            }
            if (tp.pre_splits > 1) parts = em.scratch((size_t)tp.pre_splits * rows * H * d.vdim * 4);
            tp.slice_heads = (int)each;
            launch(cl == 1 ? staged_of<1>(tk, d.dim, d.vdim, (int)units) : staged_of<2>(tk, d.dim, d.vdim, (int)units), dim3((unsigned)(tiles * cl), (unsigned)tp.pre_splits), kTalkThreads,
                   (unsigned)staged_smem(tk), "talk_prefill", (unsigned)cl);
            if (tp.pre_splits > 1) launch(talk_merge, dim3((unsigned)((H * d.vdim + 1023) / 1024), (unsigned)rows), 256, 0, "talk_merge");
        } else {
            const int64_t most = kTalkWarps * kTalkUnits / blocks;
            tp.slice_heads = (int)std::min(H, most >= 16 ? most / 16 * 16 : most);
            const int64_t slices = (H + tp.slice_heads - 1) / tp.slice_heads, g_n = std::min(d.kv_heads, (tp.slice_heads + rep - 1) / rep + (tp.slice_heads % rep != 0));
            auto smem_for = [&](int tk) {
                return (ks == 1 ? any_smem<1>(tk) : ks == 2 ? any_smem<2>(tk) : ks == 3 ? any_smem<3>(tk) : any_smem<4>(tk)) + (int)g_n * tk * value_row((int)d.vdim);
            };
            tk = smem_for(64) <= kTalkSmem ? 64 : 32;
            const TalkKernel k = ks == 1 ? any_of<1>(tk) : ks == 2 ? any_of<2>(tk) : ks == 3 ? any_of<3>(tk) : any_of<4>(tk);
            launch(k, dim3((unsigned)((rows + kTalkTokens - 1) / kTalkTokens + n_seqs), (unsigned)slices), kTalkThreads, (unsigned)smem_for(tk), "talk_prefill_any");
        }
    }
    if (!decode_only && n_seqs == 1) return;
    parts = none;
    const int nh = rep > 8;
    const int64_t groups = d.kv_heads * ((rep + 8 * nh + 7) / (8 * nh + 8)), seen = (int64_t)p.width * d.page;
    auto splits_of = [&](int64_t cells, int64_t keys_least, int64_t resident, int64_t most_parts) {  // enough CTAs for the machine, each with a few tiles
        const int64_t want = std::max<int64_t>(1, resident * sm_count() / cells), most = std::max<int64_t>(1, seen / keys_least);
        return (int)std::max<int64_t>(1, std::min<int64_t>({want, most, most_parts}));
    };
    p.splits = splits_of(n_seqs * groups, 2 * kScoreKeys, 8, 64);
    tp.span = (int)((seen + kValueKeys - 1) / kValueKeys * kValueKeys);
    scores = em.scratch((size_t)(n_seqs * H * tp.span) * 4);
    stats = em.scratch((size_t)(n_seqs * p.splits * H) * 8);
    const int64_t columns = (d.vdim + 31) / 32, per_key_head = columns * ((rep + 7) / 8), most_heads = std::max<int64_t>(1, kValueWarps * (kValueUnits / 2) / per_key_head);
    // few sequences: rather more slices than parts of the keys, which have to be added
    int64_t key_heads = std::min(most_heads, d.kv_heads);
    while (key_heads % 2 == 0 && key_heads * per_key_head > kValueWarps && n_seqs * (d.kv_heads / key_heads) * 16 < 2 * sm_count()) key_heads /= 2;
    tp.slice_heads = (int)std::min(H, key_heads * rep);  // whole key heads: at most 64 heads of 256 values share one, which is 64 units
    const int64_t slices = (H + tp.slice_heads - 1) / tp.slice_heads;
    const int64_t units = (key_heads * per_key_head + kValueWarps - 1) / kValueWarps;
    tp.value_splits = splits_of(n_seqs * slices, 2 * kValueKeys, 2, 32);
    if (n_seqs * slices > (int64_t)kCounterWords) tp.value_splits = 1;
    if (tp.value_splits > 1) parts = em.scratch((size_t)(n_seqs * slices * tp.value_splits * tp.slice_heads * d.vdim) * 4);
    const unsigned score_smem = (unsigned)(8 * (nh + 1) * query_row((int)d.dim) + d.rot_dims * 4);
    launch(nh ? talk_scores<2> : talk_scores<1>, dim3((unsigned)p.splits, (unsigned)groups, (unsigned)n_seqs), kScoreThreads, score_smem, "talk_scores");
    const TalkKernel k = ks == 1 ? values_of<1>(units) : ks == 2 ? values_of<2>(units) : ks == 3 ? values_of<3>(units) : values_of<4>(units);
    const unsigned value_smem = (unsigned)(ks == 1 ? ValueSmem<1>::total : ks == 2 ? ValueSmem<2>::total : ks == 3 ? ValueSmem<3>::total : ValueSmem<4>::total);
    launch(k, dim3((unsigned)tp.value_splits, (unsigned)slices, (unsigned)n_seqs), kValueThreads, value_smem, "talk_values");
}

}  // namespace oxk
