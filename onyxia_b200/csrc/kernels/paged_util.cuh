// Device helpers of attention over paged pools: pages, tiles of ragged prompts, merging of partial softmax results. Kernel
// parameter structs name their page table, its width, the number of pages and the page shift alike.
#pragma once
#include "tc_util.cuh"

namespace oxk {

constexpr float kLog2e = 1.4426950408889634f;

template <class P> __device__ __forceinline__ long long page_of(const P& p, int seq, int pos) {
    const int i = pos >> p.shift;
    const int pg = i < p.width ? p.table[(long long)seq * p.width + i] : -1;
    if ((unsigned)pg >= (unsigned)p.n_pages) {
        report(p.err, ERR_GATHER_OOB, p.node, pg, p.n_pages);
        return 0;
    }
    return pg;
}
// Row of a pool (its innermost axis is one key or value) of position `pos`, which lies in page `pg`.
template <class P> __device__ __forceinline__ long long key_row(const P& p, long long pg, int g, int pos) {
    return ((pg * p.kv_heads + g) << p.shift) + (pos & ((1 << p.shift) - 1));
}
// Sine and cosine of every pair at a position, by `threads` threads. `turns` [2, half]: turns per position, high and low part.
__device__ __forceinline__ void angles(const float* turns, int half, int pos, float* cs, float* sn, int tid, int threads) {
    for (int i = tid; i < half; i += threads) {
        const double t = (double)pos * ((double)turns[i] + (double)turns[half + i]);
        sincospif(2.f * (float)(t - rint(t)), sn + i, cs + i);
    }
}
// Dimension i of a head whose leading 2 · half dimensions turn: pairs 2i, 2i + 1 (interleaved) or i, i + half.
template <typename T> __device__ __forceinline__ float rotated(int half, int interleaved, const T* x, const float* cs, const float* sn, int i) {
    const float v = to_f(x[i]);
    if (i >= 2 * half) return v;
    if (interleaved) {
        const float other = to_f(x[i ^ 1]);
        return i & 1 ? v * cs[i >> 1] + other * sn[i >> 1] : v * cs[i >> 1] - other * sn[i >> 1];
    }
    const bool low = i < half;
    const int a = low ? i : i - half;
    const float other = to_f(x[low ? i + half : a]);
    return low ? v * cs[a] - other * sn[a] : v * cs[a] + other * sn[a];
}
// The tile a CTA works on: tiles of `tq` tokens are counted over the sequences with more than one new token (`least` = 2) or
// over all of them (1).
__device__ __forceinline__ bool locate_tile(const int* seqs, int n_seqs, int tile, int tq, int* seq, int* first, int least = 2) {
    const int lane = threadIdx.x & 31;
    int before = 0;
    for (int r0 = 0; r0 < n_seqs; r0 += 32) {
        int n = 0;
        if (r0 + lane < n_seqs) {
            const int len = seqs[4 * (r0 + lane) + 1];
            n = len >= least ? (len + tq - 1) / tq : 0;
        }
        int inc = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int v = __shfl_up_sync(0xffffffffu, inc, o);
            if (lane >= o) inc += v;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, before + inc > tile);
        if (hit) {
            const int at = __ffs(hit) - 1;
            *seq = r0 + at;
            *first = (tile - before - (__shfl_sync(0xffffffffu, inc, at) - __shfl_sync(0xffffffffu, n, at))) * tq;
            return true;
        }
        before += __shfl_sync(0xffffffffu, inc, 31);
    }
    return false;
}

constexpr int part_size(int rows, int values) { return rows * (values + 2); }
// Adds `n` partial results ([n][rows][DP + 2]: maximum, sum, accumulator); `out` gets head r's values divided by the sum and
// multiplied by scale(r), or with `raw` the merged partial result itself. sink(r) is a score (base 2) without a value; −inf: none.
template <int DP, int ROWS, int WARPS, class Scale, class Sink>
__device__ void merge_parts(const float* part, int n, int heads, int dim, Scale&& scale, bf16* out, float* raw, Sink&& sink) {
    constexpr int size = part_size(ROWS, DP);
    for (int r = threadIdx.x >> 5; r < heads; r += WARPS) {
        const int lane = threadIdx.x & 31;
        // lane i weighs parts i and i + 32 (n ≤ 64); a part that saw no key has maximum −inf, sum and values 0
        const float* head = part + r * (DP + 2);
        float pm[2], pl[2];
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const bool in = k * 32 + lane < n;
            pm[k] = in ? head[(k * 32 + lane) * size] : -INFINITY;
            pl[k] = in ? head[(k * 32 + lane) * size + 1] : 0.f;
        }
        float m = warp_max(fmaxf(pm[0], pm[1]));
        const float s = sink(r);
        m = fmaxf(m, s);
        const float none = m == -INFINITY ? 0.f : m;  // a split without keys: its weights are all zero
        const float f0 = exp2f(pm[0] - none), f1 = exp2f(pm[1] - none);
        const float l = warp_sum(fmaf(pl[0], f0, pl[1] * f1)) + exp2f(s - none);
        float o[(DP + 31) / 32] = {};
#pragma unroll 4
        for (int i = 0; i < n; i++) {
            const float f = __shfl_sync(0xffffffffu, i < 32 ? f0 : f1, i & 31);
#pragma unroll
            for (int c = 0; c < (DP + 31) / 32; c++)
                if (c * 32 + lane < DP) o[c] = fmaf(head[i * size + 2 + c * 32 + lane], f, o[c]);
        }
        if (raw) {
            float* q = raw + r * (DP + 2);
            if (lane == 0) {
                q[0] = m;
                q[1] = l;
            }
#pragma unroll
            for (int c = 0; c < (DP + 31) / 32; c++)
                if (c * 32 + lane < DP) q[2 + c * 32 + lane] = o[c];
        } else {
            const float f = scale(r) / l;
#pragma unroll
            for (int c = 0; c < (DP + 31) / 32; c++)
                if (c * 32 + lane < dim) out[r * dim + c * 32 + lane] = __float2bfloat16_rn(o[c] * f);
        }
    }
}

template <int DP, int ROWS, int WARPS> __device__ void merge_parts(const float* part, int n, int heads, int dim, float scale, bf16* out, float* raw) {
    merge_parts<DP, ROWS, WARPS>(part, n, heads, dim, [scale](int) { return scale; }, out, raw, [](int) { return -INFINITY; });
}

__device__ __forceinline__ unsigned transpose8x8(unsigned v) {
    unsigned r;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
    return r;
}

}  // namespace oxk
