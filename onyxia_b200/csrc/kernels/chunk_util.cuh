// Device helpers of recurrences with a matrix state that are worked off in chunks of tokens.
#pragma once
#include "paged_util.cuh"

namespace oxk {

constexpr int kCols = 64;                        // columns of the state per CTA
constexpr int kColStride = kCols * 2 + 16;       // bytes per row: conflict-free ldmatrix
__host__ __device__ constexpr int padded(int dim) { return (dim + 15) / 16 * 16; }
__host__ __device__ constexpr int row_stride(int dim) { return padded(dim) * 2 + 16; }

// 2^x, a few parts in ten million
__device__ __forceinline__ float power2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// a = hi + lo to 16 bits, two values per word
__device__ __forceinline__ void split2(float a, float b, unsigned* hi, unsigned* lo) {
    const unsigned h = pack_bf16(a, b);
    *hi = h;
    *lo = pack_bf16(a - __uint_as_float(h << 16), b - __uint_as_float(h & 0xFFFF0000u));
}
// Rows of q, k or v of a chunk into shared memory, zeros beyond its tokens and columns.
__device__ __forceinline__ void load_rows(unsigned dst, int stride, const bf16* src, long long ld, int n_tok, int cols, int padded_cols, int tid, int threads) {
    // a row per power of two of lanes
    const int per = padded_cols / 8, shift = per <= 1 ? 0 : 32 - __clz(per - 1), c = (tid & ((1 << shift) - 1)) * 8;
    if (c >= padded_cols) return;
    const int step = threads >> shift;
    int r = tid >> shift;
    const bf16* from = src + r * ld + (c < cols ? c : 0);
    if (c >= cols) n_tok = 0;
    unsigned to = dst + r * stride + c * 2;
    for (; r < kLightningChunk; r += step) {
        cp_async16(to, r < n_tok ? from : src, r < n_tok);
        from += step * ld;
        to += step * stride;
    }
}

// Chunks of the sequences before sequence `seq` (those with one new token have none). Called by whole warps.
__device__ __forceinline__ int chunks_before(const int* seqs, int seq) {
    const int lane = threadIdx.x & 31;
    int chunks = 0;
    for (int r0 = 0; r0 < seq; r0 += 32) {
        int n = 0;
        if (r0 + lane < seq) {
            const int len = seqs[4 * (r0 + lane) + 1];
            n = len > 1 ? (len + kLightningChunk - 1) / kLightningChunk : 0;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
        chunks += n;
    }
    return chunks;
}

}  // namespace oxk
