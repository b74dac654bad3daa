// Device helpers shared by the bf16 tensor-core kernels: mbarriers with bounded waits, TMA tile loads,
// tcgen05 descriptors, `mma.sync` / `ldmatrix` / `cp.async` wrappers, typed loads and stores.
#pragma once
#include "common.cuh"

namespace oxk {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ unsigned smem_u32(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }

// ── mbarriers ──
__device__ __forceinline__ void mbar_init(unsigned bar, unsigned count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory");
}
__device__ __forceinline__ void mbar_expect_tx(unsigned bar, unsigned bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool mbar_try(unsigned bar, unsigned parity) {
    unsigned ok;
    asm volatile(
        "{\n .reg .pred p;\n mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}\n"
        : "=r"(ok)
        : "r"(bar), "r"(parity)
        : "memory");
    return ok != 0;
}
// False when the phase did not complete within about a second.
__device__ __forceinline__ bool mbar_wait(unsigned bar, unsigned parity) {
    if (mbar_try(bar, parity)) return true;
    const long long t0 = clock64();
    while (clock64() - t0 < 2000000000LL)
        if (mbar_try(bar, parity)) return true;
    return false;
}

// ── TMA: one 2-D tile; x must keep the copy on a 16-byte boundary ──
__device__ __forceinline__ void tma_load_2d(unsigned dst, const void* map, int x, int y, unsigned bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
                 "l"(reinterpret_cast<unsigned long long>(map)), "r"(x), "r"(y), "r"(bar)
                 : "memory");
}

// ── tcgen05 ──
// Shared-memory matrix descriptor: K-major, 128-byte swizzle, 8-row groups 1 024 bytes apart.
__device__ __forceinline__ unsigned long long umma_kmajor_desc(unsigned smem_byte_addr) {
    return (unsigned long long)((smem_byte_addr & 0x3FFFFu) >> 4) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void umma_bf16(unsigned d, unsigned long long a, unsigned long long b, unsigned idesc, bool accumulate) {
    asm volatile(
        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
        " tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n}\n" ::"r"(d),
        "l"(a), "l"(b), "r"(idesc), "r"(accumulate ? 1u : 0u), "r"(0u)
        : "memory");
}
__device__ __forceinline__ void umma_commit(unsigned bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}

// ── warp-level tensor core ──
__device__ __forceinline__ void mma_bf16(float (&c)[4], unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void cp_async16(unsigned dst, const void* src, bool live) {
    const int n = live ? 16 : 0;  // 0: the sixteen bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async16(unsigned dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}

// ── typed scalars ──
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// The same for values that are rounded to bf16 or come from such: f32 with the approximate exponential and quotient (a few
// parts in a million).
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
__device__ __forceinline__ float gelu_tanh_fast(float z) {
    // tanh(x) = 1 − 2 / (1 + e^2x); z / (1 + e^−2x) = z (1 + tanh x) / 2
    return __fdividef(z, 1.f + __expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

// log(1 + e^z). Both terms of the sum keep their digits: a small e^−|z| is the argument of a series.
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float softplus_fast(float z) {
    const float e = __expf(-fabsf(z));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 1.f / 3.f), -0.5f), 1.f);  // e < 1/64: off by less than e^4 / 5
    return fmaxf(z, 0.f) + (e < 0.015625f ? series : __logf(1.f + e));
}

// ── ragged batches ──
struct SeqRow {
    int start, len, past, slot;
};
__device__ __forceinline__ SeqRow load_seq(const int* seqs, int r) {
    const int4 v = reinterpret_cast<const int4*>(seqs)[r];
    return SeqRow{v.x, v.y, v.z, v.w};
}
// The sequence that row `row` belongs to: the last one whose first row is not after it.
__device__ __forceinline__ int find_seq(const int* seqs, int n, int row) {
    int lo = 0, hi = n - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (seqs[4 * mid] <= row) lo = mid;
        else hi = mid - 1;
    }
    return lo;
}

}  // namespace oxk
