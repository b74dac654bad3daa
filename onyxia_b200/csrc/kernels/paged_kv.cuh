// What the kernels of attention over paged keys and values share: their parameters, visible keys, scores, factors.
#pragma once
#include "paged_util.cuh"

namespace oxk {

constexpr int kTalkHeads = 64;      // most heads of the tensor-core kernels that mix heads
constexpr float kNoScore = -1e30f;  // below every score, and finite: differences stay numbers

struct KvP {
    const void* proj;            // [rows, ld]
    const float* turns;          // [2, half]
    void *keys, *values;         // [pages, kv_heads, page, dim | vdim]
    void* q;                     // [rows, heads · dim]: prepared queries
    void* out;                   // [rows, heads · vdim]
    const int* seqs;             // [R, 4]
    const int* table;            // [R, width]
    float* part;                 // decode partial results
    unsigned* counters;
    ErrWord* err;
    const float* sinks;          // [heads], or null: 0
    const void* gate;            // [rows, gate_ld]: a factor per head, or null
    long long rows, ld, q_off, k_off, v_off, gate_ld;
    int n_seqs, width, n_pages, shift /* log2 of the page */, heads, kv_heads, dim, vdim, half, window, splits, node;
    int ldv;                     // elements from one value to the next: vdim, or dim where values are the front of the keys
    int interleaved;             // pairs of dimensions 2i, 2i + 1 instead of i, i + half
    float scale, cap, eps;       // scores in natural units
    float mul2, cap2;            // base 2: cap2 = 0: score2 = mul2 · q·k, otherwise cap2 · tanh with mul2 = 2 log2 e · scale / cap
    int norm, sink, append;
    int singles;                 // prepare: also sequences with one new token
    const float* temps;          // [heads]: factors of the scores, or null
    float* lse;                  // [rows, heads]: base-2 logarithm of the softmax's sum (the prefill kernel's form that has no values)
};

__device__ __forceinline__ int first_key(const KvP& p, int pos) { return p.window > 0 ? max(0, pos - p.window + 1) : 0; }
// log2 e · score of a dot product, `mul2` the head's; tanh x = 1 − 2 / (1 + e^2x) is off by a few 1e-7 of the cap
__device__ __forceinline__ float score2(const KvP& p, float d, float mul2) {
    const float x = d * mul2;
    return p.cap2 > 0.f ? p.cap2 - __fdividef(2.f * p.cap2, 1.f + exp2f(x)) : x;
}
__device__ __forceinline__ float temp_of(const KvP& p, int h) { return p.temps ? p.temps[h] : 1.f; }
__device__ __forceinline__ float sink_of(const KvP& p, int h) { return p.sinks ? p.sinks[h] : 0.f; }  // in natural units
template <typename T> __device__ __forceinline__ float gate_of(const KvP& p, long long row, int h) {
    return p.gate ? to_f(((const T*)p.gate)[row * p.gate_ld + h]) : 1.f;
}
// 1 / root mean square of a head, by one warp
template <typename T> __device__ __forceinline__ float head_factor(const KvP& p, const T* x) {
    if (!p.norm) return 1.f;
    float ss = 0.f;
    for (int i = threadIdx.x & 31; i < p.dim; i += 32) {
        const float v = to_f(x[i]);
        ss = fmaf(v, v, ss);
    }
    return 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
}

// Attention whose heads' softmax weights are mixed (talking_heads.cu). `p` is complete but for the pointers; new keys and values and the
// queries `q` of sequences with several new tokens are prepared.
void emit_talking_heads(Emitter&, const PagedKvDesc&, KvP p, const TRef& proj, const TRef& turns, Buf q, const TRef& keys, const TRef& values,
                        const TRef& seqs, const TRef& pages, const TRef& out);
// The form of the prefill kernel that leaves `lse` only.
void emit_kv_lse(Emitter&, const PagedKvDesc&, KvP p, Buf q, Buf lse, const TRef& keys, const TRef& seqs, const TRef& pages);

}  // namespace oxk
