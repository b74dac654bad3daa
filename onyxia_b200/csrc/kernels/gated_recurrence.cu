// Real-gated linear recurrence behind a causal convolution, over a ragged batch with per-slot state.
//
//   u = conv(x)                                   per channel, `taps` taps, inputs before the start are zero
//   r = sigmoid(ra u + ra_b), i = sigmoid(ri u + ri_b)    block-diagonal, one square matrix per block
//   log a = −decay · r · softplus(lam),  S_t = a S_{t−1} + sqrt(1 − a²) i u,  out = S · gelu(y) · out_scale
//
// x and y are columns of a fused projection. In the bf16 form u is rounded once, before the gates; the products are
// exact bf16 pairs summed in f32 and everything behind them is f32. The state of a sequence is S (f32) and a
// ring of its last inputs (row = position modulo taps); a sequence at position 0 reads neither, so slots need no
// clearing.
//
//   recurrence_step    every sequence has one new token: convolution, gates, state and output in one launch
//   recurrence_gates   convolution and gates of all tokens → a − 1 and sqrt(1 − a²) i u in f32 (`mma.sync`)
//   recurrence_scan    32 channels × one sequence per CTA; each warp scans 16 tokens in registers, the warps' (product,
//                      sum) pairs are chained through shared memory, and the scan is replayed from the right state
//   recurrence_gates_simt   f32, and block sizes that are not a multiple of 8
//
// Gates: 4 · tokens · width · n FLOPs (n = width / blocks); bytes 2 · width (x) read + 8 · width written per token. Scan: 8 ·
// width read + 4 · width (y, out) per token.
#include "tc_util.cuh"

namespace oxk {

namespace {

struct RecP {
    const void* proj;   // [rows, ld]
    const float *cw, *cb;   // [width, taps], [width]
    const void *ra, *ri;    // [blocks, n, n] (out, in)
    const float *rab, *rib, *lam;
    void* ring;             // [slots, taps, width]
    float* state;           // [slots, width]
    const int* seqs;
    float *e, *b;           // [rows, width]: a − 1, sqrt(1 − a²) i u
    void* out;              // [rows, width]
    ErrWord* err;
    long long rows, ld, x_off, y_off;
    int n_seqs, n_slots, width, blocks, n, taps, node;
    float decay, out_scale;
};

__device__ __forceinline__ int slot_of(const RecP& p, int slot) {
    if ((unsigned)slot >= (unsigned)p.n_slots) {
        report(p.err, ERR_GATHER_OOB, p.node, slot, p.n_slots);
        return 0;
    }
    return slot;
}

// Input of channel c, `back` tokens before batch row `row` of sequence `s`, whose own position is `pos`.
template <typename T> __device__ __forceinline__ float conv_input(const RecP& p, const SeqRow& s, int slot, int row, int pos, int back, int c) {
    if (pos - back < 0) return 0.f;
    if (row - back >= s.start) return to_f(((const T*)p.proj)[(long long)(row - back) * p.ld + p.x_off + c]);
    return to_f(((const T*)p.ring)[((long long)slot * p.taps + (pos - back) % p.taps) * p.width + c]);
}
template <typename T> __device__ __forceinline__ float conv_at(const RecP& p, const SeqRow& s, int slot, int row, int pos, int c) {
    float u = p.cb[c];
    for (int back = 0; back < p.taps; back++) u = fmaf(conv_input<T>(p, s, slot, row, pos, back, c), p.cw[(long long)c * p.taps + p.taps - 1 - back], u);
    return u;
}
// (pre-activations of r and i, u) of channel c → a − 1 and sqrt(1 − a²) i u. A decay next to 1 keeps its digits in a − 1;
// rounded to f32 itself it would be off by as much as 6e-8 of a state that lives for 1 / (1 − a) tokens.
__device__ __forceinline__ void gate_values(const RecP& p, int c, float zr, float zi, float u, float* e, float* b) {
    const float lam = p.lam[c], sp = fmaxf(lam, 0.f) + log1pf(expf(-fabsf(lam)));
    const float la = -p.decay * sigmoid_f(zr + p.rab[c]) * sp;
    *e = expm1f(la);
    *b = sqrtf(-*e * (2.f + *e)) * sigmoid_f(zi + p.rib[c]) * u;
}
// a S + b from e = a − 1
__device__ __forceinline__ float advance(float e, float S, float b) { return S + fmaf(e, S, b); }

// ───────────────────────────── one token per sequence ───────────────────
// CTA: 16 sequences × 16 channels of one block. Warp w forms eight outputs of one gate: w & 1 picks the gate, w >> 1 the
// eight channels; a lane reads 16 consecutive bytes of a weight row, u is read with the same permutation of k.
__global__ void __launch_bounds__(128) recurrence_step(const RecP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float z[2][16][17];
    __shared__ SeqRow sq[16];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int n = p.n, slices = (n + 15) / 16, blk = blockIdx.x / slices, o0 = (blockIdx.x % slices) * 16, r0 = blockIdx.y * 16;
    const int kc = (n + 31) / 32, stride = kc * 32 + (kc & 1 ? 0 : 32);  // 64 bytes off a multiple of 128
    bf16* us = reinterpret_cast<bf16*>(smem);
    const int o = o0 + (warp >> 1) * 8 + g;
    const bf16* w = (const bf16*)(warp & 1 ? p.ri : p.ra) + ((long long)blk * n + (o < n ? o : 0)) * n;
    auto weights = [&](int c) { return o < n && c * 32 + t * 8 < n ? __ldg(reinterpret_cast<const uint4*>(w + c * 32 + t * 8)) : make_uint4(0, 0, 0, 0); };
    pdl_trigger();
    uint4 wv[8];  // constants: may overlap the launches before this one
#pragma unroll
    for (int c = 0; c < 8; c++) wv[c] = c < kc ? weights(c) : make_uint4(0, 0, 0, 0);
    pdl_wait();
    if (tid < 16) {
        SeqRow s{0, 0, 0, 0};
        if (r0 + tid < p.n_seqs) {
            s = load_seq(p.seqs, r0 + tid);
            s.slot = slot_of(p, s.slot);
        }
        sq[tid] = s;
    }
    __syncthreads();
    const int live = min(16, p.n_seqs - r0);
#pragma unroll 2
    for (int i = tid; i < 16 * kc * 32; i += 128) {
        const int m = i / (kc * 32), k = i % (kc * 32), c = blk * n + k;
        float u = 0.f;
        if (m < live && k < n) u = conv_at<bf16>(p, sq[m], sq[m].slot, sq[m].start, sq[m].past, c);
        us[m * stride + k] = __float2bfloat16_rn(u);
    }
    __syncthreads();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int c0 = 0; c0 < kc; c0 += 8) {
#pragma unroll
        for (int j = 0; j < 8; j++) {
            const int c = c0 + j;
            if (c >= kc) break;
            const uint4 b = c0 == 0 ? wv[j] : weights(c);
            const uint4 lo = *reinterpret_cast<const uint4*>(us + g * stride + c * 32 + t * 8);
            const uint4 hi = *reinterpret_cast<const uint4*>(us + (g + 8) * stride + c * 32 + t * 8);
            mma_bf16(acc, lo.x, hi.x, lo.y, hi.y, b.x, b.y);
            mma_bf16(acc, lo.z, hi.z, lo.w, hi.w, b.z, b.w);
        }
    }
    const int col = (warp >> 1) * 8 + t * 2;
    z[warp & 1][g][col] = acc[0];
    z[warp & 1][g][col + 1] = acc[1];
    z[warp & 1][g + 8][col] = acc[2];
    z[warp & 1][g + 8][col + 1] = acc[3];
    __syncthreads();
    for (int i = tid; i < 256; i += 128) {
        const int m = i >> 4, k = o0 + (i & 15), c = blk * n + k;
        if (m >= live || k >= n) continue;
        const SeqRow s = sq[m];
        float e, b;
        gate_values(p, c, z[0][m][i & 15], z[1][m][i & 15], to_f(us[m * stride + k]), &e, &b);
        const long long st = (long long)s.slot * p.width + c;
        const float S = s.past > 0 ? advance(e, p.state[st], b) : b;
        p.state[st] = S;
        const bf16* row = (const bf16*)p.proj + (long long)s.start * p.ld;
        ((bf16*)p.out)[(long long)s.start * p.width + c] = __float2bfloat16_rn(S * gelu_tanh_f(to_f(row[p.y_off + c])) * p.out_scale);
        // this position's ring row: no other CTA reads it (they look back taps − 1 positions at most)
        ((bf16*)p.ring)[((long long)s.slot * p.taps + s.past % p.taps) * p.width + c] = row[p.x_off + c];
    }
}

// ───────────────────────────── gates of many tokens ─────────────────────
// CTA: 64 tokens × 64 channels of one block, k in chunks of 64.
constexpr int kGateStride = 72;  // bf16 per row of a staged chunk: conflict-free ldmatrix
__global__ void __launch_bounds__(128) recurrence_gates(const RecP p) {
    __shared__ __align__(16) bf16 us[64 * kGateStride], wr[64 * kGateStride], wi[64 * kGateStride], own[64 * 64];
    __shared__ SeqRow sq[64];
    __shared__ int pos[64];
    pdl_enter();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int n = p.n, slices = (n + 63) / 64, blk = blockIdx.y / slices, o0 = (blockIdx.y % slices) * 64;
    const long long m0 = (long long)blockIdx.x * 64;
    if (tid < 64) {
        const long long row = m0 + tid;
        SeqRow s{0, 0, 0, 0};
        int at = -1;
        if (row < p.rows) {
            s = load_seq(p.seqs, find_seq(p.seqs, p.n_seqs, (int)row));
            if (row < s.start + s.len) {
                s.slot = slot_of(p, s.slot);
                at = s.past + (int)row - s.start;
            }
        }
        sq[tid] = s;
        pos[tid] = at;
    }
    __syncthreads();
    float ar[8][4], ai[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) ar[j][e] = ai[j][e] = 0.f;
    for (int k0 = 0; k0 < n; k0 += 64) {
        for (int i = tid; i < 64 * 8; i += 128) {  // weight rows o0 … + 64, eight k per copy
            const int r = i >> 3, c = i & 7;
            const bool live = o0 + r < n && k0 + c * 8 < n;
            const long long off = live ? ((long long)blk * n + o0 + r) * n + k0 + c * 8 : 0;
            cp_async16(smem_u32(wr + r * kGateStride + c * 8), (const bf16*)p.ra + off, live);
            cp_async16(smem_u32(wi + r * kGateStride + c * 8), (const bf16*)p.ri + off, live);
        }
        cp_async_commit();
        {   // u: a thread follows one channel over 32 consecutive tokens, the last inputs in registers
            const int c = tid & 63, k = k0 + c, ch = blk * n + k, half = (tid >> 6) * 32;
            const bool live = k < n;
            if (live && p.taps <= 4) {
                float w[4], x[4] = {0.f, 0.f, 0.f, 0.f};  // x[j]: input j tokens back
#pragma unroll
                for (int j = 0; j < 4; j++) w[j] = j < p.taps ? p.cw[(long long)ch * p.taps + p.taps - 1 - j] : 0.f;
                const float bias = p.cb[ch];
                const bf16* src = (const bf16*)p.proj + p.x_off + ch;
#pragma unroll 8
                for (int m = half; m < half + 32; m++) {
                    float u = 0.f;
                    if (pos[m] >= 0) {
                        x[3] = x[2];
                        x[2] = x[1];
                        x[1] = x[0];
                        x[0] = to_f(src[(m0 + m) * p.ld]);
                        if (m == half || pos[m] == sq[m].past) {  // a run starts here: fetch what lies before it
#pragma unroll
                            for (int j = 1; j < 4; j++) x[j] = j < p.taps ? conv_input<bf16>(p, sq[m], sq[m].slot, (int)(m0 + m), pos[m], j, ch) : 0.f;
                        }
                        u = bias;
#pragma unroll
                        for (int j = 0; j < 4; j++) u = fmaf(x[j], w[j], u);
                    }
                    us[m * kGateStride + c] = __float2bfloat16_rn(u);
                }
            } else {
                for (int m = half; m < half + 32; m++)
                    us[m * kGateStride + c] = __float2bfloat16_rn(live && pos[m] >= 0 ? conv_at<bf16>(p, sq[m], sq[m].slot, (int)(m0 + m), pos[m], ch) : 0.f);
            }
            if (k0 == o0)
                for (int m = half; m < half + 32; m++) own[m * 64 + c] = us[m * kGateStride + c];
        }
        cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            unsigned a[4];
            ldmatrix_x4(a, smem_u32(us + (warp * 16 + (lane & 15)) * kGateStride + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                const int at = (j * 8 + (lane & 7) + (lane >> 4) * 8) * kGateStride + kk * 16 + ((lane >> 3) & 1) * 8;
                unsigned b[4];
                ldmatrix_x4(b, smem_u32(wr + at));
                mma_bf16(ar[j], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(ar[j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                ldmatrix_x4(b, smem_u32(wi + at));
                mma_bf16(ai[j], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(ai[j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
        for (int v = 0; v < 4; v++) {
            const int m = warp * 16 + g + 8 * (v >> 1), k = o0 + j * 8 + t * 2 + (v & 1), c = blk * n + k;
            if (k >= n || pos[m] < 0) continue;
            float e, b;
            gate_values(p, c, ar[j][v], ai[j][v], to_f(own[m * 64 + k - o0]), &e, &b);
            p.e[(m0 + m) * p.width + c] = e;
            p.b[(m0 + m) * p.width + c] = b;
        }
}

// One CTA per (token, block).
template <typename T> __global__ void __launch_bounds__(128) recurrence_gates_simt(const RecP p) {
    extern __shared__ float uf[];
    pdl_enter();
    const int row = blockIdx.x, blk = blockIdx.y, n = p.n;
    const SeqRow s = load_seq(p.seqs, find_seq(p.seqs, p.n_seqs, row));
    if (row >= s.start + s.len) return;
    const int slot = slot_of(p, s.slot), pos = s.past + row - s.start;
    for (int k = threadIdx.x; k < n; k += 128) uf[k] = to_f(from_f<T>(conv_at<T>(p, s, slot, row, pos, blk * n + k)));
    __syncthreads();
    for (int k = threadIdx.x; k < n; k += 128) {
        const int c = blk * n + k;
        const T *wr = (const T*)p.ra + (long long)c * n, *wi = (const T*)p.ri + (long long)c * n;
        float zr = 0.f, zi = 0.f;
        for (int j = 0; j < n; j++) {
            zr = fmaf(uf[j], to_f(wr[j]), zr);
            zi = fmaf(uf[j], to_f(wi[j]), zi);
        }
        float e, b;
        gate_values(p, c, zr, zi, uf[k], &e, &b);
        p.e[(long long)row * p.width + c] = e;
        p.b[(long long)row * p.width + c] = b;
    }
}

// ───────────────────────────── scan ─────────────────────────────────────
constexpr int kScanWarps = 16, kScanTokens = 16;
template <typename T> __global__ void __launch_bounds__(kScanWarps * 32) recurrence_scan(const RecP p) {
    __shared__ float pa[kScanWarps][32], pb[kScanWarps][32], carry[32];
    pdl_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    const SeqRow s = load_seq(p.seqs, blockIdx.y);
    const int slot = slot_of(p, s.slot);
    const bool live = c < p.width;
    if (s.len <= 0) return;
    if (warp == 0) carry[lane] = live && s.past > 0 ? p.state[(long long)slot * p.width + c] : 0.f;
    const T* proj = (const T*)p.proj;
    for (int t0 = 0; t0 < s.len; t0 += kScanWarps * kScanTokens) {
        const int lo = t0 + warp * kScanTokens;
        float e[kScanTokens], b[kScanTokens], y[kScanTokens];
#pragma unroll
        for (int j = 0; j < kScanTokens; j++) {
            const bool in = live && lo + j < s.len;
            const long long row = s.start + lo + j;
            e[j] = in ? p.e[row * p.width + c] : 0.f;
            b[j] = in ? p.b[row * p.width + c] : 0.f;
            y[j] = in ? to_f(proj[row * p.ld + p.y_off + c]) : 0.f;
        }
        float E = 0.f, B = 0.f;  // E: product of the decays, minus 1
#pragma unroll
        for (int j = 0; j < kScanTokens; j++) {
            E = advance(e[j], E, e[j]);
            B = advance(e[j], B, b[j]);
        }
        pa[warp][lane] = E;
        pb[warp][lane] = B;
        __syncthreads();
        float S = carry[lane];
        for (int w = 0; w < warp; w++) S = advance(pa[w][lane], S, pb[w][lane]);
#pragma unroll
        for (int j = 0; j < kScanTokens; j++) {
            S = advance(e[j], S, b[j]);
            if (live && lo + j < s.len) ((T*)p.out)[(long long)(s.start + lo + j) * p.width + c] = from_f<T>(S * gelu_tanh_f(y[j]) * p.out_scale);
        }
        __syncthreads();
        if (warp == kScanWarps - 1) carry[lane] = S;  // tokens past the end leave it alone
        __syncthreads();
    }
    if (warp == 0 && live) {
        p.state[(long long)slot * p.width + c] = carry[lane];
        for (int back = min(p.taps, s.len) - 1; back >= 0; back--) {
            const int pos = s.past + s.len - 1 - back;
            ((T*)p.ring)[((long long)slot * p.taps + pos % p.taps) * p.width + c] = proj[(long long)(s.start + s.len - 1 - back) * p.ld + p.x_off + c];
        }
    }
}

}  // namespace

void emit_gated_recurrence(Emitter& em, const GatedRecurrenceDesc& d, const TRef& proj, const TRef& conv_w, const TRef& conv_b,
                           const TRef& ra, const TRef& ra_b, const TRef& ri, const TRef& ri_b, const TRef& lam, const TRef& conv_state,
                           const TRef& state, const TRef& seqs, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    RecP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.x_off = d.x_off;
    p.y_off = d.y_off;
    p.n_seqs = (int)n_seqs;
    p.n_slots = (int)state.shape[0];
    p.width = (int)d.width;
    p.blocks = (int)d.blocks;
    p.n = (int)(d.width / d.blocks);
    p.taps = (int)d.taps;
    p.decay = (float)d.decay;
    p.out_scale = (float)d.out_scale;
    p.node = em.node;
    const bool bf = proj.dtype == DT_BF16, tc = bf && p.n % 8 == 0;
    const int kc = (p.n + 31) / 32;
    const unsigned step_smem = 16u * (unsigned)(kc * 32 + (kc & 1 ? 0 : 32)) * 2u;
    const bool step = tc && rows == n_seqs && step_smem <= 200 * 1024;
    const Buf none{kSlotNull, 0};
    const Buf e = step ? none : em.scratch((size_t)rows * d.width * 4), b = step ? none : em.scratch((size_t)rows * d.width * 4);
    auto launch = [&](void (*k)(const RecP), dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.cw, conv_w.buf}, {&p.cb, conv_b.buf}, {&p.ra, ra.buf}, {&p.ri, ri.buf}, {&p.rab, ra_b.buf}, {&p.rib, ri_b.buf},
                   {&p.lam, lam.buf}, {&p.ring, conv_state.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf}, {&p.e, e}, {&p.b, b}, {&p.out, out.buf},
                   {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    if (step) {
        ensure_max_dynamic_smem((const void*)recurrence_step, 200 * 1024);
        launch(recurrence_step, dim3((unsigned)(p.blocks * ((p.n + 15) / 16)), (unsigned)((n_seqs + 15) / 16)), 128, step_smem, "recurrence_step");
        return;
    }
    if (tc) {
        launch(recurrence_gates, dim3((unsigned)((rows + 63) / 64), (unsigned)(p.blocks * ((p.n + 63) / 64))), 128, 0, "recurrence_gates");
    } else {
        const auto k = bf ? recurrence_gates_simt<bf16> : recurrence_gates_simt<float>;
        ensure_max_dynamic_smem((const void*)k, 200 * 1024);
        launch(k, dim3((unsigned)rows, (unsigned)p.blocks), 128, (unsigned)p.n * 4, "recurrence_gates_simt");
    }
    launch(bf ? recurrence_scan<bf16> : recurrence_scan<float>, dim3((unsigned)((d.width + 31) / 32), (unsigned)n_seqs), kScanWarps * 32, 0, "recurrence_scan");
}

}  // namespace oxk
