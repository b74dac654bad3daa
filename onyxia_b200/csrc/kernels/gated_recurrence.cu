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
//   recurrence_gates   convolution and gates of all tokens → a − 1 and sqrt(1 − a²) i u in f32 (`mma.sync`), and what
//                      each tile of 64 batch rows does to a state that enters it
//   recurrence_scan    128 batch rows × 32 channels per CTA: the state that enters them from the tiles before, then each
//                      warp scans 16 rows in registers and the warps' effects are chained through shared memory
//   recurrence_gates_simt, recurrence_tiles   the gates in f32 (and for block sizes that are not a multiple of 8)
//
// The first token of a sequence is stored as a = 0, b = its state after the token. The scan therefore runs over the
// rows of the whole batch and needs to know nothing of where sequences begin.
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
    float *te, *tb;         // [tiles of 64 rows, width]: the same of a whole tile
    void* out;              // [rows, width]
    ErrWord* err;
    long long rows, ld, x_off, y_off;
    int n_seqs, n_slots, width, blocks, n, taps, node;
    float decay, out_scale;
    int vec;                // columns and rows of x are 16-byte aligned
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
// Gate pre-activations (with bias) and u → a − 1 and sqrt(1 − a²) i u; `rate` = −decay · softplus(lam). A decay next to 1
// keeps its digits in a − 1; rounded to f32 itself it would be off by as much as 6e-8 of a state that lives for
// 1 / (1 − a) tokens.
__device__ __forceinline__ void gate_values(float rate, float zr, float zi, float u, float* e, float* b) {
    *e = expm1f(rate * sigmoid_f(zr));
    *b = sqrtf(-*e * (2.f + *e)) * sigmoid_f(zi) * u;
}
// The same to a few parts in a million, for u that was rounded to bf16. Near zero e^x − 1 is its Taylor polynomial
// (|x| < 0.35: the first term left out is below 2e-8 of the sum), elsewhere nothing cancels.
__device__ __forceinline__ void gate_values_fast(float rate, float zr, float zi, float u, float* e, float* b) {
    const float x = rate * sigmoid_fast(zr);
    float s = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
    s = fmaf(x, s, 1.f / 120.f);
    s = fmaf(x, s, 1.f / 24.f);
    s = fmaf(x, s, 1.f / 6.f);
    s = fmaf(x, s, 0.5f);
    s = fmaf(x * x, s, x);
    *e = x > -0.35f ? s : __expf(x) - 1.f;
    const float q = -*e * (2.f + *e);
    *b = q * rsqrtf(fmaxf(q, 1e-30f)) * sigmoid_fast(zi) * u;
}
// a S + b from e = a − 1; with a = 0 nothing of S remains, not even in the rounding
__device__ __forceinline__ float advance(float e, float S, float b) { return e == -1.f ? b : S + fmaf(e, S, b); }
// A sequence's first new token takes up the state it left: a = 0, b = the state after the token.
__device__ __forceinline__ void enter(const RecP& p, const SeqRow& s, int slot, int c, float* e, float* b) {
    if (s.past > 0) *b = advance(*e, p.state[(long long)slot * p.width + c], *b);
    *e = -1.f;
}

// Where the inputs of a token lie (channel 0; null: before the start), for up to kVecTaps taps.
constexpr int kVecTaps = 4;
struct ConvInputs {
    const bf16* back[kVecTaps];
};
__device__ __forceinline__ void find_inputs(const RecP& p, const SeqRow& s, int slot, int row, int pos, ConvInputs* in) {
#pragma unroll
    for (int back = 0; back < kVecTaps; back++) {
        const bf16* at = nullptr;
        if (back < p.taps && pos >= back)
            at = row - back >= s.start ? (const bf16*)p.proj + (long long)(row - back) * p.ld + p.x_off
                                       : (const bf16*)p.ring + ((long long)slot * p.taps + (pos - back) % p.taps) * p.width;
        in->back[back] = at;
    }
}
// Convolution of eight channels from `c` on, four tokens. The loads depend on no branch, so that they are in flight together.
__device__ __forceinline__ void conv4x8(const RecP& p, int c, const ConvInputs* in, float (&u)[4][8]) {
    uint4 x[4][kVecTaps];
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
        for (int back = 0; back < kVecTaps; back++) {
            const bf16* at = in[j].back[back];
            const uint4 v = *reinterpret_cast<const uint4*>((at ? at : (const bf16*)p.proj + p.x_off) + c);
            x[j][back] = at ? v : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
    for (int e = 0; e < 8; e++) {
        const float b = p.cb[c + e];
#pragma unroll
        for (int j = 0; j < 4; j++) u[j][e] = b;
    }
#pragma unroll
    for (int back = 0; back < kVecTaps; back++) {
        float w[8];
#pragma unroll
        for (int e = 0; e < 8; e++) w[e] = back < p.taps ? p.cw[(long long)(c + e) * p.taps + p.taps - 1 - back] : 0.f;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const unsigned v[4] = {x[j][back].x, x[j][back].y, x[j][back].z, x[j][back].w};
#pragma unroll
            for (int e = 0; e < 4; e++) {
                u[j][2 * e] = fmaf(__uint_as_float(v[e] << 16), w[2 * e], u[j][2 * e]);
                u[j][2 * e + 1] = fmaf(__uint_as_float(v[e] & 0xFFFF0000u), w[2 * e + 1], u[j][2 * e + 1]);
            }
        }
    }
}
__device__ __forceinline__ void store8(bf16* dst, const float (&u)[8], bool live) {
    const uint4 v = live ? make_uint4(pack_bf16(u[0], u[1]), pack_bf16(u[2], u[3]), pack_bf16(u[4], u[5]), pack_bf16(u[6], u[7])) : make_uint4(0, 0, 0, 0);
    *reinterpret_cast<uint4*>(dst) = v;
}

// ───────────────────────────── one token per sequence ───────────────────
// CTA: 16 sequences × 16 channels of one block. Warp w forms eight outputs of one gate: w & 1 picks the gate, w >> 1 the
// eight channels; a lane reads 16 consecutive bytes of a weight row, u is read with the same permutation of k.
__global__ void __launch_bounds__(128) recurrence_step(const RecP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float z[2][16][17];
    __shared__ SeqRow sq[16];
    __shared__ ConvInputs in[16];
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
    if (tid < 16) {  // no launch of a step writes the batch description
        SeqRow s{0, 0, 0, 0};
        if (r0 + tid < p.n_seqs) {
            s = load_seq(p.seqs, r0 + tid);
            s.slot = slot_of(p, s.slot);
        }
        sq[tid] = s;
        find_inputs(p, s, s.slot, s.start, r0 + tid < p.n_seqs ? s.past : -1, in + tid);
    }
    __syncthreads();
    const int live = min(16, p.n_seqs - r0);
    // what the end of the kernel needs: two (sequence, channel) pairs per thread; this layer's state is written by
    // no launch before this one
    const int oc = o0 + (tid & 15), ch = blk * n + (oc < n ? oc : 0);
    const float rate = -p.decay * softplus_f(p.lam[ch]), rb = p.rab[ch], ib = p.rib[ch];
    float old[2], y[2];
    bf16 x[2];
#pragma unroll
    for (int h = 0; h < 2; h++) old[h] = p.state[(long long)sq[(tid >> 4) + 8 * h].slot * p.width + ch];
    pdl_wait();
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const bf16* row = (const bf16*)p.proj + (long long)sq[(tid >> 4) + 8 * h].start * p.ld;
        y[h] = to_f(row[p.y_off + ch]);
        x[h] = row[p.x_off + ch];
    }
    if (p.vec) {  // eight channels of four sequences per thread and round
        for (int i = tid; i < 4 * kc * 4; i += 128) {
            const int k = (i % (kc * 4)) * 8, m0 = (i / (kc * 4)) * 4;
            float u[4][8];
            if (k < n) conv4x8(p, blk * n + k, in + m0, u);
#pragma unroll
            for (int j = 0; j < 4; j++) store8(us + (m0 + j) * stride + k, u[j], k < n && m0 + j < live);
        }
    } else {
        for (int i = tid; i < 16 * kc * 32; i += 128) {
            const int m = i / (kc * 32), k = i % (kc * 32), c = blk * n + k;
            float u = 0.f;
            if (m < live && k < n) u = conv_at<bf16>(p, sq[m], sq[m].slot, sq[m].start, sq[m].past, c);
            us[m * stride + k] = __float2bfloat16_rn(u);
        }
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
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int m = (tid >> 4) + 8 * h;
        if (m >= live || oc >= n) continue;
        const SeqRow s = sq[m];
        float e, b;
        gate_values_fast(rate, z[0][m][tid & 15] + rb, z[1][m][tid & 15] + ib, to_f(us[m * stride + oc]), &e, &b);
        const float S = s.past > 0 ? advance(e, old[h], b) : b;
        p.state[(long long)s.slot * p.width + ch] = S;
        ((bf16*)p.out)[(long long)s.start * p.width + ch] = __float2bfloat16_rn(S * gelu_tanh_fast(y[h]) * p.out_scale);
        // this position's ring row: no other CTA reads it (they look back taps − 1 positions at most)
        ((bf16*)p.ring)[((long long)s.slot * p.taps + s.past % p.taps) * p.width + ch] = x[h];
    }
}

// ───────────────────────────── gates of many tokens ─────────────────────
// CTA: 64 tokens × 64 channels of one block, k in chunks of 64.
constexpr int kTileRows = 64;
constexpr int kGateStride = 72;  // bf16 per row of a staged chunk: conflict-free ldmatrix
constexpr int kOutStride = 65;   // f32 per row of the results
struct GateSmem {
    union {
        struct {
            bf16 us[64 * kGateStride], wr[2][64 * kGateStride], wi[2][64 * kGateStride];
        } in;
        struct {
            float e[64 * kOutStride], b[64 * kOutStride];
        } out;
    };
    bf16 own[64 * 64];
    float rate[64], rb[64], ib[64];
    SeqRow sq[64];
    int pos[64];
    ConvInputs inputs[64];
};

// What the tile's rows do to a state that enters them, from the tile's results in shared memory.
__device__ __forceinline__ void tile_effect(const RecP& p, const float* e, const float* b, int stride, int rows, long long tile, int c0, int channels) {
    __shared__ float half[2][64];
    const int c = threadIdx.x & 63, h = threadIdx.x >> 6;
    float E = 0.f, B = 0.f;
    if (c < channels)
        for (int m = h * 32; m < min(rows, h * 32 + 32); m++) {
            E = advance(e[m * stride + c], E, e[m * stride + c]);
            B = advance(e[m * stride + c], B, b[m * stride + c]);
        }
    if (h == 0) {
        half[0][c] = E;
        half[1][c] = B;
    }
    __syncthreads();
    if (h == 1 && c < channels) {
        p.te[tile * p.width + c0 + c] = advance(E, half[0][c], E);
        p.tb[tile * p.width + c0 + c] = advance(E, half[1][c], B);
    }
}

__global__ void __launch_bounds__(128, 3) recurrence_gates(const RecP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    GateSmem& sm = *reinterpret_cast<GateSmem*>(smem);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int n = p.n, slices = (n + 63) / 64, blk = blockIdx.y / slices, o0 = (blockIdx.y % slices) * 64;
    const long long m0 = (long long)blockIdx.x * 64;
    auto load_weights = [&](int k0) {  // weight rows o0 … + 64, eight k per copy
        const int st = (k0 >> 6) & 1;
        for (int i = tid; i < 64 * 8; i += 128) {
            const int r = i >> 3, c = i & 7;
            const bool live = o0 + r < n && k0 + c * 8 < n;
            const long long off = live ? ((long long)blk * n + o0 + r) * n + k0 + c * 8 : 0;
            cp_async16(smem_u32(sm.in.wr[st] + r * kGateStride + c * 8), (const bf16*)p.ra + off, live);
            cp_async16(smem_u32(sm.in.wi[st] + r * kGateStride + c * 8), (const bf16*)p.ri + off, live);
        }
        cp_async_commit();
    };
    pdl_trigger();
    load_weights(0);  // constants: may overlap the launches before this one
    if (tid < 64) {
        const int c = blk * n + o0 + tid;
        const bool in = o0 + tid < n;
        sm.rate[tid] = in ? -p.decay * softplus_f(p.lam[c]) : 0.f;
        sm.rb[tid] = in ? p.rab[c] : 0.f;
        sm.ib[tid] = in ? p.rib[c] : 0.f;
    }
    pdl_wait();
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
        sm.sq[tid] = s;
        sm.pos[tid] = at;
        find_inputs(p, s, s.slot, (int)row, at, sm.inputs + tid);
    }
    __syncthreads();
    float ar[8][4], ai[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) ar[j][e] = ai[j][e] = 0.f;
    for (int k0 = 0; k0 < n; k0 += 64) {
        const int st = (k0 >> 6) & 1;
        if (p.vec) {  // eight channels of four tokens
            const int c = (tid & 7) * 8, m = (tid >> 3) * 4, k = k0 + c;
            float u[4][8];
            if (k < n) conv4x8(p, blk * n + k, sm.inputs + m, u);
#pragma unroll
            for (int j = 0; j < 4; j++) store8(sm.in.us + (m + j) * kGateStride + c, u[j], k < n && sm.pos[m + j] >= 0);
        } else {
            const int c = tid & 63, k = k0 + c;
            for (int m = tid >> 6; m < 64; m += 2) {
                float u = 0.f;
                if (k < n && sm.pos[m] >= 0) u = conv_at<bf16>(p, sm.sq[m], sm.sq[m].slot, (int)m0 + m, sm.pos[m], blk * n + k);
                sm.in.us[m * kGateStride + c] = __float2bfloat16_rn(u);
            }
        }
        cp_async_wait<0>();
        __syncthreads();
        if (k0 + 64 < n) load_weights(k0 + 64);  // the stage was read in the previous round
        if (k0 == o0)
            for (int i = tid; i < 64 * 8; i += 128)
                *reinterpret_cast<uint4*>(sm.own + (i >> 3) * 64 + (i & 7) * 8) = *reinterpret_cast<const uint4*>(sm.in.us + (i >> 3) * kGateStride + (i & 7) * 8);
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            unsigned a[4];
            ldmatrix_x4(a, smem_u32(sm.in.us + (warp * 16 + (lane & 15)) * kGateStride + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                const int at = (j * 8 + (lane & 7) + (lane >> 4) * 8) * kGateStride + kk * 16 + ((lane >> 3) & 1) * 8;
                unsigned b[4];
                ldmatrix_x4(b, smem_u32(sm.in.wr[st] + at));
                mma_bf16(ar[j], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(ar[j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                ldmatrix_x4(b, smem_u32(sm.in.wi[st] + at));
                mma_bf16(ai[j], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(ai[j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
        __syncthreads();
    }
    bool first = false;  // a sequence's portion starts in one of this thread's two rows
    float alive[2];
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int m = warp * 16 + g + 8 * r;
        alive[r] = sm.pos[m] >= 0 ? 1.f : 0.f;
        first |= sm.pos[m] >= 0 && sm.pos[m] == sm.sq[m].past;
    }
    // channels beyond the block have rate 0 and u 0: e = b = 0
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
        for (int v = 0; v < 2; v++) {
            const int k = j * 8 + t * 2 + v;
            const float rate = sm.rate[k], rb = sm.rb[k], ib = sm.ib[k];
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int m = warp * 16 + g + 8 * r;
                float e, b;
                gate_values_fast(rate * alive[r], ar[j][2 * r + v] + rb, ai[j][2 * r + v] + ib, to_f(sm.own[m * 64 + k]), &e, &b);
                sm.out.e[m * kOutStride + k] = e;
                sm.out.b[m * kOutStride + k] = b;
            }
        }
    if (first)
        for (int r = 0; r < 2; r++) {
            const int m = warp * 16 + g + 8 * r;
            if (sm.pos[m] < 0 || sm.pos[m] != sm.sq[m].past) continue;
            for (int i = 0; i < 16; i++) {
                const int k = (i >> 1) * 8 + t * 2 + (i & 1);
                if (o0 + k < n) enter(p, sm.sq[m], sm.sq[m].slot, blk * n + o0 + k, &sm.out.e[m * kOutStride + k], &sm.out.b[m * kOutStride + k]);
            }
        }
    __syncthreads();
    const int rows = (int)min((long long)64, p.rows - m0), channels = min(64, n - o0);
    for (int i = tid; i < rows * 64; i += 128) {
        const int m = i >> 6, k = i & 63;
        if (k < channels) {
            p.e[(m0 + m) * p.width + blk * n + o0 + k] = sm.out.e[m * kOutStride + k];
            p.b[(m0 + m) * p.width + blk * n + o0 + k] = sm.out.b[m * kOutStride + k];
        }
    }
    tile_effect(p, sm.out.e, sm.out.b, kOutStride, rows, blockIdx.x, blk * n + o0, channels);
}

// One CTA per (token, block).
template <typename T> __global__ void __launch_bounds__(128) recurrence_gates_simt(const RecP p) {
    extern __shared__ float uf[];
    pdl_enter();
    const int row = blockIdx.x, blk = blockIdx.y, n = p.n;
    const SeqRow s = load_seq(p.seqs, find_seq(p.seqs, p.n_seqs, row));
    const bool token = row < s.start + s.len;
    const int slot = slot_of(p, s.slot), pos = s.past + row - s.start;
    if (token)
        for (int k = threadIdx.x; k < n; k += 128) uf[k] = to_f(from_f<T>(conv_at<T>(p, s, slot, row, pos, blk * n + k)));
    __syncthreads();
    for (int k = threadIdx.x; k < n; k += 128) {
        const int c = blk * n + k;
        float e = 0.f, b = 0.f;
        if (token) {
            const T *wr = (const T*)p.ra + (long long)c * n, *wi = (const T*)p.ri + (long long)c * n;
            float zr = 0.f, zi = 0.f;
            for (int j = 0; j < n; j++) {
                zr = fmaf(uf[j], to_f(wr[j]), zr);
                zi = fmaf(uf[j], to_f(wi[j]), zi);
            }
            gate_values(-p.decay * softplus_f(p.lam[c]), zr + p.rab[c], zi + p.rib[c], uf[k], &e, &b);
            if (row == s.start) enter(p, s, slot, c, &e, &b);
        }
        p.e[(long long)row * p.width + c] = e;
        p.b[(long long)row * p.width + c] = b;
    }
}
// CTA: one tile of rows × 64 channels.
__global__ void __launch_bounds__(128) recurrence_tiles(const RecP p) {
    pdl_enter();
    const long long m0 = (long long)blockIdx.x * kTileRows, at = m0 * p.width + blockIdx.y * 64;
    tile_effect(p, p.e + at, p.b + at, p.width, (int)min((long long)kTileRows, p.rows - m0), blockIdx.x, (int)blockIdx.y * 64, min(64, p.width - (int)blockIdx.y * 64));
}

// ───────────────────────────── scan ─────────────────────────────────────
constexpr int kScanWarps = 8, kScanTokens = 16, kScanRows = kScanWarps * kScanTokens;
template <typename T> __global__ void __launch_bounds__(kScanWarps * 32) recurrence_scan(const RecP p) {
    __shared__ float pa[2][kScanWarps][32], pb[2][kScanWarps][32];
    __shared__ int state_slot[kScanRows], ring_row[kScanRows];  // where a row's state and input go, or −1
    pdl_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    const long long row0 = (long long)blockIdx.y * kScanRows, lo = row0 + warp * kScanTokens;
    const bool live = c < p.width;
    const T* proj = (const T*)p.proj;
    float e[kScanTokens], b[kScanTokens], y[kScanTokens];
#pragma unroll
    for (int j = 0; j < kScanTokens; j++) {
        const bool in = live && lo + j < p.rows;
        e[j] = in ? p.e[(lo + j) * p.width + c] : 0.f;
        b[j] = in ? p.b[(lo + j) * p.width + c] : 0.f;
        y[j] = in ? to_f(proj[(lo + j) * p.ld + p.y_off + c]) : 0.f;
    }
    // the tiles before these rows: each warp chains a contiguous share
    const int tiles = (int)(row0 / kTileRows), t0 = tiles * warp / kScanWarps, t1 = tiles * (warp + 1) / kScanWarps;
    float E = 0.f, B = 0.f;
#pragma unroll 4
    for (int i = t0; i < t1; i++) {
        const float te = live ? p.te[(long long)i * p.width + c] : 0.f, tb = live ? p.tb[(long long)i * p.width + c] : 0.f;
        E = advance(te, E, te);
        B = advance(te, B, tb);
    }
    pa[0][warp][lane] = E;
    pb[0][warp][lane] = B;
    if (threadIdx.x < kScanRows) {
        const long long row = row0 + threadIdx.x;
        int st = -1, rr = -1;
        if (row < p.rows) {
            const SeqRow s = load_seq(p.seqs, find_seq(p.seqs, p.n_seqs, (int)row));
            const int left = s.start + s.len - 1 - (int)row;
            if (left >= 0) {
                const int slot = slot_of(p, s.slot);
                if (left == 0) st = slot;
                if (left < p.taps) rr = slot * p.taps + (s.past + (int)row - s.start) % p.taps;
            }
        }
        state_slot[threadIdx.x] = st;
        ring_row[threadIdx.x] = rr;
    }
    E = B = 0.f;
#pragma unroll
    for (int j = 0; j < kScanTokens; j++) {
        E = advance(e[j], E, e[j]);
        B = advance(e[j], B, b[j]);
    }
    pa[1][warp][lane] = E;
    pb[1][warp][lane] = B;
    __syncthreads();
    float S = 0.f;
    for (int w = 0; w < kScanWarps; w++) S = advance(pa[0][w][lane], S, pb[0][w][lane]);
    for (int w = 0; w < warp; w++) S = advance(pa[1][w][lane], S, pb[1][w][lane]);
#pragma unroll
    for (int j = 0; j < kScanTokens; j++) {
        S = advance(e[j], S, b[j]);
        if (!live || lo + j >= p.rows) continue;
        ((T*)p.out)[(lo + j) * p.width + c] = from_f<T>(S * (sizeof(T) == 4 ? gelu_tanh_f(y[j]) : gelu_tanh_fast(y[j])) * p.out_scale);
        const int st = state_slot[warp * kScanTokens + j], rr = ring_row[warp * kScanTokens + j];
        if (st >= 0) p.state[(long long)st * p.width + c] = S;
        if (rr >= 0) ((T*)p.ring)[(long long)rr * p.width + c] = proj[(lo + j) * p.ld + p.x_off + c];
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
    p.vec = d.taps <= kVecTaps && d.width % 8 == 0 && p.ld % 8 == 0 && d.x_off % 8 == 0 && proj.buf.off % 16 == 0;
    p.decay = (float)d.decay;
    p.out_scale = (float)d.out_scale;
    p.node = em.node;
    const bool bf = proj.dtype == DT_BF16, tc = bf && p.n % 8 == 0;
    const int kc = (p.n + 31) / 32;
    const unsigned step_smem = 16u * (unsigned)(kc * 32 + (kc & 1 ? 0 : 32)) * 2u;
    const bool step = tc && rows == n_seqs && step_smem <= 200 * 1024;
    const Buf none{kSlotNull, 0};
    const Buf e = step ? none : em.scratch((size_t)rows * d.width * 4), b = step ? none : em.scratch((size_t)rows * d.width * 4);
    const int64_t tiles = (rows + kTileRows - 1) / kTileRows;
    const Buf te = step ? none : em.scratch((size_t)tiles * d.width * 4), tb = step ? none : em.scratch((size_t)tiles * d.width * 4);
    auto launch = [&](void (*k)(const RecP), dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.cw, conv_w.buf}, {&p.cb, conv_b.buf}, {&p.ra, ra.buf}, {&p.ri, ri.buf}, {&p.rab, ra_b.buf}, {&p.rib, ri_b.buf},
                   {&p.lam, lam.buf}, {&p.ring, conv_state.buf}, {&p.state, state.buf}, {&p.seqs, seqs.buf}, {&p.e, e}, {&p.b, b}, {&p.te, te}, {&p.tb, tb}, {&p.out, out.buf},
                   {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    if (step) {
        ensure_max_dynamic_smem((const void*)recurrence_step, 200 * 1024);
        launch(recurrence_step, dim3((unsigned)(p.blocks * ((p.n + 15) / 16)), (unsigned)((n_seqs + 15) / 16)), 128, step_smem, "recurrence_step");
        return;
    }
    if (tc) {
        ensure_max_dynamic_smem((const void*)recurrence_gates, (int)sizeof(GateSmem));
        launch(recurrence_gates, dim3((unsigned)tiles, (unsigned)(p.blocks * ((p.n + 63) / 64))), 128, sizeof(GateSmem), "recurrence_gates");
    } else {
        const auto k = bf ? recurrence_gates_simt<bf16> : recurrence_gates_simt<float>;
        ensure_max_dynamic_smem((const void*)k, 200 * 1024);
        launch(k, dim3((unsigned)rows, (unsigned)p.blocks), 128, (unsigned)p.n * 4, "recurrence_gates_simt");
        launch(recurrence_tiles, dim3((unsigned)tiles, (unsigned)((d.width + 63) / 64)), 128, 0, "recurrence_tiles");
    }
    launch(bf ? recurrence_scan<bf16> : recurrence_scan<float>, dim3((unsigned)((d.width + 31) / 32), (unsigned)((rows + kScanRows - 1) / kScanRows)),
           kScanWarps * 32, 0, "recurrence_scan");
}

}  // namespace oxk
