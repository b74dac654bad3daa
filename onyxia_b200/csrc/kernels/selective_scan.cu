// Selective scan (the recurrence of "Mamba: Linear-Time Sequence Modeling with Selective State Spaces", Gu and Dao) over a ragged
// batch with per-slot state.
//
//   u = silu(conv(x))                              per channel, `taps` taps, inputs before the start are zero
//   (dt, B, C) = W_x u,  dt = softplus(W_dt dt + b)
//   S[c, n] ← exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n,   y_c = Σ_n S[c, n] C_n + D_c u_c,   out = y · z
//
// x and z are columns of a fused projection (z with its silu). The state of a sequence is S (f32) and a ring of its last inputs
// (row = position modulo taps); a sequence at position 0 reads neither, so slots need no clearing.
//
//   short_conv    (short_conv.cu) u of all tokens
//   products      (linear.cu) W_x u; W_dt dt over a column range of it, softplus behind it, in f32
//   scan_step     every sequence has one new token: dt, state and results in one launch (bf16)
//   scan_serial   a sequence × some channels per CTA, token after token: the states of a channel in a few lanes, whose shares of the
//                 results are added for many tokens at once (bf16)
//   scan_tokens   any size, f32: a tile of consecutive tokens of one sequence × some channels per CTA. Two forms: the state that a
//                 tile leaves when it starts from zero, and the results from the state that enters the tile; scan_chain forms the
//                 states that enter
//
// Bytes per token and channel: 4 + 2 + 2 read, 2 written, 8 · states of state per sequence. A power per token, channel and
// state: 16 a clock and multiprocessor bound the kernels over many tokens (tiles need every one twice).
#include <type_traits>

#include "paged_util.cuh"

namespace oxk {

namespace {

constexpr int kScanThreads = 128, kScanSub = 16;  // tokens whose B and C are staged together

struct ScanP {
    const void* proj;             // [rows, ld]
    void* u;                      // [rows, width]
    const void* bc;               // [rows, rank + 2 · state]
    const float *dt, *A, *D;      // [rows, width], [width, state], [width]
    const void* wdt;              // [width, rank]
    const float* dt_b;            // [width]
    void* ring;                   // [slots, taps, width]
    float* state;                 // [slots, width, state]
    float *carry, *sum;           // [tiles, width, state], [tiles, width]: a tile's state, its sum of dt
    const int* seqs;
    void* out;                    // [rows, width]
    ErrWord* err;
    long long rows, ld, x_off, z_off;
    int n_seqs, n_slots, width, states, rank, taps, tile, lanes, node;
};

__device__ __forceinline__ int slot_of(const ScanP& p, int slot) {
    if ((unsigned)slot >= (unsigned)p.n_slots) {
        report(p.err, ERR_GATHER_OOB, p.node, slot, p.n_slots);
        return 0;
    }
    return slot;
}

// ───────────────────────────── scan ─────────────────────────────────────
// 2^x, a few parts in ten million
__device__ __forceinline__ float power2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// exp(dt A) S + b. In 32-bit through e^x − 1: a decay next to 1 that is itself rounded would be off by up to 6e-8 of a state that
// lives for many tokens.
template <bool EXACT> __device__ __forceinline__ float advance(float dt, float A, float S, float b) {
    if constexpr (EXACT) return S + fmaf(expm1f(dt * A), S, b);
    else return fmaf(power2(dt * A), S, b);  // A carries log2 e
}

// A sequence's last inputs go to its ring.
template <typename T> __device__ __forceinline__ void keep_input(const ScanP& p, const SeqRow& sq, int slot, int at, int c, const T* x) {
    if (sq.len - at <= p.taps) ((T*)p.ring)[((long long)slot * p.taps + (sq.past + at) % p.taps) * p.width + c] = *x;
}

__device__ __forceinline__ float4 widen4(uint2 v) {
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
}

// Every sequence has one new token. Grid: (channel blocks, shares of the sequences, taken kStepSeqs at a time). Four states of a channel per
// lane. OWN: the channel's lanes also share the dot product that makes dt; otherwise it is there already.
constexpr int kStepSeqs = 4, kStepWeights = 6, kStepAhead = 2, kStepCtas = 6;
template <int G, bool OWN> __global__ void __launch_bounds__(kScanThreads, OWN ? 4 : kStepCtas) scan_step(const ScanP p) {
    const int tid = threadIdx.x, sub = tid % G, c = blockIdx.x * (kScanThreads / G) + tid / G, n0 = sub * 4, ld_bc = p.rank + 2 * p.states;
    const bool live = c < p.width, mine = n0 < p.states;
    const int cc = live ? c : 0;
    pdl_trigger();
    // constants, the batch description and the states of earlier steps: may be read while the launches before this one finish. The
    // states come kStepAhead rounds ahead, each into a place that only its own thread looks at.
    __shared__ __align__(16) float4 ring[kStepAhead + 1][kStepSeqs][kScanThreads];
    auto state_at = [&](int slot) { return p.state + ((long long)slot * p.width + cc) * p.states + n0; };
    const int stride = (int)gridDim.y * kStepSeqs;
    auto ask = [&](int s0, int stage) {
#pragma unroll
        for (int j = 0; j < kStepSeqs; j++) {
            const SeqRow sq = load_seq(p.seqs, min(s0 + j, p.n_seqs - 1));
            const bool in = s0 < p.n_seqs && mine && sq.past > 0;
            cp_async16(smem_u32(&ring[stage][j][tid]), in ? state_at(slot_of(p, sq.slot)) : p.state, in);  // (zeros where there is none)
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < kStepAhead; i++) ask(blockIdx.y * kStepSeqs + i * stride, i);
    float4 A = make_float4(0.f, 0.f, 0.f, 0.f);
    if (mine) A = *reinterpret_cast<const float4*>(p.A + (long long)cc * p.states + n0);
    const float D = p.D[cc], bias = p.dt_b[cc];
    const bf16* w = (const bf16*)p.wdt + (long long)cc * p.rank;
    uint4 wv[OWN ? kStepWeights : 1];
    if constexpr (OWN)
#pragma unroll
        for (int k = 0; k < kStepWeights; k++) {
            const int r = (k * G + sub) * 8;
            wv[k] = r < p.rank ? __ldg(reinterpret_cast<const uint4*>(w + r)) : make_uint4(0, 0, 0, 0);
        }
    pdl_wait();
    int stage = 0;
    for (int s0 = blockIdx.y * kStepSeqs; s0 < p.n_seqs; s0 += stride) {
        SeqRow r[kStepSeqs];
        float4 S[kStepSeqs];
        float dt[kStepSeqs];
        bf16 u[kStepSeqs], z[kStepSeqs], x[kStepSeqs];
        uint2 B[kStepSeqs], C[kStepSeqs];
#pragma unroll
        for (int j = 0; j < kStepSeqs; j++) {
            r[j] = load_seq(p.seqs, min(s0 + j, p.n_seqs - 1));
            r[j].slot = slot_of(p, r[j].slot);
            const long long row = r[j].start;
            u[j] = ((const bf16*)p.u)[row * p.width + cc];
            z[j] = ((const bf16*)p.proj)[row * p.ld + p.z_off + cc];
            x[j] = ((const bf16*)p.proj)[row * p.ld + p.x_off + cc];
            const bf16* bc = (const bf16*)p.bc + row * ld_bc + p.rank + (mine ? n0 : 0);
            B[j] = *reinterpret_cast<const uint2*>(bc);
            C[j] = mine ? *reinterpret_cast<const uint2*>(bc + p.states) : make_uint2(0, 0);
            dt[j] = OWN ? 0.f : p.dt[row * p.width + cc];
        }
        ask(s0 + kStepAhead * stride, stage == 0 ? kStepAhead : stage - 1);  // the round before this one had it
        cp_async_wait<kStepAhead>();
#pragma unroll
        for (int j = 0; j < kStepSeqs; j++) S[j] = ring[stage][j][tid];
        stage = stage == kStepAhead ? 0 : stage + 1;
        if constexpr (OWN) {
            auto dot8 = [](float acc, uint4 a, uint4 b) {
                const unsigned x[4] = {a.x, a.y, a.z, a.w}, y[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    acc = fmaf(__uint_as_float(x[e] << 16), __uint_as_float(y[e] << 16), acc);
                    acc = fmaf(__uint_as_float(x[e] & 0xFFFF0000u), __uint_as_float(y[e] & 0xFFFF0000u), acc);
                }
                return acc;
            };
            auto low = [&](int j, int k) { return *reinterpret_cast<const uint4*>((const bf16*)p.bc + (long long)r[j].start * ld_bc + k); };
#pragma unroll
            for (int k = 0; k < kStepWeights; k++) {
                const int i = (k * G + sub) * 8;
                if (i < p.rank)
#pragma unroll
                    for (int j = 0; j < kStepSeqs; j++) dt[j] = dot8(dt[j], wv[k], low(j, i));
            }
            for (int i = (kStepWeights * G + sub) * 8; i < p.rank; i += G * 8) {
                const uint4 more = __ldg(reinterpret_cast<const uint4*>(w + i));
#pragma unroll
                for (int j = 0; j < kStepSeqs; j++) dt[j] = dot8(dt[j], more, low(j, i));
            }
#pragma unroll
            for (int j = 0; j < kStepSeqs; j++) {
#pragma unroll
                for (int o = 1; o < G; o <<= 1) dt[j] += __shfl_xor_sync(0xffffffffu, dt[j], o);
                dt[j] = softplus_fast(dt[j] + bias);
            }
        }
        float y[kStepSeqs];
#pragma unroll
        for (int j = 0; j < kStepSeqs; j++) {
            const float4 b = widen4(B[j]), k = widen4(C[j]);
            const float dx = dt[j] * to_f(u[j]), e = dt[j] * kLog2e;
            S[j].x = fmaf(power2(e * A.x), S[j].x, dx * b.x);
            S[j].y = fmaf(power2(e * A.y), S[j].y, dx * b.y);
            S[j].z = fmaf(power2(e * A.z), S[j].z, dx * b.z);
            S[j].w = fmaf(power2(e * A.w), S[j].w, dx * b.w);
            y[j] = fmaf(S[j].x, k.x, fmaf(S[j].y, k.y, fmaf(S[j].z, k.z, S[j].w * k.w)));
        }
#pragma unroll
        for (int o = 1; o < G; o <<= 1)
#pragma unroll
            for (int j = 0; j < kStepSeqs; j++) y[j] += __shfl_xor_sync(0xffffffffu, y[j], o);
#pragma unroll
        for (int j = 0; j < kStepSeqs; j++) {
            if (!live || s0 + j >= p.n_seqs) continue;
            if (mine) *reinterpret_cast<float4*>(state_at(r[j].slot)) = S[j];
            if (sub == 0) {
                ((bf16*)p.out)[(long long)r[j].start * p.width + c] = __float2bfloat16_rn(fmaf(D, to_f(u[j]), y[j]) * to_f(z[j]));
                ((bf16*)p.ring)[((long long)r[j].slot * p.taps + r[j].past % p.taps) * p.width + c] = x[j];
            }
        }
    }
}

// Two f32 lanes of one register pair
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(reinterpret_cast<unsigned long long&>(r)) : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)));
    return r;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(reinterpret_cast<unsigned long long&>(r))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)), "l"(reinterpret_cast<const unsigned long long&>(c)));
    return r;
}

// Grid: (channel blocks, sequences). P pairs of states per lane, G lanes per channel. One half of a CTA's warps computes, a tile of
// tokens after the other; the other half brings the next tile into shared memory and finishes the results of the one before.
// B and C stay bf16 there, two in a word: its bandwidth is what a lane's states share.
template <int P, int G> struct SerialShape {
    static constexpr int states = 2 * P * G, threads = G <= 8 ? 32 : 4 * G, channels = threads / G, tokens = 32;  // threads of a half
    static constexpr int batch = 16, lanes = G < 16 ? G : 16, kept = batch / lanes;  // tokens whose results are added together
    static constexpr int quads = tokens * channels / 4, quads_per_thread = (quads + threads - 1) / threads;
    static constexpr int eights = tokens * states / 8, eights_per_thread = (eights + threads - 1) / threads;
};
template <int P, int G> __global__ void __launch_bounds__(2 * SerialShape<P, G>::threads) scan_serial(const ScanP p) {
    using L = SerialShape<P, G>;
    constexpr int TT = L::tokens, CH = L::channels, NS = L::states, TB = L::batch, Q = CH / 4, E = NS / 8;
    __shared__ __align__(16) float dts[2][TT][CH], dxs[2][TT][CH];  // dt, dt u
    __shared__ __align__(16) unsigned bc[2][TT][NS];                // B above C
    __shared__ __align__(16) float ys[2][TT][CH];
    __shared__ __align__(16) uint4 uz[3][TT][Q];                    // u and z of four channels
    pdl_enter();
    bool computes = threadIdx.x < L::threads;
    if constexpr (L::threads == 32) {
        // Warps with consecutive numbers lie on consecutive schedulers: of the CTAs on a multiprocessor, the first and third pair
        // and the second and fourth pair should not compute on the same ones. (The number is a hint, nothing hangs on it.)
        __shared__ int swap;
        unsigned w;
        asm volatile("mov.u32 %0, %%warpid;" : "=r"(w));
        if (threadIdx.x == 0) swap = (w & 1) != (w >> 2 & 1);
        __syncthreads();
        computes = computes != (swap != 0);
    }
    const int tid = threadIdx.x % L::threads, sub = tid % G, cl = tid / G, c0 = blockIdx.x * CH, c = c0 + cl;
    const SeqRow sq = load_seq(p.seqs, blockIdx.y);
    const int slot = slot_of(p, sq.slot), ld_bc = p.rank + 2 * p.states, tiles = (sq.len + TT - 1) / TT;
    if (!computes) {
        float4 nd[L::quads_per_thread];
        uint2 nu[L::quads_per_thread], nz[L::quads_per_thread];
        uint4 nb[L::eights_per_thread], nc[L::eights_per_thread];
        auto fetch = [&](int t0) {
#pragma unroll
            for (int i = 0; i < L::quads_per_thread; i++) {
                const int k = i * L::threads + tid, t = t0 + k / Q, ch = c0 + k % Q * 4;
                const long long row = sq.start + t;
                const bool in = k < L::quads && t < sq.len && ch < p.width;  // tokens beyond the end have dt = 0: the state stays as it is
                nd[i] = in ? *reinterpret_cast<const float4*>(p.dt + row * p.width + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
                nu[i] = in ? *reinterpret_cast<const uint2*>((const bf16*)p.u + row * p.width + ch) : make_uint2(0, 0);
                nz[i] = in ? *reinterpret_cast<const uint2*>((const bf16*)p.proj + row * p.ld + p.z_off + ch) : make_uint2(0, 0);
            }
#pragma unroll
            for (int i = 0; i < L::eights_per_thread; i++) {
                const int k = i * L::threads + tid, t = t0 + k / E, n = k % E * 8;
                const bool in = k < L::eights && t < sq.len && n < p.states;
                const bf16* from = (const bf16*)p.bc + (in ? (long long)(sq.start + t) * ld_bc + p.rank + n : 0);
                nb[i] = in ? *reinterpret_cast<const uint4*>(from) : make_uint4(0, 0, 0, 0);
                nc[i] = in ? *reinterpret_cast<const uint4*>(from + p.states) : make_uint4(0, 0, 0, 0);
            }
        };
        auto store = [&](int tile) {
            const int buf = tile & 1;
#pragma unroll
            for (int i = 0; i < L::quads_per_thread; i++) {
                const int k = i * L::threads + tid;
                if (k >= L::quads) continue;
                const float4 v = widen4(nu[i]), d = nd[i];
                uz[tile % 3][k / Q][k % Q] = make_uint4(nu[i].x, nu[i].y, nz[i].x, nz[i].y);
                *reinterpret_cast<float4*>(&dts[buf][k / Q][k % Q * 4]) = d;
                *reinterpret_cast<float4*>(&dxs[buf][k / Q][k % Q * 4]) = make_float4(d.x * v.x, d.y * v.y, d.z * v.z, d.w * v.w);
            }
#pragma unroll
            for (int i = 0; i < L::eights_per_thread; i++) {
                const int k = i * L::threads + tid;
                if (k >= L::eights) continue;
                unsigned* to = &bc[buf][k / E][k % E * 8];
                auto two = [](unsigned b, unsigned c) { return make_uint2(__byte_perm(c, b, 0x5410), __byte_perm(c, b, 0x7632)); };
                const uint2 w0 = two(nb[i].x, nc[i].x), w1 = two(nb[i].y, nc[i].y), w2 = two(nb[i].z, nc[i].z), w3 = two(nb[i].w, nc[i].w);
                *reinterpret_cast<uint4*>(to) = make_uint4(w0.x, w0.y, w1.x, w1.y);
                *reinterpret_cast<uint4*>(to + 4) = make_uint4(w2.x, w2.y, w3.x, w3.y);
            }
        };
        fetch(0);
        store(0);
        fetch(TT);
        __syncthreads();
        for (int k = 0; k <= tiles; k++) {
            const int t0 = (k - 1) * TT;  // of the tile whose results are there
            if (k + 1 < tiles) {
                store(k + 1);
                fetch((k + 2) * TT);
            }
#pragma unroll
            for (int i = 0; i < L::quads_per_thread; i++) {
                const int q = i * L::threads + tid, t = t0 + q / Q, ch = c0 + q % Q * 4;
                if (q >= L::quads || k == 0 || t >= sq.len || ch >= p.width) continue;
                const long long row = sq.start + t;
                const uint4 raw = uz[(k - 1) % 3][q / Q][q % Q];
                const float4 y = *reinterpret_cast<const float4*>(&ys[(k - 1) & 1][q / Q][q % Q * 4]), v = widen4(make_uint2(raw.x, raw.y)), f = widen4(make_uint2(raw.z, raw.w));
                const float4 D = *reinterpret_cast<const float4*>(p.D + ch);
                *reinterpret_cast<uint2*>((bf16*)p.out + row * p.width + ch) =
                    make_uint2(pack_bf16(fmaf(D.x, v.x, y.x) * f.x, fmaf(D.y, v.y, y.y) * f.y), pack_bf16(fmaf(D.z, v.z, y.z) * f.z, fmaf(D.w, v.w, y.w) * f.w));
                if (sq.len - t <= p.taps)
                    for (int e = 0; e < 4; e++) keep_input(p, sq, slot, t, ch + e, (const bf16*)p.proj + row * p.ld + p.x_off + ch + e);
            }
            __syncthreads();
        }
        return;
    }
    // pair k of this lane: states (sub · P + k) · 2 and the next one
    float2 A[P], S[P];
    const long long at = ((long long)slot * p.width + c) * p.states;
#pragma unroll
    for (int k = 0; k < P; k++) {
        const int n = (sub * P + k) * 2;
        const bool in = c < p.width && n < p.states;  // (their number is even)
        A[k] = in ? *reinterpret_cast<const float2*>(p.A + (long long)c * p.states + n) : make_float2(0.f, 0.f);
        S[k] = in && sq.past > 0 ? *reinterpret_cast<const float2*>(p.state + at + n) : make_float2(0.f, 0.f);
        A[k].x *= kLog2e;
        A[k].y *= kLog2e;
    }
    __syncthreads();
    for (int tile = 0; tile < tiles; tile++) {
        const int buf = tile & 1;
#pragma unroll 1
        for (int b = 0; b < TT; b += TB) {
            // the powers and inputs of four tokens are formed while the state takes up the four before them: a warp is often alone on its
            // scheduler and has to cover the latencies itself
            constexpr int TQ = 4;
            float y[TB];
            float2 pw[2][TQ][P], in[2][TQ][P], cv[2][TQ][P];
            auto prepare = [&](int j0, int half) {
                float dt[TQ], dx[TQ];
                unsigned word[TQ][2 * P];
#pragma unroll
                for (int j = 0; j < TQ; j++) {
                    dt[j] = dts[buf][b + j0 + j][cl];
                    dx[j] = dxs[buf][b + j0 + j][cl];
                    const unsigned* w = &bc[buf][b + j0 + j][sub * 2 * P];
                    if constexpr (P == 1) *reinterpret_cast<uint2*>(word[j]) = *reinterpret_cast<const uint2*>(w);
                    else
#pragma unroll
                        for (int k = 0; k < 2 * P; k += 4) *reinterpret_cast<uint4*>(word[j] + k) = *reinterpret_cast<const uint4*>(w + k);
                }
#pragma unroll
                for (int j = 0; j < TQ; j++)
#pragma unroll
                    for (int k = 0; k < P; k++) pw[half][j][k] = mul2(make_float2(dt[j], dt[j]), A[k]);
#pragma unroll
                for (int j = 0; j < TQ; j++)
#pragma unroll
                    for (int k = 0; k < P; k++) pw[half][j][k] = make_float2(power2(pw[half][j][k].x), power2(pw[half][j][k].y));
#pragma unroll
                for (int j = 0; j < TQ; j++)
#pragma unroll
                    for (int k = 0; k < P; k++) {
                        in[half][j][k] = mul2(make_float2(dx[j], dx[j]), make_float2(__uint_as_float(word[j][2 * k] & 0xFFFF0000u), __uint_as_float(word[j][2 * k + 1] & 0xFFFF0000u)));
                        cv[half][j][k] = make_float2(__uint_as_float(word[j][2 * k] << 16), __uint_as_float(word[j][2 * k + 1] << 16));
                    }
            };
            prepare(0, 0);
#pragma unroll
            for (int j0 = 0; j0 < TB; j0 += TQ) {
                const int half = j0 / TQ & 1;
                if (j0 + TQ < TB) prepare(j0 + TQ, half ^ 1);
#pragma unroll
                for (int j = 0; j < TQ; j++) {
                    float2 acc;
#pragma unroll
                    for (int k = 0; k < P; k++) {
                        S[k] = fma2(pw[half][j][k], S[k], in[half][j][k]);
                        acc = k == 0 ? mul2(S[k], cv[half][j][k]) : fma2(S[k], cv[half][j][k], acc);
                    }
                    y[j0 + j] = acc.x + acc.y;
                    if constexpr (G == 32) y[j0 + j] += __shfl_xor_sync(0xffffffffu, y[j0 + j], 16);
                }
            }
            // every step halves the tokens of a lane and doubles the lanes that a sum runs over: lane l ends up with tokens
            // l · kept … of the batch
#pragma unroll
            for (int o = L::lanes / 2, n = TB / 2; o > 0; o >>= 1, n >>= 1)
#pragma unroll
                for (int j = 0; j < n; j++) {
                    const bool up = sub & o;
                    const float give = up ? y[j] : y[j + n], keep = up ? y[j + n] : y[j];
                    y[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                }
            if (sub < L::lanes)
#pragma unroll
                for (int j = 0; j < L::kept; j++) ys[buf][b + sub * L::kept + j][cl] = y[j];
        }
        __syncthreads();
    }
    __syncthreads();  // the other half's last round
    if (c >= p.width) return;
#pragma unroll
    for (int k = 0; k < P; k++) {
        const int n = (sub * P + k) * 2;
        if (n < p.states) *reinterpret_cast<float2*>(p.state + at + n) = S[k];
    }
}

// Grid: (channel blocks, tiles). A channel's states lie in `lanes` neighbouring lanes, NS in each. LOCAL: from zero, leaves the
// tile's state and its sum of dt; otherwise from the state that enters, leaves results, state and ring.
template <typename T, int NS, bool LOCAL> __global__ void __launch_bounds__(kScanThreads) scan_tokens(const ScanP p) {
    extern __shared__ __align__(16) float bc_s[];  // [kScanSub][2][lanes · NS]
    constexpr bool EXACT = sizeof(T) == 4;
    constexpr int kAhead = 4;  // tokens whose inputs are loaded together
    pdl_enter();
    const int tid = threadIdx.x, G = p.lanes, padded = G * NS, c = blockIdx.x * (kScanThreads / G) + tid / G, n0 = (tid % G) * NS;
    int seq, first;
    if (!locate_tile(p.seqs, p.n_seqs, (int)blockIdx.y, p.tile, &seq, &first, 1)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int n = min(p.tile, sq.len - first), slot = slot_of(p, sq.slot);
    if (LOCAL && first + n == sq.len) return;  // nobody asks what the last tile leaves
    const bool live = c < p.width;
    const int cc = live ? c : 0;
    alignas(16) float A[NS], S[NS];
    const bool whole = p.states % NS == 0 && NS % 4 == 0;
    auto read = [&](const float* from, float* to) {  // this thread's states of a [width, states] array
        from += (long long)cc * p.states + n0;
        if (whole && n0 < p.states) {
#pragma unroll
            for (int i = 0; i < NS; i += 4) *reinterpret_cast<float4*>(to + i) = *reinterpret_cast<const float4*>(from + i);
        } else {
#pragma unroll
            for (int i = 0; i < NS; i++) to[i] = n0 + i < p.states ? from[i] : 0.f;
        }
    };
    auto write = [&](float* to) {
        if (!live) return;
        to += (long long)c * p.states + n0;
        if (whole && n0 < p.states) {
#pragma unroll
            for (int i = 0; i < NS; i += 4) *reinterpret_cast<float4*>(to + i) = *reinterpret_cast<const float4*>(S + i);
        } else {
#pragma unroll
            for (int i = 0; i < NS; i++)
                if (n0 + i < p.states) to[i] = S[i];
        }
    };
    read(p.A, A);
    if (!EXACT)
#pragma unroll
        for (int i = 0; i < NS; i++) A[i] *= kLog2e;
    const long long per_slot = (long long)p.width * p.states;
    if (LOCAL || (sq.len <= p.tile && sq.past == 0)) {
#pragma unroll
        for (int i = 0; i < NS; i++) S[i] = 0.f;
    } else if (sq.len <= p.tile) {
        read(p.state + slot * per_slot, S);
    } else {
        read(p.carry + blockIdx.y * per_slot, S);
    }
    const float D = LOCAL ? 0.f : p.D[cc];
    const long long row0 = sq.start + first;
    const T *x = (const T*)p.proj + p.x_off + cc, *z = (const T*)p.proj + p.z_off + cc, *u = (const T*)p.u + cc;
    const int ld_bc = p.rank + 2 * p.states;
    float total = 0.f;
    for (int t0 = 0; t0 < n; t0 += kScanSub) {
        const int m = min(kScanSub, n - t0);
        __syncthreads();
        for (int i = tid; i < m * 2 * padded; i += kScanThreads) {
            const int t = i / (2 * padded), k = i % (2 * padded), which = k >= padded, s = k - which * padded;
            bc_s[i] = s < p.states ? to_f(((const T*)p.bc)[(row0 + t0 + t) * ld_bc + p.rank + which * p.states + s]) : 0.f;
        }
        __syncthreads();
        for (int t1 = 0; t1 < m; t1 += kAhead) {
            float dt[kAhead], uv[kAhead], zv[kAhead], y[kAhead];
#pragma unroll
            for (int j = 0; j < kAhead; j++) {
                const long long row = row0 + t0 + min(t1 + j, m - 1);
                dt[j] = t1 + j < m ? p.dt[row * p.width + cc] : 0.f;
                uv[j] = to_f(u[row * p.width]);
                zv[j] = LOCAL ? 0.f : to_f(z[row * p.ld]);
            }
#pragma unroll
            for (int j = 0; j < kAhead; j++) {
                y[j] = 0.f;
                if (t1 + j >= m) break;
                const float* B = bc_s + (t1 + j) * 2 * padded + n0;
                const float dx = dt[j] * uv[j];
                if (LOCAL) total += dt[j];
#pragma unroll
                for (int i = 0; i < NS; i++) {
                    S[i] = advance<EXACT>(dt[j], A[i], S[i], dx * B[i]);
                    if (!LOCAL) y[j] = fmaf(S[i], B[padded + i], y[j]);
                }
            }
            if constexpr (!LOCAL) {
                for (int o = 1; o < G; o <<= 1)
#pragma unroll
                    for (int j = 0; j < kAhead; j++) y[j] += __shfl_xor_sync(0xffffffffu, y[j], o);
                if (live && tid % G == 0)
#pragma unroll
                    for (int j = 0; j < kAhead; j++) {
                        if (t1 + j >= m) break;
                        const long long row = row0 + t0 + t1 + j;
                        ((T*)p.out)[row * p.width + c] = from_f<T>(fmaf(D, uv[j], y[j]) * zv[j]);
                        keep_input(p, sq, slot, first + t0 + t1 + j, c, x + row * p.ld);
                    }
            }
        }
    }
    if constexpr (LOCAL) {
        write(p.carry + blockIdx.y * per_slot);
        if (live && tid % G == 0) p.sum[(long long)blockIdx.y * p.width + c] = total;
    } else if (first + n == sq.len) {
        write(p.state + slot * per_slot);
    }
}

// Grid: (blocks of states, sequences). In place: a tile's own state becomes the state that enters it.
template <bool EXACT> __global__ void __launch_bounds__(256) scan_chain(const ScanP p) {
    constexpr int kAhead = 8;
    pdl_enter();
    const int seq = blockIdx.y, lane = threadIdx.x & 31;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int tiles = (sq.len + p.tile - 1) / p.tile;
    if (tiles <= 1) return;
    int before = 0;
    for (int r = lane; r < seq; r += 32) before += (p.seqs[4 * r + 1] + p.tile - 1) / p.tile;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
    const long long per_slot = (long long)p.width * p.states, i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= per_slot) return;
    const int c = (int)(i / p.states);
    const float A = p.A[i];
    float S = sq.past > 0 ? p.state[slot_of(p, sq.slot) * per_slot + i] : 0.f;
    float* at = p.carry + before * per_slot + i;
    const float* sum = p.sum + (long long)before * p.width + c;
    for (int t0 = 0; t0 < tiles; t0 += kAhead) {
        float own[kAhead], a[kAhead];
#pragma unroll
        for (int j = 0; j < kAhead; j++) {
            const bool in = t0 + j < tiles - 1;  // the last tile has left nothing
            own[j] = in ? at[(t0 + j) * per_slot] : 0.f;
            a[j] = in ? sum[(long long)(t0 + j) * p.width] * A : 0.f;
        }
#pragma unroll
        for (int j = 0; j < kAhead; j++) {
            if (t0 + j >= tiles) break;
            at[(t0 + j) * per_slot] = S;
            S = EXACT ? S + fmaf(expm1f(a[j]), S, own[j]) : fmaf(expf(a[j]), S, own[j]);
        }
    }
}

using ScanKernel = void (*)(const ScanP);
template <typename T> ScanKernel token_kernel(int ns, bool local) {
    if (local) return ns == 4 ? scan_tokens<T, 4, true> : ns == 8 ? scan_tokens<T, 8, true> : scan_tokens<T, 16, true>;
    return ns == 4 ? scan_tokens<T, 4, false> : ns == 8 ? scan_tokens<T, 8, false> : scan_tokens<T, 16, false>;
}

}  // namespace

void emit_selective_scan(Emitter& em, const SelectiveScanDesc& d, const TRef& proj, const TRef& conv_w, const TRef& conv_b, const TRef& wx, const TRef& wdt,
                         const TRef& dt_b, const TRef& A, const TRef& D, const TRef& conv_state, const TRef& state, const TRef& seqs, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    const bool bf = proj.dtype == DT_BF16;
    const int64_t element = bf ? 2 : 4, cols = d.rank + 2 * d.state;
    auto tensor = [&](int dtype, int64_t n, int64_t bytes) {
        TRef t;
        t.dtype = dtype;
        t.shape = {rows, n};
        t.buf = em.scratch((size_t)(rows * n * bytes));
        return t;
    };
    const TRef u = tensor(proj.dtype, d.width, element), bc = tensor(proj.dtype, cols, element), dt = tensor(DT_F32, d.width, 4);
    ScanP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.x_off = d.x_off;
    p.z_off = d.z_off;
    p.n_seqs = (int)n_seqs;
    p.n_slots = (int)state.shape[0];
    p.width = (int)d.width;
    p.states = (int)d.state;
    p.rank = (int)d.rank;
    p.taps = (int)d.taps;
    p.node = em.node;
    const bool decode = rows == n_seqs;

    auto lanes_for = [&](int n) {
        int g = 1;
        while (g * n < d.state) g *= 2;
        return g;
    };
    // token after token: as many pairs of states per lane as leave a warp to every scheduler
    const int schedulers = 4 * sm_count();
    int pairs = 4;
    while (pairs > 1 && (d.state <= 4 * pairs || (d.width * d.state / (64 * pairs) < schedulers && lanes_for(pairs) <= 32))) pairs /= 2;
    const int group = std::max(lanes_for(2 * pairs), 4);
    const bool serial = bf && !decode && d.state % 8 == 0 && d.state <= 64 && d.rank % 8 == 0 && d.width % 4 == 0 && p.ld % 4 == 0 && d.z_off % 4 == 0;
    const bool step = bf && decode && d.state % 4 == 0 && d.state <= 128 && d.rank % 8 == 0;

    // tokens per tile and states per thread: long tiles and many states where that leaves enough threads
    int ns = 16;
    p.tile = 64;
    auto tiles_for = [&](int64_t tile) { return std::min<int64_t>(rows, rows / tile + n_seqs); };
    auto threads = [&] { return (decode ? rows : std::max<int64_t>(rows / p.tile, 1)) * d.width * lanes_for(ns); };
    while (ns > 4 && (ns / 2 >= d.state || decode || threads() < (int64_t)sm_count() * 512)) ns /= 2;
    if (lanes_for(ns) > 32) ns = 16;
    if (!decode && threads() < (int64_t)sm_count() * 256) p.tile = 32;
    p.lanes = lanes_for(ns);
    const int64_t tiles = decode ? rows : tiles_for(p.tile);
    const bool chained = !serial && !decode && rows - n_seqs + 1 > p.tile;  // some sequence may have several tiles
    const Buf none{kSlotNull, 0};
    const Buf carry = chained ? em.scratch((size_t)(tiles * d.width * d.state) * 4) : none, sum = chained ? em.scratch((size_t)(tiles * d.width) * 4) : none;
    auto launch = [&](ScanKernel k, dim3 grid, unsigned block, unsigned smem, const char* label, bool pdl = true) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.u, u.buf}, {&p.bc, bc.buf}, {&p.dt, dt.buf}, {&p.A, A.buf}, {&p.D, D.buf}, {&p.wdt, wdt.buf}, {&p.dt_b, dt_b.buf},
                   {&p.ring, conv_state.buf}, {&p.state, state.buf}, {&p.carry, carry}, {&p.sum, sum}, {&p.seqs, seqs.buf}, {&p.out, out.buf},
                   {&p.err, Buf{kSlotErr, 0}}},
                  label, pdl);
    };
    ShortConvDesc cd;
    cd.width = d.width;
    cd.taps = d.taps;
    cd.x_off = d.x_off;
    emit_short_conv(em, cd, proj, conv_w, &conv_b, conv_state, seqs, u);
    LinearDesc ld;
    ld.rows = rows;
    ld.out = cols;
    ld.k[0] = d.width;
    ld.k[1] = 0;
    emit_linear(em, ld, &u, nullptr, wx, nullptr, nullptr, bc, nullptr);
    // the step kernel's own dot products are for few sequences
    const bool own_dt = step && n_seqs <= 2 * kStepSeqs;
    if (!own_dt) {
        ld.out = d.width;
        ld.k[0] = d.rank;
        ld.act[0] = ld.act[1] = ACT_SOFTPLUS;
        emit_linear(em, ld, &bc, nullptr, wdt, nullptr, &dt_b, dt, nullptr);
    }
    if (step) {
        const int64_t g = lanes_for(4), channels = kScanThreads / g;
        const int64_t blocks = (d.width + channels - 1) / channels, groups = (n_seqs + kStepSeqs - 1) / kStepSeqs;
        auto pick = [&](auto own) -> ScanKernel {
            constexpr bool OWN = decltype(own)::value;
            return g <= 1 ? scan_step<1, OWN> : g == 2 ? scan_step<2, OWN> : g == 4 ? scan_step<4, OWN> : g == 8 ? scan_step<8, OWN> : g == 16 ? scan_step<16, OWN> : scan_step<32, OWN>;
        };
        const int64_t shares = std::min(groups, std::max<int64_t>(1, kStepCtas * sm_count() / blocks)), rounds = (groups + shares - 1) / shares;
        launch(own_dt ? pick(std::true_type{}) : pick(std::false_type{}), dim3((unsigned)blocks, (unsigned)((groups + rounds - 1) / rounds)), kScanThreads, 0, "scan_step");
        return;
    }
    if (serial) {
        auto go = [&](ScanKernel k, int threads) {
            const int64_t channels = threads / group;
            // not ahead of the launch before it: small CTAs would crowd on the multiprocessors that it leaves first
            launch(k, dim3((unsigned)((d.width + channels - 1) / channels), (unsigned)n_seqs), 2 * (unsigned)threads, 0, "scan_serial", /*pdl=*/false);
        };
        if (pairs == 1 && group == 4) go(scan_serial<1, 4>, SerialShape<1, 4>::threads);
        else if (pairs == 1 && group == 8) go(scan_serial<1, 8>, SerialShape<1, 8>::threads);
        else if (pairs == 1 && group == 16) go(scan_serial<1, 16>, SerialShape<1, 16>::threads);
        else if (pairs == 1) go(scan_serial<1, 32>, SerialShape<1, 32>::threads);
        else if (pairs == 2 && group == 4) go(scan_serial<2, 4>, SerialShape<2, 4>::threads);
        else if (pairs == 2 && group == 8) go(scan_serial<2, 8>, SerialShape<2, 8>::threads);
        else if (pairs == 2) go(scan_serial<2, 16>, SerialShape<2, 16>::threads);
        else if (group == 4) go(scan_serial<4, 4>, SerialShape<4, 4>::threads);
        else go(scan_serial<4, 8>, SerialShape<4, 8>::threads);
        return;
    }
    const int64_t channels = kScanThreads / p.lanes;
    const dim3 grid((unsigned)((d.width + channels - 1) / channels), (unsigned)tiles);
    const unsigned smem = (unsigned)(kScanSub * 2 * p.lanes * ns * 4);
    if (chained) {
        launch(bf ? token_kernel<bf16>(ns, true) : token_kernel<float>(ns, true), grid, kScanThreads, smem, "scan_local");
        launch(bf ? scan_chain<false> : scan_chain<true>, dim3((unsigned)((d.width * d.state + 255) / 256), (unsigned)n_seqs), 256, 0, "scan_chain");
    }
    launch(bf ? token_kernel<bf16>(ns, false) : token_kernel<float>(ns, false), grid, kScanThreads, smem, "scan_tokens");
}

}  // namespace oxk
