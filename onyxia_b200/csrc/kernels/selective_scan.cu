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
//   scan_conv     u of all tokens
//   products      (linear.cu) W_x u; W_dt dt over a column range of it, softplus behind it, in f32
//   scan_tokens   a tile of consecutive tokens of one sequence × some channels per CTA: a thread holds NS states of a channel, B and
//                 C of the tile lie in shared memory. Two forms: the state that a tile leaves when it starts from zero, and
//                 the results from the state that enters the tile
//   scan_chain    the state that enters every tile of a sequence
//
// Sequences that fit one tile (all of a decode step) need the second form only. Bytes per token and channel: 2 + 2 + 4 + 2 read, 2
// written, 8 · states of state per sequence; 6 · states operations and a power per token, channel and form.
#include "paged_util.cuh"

namespace oxk {

namespace {

constexpr int kScanThreads = 128, kScanSub = 16;  // tokens whose B and C are staged together

struct ScanP {
    const void* proj;             // [rows, ld]
    const float *cw, *cb;         // [width, taps], [width]
    void* u;                      // [rows, width]
    const void* bc;               // [rows, rank + 2 · state]
    const float *dt, *A, *D;      // [rows, width], [width, state], [width]
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

// ───────────────────────────── convolution ──────────────────────────────
// V consecutive channels of one row
template <typename T, int V> struct Chan {
    float v[V];
    __device__ __forceinline__ void load(const T* from) {
        if constexpr (V == 8) {
            const uint4 x = *reinterpret_cast<const uint4*>(from);
            const unsigned w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
            for (int e = 0; e < 4; e++) {
                v[2 * e] = __uint_as_float(w[e] << 16);
                v[2 * e + 1] = __uint_as_float(w[e] & 0xFFFF0000u);
            }
        } else {
            v[0] = to_f(from[0]);
        }
    }
    __device__ __forceinline__ void store(T* to) const {
        if constexpr (V == 8) *reinterpret_cast<uint4*>(to) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
        else to[0] = from_f<T>(v[0]);
    }
};
// Thread: V channels of ROWS consecutive batch rows, the inputs of the last taps in registers where TAPS is known.
template <typename T, int V, int TAPS, int ROWS> __global__ void __launch_bounds__(128) scan_conv(const ScanP p) {
    pdl_enter();
    const int c = (blockIdx.x * 128 + threadIdx.x) * V;
    const long long row0 = (long long)blockIdx.y * ROWS;
    if (c >= p.width) return;
    const int taps = TAPS ? TAPS : p.taps;
    const T* x = (const T*)p.proj + p.x_off + c;
    const T* ring = (const T*)p.ring + c;
    Chan<T, V> now[ROWS], w[TAPS ? TAPS : 1], bias;
#pragma unroll
    for (int j = 0; j < ROWS; j++)
        if (row0 + j < p.rows) now[j].load(x + (row0 + j) * p.ld);
#pragma unroll
    for (int e = 0; e < V; e++) {
        bias.v[e] = p.cb[c + e];
        if constexpr (TAPS > 0)
#pragma unroll
            for (int k = 0; k < TAPS; k++) w[k].v[e] = p.cw[(long long)(c + e) * TAPS + TAPS - 1 - k];
    }
    int s = find_seq(p.seqs, p.n_seqs, (int)row0);
    SeqRow sq = load_seq(p.seqs, s);
    int slot = slot_of(p, sq.slot);
    // the input `back` tokens before row `row`
    auto input = [&](long long row, int back) {
        Chan<T, V> in;
        const int pos = sq.past + (int)(row - sq.start) - back;
        if (pos < 0) {
#pragma unroll
            for (int e = 0; e < V; e++) in.v[e] = 0.f;
        } else if (row - back >= sq.start) {
            in.load(x + (row - back) * p.ld);
        } else {
            in.load(ring + ((long long)slot * taps + pos % taps) * p.width);
        }
        return in;
    };
    Chan<T, V> before[TAPS > 1 ? TAPS - 1 : 1];  // the inputs 1, 2, … tokens before
    bool known = false;
#pragma unroll
    for (int j = 0; j < ROWS; j++) {
        const long long row = row0 + j;
        if (row >= p.rows) break;
        if (row >= sq.start + sq.len && s + 1 < p.n_seqs) {
            while (s + 1 < p.n_seqs && row >= sq.start + sq.len) sq = load_seq(p.seqs, ++s);
            slot = slot_of(p, sq.slot);
            known = false;
        }
        Chan<T, V> acc = bias;
        if constexpr (TAPS > 0) {
            if (!known)
#pragma unroll
                for (int k = 1; k < TAPS; k++) before[k - 1] = input(row, k);
            known = true;
#pragma unroll
            for (int e = 0; e < V; e++) {
                acc.v[e] = fmaf(now[j].v[e], w[0].v[e], acc.v[e]);
#pragma unroll
                for (int k = 1; k < TAPS; k++) acc.v[e] = fmaf(before[k - 1].v[e], w[k].v[e], acc.v[e]);
            }
#pragma unroll
            for (int k = TAPS - 1; k > 1; k--) before[k - 1] = before[k - 2];
            if constexpr (TAPS > 1) before[0] = now[j];
        } else {
            for (int k = 0; k < taps; k++) {
                const Chan<T, V> in = input(row, k);
#pragma unroll
                for (int e = 0; e < V; e++) acc.v[e] = fmaf(in.v[e], p.cw[(long long)(c + e) * taps + taps - 1 - k], acc.v[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < V; e++) acc.v[e] *= sizeof(T) == 2 ? sigmoid_fast(acc.v[e]) : sigmoid_f(acc.v[e]);
        acc.store((T*)p.u + row * p.width + c);
    }
}

// ───────────────────────────── scan ─────────────────────────────────────
// exp(dt A) S + b. In 32-bit through e^x − 1: a decay next to 1 that is itself rounded would be off by up to 6e-8 of a state that
// lives for many tokens.
template <bool EXACT> __device__ __forceinline__ float advance(float dt, float A, float S, float b) {
    if constexpr (EXACT) return S + fmaf(expm1f(dt * A), S, b);
    else return fmaf(exp2f(dt * A), S, b);  // A carries log2 e
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
                        const int at = first + t0 + t1 + j;
                        if (sq.len - at <= p.taps) ((T*)p.ring)[((long long)slot * p.taps + (sq.past + at) % p.taps) * p.width + c] = x[row * p.ld];
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

    // tokens per tile and states per thread: long tiles and many states where that leaves enough threads
    int ns = 16;
    p.tile = 64;
    auto lanes_for = [&](int n) {
        int g = 1;
        while (g * n < d.state) g *= 2;
        return g;
    };
    auto tiles_for = [&](int64_t tile) { return std::min<int64_t>(rows, rows / tile + n_seqs); };
    auto threads = [&] { return (decode ? rows : std::max<int64_t>(rows / p.tile, 1)) * d.width * lanes_for(ns); };
    while (ns > 4 && (ns / 2 >= d.state || decode || threads() < (int64_t)sm_count() * 512)) ns /= 2;
    if (lanes_for(ns) > 32) ns = 16;
    if (!decode && threads() < (int64_t)sm_count() * 256) p.tile = 32;
    p.lanes = lanes_for(ns);
    const int64_t tiles = decode ? rows : tiles_for(p.tile);
    const bool chained = !decode && rows - n_seqs + 1 > p.tile;  // some sequence may have several tiles
    const Buf none{kSlotNull, 0};
    const Buf carry = chained ? em.scratch((size_t)(tiles * d.width * d.state) * 4) : none, sum = chained ? em.scratch((size_t)(tiles * d.width) * 4) : none;
    auto launch = [&](ScanKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.cw, conv_w.buf}, {&p.cb, conv_b.buf}, {&p.u, u.buf}, {&p.bc, bc.buf}, {&p.dt, dt.buf}, {&p.A, A.buf}, {&p.D, D.buf},
                   {&p.ring, conv_state.buf}, {&p.state, state.buf}, {&p.carry, carry}, {&p.sum, sum}, {&p.seqs, seqs.buf}, {&p.out, out.buf},
                   {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    const bool vec = bf && d.width % 8 == 0 && p.ld % 8 == 0 && d.x_off % 8 == 0 && d.taps == 4;
    const int per_thread = decode ? 1 : 8;
    ScanKernel conv;
    if (vec) conv = decode ? scan_conv<bf16, 8, 4, 1> : scan_conv<bf16, 8, 4, 8>;
    else if (bf) conv = decode ? scan_conv<bf16, 1, 0, 1> : scan_conv<bf16, 1, 0, 8>;
    else conv = decode ? scan_conv<float, 1, 0, 1> : scan_conv<float, 1, 0, 8>;
    const int64_t per_cta = 128 * (vec ? 8 : 1);
    launch(conv, dim3((unsigned)((d.width + per_cta - 1) / per_cta), (unsigned)((rows + per_thread - 1) / per_thread)), 128, 0, "scan_conv");
    LinearDesc ld;
    ld.rows = rows;
    ld.out = cols;
    ld.k[0] = d.width;
    ld.k[1] = 0;
    emit_linear(em, ld, &u, nullptr, wx, nullptr, nullptr, bc, nullptr);
    ld.out = d.width;
    ld.k[0] = d.rank;
    ld.act[0] = ld.act[1] = ACT_SOFTPLUS;
    emit_linear(em, ld, &bc, nullptr, wdt, nullptr, &dt_b, dt, nullptr);

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
