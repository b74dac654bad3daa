// Causal attention of a ragged batch over paged pools of keys and values: rotary positions on the leading dimensions of
// a head, queries and keys divided by their root mean square, capped scores, a window, a sink in the softmax, a factor per head.
//
//   score(i, j) = cap(scale · q_i · k_j) for 0 ≤ i − j < window,  cap(s) = c · tanh(s / c),
//   out_i = gate_i · Σ_j exp(score) v_j / (exp(sink) + Σ_j exp(score))
//
// Keys are stored as rotated and normed, so that another layer can attend to them with queries of its own. A rotation
// keeps the length of a vector: the mean square is taken in front of it. Angles are reduced in 64-bit turns.
//
//   paged_kv_prepare, paged_kv_turn   rotated, normed queries; the new keys and values go to the pools
//   paged_kv_prefill   sequences with several new tokens: 64 (token, head) rows per CTA share each tile of 64 keys;
//                      `mma.sync`, online softmax, only the tiles that the window reaches
//   paged_kv_decode    sequences with one new token, the window's keys split over CTAs and warps, all of the above in one launch
//   paged_kv_simt      f32, and shapes the tensor-core kernels do not take
//
// Heads whose softmax weights are mixed continue in talking_heads.cu.
//
// Decode reads min(past, window) · kv_heads · (dim + vdim) · 2 bytes per sequence; prefill 2 · S · T · heads · (dim + vdim) FLOPs.
#include "paged_kv.cuh"

namespace oxk {

namespace {

// One CTA per row, one warp per head.
template <typename T> __global__ void __launch_bounds__(128) paged_kv_prepare(const KvP p) {
    extern __shared__ float angle[];  // cos[half], sin[half]
    pdl_enter();
    const int row = blockIdx.x, s = find_seq(p.seqs, p.n_seqs, row), lane = threadIdx.x & 31;
    const SeqRow sq = load_seq(p.seqs, s);
    const int pos = sq.past + row - sq.start;
    if (row >= sq.start + sq.len || (sq.len == 1 && !p.singles)) return;
    angles(p.turns, p.half, pos, angle, angle + p.half, threadIdx.x, 128);
    __syncthreads();
    const T* x = (const T*)p.proj + (long long)row * p.ld;
    const long long pg = p.append ? page_of(p, s, pos) : 0;
    for (int h = threadIdx.x >> 5; h < p.heads + (p.append ? p.kv_heads : 0); h += 4) {
        const int g = h - p.heads;
        const T* src = g < 0 ? x + p.q_off + (long long)h * p.dim : x + p.k_off + (long long)g * p.dim;
        T* dst = g < 0 ? (T*)p.q + ((long long)row * p.heads + h) * p.dim : (T*)p.keys + key_row(p, pg, g, pos) * p.dim;
        const float f = head_factor(p, src);
        for (int i = lane; i < p.dim; i += 32) dst[i] = from_f<T>(rotated(p.half, p.interleaved, src, angle, angle + p.half, i) * f);
    }
    if (p.append)
        for (int i = threadIdx.x; i < p.kv_heads * p.vdim; i += 128)
            ((T*)p.values)[key_row(p, pg, i / p.vdim, pos) * p.ldv + i % p.vdim] = x[p.v_off + i];
}

// The same in bf16 where no norm is taken and a head rotates in two halves: two neighbouring elements of both halves per lane, several heads of a
// warp in flight.
constexpr int kTurnThreads = 256;
__global__ void __launch_bounds__(kTurnThreads) paged_kv_turn(const KvP p) {
    extern __shared__ __align__(8) float angle[];  // cos[half], sin[half]
    constexpr int kWarps = kTurnThreads / 32, kAhead = 4;
    pdl_enter();
    const int row = blockIdx.x, s = find_seq(p.seqs, p.n_seqs, row), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const SeqRow sq = load_seq(p.seqs, s);
    const int pos = sq.past + row - sq.start;
    if (row >= sq.start + sq.len || (sq.len == 1 && !p.singles)) return;
    angles(p.turns, p.half, pos, angle, angle + p.half, threadIdx.x, kTurnThreads);
    __syncthreads();
    const bf16* x = (const bf16*)p.proj + (long long)row * p.ld;
    const long long pg = p.append ? page_of(p, s, pos) : 0;
    const int heads = p.heads + (p.append ? p.kv_heads : 0), turned = p.half / 2, units = turned + p.dim / 2 - p.half;
    auto word = [](const bf16* from) { return *reinterpret_cast<const unsigned*>(from); };
    auto put = [](bf16* to, unsigned v) { *reinterpret_cast<unsigned*>(to) = v; };
    for (int u = lane; u < units; u += 32) {
        const bool turns = u < turned;
        const int at = turns ? u * 2 : (u + turned) * 2;  // the other half's pair, or the first one that does not turn
        const float2 c = turns ? *reinterpret_cast<const float2*>(angle + at) : make_float2(1.f, 1.f), n = turns ? *reinterpret_cast<const float2*>(angle + p.half + at) : make_float2(0.f, 0.f);
        for (int h0 = warp; h0 < heads; h0 += kWarps * kAhead) {
            unsigned a[kAhead], b[kAhead];
#pragma unroll
            for (int i = 0; i < kAhead; i++) {
                const int h = h0 + i * kWarps, g = h - p.heads;
                const bf16* src = (g < 0 ? x + p.q_off + (long long)h * p.dim : x + p.k_off + (long long)g * p.dim) + at;
                a[i] = h < heads ? word(src) : 0u;
                b[i] = h < heads && turns ? word(src + p.half) : 0u;
            }
#pragma unroll
            for (int i = 0; i < kAhead; i++) {
                const int h = h0 + i * kWarps, g = h - p.heads;
                if (h >= heads) break;
                bf16* dst = (g < 0 ? (bf16*)p.q + ((long long)row * p.heads + h) * p.dim : (bf16*)p.keys + key_row(p, pg, g, pos) * p.dim) + at;
                if (!turns) {
                    put(dst, a[i]);
                    continue;
                }
                const float x0 = __uint_as_float(a[i] << 16), x1 = __uint_as_float(a[i] & 0xFFFF0000u), y0 = __uint_as_float(b[i] << 16), y1 = __uint_as_float(b[i] & 0xFFFF0000u);
                put(dst, pack_bf16(x0 * c.x - y0 * n.x, x1 * c.y - y1 * n.y));
                put(dst + p.half, pack_bf16(y0 * c.x + x0 * n.x, y1 * c.y + x1 * n.y));
            }
        }
    }
    if (p.append)
        for (int i = threadIdx.x; i < p.kv_heads * p.vdim / 2; i += kTurnThreads)
            put((bf16*)p.values + key_row(p, pg, 2 * i / p.vdim, pos) * p.ldv + 2 * i % p.vdim, word(x + p.v_off + 2 * i));
}

// ───────────────────────────── any shape ────────────────────────────────
// One CTA per (row, head); key chunks of 128.
template <typename T> __global__ void __launch_bounds__(128) paged_kv_simt(const KvP p) {
    extern __shared__ float sm[];  // q[dim], acc[vdim], w[128]
    __shared__ float red[32];
    pdl_enter();
    const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, s = find_seq(p.seqs, p.n_seqs, row);
    const SeqRow sq = load_seq(p.seqs, s);
    if (row >= sq.start + sq.len) return;
    const int pos = sq.past + row - sq.start, g = h / (p.heads / p.kv_heads);
    float *q = sm, *acc = sm + p.dim, *w = acc + p.vdim;
    for (int i = tid; i < p.dim; i += 128) q[i] = to_f(((const T*)p.q)[((long long)row * p.heads + h) * p.dim + i]);
    for (int i = tid; i < p.vdim; i += 128) acc[i] = 0.f;
    float m = p.sink ? sink_of(p, h) : kNoScore, l = p.sink ? 1.f : 0.f;
    __syncthreads();
    for (int j0 = first_key(p, pos); j0 <= pos; j0 += 128) {
        const int j = j0 + tid;
        float sc = -INFINITY;
        if (j <= pos) {
            const T* k = (const T*)p.keys + key_row(p, page_of(p, s, j), g, j) * p.dim;
            float d = 0.f;
            for (int i = 0; i < p.dim; i++) d = fmaf(q[i], to_f(k[i]), d);
            sc = d * p.scale * temp_of(p, h);
            if (p.cap > 0.f) sc = p.cap * tanhf(sc / p.cap);
        }
        const float m2 = fmaxf(m, block_max(sc, red));
        const float e = expf(sc - m2), keep = expf(m - m2);
        w[tid] = e;
        l = l * keep + block_sum(e, red);  // (its barriers order the stores to w)
        m = m2;
        const int live = min(128, pos + 1 - j0);
        for (int i = tid; i < p.vdim; i += 128) {
            float a = acc[i] * keep;
            long long pg = 0;
            for (int jj = 0; jj < live; jj++) {
                if (jj == 0 || ((j0 + jj) & ((1 << p.shift) - 1)) == 0) pg = page_of(p, s, j0 + jj);
                a = fmaf(w[jj], to_f(((const T*)p.values)[key_row(p, pg, g, j0 + jj) * p.ldv + i]), a);
            }
            acc[i] = a;
        }
        __syncthreads();
    }
    const float f = gate_of<T>(p, row, h) / l;
    for (int i = tid; i < p.vdim; i += 128) ((T*)p.out)[((long long)row * p.heads + h) * p.vdim + i] = from_f<T>(acc[i] * f);
}

// ───────────────────────────── prefill ──────────────────────────────────
constexpr int kPreRows = 64, kPreKeys = 64, kPreThreads = 128;

// DP: head sizes of keys and values, padded
template <int DP> struct PreSmem {
    static constexpr int stride = DP * 2 + 16;                   // bytes per row: conflict-free ldmatrix
    static constexpr int tile = kPreKeys * stride;
    static constexpr int q = 0;
    static constexpr int kv = kPreRows * stride;                 // two stages of keys and values
    static constexpr int total = kv + 4 * tile, keys_only = kv + 2 * tile;
};

// LSE: no values; the softmax's sums are the result.
template <int DP, bool LSE> __global__ void __launch_bounds__(kPreThreads) paged_kv_prefill(const KvP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    using L = PreSmem<DP>;
    pdl_enter();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    const int rep = p.heads / p.kv_heads, tq = kPreRows / rep, g = blockIdx.y;
    int seq, first;
    // long rows first: the last tiles of a sequence see the most keys
    if (!locate_tile(p.seqs, p.n_seqs, (int)gridDim.x - 1 - (int)blockIdx.x, tq, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);
    const int n_tok = min(tq, sq.len - first), pos0 = sq.past + first, last = pos0 + n_tok - 1;
    constexpr int chunks = DP / 8;
    const int dim = p.dim, vdim = p.vdim;
    const bf16 *q = (const bf16*)p.q, *keys = (const bf16*)p.keys, *values = (const bf16*)p.values;
    const unsigned sm0 = smem_u32(smem);

    auto load_tile = [&](int kt, int st) {
        const int j0 = kt * kPreKeys;
        const bool whole = (1 << p.shift) >= kPreKeys;  // the tile lies in one page
        const long long row0 = whole ? key_row(p, page_of(p, seq, j0), g, j0) : 0;
        const unsigned dst = sm0 + L::kv + st * (LSE ? 1 : 2) * L::tile;
#pragma unroll 4
        for (int i = tid; i < kPreKeys * chunks; i += kPreThreads) {
            const int key = i / chunks, c = i % chunks, j = j0 + key;
            long long row = row0 + key;
            if (!whole) row = j <= last ? key_row(p, page_of(p, seq, j), g, j) : 0;
            const bool k_live = j <= last && c * 8 < dim, v_live = j <= last && c * 8 < vdim;
            cp_async16(dst + key * L::stride + c * 16, k_live ? keys + row * dim + c * 8 : keys, k_live);
            if constexpr (!LSE) cp_async16(dst + L::tile + key * L::stride + c * 16, v_live ? values + row * p.ldv + c * 8 : values, v_live);
        }
        cp_async_commit();
    };
    for (int i = tid; i < kPreRows * chunks; i += kPreThreads) {
        const int r = i / chunks, c = i % chunks, tok = r / rep, h = g * rep + r % rep;
        const bool live = tok < n_tok && c * 8 < dim;
        const bf16* src = live ? q + ((long long)(sq.start + first + tok) * p.heads + h) * dim + c * 8 : q;
        cp_async16(sm0 + L::q + r * L::stride + c * 16, src, live);
    }
    const int kt0 = first_key(p, pos0) / kPreKeys, kt1 = last / kPreKeys + 1;
    load_tile(kt0, kt0 & 1);

    constexpr int OC = LSE ? 0 : DP / 8;
    float o[OC + 1][4];
#pragma unroll
    for (int n = 0; n < OC; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    float m[2] = {kNoScore, kNoScore}, l[2] = {0.f, 0.f};
    int pos[2], low[2];
    float mul2[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = warp * 16 + g8 + 8 * e;
        mul2[e] = p.mul2 * temp_of(p, g * rep + r % rep);
        pos[e] = r / rep < n_tok ? pos0 + r / rep : last;  // rows without a token compute something harmless
        low[e] = first_key(p, pos[e]);
    }
    const int last_low = first_key(p, last);
    for (int kt = kt0; kt < kt1; kt++) {
        const int st = kt & 1, j0 = kt * kPreKeys;
        if (kt + 1 < kt1) {
            load_tile(kt + 1, st ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        float s[kPreKeys / 8][4];
#pragma unroll
        for (int n = 0; n < kPreKeys / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[n][e] = 0.f;
        const unsigned ks = sm0 + L::kv + st * (LSE ? 1 : 2) * L::tile, vs = ks + L::tile;
#pragma unroll
        for (int kk = 0; kk < DP / 16; kk++) {
            unsigned a[4];
            ldmatrix_x4(a, sm0 + L::q + (warp * 16 + (lane & 15)) * L::stride + kk * 32 + (lane >> 4) * 16);
#pragma unroll
            for (int n = 0; n < kPreKeys / 8; n += 2) {
                unsigned b[4];  // keys 8n … 8n+7 and the next eight, 16 dims
                ldmatrix_x4(b, ks + (n * 8 + (lane & 7) + (lane >> 4) * 8) * L::stride + kk * 32 + ((lane >> 3) & 1) * 16);
                mma_bf16(s[n], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(s[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
        const bool edge = j0 + kPreKeys - 1 > pos0 || j0 < last_low;
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int n = 0; n < kPreKeys / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int j = j0 + n * 8 + t4 * 2 + (e & 1), r = e >> 1;
                float v = score2(p, s[n][e], mul2[r]);
                if (edge && (j > pos[r] || j < low[r])) v = -INFINITY;
                s[n][e] = v;
                mx[r] = fmaxf(mx[r], v);
            }
#pragma unroll
        for (int r = 0; r < 2; r++) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float keep = exp2f(m[r] - mx[r]);
            m[r] = mx[r];
            l[r] *= keep;
#pragma unroll
            for (int n = 0; n < OC; n++) {
                o[n][2 * r] *= keep;
                o[n][2 * r + 1] *= keep;
            }
        }
#pragma unroll
        for (int n = 0; n < kPreKeys / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float w = exp2f(s[n][e] - m[e >> 1]);
                s[n][e] = w;
                l[e >> 1] += w;
            }
#pragma unroll
        for (int kk = 0; kk < kPreKeys / 16; kk++) {
            const unsigned a0 = pack_bf16(s[2 * kk][0], s[2 * kk][1]), a1 = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
            const unsigned a2 = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), a3 = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
            for (int n = 0; n < OC; n += 2) {
                unsigned b[4];
                ldmatrix_x4_trans(b, vs + (kk * 16 + (lane & 15)) * L::stride + n * 16 + (lane >> 4) * 16);
                mma_bf16(o[n], a0, a1, a2, a3, b[0], b[1]);
                mma_bf16(o[n + 1], a0, a1, a2, a3, b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const int row = warp * 16 + g8 + 8 * r, tok = row / rep;
        if (tok >= n_tok) continue;
        const int head = g * rep + row % rep;
        const long long token = sq.start + first + tok;
        if constexpr (LSE) {
            if (t4 == 0) p.lse[token * p.heads + head] = m[r] + log2f(l[r]);
            continue;
        }
        float f = 1.f / l[r];
        if (p.sink) {
            const float s = sink_of(p, head) * kLog2e, top = fmaxf(m[r], s), keep = exp2f(m[r] - top);
            f = keep / (l[r] * keep + exp2f(s - top));
        }
        f *= gate_of<bf16>(p, token, head);
        bf16* out = (bf16*)p.out + (token * p.heads + head) * vdim;
#pragma unroll
        for (int n = 0; n < OC; n++) {
            const int d = n * 8 + t4 * 2;
            if (d < vdim) *reinterpret_cast<unsigned*>(out + d) = pack_bf16(o[n][2 * r] * f, o[n][2 * r + 1] * f);
        }
    }
}

// ───────────────────────────── decode ───────────────────────────────────
constexpr int kDecWarps = 4, kDecThreads = kDecWarps * 32, kDecPages = 256;

// NH groups of eight query heads of one key head
template <int DP, int NH> struct DecSmem {
    static constexpr int rows = 8 * NH;
    static constexpr int keys = DP <= 64 ? 32 : 16;              // keys of a warp's tile
    static constexpr int stages = DP <= 128 ? 3 : 2;
    static constexpr int stride = DP * 2 + 16;
    static constexpr int tile = 2 * keys * stride;               // keys, then values
    static constexpr int q = 0;                                  // [rows][stride]
    static constexpr int kv = rows * stride;                     // [warps][stages][tile]
    static constexpr int ring = kDecWarps * stages * tile;
    static constexpr int part = part_size(rows, DP);             // floats of one partial result
    static constexpr int merge = kDecWarps * part * 4;           // reuses the ring after the last key
    static constexpr int angle = kv + (ring > merge ? ring : merge);  // cos[DP / 2], sin[DP / 2]
    static constexpr int total = angle + DP * 4;
};

// Grid: (splits, kv_heads · groups of 8 · NH query heads, sequences).
template <int DP, int NH> __global__ void __launch_bounds__(kDecThreads) paged_kv_decode(const KvP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ unsigned arrived;
    __shared__ int page_s[kDecPages];  // this CTA's pages, checked
    using L = DecSmem<DP, NH>;
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    // no launch of a step writes the batch description or the keys and values of earlier steps: they may be read while the
    // launches before this one finish
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int rep = p.heads / p.kv_heads, groups = (rep + L::rows - 1) / L::rows, g = blockIdx.y / groups, h0 = g * rep + (blockIdx.y % groups) * L::rows;
    const int n_heads = min(L::rows, (g + 1) * rep - h0), seq = blockIdx.z, pos = sq.past, dim = p.dim, vdim = p.vdim;
    const bf16* x = (const bf16*)p.proj + (long long)sq.start * p.ld;
    bf16 *keys = (bf16*)p.keys, *values = (bf16*)p.values;
    const unsigned sm0 = smem_u32(smem);
    float *cs = reinterpret_cast<float*>(smem + L::angle), *sn = cs + DP / 2;

    // keys of this CTA: whole tiles of all four warps, so that a split never cuts a tile
    constexpr int step = L::keys * kDecWarps;
    const int low = first_key(p, pos), base = low / step, blocks = sq.len == 1 ? pos / step + 1 - base : 0;
    const int b0 = base + (int)((long long)blocks * blockIdx.x / p.splits), b1 = base + (int)((long long)blocks * (blockIdx.x + 1) / p.splits);
    const int lo = b0 * step, hi = min(b1 * step, pos + 1);
    const int page0 = lo >> p.shift, n_pages = lo < hi ? ((hi - 1) >> p.shift) - page0 + 1 : 0;
    for (int i = tid; i < min(n_pages, kDecPages); i += kDecThreads) page_s[i] = (int)page_of(p, seq, (page0 + i) << p.shift);
    angles(p.turns, p.half, pos, cs, sn, tid, kDecThreads);
    __syncthreads();
    auto page_at = [&](int j) {
        const int i = (j >> p.shift) - page0;
        return i < kDecPages ? (long long)page_s[i] : page_of(p, seq, j);
    };
    const unsigned ring = sm0 + L::kv + warp * L::stages * L::tile;
    const int first = lo + warp * L::keys, tiles = first < hi ? (hi - first + step - 1) / step : 0;
    auto load_tile = [&](int i) {
        const int j0 = first + i * step;
        if (i < tiles) {
            const unsigned dst = ring + (i % L::stages) * L::tile;
            const bool whole = (1 << p.shift) >= L::keys;  // a tile lies in one page when pages are a multiple of it
            const long long row0 = whole ? key_row(p, page_at(j0), g, j0) : 0;
            constexpr int per_key = DP / 8;
            if constexpr (32 % per_key == 0)
                if (whole && dim == DP && vdim == DP && p.ldv == DP && j0 + L::keys <= hi) {  // contiguous runs: a lane's copies are evenly spaced
                    const unsigned d = dst + (lane / per_key) * L::stride + (lane % per_key) * 16;
                    const bf16 *k = keys + row0 * DP + lane * 8, *v = values + row0 * DP + lane * 8;
#pragma unroll
                    for (int c = 0; c < L::keys * per_key / 32; c++) {
                        cp_async16(d + c * (32 / per_key) * L::stride, k + c * 256);
                        cp_async16(d + L::keys * L::stride + c * (32 / per_key) * L::stride, v + c * 256);
                    }
                    cp_async_commit();
                    return;
                }
#pragma unroll 4
            for (int c = lane; c < L::keys * per_key; c += 32) {
                const int key = c / per_key, ch = c % per_key;
                const bool in = j0 + key < hi, k_live = in && ch * 8 < dim, v_live = in && ch * 8 < vdim;
                long long row = row0 + key;
                if (!whole) row = in ? key_row(p, page_at(j0 + key), g, j0 + key) : 0;
                cp_async16(dst + key * L::stride + ch * 16, k_live ? keys + row * dim + ch * 8 : keys, k_live);
                cp_async16(dst + (L::keys + key) * L::stride + ch * 16, v_live ? values + row * p.ldv + ch * 8 : values, v_live);
            }
        }
        cp_async_commit();
    };
    const bool newest = hi == pos + 1 && lo < hi;  // this CTA's keys include the new one
    auto fill = [&]() {
#pragma unroll
        for (int i = 0; i < L::stages - 1; i++) load_tile(i);
    };
    if (!newest) fill();
    pdl_wait();
    if (sq.len != 1) return;
    if (newest) {
        if (p.append) {
            const long long row = key_row(p, page_at(pos), g, pos);
            if (warp == 0) {
                const bf16* k = x + p.k_off + g * dim;
                const float f = head_factor(p, k);
                for (int i = lane; i < dim; i += 32) keys[row * dim + i] = __float2bfloat16_rn(rotated(p.half, p.interleaved, k, cs, sn, i) * f);
            } else if (warp == 1) {
                for (int i = lane; i < vdim; i += 32) values[row * p.ldv + i] = x[p.v_off + g * vdim + i];
            }
            __syncthreads();
        }
        fill();
    }
    for (int r = warp; r < L::rows; r += kDecWarps) {
        const bool live = r < n_heads;
        const bf16* q = x + p.q_off + (long long)(live ? h0 + r : h0) * dim;
        const float f = head_factor(p, q);
        for (int i = lane; i < DP; i += 32)
            *reinterpret_cast<bf16*>(smem + L::q + r * L::stride + i * 2) = __float2bfloat16_rn(live && i < dim ? rotated(p.half, p.interleaved, q, cs, sn, i) * f : 0.f);
    }
    __syncthreads();

    // Keys are the rows of both products (S^T = K q^T, O^T = V^T P^T): a lane holds scores of keys g, g + 8 and heads 2t, 2t + 1.
    constexpr int MT = L::keys / 16;
    float o[DP / 16][NH][4];
#pragma unroll
    for (int n = 0; n < DP / 16; n++)
#pragma unroll
        for (int h = 0; h < NH; h++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[n][h][e] = 0.f;
    float m[NH][2], l[NH][2];
#pragma unroll
    for (int h = 0; h < NH; h++) {
        m[h][0] = m[h][1] = kNoScore;
        l[h][0] = l[h][1] = 0.f;
    }
    float mul2[NH][2];
#pragma unroll
    for (int h = 0; h < NH; h++)
#pragma unroll
        for (int e = 0; e < 2; e++) mul2[h][e] = p.mul2 * temp_of(p, h0 + min(h * 8 + t4 * 2 + e, n_heads - 1));
    for (int i = 0; i < tiles; i++) {
        cp_async_wait<L::stages - 2>();
        __syncwarp();
        load_tile(i + L::stages - 1);  // the slot was read in the previous iteration
        const unsigned ks = ring + (i % L::stages) * L::tile, vs = ks + L::keys * L::stride;
        const int j0 = first + i * step;
        float s[MT][NH][4];
#pragma unroll
        for (int a = 0; a < MT; a++)
#pragma unroll
            for (int h = 0; h < NH; h++)
#pragma unroll
                for (int e = 0; e < 4; e++) s[a][h][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DP / 32; kk++) {
            unsigned bq[NH][4];
#pragma unroll
            for (int h = 0; h < NH; h++) ldmatrix_x4(bq[h], sm0 + L::q + (h * 8 + (lane & 7)) * L::stride + kk * 64 + (lane >> 3) * 16);
#pragma unroll
            for (int a = 0; a < MT; a++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    unsigned ka[4];
                    ldmatrix_x4(ka, ks + (a * 16 + (lane & 15)) * L::stride + kk * 64 + half * 32 + (lane >> 4) * 16);
#pragma unroll
                    for (int h = 0; h < NH; h++) mma_bf16(s[a][h], ka[0], ka[1], ka[2], ka[3], bq[h][2 * half], bq[h][2 * half + 1]);
                }
        }
        float mx[NH][2];
#pragma unroll
        for (int h = 0; h < NH; h++) {
            mx[h][0] = m[h][0];
            mx[h][1] = m[h][1];
        }
        const bool edge = j0 + L::keys > hi || j0 < low;
#pragma unroll
        for (int a = 0; a < MT; a++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int j = j0 + a * 16 + g8 + 8 * r;
                const bool hidden = edge && (j >= hi || j < low);
#pragma unroll
                for (int h = 0; h < NH; h++)
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const float v = hidden ? -INFINITY : score2(p, s[a][h][2 * r + e], mul2[h][e]);
                        s[a][h][2 * r + e] = v;
                        mx[h][e] = fmaxf(mx[h][e], v);
                    }
            }
        bool moved = false;
#pragma unroll
        for (int h = 0; h < NH; h++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
#pragma unroll
                for (int d = 4; d < 32; d <<= 1) mx[h][e] = fmaxf(mx[h][e], __shfl_xor_sync(0xffffffffu, mx[h][e], d));
                moved |= mx[h][e] != m[h][e];
            }
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int h = 0; h < NH; h++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const float keep = exp2f(m[h][e] - mx[h][e]);
                    m[h][e] = mx[h][e];
                    l[h][e] *= keep;
#pragma unroll
                    for (int n = 0; n < DP / 16; n++) {
                        o[n][h][e] *= keep;
                        o[n][h][e + 2] *= keep;
                    }
                }
        }
#pragma unroll
        for (int a = 0; a < MT; a++) {
            unsigned pb[NH][2];
#pragma unroll
            for (int h = 0; h < NH; h++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const float w0 = exp2f(s[a][h][2 * r] - m[h][0]), w1 = exp2f(s[a][h][2 * r + 1] - m[h][1]);
                    l[h][0] += w0;
                    l[h][1] += w1;
                    pb[h][r] = transpose8x8(pack_bf16(w0, w1));
                }
#pragma unroll
            for (int n = 0; n < DP / 16; n++) {
                unsigned va[4];
                ldmatrix_x4_trans(va, vs + (a * 16 + (lane >> 4) * 8 + (lane & 7)) * L::stride + n * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
                for (int h = 0; h < NH; h++) mma_bf16(o[n][h], va[0], va[1], va[2], va[3], pb[h][0], pb[h][1]);
            }
        }
        __syncwarp();
    }
    cp_async_wait<0>();
    __syncthreads();  // the ring becomes the merge area
    float* parts = reinterpret_cast<float*>(smem + L::kv);
#pragma unroll
    for (int h = 0; h < NH; h++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
#pragma unroll
            for (int d = 4; d < 32; d <<= 1) l[h][e] += __shfl_xor_sync(0xffffffffu, l[h][e], d);
            float* q2 = parts + warp * L::part + (h * 8 + t4 * 2 + e) * (DP + 2);
            if (g8 == 0) {
                q2[0] = m[h][e];
                q2[1] = l[h][e];
            }
#pragma unroll
            for (int n = 0; n < DP / 16; n++) {
                q2[2 + n * 16 + g8] = o[n][h][e];
                q2[2 + n * 16 + g8 + 8] = o[n][h][e + 2];
            }
        }
    __syncthreads();
    bf16* out = (bf16*)p.out + ((long long)sq.start * p.heads + h0) * vdim;
    auto gate = [&](int r) { return gate_of<bf16>(p, sq.start, h0 + r); };
    auto sink = [&](int r) { return p.sink ? sink_of(p, h0 + r) * kLog2e : -INFINITY; };
    if (p.splits == 1) {
        merge_parts<DP, L::rows, kDecWarps>(parts, kDecWarps, n_heads, vdim, gate, out, nullptr, sink);
        return;
    }
    const long long cell = (long long)blockIdx.z * gridDim.y + blockIdx.y;
    merge_parts<DP, L::rows, kDecWarps>(parts, kDecWarps, n_heads, vdim, 0.f, nullptr, p.part + (cell * p.splits + blockIdx.x) * L::part);
    __threadfence();
    __syncthreads();
    if (tid == 0) arrived = atomicAdd(&p.counters[cell], 1u);
    __syncthreads();
    if (arrived != (unsigned)p.splits - 1) return;
    __threadfence();
    if (tid == 0) p.counters[cell] = 0;
    merge_parts<DP, L::rows, kDecWarps>(p.part + cell * p.splits * L::part, p.splits, n_heads, vdim, gate, out, nullptr, sink);
}

using KvKernel = void (*)(const KvP);
struct DimChoice {
    KvKernel prefill, lse, decode[2];
    int pre_smem, lse_smem, dec_smem[2], dec_part[2];
};
template <int DP> DimChoice choice() {
    return {paged_kv_prefill<DP, false>, paged_kv_prefill<DP, true>, {paged_kv_decode<DP, 1>, paged_kv_decode<DP, 2>}, PreSmem<DP>::total, PreSmem<DP>::keys_only,
            {DecSmem<DP, 1>::total, DecSmem<DP, 2>::total}, {DecSmem<DP, 1>::part, DecSmem<DP, 2>::part}};
}
DimChoice dim_choice(int64_t dim) {
    return dim <= 32 ? choice<32>() : dim <= 64 ? choice<64>() : dim <= 96 ? choice<96>() : dim <= 128 ? choice<128>() : dim <= 192 ? choice<192>() : choice<256>();
}

}  // namespace

void emit_paged_kv_attention(Emitter& em, const PagedKvDesc& d, const TRef& proj, const TRef& turns, const TRef& keys, const TRef& values,
                             const TRef& seqs, const TRef& pages, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    KvP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.q_off = d.q_off;
    p.k_off = d.k_off;
    p.v_off = d.v_off;
    p.n_seqs = (int)n_seqs;
    p.width = (int)pages.shape[1];
    p.n_pages = (int)keys.shape[0];
    while ((int64_t)1 << p.shift < d.page) p.shift++;
    p.heads = (int)d.heads;
    p.kv_heads = (int)d.kv_heads;
    p.dim = (int)d.dim;
    p.vdim = (int)d.vdim;
    p.half = (int)(d.rot_dims / 2);
    p.window = (int)d.window;
    p.ldv = (int)(d.latent ? d.dim : d.vdim);
    p.interleaved = d.interleaved;
    p.gate_ld = p.ld;
    p.node = em.node;
    p.splits = 1;
    p.scale = (float)d.scale;
    p.cap = (float)d.softcap;
    p.eps = (float)d.eps;
    p.cap2 = (float)(d.softcap * (double)kLog2e);
    p.mul2 = (float)(d.softcap > 0 ? 2.0 * (double)kLog2e * d.scale / d.softcap : (double)kLog2e * d.scale);
    p.norm = d.norm;
    p.sink = d.sink;
    p.append = d.append;
    const int64_t rep = d.heads / d.kv_heads, widest = std::max(d.dim, d.vdim);
    const bool bf = proj.dtype == DT_BF16;
    // 16-byte copies of key and value rows
    const bool tc = bf && d.dim % 8 == 0 && d.vdim % 8 == 0 && widest <= 256 && rep <= kPreRows && (!d.talk || d.heads <= kTalkHeads);
    const DimChoice dc = dim_choice(widest);
    const bool decode_only = tc && rows == n_seqs;  // every sequence has one new token
    p.singles = !tc;
    const Buf none{kSlotNull, 0};
    const Buf q = d.latent ? proj.buf : decode_only ? none : em.scratch((size_t)rows * d.heads * d.dim * (bf ? 2 : 4));
    const Buf temps = d.temps ? d.temps->buf : none;
    const Buf sink = d.sinks ? d.sinks->buf : none, gate = d.gate_off >= 0 ? proj.buf.at(d.gate_off * (bf ? 2 : 4)) : none;
    auto launch = [&](KvKernel k, dim3 grid, unsigned block, unsigned smem, Buf part, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.turns, turns.buf}, {&p.keys, keys.buf}, {&p.values, values.buf}, {&p.q, q}, {&p.sinks, sink}, {&p.temps, temps}, {&p.gate, gate}, {&p.out, out.buf}, {&p.seqs, seqs.buf},
                   {&p.table, pages.buf}, {&p.part, part}, {&p.counters, Buf{kSlotCounters, 0}}, {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    const bool turn = bf && !d.norm && !d.interleaved && p.half % 2 == 0 && d.dim % 2 == 0 && d.vdim % 2 == 0 && p.ld % 2 == 0 && d.q_off % 2 == 0 && d.k_off % 2 == 0 &&
                      d.v_off % 2 == 0 && proj.buf.off % 4 == 0;
    if (!decode_only && !d.latent && turn) launch(paged_kv_turn, dim3((unsigned)rows), kTurnThreads, (unsigned)(d.rot_dims * 4), none, "paged_kv_prepare");
    else if (!decode_only && !d.latent)
        launch(bf ? paged_kv_prepare<bf16> : paged_kv_prepare<float>, dim3((unsigned)rows), 128, (unsigned)(d.rot_dims * 4), none, "paged_kv_prepare");
    if (d.talk) return emit_talking_heads(em, d, p, proj, turns, q, keys, values, seqs, pages, out);
    if (!tc) {
        const KvKernel k = bf ? paged_kv_simt<bf16> : paged_kv_simt<float>;
        ensure_max_dynamic_smem((const void*)k, 220 * 1024);
        launch(k, dim3((unsigned)rows, (unsigned)d.heads), 128, (unsigned)((d.dim + d.vdim + 128) * 4), none, "paged_kv_simt");
        return;
    }
    if (!decode_only) {
        const int64_t tq = kPreRows / rep;
        ensure_max_dynamic_smem((const void*)dc.prefill, 220 * 1024);
        launch(dc.prefill, dim3((unsigned)((rows + tq - 1) / tq + n_seqs), (unsigned)d.kv_heads), kPreThreads, (unsigned)dc.pre_smem, none, "paged_kv_prefill");
    }
    if (decode_only || n_seqs > 1) {
        const int nh = rep > 8;  // two groups of eight heads per CTA
        const int64_t groups = d.kv_heads * ((rep + 8 * nh + 7) / (8 * nh + 8)), cells = n_seqs * groups;
        // splits of the most keys a sequence can see: whole waves of resident CTAs, each with a fixed cost worth about
        // 160 keys, and the pieces have to be merged
        const int64_t resident = std::max<int64_t>(1, std::min<int64_t>(nh ? (widest > 192 ? 2 : 3) : 4, 224 * 1024 / (dc.dec_smem[nh] + 2560))), slots = resident * sm_count();
        int64_t seen = (int64_t)p.width * d.page;
        if (d.window > 0) seen = std::min<int64_t>(seen, d.window + 128);
        int64_t splits = 1;
        double best = 1e300;
        for (int64_t sp = 1; sp <= 64 && sp * 128 <= std::max<int64_t>(seen, 128); sp++) {
            const double us = (double)((cells * sp + slots - 1) / slots) * ((double)seen / sp + 160.0) + 4.0 * sp;
            if (us < best) {
                best = us;
                splits = sp;
            }
        }
        if (cells > (int64_t)kCounterWords) splits = 1;
        p.splits = (int)splits;
        const Buf part = splits > 1 ? em.scratch((size_t)cells * splits * dc.dec_part[nh] * 4) : none;
        ensure_max_dynamic_smem((const void*)dc.decode[nh], dc.dec_smem[nh]);
        launch(dc.decode[nh], dim3((unsigned)splits, (unsigned)groups, (unsigned)n_seqs), kDecThreads, (unsigned)dc.dec_smem[nh], part, "paged_kv_decode");
    }
}

void emit_kv_lse(Emitter& em, const PagedKvDesc& d, KvP p, Buf q, Buf lse, const TRef& keys, const TRef& seqs, const TRef& pages) {
    const DimChoice dc = dim_choice(d.dim);
    const int64_t tq = kPreRows / (d.heads / d.kv_heads);
    const Buf none{kSlotNull, 0}, temps = d.temps ? d.temps->buf : none;
    ensure_max_dynamic_smem((const void*)dc.lse, 220 * 1024);
    em.launch(dc.lse, dim3((unsigned)((p.rows + tq - 1) / tq + p.n_seqs), (unsigned)d.kv_heads), dim3(kPreThreads), (unsigned)dc.lse_smem, p,
              {{&p.keys, keys.buf}, {&p.values, none}, {&p.q, q}, {&p.temps, temps}, {&p.lse, lse}, {&p.seqs, seqs.buf}, {&p.table, pages.buf}, {&p.err, Buf{kSlotErr, 0}}},
              "talk_lse", /*pdl=*/true);
}

}  // namespace oxk
