// Causal attention of a ragged batch over a paged key pool whose values are the keys themselves.
//
// A token's key projection is stored once, as projected; its root mean square over the whole projection (all heads)
// is kept beside it as one f32, and the norm's weights are folded into the query. So
//   score(i, j) = (q'_i · k_j) · r_j + bias[h, min(i − j, n − 1)],   out_i = Σ_j softmax_j(score) k_j
// and both products read the same tile: half the bytes of separate keys and values.
//
//   paged_prepare         query norm, temperature and scale → q'; the new keys and r go to the pool
//   paged_attn_prefill    sequences with several new tokens: 64 (token, head) rows per CTA share each key tile; `mma.sync`,
//                         online softmax
//   paged_attn_decode     sequences with one new token, keys split over CTAs and warps, all of the above in one launch
//   paged_attn_simt       f32, and shapes the tensor-core kernels do not take
//
// Decode reads past · kv_heads · dim · 2 bytes (+ 4 per token) per sequence; prefill 4 · S · T · heads · dim FLOPs.
#include "paged_util.cuh"

namespace oxk {

namespace {

struct PagedP {
    const void* proj;            // [rows, ld]
    const float *qw, *kw;        // [heads · dim], [kv_heads · dim]
    const float* bias;           // [heads, nd] or null
    void* pool;                  // [pages, kv_heads, page, dim]
    float* kscale;               // [pages, page]
    void* q;                     // [rows, heads · dim]: prepared queries
    void* out;                   // [rows, heads · dim]
    const int* seqs;             // [R, 4]
    const int* table;            // [R, width]
    float* part;                 // decode partial results
    unsigned* counters;
    ErrWord* err;
    double temp_every;
    long long rows, ld, q_off, k_off;
    int n_seqs, width, n_pages, shift /* log2 of the page */, heads, kv_heads, dim, nd, splits, node;
    float qmul, eps, temp_coef, out_scale;
    int singles;                 // prepare: also sequences with one new token
    int vec;                     // query and key rows are 16-byte aligned
};

__device__ __forceinline__ long long scale_at(const PagedP& p, long long pg, int pos) { return (pg << p.shift) + (pos & ((1 << p.shift) - 1)); }
__device__ __forceinline__ float query_factor(const PagedP& p, int pos) {
    float f = p.qmul;
    if (p.temp_every > 0.0) f *= 1.f + p.temp_coef * logf((float)floor((double)(pos + 1) / p.temp_every) + 1.f);
    return f;
}

template <typename T> __device__ __forceinline__ float row_sumsq(const T* row, int n, bool vec) {
    float ss = 0.f;
    if constexpr (sizeof(T) == 2)
        if (vec) {
#pragma unroll 4
            for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
                const uint4 x = *reinterpret_cast<const uint4*>(row + i);
                const unsigned v[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float a = __uint_as_float(v[e] << 16), b = __uint_as_float(v[e] & 0xFFFF0000u);
                    ss = fmaf(a, a, fmaf(b, b, ss));
                }
            }
            return ss;
        }
#pragma unroll 4
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = to_f(row[i]);
        ss = fmaf(v, v, ss);
    }
    return ss;
}

// One CTA per row.
template <typename T> __global__ void __launch_bounds__(128) paged_prepare(const PagedP p) {
    __shared__ float red[32];
    pdl_enter();
    const int row = blockIdx.x, s = find_seq(p.seqs, p.n_seqs, row);
    const SeqRow sq = load_seq(p.seqs, s);
    const int pos = sq.past + row - sq.start;
    if (row >= sq.start + sq.len || (sq.len == 1 && !p.singles)) return;
    const int hq = p.heads * p.dim, hk = p.kv_heads * p.dim, rep = p.heads / p.kv_heads;
    const T *q = (const T*)p.proj + (long long)row * p.ld + p.q_off, *k = (const T*)p.proj + (long long)row * p.ld + p.k_off;
    const float qr = 1.f / sqrtf(block_sum(row_sumsq(q, hq, p.vec), red) / (float)hq + p.eps) * query_factor(p, pos);
    const float kr = 1.f / sqrtf(block_sum(row_sumsq(k, hk, p.vec), red) / (float)hk + p.eps);
    T* qo = (T*)p.q + (long long)row * hq;
    for (int i = threadIdx.x; i < hq; i += blockDim.x)
        qo[i] = from_f<T>(to_f(q[i]) * qr * p.qw[i] * p.kw[(i / p.dim) / rep * p.dim + i % p.dim]);
    const long long pg = page_of(p, s, pos);
    T* pool = (T*)p.pool;
    for (int i = threadIdx.x; i < hk; i += blockDim.x) pool[key_row(p, pg, i / p.dim, pos) * p.dim + i % p.dim] = k[i];
    if (threadIdx.x == 0) p.kscale[scale_at(p, pg, pos)] = kr;
}

// ───────────────────────────── any shape ────────────────────────────────
// One CTA per (row, head); key chunks of 128.
template <typename T> __global__ void __launch_bounds__(128) paged_attn_simt(const PagedP p) {
    extern __shared__ float sm[];  // q[dim], acc[dim], w[128]
    __shared__ float red[32];
    pdl_enter();
    const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, s = find_seq(p.seqs, p.n_seqs, row);
    const SeqRow sq = load_seq(p.seqs, s);
    if (row >= sq.start + sq.len) return;
    const int pos = sq.past + row - sq.start, g = h / (p.heads / p.kv_heads);
    float *q = sm, *acc = sm + p.dim, *w = acc + p.dim;
    for (int i = tid; i < p.dim; i += 128) {
        q[i] = to_f(((const T*)p.q)[((long long)row * p.heads + h) * p.dim + i]);
        acc[i] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    __syncthreads();
    for (int j0 = 0; j0 <= pos; j0 += 128) {
        const int j = j0 + tid;
        float sc = -INFINITY;
        if (j <= pos) {
            const long long pg = page_of(p, s, j);
            const T* k = (const T*)p.pool + key_row(p, pg, g, j) * p.dim;
            float d = 0.f;
            for (int i = 0; i < p.dim; i++) d = fmaf(q[i], to_f(k[i]), d);
            sc = d * p.kscale[scale_at(p, pg, j)];
            if (p.bias) sc += p.bias[(long long)h * p.nd + min(pos - j, p.nd - 1)];
        }
        const float m2 = fmaxf(m, block_max(sc, red));
        const float e = expf(sc - m2), keep = expf(m - m2);
        w[tid] = e;
        l = l * keep + block_sum(e, red);  // (its barriers order the stores to w)
        m = m2;
        const int live = min(128, pos + 1 - j0);
        for (int i = tid; i < p.dim; i += 128) {
            float a = acc[i] * keep;
            long long pg = 0;
            for (int jj = 0; jj < live; jj++) {
                if (jj == 0 || ((j0 + jj) & ((1 << p.shift) - 1)) == 0) pg = page_of(p, s, j0 + jj);
                a = fmaf(w[jj], to_f(((const T*)p.pool)[key_row(p, pg, g, j0 + jj) * p.dim + i]), a);
            }
            acc[i] = a;
        }
        __syncthreads();
    }
    for (int i = tid; i < p.dim; i += 128) ((T*)p.out)[((long long)row * p.heads + h) * p.dim + i] = from_f<T>(acc[i] / l * p.out_scale);
}

// ───────────────────────────── prefill ──────────────────────────────────
constexpr int kPreRows = 64, kPreKeys = 64, kPreThreads = 128;

template <int DP> struct PreSmem {
    static constexpr int stride = DP * 2 + 16;                   // bytes per key / query row: conflict-free ldmatrix
    static constexpr int q = 0;
    static constexpr int k = kPreRows * stride;                  // two stages
    static constexpr int scale = k + 2 * kPreKeys * stride;      // f32 [2][keys]
    static constexpr int bias = scale + 2 * kPreKeys * 4;        // f32 [rep][nd]
};

template <int DP> __global__ void __launch_bounds__(kPreThreads) paged_attn_prefill(const PagedP p) {
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
    const int chunks = DP / 8, dim = p.dim;
    const bf16 *q = (const bf16*)p.q, *pool = (const bf16*)p.pool;
    float* bias_s = reinterpret_cast<float*>(smem + L::bias);
    float* scale_s = reinterpret_cast<float*>(smem + L::scale);
    const unsigned sm0 = smem_u32(smem);

    auto load_tile = [&](int kt, int st) {
        const int j0 = kt * kPreKeys;
        const bool whole = (1 << p.shift) >= kPreKeys;  // the tile lies in one page
        const long long pg0 = whole ? page_of(p, seq, j0) : 0;
        const bf16* base = pool + key_row(p, pg0, g, j0) * dim;
#pragma unroll 4
        for (int i = tid; i < kPreKeys * chunks; i += kPreThreads) {
            const int key = i / chunks, c = i % chunks, j = j0 + key;
            const bool live = j <= last && c * 8 < dim;
            const bf16* src = base + key * dim + c * 8;
            if (!live) src = pool;
            else if (!whole) src = pool + key_row(p, page_of(p, seq, j), g, j) * dim + c * 8;
            cp_async16(sm0 + L::k + (st * kPreKeys + key) * L::stride + c * 16, src, live);
        }
        if (tid < kPreKeys) {
            const int j = j0 + tid;
            scale_s[st * kPreKeys + tid] = j <= last ? p.kscale[scale_at(p, whole ? pg0 : page_of(p, seq, j), j)] : 0.f;
        }
        cp_async_commit();
    };
    for (int i = tid; i < kPreRows * chunks; i += kPreThreads) {
        const int r = i / chunks, c = i % chunks, tok = r / rep, h = g * rep + r % rep;
        const bool live = tok < n_tok && c * 8 < dim;
        const bf16* src = live ? q + ((long long)(sq.start + first + tok) * p.heads + h) * dim + c * 8 : q;
        cp_async16(sm0 + L::q + r * L::stride + c * 16, src, live);
    }
    if (p.bias)
        for (int i = tid; i < rep * p.nd; i += kPreThreads) bias_s[i] = p.bias[(long long)g * rep * p.nd + i] * kLog2e;
    load_tile(0, 0);

    float o[DP / 8][4];
#pragma unroll
    for (int n = 0; n < DP / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    int pos[2], head[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int r = warp * 16 + g8 + 8 * e;
        pos[e] = r / rep < n_tok ? pos0 + r / rep : last;  // rows without a token compute something harmless
        head[e] = r % rep;
    }
    const int tiles = last / kPreKeys + 1;
    for (int kt = 0; kt < tiles; kt++) {
        const int st = kt & 1, j0 = kt * kPreKeys;
        if (kt + 1 < tiles) {
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
        const unsigned ks = sm0 + L::k + st * kPreKeys * L::stride;
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
        const bool far = p.bias && pos0 - (j0 + kPreKeys - 1) >= p.nd - 1;  // one bias per head for the whole tile
        float far_bias[2] = {0.f, 0.f};
        if (far) {
            far_bias[0] = bias_s[head[0] * p.nd + p.nd - 1];
            far_bias[1] = bias_s[head[1] * p.nd + p.nd - 1];
        }
        const bool edge = j0 + kPreKeys - 1 > pos0;
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int n = 0; n < kPreKeys / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int key = n * 8 + t4 * 2 + (e & 1), r = e >> 1, d = pos[r] - (j0 + key);
                float v = s[n][e] * scale_s[st * kPreKeys + key];
                if (far) v += far_bias[r];
                else if (p.bias) v += bias_s[head[r] * p.nd + min(max(d, 0), p.nd - 1)];
                if (edge && d < 0) v = -INFINITY;
                s[n][e] = v;
                mx[r] = fmaxf(mx[r], v);
            }
#pragma unroll
        for (int r = 0; r < 2; r++) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float keep = exp2f(m[r] - mx[r]);  // key 0 is visible to every row: mx is finite from the first tile on
            m[r] = mx[r];
            l[r] *= keep;
#pragma unroll
            for (int n = 0; n < DP / 8; n++) {
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
            for (int n = 0; n < DP / 8; n += 2) {
                unsigned b[4];
                ldmatrix_x4_trans(b, ks + (kk * 16 + (lane & 15)) * L::stride + n * 16 + (lane >> 4) * 16);
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
        const float f = p.out_scale / l[r];
        bf16* out = (bf16*)p.out + ((long long)(sq.start + first + tok) * p.heads + g * rep + head[r]) * dim;
#pragma unroll
        for (int n = 0; n < DP / 8; n++) {
            const int d = n * 8 + t4 * 2;
            if (d < dim) *reinterpret_cast<unsigned*>(out + d) = pack_bf16(o[n][2 * r] * f, o[n][2 * r + 1] * f);
        }
    }
}

// ───────────────────────────── decode ───────────────────────────────────
constexpr int kDecWarps = 4, kDecThreads = kDecWarps * 32, kDecPages = 256;

// NH groups of eight query heads of one key head
template <int DP, int NH> struct DecSmem {
    static constexpr int rows = 8 * NH;
    static constexpr int keys = DP <= 128 ? 32 : 16;             // keys of a warp's tile
    static constexpr int stages = DP <= 64 ? 3 : 2;
    static constexpr int stride = DP * 2 + 16;
    static constexpr int tile = keys * stride;
    static constexpr int q = 0;                                  // [rows][stride]
    static constexpr int k = rows * stride;                      // [warps][stages][tile]
    static constexpr int ring = kDecWarps * stages * tile;
    static constexpr int part = part_size(rows, DP);             // floats of one partial result
    static constexpr int merge = kDecWarps * part * 4;           // reuses the ring after the last key
    static constexpr int total = k + (ring > merge ? ring : merge);
};

// Grid: (splits, kv_heads · groups of 8 · NH query heads, sequences).
template <int DP, int NH> __global__ void __launch_bounds__(kDecThreads) paged_attn_decode(const PagedP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float red[32];
    __shared__ unsigned arrived;
    __shared__ int page_s[kDecPages];  // this CTA's pages, checked
    using L = DecSmem<DP, NH>;
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    // no launch of a step writes the batch description or the cached keys before the step's own: they may be read
    // while the launches before this one finish
    const SeqRow sq = load_seq(p.seqs, blockIdx.z);
    const int rep = p.heads / p.kv_heads, groups = (rep + L::rows - 1) / L::rows, g = blockIdx.y / groups, h0 = g * rep + (blockIdx.y % groups) * L::rows;
    const int n_heads = min(L::rows, (g + 1) * rep - h0), seq = blockIdx.z, pos = sq.past, dim = p.dim;
    const int hq = p.heads * dim, hk = p.kv_heads * dim;
    const bf16 *q = (const bf16*)p.proj + (long long)sq.start * p.ld + p.q_off, *k = (const bf16*)p.proj + (long long)sq.start * p.ld + p.k_off;
    bf16* pool = (bf16*)p.pool;
    const unsigned sm0 = smem_u32(smem);

    // keys of this CTA: whole tiles of all four warps, so that a split never cuts a tile
    constexpr int step = L::keys * kDecWarps;
    const int blocks = sq.len == 1 ? (pos + step) / step : 0;
    const int b0 = (int)((long long)blocks * blockIdx.x / p.splits), b1 = (int)((long long)blocks * (blockIdx.x + 1) / p.splits);
    const int lo = b0 * step, hi = min(b1 * step, pos + 1);
    const int page0 = lo >> p.shift, n_pages = lo < hi ? ((hi - 1) >> p.shift) - page0 + 1 : 0;
    for (int i = tid; i < min(n_pages, kDecPages); i += kDecThreads) page_s[i] = (int)page_of(p, seq, (page0 + i) << p.shift);
    __syncthreads();
    auto page_at = [&](int j) {
        const int i = (j >> p.shift) - page0;
        return i < kDecPages ? (long long)page_s[i] : page_of(p, seq, j);
    };
    const unsigned ring = sm0 + L::k + warp * L::stages * L::tile;
    const int first = lo + warp * L::keys, tiles = first < hi ? (hi - first + step - 1) / step : 0;
    float ksc[L::stages];
    auto load_tile = [&](int i) {
        const int j0 = first + i * step;
        if (i < tiles) {
            const unsigned dst = ring + (i % L::stages) * L::tile;
            // a tile lies in one page when pages are a multiple of it
            const bool whole = (1 << p.shift) >= L::keys;
            const bf16* base = whole ? pool + key_row(p, page_at(j0), g, j0) * dim : pool;
            constexpr int per_key = DP / 8;
            if constexpr (32 % per_key == 0)
                if (whole && dim == DP && j0 + L::keys <= hi) {  // the tile is one contiguous run: a lane's copies are evenly spaced
                    const unsigned d = dst + (lane / per_key) * L::stride + (lane % per_key) * 16;
#pragma unroll
                    for (int c = 0; c < L::keys * per_key / 32; c++) cp_async16(d + c * (32 / per_key) * L::stride, base + lane * 8 + c * 256);
                    cp_async_commit();
                    return;
                }
#pragma unroll 4
            for (int c = lane; c < L::keys * (DP / 8); c += 32) {
                const int key = c / (DP / 8), ch = c % (DP / 8);
                const bool live = j0 + key < hi && ch * 8 < dim;
                const bf16* src = base + key * dim + ch * 8;
                if (!live) src = pool;
                else if (!whole) src = pool + key_row(p, page_at(j0 + key), g, j0 + key) * dim + ch * 8;
                cp_async16(dst + key * L::stride + ch * 16, src, live);
            }
        }
        cp_async_commit();
    };
    // the reciprocal root mean squares of a tile's keys, one per lane (the new key's is put in below)
    auto load_scale = [&](int i) {
        const int j = first + i * step + lane;
        return i < tiles && lane < L::keys && j < min(hi, pos) ? p.kscale[scale_at(p, page_at(j), j)] : 0.f;
    };
    const bool newest = hi == pos + 1 && lo < hi;  // this CTA's keys include the new one
    auto fill = [&]() {
#pragma unroll
        for (int i = 0; i < L::stages - 1; i++) {
            load_tile(i);
            ksc[i] = load_scale(i);
        }
    };
    if (!newest) fill();
    pdl_wait();
    if (sq.len != 1) return;
    if (newest) {
        for (int i = tid; i < dim; i += kDecThreads) pool[key_row(p, page_at(pos), g, pos) * dim + i] = k[g * dim + i];
        __syncthreads();
        fill();
    }
    // both norms in one pass over the projection's row
    float ss_q = row_sumsq(q, hq, p.vec), ss_k = newest ? row_sumsq(k, hk, p.vec) : 0.f;
    ss_q = warp_sum(ss_q);
    ss_k = warp_sum(ss_k);
    if (lane == 0) {
        red[warp] = ss_q;
        red[kDecWarps + warp] = ss_k;
    }
    __syncthreads();
    ss_q = ss_k = 0.f;
#pragma unroll
    for (int w = 0; w < kDecWarps; w++) {
        ss_q += red[w];
        ss_k += red[kDecWarps + w];
    }
    const float new_scale = 1.f / sqrtf(ss_k / (float)hk + p.eps);
    if (newest && tid == 0) p.kscale[scale_at(p, page_at(pos), pos)] = new_scale;  // every head's CTA stores the same value
    const float qr = 1.f / sqrtf(ss_q / (float)hq + p.eps) * query_factor(p, pos);
#pragma unroll 4
    for (int i = tid; i < L::rows * DP; i += kDecThreads) {
        const int r = i / DP, c = i % DP;
        float v = 0.f;
        if (r < n_heads && c < dim) v = to_f(q[(h0 + r) * dim + c]) * qr * p.qw[(h0 + r) * dim + c] * p.kw[g * dim + c];
        *reinterpret_cast<bf16*>(smem + L::q + r * L::stride + c * 2) = __float2bfloat16_rn(v);
    }
    float far_bias[NH][2];  // of this lane's heads, for keys beyond the bias table
#pragma unroll
    for (int h = 0; h < NH; h++)
#pragma unroll
        for (int e = 0; e < 2; e++)
            far_bias[h][e] = p.bias ? p.bias[(long long)(h0 + min(h * 8 + t4 * 2 + e, n_heads - 1)) * p.nd + p.nd - 1] * kLog2e : 0.f;
    __syncthreads();

    // Keys are the rows of both products (S^T = K q^T, O^T = K^T P^T): a lane holds scores of keys g, g + 8 and heads 2t, 2t + 1.
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
        m[h][0] = m[h][1] = -INFINITY;
        l[h][0] = l[h][1] = 0.f;
    }
    for (int i0 = 0; i0 < tiles; i0 += L::stages) {
#pragma unroll
        for (int u = 0; u < L::stages; u++) {
            const int i = i0 + u;
            if (i >= tiles) break;
            cp_async_wait<L::stages - 2>();
            __syncwarp();
            load_tile(i + L::stages - 1);  // the slot was read in the previous iteration
            const unsigned ks = ring + u * L::tile;
            const int j0 = first + i * step;
            const float scale = j0 + lane == pos ? new_scale : ksc[u];
            ksc[(u + L::stages - 1) % L::stages] = load_scale(i + L::stages - 1);
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
            const bool far = !p.bias || pos - (j0 + L::keys - 1) >= p.nd - 1, tail = j0 + L::keys > hi;
#pragma unroll
            for (int a = 0; a < MT; a++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int key = a * 16 + g8 + 8 * r;
                    const float f = __shfl_sync(0xffffffffu, scale, key);
                    const int d = min(max(pos - (j0 + key), 0), p.nd - 1);
#pragma unroll
                    for (int h = 0; h < NH; h++)
#pragma unroll
                        for (int e = 0; e < 2; e++) {
                            float v = s[a][h][2 * r + e] * f;
                            if (far) v += far_bias[h][e];
                            else v += p.bias[(long long)(h0 + min(h * 8 + t4 * 2 + e, n_heads - 1)) * p.nd + d] * kLog2e;
                            if (tail && j0 + key >= hi) v = -INFINITY;
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
                    moved |= mx[h][e] != m[h][e];  // the tile's first key is live: mx is finite
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
                    ldmatrix_x4_trans(va, ks + (a * 16 + (lane >> 4) * 8 + (lane & 7)) * L::stride + n * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
                    for (int h = 0; h < NH; h++) mma_bf16(o[n][h], va[0], va[1], va[2], va[3], pb[h][0], pb[h][1]);
                }
            }
            __syncwarp();
        }
    }
    cp_async_wait<0>();
    __syncthreads();  // the ring becomes the merge area
    float* parts = reinterpret_cast<float*>(smem + L::k);
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
    bf16* out = (bf16*)p.out + ((long long)sq.start * p.heads + h0) * dim;
    if (p.splits == 1) {
        merge_parts<DP, L::rows, kDecWarps>(parts, kDecWarps, n_heads, dim, p.out_scale, out, nullptr);
        return;
    }
    const long long cell = (long long)blockIdx.z * gridDim.y + blockIdx.y;
    merge_parts<DP, L::rows, kDecWarps>(parts, kDecWarps, n_heads, dim, 0.f, nullptr, p.part + (cell * p.splits + blockIdx.x) * L::part);
    __threadfence();
    __syncthreads();
    if (tid == 0) arrived = atomicAdd(&p.counters[cell], 1u);
    __syncthreads();
    if (arrived != (unsigned)p.splits - 1) return;
    __threadfence();
    if (tid == 0) p.counters[cell] = 0;
    merge_parts<DP, L::rows, kDecWarps>(p.part + cell * p.splits * L::part, p.splits, n_heads, dim, p.out_scale, out, nullptr);
}

using PagedKernel = void (*)(const PagedP);
struct DimChoice {
    int dp;
    PagedKernel prefill, decode[2];
    int pre_smem, dec_smem[2], dec_part[2];
};
template <int DP> DimChoice choice() {
    return {DP, paged_attn_prefill<DP>, {paged_attn_decode<DP, 1>, paged_attn_decode<DP, 2>}, PreSmem<DP>::bias,
            {DecSmem<DP, 1>::total, DecSmem<DP, 2>::total}, {DecSmem<DP, 1>::part, DecSmem<DP, 2>::part}};
}
DimChoice dim_choice(int64_t dim) {
    return dim <= 32 ? choice<32>() : dim <= 64 ? choice<64>() : dim <= 96 ? choice<96>() : dim <= 128 ? choice<128>() : dim <= 192 ? choice<192>() : choice<256>();
}

}  // namespace

void emit_paged_attention(Emitter& em, const PagedAttnDesc& d, const TRef& proj, const TRef& q_norm, const TRef& k_norm, const TRef* bias,
                          const TRef& pool, const TRef& key_scale, const TRef& seqs, const TRef& pages, const TRef& out) {
    const int64_t rows = proj.shape[0], n_seqs = seqs.shape[0];
    if (rows == 0) return;
    PagedP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.q_off = d.q_off;
    p.k_off = d.k_off;
    p.n_seqs = (int)n_seqs;
    p.width = (int)pages.shape[1];
    p.n_pages = (int)pool.shape[0];
    while ((int64_t)1 << p.shift < d.page) p.shift++;
    p.heads = (int)d.heads;
    p.kv_heads = (int)d.kv_heads;
    p.dim = (int)d.dim;
    p.nd = bias ? (int)bias->shape[1] : 0;
    p.eps = (float)d.eps;
    p.temp_coef = (float)d.temp_coef;
    p.temp_every = d.temp_every;
    p.out_scale = (float)d.out_scale;
    p.node = em.node;
    p.splits = 1;
    const int64_t rep = d.heads / d.kv_heads;
    const bool bf = proj.dtype == DT_BF16;
    const DimChoice dc = dim_choice(d.dim);
    const int64_t pre_smem = dc.pre_smem + rep * p.nd * 4;
    // 16-byte copies of key rows; the bias rows of a key head's queries in shared memory
    const bool tc = bf && d.dim % 8 == 0 && d.dim <= 256 && rep <= kPreRows && pre_smem <= 220 * 1024;
    const Buf bb = bias ? bias->buf : Buf{kSlotNull, 0}, err{kSlotErr, 0};
    const bool decode_only = tc && rows == n_seqs;  // every sequence has one new token
    p.qmul = (float)(tc ? d.scale * 1.4426950408889634 : d.scale);
    p.singles = !tc;
    p.vec = bf && d.dim % 8 == 0 && p.ld % 8 == 0 && d.q_off % 8 == 0 && d.k_off % 8 == 0 && proj.buf.off % 16 == 0;
    const Buf q = decode_only ? Buf{kSlotNull, 0} : em.scratch((size_t)rows * d.heads * d.dim * (bf ? 2 : 4));
    auto launch = [&](PagedKernel k, dim3 grid, unsigned block, unsigned smem, Buf part, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.proj, proj.buf}, {&p.qw, q_norm.buf}, {&p.kw, k_norm.buf}, {&p.bias, bb}, {&p.pool, pool.buf}, {&p.kscale, key_scale.buf},
                   {&p.q, q}, {&p.out, out.buf}, {&p.seqs, seqs.buf}, {&p.table, pages.buf}, {&p.part, part}, {&p.counters, Buf{kSlotCounters, 0}}, {&p.err, err}},
                  label, /*pdl=*/true);
    };
    const Buf none{kSlotNull, 0};
    if (!decode_only) launch(bf ? paged_prepare<bf16> : paged_prepare<float>, dim3((unsigned)rows), 128, 0, none, "paged_prepare");
    if (!tc) {
        const unsigned smem = (unsigned)((2 * d.dim + 128) * 4);
        const PagedKernel k = bf ? paged_attn_simt<bf16> : paged_attn_simt<float>;
        ensure_max_dynamic_smem((const void*)k, 220 * 1024);
        launch(k, dim3((unsigned)rows, (unsigned)d.heads), 128, smem, none, "paged_attn_simt");
        return;
    }
    if (!decode_only) {
        const int64_t tq = kPreRows / rep;
        ensure_max_dynamic_smem((const void*)dc.prefill, 220 * 1024);
        launch(dc.prefill, dim3((unsigned)((rows + tq - 1) / tq + n_seqs), (unsigned)d.kv_heads), kPreThreads, (unsigned)pre_smem, none, "paged_attn_prefill");
    }
    if (decode_only || n_seqs > 1) {
        const int nh = rep > 8;  // two groups of eight heads per CTA
        const int64_t groups = d.kv_heads * ((rep + 8 * nh + 7) / (8 * nh + 8)), cells = n_seqs * groups;
        // splits of the longest sequence the page tables can hold: whole waves of resident CTAs, each with a fixed cost
        // worth about 160 keys, and the pieces have to be merged
        const int64_t resident = std::max<int64_t>(1, std::min<int64_t>(nh ? (d.dim > 192 ? 2 : 3) : 4, 224 * 1024 / (dc.dec_smem[nh] + 2560))), slots = resident * sm_count();
        const int64_t keys = (int64_t)p.width * d.page;
        int64_t splits = 1;
        double best = 1e300;
        for (int64_t sp = 1; sp <= 64 && sp * 128 <= std::max<int64_t>(keys, 128); sp++) {
            const double us = (double)((cells * sp + slots - 1) / slots) * ((double)keys / sp + 160.0) + 4.0 * sp;
            if (us < best) {
                best = us;
                splits = sp;
            }
        }
        if (cells > (int64_t)kCounterWords) splits = 1;
        p.splits = (int)splits;
        const Buf part = splits > 1 ? em.scratch((size_t)cells * splits * dc.dec_part[nh] * 4) : none;
        ensure_max_dynamic_smem((const void*)dc.decode[nh], dc.dec_smem[nh]);
        launch(dc.decode[nh], dim3((unsigned)splits, (unsigned)groups, (unsigned)n_seqs), kDecThreads, (unsigned)dc.dec_smem[nh], part,
               "paged_attn_decode");
    }
}

}  // namespace oxk
