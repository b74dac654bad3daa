// Attention over one latent per token that all heads share: key = (latent, rotated part), value = latent. Queries come with their
// unrotated part mapped into the latent space, results leave in it; both maps are block-diagonal products (linear.cu).
//
//   latent_prepare   the new latents, normed, and their rotated part go to the pool; queries' rotated parts are rotated
//   latent_attend    bf16: M (token, head) rows per CTA share each tile of keys, which is read once for both products; scores and
//                    weights pass through shared memory, since the warps split the keys in the first product and the value
//                    dimensions in the second. The keys of a row tile can be split over CTAs; the last one to arrive merges.
//                    For sequences with one new token it also does latent_prepare's work
//   f32, and sizes that latent_attend does not take: paged_kv_attention.cu, one key head, values at the front of the keys
//
// Decode reads past · (rank + rot) · 2 bytes per sequence; prefill 2 · S · T · heads · (2 rank + rot) FLOPs.
#include <type_traits>

#include "paged_util.cuh"

namespace oxk {

namespace {

struct LatP {
    const void* q_latent;        // [rows, heads · rank]
    const void* q_own;           // rotated parts: row · q_ld + head · q_step
    const void* proj;            // new latents: row · ld
    const float* norm_w;         // [rank]
    const float* turns;          // [2, rot / 2]
    void* pool;                  // [pages, page, rank + rot]
    void* q;                     // [rows, heads · rot]: rotated parts; with `whole` [rows, heads · (rank + rot)], complete queries
    const int* seqs;             // [R, 4]
    const int* table;            // [R, width]
    void* out;                   // [rows, heads · rank]
    float* part;                 // [cells, splits, M, rank padded + 2]
    unsigned* counters;
    ErrWord* err;
    long long rows, ld, q_ld;
    int n_seqs, width, n_pages, shift, heads, kv_heads, rank, rot, q_step, node;
    int splits, stages, per_cta;  // per_cta: heads of a row tile
    int singles, whole;           // prepare: also sequences with one new token; complete queries
    float eps, mul2;              // log2 e · scale
};

// One CTA per row.
template <typename T> __global__ void __launch_bounds__(128) latent_prepare(const LatP p) {
    extern __shared__ float angle[];  // cos[rot / 2], sin[rot / 2]
    __shared__ float red[32];
    pdl_enter();
    const int row = blockIdx.x, s = find_seq(p.seqs, p.n_seqs, row), tid = threadIdx.x, half = p.rot / 2, dim = p.rank + p.rot;
    const SeqRow sq = load_seq(p.seqs, s);
    const int pos = sq.past + row - sq.start;
    if (row >= sq.start + sq.len || (sq.len == 1 && !p.singles)) return;
    angles(p.turns, half, pos, angle, angle + half, tid, 128);
    const T* x = (const T*)p.proj + (long long)row * p.ld;
    float ss = 0.f;
    for (int i = tid; i < p.rank; i += 128) {
        const float v = to_f(x[i]);
        ss = fmaf(v, v, ss);
    }
    const float f = 1.f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);  // (its barriers order the angles)
    T* dst = (T*)p.pool + key_row(p, page_of(p, s, pos), 0, pos) * dim;
    for (int i = tid; i < p.rank; i += 128) dst[i] = from_f<T>(to_f(x[i]) * f * p.norm_w[i]);
    for (int i = tid; i < p.rot; i += 128) dst[p.rank + i] = from_f<T>(rotated(half, 0, x + p.rank, angle, angle + half, i));
    const T *lat = (const T*)p.q_latent + (long long)row * p.heads * p.rank, *own = (const T*)p.q_own + (long long)row * p.q_ld;
    const int front = p.whole ? p.rank : 0, size = front + p.rot;
    T* q = (T*)p.q + (long long)row * p.heads * size;
    for (int k = tid; k < p.heads * p.rot; k += 128) {
        const int h = k / p.rot, i = k - h * p.rot;
        q[h * size + front + i] = from_f<T>(rotated(half, 0, own + (long long)h * p.q_step, angle, angle + half, i));
    }
    if (p.whole)
        for (int h = 0; h < p.heads; h++)
            for (int i = tid; i < p.rank; i += 128) q[h * size + i] = lat[h * p.rank + i];
}

// ───────────────────────────── tensor cores ─────────────────────────────
constexpr int kLatThreads = 256, kLatWarps = 8, kLatSplits = 32;
constexpr float kNoScore = -1e30f;  // below every score, and finite: differences stay numbers

// M rows; the rank is padded to NT · 64: a warp owns NT · 8 value dimensions.
template <int M> struct LatShape {
    static constexpr int row_tiles = M / 16, key_parts = kLatWarps / row_tiles;
    static constexpr int keys = M == 16 ? 64 : 32;                 // of a tile
    static constexpr int key_tiles = keys / key_parts / 8;         // groups of eight keys of a warp in the first product
    static constexpr int row_threads = kLatThreads / M, row_keys = keys / row_threads;  // softmax
    static constexpr int score_stride = keys + 4, weight_stride = keys * 2 + 16;  // floats; bytes
};
__host__ __device__ constexpr int lat_dim(int dim) { return (dim + 31) / 32 * 32; }
__host__ __device__ constexpr int lat_stride(int dim) { return lat_dim(dim) * 2 + 16; }  // bytes per row: conflict-free ldmatrix
template <int M> __host__ __device__ constexpr int lat_smem(int dim, int rot, int stages) {
    using L = LatShape<M>;
    return (M + stages * L::keys) * lat_stride(dim) + M * L::score_stride * 4 + M * L::weight_stride + M * 12 + rot * 4;
}

// Grid: (splits of row tiles or sequences, head groups).
template <int M, int NT, bool DECODE> __global__ void __launch_bounds__(kLatThreads, NT <= 4 ? 2 : 1) latent_attend(const LatP p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float red[32];
    __shared__ unsigned arrived;
    using L = LatShape<M>;
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    const int rank = p.rank, dim = p.rank + p.rot, half = p.rot / 2, stride = lat_stride(dim), chunks = lat_dim(dim) / 8;
    if constexpr (!DECODE) pdl_wait();
    const int unit = (int)blockIdx.x / p.splits, split = (int)blockIdx.x - unit * p.splits, tq = M / p.per_cta;
    int seq = unit, first = 0;
    // long rows first: the last tiles of a sequence see the most keys
    if (!DECODE && !locate_tile(p.seqs, p.n_seqs, (int)gridDim.x / p.splits - 1 - unit, tq, &seq, &first)) return;
    const SeqRow sq = load_seq(p.seqs, seq);  // no launch of a step writes the batch description
    const int h0 = blockIdx.y * p.per_cta, n_heads = min(p.per_cta, p.heads - h0);
    const int n_tok = DECODE ? 1 : min(tq, sq.len - first), pos0 = sq.past + first, last = pos0 + n_tok - 1;
    const int all = last / L::keys + 1;
    int kt0 = (int)((long long)all * split / p.splits), kt1 = (int)((long long)all * (split + 1) / p.splits);
    if (DECODE && sq.len != 1) kt0 = kt1 = 0;

    const unsigned sm_q = smem_u32(smem), sm_kv = sm_q + M * stride;
    unsigned char* after = smem + (size_t)(M + p.stages * L::keys) * stride;
    float* scores = reinterpret_cast<float*>(after);                       // [M][score_stride]
    unsigned char* weights = after + M * L::score_stride * 4;              // [M][weight_stride]
    float* row_scale = reinterpret_cast<float*>(weights + M * L::weight_stride);
    float *row_max = row_scale + M, *row_sum = row_max + M;
    float *cs = row_sum + M, *sn = cs + half;
    bf16* pool = (bf16*)p.pool;

    auto load_tile = [&](int kt) {
        if (kt < kt1) {
            const int j0 = kt * L::keys;
            const bool whole = (1 << p.shift) >= L::keys;  // the tile lies in one page
            const long long row0 = whole ? key_row(p, page_of(p, seq, j0), 0, j0) : 0;
            const unsigned dst = sm_kv + (unsigned)(kt % p.stages) * L::keys * stride;
#pragma unroll 4
            for (int i = tid; i < L::keys * chunks; i += kLatThreads) {
                const int key = i / chunks, c = i - key * chunks;
                const bool live = j0 + key <= last && c * 8 < dim;
                long long row = row0 + key;
                if (!whole) row = live ? key_row(p, page_of(p, seq, j0 + key), 0, j0 + key) : 0;
                cp_async16(dst + key * stride + c * 16, live ? pool + row * dim + c * 8 : pool, live);
            }
        }
        cp_async_commit();
    };
    auto fill = [&]() {
        for (int i = 0; i < p.stages - 1; i++) load_tile(kt0 + i);
    };
    if constexpr (DECODE) {
        const bool newest = kt1 == all && kt0 < kt1;  // this CTA's keys include the new one
        if (!newest) fill();  // earlier steps' keys: may overlap the launches before this one
        angles(p.turns, half, pos0, cs, sn, tid, kLatThreads);
        pdl_wait();
        if (sq.len != 1) return;
        __syncthreads();
        if (newest) {
            const bf16* x = (const bf16*)p.proj + (long long)sq.start * p.ld;
            float ss = 0.f;
            for (int i = tid; i < rank; i += kLatThreads) {
                const float v = to_f(x[i]);
                ss = fmaf(v, v, ss);
            }
            const float f = 1.f / sqrtf(block_sum(ss, red) / (float)rank + p.eps);
            bf16* dst = pool + key_row(p, page_of(p, seq, pos0), 0, pos0) * dim;
            for (int i = tid; i < rank; i += kLatThreads) dst[i] = __float2bfloat16_rn(to_f(x[i]) * f * p.norm_w[i]);
            for (int i = tid; i < p.rot; i += kLatThreads) dst[rank + i] = __float2bfloat16_rn(rotated(half, 0, x + rank, cs, sn, i));
            __syncthreads();
            fill();
        }
        const bf16 *lat = (const bf16*)p.q_latent + ((long long)sq.start * p.heads + h0) * rank, *own = (const bf16*)p.q_own + (long long)sq.start * p.q_ld;
        for (int i = tid; i < M * chunks; i += kLatThreads) {
            const int r = i / chunks, c = i - r * chunks;
            bf16* to = reinterpret_cast<bf16*>(smem + r * stride + c * 16);
            if (r < n_heads && c * 8 < rank) {
                *reinterpret_cast<uint4*>(to) = *reinterpret_cast<const uint4*>(lat + (long long)r * rank + c * 8);
            } else {
#pragma unroll
                for (int e = 0; e < 8; e++) {
                    const int d = c * 8 + e - rank;
                    to[e] = __float2bfloat16_rn(r < n_heads && d < p.rot ? rotated(half, 0, own + (long long)(h0 + r) * p.q_step, cs, sn, d) : 0.f);
                }
            }
        }
    } else {
        const bf16 *lat = (const bf16*)p.q_latent, *own = (const bf16*)p.q;
        for (int i = tid; i < M * chunks; i += kLatThreads) {
            const int r = i / chunks, c = i - r * chunks, tok = r / p.per_cta, h = r - tok * p.per_cta;
            const bool live = tok < n_tok && h < n_heads && c * 8 < dim;
            const long long at = (long long)(sq.start + first + tok) * p.heads + h0 + h;
            cp_async16(sm_q + r * stride + c * 16, !live ? lat : c * 8 < rank ? lat + at * rank + c * 8 : own + at * p.rot + c * 8 - rank, live);
        }
        fill();
    }

    float o[L::row_tiles][NT][4];
#pragma unroll
    for (int r = 0; r < L::row_tiles; r++)
#pragma unroll
        for (int n = 0; n < NT; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[r][n][e] = 0.f;
    const int s_row = tid / L::row_threads, s_key = (tid % L::row_threads) * L::row_keys;  // softmax: this thread's row and keys
    const int s_tok = s_row / p.per_cta, s_pos = s_tok < n_tok ? pos0 + s_tok : last;      // rows without a token compute something harmless
    float m = kNoScore, l = 0.f;
    for (int kt = kt0; kt < kt1; kt++) {
        if (p.stages == 2) cp_async_wait<0>();
        else if (p.stages == 3) cp_async_wait<1>();
        else cp_async_wait<2>();
        __syncthreads();
        load_tile(kt + p.stages - 1);  // that slot was read in the previous iteration
        const unsigned ks = sm_kv + (unsigned)(kt % p.stages) * L::keys * stride;
        {
            const int rt = warp % L::row_tiles, key0 = warp / L::row_tiles * (L::key_tiles * 8);
            float s[L::key_tiles][4];
#pragma unroll
            for (int n = 0; n < L::key_tiles; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) s[n][e] = 0.f;
            const unsigned qa = sm_q + (rt * 16 + (lane & 15)) * stride + (lane >> 4) * 16;
            const unsigned ka = ks + (key0 + (lane & 7)) * stride + (lane >> 3) * 16;
#pragma unroll 3
            for (int kk = 0; kk < chunks / 4; kk++) {
                unsigned a0[4], a1[4];
                ldmatrix_x4(a0, qa + kk * 64);
                ldmatrix_x4(a1, qa + kk * 64 + 32);
#pragma unroll
                for (int n = 0; n < L::key_tiles; n++) {
                    unsigned b[4];  // eight keys, 32 dimensions
                    ldmatrix_x4(b, ka + n * 8 * stride + kk * 64);
                    mma_bf16(s[n], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                    mma_bf16(s[n], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int n = 0; n < L::key_tiles; n++)
#pragma unroll
                for (int r = 0; r < 2; r++)
                    *reinterpret_cast<float2*>(scores + (rt * 16 + g8 + 8 * r) * L::score_stride + key0 + n * 8 + t4 * 2) = make_float2(s[n][2 * r], s[n][2 * r + 1]);
        }
        __syncthreads();
        bool moved;
        {
            float v[L::row_keys], mx = m;
#pragma unroll
            for (int i = 0; i < L::row_keys; i += 4) *reinterpret_cast<float4*>(v + i) = *reinterpret_cast<const float4*>(scores + s_row * L::score_stride + s_key + i);
            const int j0 = kt * L::keys + s_key;
#pragma unroll
            for (int i = 0; i < L::row_keys; i++) {
                v[i] = j0 + i > s_pos ? -INFINITY : v[i] * p.mul2;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int d = 1; d < L::row_threads; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float keep = exp2f(m - mx);
            moved = mx != m;
            m = mx;
            l *= keep;
            unsigned packed[L::row_keys / 2];
#pragma unroll
            for (int i = 0; i < L::row_keys; i += 2) {
                const float a = exp2f(v[i] - m), b = exp2f(v[i + 1] - m);
                l += a + b;
                packed[i / 2] = pack_bf16(a, b);
            }
#pragma unroll
            for (int i = 0; i < L::row_keys / 2; i += 2)
                *reinterpret_cast<uint2*>(weights + s_row * L::weight_stride + (s_key + 2 * i) * 2) = make_uint2(packed[i], packed[i + 1]);
            if (tid % L::row_threads == 0) row_scale[s_row] = keep;
        }
        if (__syncthreads_or(moved)) {
#pragma unroll
            for (int r = 0; r < L::row_tiles; r++) {
                const float f0 = row_scale[r * 16 + g8], f1 = row_scale[r * 16 + g8 + 8];
#pragma unroll
                for (int n = 0; n < NT; n++) {
                    o[r][n][0] *= f0;
                    o[r][n][1] *= f0;
                    o[r][n][2] *= f1;
                    o[r][n][3] *= f1;
                }
            }
        }
        const unsigned wa = smem_u32(weights) + (lane & 15) * L::weight_stride + (lane >> 4) * 16;
        const unsigned va = ks + (lane & 15) * stride + warp * (NT * 16) + (lane >> 4) * 16;
#pragma unroll
        for (int kk = 0; kk < L::keys / 16; kk++) {
            unsigned a[L::row_tiles][4];
#pragma unroll
            for (int r = 0; r < L::row_tiles; r++) ldmatrix_x4(a[r], wa + r * 16 * L::weight_stride + kk * 32);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                // dimensions beyond the row are another tile's bytes or this tile's next row: finite, and never stored
                unsigned b[4];
                ldmatrix_x4_trans(b, va + kk * 16 * stride + n * 16);
#pragma unroll
                for (int r = 0; r < L::row_tiles; r++) {
                    mma_bf16(o[r][n], a[r][0], a[r][1], a[r][2], a[r][3], b[0], b[1]);
                    mma_bf16(o[r][n + 1], a[r][0], a[r][1], a[r][2], a[r][3], b[2], b[3]);
                }
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int d = 1; d < L::row_threads; d <<= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
    if (tid % L::row_threads == 0) {
        row_max[s_row] = m;
        row_sum[s_row] = l;
    }
    __syncthreads();
    constexpr int RP = NT * 64, part_floats = M * (RP + 2);
    auto row_out = [&](int row) { return (bf16*)p.out + ((long long)(sq.start + first + row / p.per_cta) * p.heads + h0 + row % p.per_cta) * rank; };
    auto wanted = [&](int row) { return row / p.per_cta < n_tok && row % p.per_cta < n_heads; };
    const long long cell = (long long)unit * gridDim.y + blockIdx.y;
    float* mine = p.part + (cell * p.splits + split) * part_floats;
#pragma unroll
    for (int r = 0; r < L::row_tiles; r++)
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int row = r * 16 + g8 + 8 * k;
            if (!wanted(row)) continue;
            const float f = p.splits == 1 ? 1.f / row_sum[row] : 1.f;
#pragma unroll
            for (int n = 0; n < NT; n++) {
                const int d = warp * (NT * 8) + n * 8 + t4 * 2;
                if (d >= rank) continue;
                if (p.splits == 1) *reinterpret_cast<unsigned*>(row_out(row) + d) = pack_bf16(o[r][n][2 * k] * f, o[r][n][2 * k + 1] * f);
                else *reinterpret_cast<float2*>(mine + row * (RP + 2) + 2 + d) = make_float2(o[r][n][2 * k], o[r][n][2 * k + 1]);
            }
        }
    if (p.splits == 1) return;
    if (tid < M) *reinterpret_cast<float2*>(mine + tid * (RP + 2)) = make_float2(row_max[tid], row_sum[tid]);
    __threadfence();
    __syncthreads();
    if (tid == 0) arrived = atomicAdd(&p.counters[cell], 1u);
    __syncthreads();
    if (arrived != (unsigned)p.splits - 1) return;
    __threadfence();
    if (tid == 0) p.counters[cell] = 0;
    const float* parts = p.part + cell * p.splits * part_floats;
    float* factor = scores;  // [splits][M]: splits · M ≤ M · score_stride
    if (tid < M) {
        float top = kNoScore, sum = 0.f;
        for (int i = 0; i < p.splits; i++) top = fmaxf(top, parts[(long long)i * part_floats + tid * (RP + 2)]);
        for (int i = 0; i < p.splits; i++) {
            const float2 v = *reinterpret_cast<const float2*>(parts + (long long)i * part_floats + tid * (RP + 2));
            const float f = exp2f(v.x - top);
            factor[i * M + tid] = f;
            sum = fmaf(v.y, f, sum);
        }
        row_sum[tid] = 1.f / sum;
    }
    __syncthreads();
    const int pairs = rank / 2;
    for (int i = tid; i < M * pairs; i += kLatThreads) {
        const int row = i / pairs, d = (i - row * pairs) * 2;
        if (!wanted(row)) continue;
        float a = 0.f, b = 0.f;
#pragma unroll 4
        for (int k = 0; k < p.splits; k++) {
            const float2 v = *reinterpret_cast<const float2*>(parts + (long long)k * part_floats + row * (RP + 2) + 2 + d);
            a = fmaf(v.x, factor[k * M + row], a);
            b = fmaf(v.y, factor[k * M + row], b);
        }
        *reinterpret_cast<unsigned*>(row_out(row) + d) = pack_bf16(a * row_sum[row], b * row_sum[row]);
    }
}

using LatKernel = void (*)(const LatP);
template <int M, bool DECODE> LatKernel latent_kernel(int64_t rank) {
    return rank <= 128 ? latent_attend<M, 2, DECODE> : rank <= 256 ? latent_attend<M, 4, DECODE> : rank <= 384 ? latent_attend<M, 6, DECODE> : latent_attend<M, 8, DECODE>;
}

}  // namespace

void emit_latent_attention(Emitter& em, const LatentAttnDesc& d, const TRef& q_latent, const TRef& q, const TRef& proj, const TRef& norm_w, const TRef& turns,
                           const TRef& pool, const TRef& seqs, const TRef& pages, const TRef& out) {
    const int64_t rows = proj.shape[0], dim = d.rank + d.rot;
    if (rows == 0) return;
    const bool bf = proj.dtype == DT_BF16;
    const int64_t element = bf ? 2 : 4;
    LatP p{};
    p.rows = rows;
    p.ld = proj.shape[1];
    p.q_ld = q.shape[1];
    p.n_seqs = (int)seqs.shape[0];
    p.width = (int)pages.shape[1];
    p.n_pages = (int)pool.shape[0];
    while ((int64_t)1 << p.shift < d.page) p.shift++;
    p.heads = (int)d.heads;
    p.kv_heads = 1;
    p.rank = (int)d.rank;
    p.rot = (int)d.rot;
    p.q_step = (int)d.q_step;
    p.node = em.node;
    p.eps = (float)d.eps;
    p.mul2 = (float)(d.scale * (double)kLog2e);
    const Buf none{kSlotNull, 0};
    auto launch = [&](LatKernel k, dim3 grid, unsigned block, unsigned smem, Buf q_ready, Buf part, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.q_latent, q_latent.buf}, {&p.q_own, q.buf.at(d.q_off * element)}, {&p.proj, proj.buf.at(d.kv_off * element)}, {&p.norm_w, norm_w.buf},
                   {&p.turns, turns.buf}, {&p.pool, pool.buf}, {&p.q, q_ready}, {&p.seqs, seqs.buf}, {&p.table, pages.buf}, {&p.out, out.buf}, {&p.part, part},
                   {&p.counters, Buf{kSlotCounters, 0}}, {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
    };
    const int64_t n_seqs = seqs.shape[0];
    // 16-byte copies of latents and rotated parts
    const bool tc = bf && d.rank % 8 == 0 && d.rot % 8 == 0 && d.rank <= 512 && lat_smem<64>((int)dim, (int)d.rot, 2) <= 220 * 1024;
    const bool decode_only = tc && rows == n_seqs;  // every sequence has one new token
    p.singles = p.whole = !tc;
    TRef ready;
    ready.dtype = proj.dtype;
    ready.shape = {rows, d.heads * (tc ? d.rot : dim)};
    ready.buf = none;
    if (!decode_only) {
        ready.buf = em.scratch((size_t)(rows * ready.shape[1] * element));
        launch(bf ? latent_prepare<bf16> : latent_prepare<float>, dim3((unsigned)rows), 128, (unsigned)(d.rot * 4), ready.buf, none, "latent_prepare");
    }
    if (!tc) {
        PagedKvDesc kd{};
        kd.heads = d.heads;
        kd.kv_heads = 1;
        kd.dim = dim;
        kd.vdim = d.rank;
        kd.page = d.page;
        kd.scale = d.scale;
        kd.latent = true;
        emit_paged_kv_attention(em, kd, ready, turns, pool, pool, seqs, pages, out);
        return;
    }
    auto attend = [&](auto rows_per_tile, LatKernel k, int64_t cells, int64_t groups, bool decode, const char* label) {
        constexpr int M = decltype(rows_per_tile)::value;
        const int resident = d.rank <= 256 ? 2 : 1;
        const int64_t limit = resident == 2 ? 110 * 1024 : 220 * 1024;
        p.stages = 2;
        while (p.stages < 4 && lat_smem<M>((int)dim, (int)d.rot, p.stages + 1) <= limit) p.stages++;
        // splits of the most keys a sequence can see: whole waves of resident CTAs, each with a fixed cost worth some keys
        const int64_t smem = lat_smem<M>((int)dim, (int)d.rot, p.stages), slots = (smem <= limit ? resident : 1) * sm_count(), seen = (int64_t)p.width * d.page;
        int64_t splits = 1;
        double best = 1e300;
        for (int64_t sp = 1; sp <= kLatSplits && sp * LatShape<M>::keys <= std::max<int64_t>(seen, LatShape<M>::keys); sp++) {
            if (sp > 1 && !decode && cells * groups * sp > 2 * slots) break;  // row tiles fill the device by themselves
            const double cost = (double)((cells * groups * sp + slots - 1) / slots) * ((double)seen / sp + 192.0) + 8.0 * sp;
            if (cost < best) {
                best = cost;
                splits = sp;
            }
        }
        if (cells * groups > (int64_t)kCounterWords) splits = 1;
        p.splits = (int)splits;
        const int64_t padded = (d.rank + 127) / 128 * 128;
        const Buf part = splits > 1 ? em.scratch((size_t)(cells * groups * splits * M * (padded + 2)) * 4) : none;
        ensure_max_dynamic_smem((const void*)k, 222 * 1024);
        launch(k, dim3((unsigned)(cells * splits), (unsigned)groups), kLatThreads, (unsigned)smem, ready.buf, part, label);
    };
    if (!decode_only) {
        p.per_cta = (int)std::min<int64_t>(d.heads, 64);
        const int64_t tq = 64 / p.per_cta;
        attend(std::integral_constant<int, 64>{}, latent_kernel<64, false>(d.rank), std::min<int64_t>(rows, rows / tq + n_seqs), (d.heads + p.per_cta - 1) / p.per_cta,
               false, "latent_prefill");
    }
    if (decode_only || n_seqs > 1) {
        const int M = d.heads <= 16 ? 16 : d.heads <= 32 ? 32 : 64;
        p.per_cta = (int)std::min<int64_t>(d.heads, M);
        const int64_t groups = (d.heads + M - 1) / M;
        if (M == 16) attend(std::integral_constant<int, 16>{}, latent_kernel<16, true>(d.rank), n_seqs, groups, true, "latent_decode");
        else if (M == 32) attend(std::integral_constant<int, 32>{}, latent_kernel<32, true>(d.rank), n_seqs, groups, true, "latent_decode");
        else attend(std::integral_constant<int, 64>{}, latent_kernel<64, true>(d.rank), n_seqs, groups, true, "latent_decode");
    }
}

}  // namespace oxk
