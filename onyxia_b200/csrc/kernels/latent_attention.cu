// Attention over one latent per token that all heads share: key = (latent, rotated part), value = latent. Queries come with their
// unrotated part mapped into the latent space, results leave in it; both maps are block-diagonal products (linear.cu).
//
//   latent_prepare   the new latents, normed, and their rotated part go to the pool; queries' rotated parts are rotated
//   latent_attend    bf16: M (token, head) rows per CTA share each tile of keys, which is read once for both products; scores and
//                    weights pass through shared memory, since the warps split the keys in the first product and the value
//                    dimensions in the second. Keys come by TMA, several tiles ahead. The keys of a row tile
//                    can be split over CTAs (latent_merge). For sequences with one new token it also does latent_prepare's work
//   f32, and sizes that latent_attend does not take: paged_kv_attention.cu, one key head, values at the front of the keys
//
// Decode reads past · (rank + rot) · 2 bytes per sequence; prefill 2 · S · T · heads · (2 rank + rot) FLOPs.
#include <type_traits>

#include "paged_util.cuh"

namespace oxk {

namespace {

struct LatP {
    alignas(64) unsigned char map[128];  // the pool as [pages · page, rank + rot]
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
    float *part, *stats;         // [cells, splits, M, rank padded], [cells, splits, M, 2]: results that are to be merged
    ErrWord* err;
    long long rows, ld, q_ld;
    int n_seqs, width, n_pages, shift, heads, kv_heads, rank, rot, q_step, node;
    int splits, slots, ring, per_cta;  // tiles in flight per team, bytes of the ring, heads of a row tile
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
constexpr int kLatSplits = 64, kLatSlots = 8;
constexpr float kNoScore = -1e30f;  // below every score, and finite: differences stay numbers

// M rows. Teams of warps take turns at the tiles of `keys` keys and never wait for one another; their results are added at the end.
// Within a team the warps split the keys (and dimensions, in `halves`) in the first product, the rows and keys in the softmax and the value dimensions in the second.
template <int M, bool DECODE> struct LatShape {
    static constexpr int teams = !DECODE || M == 64 ? 1 : M == 32 ? 2 : 4, warps = M == 16 ? 4 : 8;  // warps of a team
    static constexpr int team_threads = warps * 32, threads = teams * team_threads;
    static constexpr int keys = M == 16 ? 16 : 32, panel = keys * 128, halves = M == 16 ? 2 : 1;
    static constexpr int row_tiles = M / 16, key_parts = warps / row_tiles / halves, key_tiles = keys / key_parts / 8;  // groups of eight keys of a warp in the first product
    static constexpr int row_threads = team_threads / M, row_keys = keys / row_threads;              // softmax
    static constexpr int score_stride = keys + 4, weight_stride = keys * 2 + 16;                     // floats; bytes
    static constexpr int team_bytes = halves * M * score_stride * 4 + M * weight_stride + M * 12;    // scores, weights; scale, maximum and sum of every row
};
__host__ __device__ constexpr int lat_dim(int dim) { return (dim + 31) / 32 * 32; }
__host__ __device__ constexpr int lat_stride(int dim) { return lat_dim(dim) * 2 + 16; }  // bytes per row: conflict-free ldmatrix
// A tile of keys lies in panels of 64 dimensions, 128 bytes per key, swizzled as TMA does: 16-byte chunk c of key k at chunk c ^ (k & 7).
__host__ __device__ constexpr int lat_panels(int dim) { return (dim + 63) / 64; }
constexpr int lat_out_stride(int padded) { return padded + 8; }  // floats per row of a team's results
template <int M, bool DECODE> constexpr int lat_smem(int dim, int rank, int rot, int slots) {
    using L = LatShape<M, DECODE>;
    const int ring = L::teams * slots * lat_panels(dim) * L::panel, results = L::teams > 1 ? L::teams * M * lat_out_stride((rank + 127) / 128 * 128) * 4 : 0;
    return 1024 + (ring > results ? ring : results) + M * lat_stride(dim) + L::teams * L::team_bytes + rot * 4;
}
// Chunk `c` (of eight dimensions) of key `k` in a tile of panels of PANEL bytes.
template <int PANEL> __device__ __forceinline__ unsigned lat_chunk(unsigned tile, int k, int c) { return tile + (c >> 3) * PANEL + k * 128 + (((c ^ k) & 7) << 4); }

// The rows of a CTA: tokens of one sequence × heads.
struct LatTile {
    int seq, first, n_tok, h0, n_heads;
    SeqRow sq;
};
template <int M, bool DECODE> __device__ __forceinline__ bool lat_tile(const LatP& p, int unit, int units, int group, LatTile* t) {
    t->seq = unit;
    t->first = 0;
    const int tq = M / p.per_cta;
    // long rows first: the last tiles of a sequence see the most keys
    if (!DECODE && !locate_tile(p.seqs, p.n_seqs, units - 1 - unit, tq, &t->seq, &t->first)) return false;
    t->sq = load_seq(p.seqs, t->seq);
    t->n_tok = DECODE ? 1 : min(tq, t->sq.len - t->first);
    t->h0 = group * p.per_cta;
    t->n_heads = min(p.per_cta, p.heads - t->h0);
    return true;
}
__device__ __forceinline__ bool lat_wanted(const LatP& p, const LatTile& t, int row) { return row / p.per_cta < t.n_tok && row % p.per_cta < t.n_heads; }
__device__ __forceinline__ bf16* lat_out(const LatP& p, const LatTile& t, int row) {
    return (bf16*)p.out + ((long long)(t.sq.start + t.first + row / p.per_cta) * p.heads + t.h0 + row % p.per_cta) * p.rank;
}

// Grid: (splits of row tiles or sequences, head groups). The rank is padded to NT · 128.
template <int M, int NT, bool DECODE> __global__ void __launch_bounds__(LatShape<M, DECODE>::threads, LatShape<M, DECODE>::threads == 256 && NT <= 2 ? 2 : 1)
    latent_attend(const __grid_constant__ LatP p) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ float red[32];
    __shared__ __align__(8) unsigned long long full[kLatSlots];
    using L = LatShape<M, DECODE>;
    constexpr int KEYS = L::keys, TEAMS = L::teams, TT = L::team_threads, RP = NT * 128, NW = RP / 8 / L::warps;  // NW: groups of eight value dimensions of a warp
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, team = tid / TT, warp = (tid % TT) >> 5, tt = tid % TT, g8 = lane >> 2, t4 = lane & 3;
    const int rank = p.rank, dim = p.rank + p.rot, half = p.rot / 2, stride = lat_stride(dim), chunks = lat_dim(dim) / 8;
    if constexpr (!DECODE) pdl_wait();
    const int unit = (int)blockIdx.x / p.splits, split = (int)blockIdx.x - unit * p.splits;
    LatTile tile;  // no launch of a step writes the batch description
    if (!lat_tile<M, DECODE>(p, unit, (int)gridDim.x / p.splits, (int)blockIdx.y, &tile)) return;
    const SeqRow sq = tile.sq;
    const int pos0 = sq.past + tile.first, last = pos0 + tile.n_tok - 1, all = last / KEYS + 1;
    int kt0 = (int)((long long)all * split / p.splits), kt1 = (int)((long long)all * (split + 1) / p.splits);
    if (DECODE && sq.len != 1) kt0 = kt1 = 0;

    const int tile_bytes = lat_panels(dim) * L::panel, ring_bytes = p.ring;
    unsigned char *smem_q = ring + ring_bytes, *teams = smem_q + (size_t)M * stride, *mine = teams + team * L::team_bytes;
    const unsigned sm_q = smem_u32(smem_q), sm_kv = smem_u32(ring);
    float* scores = reinterpret_cast<float*>(mine);                                  // [halves][M][score_stride]
    unsigned char* weights = mine + L::halves * M * L::score_stride * 4;             // [M][weight_stride]
    float* row_scale = reinterpret_cast<float*>(weights + M * L::weight_stride);
    float *row_max = row_scale + M, *row_sum = row_max + M;
    float *cs = reinterpret_cast<float*>(teams + TEAMS * L::team_bytes), *sn = cs + half;
    bf16* pool = (bf16*)p.pool;
    bool ok = true;

    if (tid == 0) {
        for (int i = 0; i < TEAMS * p.slots; i++) mbar_init(smem_u32(full + i), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    // The team's i-th tile into its slot `in`, a panel per copy: its keys lie in one page; columns beyond the pool's come as zeros.
    auto load_tile = [&](int i, int in) {
        const int kt = kt0 + team + i * TEAMS;
        if (kt >= kt1 || tt != 0) return;
        const int slot = team * p.slots + in, j0 = kt * KEYS;
        const unsigned bar = smem_u32(full + slot), dst = sm_kv + (unsigned)(slot * tile_bytes);
        const int row = (int)key_row(p, page_of(p, tile.seq, j0), 0, j0);
        mbar_expect_tx(bar, (unsigned)tile_bytes);
        for (int k = 0; k < lat_panels(dim); k++) tma_load_2d(dst + k * L::panel, p.map, k * 64, row, bar);
    };
    auto team_sync = [&]() {
        if constexpr (TEAMS == 1) __syncthreads();
        else asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "n"(TT) : "memory");
    };
    auto team_any = [&](bool v) -> bool {
        if constexpr (TEAMS == 1) return __syncthreads_or(v);
        int r;
        asm volatile("{\n .reg .pred p, q;\n setp.ne.u32 p, %1, 0;\n bar.red.or.pred q, %2, %3, p;\n selp.u32 %0, 1, 0, q;\n}\n"
                     : "=r"(r)
                     : "r"((int)v), "r"(1 + team), "n"(TT)
                     : "memory");
        return r != 0;
    };
    if constexpr (DECODE) {
        // Tiles of earlier steps' keys may be loaded while the launches before this one finish; the one with the new key has to wait.
        const bool newest = kt1 == all && kt0 < kt1;
        const int late = newest && (all - 1 - kt0) % TEAMS == team ? (all - 1 - kt0) / TEAMS : -1;
        for (int i = 0; i < p.slots; i++)
            if (i != late) load_tile(i, i);
        angles(p.turns, half, pos0, cs, sn, tid, L::threads);
        pdl_wait();
        if (sq.len != 1) return;
        __syncthreads();
        const bf16 *lat = (const bf16*)p.q_latent + ((long long)sq.start * p.heads + tile.h0) * rank, *own = (const bf16*)p.q_own + (long long)sq.start * p.q_ld;
        for (int i = tid; i < M * chunks; i += L::threads) {
            const int r = i / chunks, c = i - r * chunks;
            bf16* to = reinterpret_cast<bf16*>(smem_q + r * stride + c * 16);
            if (r < tile.n_heads && c * 8 < rank) {
                *reinterpret_cast<uint4*>(to) = *reinterpret_cast<const uint4*>(lat + (long long)r * rank + c * 8);
            } else {
float v[8];  // (all loads before the store)
#pragma unroll
                for (int e = 0; e < 8; e++) {
                    const int d = c * 8 + e - rank;
                    v[e] = r < tile.n_heads && d < p.rot ? rotated(half, 0, own + (long long)(tile.h0 + r) * p.q_step, cs, sn, d) : 0.f;
                }
                *reinterpret_cast<uint4*>(to) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
            }
        }
        if (newest) {
            const bf16* x = (const bf16*)p.proj + (long long)sq.start * p.ld;
            bf16* dst = pool + key_row(p, page_of(p, tile.seq, pos0), 0, pos0) * dim;
            constexpr int PER = 512 / L::threads;  // the rank is at most 512
            float v[PER], w[PER], ss = 0.f;
#pragma unroll
            for (int j = 0; j < PER; j++) {
                const int i = j * L::threads + tid;
                v[j] = i < rank ? to_f(x[i]) : 0.f;
                w[j] = i < rank ? p.norm_w[i] : 0.f;
            }
            for (int i = tid; i < p.rot; i += L::threads) dst[rank + i] = __float2bfloat16_rn(rotated(half, 0, x + rank, cs, sn, i));
#pragma unroll
            for (int j = 0; j < PER; j++) ss = fmaf(v[j], v[j], ss);
            const float f = 1.f / sqrtf(block_sum(ss, red) / (float)rank + p.eps);
#pragma unroll
            for (int j = 0; j < PER; j++)
                if (j * L::threads + tid < rank) dst[j * L::threads + tid] = __float2bfloat16_rn(v[j] * f * w[j]);
            asm volatile("fence.proxy.async;" ::: "memory");  // the copy below reads what was just written
            __syncthreads();
            if (late >= 0 && late < p.slots) load_tile(late, late);
        }
    } else {
        for (int i = 0; i < p.slots; i++) load_tile(i, i);
        const bf16 *lat = (const bf16*)p.q_latent, *own = (const bf16*)p.q;
        for (int i = tid; i < M * chunks; i += L::threads) {
            const int r = i / chunks, c = i - r * chunks;
            const bool live = lat_wanted(p, tile, r) && c * 8 < dim;
            const long long at = (long long)(sq.start + tile.first + r / p.per_cta) * p.heads + tile.h0 + r % p.per_cta;
            cp_async16(sm_q + r * stride + c * 16, !live ? lat : c * 8 < rank ? lat + at * rank + c * 8 : own + at * p.rot + c * 8 - rank, live);
        }
        cp_async_commit();
        cp_async_wait<0>();
    }
    __syncthreads();

    float o[L::row_tiles][NW][4];
#pragma unroll
    for (int r = 0; r < L::row_tiles; r++)
#pragma unroll
        for (int n = 0; n < NW; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[r][n][e] = 0.f;
    const int s_row = tt / L::row_threads, s_key = (tt % L::row_threads) * L::row_keys;    // softmax: this thread's row and keys
    const int s_tok = s_row / p.per_cta, s_pos = s_tok < tile.n_tok ? pos0 + s_tok : last; // rows without a token compute something harmless
    float m = kNoScore, l = 0.f;
    // Where a lane's rows of ldmatrix lie in a tile, the swizzle applied: chunk c of key k is at chunk c ^ (k & 7) of its panel, and the chunks that a
    // lane visits differ in bits that its own offset does not have.
    const int l7 = lane & 7;
    const unsigned key_row0 = (unsigned)(warp / L::row_tiles % L::key_parts * (L::key_tiles * 8) + l7) * 128, key_chunk = (unsigned)((lane >> 3) ^ l7) << 4;
    const int c0 = warp * NW;
    constexpr bool simple = (NW & (NW - 1)) == 0;
    const unsigned value0 = (unsigned)(lane & 15) * 128 + (c0 >> 3) * L::panel, value_chunk = (unsigned)((c0 & 7) ^ (lane >> 4) ^ l7) << 4;
    int i = 0, at = 0, phase = 0;  // tiles done, slot, its phase
    for (int kt = kt0 + team; kt < kt1; kt += TEAMS, i++) {
        const int slot = team * p.slots + at;
        if (ok && !mbar_wait(smem_u32(full + slot), phase)) ok = false;
        __syncwarp();
        const unsigned ks = sm_kv + (unsigned)(slot * tile_bytes);
        if (const int live = last + 1 - kt * KEYS; live < KEYS) {  // what lies behind the newest key must be numbers
            for (int k = tt; k < (KEYS - live) * lat_panels(dim) * 8; k += TT) {
                const int key = live + k % (KEYS - live), c = k / (KEYS - live);
                *reinterpret_cast<uint4*>(ring + (lat_chunk<L::panel>(ks, key, c) - sm_kv)) = make_uint4(0, 0, 0, 0);
            }
            __syncwarp();
            team_sync();
        }
        {
            const int rt = warp % L::row_tiles, piece = warp / L::row_tiles, key0 = piece % L::key_parts * (L::key_tiles * 8), h = piece / L::key_parts;
            const int steps = chunks / 4, lo = steps * h / L::halves, hi = steps * (h + 1) / L::halves;
            float s[L::key_tiles][2][4];
#pragma unroll
            for (int n = 0; n < L::key_tiles; n++)
#pragma unroll
                for (int e = 0; e < 8; e++) s[n][e >> 2][e & 3] = 0.f;
            const unsigned qa = sm_q + (rt * 16 + (lane & 15)) * stride + (lane >> 4) * 16;
#pragma unroll 3
            for (int kk = lo; kk < hi; kk++) {
                unsigned a0[4], a1[4];
                ldmatrix_x4(a0, qa + kk * 64);
                ldmatrix_x4(a1, qa + kk * 64 + 32);
#pragma unroll
                for (int n = 0; n < L::key_tiles; n++) {
                    unsigned b[4];  // eight keys, 32 dimensions
                    ldmatrix_x4(b, ks + key_row0 + n * 1024 + (kk >> 1) * L::panel + (key_chunk ^ ((kk & 1) << 6)));
                    mma_bf16(s[n][0], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                    mma_bf16(s[n][1], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int n = 0; n < L::key_tiles; n++)
#pragma unroll
                for (int r = 0; r < 2; r++)
                    *reinterpret_cast<float2*>(scores + (h * M + rt * 16 + g8 + 8 * r) * L::score_stride + key0 + n * 8 + t4 * 2) =
                        make_float2(s[n][0][2 * r] + s[n][1][2 * r], s[n][0][2 * r + 1] + s[n][1][2 * r + 1]);
        }
        team_sync();
        if (TEAMS == 1 && i > 0 && ok) load_tile(i - 1 + p.slots, at == 0 ? p.slots - 1 : at - 1);  // its slot was read in the previous iteration
        __syncwarp();
        bool moved;
        {
            float v[L::row_keys], mx = m;
            const int j0 = kt * KEYS + s_key;
#pragma unroll
            for (int k = 0; k < L::row_keys; k += 2) {
                float2 x = *reinterpret_cast<const float2*>(scores + s_row * L::score_stride + s_key + k);
                if constexpr (L::halves == 2) {
                    const float2 y = *reinterpret_cast<const float2*>(scores + (M + s_row) * L::score_stride + s_key + k);
                    x = make_float2(x.x + y.x, x.y + y.y);
                }
                v[k] = j0 + k > s_pos ? -INFINITY : x.x * p.mul2;
                v[k + 1] = j0 + k + 1 > s_pos ? -INFINITY : x.y * p.mul2;
                mx = fmaxf(mx, fmaxf(v[k], v[k + 1]));
            }
#pragma unroll
            for (int d = 1; d < L::row_threads; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float keep = exp2f(m - mx);
            moved = mx != m;
            m = mx;
            l *= keep;
#pragma unroll
            for (int k = 0; k < L::row_keys; k += 2) {
                const float a = exp2f(v[k] - m), b = exp2f(v[k + 1] - m);
                l += a + b;
                *reinterpret_cast<unsigned*>(weights + s_row * L::weight_stride + (s_key + k) * 2) = pack_bf16(a, b);
            }
            if (tt % L::row_threads == 0) row_scale[s_row] = keep;
            __syncwarp();
        }
        if (team_any(moved)) {
#pragma unroll
            for (int r = 0; r < L::row_tiles; r++) {
                const float f0 = row_scale[r * 16 + g8], f1 = row_scale[r * 16 + g8 + 8];
#pragma unroll
                for (int n = 0; n < NW; n++) {
                    o[r][n][0] *= f0;
                    o[r][n][1] *= f0;
                    o[r][n][2] *= f1;
                    o[r][n][3] *= f1;
                }
            }
        }
        const unsigned wa = smem_u32(weights) + (lane & 15) * L::weight_stride + (lane >> 4) * 16;
#pragma unroll
        for (int kk = 0; kk < KEYS / 16; kk++) {
            unsigned a[L::row_tiles][4];
#pragma unroll
            for (int r = 0; r < L::row_tiles; r++) ldmatrix_x4(a[r], wa + r * 16 * L::weight_stride + kk * 32);
#pragma unroll
            for (int n = 0; n < NW; n += 2) {
                // dimensions beyond the tile are other bytes of this CTA's shared memory: a column that is never stored
                unsigned b[4];
                if constexpr (simple) ldmatrix_x4_trans(b, ks + value0 + kk * 2048 + (n >> 3) * L::panel + (value_chunk ^ ((n & 7) << 4)));
                else ldmatrix_x4_trans(b, lat_chunk<L::panel>(ks, kk * 16 + (lane & 15), c0 + n + (lane >> 4)));
#pragma unroll
                for (int r = 0; r < L::row_tiles; r++) {
                    mma_bf16(o[r][n], a[r][0], a[r][1], a[r][2], a[r][3], b[0], b[1]);
                    mma_bf16(o[r][n + 1], a[r][0], a[r][1], a[r][2], a[r][3], b[2], b[3]);
                }
            }
        }
        if constexpr (TEAMS > 1) {  // few slots per team: the next tile is asked for at once
            team_sync();
            if (ok) load_tile(i + p.slots, at);
            __syncwarp();
        }
        if (++at == p.slots) {
            at = 0;
            phase ^= 1;
        }
    }
    if (!ok) {
        report(p.err, ERR_WAIT_TIMEOUT, p.node, (long long)blockIdx.x, (long long)warp);
        for (int k = 0; k < TEAMS * p.slots; k++) mbar_wait(smem_u32(full + k), 0);  // copies in flight get a last chance to land
    }
    __syncwarp();
#pragma unroll
    for (int d = 1; d < L::row_threads; d <<= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
    if (tt % L::row_threads == 0) {
        row_max[s_row] = m;
        row_sum[s_row] = l;
    }
    __syncthreads();
    const long long part = ((long long)unit * gridDim.y + blockIdx.y) * p.splits + split;
    if constexpr (TEAMS == 1) {
#pragma unroll
        for (int r = 0; r < L::row_tiles; r++)
#pragma unroll
            for (int k = 0; k < 2; k++) {
                const int row = r * 16 + g8 + 8 * k;
                if (!lat_wanted(p, tile, row)) continue;
                const float f = p.splits == 1 ? 1.f / row_sum[row] : 1.f;
#pragma unroll
                for (int n = 0; n < NW; n++) {
                    const int d = warp * (NW * 8) + n * 8 + t4 * 2;
                    if (d >= rank) continue;
                    if (p.splits == 1) *reinterpret_cast<unsigned*>(lat_out(p, tile, row) + d) = pack_bf16(o[r][n][2 * k] * f, o[r][n][2 * k + 1] * f);
                    else *reinterpret_cast<float2*>(p.part + (part * M + row) * RP + d) = make_float2(o[r][n][2 * k], o[r][n][2 * k + 1]);
                }
            }
        if (p.splits > 1 && tid < M) *reinterpret_cast<float2*>(p.stats + (part * M + tid) * 2) = make_float2(row_max[tid], row_sum[tid]);
    } else {
        // the ring becomes the teams' results
        constexpr int OS = lat_out_stride(RP);
        float* results = reinterpret_cast<float*>(ring);
#pragma unroll
        for (int r = 0; r < L::row_tiles; r++)
#pragma unroll
            for (int k = 0; k < 2; k++)
#pragma unroll
                for (int n = 0; n < NW; n++)
                    *reinterpret_cast<float2*>(results + ((size_t)team * M + r * 16 + g8 + 8 * k) * OS + warp * (NW * 8) + n * 8 + t4 * 2) =
                        make_float2(o[r][n][2 * k], o[r][n][2 * k + 1]);
        __syncthreads();
        const int fours = rank / 4;
        for (int k = tid; k < tile.n_heads * fours; k += L::threads) {
            const int row = k / fours, d = (k - row * fours) * 4;
            float f[TEAMS], top = kNoScore, sum = 0.f;
            auto stat = [&](int t, int which) { return reinterpret_cast<const float*>(teams + t * L::team_bytes + L::team_bytes - M * 8)[which * M + row]; };
#pragma unroll
            for (int t = 0; t < TEAMS; t++) top = fmaxf(top, stat(t, 0));
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int t = 0; t < TEAMS; t++) {
                f[t] = exp2f(stat(t, 0) - top);
                sum = fmaf(stat(t, 1), f[t], sum);
                const float4 x = *reinterpret_cast<const float4*>(results + ((size_t)t * M + row) * OS + d);
                v = make_float4(fmaf(x.x, f[t], v.x), fmaf(x.y, f[t], v.y), fmaf(x.z, f[t], v.z), fmaf(x.w, f[t], v.w));
            }
            if (p.splits == 1) {
                const float g = 1.f / sum;
                *reinterpret_cast<uint2*>(lat_out(p, tile, row) + d) = make_uint2(pack_bf16(v.x * g, v.y * g), pack_bf16(v.z * g, v.w * g));
            } else {
                *reinterpret_cast<float4*>(p.part + (part * M + row) * RP + d) = v;
                if (d == 0) *reinterpret_cast<float2*>(p.stats + (part * M + row) * 2) = make_float2(top, sum);
            }
        }
    }
}

// Adds the splits of a row. Grid: (row tiles or sequences, head groups, rows); a thread takes four dimensions.
template <int M, bool DECODE> __global__ void __launch_bounds__(128) latent_merge(const LatP p) {
    __shared__ float factor[kLatSplits];
    pdl_enter();
    const int tid = threadIdx.x, row = blockIdx.z, RP = (p.rank + 127) / 128 * 128;
    LatTile tile;
    if (!lat_tile<M, DECODE>(p, (int)blockIdx.x, (int)gridDim.x, (int)blockIdx.y, &tile)) return;
    if ((DECODE && tile.sq.len != 1) || !lat_wanted(p, tile, row)) return;
    const long long part = ((long long)blockIdx.x * gridDim.y + blockIdx.y) * p.splits;
    if (tid < 32) {
        float2 v[kLatSplits / 32];
        float top = kNoScore, sum = 0.f;
#pragma unroll
        for (int k = 0; k < kLatSplits / 32; k++) {
            v[k] = k * 32 + tid < p.splits ? *reinterpret_cast<const float2*>(p.stats + ((part + k * 32 + tid) * M + row) * 2) : make_float2(kNoScore, 0.f);
            top = fmaxf(top, v[k].x);
        }
        top = warp_max(top);
#pragma unroll
        for (int k = 0; k < kLatSplits / 32; k++) sum = fmaf(v[k].y, exp2f(v[k].x - top), sum);
        sum = warp_sum(sum);
#pragma unroll
        for (int k = 0; k < kLatSplits / 32; k++) factor[k * 32 + tid] = exp2f(v[k].x - top) / sum;
    }
    __syncthreads();
    const int d = tid * 4;
    if (d >= p.rank) return;
    const float* from = p.part + (part * M + row) * RP + d;
    const long long step = (long long)M * RP;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < p.splits; k++) {
        const float4 v = *reinterpret_cast<const float4*>(from + k * step);
        const float f = factor[k];
        o = make_float4(fmaf(v.x, f, o.x), fmaf(v.y, f, o.y), fmaf(v.z, f, o.z), fmaf(v.w, f, o.w));
    }
    *reinterpret_cast<uint2*>(lat_out(p, tile, row) + d) = make_uint2(pack_bf16(o.x, o.y), pack_bf16(o.z, o.w));
}

using LatKernel = void (*)(const LatP);
template <int M, bool DECODE> LatKernel latent_kernel(int64_t rank) {
    return rank <= 128 ? latent_attend<M, 1, DECODE> : rank <= 256 ? latent_attend<M, 2, DECODE> : rank <= 384 ? latent_attend<M, 3, DECODE> : latent_attend<M, 4, DECODE>;
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
    Buf q_ready = none, part = none, stats = none;
    auto launch = [&](LatKernel k, dim3 grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, grid, dim3(block), smem, p,
                  {{&p.q_latent, q_latent.buf}, {&p.q_own, q.buf.at(d.q_off * element)}, {&p.proj, proj.buf.at(d.kv_off * element)}, {&p.norm_w, norm_w.buf},
                   {&p.turns, turns.buf}, {&p.pool, pool.buf}, {&p.q, q_ready}, {&p.seqs, seqs.buf}, {&p.table, pages.buf}, {&p.out, out.buf}, {&p.part, part},
                   {&p.stats, stats}, {&p.err, Buf{kSlotErr, 0}}},
                  label, /*pdl=*/true);
        return &em.recs.back();
    };
    const int64_t n_seqs = seqs.shape[0];
    // whole 16-byte chunks of latents and rotated parts
    const bool tc = bf && d.page % 32 == 0 && d.rank % 8 == 0 && d.rot % 8 == 0 && d.rank <= 512 && lat_smem<64, false>((int)dim, (int)d.rank, (int)d.rot, 2) <= 220 * 1024;
    const bool decode_only = tc && rows == n_seqs;  // every sequence has one new token
    p.singles = p.whole = !tc;
    const int64_t per_head = tc ? d.rot : dim;
    if (!decode_only) {
        q_ready = em.scratch((size_t)(rows * d.heads * per_head * element));
        launch(bf ? latent_prepare<bf16> : latent_prepare<float>, dim3((unsigned)rows), 128, (unsigned)(d.rot * 4), "latent_prepare");
    }
    if (!tc) {
        TRef ready;
        ready.dtype = proj.dtype;
        ready.shape = {rows, d.heads * dim};
        ready.buf = q_ready;
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
    auto attend = [&](auto rows_per_tile, auto decode, int64_t cells, int64_t groups) {
        constexpr int M = decltype(rows_per_tile)::value;
        constexpr bool DECODE = decltype(decode)::value;
        using L = LatShape<M, DECODE>;
        const int resident = L::threads == 256 && d.rank <= 256 ? 2 : 1, most = L::teams == 1 ? 6 : kLatSlots / L::teams;
        const int64_t limit = resident == 2 ? 110 * 1024 : 220 * 1024;
        const int idim = (int)dim, irank = (int)d.rank, irot = (int)d.rot;
        p.slots = L::teams == 1 ? 2 : 1;
        while (p.slots < most && lat_smem<M, DECODE>(idim, irank, irot, p.slots + 1) <= limit) p.slots++;
        const int64_t smem = lat_smem<M, DECODE>(idim, irank, irot, p.slots);
        p.ring = (int)smem - lat_smem<M, DECODE>(idim, irank, irot, 0) + (L::teams > 1 ? L::teams * M * lat_out_stride((irank + 127) / 128 * 128) * 4 : 0);
        // splits of the most keys a sequence can see: whole waves of resident CTAs, each with a fixed cost worth some keys
        const int64_t slots = (smem <= limit ? resident : 1) * sm_count(), seen = (int64_t)p.width * d.page;
        int64_t splits = 1;
        double best = 1e300;
        for (int64_t sp = 1; sp <= kLatSplits && sp * 2 * L::keys * L::teams <= std::max<int64_t>(seen, 2 * L::keys * L::teams); sp++) {
            if (sp > 1 && !DECODE && cells * groups * sp > 2 * slots) break;  // row tiles fill the device by themselves
            const double cost = (double)((cells * groups * sp + slots - 1) / slots) * ((double)seen / sp + 160.0) + (sp > 1 ? 100.0 + 2.0 * sp : 0.0);
            if (cost < best) {
                best = cost;
                splits = sp;
            }
        }
        p.splits = (int)splits;
        const int64_t padded = (d.rank + 127) / 128 * 128;
        part = splits > 1 ? em.scratch((size_t)(cells * groups * splits * M * padded) * 4) : none;
        stats = splits > 1 ? em.scratch((size_t)(cells * groups * splits * M) * 8) : none;
        const LatKernel k = latent_kernel<M, DECODE>(d.rank);
        ensure_max_dynamic_smem((const void*)k, 222 * 1024);
        LaunchRec* rec = launch(k, dim3((unsigned)(cells * splits), (unsigned)groups), L::threads, (unsigned)smem, DECODE ? "latent_decode" : "latent_prefill");
        rec->tmaps.push_back(TmapReloc{(uint32_t)offsetof(LatP, map), pool.buf, (uint64_t)dim, (uint64_t)(pool.shape[0] * d.page), (uint64_t)dim * 2, 64u, (uint32_t)L::keys});
        if (splits > 1)
            launch(latent_merge<M, DECODE>, dim3((unsigned)cells, (unsigned)groups, (unsigned)(DECODE ? p.per_cta : M)), 128, 0, "latent_merge");
    };
    if (!decode_only) {
        p.per_cta = (int)std::min<int64_t>(d.heads, 64);
        const int64_t tq = 64 / p.per_cta;
        attend(std::integral_constant<int, 64>{}, std::false_type{}, std::min<int64_t>(rows, rows / tq + n_seqs), (d.heads + p.per_cta - 1) / p.per_cta);
    }
    if (decode_only || n_seqs > 1) {
        const int M = d.heads <= 16 ? 16 : d.heads <= 32 ? 32 : 64;
        p.per_cta = (int)std::min<int64_t>(d.heads, M);
        const int64_t groups = (d.heads + M - 1) / M;
        if (M == 16) attend(std::integral_constant<int, 16>{}, std::true_type{}, n_seqs, groups);
        else if (M == 32) attend(std::integral_constant<int, 32>{}, std::true_type{}, n_seqs, groups);
        else attend(std::integral_constant<int, 64>{}, std::true_type{}, n_seqs, groups);
    }
}

}  // namespace oxk
