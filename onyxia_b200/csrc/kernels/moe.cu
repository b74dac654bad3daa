// Mixture of experts behind a residual norm: y = Σ over a token's chosen experts of weight · down(glu(gate h, up h)), plus the same
// of a shared expert (two ordinary products, whose result is the sums' first term).
//
// Router logits are an ordinary product (f32 result) unless moe_route forms them. What follows depends on the batch:
//   up to 32 rows (bf16)   moe_stream_up     the chosen experts' gate and up rows read once, straight into `mma.sync` A fragments;
//                          every CTA chooses the experts again from the logits (a few KB), CTA 0 leaves the choice for
//                          moe_stream_down   the down rows of all chosen experts as one long dot product per output row: a chunk's
//                                            partial sum is scaled by its token's expert weight in f32 as it is added
//   more rows, and f32     moe_top           choice, weights, and every token's place among its expert's tokens
//                          moe_route         the same with the logits, 16 tokens per CTA (bf16, routers of a moderate size)
//                          moe_sort          the rows in expert order
//                          grouped products  (linear.cu) one weight matrix per expert
//                          moe_combine       the weighted sum of a token's results
//
// Bytes: decode, chosen experts · 3 · ff · width · 2. FLOPs: 6 · tokens · top · ff · width.
#include <cooperative_groups.h>

#include "tc_util.cuh"

namespace oxk {

namespace cg = cooperative_groups;

namespace {

struct MoeP {
    const float* logits;   // [rows, experts]
    const void* router;    // [experts, width]
    const float* router_bias;
    const void* h;         // [rows, width]
    const void *up, *down;
    void* act;             // stream: [rows · top, ff]; sorted: unused
    void* sorted;          // [rows · top, width]
    const float* parts;    // [rows · top, width], sorted
    float* y;              // [rows, width]
    const float* base;     // [rows, width]: what is added to the experts' sum, or null
    int *ids, *rank, *counts;   // [rows, top], [rows, top], [experts]
    float* weights;        // [rows, top]
    long long rows, width, ff;
    int experts, top, up_tiles, down_tiles, max_active;
    int share, ctas;       // stream: warps per row tile of the first product, CTAs (a cluster) per row tile of the second
    unsigned per_expert_inv;  // 2^32 / (chunks of an expert's second product), rounded up
    float alpha, limit, shift;
    int scores, groups, keep, renorm, group_max;
    float route_scale;
    const float* correction;  // [experts], or null
    float* gates;             // [rows]: the shared expert's factor, or null
    int ld;                   // logits of a row: experts, and the shared expert's
};

// Shuts the experts of all groups but the best: scores of −inf. By one warp; lane l looks after groups l, l + 32, …
__device__ __forceinline__ void keep_groups(float* z, int n, int groups, int keep, int only_max) {
    constexpr int kMine = kMoeMaxGroups / 32;
    const int lane = threadIdx.x & 31, size = n / groups;
    float sum[kMine];
    int ahead[kMine];  // groups in front of mine
#pragma unroll
    for (int i = 0; i < kMine; i++) {
        const int g = i * 32 + lane;
        float a = -INFINITY, b = -INFINITY;
        if (g < groups)
            for (int e = g * size; e < (g + 1) * size; e++) {
                const float v = z[e];
                b = fmaxf(b, fminf(a, v));
                a = fmaxf(a, v);
            }
        sum[i] = size > 1 && !only_max ? a + b : a;
        ahead[i] = 0;
    }
#pragma unroll
    for (int i = 0; i < kMine; i++)
        for (int l = 0; l < 32 && i * 32 + l < groups; l++) {
            const float other = __shfl_sync(0xffffffffu, sum[i], l);
#pragma unroll
            for (int k = 0; k < kMine; k++) ahead[k] += other > sum[k] || (other == sum[k] && i * 32 + l < k * 32 + lane);
        }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < kMine; i++)
        if (i * 32 + lane < groups && ahead[i] >= keep)
            for (int e = (i * 32 + lane) * size; e < (i * 32 + lane + 1) * size; e++) z[e] = -INFINITY;
    __syncwarp();
}
// A token's choice from its router logits, by one warp; `z` is the warp's own copy in shared memory and is overwritten, `raw` another one
// that is not (MOE_CHOSEN does not look at it). Lane j < top ends up with the j-th choice and its weight.
__device__ __forceinline__ void choose(const MoeP& p, float* z, const float* raw, int* id, float* weight) {
    const int lane = threadIdx.x & 31, n = p.experts, top = p.top;
    float most = 0.f, inv = 1.f;  // softmax over all: of the largest logit, one over the sum
    if (p.scores == MOE_SOFTMAX) {
        most = -INFINITY;
        for (int i = lane; i < n; i += 32) most = fmaxf(most, z[i]);
        most = warp_max(most);
        float s = 0.f;
        for (int i = lane; i < n; i += 32) s += expf(z[i] - most);
        inv = 1.f / warp_sum(s);
    }
    auto score = [&](float logit) { return p.scores == MOE_SOFTMAX ? expf(logit - most) * inv : sigmoid_f(logit); };
    if (p.scores != MOE_CHOSEN) {
        for (int i = lane; i < n; i += 32) z[i] = score(z[i]) + (p.correction ? p.correction[i] : 0.f);
        __syncwarp();
        if (p.groups) keep_groups(z, n, p.groups, p.keep, p.group_max);
    }
    float mine = -INFINITY, first = 0.f;
    int chosen = 0;
    for (int j = 0; j < top; j++) {
        float best = -INFINITY;
        int at = INT32_MAX;
        for (int i = lane; i < n; i += 32)
            if (z[i] > best || at == INT32_MAX) {
                best = z[i];
                at = i;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float b = __shfl_xor_sync(0xffffffffu, best, o);
            const int a = __shfl_xor_sync(0xffffffffu, at, o);
            if (a != INT32_MAX && (at == INT32_MAX || b > best || (b == best && a < at))) {
                best = b;
                at = a;
            }
        }
        if (j == 0) first = best;
        if (lane == j) {
            mine = best;
            chosen = at;
        }
        if (lane == (at & 31)) z[at] = -INFINITY;
        __syncwarp();
    }
    *id = chosen;
    if (p.scores != MOE_CHOSEN) {
        const float s = lane < top ? score(raw[chosen]) : 0.f;
        *weight = (p.renorm ? s / (warp_sum(s) + 1e-20f) : s) * p.route_scale;
    } else {
        const float e = lane < top ? expf(mine - first) : 0.f;
        *weight = e / warp_sum(e);
    }
}

// ───────────────────────────── few rows ─────────────────────────────────
constexpr int kMoeWarps = 8, kMoeRows = 32;

__device__ __forceinline__ uint4 ld_weights(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// The experts that anybody chose, ascending, and who chose them.
struct Chosen {
    int* expert;           // [max_active]
    float* weight;         // [max_active][rows]; 0: not chosen by that token
    signed char* place;    // [max_active][rows]: the expert's place among the token's choices, or −1
    int n;
};

// Shared memory: expert, weight, place, then a map of all experts. `ids` / `wts` are the rows' choices in shared memory.
__device__ __forceinline__ Chosen list_chosen(const MoeP& p, unsigned char* smem, const int* ids, const float* wts, int* n_out) {
    const int rows = (int)p.rows, tid = threadIdx.x, cells = p.max_active * rows;
    Chosen c;
    c.expert = reinterpret_cast<int*>(smem);
    c.weight = reinterpret_cast<float*>(c.expert + p.max_active);
    int* index = reinterpret_cast<int*>(c.weight + cells);
    c.place = reinterpret_cast<signed char*>(index + p.experts);
    for (int i = tid; i < cells; i += kMoeWarps * 32) {
        c.weight[i] = 0.f;
        c.place[i] = -1;
    }
    for (int i = tid; i < p.experts; i += kMoeWarps * 32) index[i] = 0;
    __syncthreads();
    for (int i = tid; i < rows * p.top; i += kMoeWarps * 32) index[ids[i]] = 1;
    __syncthreads();
    if (tid < 32) {
        int n = 0;
        for (int e0 = 0; e0 < p.experts; e0 += 32) {
            const bool in = e0 + tid < p.experts && index[e0 + tid];
            const unsigned mask = __ballot_sync(0xffffffffu, in);
            const int at = n + __popc(mask & ((1u << tid) - 1));
            if (in) {
                index[e0 + tid] = at;
                c.expert[at] = e0 + tid;
            }
            n += __popc(mask);
        }
        if (tid == 0) *n_out = n;
    }
    __syncthreads();
    for (int i = tid; i < rows * p.top; i += kMoeWarps * 32) {
        const int at = index[ids[i]] * rows + i / p.top;
        c.weight[at] = wts[i];
        c.place[at] = (signed char)(i % p.top);
    }
    __syncthreads();
    c.n = *n_out;
    return c;
}
size_t stream_smem(const MoeP& p) {
    const size_t rows = (size_t)p.rows, cells = (size_t)p.max_active * rows;
    return rows * p.top * 8 + (size_t)p.max_active * 4 + cells * 4 + (size_t)p.experts * 4 + (cells + 15) / 16 * 16 + kMoeWarps * (size_t)p.experts * 4;
}

// NT groups of eight tokens. The first product deals its row tiles to groups of `share` warps, which split k; in the second
// one (DOWN) all warps of a cluster of `ctas` CTAs split the chunks of all experts.
template <int NT, bool DOWN> __global__ void __launch_bounds__(kMoeWarps * 32, 2) moe_stream(const MoeP p) {
    constexpr int kBatch = NT == 4 ? 2 : 4;  // 32-k chunks a warp has in flight
    constexpr int kCells = 16 * NT * 8;      // results of a row tile
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float red[kMoeWarps][16][NT * 8 + 1];
    __shared__ float sums[DOWN ? 2 * kCells : 1];
    __shared__ int n_active;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int rows = (int)p.rows, pairs = rows * p.top;
    int* ids = reinterpret_cast<int*>(smem);
    float* wts = reinterpret_cast<float*>(ids + pairs);
    pdl_enter();
    if constexpr (DOWN) {
        for (int i = tid; i < pairs; i += kMoeWarps * 32) {
            ids[i] = p.ids[i];
            wts[i] = p.weights[i];
        }
    } else {
        float* z = reinterpret_cast<float*>(smem + pairs * 8) + warp * p.experts;
        for (int r = warp; r < rows; r += kMoeWarps) {
            const float* raw = p.logits + (long long)r * p.ld;
            for (int i = lane; i < p.experts; i += 32) z[i] = raw[i];
            __syncwarp();
            int id;
            float w;
            choose(p, z, raw, &id, &w);
            if (p.gates && blockIdx.x == 0 && lane == 0) p.gates[r] = sigmoid_f(raw[p.experts]);
            if (lane < p.top) {
                ids[r * p.top + lane] = id;
                wts[r * p.top + lane] = w;
                if (blockIdx.x == 0) {
                    p.ids[r * p.top + lane] = id;
                    p.weights[r * p.top + lane] = w;
                }
            }
            __syncwarp();
        }
    }
    __syncthreads();
    const Chosen chosen = list_chosen(p, smem + pairs * 8, ids, wts, &n_active);

    const long long K = DOWN ? p.ff : p.width, out = DOWN ? p.width : 2 * p.ff;
    const int per_expert = (int)((K + 31) / 32);
    const int share = DOWN ? kMoeWarps : p.share, group = warp / share, sub = warp % share;
    const int parts = DOWN ? p.ctas : 1, part = (int)blockIdx.x % parts;
    const int all = DOWN ? per_expert * chosen.n : per_expert;
    const int lo = (int)((long long)all * part / parts), hi = (int)((long long)all * (part + 1) / parts);
    const int tiles = DOWN ? p.down_tiles : p.up_tiles * chosen.n, lanes = DOWN ? 1 : kMoeWarps / share;  // tiles at a time
    const int first = (int)blockIdx.x / parts * lanes + group, stride = (int)gridDim.x / parts * lanes;
    const int per_tile = max(1, (hi - lo + share * kBatch - 1) / (share * kBatch));
    const int my_tiles = first < tiles ? (tiles - 1 - first) / stride + 1 : 0, total = my_tiles * per_tile;
    // chunk j of batch `it` → index of its expert, first k of this lane, row tile
    auto where = [&](int it, int j, int& a, long long& k, int& tile) {
        const int unit = first + (it / per_tile) * stride, c = lo + ((it % per_tile) * kBatch + j) * share + sub;
        if constexpr (DOWN) {
            a = per_expert == 1 ? c : (int)__umulhi((unsigned)c, p.per_expert_inv);
            k = (long long)(c - a * per_expert) * 32 + t * 8;
            tile = unit;
        } else {
            a = unit / p.up_tiles;
            k = (long long)c * 32 + t * 8;
            tile = unit - a * p.up_tiles;
        }
        return it < total && c < hi && k < K;
    };
    auto meet = [&]() {  // the warps that share a tile
        if (DOWN) __syncthreads();
        else if (share == 1) __syncwarp();
        else asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "r"(share * 32) : "memory");
    };
    const bf16* W = (const bf16*)(DOWN ? p.down : p.up);
    uint4 wl[kBatch], wh[kBatch];
    auto fetch = [&](int it) {
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            int a, tile;
            long long k;
            wl[j] = wh[j] = make_uint4(0, 0, 0, 0);
            if (!where(it, j, a, k, tile)) continue;
            const long long r0 = (long long)tile * 16 + g, at = ((long long)chosen.expert[a] * out + r0) * K + k;
            if (r0 < out) wl[j] = ld_weights(W + at);
            if (r0 + 8 < out) wh[j] = ld_weights(W + at + 8 * K);
        }
    };
    fetch(0);
    float acc[NT][4];
    for (int it = 0; it < total; it++) {
        if (it % per_tile == 0) {
#pragma unroll
            for (int n = 0; n < NT; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[n][e] = 0.f;
        }
        uint4 a[kBatch], b[kBatch], xv[kBatch][NT];
        int expert[kBatch];
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            a[j] = wl[j];
            b[j] = wh[j];
            int tile;
            long long k;
            const bool live = where(it, j, expert[j], k, tile);
            // also for lanes whose own k lies beyond the chunk's end: their columns take part in the sum
            if (expert[j] >= chosen.n) expert[j] = 0;
#pragma unroll
            for (int n = 0; n < NT; n++) {
                const int row = n * 8 + g;
                xv[j][n] = make_uint4(0, 0, 0, 0);
                if (!live || row >= rows) continue;
                const int place = chosen.place[expert[j] * rows + row];
                if (place < 0) continue;
                const bf16* x = DOWN ? (const bf16*)p.act + ((long long)row * p.top + place) * K : (const bf16*)p.h + row * K;
                xv[j][n] = *reinterpret_cast<const uint4*>(x + k);
            }
        }
        fetch(it + 1);
#pragma unroll
        for (int j = 0; j < kBatch; j++)
#pragma unroll
            for (int n = 0; n < NT; n++) {
                if constexpr (DOWN) {
                    float sum[4] = {0.f, 0.f, 0.f, 0.f};
                    mma_bf16(sum, a[j].x, b[j].x, a[j].y, b[j].y, xv[j][n].x, xv[j][n].y);
                    mma_bf16(sum, a[j].z, b[j].z, a[j].w, b[j].w, xv[j][n].z, xv[j][n].w);
                    const int m = n * 8 + t * 2;
                    const float w0 = m < rows ? chosen.weight[expert[j] * rows + m] : 0.f, w1 = m + 1 < rows ? chosen.weight[expert[j] * rows + m + 1] : 0.f;
                    acc[n][0] = fmaf(sum[0], w0, acc[n][0]);
                    acc[n][1] = fmaf(sum[1], w1, acc[n][1]);
                    acc[n][2] = fmaf(sum[2], w0, acc[n][2]);
                    acc[n][3] = fmaf(sum[3], w1, acc[n][3]);
                } else {
                    mma_bf16(acc[n], a[j].x, b[j].x, a[j].y, b[j].y, xv[j][n].x, xv[j][n].y);
                    mma_bf16(acc[n], a[j].z, b[j].z, a[j].w, b[j].w, xv[j][n].z, xv[j][n].w);
                }
            }
        if (it % per_tile != per_tile - 1) continue;
#pragma unroll
        for (int n = 0; n < NT; n++) {
            red[warp][g][n * 8 + t * 2] = acc[n][0];
            red[warp][g][n * 8 + t * 2 + 1] = acc[n][1];
            red[warp][g + 8][n * 8 + t * 2] = acc[n][2];
            red[warp][g + 8][n * 8 + t * 2 + 1] = acc[n][3];
        }
        meet();
        auto total_of = [&](int r, int m) {
            float s = 0.f;
            for (int w = 0; w < share; w++) s += red[group * share + w][r][m];
            return s;
        };
        const int unit = first + (it / per_tile) * stride;
        if constexpr (DOWN) {
            auto put = [&](int i, float v) {
                const int m = i >> 4;
                const long long o = (long long)unit * 16 + (i & 15);
                if (m < rows && o < out) p.y[m * out + o] = p.base ? fmaf(p.base[m * out + o], p.gates ? p.gates[m] : 1.f, v) : v;
            };
            if (parts == 1) {
                for (int i = tid; i < kCells; i += kMoeWarps * 32) put(i, total_of(i & 15, i >> 4));
                __syncthreads();
            } else {
                // sums of this CTA; the cluster's CTAs finish a share of the cells each. The other half of `sums` is written
                // next, and this one only after the meeting that every reader of it has come to
                float* mine = sums + (it / per_tile & 1) * kCells;
                for (int i = tid; i < kCells; i += kMoeWarps * 32) mine[i] = total_of(i & 15, i >> 4);
                cg::cluster_group cluster = cg::this_cluster();
                cluster.sync();
                for (int i = part * kMoeWarps * 32 + tid; i < kCells; i += parts * kMoeWarps * 32) {
                    float s = 0.f;
                    for (int q = 0; q < parts; q++) s += cluster.map_shared_rank(mine, q)[i];
                    put(i, s);
                }
            }
        } else {
            const int e = unit / p.up_tiles;
            for (int i = sub * 32 + lane; i < 8 * NT * 8; i += share * 32) {
                const int r = i & 7, m = i >> 3;
                const long long o = (long long)(unit - e * p.up_tiles) * 8 + r;
                if (m >= rows || o >= p.ff) continue;
                const int place = chosen.place[e * rows + m];
                if (place < 0) continue;
                const float gate = fminf(total_of(2 * r, m), p.limit), u = fminf(fmaxf(total_of(2 * r + 1, m), -p.limit), p.limit);
                ((bf16*)p.act)[((long long)m * p.top + place) * p.ff + o] = __float2bfloat16_rn(gate * sigmoid_fast(p.alpha * gate) * (u + p.shift));
            }
            meet();
        }
    }
    if (DOWN && parts > 1) cg::this_cluster().sync();  // nobody reads this CTA's sums any more
}

// ───────────────────────────── many rows ────────────────────────────────
// One warp per token. `counts` was cleared by an earlier launch; the places that a CTA's tokens take among an expert's
// are handed out by one addition per CTA and expert (their order changes nothing but where a row lies).
constexpr int kTopWarps = 16;
__global__ void __launch_bounds__(kTopWarps * 32) moe_top(const MoeP p) {
    extern __shared__ __align__(16) unsigned char smem[];  // count[experts], base[experts], z[warps][experts]
    pdl_enter();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    int *count = reinterpret_cast<int*>(smem), *base = count + p.experts;
    float* z = reinterpret_cast<float*>(base + p.experts) + warp * p.experts;
    const long long row = (long long)blockIdx.x * kTopWarps + warp;
    for (int i = tid; i < p.experts; i += kTopWarps * 32) count[i] = 0;
    int id = 0, place = 0;
    float w = 0.f;
    __syncthreads();
    const bool live = row < p.rows;
    if (live) {
        const float* raw = p.logits + row * p.ld;
        for (int i = lane; i < p.experts; i += 32) z[i] = raw[i];
        __syncwarp();
        choose(p, z, raw, &id, &w);
        if (p.gates && lane == 0) p.gates[row] = sigmoid_f(raw[p.experts]);
        if (lane < p.top) place = atomicAdd(count + id, 1);
    }
    __syncthreads();
    for (int i = tid; i < p.experts; i += kTopWarps * 32)
        if (count[i]) base[i] = atomicAdd(p.counts + i, count[i]);
    __syncthreads();
    if (live && lane < p.top) {
        p.ids[row * p.top + lane] = id;
        p.weights[row * p.top + lane] = w;
        p.rank[row * p.top + lane] = base[id] + place;
    }
}

constexpr int kRouteRows = 16;
__global__ void __launch_bounds__(kMoeWarps * 32, 2) moe_route(const MoeP p) {
    constexpr int kBatch = 4;
    extern __shared__ __align__(16) unsigned char smem[];  // count[experts], base[experts], z[rows][ld] [, the same once more]
    __shared__ float red[kMoeWarps][16][kRouteRows + 1];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3, E = p.experts, L = p.ld;
    int *count = reinterpret_cast<int*>(smem), *base = count + E;
    float* z = reinterpret_cast<float*>(base + E);
    const long long row0 = (long long)blockIdx.x * kRouteRows, K = p.width;
    const int chunks = (int)((K + 31) / 32), per_tile = (chunks + kMoeWarps * kBatch - 1) / (kMoeWarps * kBatch), total = (L + 15) / 16 * per_tile;
    const bf16* W = (const bf16*)p.router;
    auto k_of = [&](int it, int j) { return (long long)(((it % per_tile) * kBatch + j) * kMoeWarps + warp) * 32 + t * 8; };
    uint4 wl[kBatch], wh[kBatch];
    auto fetch = [&](int it) {
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            const long long k = k_of(it, j), at = (long long)(it / per_tile * 16 + g) * K + k;
            const bool live = it < total && k < K;
            wl[j] = wh[j] = make_uint4(0, 0, 0, 0);
            if (live && it / per_tile * 16 + g < L) wl[j] = *reinterpret_cast<const uint4*>(W + at);
            if (live && it / per_tile * 16 + g + 8 < L) wh[j] = *reinterpret_cast<const uint4*>(W + at + 8 * K);
        }
    };
    fetch(0);  // constants: may overlap the launches before this one
    for (int i = tid; i < E; i += kMoeWarps * 32) count[i] = 0;
    pdl_wait();
    float acc[2][4];
    for (int it = 0; it < total; it++) {
        if (it % per_tile == 0) {
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[n][e] = 0.f;
        }
        uint4 a[kBatch], b[kBatch], xv[kBatch][2];
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            a[j] = wl[j];
            b[j] = wh[j];
            const long long k = k_of(it, j);
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const long long row = row0 + n * 8 + g;
                xv[j][n] = k < K && row < p.rows ? *reinterpret_cast<const uint4*>((const bf16*)p.h + row * K + k) : make_uint4(0, 0, 0, 0);
            }
        }
        fetch(it + 1);
#pragma unroll
        for (int j = 0; j < kBatch; j++)
#pragma unroll
            for (int n = 0; n < 2; n++) {
                mma_bf16(acc[n], a[j].x, b[j].x, a[j].y, b[j].y, xv[j][n].x, xv[j][n].y);
                mma_bf16(acc[n], a[j].z, b[j].z, a[j].w, b[j].w, xv[j][n].z, xv[j][n].w);
            }
        if (it % per_tile != per_tile - 1) continue;
#pragma unroll
        for (int n = 0; n < 2; n++) {
            red[warp][g][n * 8 + t * 2] = acc[n][0];
            red[warp][g][n * 8 + t * 2 + 1] = acc[n][1];
            red[warp][g + 8][n * 8 + t * 2] = acc[n][2];
            red[warp][g + 8][n * 8 + t * 2 + 1] = acc[n][3];
        }
        __syncthreads();
        const int o = it / per_tile * 16 + (tid & 15), m = tid >> 4;
        if (o < L) {
            float s = 0.f;
#pragma unroll
            for (int w = 0; w < kMoeWarps; w++) s += red[w][tid & 15][m];
            z[m * L + o] = s + p.router_bias[o];
            if (p.scores != MOE_CHOSEN) z[(kRouteRows + m) * L + o] = s + p.router_bias[o];
        }
        __syncthreads();
    }
    int id[2], place[2];
    float w[2];
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const float* raw = z + (kRouteRows + warp + h * kMoeWarps) * L;
        choose(p, z + (warp + h * kMoeWarps) * L, raw, id + h, w + h);
        if (p.gates && lane == 0 && row0 + warp + h * kMoeWarps < p.rows) p.gates[row0 + warp + h * kMoeWarps] = sigmoid_f(raw[E]);
        place[h] = row0 + warp + h * kMoeWarps < p.rows && lane < p.top ? atomicAdd(count + id[h], 1) : 0;
    }
    __syncthreads();
    for (int i = tid; i < E; i += kMoeWarps * 32)
        if (count[i]) base[i] = atomicAdd(p.counts + i, count[i]);
    __syncthreads();
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const long long row = row0 + warp + h * kMoeWarps;
        if (row >= p.rows || lane >= p.top) continue;
        p.ids[row * p.top + lane] = id[h];
        p.weights[row * p.top + lane] = w[h];
        p.rank[row * p.top + lane] = base[id[h]] + place[h];
    }
}

// One CTA per token: its row goes to every chosen expert's part of the sorted rows; `rank` becomes the row there.
constexpr int kSortThreads = 128;
template <int BYTES> struct Unit;
template <> struct Unit<16> { using T = uint4; };
template <> struct Unit<2> { using T = unsigned short; };
template <> struct Unit<4> { using T = unsigned; };
template <int BYTES> __global__ void __launch_bounds__(kSortThreads) moe_sort(const MoeP p) {
    using T = typename Unit<BYTES>::T;
    __shared__ int at[32];
    pdl_enter();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const long long row = blockIdx.x;
    for (int j = warp; j < p.top; j += kSortThreads / 32) {
        const int e = p.ids[row * p.top + j];
        int before = 0;
        for (int i = lane; i < e; i += 32) before += p.counts[i];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
        if (lane == 0) {
            at[j] = before + p.rank[row * p.top + j];
            p.rank[row * p.top + j] = at[j];
        }
    }
    __syncthreads();
    const long long n = p.width;  // in units
    const T* src = (const T*)p.h + row * n;
    for (long long i = tid; i < n; i += kSortThreads) {
        const T v = src[i];
        for (int j = 0; j < p.top; j++) ((T*)p.sorted)[at[j] * n + i] = v;
    }
}

// One CTA per token; V consecutive elements per thread.
template <int V> __global__ void __launch_bounds__(256) moe_combine(const MoeP p) {
    pdl_enter();
    const long long row = blockIdx.x;
    __shared__ long long at[32];
    __shared__ float w[32];
    const float gate = p.gates ? p.gates[row] : 1.f;
    if (threadIdx.x < p.top) {
        at[threadIdx.x] = p.rank[row * p.top + threadIdx.x] * p.width;
        w[threadIdx.x] = p.weights[row * p.top + threadIdx.x];
    }
    __syncthreads();
    for (long long i = threadIdx.x * V; i < p.width; i += 256 * V) {
        float s[V];
#pragma unroll
        for (int e = 0; e < V; e++) s[e] = p.base ? p.base[row * p.width + i + e] * gate : 0.f;
#pragma unroll 4
        for (int j = 0; j < p.top; j++) {
            float v[V];
            if constexpr (V == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p.parts + at[j] + i);
            else v[0] = p.parts[at[j] + i];
#pragma unroll
            for (int e = 0; e < V; e++) s[e] = fmaf(w[j], v[e], s[e]);
        }
        if constexpr (V == 4) *reinterpret_cast<float4*>(p.y + row * p.width + i) = *reinterpret_cast<float4*>(s);
        else p.y[row * p.width + i] = s[0];
    }
}

}  // namespace

void emit_moe(Emitter& em, const MoeDesc& d, const ResidualNormDesc& norm, const TRef& router, const TRef& router_bias, const TRef& up_w, const TRef& down,
              const TRef* shared_up, const TRef* shared_down, const TRef& y) {
    if (d.rows == 0) return;
    const bool bf = up_w.dtype == DT_BF16;
    const int64_t element = bf ? 2 : 4, pairs = d.rows * d.top;
    MoeP p{};
    p.rows = d.rows;
    p.width = d.width;
    p.ff = d.ff;
    p.experts = (int)d.experts;
    p.top = (int)d.top;
    p.up_tiles = (int)((2 * d.ff + 15) / 16);
    p.down_tiles = (int)((d.width + 15) / 16);
    p.max_active = (int)std::min(d.experts, pairs);
    const uint64_t per_expert = (uint64_t)((d.ff + 31) / 32);
    p.per_expert_inv = (unsigned)(((1ull << 32) + per_expert - 1) / per_expert);  // (of no use, and 0, for 1)
    p.alpha = d.alpha;
    p.limit = d.limit;
    p.shift = d.shift;
    p.scores = d.scores;
    p.renorm = d.renorm;
    p.group_max = d.group_max;
    p.ld = (int)d.experts + d.shared_gate;
    p.groups = (int)d.groups;
    p.keep = (int)d.keep;
    p.route_scale = d.route_scale;
    auto tensor = [&](int dtype, std::vector<int64_t> shape, size_t bytes) {
        TRef t;
        t.dtype = dtype;
        t.shape = std::move(shape);
        t.buf = em.scratch(bytes);
        return t;
    };
    const TRef h = tensor(up_w.dtype, {d.rows, d.width}, (size_t)(d.rows * d.width * element));
    const TRef logits = tensor(DT_F32, {d.rows, p.ld}, (size_t)(d.rows * p.ld) * 4);
    const Buf none{kSlotNull, 0}, correction = d.correction ? d.correction->buf : none, gates = d.shared_gate ? em.scratch((size_t)d.rows * 4) : none;
    const Buf ids = em.scratch((size_t)pairs * 4), weights = em.scratch((size_t)pairs * 4);
    LinearDesc rd;
    rd.rows = d.rows;
    rd.out = p.ld;
    rd.k[0] = d.width;
    rd.k[1] = 0;
    // the shared expert, once the rows lie in `h`
    const TRef base = d.shared_ff ? tensor(DT_F32, {d.rows, d.width}, (size_t)(d.rows * d.width) * 4) : TRef{};
    const Buf base_buf = d.shared_ff ? base.buf : Buf{kSlotNull, 0};
    auto shared = [&] {
        if (!d.shared_ff) return;
        const TRef act = tensor(up_w.dtype, {d.rows, d.shared_ff}, (size_t)(d.rows * d.shared_ff * element));
        LinearDesc sd;
        sd.rows = d.rows;
        sd.out = 2 * d.shared_ff;
        sd.k[0] = d.width;
        sd.k[1] = 0;
        sd.glu = true;
        sd.alpha = d.alpha;
        sd.limit = d.shared_limit;
        sd.shift = d.shift;
        emit_linear(em, sd, &h, nullptr, *shared_up, nullptr, nullptr, act, nullptr);
        sd = LinearDesc{};
        sd.rows = d.rows;
        sd.out = d.width;
        sd.k[0] = d.shared_ff;
        sd.k[1] = 0;
        emit_linear(em, sd, &act, nullptr, *shared_down, nullptr, nullptr, base, nullptr);
    };
    const bool stream = bf && d.rows <= kMoeRows && d.width % 8 == 0 && d.ff % 8 == 0 && stream_smem(p) <= 90 * 1024;
    if (stream) {
        emit_linear(em, rd, nullptr, nullptr, router, nullptr, &router_bias, logits, &norm, &h);
        shared();
        const Buf act = em.scratch((size_t)(pairs * d.ff) * 2);
        const unsigned smem = (unsigned)stream_smem(p);
        const int nt = d.rows <= 8 ? 1 : d.rows <= 16 ? 2 : 4, batch = nt == 4 ? 2 : 4;
        // Batches of loads that follow one another: waves of row tiles times batches per tile. Experts in use: as many as
        // random choices reach.
        const double met = std::max((double)d.top, (double)d.experts * (1.0 - std::pow(1.0 - (double)d.top / (double)d.experts, (double)d.rows)));
        const int64_t slots = 2 * sm_count();
        auto up = [](int64_t a, int64_t b) { return (a + b - 1) / b; };
        double best = 1e300;
        for (int share : {1, 2, 4, 8}) {
            const double rounds = std::ceil(met * p.up_tiles * share / (double)(slots * kMoeWarps)) * ((double)up(up(d.width, 32), share * batch) + (share > 1 ? 0.5 : 0.0));
            if (rounds < best) {
                best = rounds;
                p.share = share;
            }
        }
        best = 1e300;
        for (int parts : {1, 2, 4, 8}) {
            const double rounds = (double)up(p.down_tiles * parts, slots) *
                                  (std::ceil(met * (double)up(d.ff, 32) / (parts * kMoeWarps * batch)) + (parts > 1 ? 1.0 : 0.5));
            if (rounds < best) {
                best = rounds;
                p.ctas = parts;
            }
        }
        auto launch = [&](void (*k)(const MoeP), int64_t ctas, int cluster, const char* label) {
            ensure_max_dynamic_smem((const void*)k, 90 * 1024);
            LaunchRec& rec = em.launch(k, dim3((unsigned)ctas), dim3(kMoeWarps * 32), smem, p,
                                       {{&p.logits, logits.buf}, {&p.h, h.buf}, {&p.up, up_w.buf}, {&p.down, down.buf}, {&p.act, act}, {&p.y, y.buf}, {&p.base, base_buf}, {&p.ids, ids},
                                        {&p.weights, weights}, {&p.correction, correction}, {&p.gates, gates}},
                                       label, /*pdl=*/true);
            if (cluster > 1) rec.cluster = dim3((unsigned)cluster, 1, 1);
        };
        launch(nt == 1 ? moe_stream<1, false> : nt == 2 ? moe_stream<2, false> : moe_stream<4, false>,
               std::min(up((int64_t)p.max_active * p.up_tiles * p.share, kMoeWarps), slots), 1, "moe_stream_up");
        launch(nt == 1 ? moe_stream<1, true> : nt == 2 ? moe_stream<2, true> : moe_stream<4, true>,
               std::min<int64_t>(p.down_tiles, slots / p.ctas) * p.ctas, p.ctas, "moe_stream_down");
        return;
    }
    TRef counts = tensor(DT_I32, {d.experts}, (size_t)d.experts * 4);
    emit_residual_norm(em, norm, &h, counts.buf, (int)d.experts);
    shared();
    // one launch forms the logits and chooses where the router is small enough to be read by every 16 tokens
    const unsigned route_smem = (unsigned)((2 * d.experts + (d.scores == MOE_CHOSEN ? 1 : 2) * kRouteRows * p.ld) * 4);
    const bool route = bf && d.width % 8 == 0 && p.ld * d.width <= (1 << 19) && route_smem <= 64 * 1024;
    if (!route) emit_linear(em, rd, &h, nullptr, router, nullptr, &router_bias, logits, nullptr);
    const Buf rank = em.scratch((size_t)pairs * 4);
    const TRef sorted = tensor(up_w.dtype, {pairs, d.width}, (size_t)(pairs * d.width * element));
    const TRef act = tensor(up_w.dtype, {pairs, d.ff}, (size_t)(pairs * d.ff * element));
    const TRef parts = tensor(DT_F32, {pairs, d.width}, (size_t)(pairs * d.width) * 4);
    auto launch = [&](void (*k)(const MoeP), unsigned grid, unsigned block, unsigned smem, const char* label) {
        em.launch(k, dim3(grid), dim3(block), smem, p,
                  {{&p.logits, logits.buf}, {&p.router, router.buf}, {&p.router_bias, router_bias.buf}, {&p.h, h.buf}, {&p.sorted, sorted.buf}, {&p.parts, parts.buf}, {&p.y, y.buf}, {&p.base, base_buf}, {&p.ids, ids}, {&p.rank, rank},
                   {&p.counts, counts.buf}, {&p.weights, weights}, {&p.correction, correction}, {&p.gates, gates}},
                  label, /*pdl=*/true);
    };
    if (route) {
        ensure_max_dynamic_smem((const void*)moe_route, 64 * 1024);
        launch(moe_route, (unsigned)((d.rows + kRouteRows - 1) / kRouteRows), kMoeWarps * 32, route_smem, "moe_route");
    } else {
        const unsigned top_smem = (unsigned)((2 + kTopWarps) * d.experts * 4);
        ensure_max_dynamic_smem((const void*)moe_top, 200 * 1024);
        launch(moe_top, (unsigned)((d.rows + kTopWarps - 1) / kTopWarps), kTopWarps * 32, top_smem, "moe_top");
    }
    const int64_t row_bytes = d.width * element;
    const int unit = row_bytes % 16 == 0 ? 16 : (int)element;
    p.width = row_bytes / unit;
    launch(unit == 16 ? moe_sort<16> : unit == 4 ? moe_sort<4> : moe_sort<2>, (unsigned)d.rows, kSortThreads, 0, "moe_sort");
    p.width = d.width;
    GroupedLinearDesc gd;
    gd.rows = pairs;
    gd.groups = d.experts;
    gd.out = 2 * d.ff;
    gd.k = d.width;
    gd.glu = true;
    gd.alpha = d.alpha;
    gd.limit = d.limit;
    gd.shift = d.shift;
    emit_grouped_linear(em, gd, sorted, up_w, counts, act);
    gd = GroupedLinearDesc{};
    gd.rows = pairs;
    gd.groups = d.experts;
    gd.out = d.width;
    gd.k = d.ff;
    emit_grouped_linear(em, gd, act, down, counts, parts);
    const bool wide = d.width % 4 == 0;
    launch(wide ? moe_combine<4> : moe_combine<1>, (unsigned)d.rows, 256, 0, "moe_combine");
}

}  // namespace oxk
