// Dense products over unquantised weights, y = x · Wᵀ, and the residual norm in front of them.
//
//   linear_stream   up to 32 rows (decode): a warp reads 16 weight rows × 32 k straight into `mma.sync` A fragments (a dot
//                   product does not care in which order its k are visited, so a lane takes 16 consecutive bytes of
//                   a row), eight warps share a row tile's k. Weight loads run one batch ahead and start before the
//                   grid dependency resolves. For up to eight rows the residual norm that makes x runs as the
//                   prologue, in every CTA.
//   linear_tc       more rows: tcgen05 GEMM. Weights are the MMA's A operand (128 rows), activations its B operand
//                   (32–256 rows), both loaded by TMA into 128-byte-swizzled stages; accumulator in tensor memory.
//                   Grids that would leave SMs idle are cut along k; `linear_reduce` adds the pieces in order.
//   linear_simt     f32 (true 32-bit), and bf16 shapes whose rows are not 16-byte aligned.
//
// linear_tc and linear_simt also run grouped: activation rows sorted by group, one weight matrix per group, the groups'
// row counts known on the device only. A CTA finds its group from the counts; the grid covers the most tiles
// that any counts can give.
//
// Bytes per launch: out · k · 2 once per 256 activation rows; FLOPs 2 · rows · out · k.
#include <cstdio>
#include <cstdlib>

#include "tc_util.cuh"

namespace oxk {

namespace {

struct LinP {
    alignas(64) unsigned char maps[4][128];  // x0, w0, x1, w1 (linear_tc)
    const void* x[2];
    const void* w[2];
    const float* bias;
    void* y;
    float* partial;
    ErrWord* err;
    // residual norm (linear_stream prologue)
    const void* ny;
    const float *nw, *ngain, *nres;
    const bf16* ngate;
    const float *npost, *noffset;
    const void* nadd;
    float* stream;
    bf16* low;
    long long gate_ld, ny_ld;
    float eps, y_scale, add_scale;
    int ny_bf16, pre, add_bf16, streams, norm_groups;
    const float *connect, *npost2;
    const void* ny2;
    long long rows, out, k[2];
    // block-diagonal products: x rows are ldx apart, block b reads its columns from x_off + b · x_step on; y rows are ldy apart
    const void* mul;
    long long ldx, x_off, x_step, ldy, mul_ld;
    int blocks;
    int y_bf16, fast, glu;  // fast: the operands are bf16
    float alpha, limit, shift;
    int act[2];           // functions of the columns before and from act_split on; none from act_end on
    long long act_split, act_end;
    int nb, stages, splits, node;  // linear_tc
    const int* counts;    // grouped: rows of every group
    int groups;
};

// Grouped: the `tile`-th tile of `size` rows, counted group by group → its group, first row and rows. Called by whole warps.
__device__ __forceinline__ bool locate_group(const LinP& p, int tile, int size, int* group, int* row, int* live) {
    const int lane = threadIdx.x & 31;
    int tiles = 0, rows = 0;
    for (int g0 = 0; g0 < p.groups; g0 += 32) {
        const int n = g0 + lane < p.groups ? p.counts[g0 + lane] : 0, mine = (n + size - 1) / size;
        int t_inc = mine, r_inc = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int t = __shfl_up_sync(0xffffffffu, t_inc, o), r = __shfl_up_sync(0xffffffffu, r_inc, o);
            if (lane >= o) {
                t_inc += t;
                r_inc += r;
            }
        }
        const unsigned hit = __ballot_sync(0xffffffffu, tiles + t_inc > tile);
        if (hit) {
            const int at = __ffs(hit) - 1;
            const int count = __shfl_sync(0xffffffffu, n, at);
            const int first = (tile - tiles - (__shfl_sync(0xffffffffu, t_inc, at) - __shfl_sync(0xffffffffu, mine, at))) * size;
            *group = g0 + at;
            *row = rows + __shfl_sync(0xffffffffu, r_inc, at) - count + first;
            *live = min(size, count - first);
            return true;
        }
        tiles += __shfl_sync(0xffffffffu, t_inc, 31);
        rows += __shfl_sync(0xffffffffu, r_inc, 31);
    }
    return false;
}

__device__ __forceinline__ float glu_value(const LinP& p, float gate, float up) {
    const float g = fminf(gate, p.limit), u = fminf(fmaxf(up, -p.limit), p.limit);
    return g * (p.y_bf16 ? sigmoid_fast(p.alpha * g) : sigmoid_f(p.alpha * g)) * (u + p.shift);
}
// act: per column range
__device__ __forceinline__ float activate(const LinP& p, long long col, float v) {
    const int f = col < p.act_end ? p.act[col >= p.act_split] : ACT_NONE;
    if (f == ACT_NONE) return v;
    if (f == ACT_SOFTPLUS) return p.fast ? softplus_fast(v) : softplus_f(v);
    const float s = p.y_bf16 ? sigmoid_fast(v) : sigmoid_f(v);
    return f == ACT_SILU ? v * s : s;
}
// The factor of a block-diagonal product's result; the matrix has the weights' type.
template <typename T> __device__ __forceinline__ float factor(const LinP& p, long long row, long long col) {
    return p.mul ? to_f(((const T*)p.mul)[row * p.mul_ld + col]) : 1.f;
}
__device__ __forceinline__ void put(const LinP& p, long long row, long long width, long long col, float v) {
    if (p.y_bf16) ((bf16*)p.y)[row * width + col] = __float2bfloat16_rn(v);
    else ((float*)p.y)[row * width + col] = v;
}

// ───────────────────────────── decode ───────────────────────────────────
constexpr int kStreamWarps = 8, kThreads = kStreamWarps * 32;

__device__ __forceinline__ uint4 ld_weights(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

template <bool YB> __device__ __forceinline__ float4 ld_y4(const void* y, long long i) {
    if constexpr (YB) {
        const uint2 v = *reinterpret_cast<const uint2*>((const bf16*)y + i);
        return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
    } else {
        return *reinterpret_cast<const float4*>((const float*)y + i);
    }
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
// Rows 0 … rows−1 of the residual norm into shared memory (bf16, `stride` elements per row); CTA 0 stores the residual
// and the low-precision copy. Eight warps; `per` of them work on one row. K is a multiple of 8.
template <bool YB> __device__ void norm_prologue(const LinP& p, bf16* xs, int stride, float* red) {
    const int rows = (int)p.rows, K = (int)p.k[0], warp = threadIdx.x >> 5;
    const int per = rows <= 1 ? 8 : rows <= 2 ? 4 : rows <= 4 ? 2 : 1;
    const int row = warp / per, t = ((warp % per) * 32 + (threadIdx.x & 31)) * 4, step = per * 128;
    const long long base = (long long)row * K, y0 = (long long)row * p.ny_ld;
    auto rstd_of = [&](float ss) {  // of this row, from every thread's share of the squares
        ss = warp_sum(ss);
        if ((threadIdx.x & 31) == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
        if (row < rows)
            for (int i = 0; i < per; i++) tot += red[row * per + i];
        return 1.f / sqrtf(tot / (float)K + p.eps);
    };
    float inner = p.y_scale;  // with `post`: one over the root mean square of y
    if (p.npost) {
        float ss = 0.f;
        if (row < rows) {
#pragma unroll 8
            for (int i = t; i < K; i += step) {
                const float4 v = ld_y4<YB>(p.ny, y0 + i);
                ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
            }
        }
        inner = rstd_of(ss);
        __syncthreads();  // red is written again
    }
    auto normed = [&](int i) {  // what the mean square is taken of
        float4 v = ld_y4<YB>(p.ny, y0 + i);
        if (p.pre) {
            v = make_float4(v.x * inner, v.y * inner, v.z * inner, v.w * inner);
            if (p.npost) v = mul4(v, *reinterpret_cast<const float4*>(p.npost + i));
            if (p.nres) v = add4(v, *reinterpret_cast<const float4*>(p.nres + base + i));
            if (p.nadd) {
                const float4 r = p.add_bf16 ? ld_y4<true>(p.nadd, base + i) : ld_y4<false>(p.nadd, base + i);
                v = make_float4(fmaf(r.x, p.add_scale, v.x), fmaf(r.y, p.add_scale, v.y), fmaf(r.z, p.add_scale, v.z), fmaf(r.w, p.add_scale, v.w));
            }
            if (p.noffset) v = add4(v, *reinterpret_cast<const float4*>(p.noffset + i));
        }
        return v;
    };
    float ss = 0.f;
    if (row < rows) {
#pragma unroll 8
        for (int i = t; i < K; i += step) {
            const float4 v = normed(i);
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    }
    const float rstd = rstd_of(ss);
    if (row < rows) {
#pragma unroll 4
        for (int i = t; i < K; i += step) {
            const float4 sum = normed(i), w = *reinterpret_cast<const float4*>(p.nw + i);
            float4 v = mul4(make_float4(sum.x * rstd, sum.y * rstd, sum.z * rstd, sum.w * rstd), w);
            if (p.ngain) v = mul4(v, *reinterpret_cast<const float4*>(p.ngain + i));
            if (p.ngate) v = mul4(v, ld_y4<true>(p.ngate, row * p.gate_ld + i));
            if (!p.pre && p.nres) v = add4(v, *reinterpret_cast<const float4*>(p.nres + base + i));
            const uint2 packed = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
            *reinterpret_cast<uint2*>(xs + (long long)row * stride + i) = packed;
            if (blockIdx.x == 0 && p.stream) *reinterpret_cast<float4*>(p.stream + base + i) = p.pre ? sum : v;
            if (blockIdx.x == 0 && p.low) *reinterpret_cast<uint2*>(p.low + base + i) = packed;
        }
    }
    __syncthreads();
}

// The same for a residual of several streams. Every CTA forms the norm's operand, and stores its share of the new streams.
template <bool YB> __device__ void streams_prologue(const LinP& p, bf16* xs, int stride, float* red) {
    const int rows = (int)p.rows, K = (int)p.k[0], S = p.streams, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per = rows <= 1 ? 8 : rows <= 2 ? 4 : rows <= 4 ? 2 : 1;
    const int row = warp / per, t = ((warp % per) * 32 + lane) * 4, step = per * 128;
    const long long y0 = (long long)row * p.ny_ld, base = (long long)row * K;
    const float* res = p.nres + base * S;
    __shared__ float con[kMaxStreams * (kMaxStreams + 2)], take[kMaxStreams + 1];  // take: what the operand takes of every old stream and of y
    for (int i = threadIdx.x; i < S * (S + 2); i += kThreads) con[i] = p.connect[i];
    __syncthreads();
    const float *out = con + S * S, *in = out + S;
    if ((int)threadIdx.x <= S) {
        float a = 0.f;
        for (int u = 0; u < S; u++) a = fmaf(in[u], (int)threadIdx.x < S ? con[threadIdx.x * S + u] : out[u], a);
        take[threadIdx.x] = a;
    }
    float f1 = p.y_scale, f2 = 0.f;
    auto total_of = [&](float ss) {  // of this row
        ss = warp_sum(ss);
        __syncthreads();
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
        if (row < rows)
            for (int i = 0; i < per; i++) tot += red[row * per + i];
        return 1.f / sqrtf(tot / (float)K + p.eps);
    };
    auto squares = [&](const void* y, long long at) {
        float ss = 0.f;
        if (row < rows) {
#pragma unroll 4
            for (int i = t; i < K; i += step) {
                const float4 v = ld_y4<YB>(y, at + i);
                ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
            }
        }
        return ss;
    };
    if (p.npost) f1 = total_of(squares(p.ny, y0));
    if (p.ny2) f2 = total_of(squares(p.ny2, base));
    __syncthreads();
    auto result = [&](int i) {  // y'
        float4 v = ld_y4<YB>(p.ny, y0 + i);
        v = make_float4(v.x * f1, v.y * f1, v.z * f1, v.w * f1);
        if (p.npost) v = mul4(v, *reinterpret_cast<const float4*>(p.npost + i));
        if (p.ny2) {
            const float4 o = ld_y4<YB>(p.ny2, base + i), w = *reinterpret_cast<const float4*>(p.npost2 + i);
            v = add4(v, make_float4(o.x * f2 * w.x, o.y * f2 * w.y, o.z * f2 * w.z, o.w * f2 * w.w));
        }
        return v;
    };
    auto plus = [](float4 a, float f, float4 b) { return make_float4(fmaf(f, b.x, a.x), fmaf(f, b.y, a.y), fmaf(f, b.z, a.z), fmaf(f, b.w, a.w)); };
    auto operand = [&](int i, float4 y) {
        float4 v = plus(make_float4(0.f, 0.f, 0.f, 0.f), take[S], y);
        if (p.nres)
#pragma unroll 4
            for (int r = 0; r < S; r++) v = plus(v, take[r], *reinterpret_cast<const float4*>(res + (long long)r * K + i));
        return v;
    };
    float ss = 0.f;
    if (row < rows)
#pragma unroll 2
        for (int i = t; i < K; i += step) {
            const float4 y = result(i), v = operand(i, y);
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
            if (p.stream && (row + i / 128 * rows) % gridDim.x == blockIdx.x)  // (128 elements of a row: one warp)
                for (int u = 0; u < S; u++) {
                    float4 s = plus(make_float4(0.f, 0.f, 0.f, 0.f), out[u], y);
                    if (p.nres)
                        for (int r = 0; r < S; r++) s = plus(s, con[r * S + u], *reinterpret_cast<const float4*>(res + (long long)r * K + i));
                    *reinterpret_cast<float4*>(p.stream + base * S + (long long)u * K + i) = s;
                }
        }
    const float rstd = total_of(ss);
    if (row < rows) {
#pragma unroll 2
        for (int i = t; i < K; i += step) {
            const float4 u = operand(i, result(i)), w = *reinterpret_cast<const float4*>(p.nw + i);
            const uint2 packed = make_uint2(pack_bf16(u.x * rstd * w.x, u.y * rstd * w.y), pack_bf16(u.z * rstd * w.z, u.w * rstd * w.w));
            *reinterpret_cast<uint2*>(xs + (long long)row * stride + i) = packed;
            if (blockIdx.x == 0 && p.low) *reinterpret_cast<uint2*>(p.low + base + i) = packed;
        }
    }
    __syncthreads();
}

// The same for a norm of several runs of columns: a warp takes a row's run at a time.
template <bool YB> __device__ void groups_prologue(const LinP& p, bf16* xs, int stride) {
    const int rows = (int)p.rows, K = (int)p.k[0], G = p.norm_groups, size = K / G, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int unit = warp; unit < rows * G; unit += kThreads / 32) {
        const int row = unit / G, at = unit % G * size;
        const long long y0 = (long long)row * p.ny_ld + at;
        float ss = 0.f;
        for (int i = lane * 4; i < size; i += 128) {
            const float4 v = ld_y4<YB>(p.ny, y0 + i);
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
        const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)size + p.eps);
        for (int i = lane * 4; i < size; i += 128) {
            float4 v = ld_y4<YB>(p.ny, y0 + i);
            v = mul4(make_float4(v.x * rstd, v.y * rstd, v.z * rstd, v.w * rstd), *reinterpret_cast<const float4*>(p.nw + at + i));
            if (p.ngate) v = mul4(v, ld_y4<true>(p.ngate, row * p.gate_ld + at + i));
            const uint2 packed = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
            *reinterpret_cast<uint2*>(xs + (long long)row * stride + at + i) = packed;
            if (blockIdx.x == 0 && p.low) *reinterpret_cast<uint2*>(p.low + (long long)row * K + at + i) = packed;
            if (blockIdx.x == 0 && p.stream) *reinterpret_cast<float4*>(p.stream + (long long)row * K + at + i) = v;
        }
    }
    __syncthreads();
}

// NT groups of eight activation rows
// NORM: what runs in front of the product
enum : int { PRO_NONE, PRO_NORM, PRO_STREAMS, PRO_GROUPS };
// BLOCKS: block-diagonal products; a row tile belongs to one block.
template <int NT, int NORM, bool BLOCKS> __global__ void __launch_bounds__(kStreamWarps * 32, 2) linear_stream(const __grid_constant__ LinP p) {
    constexpr int kBatch = NT == 4 ? 2 : 4;  // 32-k chunks a warp has in flight
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float red[kStreamWarps][16][NT * 8 + 1];
    __shared__ float norm_red[kStreamWarps];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int c0 = (int)((p.k[0] + 31) / 32), c1 = (int)((p.k[1] + 31) / 32), chunks = c0 + c1;
    const int block_tiles = (int)((p.out + 15) / 16), tiles = BLOCKS ? block_tiles * p.blocks : block_tiles;
    const int per_tile = (chunks + kStreamWarps * kBatch - 1) / (kStreamWarps * kBatch);  // batches of a warp per row tile
    const int my_tiles = blockIdx.x < tiles ? (tiles - 1 - (int)blockIdx.x) / (int)gridDim.x + 1 : 0;
    const int total = my_tiles * per_tile;

    // chunk `c` of the joint k range → operand and first k of this lane
    auto where = [&](int c, int& op, long long& k) {
        op = c >= c0 ? 1 : 0;
        k = (long long)(op ? c - c0 : c) * 32 + t * 8;
        return c < chunks && k < p.k[op];
    };
    uint4 wl[kBatch], wh[kBatch];
    auto fetch = [&](int it) {
        const int tile = (int)blockIdx.x + (it / per_tile) * (int)gridDim.x;
        const int block = BLOCKS ? tile / block_tiles : 0;
        const long long r0 = (long long)(tile - block * block_tiles) * 16 + g, r1 = r0 + 8;
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            const int c = ((it % per_tile) * kBatch + j) * kStreamWarps + warp;
            int op;
            long long k;
            const bool live = it < total && where(c, op, k);
            const bf16* w = (const bf16*)p.w[live ? op : 0];
            if constexpr (BLOCKS) w += block * p.out * p.k[0];
            wl[j] = wh[j] = make_uint4(0, 0, 0, 0);
            if (live && r0 < p.out) wl[j] = ld_weights(w + r0 * p.k[op] + k);
            if (live && r1 < p.out) wh[j] = ld_weights(w + r1 * p.k[op] + k);
        }
    };
    pdl_trigger();
    fetch(0);
    pdl_wait();
    bf16* xs = reinterpret_cast<bf16*>(smem);
    const int stride = ((int)p.k[0] + 63) / 64 * 64 + 32;  // 64 bytes off a multiple of 128: conflict-free fragment loads
    if constexpr (NORM == PRO_NORM) {
        if (p.ny_bf16) norm_prologue<true>(p, xs, stride, norm_red);
        else norm_prologue<false>(p, xs, stride, norm_red);
    } else if constexpr (NORM == PRO_STREAMS) {
        if (p.ny_bf16) streams_prologue<true>(p, xs, stride, norm_red);
        else streams_prologue<false>(p, xs, stride, norm_red);
    } else if constexpr (NORM == PRO_GROUPS) {
        if (p.ny_bf16) groups_prologue<true>(p, xs, stride);
        else groups_prologue<false>(p, xs, stride);
    }
    float acc[NT][4];
    for (int it = 0; it < total; it++) {
        if (it % per_tile == 0) {
#pragma unroll
            for (int n = 0; n < NT; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[n][e] = 0.f;
        }
        uint4 a[kBatch], b[kBatch];
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            a[j] = wl[j];
            b[j] = wh[j];
        }
        uint4 xv[kBatch][NT];
        long long x0 = 0;
        if constexpr (BLOCKS) x0 = p.x_off + ((int)blockIdx.x + (it / per_tile) * (int)gridDim.x) / block_tiles * p.x_step;
#pragma unroll
        for (int j = 0; j < kBatch; j++) {
            const int c = ((it % per_tile) * kBatch + j) * kStreamWarps + warp;
            int op;
            long long k;
            const bool live = where(c, op, k);
#pragma unroll
            for (int n = 0; n < NT; n++) {
                const long long row = n * 8 + g;
                xv[j][n] = make_uint4(0, 0, 0, 0);
                if (live && row < p.rows) {
                    if constexpr (NORM != PRO_NONE) xv[j][n] = *reinterpret_cast<const uint4*>(xs + row * stride + k);
                    else if constexpr (BLOCKS) xv[j][n] = *reinterpret_cast<const uint4*>((const bf16*)p.x[0] + row * p.ldx + x0 + k);
                    else xv[j][n] = *reinterpret_cast<const uint4*>((const bf16*)p.x[op] + row * p.k[op] + k);
                }
            }
        }
        fetch(it + 1);
#pragma unroll
        for (int j = 0; j < kBatch; j++)
#pragma unroll
            for (int n = 0; n < NT; n++) {
                mma_bf16(acc[n], a[j].x, b[j].x, a[j].y, b[j].y, xv[j][n].x, xv[j][n].y);
                mma_bf16(acc[n], a[j].z, b[j].z, a[j].w, b[j].w, xv[j][n].z, xv[j][n].w);
            }
        if (it % per_tile == per_tile - 1) {
#pragma unroll
            for (int n = 0; n < NT; n++) {
                red[warp][g][n * 8 + t * 2] = acc[n][0];
                red[warp][g][n * 8 + t * 2 + 1] = acc[n][1];
                red[warp][g + 8][n * 8 + t * 2] = acc[n][2];
                red[warp][g + 8][n * 8 + t * 2 + 1] = acc[n][3];
            }
            __syncthreads();
            long long tile = (long long)blockIdx.x + (it / per_tile) * (long long)gridDim.x, col0 = 0;  // col0: the block's first column
            if constexpr (BLOCKS) {
                col0 = tile / block_tiles * p.out;
                tile %= block_tiles;
            }
            auto total_of = [&](int r, int m) {
                float s = 0.f;
#pragma unroll
                for (int w = 0; w < kStreamWarps; w++) s += red[w][r][m];
                const long long o = tile * 16 + r;
                return s + (p.bias && o < p.out ? p.bias[col0 + o] : 0.f);
            };
            if constexpr (BLOCKS) {
                for (int i = tid; i < 16 * NT * 8; i += kStreamWarps * 32) {
                    const int r = i & 15, m = i >> 4;
                    const long long o = tile * 16 + r;
                    if (m < p.rows && o < p.out) put(p, m, p.ldy, col0 + o, activate(p, col0 + o, total_of(r, m)) * factor<bf16>(p, m, col0 + o));
                }
            } else if (p.glu) {
                for (int i = tid; i < 8 * NT * 8; i += kStreamWarps * 32) {
                    const int r = i & 7, m = i >> 3;
                    const long long o = tile * 8 + r;
                    if (m < p.rows && o < p.out / 2) put(p, m, p.out / 2, o, glu_value(p, total_of(2 * r, m), total_of(2 * r + 1, m)));
                }
            } else {
                for (int i = tid; i < 16 * NT * 8; i += kStreamWarps * 32) {
                    const int r = i & 15, m = i >> 4;
                    const long long o = tile * 16 + r;
                    if (m < p.rows && o < p.out) put(p, m, p.out, o, activate(p, o, total_of(r, m)));
                }
            }
            __syncthreads();
        }
    }
}

// ───────────────────────────── tcgen05 GEMM ─────────────────────────────
constexpr int kTcThreads = 192;      // warps 0-3 epilogue, 4 TMA, 5 MMA
constexpr int kTcPanelA = 128 * 128; // bytes: 128 weight rows × 64 k

// What the epilogue does: EPI_PLAIN bias only, EPI_GLU the gated unit, EPI_ACT functions of columns and factors. Kernels of their own: the
// paths of one are short enough to stay in the instruction cache.
enum : int { EPI_PLAIN, EPI_GLU, EPI_ACT };
template <int EPI> __global__ void __launch_bounds__(kTcThreads) linear_tc(const __grid_constant__ LinP p) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nb = p.nb, S = p.stages;
    const int stage_bytes = kTcPanelA + nb * 128;
    int group = 0, n0 = (int)blockIdx.x * nb, n_live = nb;
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(smem + (size_t)S * stage_bytes);  // full[S], empty[S], done
    unsigned* tmem_slot = reinterpret_cast<unsigned*>(bars + 2 * S + 1);
    pdl_trigger();
    if (p.groups) {  // the counts come from an earlier launch
        pdl_wait();
        if (!locate_group(p, (int)blockIdx.x, nb, &group, &n0, &n_live)) return;
    }
    if (tid == 0) {
        for (int s = 0; s < 2 * S + 1; s++) mbar_init(smem_u32(bars + s), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    int cols = 32;
    while (cols < nb) cols <<= 1;
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned tmem = *tmem_slot;

    const int s0 = (int)((p.k[0] + 63) / 64), all = s0 + (int)((p.k[1] + 63) / 64);
    const int lo = (int)((long long)all * blockIdx.z / p.splits), steps = (int)((long long)all * (blockIdx.z + 1) / p.splits) - lo;
    // activation tiles first: they share a weight tile while it is in L2
    const int block_tiles = (int)((p.out + 127) / 128), block = p.blocks > 1 ? (int)blockIdx.y / block_tiles : 0;
    const int m0 = ((int)blockIdx.y - block * block_tiles) * 128, w0 = (group + block) * (int)p.out + m0;
    const int x0 = (int)(p.x_off + block * p.x_step);
    bool ok = true;

    if (warp == 4) {
        if (lane == 0) {
            auto load_w = [&](int i) {
                const int s = i % S, c = lo + i, op = c >= s0;
                mbar_expect_tx(smem_u32(bars + s), (unsigned)stage_bytes);
                tma_load_2d(smem_u32(smem + (size_t)s * stage_bytes), p.maps[op * 2 + 1], (op ? c - s0 : c) * 64, w0, smem_u32(bars + s));
            };
            auto load_x = [&](int i) {
                const int s = i % S, c = lo + i, op = c >= s0;
                tma_load_2d(smem_u32(smem + (size_t)s * stage_bytes + kTcPanelA), p.maps[op * 2], (op ? c - s0 : c) * 64 + x0, n0, smem_u32(bars + s));
            };
            const int head = min(S, steps);
            for (int i = 0; i < head; i++) load_w(i);  // constants: may overlap the launches before this one
            pdl_wait();
            for (int i = 0; i < head; i++) load_x(i);
            int issued = head;
            for (; issued < steps; issued++) {
                if (!mbar_wait(smem_u32(bars + S + issued % S), ((issued / S) - 1) & 1)) {
                    ok = false;
                    break;
                }
                load_w(issued);
                load_x(issued);
            }
            // every copy has landed before this CTA's shared memory can be given away
            for (int s = 0; s < head; s++)
                if (!mbar_wait(smem_u32(bars + s), ((issued - 1 - s) / S) & 1)) ok = false;
        } else {
            pdl_wait();
        }
    } else if (warp == 5) {
        pdl_wait();
        const unsigned idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(nb >> 3) << 17) | (8u << 24);  // bf16 × bf16 → f32, M 128 × N nb
        for (int i = 0; i < steps; i++) {
            const int s = i % S;
            if (ok && !mbar_wait(smem_u32(bars + s), (i / S) & 1)) ok = false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (lane == 0 && ok) {
                const unsigned a0 = smem_u32(smem + (size_t)s * stage_bytes), b0 = a0 + kTcPanelA;
#pragma unroll
                for (int j = 0; j < 4; j++) umma_bf16(tmem, umma_kmajor_desc(a0 + j * 32), umma_kmajor_desc(b0 + j * 32), idesc, i > 0 || j > 0);
                umma_commit(smem_u32(bars + S + s));
            }
            __syncwarp();
        }
        if (lane == 0) umma_commit(smem_u32(bars + 2 * S));
        __syncwarp();
    } else {
        pdl_wait();
        if (!mbar_wait(smem_u32(bars + 2 * S), 0)) ok = false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const long long o = (long long)m0 + warp * 32 + lane;  // weight row = accumulator lane
        const long long col0 = block * p.out;
        const float bias = p.bias && p.splits == 1 && o < p.out ? p.bias[col0 + o] : 0.f;
        const long long live = min((long long)n_live, p.rows - n0);
        const int f = EPI == EPI_ACT && col0 + o < p.act_end ? p.act[col0 + o >= p.act_split] : ACT_NONE;
        for (int c = 0; c < nb && c < live; c += 16) {
            unsigned v[16];
            asm volatile(
                "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n"
                : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]),
                  "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
                : "r"(tmem + ((unsigned)(warp * 32) << 16) + (unsigned)c));
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            if (p.splits > 1) {
                float* part = p.partial + ((size_t)blockIdx.z * p.rows + n0 + c) * p.ldy + col0 + o;
#pragma unroll
                for (int j = 0; j < 16; j++)
                    if (ok && o < p.out && c + j < live) part[(size_t)j * p.ldy] = __uint_as_float(v[j]);
            } else if constexpr (EPI == EPI_GLU) {
                // lanes 2i and 2i + 1 hold gate and up; of two activation rows the even lane finishes the first, the odd one
                // the second
                const int odd = lane & 1;
                const long long width = p.out / 2, at = (n0 + c + odd) * width + (o >> 1);
                const bool mine = ok && (o | 1) < p.out;
#pragma unroll
                for (int j = 0; j < 16; j += 2) {
                    const float lo = __uint_as_float(v[j]) + bias, hi = __uint_as_float(v[j + 1]) + bias;
                    const float got = __shfl_xor_sync(0xffffffffu, odd ? lo : hi, 1);
                    const float y = glu_value(p, odd ? got : lo, odd ? hi : got);
                    if (!mine || c + j + odd >= live) continue;
                    if (p.y_bf16) ((bf16*)p.y)[at + j * width] = __float2bfloat16_rn(y);
                    else ((float*)p.y)[at + j * width] = y;
                }
            } else if (ok && o < p.out) {
                float y[16];
#pragma unroll
                for (int j = 0; j < 16; j++) y[j] = __uint_as_float(v[j]) + bias;
                if constexpr (EPI == EPI_ACT) {
                    if (f == ACT_SOFTPLUS) {
#pragma unroll
                        for (int j = 0; j < 16; j++) y[j] = softplus_fast(y[j]);
                    } else if (f != ACT_NONE && p.y_bf16) {
#pragma unroll
                        for (int j = 0; j < 16; j++) y[j] = sigmoid_fast(y[j]) * (f == ACT_SILU ? y[j] : 1.f);
                    } else if (f != ACT_NONE) {
#pragma unroll
                        for (int j = 0; j < 16; j++) y[j] = sigmoid_f(y[j]) * (f == ACT_SILU ? y[j] : 1.f);
                    }
                    if (p.mul)
#pragma unroll
                        for (int j = 0; j < 16; j++)
                            if (c + j < live) y[j] *= factor<bf16>(p, n0 + c + j, col0 + o);
                }
                const long long at = (n0 + c) * p.ldy + col0 + o;
                if (p.y_bf16) {
                    bf16* to = (bf16*)p.y + at;
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (c + j < live) to[j * p.ldy] = __float2bfloat16_rn(y[j]);
                } else {
                    float* to = (float*)p.y + at;
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (c + j < live) to[j * p.ldy] = y[j];
                }
            }
        }
    }
    if (!ok && lane == 0) report(p.err, ERR_WAIT_TIMEOUT, p.node, (long long)blockIdx.x, (long long)warp);
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 5) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}

// Adds the pieces of a product that was cut along k, in piece order, with bias and gating. blockIdx.y is the activation
// row; V consecutive weight rows per thread (V = 4: out is a multiple of 4).
template <int V> __global__ void __launch_bounds__(256) linear_reduce(const __grid_constant__ LinP p) {
    pdl_enter();
    const long long row = blockIdx.y, o = ((long long)blockIdx.x * 256 + threadIdx.x) * V;
    if (o >= p.out) return;
    const size_t piece = (size_t)p.rows * p.out;
    const float* src = p.partial + row * p.out + o;
    float s[V];
#pragma unroll
    for (int e = 0; e < V; e++) s[e] = 0.f;
#pragma unroll 4
    for (int z = 0; z < p.splits; z++) {
        if constexpr (V == 4) {
            const float4 f = *reinterpret_cast<const float4*>(src + z * piece);
            s[0] += f.x;
            s[1] += f.y;
            s[2] += f.z;
            s[3] += f.w;
        } else {
#pragma unroll
            for (int e = 0; e < V; e++) s[e] += src[z * piece + e];
        }
    }
    if (p.bias)
#pragma unroll
        for (int e = 0; e < V; e++) s[e] += p.bias[o + e];
    if (!p.glu)
#pragma unroll
        for (int e = 0; e < V; e++) s[e] = activate(p, o + e, s[e]) * factor<bf16>(p, row, o + e);
    if (p.glu) {  // out is even, and so are o and V
#pragma unroll
        for (int e = 0; e < V; e += 2) put(p, row, p.out / 2, (o + e) / 2, glu_value(p, s[e], s[e + 1]));
    } else if (V == 4 && !p.y_bf16) {
        *reinterpret_cast<float4*>((float*)p.y + row * p.out + o) = make_float4(s[0], s[1 % V], s[2 % V], s[3 % V]);
    } else {
#pragma unroll
        for (int e = 0; e < V; e++)
            if (o + e < p.out) put(p, row, p.out, o + e, s[e]);
    }
}

// ───────────────────────────── any shape ────────────────────────────────
template <typename T> __global__ void __launch_bounds__(256) linear_simt(const __grid_constant__ LinP p) {
    __shared__ float xs[16][65], ws[16][65];
    pdl_enter();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int block_tiles = (int)((p.out + 63) / 64), block = p.blocks > 1 ? (int)blockIdx.x / block_tiles : 0;
    const long long m0 = (long long)((int)blockIdx.x - block * block_tiles) * 64, x0 = p.x_off + block * p.x_step, col0 = block * p.out;
    long long n0 = (long long)blockIdx.y * 64, rows = p.rows, w_at = col0;  // w_at: first row of the group's or block's weights
    if (p.groups) {
        int group, row, live;
        if (!locate_group(p, (int)blockIdx.y, 64, &group, &row, &live)) return;
        n0 = row;
        rows = row + live;
        w_at = group * p.out;
    }
    float acc[4][4] = {};  // [row][weight row]
    for (int op = 0; op < 2; op++) {
        const T *x = (const T*)p.x[op], *w = (const T*)p.w[op];
        const long long ldx = p.ldx ? p.ldx : p.k[op];
        for (long long k0 = 0; k0 < p.k[op]; k0 += 16) {
            for (int i = tid; i < 1024; i += 256) {
                const int kk = i & 15, r = i >> 4;
                const bool kl = k0 + kk < p.k[op];
                xs[kk][r] = kl && n0 + r < rows ? to_f(x[(n0 + r) * ldx + x0 + k0 + kk]) : 0.f;
                ws[kk][r] = kl && m0 + r < p.out ? to_f(w[(w_at + m0 + r) * p.k[op] + k0 + kk]) : 0.f;
            }
            __syncthreads();
#pragma unroll
            for (int kk = 0; kk < 16; kk++) {
                float a[4], b[4];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    a[i] = xs[kk][ty * 4 + i];
                    b[i] = ws[kk][tx * 4 + i];
                }
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
            }
            __syncthreads();
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const long long row = n0 + ty * 4 + i;
        if (row >= rows) continue;
        float v[4];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const long long o = m0 + tx * 4 + j;
            v[j] = acc[i][j] + (p.bias && o < p.out ? p.bias[col0 + o] : 0.f);
        }
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const long long o = m0 + tx * 4 + j;
            if (p.glu) {
                if (!(j & 1) && o + 1 < p.out) put(p, row, p.out / 2, o >> 1, glu_value(p, v[j], v[j + 1]));
            } else if (o < p.out) {
                put(p, row, p.ldy, col0 + o, activate(p, col0 + o, v[j]) * factor<T>(p, row, col0 + o));
            }
        }
    }
}

// ───────────────────────────── residual norm ────────────────────────────
struct ResNormP {
    const void* y;
    const float *w, *gain, *res, *post, *offset;
    const void *gate, *add;
    float* stream;
    void* low;
    int* zero;
    long long rows, width, y_ld, gate_ld;
    float eps, y_scale, add_scale;
    int y_bf16, low_bf16, gate_bf16, add_bf16, pre, n_zero, groups;
};
// One CTA per row; V consecutive elements per load.
template <int V> struct Pack {
    float v[V];
};
template <int V> __device__ __forceinline__ Pack<V> ld_pack(const void* p, long long i, bool is_bf16) {
    Pack<V> o;
    if constexpr (V == 4) {
        const float4 f = is_bf16 ? ld_y4<true>(p, i) : ld_y4<false>(p, i);
        o.v[0] = f.x;
        o.v[1] = f.y;
        o.v[2] = f.z;
        o.v[3] = f.w;
    } else {
        o.v[0] = is_bf16 ? __bfloat162float(((const bf16*)p)[i]) : ((const float*)p)[i];
    }
    return o;
}
template <int V> __device__ __forceinline__ void st_pack(void* p, long long i, const Pack<V>& v, bool is_bf16) {
    if constexpr (V == 4) {
        if (is_bf16) *reinterpret_cast<uint2*>((bf16*)p + i) = make_uint2(pack_bf16(v.v[0], v.v[1]), pack_bf16(v.v[2], v.v[3]));
        else *reinterpret_cast<float4*>((float*)p + i) = make_float4(v.v[0], v.v[1], v.v[2], v.v[3]);
    } else {
        if (is_bf16) ((bf16*)p)[i] = __float2bfloat16_rn(v.v[0]);
        else ((float*)p)[i] = v.v[0];
    }
}
template <int V> __global__ void __launch_bounds__(256) residual_norm(const ResNormP p) {
    __shared__ float red[32];
    pdl_enter();
    const long long row = blockIdx.x, base = row * p.width;
    if (row == 0)
        for (int i = threadIdx.x; i < p.n_zero; i += 256) p.zero[i] = 0;
    const long long y0 = row * p.y_ld;
    auto rstd_of = [&](auto&& value) {
        float ss = 0.f;
#pragma unroll 4
        for (long long i = threadIdx.x * V; i < p.width; i += 256 * V) {
            const Pack<V> y = value(i);
#pragma unroll
            for (int e = 0; e < V; e++) ss = fmaf(y.v[e], y.v[e], ss);
        }
        return 1.f / sqrtf(block_sum(ss, red) / (float)p.width + p.eps);
    };
    const float inner = p.post ? rstd_of([&](long long i) { return ld_pack<V>(p.y, y0 + i, p.y_bf16); }) : p.y_scale;
    auto normed = [&](long long i) {  // what the mean square is taken of
        Pack<V> y = ld_pack<V>(p.y, y0 + i, p.y_bf16);
        auto plus = [&](const void* from, long long at, bool is_bf16, float scale) {
            const Pack<V> r = ld_pack<V>(from, at, is_bf16);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] = fmaf(r.v[e], scale, y.v[e]);
        };
        if (p.pre) {
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] *= inner;
            if (p.post) {
                const Pack<V> w = ld_pack<V>(p.post, i, false);
#pragma unroll
                for (int e = 0; e < V; e++) y.v[e] *= w.v[e];
            }
            if (p.res) plus(p.res, base + i, false, 1.f);
            if (p.add) plus(p.add, base + i, p.add_bf16, p.add_scale);
            if (p.offset) plus(p.offset, i, false, 1.f);
        }
        return y;
    };
    const float rstd = rstd_of(normed);
#pragma unroll 2
    for (long long i = threadIdx.x * V; i < p.width; i += 256 * V) {
        const Pack<V> sum = normed(i), w = ld_pack<V>(p.w, i, false);
        Pack<V> y;
#pragma unroll
        for (int e = 0; e < V; e++) y.v[e] = sum.v[e] * (rstd * w.v[e]);
        if (p.gain) {
            const Pack<V> g = ld_pack<V>(p.gain, i, false);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] *= g.v[e];
        }
        if (p.gate) {
            const Pack<V> g = ld_pack<V>(p.gate, row * p.gate_ld + i, p.gate_bf16);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] *= g.v[e];
        }
        if (!p.pre && p.res) {
            const Pack<V> r = ld_pack<V>(p.res, base + i, false);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] += r.v[e];
        }
        if (p.stream) st_pack<V>(p.stream, base + i, p.pre ? sum : y, false);
        if (p.low) st_pack<V>(p.low, base + i, y, p.low_bf16);
    }
}

// A residual of several streams: one CTA per row, the norm's operand in shared memory in between. S: the most streams.
struct StreamsP {
    const void *y, *y2;
    const float *w, *res, *post, *post2, *connect;
    float* stream;
    void* low;
    int* zero;
    long long width, y_ld;
    float eps, y_scale;
    int y_bf16, low_bf16, streams, n_zero;
};
template <int V, int S> __global__ void __launch_bounds__(256) streams_norm(const StreamsP p) {
    extern __shared__ __align__(16) float operand[];
    __shared__ float red[32], con[S * (S + 2)];
    pdl_trigger();
    const int n = p.streams, tid = threadIdx.x;
    for (int i = tid; i < n * (n + 2); i += 256) con[i] = p.connect[i];  // constants
    pdl_wait();
    const long long row = blockIdx.x, base = row * p.width, y0 = row * p.y_ld;
    if (row == 0)
        for (int i = tid; i < p.n_zero; i += 256) p.zero[i] = 0;
    auto factor_of = [&](const void* y, long long at) {
        float ss = 0.f;
#pragma unroll 4
        for (long long i = tid * V; i < p.width; i += 256 * V) {
            const Pack<V> v = ld_pack<V>(y, at + i, p.y_bf16);
#pragma unroll
            for (int e = 0; e < V; e++) ss = fmaf(v.v[e], v.v[e], ss);
        }
        return 1.f / sqrtf(block_sum(ss, red) / (float)p.width + p.eps);
    };
    const float f1 = p.post ? factor_of(p.y, y0) : p.y_scale, f2 = p.y2 ? factor_of(p.y2, base) : 0.f;
    __syncthreads();
    const float *out = con + n * n, *in = out + n;
    float ss = 0.f;
#pragma unroll 2
    for (long long i = tid * V; i < p.width; i += 256 * V) {
        Pack<V> y = ld_pack<V>(p.y, y0 + i, p.y_bf16), x[S], u;
        if (p.res)
#pragma unroll
            for (int r = 0; r < S; r++)
                if (r < n) x[r] = ld_pack<V>(p.res, base * n + r * p.width + i, false);
#pragma unroll
        for (int e = 0; e < V; e++) y.v[e] *= f1;
        if (p.post) {
            const Pack<V> w = ld_pack<V>(p.post, i, false);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] *= w.v[e];
        }
        if (p.y2) {
            const Pack<V> o = ld_pack<V>(p.y2, base + i, p.y_bf16), w = ld_pack<V>(p.post2, i, false);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] = fmaf(o.v[e] * f2, w.v[e], y.v[e]);
        }
#pragma unroll
        for (int e = 0; e < V; e++) u.v[e] = 0.f;
#pragma unroll
        for (int t = 0; t < S; t++) {
            if (t >= n) break;
            Pack<V> s;
#pragma unroll
            for (int e = 0; e < V; e++) s.v[e] = out[t] * y.v[e];
            if (p.res)
#pragma unroll
                for (int r = 0; r < S; r++)
                    if (r < n)
#pragma unroll
                        for (int e = 0; e < V; e++) s.v[e] = fmaf(con[r * n + t], x[r].v[e], s.v[e]);
#pragma unroll
            for (int e = 0; e < V; e++) u.v[e] = fmaf(in[t], s.v[e], u.v[e]);
            if (p.stream) st_pack<V>(p.stream, base * n + t * p.width + i, s, false);
        }
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(u.v[e], u.v[e], ss);
        st_pack<V>(operand, i, u, false);
    }
    const float rstd = 1.f / sqrtf(block_sum(ss, red) / (float)p.width + p.eps);
    if (!p.low) return;
#pragma unroll 4
    for (long long i = tid * V; i < p.width; i += 256 * V) {
        Pack<V> u = ld_pack<V>(operand, i, false);
        const Pack<V> w = ld_pack<V>(p.w, i, false);
#pragma unroll
        for (int e = 0; e < V; e++) u.v[e] *= rstd * w.v[e];
        st_pack<V>(p.low, base + i, u, p.low_bf16);
    }
}

// A norm of several runs of columns, times a gate: one warp per row and run.
template <int V> __global__ void __launch_bounds__(256) groups_norm(const ResNormP p) {
    pdl_enter();
    const int size = (int)p.width / p.groups, lane = threadIdx.x & 31;
    if (blockIdx.x == 0)
        for (int i = threadIdx.x; i < p.n_zero; i += 256) p.zero[i] = 0;
    const long long unit = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (unit >= p.rows * p.groups) return;
    const long long row = unit / p.groups, at = unit % p.groups * size, y0 = row * p.y_ld + at;
    float ss = 0.f;
#pragma unroll 4
    for (int i = lane * V; i < size; i += 32 * V) {
        const Pack<V> y = ld_pack<V>(p.y, y0 + i, p.y_bf16);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(y.v[e], y.v[e], ss);
    }
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)size + p.eps);
#pragma unroll 4
    for (int i = lane * V; i < size; i += 32 * V) {
        Pack<V> y = ld_pack<V>(p.y, y0 + i, p.y_bf16);
        const Pack<V> w = ld_pack<V>(p.w, at + i, false);
#pragma unroll
        for (int e = 0; e < V; e++) y.v[e] *= rstd * w.v[e];
        if (p.gate) {
            const Pack<V> g = ld_pack<V>(p.gate, row * p.gate_ld + at + i, p.gate_bf16);
#pragma unroll
            for (int e = 0; e < V; e++) y.v[e] *= g.v[e];
        }
        if (p.stream) st_pack<V>(p.stream, row * p.width + at + i, y, false);
        if (p.low) st_pack<V>(p.low, row * p.width + at + i, y, p.low_bf16);
    }
}

constexpr Buf kNull{kSlotNull, 0};
constexpr int64_t kFusedNormElements = 12288;
Buf buf_of(const TRef* t) { return t ? t->buf : kNull; }

}  // namespace

static void emit_streams_norm(Emitter& em, const ResidualNormDesc& d, const TRef* low, Buf zero, int n_zero) {
    StreamsP p{};
    p.width = d.w->numel();
    p.y_ld = d.y->shape[1];
    p.eps = (float)d.eps;
    p.y_scale = (float)d.y_scale;
    p.y_bf16 = d.y->dtype == DT_BF16;
    p.low_bf16 = low && low->dtype == DT_BF16;
    p.streams = (int)d.streams;
    p.n_zero = n_zero;
    bool wide = p.width % 4 == 0 && p.y_ld % 4 == 0 && d.y_off % 4 == 0;
    for (const TRef* t : {d.y, d.w, d.res, d.post, d.y2, d.post2, d.stream, low}) wide = wide && (!t || t->buf.off % 16 == 0);
    const auto k = wide ? (p.streams <= 2 ? streams_norm<4, 2> : p.streams <= 4 ? streams_norm<4, 4> : p.streams <= 8 ? streams_norm<4, 8> : streams_norm<1, kMaxStreams>)
                        : (p.streams <= 4 ? streams_norm<1, 4> : streams_norm<1, kMaxStreams>);
    const unsigned smem = (unsigned)p.width * 4;
    ensure_max_dynamic_smem((const void*)k, 200 * 1024);
    em.launch(k, dim3((unsigned)d.y->shape[0]), dim3(256), smem, p,
              {{&p.y, d.y->buf.at(d.y_off * (p.y_bf16 ? 2 : 4))}, {&p.y2, buf_of(d.y2)}, {&p.w, d.w->buf}, {&p.res, buf_of(d.res)}, {&p.post, buf_of(d.post)}, {&p.post2, buf_of(d.post2)},
               {&p.connect, d.connect->buf}, {&p.stream, buf_of(d.stream)}, {&p.low, buf_of(low)}, {&p.zero, n_zero ? zero : kNull}},
              "streams_norm", /*pdl=*/true);
}

void emit_residual_norm(Emitter& em, const ResidualNormDesc& d, const TRef* low, Buf zero, int n_zero) {
    ResNormP p{};
    p.width = d.w->numel();
    const long long rows = d.y->shape[0];
    if (rows == 0) return;
    if (d.streams > 0) return emit_streams_norm(em, d, low, zero, n_zero);
    p.rows = rows;
    p.groups = (int)d.groups;
    p.y_ld = d.y->shape[1];
    p.add_scale = (float)d.add_scale;
    p.add_bf16 = d.add && d.add->dtype == DT_BF16;
    p.eps = (float)d.eps;
    p.y_scale = (float)d.y_scale;
    p.pre = d.pre;
    p.y_bf16 = d.y->dtype == DT_BF16;
    p.low_bf16 = low && low->dtype == DT_BF16;
    p.n_zero = n_zero;
    bool wide = p.width % 4 == 0;  // every row is 16-byte aligned when the tensors are
    wide = wide && p.y_ld % 4 == 0 && d.y_off % 4 == 0;
    for (const TRef* t : {d.y, d.w, d.gain, d.res, d.post, d.add, d.offset, d.stream, low}) wide = wide && (!t || t->buf.off % 16 == 0);
    Buf gate = kNull;
    if (d.gate) {
        p.gate_bf16 = d.gate->dtype == DT_BF16;
        p.gate_ld = d.gate->shape[1];
        gate = d.gate->buf.at(d.gate_off * (p.gate_bf16 ? 2 : 4));
        wide = wide && p.gate_ld % 4 == 0 && d.gate_off % 4 == 0 && d.gate->buf.off % 16 == 0;
    }
    wide = wide && (p.width / d.groups) % 4 == 0;
    const auto k = d.groups > 1 ? (wide ? groups_norm<4> : groups_norm<1>) : wide ? residual_norm<4> : residual_norm<1>;
    em.launch(k, dim3((unsigned)(d.groups > 1 ? (rows * d.groups + 7) / 8 : rows)), dim3(256), 0, p,
              {{&p.y, d.y->buf.at(d.y_off * (p.y_bf16 ? 2 : 4))}, {&p.post, buf_of(d.post)}, {&p.add, buf_of(d.add)}, {&p.offset, buf_of(d.offset)}, {&p.w, d.w->buf}, {&p.gain, buf_of(d.gain)}, {&p.res, buf_of(d.res)}, {&p.gate, gate}, {&p.stream, buf_of(d.stream)},
               {&p.low, buf_of(low)}, {&p.zero, n_zero ? zero : kNull}},
              "residual_norm", /*pdl=*/true);
}

void emit_linear(Emitter& em, const LinearDesc& d, const TRef* x0, const TRef* x1, const TRef& w0, const TRef* w1, const TRef* bias,
                 const TRef& y, const ResidualNormDesc* norm, const TRef* low) {
    if (d.rows == 0) return;
    const bool tc_type = w0.dtype == DT_BF16;
    const bool blocks = d.blocks > 1 || d.x_off > 0 || d.mul || (x0 && x0->shape[1] != d.k[0]);
    const long long ldx = x0 ? x0->shape[1] : d.k[0];
    const bool aligned = d.k[0] % 8 == 0 && d.k[1] % 8 == 0 && (!blocks || (ldx % 8 == 0 && d.x_off % 8 == 0 && d.x_step % 8 == 0));
    const size_t norm_smem = (size_t)d.rows * ((d.k[0] + 63) / 64 * 64 + 32) * 2;
    const bool gate_fits = !norm || !norm->gate || (norm->gate->shape[1] % 4 == 0 && norm->gate_off % 4 == 0 && norm->gate->buf.off % 16 == 0);
    const bool y_fits = norm && norm->y->shape[1] % 4 == 0 && norm->y_off % 4 == 0;
    // every CTA of the product repeats the norm: beyond some elements a launch of its own is shorter
    const int pro = !norm ? PRO_NONE : norm->streams > 0 ? PRO_STREAMS : norm->groups > 1 ? PRO_GROUPS : PRO_NORM;
    const bool parts_fit = pro == PRO_GROUPS ? (d.k[0] / norm->groups) % 4 == 0 : pro != PRO_STREAMS || !norm->y2 || norm->y2->dtype == norm->y->dtype;
    const int64_t read = d.rows * d.k[0] * (pro == PRO_STREAMS ? (norm->streams + 1) / 2 : 1);
    const bool fuse_norm = norm && tc_type && aligned && gate_fits && y_fits && parts_fit && d.rows <= 8 && read <= kFusedNormElements;
    TRef made;
    if (norm && !fuse_norm) {
        made.dtype = w0.dtype;
        made.shape = {d.rows, d.k[0]};
        // in 32-bit the sum of a norm that is not followed by another operation is the operand itself
        const bool own = w0.dtype == DT_F32 && norm->stream && !norm->pre && !low;
        if (low) made.buf = low->buf;
        else made.buf = own ? norm->stream->buf : em.scratch((size_t)d.rows * d.k[0] * (tc_type ? 2 : 4));
        emit_residual_norm(em, *norm, own ? nullptr : &made);
        x0 = &made;
    }
    LinP p{};
    p.ldx = blocks ? ldx : 0;
    p.x_off = d.x_off;
    p.x_step = d.x_step;
    p.blocks = (int)d.blocks;
    p.ldy = d.blocks * d.out;
    p.mul_ld = d.mul ? d.mul->shape[1] : 0;
    const Buf mul = d.mul ? d.mul->buf.at(d.mul_off * (tc_type ? 2 : 4)) : kNull;
    p.rows = d.rows;
    p.out = d.out;
    p.k[0] = d.k[0];
    p.k[1] = d.k[1];
    p.y_bf16 = y.dtype == DT_BF16;
    p.fast = tc_type;
    p.glu = d.glu;
    p.alpha = d.alpha;
    p.limit = d.limit;
    p.shift = d.shift;
    p.act[0] = d.act[0];
    p.act[1] = d.act[1];
    p.act_split = d.act_split;
    p.act_end = d.act_end > 0 ? d.act_end : d.blocks * d.out;
    p.node = em.node;
    p.splits = 1;
    const Buf bx0 = fuse_norm ? kNull : x0->buf, bx1 = buf_of(x1), bw1 = buf_of(w1), bb = buf_of(bias);
    if (!tc_type || !aligned) {
        const dim3 grid((unsigned)((d.out + 63) / 64 * d.blocks), (unsigned)((d.rows + 63) / 64));
        const auto k = tc_type ? linear_simt<bf16> : linear_simt<float>;
        em.launch(k, grid, dim3(256), 0, p, {{&p.mul, mul}, {&p.x[0], bx0}, {&p.x[1], bx1}, {&p.w[0], w0.buf}, {&p.w[1], bw1}, {&p.bias, bb}, {&p.y, y.buf}},
                  "linear_simt", /*pdl=*/true);
        return;
    }
    if (d.rows <= 32) {
        const long long tiles = (d.out + 15) / 16 * d.blocks;
        const dim3 grid((unsigned)std::min<long long>(tiles, 2 * sm_count()));
        const int nt = d.rows <= 8 ? 1 : d.rows <= 16 ? 2 : 4;
        auto k = nt == 1 ? linear_stream<1, PRO_NONE, false> : nt == 2 ? linear_stream<2, PRO_NONE, false> : linear_stream<4, PRO_NONE, false>;
        if (blocks) k = nt == 1 ? linear_stream<1, PRO_NONE, true> : nt == 2 ? linear_stream<2, PRO_NONE, true> : linear_stream<4, PRO_NONE, true>;
        unsigned smem = 0;
        if (fuse_norm) {
            k = pro == PRO_STREAMS ? linear_stream<1, PRO_STREAMS, false> : pro == PRO_GROUPS ? linear_stream<1, PRO_GROUPS, false> : linear_stream<1, PRO_NORM, false>;
            p.streams = (int)norm->streams;
            p.norm_groups = (int)norm->groups;
            smem = (unsigned)norm_smem;
            ensure_max_dynamic_smem((const void*)k, 100 * 1024);
            p.eps = (float)norm->eps;
            p.ny_bf16 = norm->y->dtype == DT_BF16;
            p.y_scale = (float)norm->y_scale;
            p.pre = norm->pre;
            p.ny_ld = norm->y->shape[1];
            p.add_scale = (float)norm->add_scale;
            p.add_bf16 = norm->add && norm->add->dtype == DT_BF16;
            p.gate_ld = norm->gate ? norm->gate->shape[1] : 0;
        }
        em.launch(k, grid, dim3(kStreamWarps * 32), smem, p,
                  {{&p.x[0], bx0}, {&p.x[1], bx1}, {&p.w[0], w0.buf}, {&p.w[1], bw1}, {&p.bias, bb}, {&p.y, y.buf}, {&p.mul, mul},
                   {&p.npost, fuse_norm ? buf_of(norm->post) : kNull}, {&p.nadd, fuse_norm ? buf_of(norm->add) : kNull},
                   {&p.noffset, fuse_norm ? buf_of(norm->offset) : kNull}, {&p.connect, fuse_norm ? buf_of(norm->connect) : kNull},
                   {&p.ny2, fuse_norm ? buf_of(norm->y2) : kNull}, {&p.npost2, fuse_norm ? buf_of(norm->post2) : kNull},
                   {&p.ny, fuse_norm ? norm->y->buf.at(norm->y_off * (p.ny_bf16 ? 2 : 4)) : kNull}, {&p.nw, fuse_norm ? norm->w->buf : kNull},
                   {&p.ngain, fuse_norm ? buf_of(norm->gain) : kNull}, {&p.nres, fuse_norm ? buf_of(norm->res) : kNull},
                   {&p.ngate, fuse_norm && norm->gate ? norm->gate->buf.at(norm->gate_off * 2) : kNull},
                   {&p.stream, fuse_norm ? buf_of(norm->stream) : kNull}, {&p.low, fuse_norm ? buf_of(low) : kNull}},
                  "linear_stream", /*pdl=*/true);
        return;
    }
    // Activation rows per tile and pieces along k: the choice with the smallest modelled time, waves × (64-k steps of a
    // CTA × cost of a step + set-up and drain), plus the trip of the partial sums and a second launch where k is cut.
    const long long mt = (d.out + 127) / 128 * d.blocks, steps = (d.k[0] + 63) / 64 + (d.k[1] + 63) / 64;
    double best = 1e300;
    for (int nb : {32, 64, 128, 256}) {
        if (nb > 32 && nb / 2 >= d.rows) break;
        const int resident = nb <= 128 ? 2 : 1;
        const long long slots = (long long)sm_count() * resident, tiles = mt * ((d.rows + nb - 1) / nb);
        for (int sp = 1; sp <= (d.rows < 65536 ? 16 : 1) && sp * 2 <= std::max<long long>(steps, 2); sp++) {
            const long long waves = (tiles * sp + slots - 1) / slots;
            // measured: a 64-k step of the CTAs that share an SM, and what a wave costs besides its steps
            const double step_us = nb == 32 ? 0.36 : nb == 64 ? 0.38 : nb == 128 ? 0.42 : 0.45;
            double us = (double)waves * ((double)((steps + sp - 1) / sp) * step_us + (nb == 256 ? 10.0 : 7.0));
            if (sp > 1) us += 3.0 + (double)(sp + 1) * d.rows * p.ldy * 4.0 / 3e6;
            if (us < best * (sp > 1 ? 0.97 : 1.0)) {
                best = us;
                p.nb = nb;
                p.splits = sp;
            }
        }
    }
    if (const char* e = std::getenv("ONYXIA_LINEAR_TILE")) {  // diagnostics: "rows,pieces"
        int nb = 0, sp = 0;
        if (std::sscanf(e, "%d,%d", &nb, &sp) == 2 && (nb == 32 || nb == 64 || nb == 128 || nb == 256) && sp >= 1 && sp <= 16 && sp * 2 <= std::max<long long>(steps, 2)) {
            p.nb = nb;
            p.splits = sp;
        }
    }
    const size_t stage = kTcPanelA + (size_t)p.nb * 128;
    const bool alone = mt * ((d.rows + p.nb - 1) / p.nb) * p.splits <= sm_count();  // one CTA per SM: all of its shared memory
    p.stages = (int)std::min<size_t>(8, (p.nb <= 128 && !alone ? 108 * 1024 : 208 * 1024) / stage);
    const size_t smem = stage * p.stages + 1024 + (2 * p.stages + 1) * 8 + 16;
    const auto kernel = d.glu ? linear_tc<EPI_GLU> : d.act[0] || d.act[1] || d.mul ? linear_tc<EPI_ACT> : linear_tc<EPI_PLAIN>;
    ensure_max_dynamic_smem((const void*)kernel, 220 * 1024);
    const Buf partial = p.splits > 1 ? em.scratch((size_t)p.splits * d.rows * p.ldy * 4) : kNull;
    LaunchRec& rec = em.launch(kernel, dim3((unsigned)((d.rows + p.nb - 1) / p.nb), (unsigned)mt, (unsigned)p.splits), dim3(kTcThreads), (unsigned)smem, p,
                               {{&p.bias, bb}, {&p.y, y.buf}, {&p.mul, mul}, {&p.partial, partial}, {&p.err, Buf{kSlotErr, 0}}}, "linear_tc", /*pdl=*/true);
    auto add_map = [&](int i, const Buf& b, int64_t k, int64_t rows, uint32_t box) {
        rec.tmaps.push_back(TmapReloc{(uint32_t)(offsetof(LinP, maps) + 128 * i), b, (uint64_t)k, (uint64_t)rows, (uint64_t)k * 2, 64u, box});
    };
    add_map(0, bx0, blocks ? ldx : d.k[0], d.rows, (uint32_t)p.nb);
    add_map(1, w0.buf, d.k[0], d.blocks * d.out, 128u);
    if (d.k[1]) {
        add_map(2, bx1, d.k[1], d.rows, (uint32_t)p.nb);
        add_map(3, bw1, d.k[1], d.out, 128u);
    }
    if (p.splits > 1) {
        const bool wide = p.ldy % 4 == 0 && y.buf.off % 16 == 0;
        const int v = wide ? 4 : p.ldy % 2 == 0 ? 2 : 1;  // gating needs pairs; out is even then
        p.out = p.ldy;                                    // all blocks' columns
        em.launch(wide ? linear_reduce<4> : v == 2 ? linear_reduce<2> : linear_reduce<1>,
                  dim3((unsigned)((p.out + 256 * v - 1) / (256 * v)), (unsigned)d.rows), dim3(256), 0, p,
                  {{&p.bias, bb}, {&p.y, y.buf}, {&p.mul, mul}, {&p.partial, partial}}, "linear_reduce", /*pdl=*/true);
    }
}

// One product per group of sorted rows.
void emit_grouped_linear(Emitter& em, const GroupedLinearDesc& d, const TRef& x, const TRef& w, const TRef& counts, const TRef& y) {
    if (d.rows == 0) return;
    LinP p{};
    p.rows = d.rows;
    p.out = d.out;
    p.ldy = d.out;
    p.blocks = 1;
    p.k[0] = d.k;
    p.y_bf16 = y.dtype == DT_BF16;
    p.glu = d.glu;
    p.alpha = d.alpha;
    p.limit = d.limit;
    p.shift = d.shift;
    p.node = em.node;
    p.splits = 1;
    p.groups = (int)d.groups;
    auto tiles_of = [&](int64_t size) { return std::min<int64_t>(d.rows / size + std::min(d.groups, d.rows), d.rows); };
    const bool tc_type = w.dtype == DT_BF16;
    if (!tc_type || d.k % 8 != 0) {
        const auto k = tc_type ? linear_simt<bf16> : linear_simt<float>;
        em.launch(k, dim3((unsigned)((d.out + 63) / 64), (unsigned)tiles_of(64)), dim3(256), 0, p,
                  {{&p.x[0], x.buf}, {&p.x[1], kNull}, {&p.w[0], w.buf}, {&p.w[1], kNull}, {&p.bias, kNull}, {&p.y, y.buf}, {&p.counts, counts.buf}},
                  "grouped_simt", /*pdl=*/true);
        return;
    }
    // Rows per tile: whole tiles plus half a tile per group are expected to be filled.
    const long long mt = (d.out + 127) / 128, steps = (d.k + 63) / 64;
    double best = 1e300;
    for (int nb : {32, 64, 128, 256}) {
        const long long slots = (long long)sm_count() * (nb <= 128 ? 2 : 1);
        const double groups = (double)std::min(d.groups, d.rows), tiles = std::max(groups, (double)d.rows / nb + 0.5 * groups);
        const double step_us = nb == 32 ? 0.36 : nb == 64 ? 0.38 : nb == 128 ? 0.42 : 0.45;
        const double waves = std::max(1.0, tiles * (double)mt / (double)slots);
        const double us = waves * ((double)steps * step_us + (nb == 256 ? 10.0 : 7.0));
        if (us < best) {
            best = us;
            p.nb = nb;
        }
    }
    if (const char* e = std::getenv("ONYXIA_GROUPED_TILE")) {  // diagnostics: rows
        const int nb = std::atoi(e);
        if (nb == 32 || nb == 64 || nb == 128 || nb == 256) p.nb = nb;
    }
    const size_t stage = kTcPanelA + (size_t)p.nb * 128;
    p.stages = (int)std::min<size_t>(8, (p.nb <= 128 ? 108 * 1024 : 208 * 1024) / stage);
    const size_t smem = stage * p.stages + 1024 + (2 * p.stages + 1) * 8 + 16;
    const auto kernel = d.glu ? linear_tc<EPI_GLU> : linear_tc<EPI_PLAIN>;
    ensure_max_dynamic_smem((const void*)kernel, 220 * 1024);
    LaunchRec& rec = em.launch(kernel, dim3((unsigned)tiles_of(p.nb), (unsigned)mt, 1), dim3(kTcThreads), (unsigned)smem, p,
                               {{&p.bias, kNull}, {&p.y, y.buf}, {&p.partial, kNull}, {&p.err, Buf{kSlotErr, 0}}, {&p.counts, counts.buf}}, "grouped_tc",
                               /*pdl=*/true);
    auto add_map = [&](int i, const Buf& b, int64_t rows, uint32_t box) {
        rec.tmaps.push_back(TmapReloc{(uint32_t)(offsetof(LinP, maps) + 128 * i), b, (uint64_t)d.k, (uint64_t)rows, (uint64_t)d.k * 2, 64u, box});
    };
    add_map(0, x.buf, d.rows, (uint32_t)p.nb);
    add_map(1, w.buf, d.groups * d.out, 128u);
}

}  // namespace oxk
