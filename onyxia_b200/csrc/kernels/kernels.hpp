// Host-side interface to the CUDA kernels: one `emit_*` function per kernel
// family. An emit function does not launch; it appends launch records
// ({function, grid, block, shared memory, parameter bytes, pointer
// relocations}) to an Emitter. The session replays the records — directly, or
// as nodes of a CUDA graph — after patching pointer fields with the current
// buffer addresses.
#pragma once
#include <cuda_runtime.h>

#include <cstdint>
#include <cstring>
#include <algorithm>
#include <cmath>
#include <initializer_list>
#include <memory>
#include <stdexcept>
#include <string>
#include <utility>
#include <vector>

namespace oxk {

// Error codes written to the error word (first writer wins).
enum : int {
    ERR_NONE = 0,
    ERR_GATHER_OOB = 1,
    ERR_SCATTER_OOB = 2,
    ERR_INT_DIV_ZERO = 3,
    ERR_INT_POW_NEG = 4,
    ERR_SLICE_OOB = 5,
    ERR_WAIT_TIMEOUT = 6,
    ERR_SAMPLE_NO_FINITE = 7,
};

struct ErrWord {
    int code;
    int node;      // launch tag (IR node index)
    long long a;   // offending value
    long long b;   // bound
};

// A device address known only at execution time: a runtime value slot plus a
// byte offset into it.
struct Buf {
    uint32_t slot = 0xFFFFFFFFu;
    int64_t off = 0;
    Buf at(int64_t bytes) const { return Buf{slot, off + bytes}; }
    bool valid() const { return slot != 0xFFFFFFFFu; }
};
// Reserved slots resolved by the session.
constexpr uint32_t kSlotErr = 0xFFFFFFF0u;      // the session's ErrWord
constexpr uint32_t kSlotScratch = 0xFFFFFFF1u;  // the plan's scratch area (offset = position in it)
constexpr uint32_t kSlotNull = 0xFFFFFFF2u;     // resolves to nullptr
// A session-lifetime array of kCounterWords zeroed 32-bit arrival counters;
// kernels that use it leave every word zero again when they finish.
constexpr uint32_t kSlotCounters = 0xFFFFFFF3u;
constexpr size_t kCounterWords = 1 << 16;
// The plan's block of per-run scalars (int64 each; offset = byte position).
// Values that change from run to run without changing the launch geometry —
// the KV length of a decode step — are read from here by the kernels, so the
// parameter bytes of their launches stay identical and a CUDA graph replays
// unmodified. The session refreshes the block before every run.
constexpr uint32_t kSlotDyn = 0xFFFFFFF4u;
constexpr int kDynPerNode = 4;

struct Reloc {
    uint32_t field_off;  // byte offset of a pointer field inside the parameter struct
    Buf buf;
};

// A 2-D tiled tensor map over f16 elements that has to be encoded into the parameter bytes once the
// address of its tensor is known (TMA loads: `cp.async.bulk.tensor`).
struct TmapReloc {
    uint32_t field_off;      // byte offset of the 128-byte map inside the parameter struct (64-byte aligned there)
    Buf buf;                 // base of the tensor
    uint64_t dim0, dim1;     // extents in elements: contiguous axis, outer axis
    uint64_t stride1_bytes;  // bytes between outer rows (a multiple of 16)
    uint32_t box0, box1;     // tile extents in elements (box0·2 ≤ 128 bytes with the 128-byte swizzle)
    // Byte offset of an int32 field of the parameter struct that the kernel reads as "use the map"; it is
    // cleared when the tensor's address in a run turns out not to be 16-byte aligned (the kernel then takes
    // its plain-load path). 0xFFFFFFFF: no such field, a misaligned tensor is an error.
    uint32_t enable_off = 0xFFFFFFFFu;
};

struct PersistOp;  // persist.hpp

struct LaunchRec {
    const void* func = nullptr;
    dim3 grid{1, 1, 1}, block{1, 1, 1};
    dim3 cluster{0, 0, 0};  // thread-block cluster shape; x = 0 launches without clusters
    unsigned smem = 0;
    std::vector<uint8_t> params;
    std::vector<Reloc> relocs;
    std::vector<TmapReloc> tmaps;
    const char* label = "";
    int node = -1;  // IR node index, for error messages and profiling
    // The kernel executes `griddepcontrol.wait` before it reads anything an
    // earlier launch wrote and before it writes anything at all, on every path
    // to its exit. Such a kernel may be launched while its predecessor in the
    // stream is still running (programmatic dependent launch): its prologue —
    // barrier set-up, prefetch of constant weights — overlaps the predecessor.
    // Every such kernel triggers its own dependents at entry, so the section
    // before its wait may overlap not only the launch before it but several
    // earlier ones: it may read only memory that NO launch of the same run
    // writes (constants, rows of a KV cache below the step's first new row).
    bool pdl = false;
    // Not a kernel of this library: a collective the session enqueues itself. The parameter bytes
    // are a CollP (with the usual pointer relocations); `func` is null.
    int coll = 0;  // 1 = sum over the tensor-parallel ranks
    // The grid's CTAs wait on one another: the launch must be cooperative (all CTAs co-resident).
    bool cooperative = false;
    // What this launch does, in the form the persistent step kernel executes: a run of consecutive
    // launches that all carry one can be replaced by a single launch of that kernel.
    std::shared_ptr<const PersistOp> pop;
};

struct CollP {
    const void* send;
    void* recv;
    unsigned long long count;
    int dtype;
};

class Emitter {
public:
    std::vector<LaunchRec> recs;
    int node = -1;
    size_t scratch_bytes = 0;  // high-water mark of scratch requested by this plan

    // Reserve `bytes` of scratch that lives for the duration of one node.
    Buf scratch(size_t bytes, size_t align = 256) {
        size_t off = (scratch_cursor_ + align - 1) / align * align;
        scratch_cursor_ = off + bytes;
        if (scratch_cursor_ > scratch_bytes) scratch_bytes = scratch_cursor_;
        return Buf{kSlotScratch, (int64_t)off};
    }
    void begin_node(int n) {
        node = n;
        scratch_cursor_ = 0;
        dyn_vals.clear();
    }
    // Register a per-run scalar of the current node; kernels read it through
    // the returned address instead of from their parameter bytes.
    std::vector<int64_t> dyn_vals;
    Buf dyn(int64_t value) {
        if ((int)dyn_vals.size() >= kDynPerNode) throw std::runtime_error("too many per-run scalars for one node");
        dyn_vals.push_back(value);
        return Buf{kSlotDyn, (int64_t)((node * kDynPerNode + (int)dyn_vals.size() - 1) * 8)};
    }

    template <class P>
    LaunchRec& launch(void (*kernel)(const P), dim3 grid, dim3 block, unsigned smem, const P& p,
                std::initializer_list<std::pair<const void*, Buf>> ptrs, const char* label, bool pdl = false) {
        static_assert(sizeof(P) <= 4000, "kernel parameter struct too large");
        LaunchRec r;
        r.func = (const void*)kernel;
        r.grid = grid;
        r.block = block;
        r.smem = smem;
        r.params.resize(sizeof(P));
        std::memcpy(r.params.data(), &p, sizeof(P));
        for (auto& pr : ptrs) {
            Reloc rl;
            rl.field_off = (uint32_t)((const char*)pr.first - (const char*)&p);
            rl.buf = pr.second;
            r.relocs.push_back(rl);
        }
        r.label = label;
        r.node = node;
        r.pdl = pdl;
        recs.push_back(std::move(r));
        return recs.back();
    }

private:
    size_t scratch_cursor_ = 0;
};

// A tensor operand at lowering time: symbolic address, dtype code, concrete dims.
struct TRef {
    Buf buf;
    int dtype = 0;
    std::vector<int64_t> shape;
    // Physical row capacity of axis 2 for KV-cache tensors ([B, KV, T, D] whose
    // buffer holds `cap` rows per head); 0 = densely packed.
    int64_t cap = 0;
    int64_t numel() const {
        int64_t n = 1;
        for (auto d : shape) n *= d;
        return n;
    }
};

// Streaming multiprocessors of the current device (cached per device; thread-safe).
int sm_count();
// Raises a kernel's dynamic shared-memory limit on the current device once (thread-safe); throws on failure.
void ensure_max_dynamic_smem(const void* func, int bytes);

inline unsigned grid_for(int64_t n, int block, int64_t max_blocks = 0) {
    if (max_blocks <= 0) max_blocks = (int64_t)sm_count() * 16;
    int64_t g = (n + block - 1) / block;
    if (g < 1) g = 1;
    if (g > max_blocks) g = max_blocks;
    return (unsigned)g;
}

// ── primitives (one kernel family per IR primitive) ─────────────────────
void emit_unary(Emitter&, int op, const TRef& x, const TRef& y);
void emit_binary(Emitter&, int op, const TRef& a, const TRef& b, const TRef& y);
void emit_compare(Emitter&, int op, const TRef& a, const TRef& b, const TRef& y);
void emit_select(Emitter&, const TRef& c, const TRef& a, const TRef& b, const TRef& y);
void emit_cast(Emitter&, const TRef& x, const TRef& y);
void emit_matmul(Emitter&, const TRef& a, const TRef& b, const TRef& y, bool trans_a, bool trans_b);
void emit_reduce(Emitter&, int op, const TRef& x, const TRef& y, const std::vector<size_t>& axes);
void emit_reshape_copy(Emitter&, const TRef& x, const TRef& y);
void emit_transpose(Emitter&, const TRef& x, const TRef& y, const std::vector<size_t>& perm);
void emit_broadcast(Emitter&, const TRef& x, const TRef& y);
void emit_concat(Emitter&, const std::vector<TRef>& xs, const TRef& y, size_t axis);
void emit_slice(Emitter&, const TRef& x, const TRef& y, const std::vector<int64_t>& starts,
                const std::vector<int64_t>& steps);
void emit_gather(Emitter&, const TRef& data, const TRef& idx, const TRef& y, size_t axis);
void emit_scatter(Emitter&, const TRef& data, const TRef& idx, const TRef& upd, const TRef& y);
void emit_iota(Emitter&, const TRef& y);
void emit_dim_values(Emitter&, const std::vector<int64_t>& vals, const TRef& y);
void emit_dequantize(Emitter&, const TRef& q, const TRef& scales, const TRef* zp, const TRef& y, int64_t block_size);

// ── fused composites ────────────────────────────────────────────────────
void emit_softmax(Emitter&, const TRef& x, const TRef& y);  // last axis
// y = x · rsqrt(mean(x²) + eps) · w over the last axis; with `res` the input is
// x + res and the sum is also written to `sum_out`.
void emit_rmsnorm(Emitter&, const TRef& x, const TRef& w, const TRef& y, double eps, const TRef* res,
                  const TRef* sum_out);
void emit_gelu(Emitter&, const TRef& x, const TRef& y, bool tanh_approx, const TRef* mul);  // optional ·mul (GeGLU)
void emit_rotary(Emitter&, const TRef& x, const TRef& pos, const TRef& cos, const TRef& sin, const TRef& y,
                 int64_t heads, int64_t half);

struct GqaDesc {
    int64_t batch, seq, heads, kv_heads, head_dim, past;  // past = P (logical rows of the past tensors)
    double scale;
    int64_t window;        // -1 = none
    int64_t rot_half;      // 0 = no rotary
    int64_t cache_rows;    // rows of cos/sin
    bool has_bias;
    int64_t bias_b, bias_h;  // bias batch/head extents (1 = broadcast)
    bool in_place;         // present aliases past: only new rows are written
    // > 0: size the key split for this many rows (a bucket ≥ past + seq) and let
    // the kernels read the true length from the plan's per-run scalars, so a
    // decode step changes no launch parameter until the bucket is outgrown.
    int64_t t_bucket;
};
void emit_gqa(Emitter&, const GqaDesc&, const TRef& q, const TRef& k, const TRef& v, const TRef& past_k,
              const TRef& past_v, const TRef& seqlens, const TRef* cos, const TRef* sin, const TRef* bias,
              const TRef& out, const TRef& present_k, const TRef& present_v);

// The decode step (S = 1) over an in-place cache as one launch of thread-block
// clusters; false when the shape is outside what that kernel handles. `t_size`
// bounds the present length the launch is sized for; the true length is read
// from `dyn_t` at run time.
// One token per row of `logits` by temperature / top-k / top-p sampling (crates/onyxia-cli/src/sampling.rs:36-195);
// `u` holds one uniform number in [0, 1] per row.
void emit_sample_rows(Emitter&, const TRef& logits, const TRef& out, Buf u, float temperature, long long top_k, float top_p);
// Attention over many new positions on the tensor cores (f16, no bias; after gqa_prepare). False = shape not taken.
bool emit_gqa_prefill_tc(Emitter&, const GqaDesc&, Buf q_rot, const TRef& seqlens, const TRef& out, const TRef& present_k,
                         const TRef& present_v, Buf dyn_t, long long T, long long cap);
bool emit_gqa_decode(Emitter&, const GqaDesc&, const TRef& q, const TRef& k, const TRef& v, const TRef& seqlens,
                     const TRef* cos, const TRef* sin, const TRef& out, const TRef& present_k, const TRef& present_v,
                     Buf dyn_t, long long t_size);

struct NBitsDesc {
    int64_t m, k, n, block_size, n_blocks;
    int act_dtype, scale_dtype;
    bool has_zp;
    // The weight constant was re-laid out by emit_nbits_interleave (backend-
    // private layout for the tensor-core decode kernel).
    bool interleaved;
    // The weight constant was replaced by tile records holding nibbles, scales
    // and zero points together (emit_nbits_pack_tiles); `scales` and `zp` are
    // not read by the kernel.
    bool tiled;
};
// y[m, n] = a[m, :] · dequant(w)[n, :]ᵀ for packed u4 weights [N, n_blocks, bs].
void emit_matmul_nbits(Emitter&, const NBitsDesc&, const TRef& a, const TRef& w, const TRef& scales,
                       const TRef* zp, const TRef& y);

// Tensor-core decode kernel for f16 activations and scales over interleaved weights.
void emit_matmul_nbits_mma(Emitter&, const NBitsDesc&, const TRef& a, const TRef& w, const TRef& scales,
                           const TRef* zp, const TRef& y);
// One-time re-layout of a packed u4 weight constant: within each 32-bit word,
// nibble j moves to position (j >> 1) + 4·(j & 1).
void emit_nbits_interleave(Emitter&, Buf src, Buf dst, long long bytes);

// Streaming decode kernel over tile-major weight records (f16 activations and scales).
void emit_matmul_nbits_stream(Emitter&, const NBitsDesc&, const TRef& a, const TRef& tiles, const TRef& y);
// One-time gathering of a packed u4 weight [N, n_blocks, 32], its f16 scales
// and optional u4 zero points into tile records; `dst` needs nbits_tiled_bytes.
// Row tile rt of the matrix becomes row tile rt·rt_mul + rt_add of the
// destination stream, so several matrices can share one stream (one after the
// other, or interleaved row tile by row tile).
size_t nbits_tiled_bytes(long long n, long long n_blocks, bool has_zp);
void emit_nbits_pack_tiles(Emitter&, Buf w, Buf scales, Buf zp, Buf dst, long long n, long long n_blocks, bool has_zp,
                           long long rt_mul = 1, long long rt_add = 0);

// Several MatMulNBits over the same activations as one launch of the streaming
// kernel, optionally with a prologue on the activations and a GeGLU epilogue:
//   v = a;  [v = rmsnorm(v, eps1)·w1;]  [v = res + v, also stored to sum_out;]  [v = rmsnorm(v, eps2)·w2;]
//   plain:  y[i] = v · W_iᵀ for each segment i (the stream holds W_0's row tiles, then W_1's, …)
//   geglu:  y[0] = gelu(v · W_0ᵀ) · (v · W_1ᵀ), the stream alternating row tiles of W_0 and W_1
// Every step rounds where the primitives of the corresponding decompositions store a tensor.
struct NBitsGroup {
    long long m, k;
    bool has_zp;
    int n_seg;            // 1..3
    long long seg_n[3];
    TRef y[3];
    int geglu;            // 0 none, 1 tanh form, 2 erf form
    const TRef* w1;
    double eps1;
    const TRef* res;
    const TRef* sum_out;
    const TRef* w2;
    double eps2;
};
void emit_nbits_group(Emitter&, const NBitsGroup&, const TRef& a, const TRef& tiles);
// The tcgen05 GEMM form of a group's matrices (any number of activation rows, in passes of up to
// 256): no prologue, no epilogue. `interleave2`: the stream alternates row tiles of segments 0 and 1.
void emit_nbits_gemm_tc(Emitter&, const NBitsGroup&, const TRef& x, const TRef& tiles, bool interleave2);

// y = Σ over the tensor-parallel ranks of x (executed by the session through its communicator).
void emit_allreduce(Emitter&, const TRef& x, const TRef& y);

// ── dense products over unquantised weights ─────────────────────────────
// y[rows, ·] = x0 · W0ᵀ (+ x1 · W1ᵀ) + bias, f32 accumulation; W is [out, k], stored like the activations
// (bf16 on the tensor cores, f32 in true 32-bit).
enum : int { ACT_NONE = 0, ACT_SILU = 1, ACT_SIGMOID = 2, ACT_SOFTPLUS = 3 };
struct LinearDesc {
    int64_t rows, out;
    int64_t k[2];          // k[1] = 0: a single product
    // Block-diagonal products (no second operand, gated unit or norm): block b's columns of y, `out` wide, are
    //   y_b = act(x[:, x_off + b · x_step …+ k] · W_bᵀ + bias_b) · mul[:, mul_off + b · out …],  W [blocks · out, k].
    // One block is a product over a column range of x.
    int64_t blocks = 1, x_off = 0, x_step = 0;
    const struct TRef* mul = nullptr;  // a matrix in the activation type, optional
    int64_t mul_off = 0;
    // Gated unit over interleaved weight rows (row 2i = gate, row 2i + 1 = up):
    //   g = min(gate, limit), u = clamp(up, ±limit), y = g · sigmoid(alpha · g) · (u + shift)
    bool glu = false;
    float alpha = 1.f, limit = INFINITY, shift = 0.f;
    // Without a gated unit: functions of the columns before act_split and of those from there on, to act_end (> 0) at most.
    int act[2] = {ACT_NONE, ACT_NONE};
    int64_t act_split = 0, act_end = 0;
};
// What turns a sublayer's result into the next product's operand.
//   norm of the result:  v = rmsnorm(y, eps) · w · gain · gate + res, and the new residual is v
//   norm of the sum:     s = y · y_scale + res, v = rmsnorm(s, eps) · w · gain · gate, and the new residual is s   (`pre`)
//                        with `post`, y is normed on its way into the sum: s = rmsnorm(y, eps) · post + res
//                        with `add` / `offset`, s also contains add · add_scale / a vector that is the same for all rows
//   norm of a sum of streams (`streams` = S > 0, `pre`): the residual is S streams side by side, and
//                        s_t = Σ_r mix[r, t] res_r + out[t] · y',  v = rmsnorm(Σ_t in[t] s_t) · w,  the new residual is all s_t
//                        y' = y · y_scale or rmsnorm(y) · post, with `y2` / `post2` plus the same of a second result; without a
//                        residual s_t = out[t] · y'
//   `groups` > 1 (neither a residual nor `pre`): the norm is taken of that many runs of columns, each for itself
// The new residual is stored to `stream` when there is one.
constexpr int kMaxStreams = 32;
struct ResidualNormDesc {
    const TRef* y = nullptr;      // f32 or the activation type; columns from y_off on of a matrix
    const TRef* w = nullptr;      // f32
    const TRef* gain = nullptr;   // f32, optional
    const TRef* res = nullptr;    // f32, optional
    const TRef* gate = nullptr;   // columns of a matrix in the activation type, optional
    const TRef* post = nullptr;   // f32, optional
    const TRef* add = nullptr;    // f32 or the activation type, optional
    const TRef* offset = nullptr; // f32, optional
    double add_scale = 1.0;
    int64_t y_off = 0, gate_off = 0;
    const TRef* stream = nullptr; // f32 result, optional
    double eps = 1e-6, y_scale = 1.0;
    bool pre = false;
    int64_t streams = 0, groups = 1;
    const TRef* connect = nullptr;              // f32 [streams² + 2 · streams]: mix (by origin), out, in
    const TRef *y2 = nullptr, *post2 = nullptr; // like y and post
};
// `low`, when given, receives v in its own type. `zero`: integers to clear on the way.
void emit_residual_norm(Emitter&, const ResidualNormDesc&, const TRef* low, Buf zero = {}, int n_zero = 0);
// With `norm` the (single) operand x0 is the residual norm's result v: one launch for up to eight rows, otherwise
// a launch of its own in front of the product. `x0` is ignored then. `low` receives v as the product reads it.
void emit_linear(Emitter&, const LinearDesc&, const TRef* x0, const TRef* x1, const TRef& w0, const TRef* w1, const TRef* bias,
                 const TRef& y, const ResidualNormDesc* norm, const TRef* low = nullptr);
// y[r] = x[r] · W_gᵀ for rows sorted by group g: counts I32 [groups] of the rows of every group lie on the device, W is
// [groups · out, k].
struct GroupedLinearDesc {
    int64_t rows, groups, out, k;
    bool glu = false;
    float alpha = 1.f, limit = INFINITY, shift = 0.f;
};
void emit_grouped_linear(Emitter&, const GroupedLinearDesc&, const TRef& x, const TRef& w, const TRef& counts, const TRef& y);

// ── mixture of experts ──────────────────────────────────────────────────
// h = the residual norm's result; z = router · h + bias; the `top` experts with the largest z, weighted by the softmax over
// their z; y = Σ weight · down_e (glu(up_e h)). `up` is [experts · 2 ff, k] with gate and up rows interleaved, `down`
// [experts · k, ff].
// With `scores` MOE_SIGMOID or MOE_SOFTMAX the scores are sigmoid(z) or the softmax over all z; a choice's weight is its score, with
// `renorm` divided by the sum of the chosen ones, times `route_scale`. `correction` is added to the scores where they are compared.
// With `groups` > 0 the experts form that many runs, and only those of the `keep` runs with the largest sums of their two largest scores
// (`group_max`: the largest score) can be chosen. A shared expert (`shared_ff` > 0), a gated unit of its own size and limit, is added for every
// token; with `shared_gate` times the sigmoid of one more row of the router.
enum : int { MOE_CHOSEN = 0, MOE_SIGMOID = 1, MOE_SOFTMAX = 2 };
struct MoeDesc {
    int64_t rows, width, experts, top, ff;
    float alpha = 1.f, limit = INFINITY, shift = 0.f;
    int scores = MOE_CHOSEN;
    bool renorm = true, group_max = false, shared_gate = false;
    int64_t groups = 0, keep = 0, shared_ff = 0;
    float route_scale = 1.f, shared_limit = INFINITY;
    const TRef* correction = nullptr;  // F32 [experts]
};
constexpr int kMoeMaxGroups = 128;
void emit_moe(Emitter&, const MoeDesc&, const ResidualNormDesc& norm, const TRef& router, const TRef& router_bias, const TRef& up, const TRef& down,
              const TRef* shared_up, const TRef* shared_down, const TRef& y);

// ── ragged batches over pools ───────────────────────────────────────────
// `seqs` is I32 [R, 4]: first row in the batch, new tokens, tokens before them, slot. Rows of one sequence are
// consecutive and ascend with the sequence index; positions count from the tokens before.
// `pages` is I32 [R, width]: the pool pages of a sequence in order.
struct PagedAttnDesc {
    int64_t heads, kv_heads, dim, page;  // page: a power of two
    int64_t q_off, k_off;        // columns of the fused projection
    double scale, eps, out_scale;
    double temp_coef, temp_every;  // queries times 1 + coef · ln(floor((p + 1) / every) + 1); every = 0: none
};
// Causal attention whose values are the keys as projected: the pool [pages, kv_heads, page, dim] holds a token's key
// once, `key_scale` [pages, page] the reciprocal root mean square of its whole key projection. `bias` [heads, n] is
// added to the scaled score of distance d from column min(d, n − 1).
void emit_paged_attention(Emitter&, const PagedAttnDesc&, const TRef& proj, const TRef& q_norm, const TRef& k_norm, const TRef* bias,
                          const TRef& pool, const TRef& key_scale, const TRef& seqs, const TRef& pages, const TRef& out);

struct PagedKvDesc {
    int64_t heads, kv_heads, dim, vdim, page;  // page: a power of two
    int64_t q_off, k_off, v_off;  // columns of the fused projection
    int64_t rot_dims;             // leading dimensions of a head that rotate in two halves; 0: none
    int64_t window;               // keys a position sees, itself among them; 0: all
    double scale, softcap, eps;   // softcap 0: none
    bool norm;                    // queries and keys divided by their root mean square over `dim` after the rotation
    bool sink;                    // a score without a value in every softmax: 0, or `sinks`
    bool append;                  // the new keys and values go to the pools; otherwise they are there already
    bool interleaved = false;     // dimensions 2i and 2i + 1 are a pair instead of i and i + rot_dims / 2
    const struct TRef* sinks = nullptr;  // F32 [heads], natural units, neither scaled nor capped
    int64_t gate_off = -1;        // column of the projection with a factor of every head's result; −1: none
    const struct TRef* temps = nullptr;  // F32 [heads]: factors of the scores
    const struct TRef* talk = nullptr;   // F32 [heads, heads]: row h mixes all heads' softmax weights into those of head h; no window, sink or cap
    bool latent = false;          // `proj` [rows, heads · dim] are finished queries, the values are the leading vdim elements of the keys
};
// Causal attention over pools of keys [pages, kv_heads, page, dim] (as rotated and normed) and values
// [pages, kv_heads, page, vdim]. `turns` F32 [2, rot_dims / 2]: turns per position of every pair, high and low part.
void emit_paged_kv_attention(Emitter&, const PagedKvDesc&, const TRef& proj, const TRef& turns, const TRef& keys, const TRef& values,
                             const TRef& seqs, const TRef& pages, const TRef& out);

// Attention whose keys and values are one latent per token that all heads share: key = (latent, rotated part), value =
// latent. Queries come with their unrotated part already mapped into the latent space (`q_latent` [rows, heads · rank]) and with
// their rotated part in `q` (head h's from column h · q_step + q_off on). The new latents are columns of `proj` from kv_off
// on, `rank` to be normed with `norm_w` and `rot` to be rotated in two halves; `pool` [pages, 1, page, rank + rot] gets both.
// `out` [rows, heads · rank] is the attention's result in the latent space.
struct LatentAttnDesc {
    int64_t heads, rank, rot, page, q_off, q_step, kv_off;
    double scale, eps;
};
void emit_latent_attention(Emitter&, const LatentAttnDesc&, const TRef& q_latent, const TRef& q, const TRef& proj, const TRef& norm_w, const TRef& turns,
                           const TRef& pool, const TRef& seqs, const TRef& pages, const TRef& out);

// u [rows, width] = silu of a causal convolution per channel over columns of `proj` from x_off on; `w` F32 [width, taps] (last column: the
// current token). `ring` [slots, taps, width] keeps the last inputs by position modulo taps; it is only read but with `keep`, which is for batches
// of one new token per sequence.
struct ShortConvDesc {
    int64_t width, taps, x_off;
    bool keep = false;
};
void emit_short_conv(Emitter&, const ShortConvDesc&, const TRef& proj, const TRef& w, const TRef* bias, const TRef& ring, const TRef& seqs, const TRef& u);

// Selective scan behind a causal convolution with silu. Columns of `proj`: `width` inputs from x_off on and as many factors of
// the result from z_off on. u = silu(conv(x)); (dt, B, C) = W_x u with rank + 2 · state columns; dt ← softplus(W_dt dt + dt_b);
//   S[c, n] ← exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n,   out_c = (Σ_n S[c, n] C_n + D_c u_c) · z_c
// `conv_state` [slots, taps, width] keeps the last inputs by position modulo taps, `state` F32 [slots, width, state].
struct SelectiveScanDesc {
    int64_t width, state, rank, taps, x_off, z_off;
};
void emit_selective_scan(Emitter&, const SelectiveScanDesc&, const TRef& proj, const TRef& conv_w, const TRef& conv_b, const TRef& wx, const TRef& wdt,
                         const TRef& dt_b, const TRef& A, const TRef& D, const TRef& conv_state, const TRef& state, const TRef& seqs, const TRef& out);

struct LightningDesc {
    int64_t heads, dim, vdim;
    int64_t q_off, k_off, v_off;  // columns of the fused projection
};
constexpr int kLightningChunk = 64;
// Per head S ← decay S + k vᵀ, o = Sᵀ q with S [slots, heads, dim, vdim] in f32. `decay` F32 [heads, chunk + 2]: the powers
// 0 … chunk of every head's decay, then decay − 1. `out` is F32 [rows, heads · vdim].
void emit_lightning(Emitter&, const LightningDesc&, const TRef& proj, const TRef& decay, const TRef& state, const TRef& seqs, const TRef& out);

// Linear attention with a decay per key channel: per head S ← diag(α) S + k vᵀ, o = Sᵀ (q_scale q), α = sigmoid(z)^(1 / tau) with z F32
// [rows, heads · dim]; q, k and v are columns of `proj`, S [slots, heads, dim, vdim] in f32. `out` is F32 [rows, heads · vdim].
struct GatedLinearDesc {
    int64_t heads, dim, vdim;
    int64_t q_off, k_off, v_off;
    double tau, q_scale;
};
void emit_gated_linear(Emitter&, const GatedLinearDesc&, const TRef& proj, const TRef& z, const TRef& state, const TRef& seqs, const TRef& out);

// Gated delta rule behind a short convolution with silu over the columns q, k, v of `proj` (side by side from q_off on): q and k as unit vectors
// (x / sqrt(Σ x² + unit_eps)), head h reading those of head h / (heads / kv_heads), q times q_scale; per head, with
// g = exp(−decay · softplus(a + dt_bias)) and beta = sigmoid(b) from columns of `proj` (`decay`, `dt_bias` F32 [heads]):
//   S ← g S,  S ← S + k (beta (v − Sᵀ k))ᵀ,  o = Sᵀ q
// `conv_state` [slots, taps, 2 · kv_heads · dim + heads · vdim], `state` F32 [slots, heads, dim, vdim]; `out` is F32 [rows, heads · vdim].
struct DeltaRuleDesc {
    int64_t heads, kv_heads, dim, vdim, taps;
    int64_t q_off, a_off, b_off;
    double q_scale, unit_eps;
};
void emit_delta_rule(Emitter&, const DeltaRuleDesc&, const TRef& proj, const TRef& conv_w, const TRef& decay, const TRef& dt_bias, const TRef& conv_state,
                     const TRef& state, const TRef& seqs, const TRef& out);

struct GatedRecurrenceDesc {
    int64_t width, blocks, taps;
    int64_t x_off, y_off;        // columns of the fused projection: recurrence branch, gelu branch
    double decay, out_scale;     // a = exp(−decay · r · softplus(lam))
};
// Real-gated linear recurrent unit behind a causal convolution, times gelu of the other branch. `conv_state`
// [slots, taps, width] keeps the last inputs by position modulo taps, `state` [slots, width] the f32 recurrence.
void emit_gated_recurrence(Emitter&, const GatedRecurrenceDesc&, const TRef& proj, const TRef& conv_w, const TRef& conv_b,
                           const TRef& ra, const TRef& ra_b, const TRef& ri, const TRef& ri_b, const TRef& lam, const TRef& conv_state,
                           const TRef& state, const TRef& seqs, const TRef& out);

// argmax over the last axis, highest index among equal maxima → i64.
// `part` is scratch of argmax_scratch_bytes(rows) bytes, `counters` the zeroed arrival counters.
constexpr int kArgmaxMaxBlocks = 128;
inline size_t argmax_scratch_bytes(int64_t rows) { return (size_t)rows * kArgmaxMaxBlocks * 12 + 64; }
void emit_argmax_last(Emitter&, const TRef& x, const TRef& y, Buf part, Buf counters);

// The same argmax with its scratch in a fixed array of the module's global
// data: launches one kernel on `stream` and allocates nothing. At most
// kStaticArgmaxMaxRows rows per call; calls on one device share the array and
// must not overlap. Returns nullptr, or a message describing the failure.
constexpr int kStaticArgmaxMaxRows = 64;
const char* argmax_last_static(int device, cudaStream_t stream, const void* x, int dtype, long long rows,
                               long long cols, long long* y);

// Clear the error word (one tiny launch at the head of a plan is not needed:
// the session clears it with a memset when it reads it).
}  // namespace oxk
