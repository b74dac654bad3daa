// Attention over one latent per token that all heads share: key = (latent, rotated part), value = latent. Queries come with their
// unrotated part mapped into the latent space, results leave in it; both maps are block-diagonal products (linear.cu).
//
//   latent_prepare   the new latents, normed, and their rotated part go to the pool; queries are put together
//   the rest         paged_kv_attention.cu: one key head, values at the front of the keys
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
    void* q;                     // [rows, heads · (rank + rot)]
    const int* seqs;             // [R, 4]
    const int* table;            // [R, width]
    ErrWord* err;
    long long rows, ld, q_ld;
    int n_seqs, width, n_pages, shift, heads, kv_heads, rank, rot, q_step, node;
    float eps;
};

// One CTA per row.
template <typename T> __global__ void __launch_bounds__(128) latent_prepare(const LatP p) {
    extern __shared__ float angle[];  // cos[rot / 2], sin[rot / 2]
    __shared__ float red[32];
    pdl_enter();
    const int row = blockIdx.x, s = find_seq(p.seqs, p.n_seqs, row), tid = threadIdx.x, half = p.rot / 2, dim = p.rank + p.rot;
    const SeqRow sq = load_seq(p.seqs, s);
    const int pos = sq.past + row - sq.start;
    if (row >= sq.start + sq.len) return;
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
    T* q = (T*)p.q + (long long)row * p.heads * dim;
    for (int h = 0; h < p.heads; h++) {
        for (int i = tid; i < p.rank; i += 128) q[h * dim + i] = lat[h * p.rank + i];
        for (int i = tid; i < p.rot; i += 128) q[h * dim + p.rank + i] = from_f<T>(rotated(half, 0, own + (long long)h * p.q_step, angle, angle + half, i));
    }
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
    TRef ready;
    ready.dtype = proj.dtype;
    ready.shape = {rows, d.heads * dim};
    ready.buf = em.scratch((size_t)(rows * d.heads * dim * element));
    em.launch(bf ? latent_prepare<bf16> : latent_prepare<float>, dim3((unsigned)rows), dim3(128), (unsigned)(d.rot * 4), p,
              {{&p.q_latent, q_latent.buf}, {&p.q_own, q.buf.at(d.q_off * element)}, {&p.proj, proj.buf.at(d.kv_off * element)}, {&p.norm_w, norm_w.buf},
               {&p.turns, turns.buf}, {&p.pool, pool.buf}, {&p.q, ready.buf}, {&p.seqs, seqs.buf}, {&p.table, pages.buf}, {&p.err, Buf{kSlotErr, 0}}},
              "latent_prepare", /*pdl=*/true);
    PagedKvDesc kd{};
    kd.heads = d.heads;
    kd.kv_heads = 1;
    kd.dim = dim;
    kd.vdim = d.rank;
    kd.page = d.page;
    kd.scale = d.scale;
    kd.latent = true;
    emit_paged_kv_attention(em, kd, ready, turns, pool, pool, seqs, pages, out);
}

}  // namespace oxk
