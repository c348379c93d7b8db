// Models described layer by layer on the engine's shared loop: per layer one norm whose output both
// sublayers read (parallel residual), a mixer -- lightning (decaying linear attention) or latent
// attention -- and a dense feed-forward.
//
//   in   one stacked linear for everything that reads the normed input, the norm folded into its input
//        staging for small batches
//   mix  the mixer, leaving its gated heads beside the feed-forward activations
//   out  one linear over [heads | activations] that adds both sublayers into the fp32 residual
//
// A decode step takes one token of every row of the batch (each with its own slot and position, read from
// device arrays, so the captured graph serves any set of sequences); a prompt portion takes consecutive
// tokens of one slot.  Both run the same layer code.
#include <algorithm>
#include <cmath>
#include <cstring>

#include "layered.hpp"

namespace prism {

// ---- construction --------------------------------------------------------------------------------------

static int model_alloc(prism_cuda_engine *e, void **p, size_t bytes) {
    *p = nullptr;
    cudaError_t ce = cudaMalloc(p, (bytes + 255) / 256 * 256);
    if (ce != cudaSuccess) return cuda_fail(e->ctx, ce, "cudaMalloc(model)");
    e->lm->allocs.push_back(*p);
    // padding that a kernel reads must be finite
    PRISM_CUDA_TRY(e->ctx, cudaMemsetAsync(*p, 0, (bytes + 255) / 256 * 256, e->ctx->stream));
    return PRISM_OK;
}
template <typename T>
static int model_alloc(prism_cuda_engine *e, T *&p, size_t n) {
    return model_alloc(e, reinterpret_cast<void **>(&p), n * sizeof(T));
}

static uint32_t add_seg(DenseLinear &l, uint32_t rows, uint32_t act) {
    DenseSeg &s = l.seg[l.n_segs];
    s.row0 = l.n_tiles * 128;
    s.rows = rows;
    s.act = act;
    l.n_tiles += (rows + 127) / 128;
    return l.n_segs++;
}
static int finish_linear(prism_cuda_engine *e, DenseLinear &l, uint32_t k_pad) {
    const int rc = dense_alloc(e->ctx, l, k_pad, l.n_tiles);
    if (l.w) e->lm->allocs.push_back(l.w);
    return rc;
}
static LayeredDst &add_name(LayeredModel *m, const std::string &name, uint64_t rows, uint64_t cols) {
    LayeredDst &d = m->names[name];
    d.rows = rows;
    d.cols = cols;
    m->order.push_back(name);
    return d;
}
static void name_packed(LayeredModel *m, const std::string &name, uint32_t rows, uint32_t cols, DenseLinear &l, uint32_t seg, uint32_t k0 = 0) {
    LayeredDst &d = add_name(m, name, rows, cols);
    d.lin = &l;
    d.row0 = l.seg[seg].row0;
    d.k0 = k0;
}
static int name_vector(prism_cuda_engine *e, const std::string &name, uint32_t n, float *&vec, bool is_norm) {
    PRISM_TRY(model_alloc(e, vec, n));
    LayeredDst &d = add_name(e->lm, name, n, 1);
    d.vec = vec;
    d.is_norm = is_norm;
    return PRISM_OK;
}

static int build_layer(prism_cuda_engine *e, uint32_t i, const prism_layer_config &c) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    LayeredLayer &ly = m->layers[i];
    ly.c = c;
    ly.c.decay = ly.c.rot_freq = nullptr;
    const uint32_t D = m->c.width, slots = m->c.max_batch, hv = c.heads * c.vdim;
    const std::string p = "l" + std::to_string(i) + ".", bad = "layer " + std::to_string(i) + ": ";
    if (!c.heads || !c.dim || !c.vdim) return fail(ctx, PRISM_E_ARG, bad + "a mixer size is zero");
    PRISM_TRY(name_vector(e, p + "norm1", D, ly.norm1, true));
    if (c.mixer == PRISM_MIXER_LIGHTNING) {
        if (!c.decay) return fail(ctx, PRISM_E_ARG, bad + "no decays");
        const uint32_t hk = c.heads * c.dim;
        const uint32_t sq = add_seg(ly.in, hk, ACT_SILU), sk = add_seg(ly.in, hk, ACT_SILU), sv = add_seg(ly.in, hv, ACT_SILU),
                       sg = add_seg(ly.in, hv, ACT_SIGMOID);
        name_packed(m, p + "mix.q", hk, D, ly.in, sq);
        name_packed(m, p + "mix.k", hk, D, ly.in, sk);
        name_packed(m, p + "mix.v", hv, D, ly.in, sv);
        name_packed(m, p + "mix.g", hv, D, ly.in, sg);
        PRISM_TRY(name_vector(e, p + "mix.norm", hv, ly.mix_norm, true));
        PRISM_TRY(model_alloc(e, ly.decay, c.heads));
        PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(ly.decay, c.decay, c.heads * 4, cudaMemcpyHostToDevice, ctx->stream));
        PRISM_TRY(model_alloc(e, ly.state, (size_t)slots * c.heads * c.dim * c.vdim));
    } else if (c.mixer == PRISM_MIXER_LATENT_ATTENTION) {
        if (!c.q_rank || !c.kv_rank || 2 * c.rot_pairs > c.rot_dim || (c.rot_pairs && !c.rot_freq))
            return fail(ctx, PRISM_E_ARG, bad + "latent attention needs q_rank, kv_rank and rotation pairs inside rot_dim");
        const uint32_t sdq = add_seg(ly.in, c.q_rank, ACT_NONE), skv = add_seg(ly.in, c.kv_rank + c.rot_dim, ACT_NONE),
                       sg = add_seg(ly.in, hv, ACT_SIGMOID);
        name_packed(m, p + "mix.dq", c.q_rank, D, ly.in, sdq);
        name_packed(m, p + "mix.dkv", c.kv_rank + c.rot_dim, D, ly.in, skv);
        name_packed(m, p + "mix.g", hv, D, ly.in, sg);
        PRISM_TRY(name_vector(e, p + "mix.dq.norm", c.q_rank, ly.dq_norm, true));
        float *dkv_norm = nullptr;
        PRISM_TRY(name_vector(e, p + "mix.dkv.norm", c.kv_rank, dkv_norm, true));
        const uint32_t hq = c.heads * (c.dim + c.rot_dim);
        add_seg(ly.uq, hq, ACT_NONE);
        PRISM_TRY(finish_linear(e, ly.uq, round_up_u32(c.q_rank, 64)));
        name_packed(m, p + "mix.uq", hq, c.q_rank, ly.uq, 0);
        LatentArgs &la = ly.la;
        la.heads = c.heads; la.dim = c.dim; la.rot_dim = c.rot_dim; la.rot_pairs = c.rot_pairs; la.vdim = c.vdim; la.kv_rank = c.kv_rank;
        la.window = c.window; la.scale = c.scale; la.eps = m->c.norm_eps; la.rot_mul = c.rot_mul;
        la.dkv_norm = dkv_norm;
        la.uk_pitch = round_up_u32(c.kv_rank, 8);
        float *freq = nullptr;
        bf16 *uk = nullptr, *uv = nullptr;
        PRISM_TRY(model_alloc(e, freq, std::max(1u, c.rot_pairs)));
        if (c.rot_pairs) PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(freq, c.rot_freq, c.rot_pairs * 4, cudaMemcpyHostToDevice, ctx->stream));
        PRISM_TRY(model_alloc(e, uk, (size_t)c.heads * c.dim * la.uk_pitch));
        PRISM_TRY(model_alloc(e, uv, (size_t)hv * la.uk_pitch));
        la.rot_freq = freq; la.uk = uk; la.uv = uv;
        const bool expand = !m->act32 && latent_expand_ok(la);
        const uint32_t suk = add_seg(ly.ukv, c.heads * c.dim, ACT_NONE), suv = add_seg(ly.ukv, hv, ACT_NONE);
        if (expand) PRISM_TRY(finish_linear(e, ly.ukv, round_up_u32(c.kv_rank, 64)));
        for (int j = 0; j < 2; j++) {
            LayeredDst &d = add_name(m, p + (j ? "mix.uv" : "mix.uk"), j ? hv : c.heads * c.dim, c.kv_rank);
            d.rowmajor = j ? uv : uk;
            d.pitch = la.uk_pitch;
            if (expand) {
                d.lin = &ly.ukv;
                d.row0 = ly.ukv.seg[j ? suv : suk].row0;
            }
        }
        la.cache.pitch = round_up_u32(c.kv_rank + c.rot_dim, 16);
        la.cache.ring = c.window ? (uint32_t)std::min<uint64_t>(m->c.max_seq, (uint64_t)c.window - 1 + m->chunk) : m->c.max_seq;
        PRISM_TRY(model_alloc(e, &la.cache.rows, (size_t)slots * la.cache.ring * la.cache.pitch * (m->act32 ? 4 : 2)));
        ly.splits = latent_rows_splits(la, m->c.max_seq);
    } else {
        return fail(ctx, PRISM_E_ARG, bad + "unknown mixer");
    }
    ly.k_mix = round_up_u32(hv, 64);
    m->proj_pitch = std::max(m->proj_pitch, ly.in.n_tiles * 128);
    if (c.ff) {
        ly.seg_up = add_seg(ly.in, c.ff, ACT_GELU_TANH);
        name_packed(m, p + "mlp.up", c.ff, D, ly.in, ly.seg_up);
        PRISM_TRY(name_vector(e, p + "mlp.up.b", c.ff, ly.up_b, false));
        ly.in.seg[ly.seg_up].bias = ly.up_b;
    }
    PRISM_TRY(finish_linear(e, ly.in, m->width_pad));
    add_seg(ly.out, D, ACT_NONE);
    ly.out.seg[0].mul = m->c.residual_mult;
    PRISM_TRY(finish_linear(e, ly.out, ly.k_mix + round_up_u32(c.ff, 64)));
    name_packed(m, p + "mix.o", D, hv, ly.out, 0);
    if (c.ff) {
        name_packed(m, p + "mlp.down", D, c.ff, ly.out, 0, ly.k_mix);
        PRISM_TRY(name_vector(e, p + "mlp.down.b", D, ly.down_b, false));
        ly.out.seg[0].bias = ly.down_b;
    }
    m->cat_pitch = std::max(m->cat_pitch, ly.out.k_pad);
    if (c.mixer == PRISM_MIXER_LATENT_ATTENTION) {
        m->q_pitch = std::max(m->q_pitch, ly.uq.n_tiles * 128);
        m->cq_pitch = std::max(m->cq_pitch, ly.uq.k_pad);
    }
    return PRISM_OK;
}

static int build_model(prism_cuda_engine *e, const prism_layer_config *layers) {
    LayeredModel *m = e->lm;
    const prism_layered_config &c = m->c;
    const size_t es = m->act32 ? 4 : 2;
    m->width_pad = round_up_u32(c.width, 64);
    m->vocab_pad = round_up_u32(c.vocab, 4);
    m->cap = std::max(m->chunk, c.max_batch);
    m->layers.resize(c.num_layers);  // never resized again: names point into it
    PRISM_TRY(model_alloc(e, m->embed, (size_t)c.vocab * c.width));
    LayeredDst &em = add_name(m, "embed", c.vocab, c.width);
    em.rowmajor = m->embed;
    em.pitch = c.width;
    for (uint32_t i = 0; i < c.num_layers; i++) PRISM_TRY(build_layer(e, i, layers[i]));
    PRISM_TRY(name_vector(e, "final.norm", c.width, m->final_norm, true));
    add_seg(m->head, c.vocab, ACT_NONE);
    m->head.seg[0].mul = c.logit_scale;
    PRISM_TRY(finish_linear(e, m->head, m->width_pad));
    name_packed(m, "head", c.vocab, c.width, m->head, 0);
    m->lg_cap = std::max(64u, c.max_batch);
    PRISM_TRY(model_alloc(e, m->x, (size_t)m->cap * c.width));
    PRISM_TRY(model_alloc(e, m->xw, (size_t)m->lg_cap * c.width));
    PRISM_TRY(model_alloc(e, m->logits, (size_t)m->lg_cap * m->vocab_pad));
    PRISM_TRY(model_alloc(e, &m->xn, (size_t)m->cap * m->width_pad * es));
    PRISM_TRY(model_alloc(e, &m->proj, (size_t)m->cap * m->proj_pitch * es));
    PRISM_TRY(model_alloc(e, &m->cat, (size_t)m->cap * m->cat_pitch * es));
    if (m->q_pitch) {
        PRISM_TRY(model_alloc(e, &m->q, (size_t)m->cap * m->q_pitch * es));
        PRISM_TRY(model_alloc(e, &m->cq, (size_t)m->cap * m->cq_pitch * es));
    }
    PRISM_TRY(model_alloc(e, m->want_idx, m->cap));
    PRISM_TRY(model_alloc(e, m->pf_tok, m->cap));
    PRISM_TRY(model_alloc(e, m->row_slot, c.max_batch));
    PRISM_TRY(model_alloc(e, m->row_pos, c.max_batch));
    size_t qa = 0, part = 0, ml = 0;
    for (const LayeredLayer &ly : m->layers)
        if (ly.c.mixer == PRISM_MIXER_LATENT_ATTENTION) {
            size_t q1, p1, m1;
            latent_rows_scratch_floats(ly.la, ly.splits, &q1, &p1, &m1);
            qa = std::max(qa, q1);
            part = std::max(part, p1);
            ml = std::max(ml, m1);
        }
    if (qa) {
        m->rows_scratch.rows_cap = std::max(c.max_batch, DENSE_GEMV_ROWS);
        PRISM_TRY(model_alloc(e, m->rows_scratch.qa, qa * m->rows_scratch.rows_cap));
        PRISM_TRY(model_alloc(e, m->rows_scratch.part, part * m->rows_scratch.rows_cap));
        PRISM_TRY(model_alloc(e, m->rows_scratch.ml, ml * m->rows_scratch.rows_cap));
    }
    m->slot_pos.assign(c.max_batch, -1);
    return PRISM_OK;
}

void layered_destroy(prism_cuda_engine *e) {
    LayeredModel *m = e->lm;
    for (void *p : m->allocs) cudaFree(p);
    cudaFree(m->ex_lat);
    cudaFree(m->ex_krot);
    cudaFree(m->ex_kv);
    delete m;
    e->lm = nullptr;
}

// ---- weights -------------------------------------------------------------------------------------------

static int place_tensor(prism_cuda_engine *e, LayeredDst &d, const bf16 *src_dev) {
    prism_cuda_ctx *ctx = e->ctx;
    if (d.lin) PRISM_TRY(launch_dense_pack(ctx, *d.lin, src_dev, (uint32_t)d.rows, (uint32_t)d.cols, d.row0, d.k0));
    if (d.rowmajor) PRISM_TRY(launch_bf16_pitch_copy(ctx, src_dev, d.rowmajor, (uint32_t)d.rows, (uint32_t)d.cols, d.pitch));
    if (d.vec) PRISM_TRY(launch_bf16_to_f32(ctx, src_dev, d.vec, d.rows * d.cols));
    d.bound = true;
    return PRISM_OK;
}

int layered_check_bound(prism_cuda_engine *e) {
    LayeredModel *m = e->lm;
    if (m->bound_ok) return PRISM_OK;
    for (const std::string &n : m->order)
        if (!m->names[n].bound) return fail(e->ctx, PRISM_E_STATE, "tensor " + n + " has not been set");
    m->bound_ok = true;
    return PRISM_OK;
}

int layered_synth(prism_cuda_engine *e, uint64_t seed, float sigma) {
    LayeredModel *m = e->lm;
    uint64_t id = 0;
    for (const std::string &n : m->order) {
        LayeredDst &d = m->names[n];
        PRISM_TRY(ensure_stage(e->ctx, d.rows * d.cols * 2, 0));
        bf16 *tmp = reinterpret_cast<bf16 *>(e->ctx->stage_in);
        PRISM_TRY(launch_dense_synth(e->ctx, tmp, d.rows * d.cols, seed * 1000003ull + id++, d.is_norm ? 1.0f : 0.0f, sigma));
        PRISM_TRY(place_tensor(e, d, tmp));
    }
    return PRISM_OK;
}

// ---- the step --------------------------------------------------------------------------------------------

// y = W (norm of) x for `rows` rows: the small-batch kernel with the norm folded in, or norm, then the tensor-core
// GEMM (fp32: the 32-bit kernel).  `normed` receives the normed rows of the unfused path (pitch normed_pitch); when
// only a prefix of the row is normed it is done in place.
static int linear(prism_cuda_engine *e, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows, void *normed,
                  uint32_t normed_pitch) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    if (!m->act32 && ctx->fuse && dense_gemv_ok(in, rows)) return launch_dense_gemv(ctx, l, in, outs, rows);
    const void *x = in.x;
    uint32_t pitch = in.pitch;
    if (in.norm_w) {
        PRISM_TRY(launch_dense_norm(ctx, in, normed, normed_pitch, rows, m->act32));
        x = normed;
        pitch = normed_pitch;
        if (!m->act32 && ctx->fuse && rows <= DENSE_GEMV_ROWS) {
            DenseIn plain{};
            plain.x = x; plain.pitch = pitch;
            return launch_dense_gemv(ctx, l, plain, outs, rows);
        }
    }
    if (m->act32) return launch_dense_f32(ctx, l, (const float *)x, pitch, outs, rows);
    return launch_dense_gemm_tc5(ctx, l, (const bf16 *)x, pitch, outs, rows);
}

static void *at(const LayeredModel *m, void *p, size_t elems) { return (char *)p + elems * (m->act32 ? 4 : 2); }

static int grow_bf16(prism_cuda_engine *e, bf16 *&p, size_t &have, size_t want) {
    if (want <= have) return PRISM_OK;
    PRISM_CUDA_TRY(e->ctx, cudaStreamSynchronize(e->ctx->stream));
    cudaFree(p);
    p = nullptr;
    have = 0;
    cudaError_t ce = cudaMalloc((void **)&p, want * 2);
    if (ce != cudaSuccess) return cuda_fail(e->ctx, ce, "cudaMalloc(expanded keys and values)");
    PRISM_CUDA_TRY(e->ctx, cudaMemsetAsync(p, 0, want * 2, e->ctx->stream));
    have = want;
    return PRISM_OK;
}

static int mix_lightning(prism_cuda_engine *e, LayeredLayer &ly, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    LightningArgs a{};
    a.q = at(m, m->proj, ly.in.seg[0].row0);
    a.k = at(m, m->proj, ly.in.seg[1].row0);
    a.v = at(m, m->proj, ly.in.seg[2].row0);
    a.pitch = m->proj_pitch;
    a.o = m->cat;
    a.o_pitch = m->cat_pitch;
    a.state = ly.state;
    a.decay = ly.decay;
    a.heads = ly.c.heads; a.dim = ly.c.dim; a.vdim = ly.c.vdim; a.rows = n;
    return seq ? launch_lightning_seq(e->ctx, a, rows, m->act32) : launch_lightning_step(e->ctx, a, rows, m->act32);
}

static int mix_latent(prism_cuda_engine *e, LayeredLayer &ly, const RowMap &rows, uint32_t n, bool seq) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    const LatentArgs &la = ly.la;
    void *dq = at(m, m->proj, ly.in.seg[0].row0), *dkv = at(m, m->proj, ly.in.seg[1].row0), *gate = at(m, m->proj, ly.in.seg[2].row0);
    DenseIn qi{};
    qi.x = dq; qi.pitch = m->proj_pitch; qi.norm_w = ly.dq_norm; qi.n_norm = ly.c.q_rank; qi.eps = m->c.norm_eps;
    const DenseOut qo{m->q, m->q_pitch, ST_ACT};
    PRISM_TRY(linear(e, ly.uq, qi, &qo, n, m->cq, m->cq_pitch));
    if (seq && n > DENSE_GEMV_ROWS && ly.ukv.w) {
        const uint32_t pos0 = (uint32_t)rows.pos0, lo = la.window && pos0 + 1 > la.window ? pos0 + 1 - la.window : 0, nk = pos0 + n - lo;
        const uint32_t kv_pitch = ly.ukv.n_tiles * 128, v0 = ly.ukv.seg[1].row0;
        PRISM_TRY(launch_latent_append(ctx, la, dkv, m->proj_pitch, rows, n, false));
        PRISM_TRY(grow_bf16(e, m->ex_lat, m->ex_lat_n, (size_t)nk * ly.ukv.k_pad));
        PRISM_TRY(grow_bf16(e, m->ex_krot, m->ex_krot_n, (size_t)nk * la.rot_dim + 8));
        PRISM_TRY(grow_bf16(e, m->ex_kv, m->ex_kv_n, (size_t)nk * kv_pitch));
        PRISM_TRY(launch_latent_gather(ctx, la, rows.slot0, lo, nk, m->ex_lat, ly.ukv.k_pad, m->ex_krot));
        const DenseOut ko[2] = {{m->ex_kv, kv_pitch, ST_ACT}, {m->ex_kv + v0, kv_pitch, ST_ACT}};
        PRISM_TRY(launch_dense_gemm_tc5(ctx, ly.ukv, m->ex_lat, ly.ukv.k_pad, ko, nk));
        return launch_latent_prefill(ctx, la, (const bf16 *)m->q, m->q_pitch, m->ex_kv, kv_pitch, m->ex_kv + v0, kv_pitch, m->ex_krot, lo,
                                     (const bf16 *)gate, m->proj_pitch, (bf16 *)m->cat, m->cat_pitch, pos0, n);
    }
    LatentRowsScratch s = m->rows_scratch;
    s.splits = ly.splits;
    for (uint32_t r = 0; r < n; r += (uint32_t)s.rows_cap) {
        const uint32_t k = std::min<uint32_t>(n - r, (uint32_t)s.rows_cap);
        RowMap sub = rows;
        if (sub.slot) {
            sub.slot += r;
            sub.pos += r;
        } else {
            sub.pos0 += (int32_t)r;
        }
        PRISM_TRY(launch_latent_rows(ctx, la, s, at(m, m->q, (size_t)r * m->q_pitch), m->q_pitch, at(m, dkv, (size_t)r * m->proj_pitch),
                                     m->proj_pitch, at(m, gate, (size_t)r * m->proj_pitch), m->proj_pitch,
                                     at(m, m->cat, (size_t)r * m->cat_pitch), m->cat_pitch, sub, k, m->act32));
    }
    return PRISM_OK;
}

// `n` rows of m->x through every layer.
static int forward_layers(prism_cuda_engine *e, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    const uint32_t D = m->c.width;
    for (LayeredLayer &ly : m->layers) {
        DenseIn in{};
        in.x = m->x; in.pitch = D; in.f32 = 1; in.norm_w = ly.norm1; in.n_norm = D; in.eps = m->c.norm_eps;
        DenseOut outs[DENSE_MAX_SEGS];
        for (uint32_t s = 0; s < ly.in.n_segs; s++) outs[s] = DenseOut{at(m, m->proj, ly.in.seg[s].row0), m->proj_pitch, ST_ACT};
        if (ly.c.ff) outs[ly.seg_up] = DenseOut{at(m, m->cat, ly.k_mix), m->cat_pitch, ST_ACT};
        PRISM_TRY(linear(e, ly.in, in, outs, n, m->xn, m->width_pad));
        DenseIn oi{};
        oi.x = m->cat; oi.pitch = m->cat_pitch;
        if (ly.c.mixer == PRISM_MIXER_LIGHTNING) {
            PRISM_TRY(mix_lightning(e, ly, rows, n, seq));
            // all heads normed together, then gated
            oi.norm_w = ly.mix_norm; oi.n_norm = ly.c.heads * ly.c.vdim; oi.eps = m->c.norm_eps;
            oi.gate = at(m, m->proj, ly.in.seg[3].row0); oi.gate_pitch = m->proj_pitch;
        } else {
            PRISM_TRY(mix_latent(e, ly, rows, n, seq));
        }
        const DenseOut ro{m->x, D, ST_RESID};
        PRISM_TRY(linear(e, ly.out, oi, &ro, n, m->cat, m->cat_pitch));
    }
    return PRISM_OK;
}

// Logits of `n` fp32 residual rows into m->logits.
static int head_rows(prism_cuda_engine *e, const float *x, uint32_t n) {
    LayeredModel *m = e->lm;
    DenseIn in{};
    in.x = x; in.pitch = m->c.width; in.f32 = 1; in.norm_w = m->final_norm; in.n_norm = m->c.width; in.eps = m->c.norm_eps;
    const DenseOut o{m->logits, m->vocab_pad, ST_F32};
    return linear(e, m->head, in, &o, n, m->xn, m->width_pad);
}

int layered_enqueue_step(prism_cuda_engine *e) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    const uint32_t B = e->batch;
    RowMap rows;
    rows.slot = m->row_slot;
    rows.pos = m->row_pos;
    PRISM_TRY(launch_dense_embed(ctx, m->embed, m->c.width, m->c.vocab, e->tok, B, m->x));
    PRISM_TRY(forward_layers(e, rows, B, false));
    PRISM_TRY(head_rows(e, m->x, B));
    PRISM_TRY(launch_argmax(ctx, m->logits, m->c.vocab, m->vocab_pad, B, e->next));
    return enqueue_advance(e, m->row_pos);
}

// ---- rows and slots ---------------------------------------------------------------------------------------

static int upload_rows(prism_cuda_engine *e, const std::vector<int32_t> &slot, const std::vector<int32_t> &pos) {
    LayeredModel *m = e->lm;
    // pageable sources: copied before the calls return
    PRISM_CUDA_TRY(e->ctx, cudaMemcpyAsync(m->row_slot, slot.data(), slot.size() * 4, cudaMemcpyHostToDevice, e->ctx->stream));
    PRISM_CUDA_TRY(e->ctx, cudaMemcpyAsync(m->row_pos, pos.data(), pos.size() * 4, cudaMemcpyHostToDevice, e->ctx->stream));
    PRISM_CUDA_TRY(e->ctx, cudaStreamSynchronize(e->ctx->stream));
    return PRISM_OK;
}
int layered_set_rows(prism_cuda_engine *e, uint32_t pos) {
    std::vector<int32_t> s(e->batch), p(e->batch, (int32_t)pos);
    for (uint32_t b = 0; b < e->batch; b++) {
        if (e->lm->slot_pos[b] != (int64_t)pos)
            return fail(e->ctx, PRISM_E_STATE, "sequence " + std::to_string(b) + " is not where the batch is: reset() first, or use extend()");
        s[b] = (int32_t)b;
    }
    return upload_rows(e, s, p);
}
void layered_advance(prism_cuda_engine *e, uint32_t n) {
    for (uint32_t b = 0; b < e->batch; b++) e->lm->slot_pos[b] += n;
}

static int open_slot(prism_cuda_engine *e, uint32_t slot) {
    LayeredModel *m = e->lm;
    for (LayeredLayer &ly : m->layers)
        if (ly.state) {
            const size_t n = (size_t)ly.c.heads * ly.c.dim * ly.c.vdim;
            PRISM_CUDA_TRY(e->ctx, cudaMemsetAsync(ly.state + slot * n, 0, n * 4, e->ctx->stream));
        }
    m->slot_pos[slot] = 0;  // cached latents need no clearing: only positions below the slot's are ever read
    return PRISM_OK;
}
int layered_reset(prism_cuda_engine *e, uint32_t batch) {
    LayeredModel *m = e->lm;
    std::fill(m->slot_pos.begin(), m->slot_pos.end(), (int64_t)-1);
    for (uint32_t b = 0; b < batch; b++) PRISM_TRY(open_slot(e, b));
    return PRISM_OK;
}

// Prompt tokens of one slot, in chunks; after_chunk(first token, count) runs once a chunk's residual rows are in m->x.
template <typename F>
static int run_portion(prism_cuda_engine *e, uint32_t slot, const uint32_t *tokens, uint32_t n, F &&after_chunk) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    for (uint32_t t0 = 0; t0 < n; t0 += m->chunk) {
        const uint32_t k = std::min(m->chunk, n - t0);
        PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(m->pf_tok, tokens + t0, (size_t)k * 4, cudaMemcpyHostToDevice, ctx->stream));
        RowMap rows;
        rows.slot0 = (int32_t)slot;
        rows.pos0 = (int32_t)m->slot_pos[slot];
        PRISM_TRY(launch_dense_embed(ctx, m->embed, m->c.width, m->c.vocab, m->pf_tok, k, m->x));
        PRISM_TRY(forward_layers(e, rows, k, true));
        m->slot_pos[slot] += k;
        PRISM_TRY(after_chunk(t0, k));
    }
    return PRISM_OK;
}
int layered_prefill(prism_cuda_engine *e, uint32_t slot, const uint32_t *tokens, uint32_t n) {
    for (uint32_t i = 0; i < n; i++)
        if (tokens[i] >= e->lm->c.vocab) return fail(e->ctx, PRISM_E_ARG, "token id outside the vocabulary");
    return run_portion(e, slot, tokens, n, [](uint32_t, uint32_t) { return PRISM_OK; });
}

int layered_logits_f16(prism_cuda_engine *e, uint16_t *host) {
    LayeredModel *m = e->lm;
    prism_cuda_ctx *ctx = e->ctx;
    const size_t n = (size_t)e->batch * m->c.vocab;
    PRISM_TRY(ensure_stage(ctx, 0, n * 2));
    PRISM_TRY(launch_f32_to_f16(ctx, m->logits, e->batch, m->c.vocab, m->vocab_pad, reinterpret_cast<uint16_t *>(ctx->stage_out), m->c.vocab));
    PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(host, ctx->stage_out, n * 2, cudaMemcpyDeviceToHost, ctx->stream));
    return PRISM_OK;
}

uint64_t layered_step_bytes(const prism_cuda_engine *e) {
    const LayeredModel *m = e->lm;
    const uint64_t es = m->act32 ? 4 : 2, B = std::max(1u, e->batch), keys = e->pos + 1;
    uint64_t bytes = (uint64_t)m->c.vocab * m->c.width * 2;
    for (const LayeredLayer &ly : m->layers) {
        const uint64_t hv = (uint64_t)ly.c.heads * ly.c.vdim;
        bytes += (ly.in.valid_rows() * m->c.width + (hv + ly.c.ff) * m->c.width) * 2;
        if (ly.c.mixer == PRISM_MIXER_LIGHTNING) {
            bytes += B * 8 * (uint64_t)ly.c.heads * ly.c.dim * ly.c.vdim;  // state read and written
        } else {
            bytes += ly.uq.valid_rows() * ly.c.q_rank * 2 + ((uint64_t)ly.c.heads * ly.c.dim + hv) * ly.c.kv_rank * 2;
            const uint64_t seen = ly.c.window ? std::min<uint64_t>(keys, ly.c.window) : keys;
            bytes += B * seen * (ly.c.kv_rank + ly.c.rot_dim) * es;
        }
    }
    return bytes;
}

// Logits of rows `idx` (places in m->x) of a portion's chunk, row i to host row dst[i]; next_host: the greedy
// token of a single row instead.
static int logits_of(prism_cuda_engine *e, const uint32_t *idx, const uint32_t *dst, uint32_t n, float *host, uint32_t *next_host) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    for (uint32_t i = 0; i < n; i += m->lg_cap) {
        const uint32_t k = std::min(m->lg_cap, n - i);
        PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(m->want_idx, idx + i, (size_t)k * 4, cudaMemcpyHostToDevice, ctx->stream));
        PRISM_TRY(launch_gather_rows_f32(ctx, m->x, m->want_idx, k, m->c.width, m->xw));
        PRISM_TRY(head_rows(e, m->xw, k));
        for (uint32_t j = 0, run; host && j < k; j += run) {  // runs of consecutive host rows
            for (run = 1; j + run < k && dst[i + j + run] == dst[i + j] + run;) run++;
            PRISM_CUDA_TRY(ctx, cudaMemcpy2DAsync(host + (size_t)dst[i + j] * m->c.vocab, (size_t)m->c.vocab * 4, m->logits + (size_t)j * m->vocab_pad,
                                                  (size_t)m->vocab_pad * 4, (size_t)m->c.vocab * 4, run, cudaMemcpyDeviceToHost, ctx->stream));
        }
        if (next_host) {  // one row
            PRISM_TRY(launch_argmax(ctx, m->logits, m->c.vocab, m->vocab_pad, 1, e->next));
            PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(next_host, e->next, 4, cudaMemcpyDeviceToHost, ctx->stream));
        }
        PRISM_CUDA_TRY(ctx, cudaStreamSynchronize(ctx->stream));  // idx and the buffers are used again
    }
    return PRISM_OK;
}

}  // namespace prism

using namespace prism;

extern "C" {

int prism_cuda_engine_create_layered(prism_cuda_ctx *ctx, const prism_layered_config *cfg, const prism_layer_config *layers,
                                     prism_cuda_engine **out) {
    if (!ctx || !cfg || !layers || !out) return fail(ctx, PRISM_E_NULL, "null argument");
    *out = nullptr;
    const prism_layered_config &c = *cfg;
    if (!c.vocab || !c.width || !c.num_layers || !c.max_seq || !c.max_batch) return fail(ctx, PRISM_E_ARG, "model config has a zero dimension");
    if (c.dtype != PRISM_DTYPE_BF16 && c.dtype != PRISM_DTYPE_F32) return fail(ctx, PRISM_E_ARG, "dtype must be bf16 or f32");
    if (ctx->tp_world > 1 || ctx->tp_loopback) return fail(ctx, PRISM_E_STATE, "layered models run on one GPU");
    PRISM_CUDA_TRY(ctx, cudaSetDevice(ctx->device));
    prism_cuda_engine *e = new prism_cuda_engine();
    e->ctx = ctx;
    e->lm = new LayeredModel();
    e->lm->c = c;
    e->lm->act32 = c.dtype == PRISM_DTYPE_F32;
    e->lm->chunk = std::min(c.max_seq, (uint32_t)std::max(1, ctx->layered_chunk));
    // what the shared loop reads of the palettized configuration
    e->cfg.num_layers = c.num_layers; e->cfg.hidden_size = c.width; e->cfg.vocab_size = c.vocab; e->cfg.norm_eps = c.norm_eps;
    e->cfg.max_seq = c.max_seq; e->cfg.max_batch = c.max_batch;
    e->kv_slots = c.max_seq;
    e->out_cap = c.max_seq;
    e->batch = 1;
    int rc = engine_alloc_common(e, c.max_batch);
    if (rc == PRISM_OK) rc = build_model(e, layers);
    if (rc == PRISM_OK) rc = layered_reset(e, 0);
    if (rc == PRISM_OK && cudaStreamSynchronize(ctx->stream) != cudaSuccess) rc = fail(ctx, PRISM_E_CUDA, "model set-up failed");
    if (rc != PRISM_OK) {
        prism_cuda_engine_destroy(e);
        return rc;
    }
    *out = e;
    return PRISM_OK;
}

int prism_cuda_engine_set_tensor(prism_cuda_engine *e, const char *name, const uint16_t *data, uint64_t rows, uint64_t cols) {
    if (!e || !name || !data) return fail(e ? e->ctx : nullptr, PRISM_E_NULL, "null argument");
    prism_cuda_ctx *ctx = e->ctx;
    if (!e->lm) return fail(ctx, PRISM_E_STATE, "palettized models bind uploaded tensors");
    auto it = e->lm->names.find(name);
    if (it == e->lm->names.end()) return fail(ctx, PRISM_E_NOTFOUND, std::string("miss ") + name);
    LayeredDst &d = it->second;
    const bool vec = d.cols == 1 && rows * cols == d.rows && (rows == 1 || cols == 1);
    if (!vec && (rows != d.rows || cols != d.cols))
        return fail(ctx, PRISM_E_ARG, std::string("tensor ") + name + " is " + std::to_string(rows) + "x" + std::to_string(cols) + ", the model needs " +
                                          std::to_string(d.rows) + "x" + std::to_string(d.cols));
    PRISM_CUDA_TRY(ctx, cudaSetDevice(ctx->device));
    const size_t bytes = d.rows * d.cols * 2;
    PRISM_TRY(ensure_stage(ctx, bytes, 0));
    PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(ctx->stage_in, data, bytes, cudaMemcpyHostToDevice, ctx->stream));
    PRISM_TRY(place_tensor(e, d, reinterpret_cast<const bf16 *>(ctx->stage_in)));
    PRISM_CUDA_TRY(ctx, cudaStreamSynchronize(ctx->stream));
    return PRISM_OK;
}

int prism_cuda_engine_seq_open(prism_cuda_engine *e, uint32_t *seq) {
    if (!e || !seq) return fail(e ? e->ctx : nullptr, PRISM_E_NULL, "null argument");
    if (!e->lm) return fail(e->ctx, PRISM_E_STATE, "palettized models decode their batch in step: use reset()");
    PRISM_CUDA_TRY(e->ctx, cudaSetDevice(e->ctx->device));
    for (uint32_t s = 0; s < e->lm->slot_pos.size(); s++)
        if (e->lm->slot_pos[s] < 0) {
            *seq = s;
            return open_slot(e, s);
        }
    return fail(e->ctx, PRISM_E_STATE, "all " + std::to_string(e->lm->slot_pos.size()) + " sequences are in use");
}

static int open_seq(prism_cuda_engine *e, uint32_t seq) {
    if (!e->lm) return fail(e->ctx, PRISM_E_STATE, "palettized models have no sequence slots");
    if (seq >= e->lm->slot_pos.size() || e->lm->slot_pos[seq] < 0) return fail(e->ctx, PRISM_E_ARG, "sequence " + std::to_string(seq) + " is not open");
    return PRISM_OK;
}
int prism_cuda_engine_seq_close(prism_cuda_engine *e, uint32_t seq) {
    if (!e) return PRISM_E_NULL;
    PRISM_TRY(open_seq(e, seq));
    e->lm->slot_pos[seq] = -1;
    return PRISM_OK;
}
int prism_cuda_engine_seq_position(prism_cuda_engine *e, uint32_t seq, uint32_t *pos) {
    if (!e || !pos) return fail(e ? e->ctx : nullptr, PRISM_E_NULL, "null argument");
    PRISM_TRY(open_seq(e, seq));
    *pos = (uint32_t)e->lm->slot_pos[seq];
    return PRISM_OK;
}

int prism_cuda_engine_extend(prism_cuda_engine *e, uint32_t n, const uint32_t *seqs, const uint32_t *n_tokens, const uint32_t *tokens,
                             const uint32_t *n_want, const uint32_t *want, float *logits, uint32_t *next_tokens) {
    if (!e || !seqs || !n_tokens || !tokens) return fail(e ? e->ctx : nullptr, PRISM_E_NULL, "null argument");
    prism_cuda_ctx *ctx = e->ctx;
    if (!e->lm) return fail(ctx, PRISM_E_STATE, "palettized models decode their batch in step: use step() or generate()");
    LayeredModel *m = e->lm;
    PRISM_CUDA_TRY(ctx, cudaSetDevice(ctx->device));
    PRISM_TRY(layered_check_bound(e));
    // everything is checked before anything runs
    std::vector<size_t> tok0(n), want0(n);
    std::vector<bool> seen(m->slot_pos.size(), false);
    size_t nt = 0, nw = 0;
    for (uint32_t i = 0; i < n; i++) {
        PRISM_TRY(open_seq(e, seqs[i]));
        if (seen[seqs[i]]) return fail(ctx, PRISM_E_ARG, "a sequence appears twice in one step");
        seen[seqs[i]] = true;
        if (!n_tokens[i]) return fail(ctx, PRISM_E_ARG, "an entry without tokens");
        if (m->slot_pos[seqs[i]] + n_tokens[i] > m->c.max_seq) return fail(ctx, PRISM_E_STATE, "sequence " + std::to_string(seqs[i]) + " would exceed max_seq");
        tok0[i] = nt;
        want0[i] = nw;
        for (uint32_t t = 0; t < n_tokens[i]; t++)
            if (tokens[nt + t] >= m->c.vocab) return fail(ctx, PRISM_E_ARG, "token id outside the vocabulary");
        const uint32_t w = n_want ? n_want[i] : 0;
        for (uint32_t k = 0; k < w; k++)
            if (want[nw + k] >= n_tokens[i]) return fail(ctx, PRISM_E_ARG, "a wanted place lies outside the entry");
        nt += n_tokens[i];
        nw += w;
    }
    if (nw && !logits) return fail(ctx, PRISM_E_NULL, "null argument");
    // decode rows: one captured step for all entries of one token
    std::vector<uint32_t> one;
    for (uint32_t i = 0; i < n; i++)
        if (n_tokens[i] == 1) one.push_back(i);
    if (!one.empty()) {
        std::vector<int32_t> slot, pos;
        std::vector<uint32_t> tk, nx(one.size());
        for (uint32_t i : one) {
            slot.push_back((int32_t)seqs[i]);
            pos.push_back((int32_t)m->slot_pos[seqs[i]]);
            tk.push_back(tokens[tok0[i]]);
        }
        e->batch = (uint32_t)one.size();
        PRISM_TRY(upload_rows(e, slot, pos));
        PRISM_TRY(set_scalars(e, 0, 0, 0));
        PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(e->tok, tk.data(), tk.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
        PRISM_TRY(run_step(e));
        for (size_t r = 0; r < one.size(); r++) {
            const uint32_t i = one[r];
            m->slot_pos[seqs[i]] += 1;
            for (uint32_t k = 0; n_want && k < n_want[i]; k++)
                PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(logits + (want0[i] + k) * m->c.vocab, m->logits + r * m->vocab_pad, (size_t)m->c.vocab * 4,
                                                    cudaMemcpyDeviceToHost, ctx->stream));
        }
        PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(nx.data(), e->next, nx.size() * 4, cudaMemcpyDeviceToHost, ctx->stream));
        PRISM_CUDA_TRY(ctx, cudaStreamSynchronize(ctx->stream));
        if (next_tokens)
            for (size_t r = 0; r < one.size(); r++) next_tokens[one[r]] = nx[r];
    }
    for (uint32_t i = 0; i < n; i++) {
        if (n_tokens[i] == 1) continue;
        const uint32_t nwi = n_want ? n_want[i] : 0;
        const uint32_t *w = want + want0[i];
        PRISM_TRY(run_portion(e, seqs[i], tokens + tok0[i], n_tokens[i], [&](uint32_t t0, uint32_t k) -> int {
            std::vector<uint32_t> idx, dst;
            for (uint32_t j = 0; j < nwi; j++)
                if (w[j] >= t0 && w[j] < t0 + k) {
                    idx.push_back(w[j] - t0);
                    dst.push_back((uint32_t)want0[i] + j);
                }
            if (!idx.empty()) PRISM_TRY(logits_of(e, idx.data(), dst.data(), (uint32_t)idx.size(), logits, nullptr));
            if (next_tokens && t0 + k == n_tokens[i]) {
                const uint32_t last = k - 1;
                PRISM_TRY(logits_of(e, &last, nullptr, 1, nullptr, next_tokens + i));
            }
            return PRISM_OK;
        }));
    }
    return check_device_error(ctx);
}

}  // extern "C"
