// Models described layer by layer on the engine's shared loop, in one of two arrangements.
//
// Parallel: per layer one norm whose output both sublayers read, a mixer and a dense feed-forward.
//   in   one stacked linear for everything that reads the normed input, the norm folded into its input
//        staging for small batches
//   mix  the mixer, leaving its gated heads beside the feed-forward activations
//   out  one linear over [heads | activations] that adds both sublayers into the fp32 residual
//
// Sequential: mixer, then feed-forward, each with its norm, and optionally an input convolution, a gate on its
// result and a weighted sum over the depth; everything between two linears is one row-wise kernel.
//   in   one stacked linear: projections from the convolved norm, the gate from the norm itself
//   mix  one mixer or a pair, each leaving its heads in its own columns
//   out  their output linears; in2, experts or dense feed-forward
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

static uint32_t add_seg(DenseLinear &l, uint32_t rows, uint32_t act, uint32_t in = 0, uint32_t k = 0) {
    if (l.n_segs && (l.seg[l.n_segs - 1].in != in || l.seg[l.n_segs - 1].k != k)) l.n_tiles += l.n_tiles & 1;
    DenseSeg &s = l.seg[l.n_segs];
    s.row0 = l.n_tiles * 128;
    s.rows = rows;
    s.act = act;
    s.in = in;
    s.k = k;
    l.n_tiles += (rows + 127) / 128;
    return l.n_segs++;  // at most 11: a pair of mixers takes at most ten
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
static void name_packed(LayeredModel *m, const std::string &name, uint32_t rows, uint32_t cols, DenseLinear &l, uint32_t seg, uint32_t k0 = 0, uint32_t row = 0) {
    LayeredDst &d = add_name(m, name, rows, cols);
    d.lin = &l;
    d.row0 = l.seg[seg].row0 + row;
    d.k0 = k0;
}
static int name_vector(prism_cuda_engine *e, const std::string &name, uint32_t n, float *&vec, float mean, float add = 0.0f) {
    PRISM_TRY(model_alloc(e, vec, n));
    LayeredDst &d = add_name(e->lm, name, n, 1);
    d.vec = vec;
    d.vec_pitch = n;
    d.mean = mean;
    d.add = add;
    return PRISM_OK;
}
// [channels][taps] of a convolution, kept as [taps][pitch]
static void name_conv(LayeredModel *m, const std::string &name, uint32_t channels, uint32_t taps, float *vec, uint32_t pitch) {
    LayeredDst &d = add_name(m, name, channels, taps);
    d.vec = vec;
    d.vec_pitch = pitch;
    d.mean = 0.2f;
}

// A tensor that a checkpoint may carry although no sublayer reads it.
static void name_unused(LayeredModel *m, const std::string &name, uint64_t rows, uint64_t cols) {
    LayeredDst &d = m->names[name];
    d.rows = rows;
    d.cols = cols;
    d.bound = true;
}

static uint32_t ring_size(const LayeredModel *m, uint32_t window) {
    return window ? (uint32_t)std::min<uint64_t>(m->c.max_seq, (uint64_t)window - 1 + m->chunk) : m->c.max_seq;
}

// Segments, names, small weights, caches and state of a mixer.
static int build_mixer(prism_cuda_engine *e, LayeredLayer &ly, LayeredMixer &mx, const prism_layer_config &c, const std::string &p, const std::string &bad) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    mx.c = c;
    mx.c.decay = mx.c.rot_freq = nullptr;
    mx.c.left = mx.c.right = nullptr;
    mx.name = p;
    const uint32_t D = m->c.width, slots = m->c.max_batch, hv = c.heads * c.vdim;
    const size_t es = m->act32 ? 4 : 2;
    if (!c.heads || !c.dim || !c.vdim) return fail(ctx, PRISM_E_ARG, bad + "a mixer size is zero");
    mx.seg0 = ly.in.n_segs;
    auto seg = [&](const char *name, uint32_t rows, uint32_t act) { name_packed(m, p + name, rows, D, ly.in, add_seg(ly.in, rows, act)); };
    if (c.mixer == PRISM_MIXER_LIGHTNING) {
        if (!c.decay) return fail(ctx, PRISM_E_ARG, bad + "no decays");
        const uint32_t hk = c.heads * c.dim;
        seg("q", hk, ACT_SILU);
        seg("k", hk, ACT_SILU);
        seg("v", hv, ACT_SILU);
        seg("g", hv, ACT_SIGMOID);
        PRISM_TRY(name_vector(e, p + "norm", hv, mx.mix_norm, 1.0f));
        PRISM_TRY(model_alloc(e, mx.decay, c.heads));
        PRISM_CUDA_TRY(ctx, cudaMemcpyAsync(mx.decay, c.decay, c.heads * 4, cudaMemcpyHostToDevice, ctx->stream));
        PRISM_TRY(model_alloc(e, mx.state, (size_t)slots * c.heads * c.dim * c.vdim));
    } else if (c.mixer == PRISM_MIXER_LATENT_ATTENTION) {
        if (!c.q_rank || !c.kv_rank || 2 * c.rot_pairs > c.rot_dim || (c.rot_pairs && !c.rot_freq))
            return fail(ctx, PRISM_E_ARG, bad + "latent attention needs q_rank, kv_rank and rotation pairs inside rot_dim");
        seg("dq", c.q_rank, ACT_NONE);
        seg("dkv", c.kv_rank + c.rot_dim, ACT_NONE);
        seg("g", hv, ACT_SIGMOID);
        PRISM_TRY(name_vector(e, p + "dq.norm", c.q_rank, mx.dq_norm, 1.0f));
        float *dkv_norm = nullptr;
        PRISM_TRY(name_vector(e, p + "dkv.norm", c.kv_rank, dkv_norm, 1.0f));
        const uint32_t hq = c.heads * (c.dim + c.rot_dim);
        add_seg(mx.uq, hq, ACT_NONE);
        PRISM_TRY(finish_linear(e, mx.uq, round_up_u32(c.q_rank, 64)));
        name_packed(m, p + "uq", hq, c.q_rank, mx.uq, 0);
        LatentArgs &la = mx.la;
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
        const uint32_t suk = add_seg(mx.ukv, c.heads * c.dim, ACT_NONE), suv = add_seg(mx.ukv, hv, ACT_NONE);
        if (expand) PRISM_TRY(finish_linear(e, mx.ukv, round_up_u32(c.kv_rank, 64)));
        for (int j = 0; j < 2; j++) {
            LayeredDst &d = add_name(m, p + (j ? "uv" : "uk"), j ? hv : c.heads * c.dim, c.kv_rank);
            d.rowmajor = j ? uv : uk;
            d.pitch = la.uk_pitch;
            if (expand) {
                d.lin = &mx.ukv;
                d.row0 = mx.ukv.seg[j ? suv : suk].row0;
            }
        }
        la.cache.pitch = round_up_u32(c.kv_rank + c.rot_dim, 16);
        la.cache.ring = ring_size(m, c.window);
        PRISM_TRY(model_alloc(e, &la.cache.rows, (size_t)slots * la.cache.ring * la.cache.pitch * es));
        mx.splits = latent_rows_splits(la, m->c.max_seq);
        m->q_pitch = std::max(m->q_pitch, mx.uq.n_tiles * 128);
        m->cq_pitch = std::max(m->cq_pitch, mx.uq.k_pad);
    } else if (c.mixer == PRISM_MIXER_ATTENTION) {
        if (!c.kv_heads || c.heads % c.kv_heads) return fail(ctx, PRISM_E_ARG, bad + "attention: kv_heads must divide heads");
        seg("q", c.heads * c.dim, ACT_NONE);
        seg("k", c.kv_heads * c.dim, ACT_NONE);
        seg("v", c.kv_heads * c.vdim, ACT_NONE);
        GroupedArgs &ga = mx.ga;
        ga.heads = c.heads; ga.kv_heads = c.kv_heads; ga.dim = c.dim; ga.vdim = c.vdim; ga.window = c.window; ga.scale = c.scale;
        ga.dp = round_up_u32(c.dim, 8); ga.vp = round_up_u32(c.vdim, 8);
        ga.ring = ring_size(m, c.window);
        ga.splits = grouped_splits(ga, m->c.max_seq);
        PRISM_TRY(model_alloc(e, &ga.kc, (size_t)slots * ga.ring * c.kv_heads * ga.dp * es));
        PRISM_TRY(model_alloc(e, &ga.vc, (size_t)slots * ga.ring * c.kv_heads * ga.vp * es));
    } else if (c.mixer == PRISM_MIXER_GATED_DELTA) {
        if (!c.kv_heads || c.heads % c.kv_heads || !c.conv) return fail(ctx, PRISM_E_ARG, bad + "gated delta: kv_heads must divide heads, and a convolution has taps");
        const uint32_t hk = c.kv_heads * c.dim, C = 2 * hk + hv;
        seg("q", hk, ACT_NONE);
        seg("k", hk, ACT_NONE);
        seg("v", hv, ACT_NONE);
        const uint32_t sba = add_seg(ly.in, 2 * c.heads, ACT_NONE);
        name_packed(m, p + "b", c.heads, D, ly.in, sba);
        name_packed(m, p + "a", c.heads, D, ly.in, sba, 0, c.heads);
        seg("g", hv, ACT_SILU);
        DeltaArgs &da = mx.da;
        da.heads = c.heads; da.kv_heads = c.kv_heads; da.dim = c.dim; da.vdim = c.vdim; da.taps = c.conv; da.eps = m->c.norm_eps; da.channels = C;
        float *w = nullptr, *v = nullptr;
        PRISM_TRY(model_alloc(e, w, (size_t)c.conv * C));
        name_conv(m, p + "q.conv", hk, c.conv, w, C);
        name_conv(m, p + "k.conv", hk, c.conv, w + hk, C);
        name_conv(m, p + "v.conv", hv, c.conv, w + 2 * hk, C);
        da.conv_w = w;
        PRISM_TRY(name_vector(e, p + "A_log", c.heads, v, 0.0f));
        da.a_log = v;
        PRISM_TRY(name_vector(e, p + "dt_bias", c.heads, v, 0.0f));
        da.dt_bias = v;
        PRISM_TRY(name_vector(e, p + "norm", c.vdim, v, 1.0f));
        da.norm = v;
        PRISM_TRY(model_alloc(e, &da.ring, (size_t)slots * c.conv * C * es));
        PRISM_TRY(model_alloc(e, da.state, (size_t)slots * c.heads * c.dim * c.vdim));
        for (int i = 0; i < 3; i++) mx.conv_col[i] = i ? mx.conv_col[i - 1] + round_up_u32(hk, 8) : 0;
        m->conv_pitch = std::max(m->conv_pitch, mx.conv_col[2] + round_up_u32(hv, 8));
        m->o32_width = std::max(m->o32_width, hv);
        m->aux_pitch = std::max(m->aux_pitch, round_up_u32(2 * c.heads, 4));
    } else {
        return fail(ctx, PRISM_E_ARG, bad + "unknown mixer");
    }
    return PRISM_OK;
}

static int build_parallel_layer(prism_cuda_engine *e, LayeredLayer &ly, const std::string &p, const std::string &bad) {
    LayeredModel *m = e->lm;
    const uint32_t D = m->c.width, ff = ly.c.ff, hv = ly.mix[0].width();
    if (ly.mix.size() != 1 || ly.c.experts) return fail(e->ctx, PRISM_E_ARG, bad + "pairs of mixers and experts need the sequential arrangement");
    ly.k_mix = round_up_u32(hv, 64);
    if (ff) {
        ly.seg_up = add_seg(ly.in, ff, ACT_GELU_TANH);
        name_packed(m, p + "mlp.up", ff, D, ly.in, ly.seg_up);
        PRISM_TRY(name_vector(e, p + "mlp.up.b", ff, ly.up_b, 0.0f));
        ly.in.seg[ly.seg_up].bias = ly.up_b;
    }
    PRISM_TRY(finish_linear(e, ly.in, m->width_pad));
    add_seg(ly.out, D, ACT_NONE);
    ly.out.seg[0].mul = m->c.residual_mult;
    PRISM_TRY(finish_linear(e, ly.out, ly.k_mix + round_up_u32(ff, 64)));
    name_packed(m, ly.mix[0].name + "o", D, hv, ly.out, 0);
    if (ff) {
        name_packed(m, p + "mlp.down", D, ff, ly.out, 0, ly.k_mix);
        PRISM_TRY(name_vector(e, p + "mlp.down.b", D, ly.down_b, 0.0f));
        ly.out.seg[0].bias = ly.down_b;
    }
    m->cat_pitch = std::max(m->cat_pitch, ly.out.k_pad);
    return PRISM_OK;
}

// Gate and input convolution of sublayer `n` ("1", "2"); `in`: the linear the gate is a segment of.
static int build_sublayer(prism_cuda_engine *e, const std::string &p, const char *n, DenseLinear &in, uint32_t &seg_gate, float *&gate_b, float *&canon,
                          void *&ring) {
    LayeredModel *m = e->lm;
    const uint32_t D = m->c.width, taps = m->c.canon_taps;
    if (m->c.gated_residual) {
        seg_gate = add_seg(in, D, ACT_SIGMOID, taps ? 1 : 0);  // from the norm before its convolution
        name_packed(m, p + "rg" + n, D, D, in, seg_gate);
        PRISM_TRY(name_vector(e, p + "rg" + n + ".b", D, gate_b, 0.0f));
        in.seg[seg_gate].bias = gate_b;
    }
    if (taps) {
        PRISM_TRY(model_alloc(e, canon, (size_t)taps * D));
        name_conv(m, p + "canon" + n, D, taps, canon, D);
        PRISM_TRY(model_alloc(e, &ring, (size_t)m->c.max_batch * taps * D * (m->act32 ? 4 : 2)));
    }
    return finish_linear(e, in, m->width_pad);
}

static int build_sequential_layer(prism_cuda_engine *e, LayeredLayer &ly, uint32_t i, const std::string &p, const std::string &bad) {
    LayeredModel *m = e->lm;
    const prism_layer_config &c = ly.c;
    const uint32_t D = m->c.width;
    PRISM_TRY(build_sublayer(e, p, "1", ly.in, ly.seg_gate1, ly.gate1_b, ly.canon1, ly.ring1));
    uint32_t col = 0, k_max = 0;
    for (size_t j = 0; j < ly.mix.size(); j++) {
        LayeredMixer &mx = ly.mix[j];
        const uint32_t k = round_up_u32(mx.width(), 64);
        mx.col = col;
        col += k;
        k_max = std::max(k_max, k);
        add_seg(ly.out, D, ACT_NONE, (uint32_t)j, k);
    }
    PRISM_TRY(finish_linear(e, ly.out, k_max));
    for (size_t j = 0; j < ly.mix.size(); j++) {
        LayeredMixer &mx = ly.mix[j];
        name_packed(m, mx.name + "o", D, mx.width(), ly.out, (uint32_t)j);
        if (ly.mix.size() > 1) PRISM_TRY(name_vector(e, mx.name + "out", D, mx.out_norm, 1.0f));
    }
    m->cat_pitch = std::max(m->cat_pitch, col);
    if (c.ff) {
        PRISM_TRY(name_vector(e, p + "norm2", D, ly.norm2, 1.0f - m->c.norm_offset, m->c.norm_offset));
        if (c.experts) {
            const uint32_t groups = std::max(1u, c.expert_groups), keep = c.groups_keep ? c.groups_keep : groups;
            if (!c.top || c.experts % groups || keep > groups || c.top > c.experts / groups * keep)
                return fail(e->ctx, PRISM_E_ARG, bad + "experts: the groups must be equal and those kept hold at least `top` experts");
            ly.c.expert_groups = groups;
            ly.c.groups_keep = keep;
            ly.seg_up = add_seg(ly.in2, c.experts, ACT_NONE);
            name_packed(m, p + "mlp.router", c.experts, D, ly.in2, ly.seg_up);
            PRISM_TRY(name_vector(e, p + "mlp.correction", c.experts, ly.correction, 0.0f));
            add_seg(ly.up, c.ff, ACT_RELU2);
            add_seg(ly.down, D, ACT_NONE);
            ly.up.experts = ly.down.experts = c.experts;
            PRISM_TRY(finish_linear(e, ly.up, m->width_pad));
            PRISM_TRY(finish_linear(e, ly.down, round_up_u32(c.ff, 64)));
            for (uint32_t x = 0; x < c.experts; x++) {
                const std::string q = p + "mlp.e" + std::to_string(x);
                name_packed(m, q + ".up", c.ff, D, ly.up, 0, 0, x * ly.up.n_tiles * 128);
                name_packed(m, q + ".down", D, c.ff, ly.down, 0, 0, x * ly.down.n_tiles * 128);
            }
            m->aux_pitch = std::max(m->aux_pitch, round_up_u32(c.experts, 4));
            m->pairs_cap = std::max(m->pairs_cap, (size_t)m->cap * c.top);
            m->plan.experts = std::max(m->plan.experts, c.experts);
            m->plan.top = std::max(m->plan.top, c.top);
        } else {
            ly.seg_up = add_seg(ly.in2, c.ff, ACT_GELU_TANH);
            name_packed(m, p + "mlp.up", c.ff, D, ly.in2, ly.seg_up);
            PRISM_TRY(name_vector(e, p + "mlp.up.b", c.ff, ly.up_b, 0.0f));
            ly.in2.seg[ly.seg_up].bias = ly.up_b;
            add_seg(ly.down, D, ACT_NONE);
            PRISM_TRY(finish_linear(e, ly.down, round_up_u32(c.ff, 64)));
            name_packed(m, p + "mlp.down", D, c.ff, ly.down, 0);
            PRISM_TRY(name_vector(e, p + "mlp.down.b", D, ly.down_b, 0.0f));
            ly.down.seg[0].bias = ly.down_b;
        }
        m->act_pitch = std::max(m->act_pitch, ly.down.k_pad);
        PRISM_TRY(build_sublayer(e, p, "2", ly.in2, ly.seg_gate2, ly.gate2_b, ly.canon2, ly.ring2));
        m->proj_pitch = std::max(m->proj_pitch, ly.in2.n_tiles * 128);
    } else {
        name_unused(m, p + "norm2", D, 1);
        if (m->c.canon_taps) name_unused(m, p + "canon2", D, m->c.canon_taps);
        if (m->c.gated_residual) {
            name_unused(m, p + "rg2", D, D);
            name_unused(m, p + "rg2.b", D, 1);
        }
    }
    if (m->c.depth_average) PRISM_TRY(name_vector(e, p + "dwa", i + 2, ly.avg, 0.5f));
    return PRISM_OK;
}

static int build_layer(prism_cuda_engine *e, uint32_t i, const prism_layer_config &c) {
    LayeredModel *m = e->lm;
    LayeredLayer &ly = m->layers[i];
    ly.c = c;
    ly.c.decay = ly.c.rot_freq = nullptr;
    ly.c.left = ly.c.right = nullptr;
    const std::string p = "l" + std::to_string(i) + ".", bad = "layer " + std::to_string(i) + ": ";
    PRISM_TRY(name_vector(e, p + "norm1", m->c.width, ly.norm1, 1.0f - m->c.norm_offset, m->c.norm_offset));
    if (c.mixer == PRISM_MIXER_PAIR) {
        if (!c.left || !c.right) return fail(e->ctx, PRISM_E_ARG, bad + "a pair needs two mixers");
        ly.mix.resize(2);  // never resized again: names point into it
        PRISM_TRY(build_mixer(e, ly, ly.mix[0], *c.left, p + "mix.left.", bad));
        PRISM_TRY(build_mixer(e, ly, ly.mix[1], *c.right, p + "mix.right.", bad));
    } else {
        ly.mix.resize(1);
        PRISM_TRY(build_mixer(e, ly, ly.mix[0], c, p + "mix.", bad));
    }
    PRISM_TRY(m->c.arrangement == PRISM_ARRANGE_SEQUENTIAL ? build_sequential_layer(e, ly, i, p, bad) : build_parallel_layer(e, ly, p, bad));
    m->proj_pitch = std::max(m->proj_pitch, ly.in.n_tiles * 128);
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
    if (c.max_positions) {
        PRISM_TRY(model_alloc(e, m->pos, (size_t)c.max_positions * c.width));
        LayeredDst &ps = add_name(m, "pos", c.max_positions, c.width);
        ps.rowmajor = m->pos;
        ps.pitch = c.width;
    }
    for (uint32_t i = 0; i < c.num_layers; i++) PRISM_TRY(build_layer(e, i, layers[i]));
    PRISM_TRY(name_vector(e, "final.norm", c.width, m->final_norm, 1.0f - c.norm_offset, c.norm_offset));
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
    size_t delta = 0;
    for (const LayeredLayer &ly : m->layers)
        for (const LayeredMixer &mx : ly.mix)
            if (mx.c.mixer == PRISM_MIXER_LATENT_ATTENTION) {
                size_t q1, p1, m1;
                latent_rows_scratch_floats(mx.la, mx.splits, &q1, &p1, &m1);
                qa = std::max(qa, q1);
                part = std::max(part, p1);
                ml = std::max(ml, m1);
            } else if (mx.c.mixer == PRISM_MIXER_GATED_DELTA) {
                delta = std::max(delta, delta_scratch_bytes(mx.da, m->cap));
            }
    if (delta) {
        PRISM_TRY(model_alloc(e, &m->conv, (size_t)m->cap * m->conv_pitch * es));
        PRISM_TRY(model_alloc(e, m->o32, (size_t)m->cap * m->o32_width));
        if (!m->act32) PRISM_TRY(model_alloc(e, &m->delta, delta));
    }
    if (m->aux_pitch) PRISM_TRY(model_alloc(e, m->aux, (size_t)m->cap * m->aux_pitch));
    if (c.arrangement == PRISM_ARRANGE_SEQUENTIAL) {
        m->y_pitch = round_up_u32(c.width, 8);
        if (c.canon_taps) PRISM_TRY(model_alloc(e, &m->xc, (size_t)m->cap * m->width_pad * es));
        PRISM_TRY(model_alloc(e, &m->y, std::max((size_t)2 * m->cap, m->pairs_cap) * m->y_pitch * es));
        if (m->act_pitch) PRISM_TRY(model_alloc(e, &m->act, std::max((size_t)m->cap, m->pairs_cap) * m->act_pitch * es));
        if (c.depth_average) PRISM_TRY(model_alloc(e, m->history, (size_t)(c.num_layers + 1) * m->cap * c.width));
    }
    if (m->pairs_cap) {
        MoePlan &pl = m->plan;
        PRISM_TRY(model_alloc(e, &m->moe_x, m->pairs_cap * m->width_pad * es));
        PRISM_TRY(model_alloc(e, pl.idx, m->pairs_cap));
        PRISM_TRY(model_alloc(e, pl.wgt, m->pairs_cap));
        PRISM_TRY(model_alloc(e, pl.order, m->pairs_cap));
        PRISM_TRY(model_alloc(e, pl.inv, m->pairs_cap));
        PRISM_TRY(model_alloc(e, pl.count, pl.experts));
        PRISM_TRY(model_alloc(e, pl.n_active, 1));
        PRISM_TRY(model_alloc(e, pl.active, DENSE_GEMV_ROWS * pl.top));
        PRISM_TRY(model_alloc(e, pl.pair_of, DENSE_GEMV_ROWS * DENSE_GEMV_ROWS * pl.top));
    }
    if (qa) {
        m->rows_scratch.rows_cap = std::max(c.max_batch, DENSE_GEMV_ROWS);
        PRISM_TRY(model_alloc(e, m->rows_scratch.qa, qa * m->rows_scratch.rows_cap));
        PRISM_TRY(model_alloc(e, m->rows_scratch.part, part * m->rows_scratch.rows_cap));
        PRISM_TRY(model_alloc(e, m->rows_scratch.ml, ml * m->rows_scratch.rows_cap));
    }
    m->slot_pos.assign(c.max_batch, -1);
    PRISM_CUDA_TRY(e->ctx, cudaStreamCreateWithFlags(&m->side, cudaStreamNonBlocking));
    PRISM_CUDA_TRY(e->ctx, cudaEventCreateWithFlags(&m->fork, cudaEventDisableTiming));
    PRISM_CUDA_TRY(e->ctx, cudaEventCreateWithFlags(&m->join, cudaEventDisableTiming));
    return PRISM_OK;
}

void layered_destroy(prism_cuda_engine *e) {
    LayeredModel *m = e->lm;
    for (void *p : m->allocs) cudaFree(p);
    cudaFree(m->ex_lat);
    cudaFree(m->ex_krot);
    cudaFree(m->ex_kv);
    if (m->fork) cudaEventDestroy(m->fork);
    if (m->join) cudaEventDestroy(m->join);
    if (m->side) cudaStreamDestroy(m->side);
    delete m;
    e->lm = nullptr;
}

// ---- weights -------------------------------------------------------------------------------------------

static int place_tensor(prism_cuda_engine *e, LayeredDst &d, const bf16 *src_dev) {
    prism_cuda_ctx *ctx = e->ctx;
    if (d.lin) PRISM_TRY(launch_dense_pack(ctx, *d.lin, src_dev, (uint32_t)d.rows, (uint32_t)d.cols, d.row0, d.k0));
    if (d.rowmajor) PRISM_TRY(launch_bf16_pitch_copy(ctx, src_dev, d.rowmajor, (uint32_t)d.rows, (uint32_t)d.cols, d.pitch));
    if (d.vec) PRISM_TRY(launch_bf16_to_f32(ctx, src_dev, d.vec, d.rows * d.cols, d.add, (uint32_t)d.cols, d.vec_pitch));
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
        PRISM_TRY(launch_dense_synth(e->ctx, tmp, d.rows * d.cols, seed * 1000003ull + id++, d.mean, sigma));
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
    }
    DenseIn plain{};
    plain.x = x; plain.pitch = pitch; plain.x2 = in.x2; plain.pitch2 = in.pitch2;
    if (m->act32) return launch_dense_f32(ctx, l, plain, outs, rows);
    if (ctx->fuse && dense_gemv_ok(plain, rows)) return launch_dense_gemv(ctx, l, plain, outs, rows);
    return launch_dense_gemm_tc5(ctx, l, plain, outs, rows);
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

// The mixers leave their heads in the rows of `cat`, from column mx.col on.
static int mix_lightning(prism_cuda_engine *e, LayeredLayer &ly, LayeredMixer &mx, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    const DenseSeg *seg = ly.in.seg + mx.seg0;
    LightningArgs a{};
    a.q = at(m, m->proj, seg[0].row0);
    a.k = at(m, m->proj, seg[1].row0);
    a.v = at(m, m->proj, seg[2].row0);
    a.pitch = m->proj_pitch;
    a.o = at(m, m->cat, mx.col);
    a.o_pitch = m->cat_pitch;
    a.state = mx.state;
    a.decay = mx.decay;
    a.heads = mx.c.heads; a.dim = mx.c.dim; a.vdim = mx.c.vdim; a.rows = n;
    return seq ? launch_lightning_seq(e->ctx, a, rows, m->act32) : launch_lightning_step(e->ctx, a, rows, m->act32);
}

static int mix_attention(prism_cuda_engine *e, LayeredLayer &ly, LayeredMixer &mx, const RowMap &rows, uint32_t n, bool seq, bool late) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    const DenseSeg *seg = ly.in.seg + mx.seg0;
    const void *q = at(m, m->proj, seg[0].row0), *k = at(m, m->proj, seg[1].row0), *v = at(m, m->proj, seg[2].row0);
    void *out = at(m, m->cat, mx.col);
    if (!seq) return launch_grouped_rows(ctx, mx.ga, q, k, v, m->proj_pitch, out, m->cat_pitch, rows, n, m->act32, late);
    PRISM_TRY(launch_grouped_append(ctx, mx.ga, k, v, m->proj_pitch, rows, n, m->act32));
    if (!m->act32 && n > DENSE_GEMV_ROWS && tiled_attn_ok(mx.ga.dp, mx.ga.vp))
        return launch_grouped_prefill(ctx, mx.ga, (const bf16 *)q, m->proj_pitch, (bf16 *)out, m->cat_pitch, rows, n);
    return launch_grouped_rows(ctx, mx.ga, q, nullptr, nullptr, m->proj_pitch, out, m->cat_pitch, rows, n, m->act32);
}

static int mix_delta(prism_cuda_engine *e, LayeredLayer &ly, LayeredMixer &mx, const RowMap &rows, uint32_t n, bool seq, bool beside) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    const DenseSeg *seg = ly.in.seg + mx.seg0;
    DeltaArgs a = mx.da;
    a.rows = n;
    a.q = at(m, m->proj, seg[0].row0); a.k = at(m, m->proj, seg[1].row0); a.v = at(m, m->proj, seg[2].row0); a.pitch = m->proj_pitch;
    a.ba = m->aux; a.ba_pitch = m->aux_pitch;
    a.gate = at(m, m->proj, seg[4].row0); a.gate_pitch = m->proj_pitch;
    a.o = at(m, m->cat, mx.col); a.o_pitch = m->cat_pitch;
    a.beside = beside;
    if (!seq) return launch_delta_step(ctx, a, rows, m->act32);
    const uint32_t hk = a.kv_heads * a.dim;
    ConvArgs c{};
    c.pieces = 3; c.x_pitch = m->proj_pitch; c.y_pitch = m->conv_pitch; c.taps = a.taps; c.channels = a.channels; c.w = a.conv_w; c.ring = a.ring; c.silu = 1;
    c.piece[0] = ConvPiece{a.q, at(m, m->conv, mx.conv_col[0]), hk, 0};
    c.piece[1] = ConvPiece{a.k, at(m, m->conv, mx.conv_col[1]), hk, hk};
    c.piece[2] = ConvPiece{a.v, at(m, m->conv, mx.conv_col[2]), a.heads * a.vdim, 2 * hk};
    PRISM_TRY(launch_conv_seq(ctx, c, rows, n, m->act32));
    a.q = c.piece[0].y; a.k = c.piece[1].y; a.v = c.piece[2].y; a.pitch = m->conv_pitch;
    a.o32 = m->o32; a.chunk_scratch = m->delta;
    return launch_delta_seq(ctx, a, rows, m->act32);
}

static int mix_latent(prism_cuda_engine *e, LayeredLayer &ly, LayeredMixer &mx, const RowMap &rows, uint32_t n, bool seq) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    const LatentArgs &la = mx.la;
    const DenseSeg *seg = ly.in.seg + mx.seg0;
    void *dq = at(m, m->proj, seg[0].row0), *dkv = at(m, m->proj, seg[1].row0), *gate = at(m, m->proj, seg[2].row0), *out = at(m, m->cat, mx.col);
    DenseIn qi{};
    qi.x = dq; qi.pitch = m->proj_pitch; qi.norm_w = mx.dq_norm; qi.n_norm = mx.c.q_rank; qi.eps = m->c.norm_eps;
    const DenseOut qo{m->q, m->q_pitch, ST_ACT};
    PRISM_TRY(linear(e, mx.uq, qi, &qo, n, m->cq, m->cq_pitch));
    if (seq && n > DENSE_GEMV_ROWS && mx.ukv.w) {
        const uint32_t pos0 = (uint32_t)rows.pos0, lo = la.window && pos0 + 1 > la.window ? pos0 + 1 - la.window : 0, nk = pos0 + n - lo;
        const uint32_t kv_pitch = mx.ukv.n_tiles * 128, v0 = mx.ukv.seg[1].row0;
        PRISM_TRY(launch_latent_append(ctx, la, dkv, m->proj_pitch, rows, n, false));
        PRISM_TRY(grow_bf16(e, m->ex_lat, m->ex_lat_n, (size_t)nk * mx.ukv.k_pad));
        PRISM_TRY(grow_bf16(e, m->ex_krot, m->ex_krot_n, (size_t)nk * la.rot_dim + 8));
        PRISM_TRY(grow_bf16(e, m->ex_kv, m->ex_kv_n, (size_t)nk * kv_pitch));
        PRISM_TRY(launch_latent_gather(ctx, la, rows.slot0, lo, nk, m->ex_lat, mx.ukv.k_pad, m->ex_krot));
        const DenseOut ko[2] = {{m->ex_kv, kv_pitch, ST_ACT}, {m->ex_kv + v0, kv_pitch, ST_ACT}};
        DenseIn ki{};
        ki.x = m->ex_lat; ki.pitch = mx.ukv.k_pad;
        PRISM_TRY(launch_dense_gemm_tc5(ctx, mx.ukv, ki, ko, nk));
        return launch_latent_prefill(ctx, la, (const bf16 *)m->q, m->q_pitch, m->ex_kv, kv_pitch, m->ex_kv + v0, kv_pitch, m->ex_krot, lo,
                                     (const bf16 *)gate, m->proj_pitch, (bf16 *)out, m->cat_pitch, pos0, n);
    }
    LatentRowsScratch s = m->rows_scratch;
    s.splits = mx.splits;
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
                                     at(m, out, (size_t)r * m->cat_pitch), m->cat_pitch, sub, k, m->act32));
    }
    return PRISM_OK;
}

// In a decode step the two kernels of an attention and a gated delta rule run side by side: neither needs the other.
static int run_mixer(prism_cuda_engine *e, LayeredLayer &ly, LayeredMixer &mx, const RowMap &rows, uint32_t n, bool seq) {
    const bool side = !seq && ly.mix.size() == 2 && ly.mix[0].c.mixer == PRISM_MIXER_ATTENTION && ly.mix[1].c.mixer == PRISM_MIXER_GATED_DELTA;
    switch (mx.c.mixer) {
    case PRISM_MIXER_LIGHTNING: return mix_lightning(e, ly, mx, rows, n, seq);
    case PRISM_MIXER_LATENT_ATTENTION: return mix_latent(e, ly, mx, rows, n, seq);
    case PRISM_MIXER_ATTENTION: return mix_attention(e, ly, mx, rows, n, seq, side);
    default: return mix_delta(e, ly, mx, rows, n, seq, side);
    }
}
// Lightning: all heads normed together, then gated, as the input of the output linear takes it.
static void lightning_norm(LayeredModel *m, const LayeredLayer &ly, const LayeredMixer &mx, DenseIn &in) {
    in.norm_w = mx.mix_norm; in.n_norm = mx.width(); in.eps = m->c.norm_eps;
    in.gate = at(m, m->proj, ly.in.seg[mx.seg0 + 3].row0); in.gate_pitch = m->proj_pitch;
}
// Where the segments of a layer's `in` go: rows of proj, the fp32 projections to aux.
static void in_outs(const LayeredModel *m, const LayeredLayer &ly, DenseOut *outs) {
    for (uint32_t s = 0; s < ly.in.n_segs; s++) outs[s] = DenseOut{at(m, m->proj, ly.in.seg[s].row0), m->proj_pitch, ST_ACT};
    for (const LayeredMixer &mx : ly.mix)
        if (mx.c.mixer == PRISM_MIXER_GATED_DELTA) outs[mx.seg0 + 3] = DenseOut{m->aux, m->aux_pitch, ST_F32};
}

static int forward_parallel(prism_cuda_engine *e, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    const uint32_t D = m->c.width;
    for (LayeredLayer &ly : m->layers) {
        DenseIn in{};
        in.x = m->x; in.pitch = D; in.f32 = 1; in.norm_w = ly.norm1; in.n_norm = D; in.eps = m->c.norm_eps;
        DenseOut outs[DENSE_MAX_SEGS];
        in_outs(m, ly, outs);
        if (ly.c.ff) outs[ly.seg_up] = DenseOut{at(m, m->cat, ly.k_mix), m->cat_pitch, ST_ACT};
        PRISM_TRY(linear(e, ly.in, in, outs, n, m->xn, m->width_pad));
        PRISM_TRY(run_mixer(e, ly, ly.mix[0], rows, n, seq));
        DenseIn oi{};
        oi.x = m->cat; oi.pitch = m->cat_pitch;
        if (ly.c.mixer == PRISM_MIXER_LIGHTNING) lightning_norm(m, ly, ly.mix[0], oi);
        const DenseOut ro{m->x, D, ST_RESID};
        PRISM_TRY(linear(e, ly.out, oi, &ro, n, m->cat, m->cat_pitch));
    }
    return PRISM_OK;
}

// The row-wise kernel between two sublayers, ending with the norm (and convolution) of sublayer `which` of `next`.
static int row_step(prism_cuda_engine *e, RowUpdate &u, const LayeredLayer *next, int which, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    const uint32_t D = m->c.width, taps = m->c.canon_taps;
    u.x = m->x; u.width = D; u.eps = m->c.norm_eps; u.mul = m->c.residual_mult;
    if (next) {
        u.norm = which == 1 ? next->norm1 : next->norm2;
        u.h = m->xn; u.h_pitch = m->width_pad;
        if (taps && !seq) {
            u.conv_w = which == 1 ? next->canon1 : next->canon2;
            u.ring = which == 1 ? next->ring1 : next->ring2;
            u.taps = taps; u.hc = m->xc;
        }
    }
    PRISM_TRY(launch_row_update(e->ctx, u, rows, n, m->act32));
    if (!next || !taps || !seq) return PRISM_OK;
    ConvArgs c{};
    c.pieces = 1; c.x_pitch = c.y_pitch = m->width_pad; c.taps = taps; c.channels = D;
    c.w = which == 1 ? next->canon1 : next->canon2;
    c.ring = which == 1 ? next->ring1 : next->ring2;
    c.piece[0] = ConvPiece{m->xn, m->xc, D, 0};
    return launch_conv_seq(e->ctx, c, rows, n, m->act32);
}

// Feed-forward of the rows in m->xc / m->xn, up to its result: a row each, or rows of the experts with the plan.
static int feed_forward(prism_cuda_engine *e, LayeredLayer &ly, const DenseIn &in, uint32_t n, RowUpdate &u) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    DenseOut outs[DENSE_MAX_SEGS];
    for (uint32_t s = 0; s < ly.in2.n_segs; s++) outs[s] = DenseOut{at(m, m->proj, ly.in2.seg[s].row0), m->proj_pitch, ST_ACT};
    outs[ly.seg_up] = ly.c.experts ? DenseOut{m->aux, m->aux_pitch, ST_F32} : DenseOut{m->act, m->act_pitch, ST_ACT};
    PRISM_TRY(linear(e, ly.in2, in, outs, n, nullptr, 0));
    if (m->c.gated_residual) {
        u.gate = at(m, m->proj, ly.in2.seg[ly.seg_gate2].row0);
        u.gate_pitch = m->proj_pitch;
    }
    const DenseOut ao{m->act, m->act_pitch, ST_ACT}, yo{m->y, m->y_pitch, ST_ACT};
    DenseIn act{};
    act.x = m->act; act.pitch = m->act_pitch;
    u.y = m->y; u.y_pitch = m->y_pitch;
    if (!ly.c.experts) {
        u.add = ROW_ADD_ONE;
        return linear(e, ly.down, act, &yo, n, nullptr, 0);
    }
    MoePlan plan = m->plan;
    plan.experts = ly.c.experts;
    plan.top = ly.c.top;
    const bool few = !m->act32 && ctx->fuse && n <= DENSE_GEMV_ROWS;
    const uint32_t pairs = n * plan.top;
    PRISM_TRY(launch_moe_route(ctx, MoeRouter{ly.c.expert_groups, ly.c.groups_keep, m->aux, ly.correction, m->aux_pitch}, plan, n, !few));
    u.add = ROW_ADD_EXPERTS; u.wgt = plan.wgt; u.inv = few ? nullptr : plan.inv; u.top = plan.top;
    if (few) {
        PRISM_TRY(launch_moe_gemv(ctx, ly.up, plan, in, false, ao, n));
        return launch_moe_gemv(ctx, ly.down, plan, act, true, yo, n);
    }
    PRISM_TRY(launch_moe_gather(ctx, plan, in.x, in.pitch, m->moe_x, m->width_pad, m->width_pad, pairs, m->act32));
    DenseIn rows{};
    rows.x = m->moe_x; rows.pitch = m->width_pad;
    if (m->act32) {
        PRISM_TRY(launch_moe_f32(ctx, ly.up, plan, rows, ao, pairs));
        return launch_moe_f32(ctx, ly.down, plan, act, yo, pairs);
    }
    PRISM_TRY(launch_moe_gemm_tc5(ctx, ly.up, plan, rows, ao, pairs));
    return launch_moe_gemm_tc5(ctx, ly.down, plan, act, yo, pairs);
}

// All mixers of a layer.  In a prompt portion the second of a pair runs on a stream of its own: its chunks follow one
// another on a part of the GPU.
static int run_mixers(prism_cuda_engine *e, LayeredLayer &ly, const RowMap &rows, uint32_t n, bool seq) {
    prism_cuda_ctx *ctx = e->ctx;
    LayeredModel *m = e->lm;
    auto whole = [&](LayeredMixer &mx) -> int {
        PRISM_TRY(run_mixer(e, ly, mx, rows, n, seq));
        if (mx.c.mixer != PRISM_MIXER_LIGHTNING) return PRISM_OK;
        DenseIn h{};
        h.x = at(m, m->cat, mx.col); h.pitch = m->cat_pitch;
        lightning_norm(m, ly, mx, h);
        return launch_dense_norm(ctx, h, at(m, m->cat, mx.col), m->cat_pitch, n, m->act32);
    };
    if (!seq || ly.mix.size() != 2 || ly.mix[0].c.mixer == ly.mix[1].c.mixer || n <= DENSE_GEMV_ROWS) {  // mixers of a kind share scratch
        for (LayeredMixer &mx : ly.mix) PRISM_TRY(whole(mx));
        return PRISM_OK;
    }
    const cudaStream_t main = ctx->stream;
    PRISM_CUDA_TRY(ctx, cudaEventRecord(m->fork, main));
    PRISM_CUDA_TRY(ctx, cudaStreamWaitEvent(m->side, m->fork, 0));
    ctx->stream = m->side;
    const int rc = whole(ly.mix[1]);
    ctx->stream = main;
    PRISM_TRY(rc);
    PRISM_CUDA_TRY(ctx, cudaEventRecord(m->join, m->side));
    PRISM_TRY(whole(ly.mix[0]));
    PRISM_CUDA_TRY(ctx, cudaStreamWaitEvent(main, m->join, 0));
    return PRISM_OK;
}

static int forward_sequential(prism_cuda_engine *e, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    const uint32_t D = m->c.width, L = m->c.num_layers;
    DenseIn in{};  // what the sublayers read: the convolved norm, and the norm itself
    in.x = m->c.canon_taps ? m->xc : m->xn;
    in.x2 = m->xn;
    in.pitch = in.pitch2 = m->width_pad;
    RowUpdate u{};
    PRISM_TRY(row_step(e, u, &m->layers[0], 1, rows, n, seq));
    for (uint32_t i = 0; i < L; i++) {
        LayeredLayer &ly = m->layers[i];
        const LayeredLayer *next = i + 1 < L ? &m->layers[i + 1] : nullptr;
        auto layer_end = [&](RowUpdate &r) {
            if (!m->c.depth_average) return;
            r.history = m->history; r.history_stride = (size_t)m->cap * D; r.avg = ly.avg; r.n_history = i + 1;
        };
        DenseOut outs[DENSE_MAX_SEGS];
        in_outs(m, ly, outs);
        PRISM_TRY(linear(e, ly.in, in, outs, n, nullptr, 0));
        PRISM_TRY(run_mixers(e, ly, rows, n, seq));
        DenseIn oi{};
        oi.x = m->cat; oi.pitch = m->cat_pitch;
        const bool pair = ly.mix.size() > 1;
        if (pair) {
            oi.x2 = at(m, m->cat, ly.mix[1].col);
            oi.pitch2 = m->cat_pitch;
        }
        const DenseOut yo[2] = {{m->y, m->y_pitch, ST_ACT}, {at(m, m->y, (size_t)m->cap * m->y_pitch), m->y_pitch, ST_ACT}};
        PRISM_TRY(linear(e, ly.out, oi, yo, n, nullptr, 0));
        u = RowUpdate{};
        u.x_out = m->x;
        u.add = pair ? ROW_ADD_PAIR : ROW_ADD_ONE;
        u.y = yo[0].p; u.y_pitch = m->y_pitch;
        if (pair) {
            u.y2 = yo[1].p; u.y2_pitch = m->y_pitch;
            u.w = ly.mix[0].out_norm; u.w2 = ly.mix[1].out_norm;
        }
        if (m->c.gated_residual) {
            u.gate = at(m, m->proj, ly.in.seg[ly.seg_gate1].row0);
            u.gate_pitch = m->proj_pitch;
        }
        if (!ly.c.ff) {
            layer_end(u);
            PRISM_TRY(row_step(e, u, next, 1, rows, n, seq));
            continue;
        }
        PRISM_TRY(row_step(e, u, &ly, 2, rows, n, seq));
        u = RowUpdate{};
        u.x_out = m->x;
        PRISM_TRY(feed_forward(e, ly, in, n, u));
        layer_end(u);
        PRISM_TRY(row_step(e, u, next, 1, rows, n, seq));
    }
    return PRISM_OK;
}

// `n` tokens (device ids) through every layer, their residual rows in m->x.
static int forward_tokens(prism_cuda_engine *e, const uint32_t *tokens, const RowMap &rows, uint32_t n, bool seq) {
    LayeredModel *m = e->lm;
    PRISM_TRY(launch_dense_embed(e->ctx, m->embed, m->c.width, m->c.vocab, tokens, n, m->x, m->pos, m->c.max_positions, rows, m->history));
    return m->c.arrangement == PRISM_ARRANGE_SEQUENTIAL ? forward_sequential(e, rows, n, seq) : forward_parallel(e, rows, n, seq);
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
    PRISM_TRY(forward_tokens(e, e->tok, rows, B, false));
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
        for (LayeredMixer &mx : ly.mix)
            if (float *state = mx.state ? mx.state : mx.da.state) {
                const size_t n = (size_t)mx.c.heads * mx.c.dim * mx.c.vdim;
                PRISM_CUDA_TRY(e->ctx, cudaMemsetAsync(state + slot * n, 0, n * 4, e->ctx->stream));
            }
    m->slot_pos[slot] = 0;  // caches and convolution rings need no clearing: only positions below the slot's are ever read
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
        PRISM_TRY(forward_tokens(e, m->pf_tok, rows, k, true));
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
    const bool sequential = m->c.arrangement == PRISM_ARRANGE_SEQUENTIAL;
    for (const LayeredLayer &ly : m->layers) {
        const uint64_t D = m->c.width, experts = ly.c.experts ? std::min<uint64_t>(B * ly.c.top, ly.c.experts) : 1;
        bytes += ly.in.valid_rows() * D * 2;
        if (sequential) bytes += (ly.in2.valid_rows() * D + experts * (ly.c.experts ? 2 : 1) * ly.c.ff * D) * 2;
        else bytes += (uint64_t)ly.c.ff * D * 2;
        for (const LayeredMixer &mx : ly.mix) {
            const prism_layer_config &c = mx.c;
            const uint64_t hv = mx.width(), seen = c.window ? std::min<uint64_t>(keys, c.window) : keys;
            bytes += hv * D * 2;
            if (c.mixer == PRISM_MIXER_LIGHTNING || c.mixer == PRISM_MIXER_GATED_DELTA) {
                bytes += B * 8 * (uint64_t)c.heads * c.dim * c.vdim;  // state read and written
            } else if (c.mixer == PRISM_MIXER_ATTENTION) {
                bytes += B * seen * c.kv_heads * (c.dim + c.vdim) * es;
            } else {
                bytes += mx.uq.valid_rows() * c.q_rank * 2 + ((uint64_t)c.heads * c.dim + hv) * c.kv_rank * 2;
                bytes += B * seen * (c.kv_rank + c.rot_dim) * es;
            }
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
    if (c.max_positions && c.max_seq > c.max_positions) return fail(ctx, PRISM_E_ARG, "max_seq exceeds the position table");
    if (c.arrangement > PRISM_ARRANGE_SEQUENTIAL || (c.arrangement == PRISM_ARRANGE_PARALLEL && (c.canon_taps || c.gated_residual || c.depth_average)))
        return fail(ctx, PRISM_E_ARG, "input convolutions, gated residuals and depth averages belong to the sequential arrangement");
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
