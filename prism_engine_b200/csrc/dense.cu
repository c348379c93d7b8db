// Dense bf16 linears for few rows, the same linears in 32-bit, and the element-wise kernels around
// them: weight packing, RMS norm with a weight, embedding gather, fp32 argmax.
#include <cooperative_groups.h>

#include <algorithm>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace prism {

// ---- weights -------------------------------------------------------------------------------------

int dense_alloc(prism_cuda_ctx *ctx, DenseLinear &l, uint32_t k_pad, uint32_t n_tiles) {
    l.k_pad = k_pad;
    l.n_tiles = n_tiles;
    PRISM_CUDA_TRY(ctx, cudaMalloc((void **)&l.w, l.bytes()));
    PRISM_CUDA_TRY(ctx, cudaMemsetAsync(l.w, 0, l.bytes(), ctx->stream));
    return PRISM_OK;
}

__global__ void dense_pack_kernel(const bf16 *__restrict__ src, uint32_t rows, uint32_t cols, bf16 *__restrict__ w, uint32_t k_pad,
                                  uint32_t row0, uint32_t k0) {
    const size_t n = (size_t)rows * cols;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const uint32_t r = row0 + (uint32_t)(i / cols), k = k0 + (uint32_t)(i % cols);
        w[(((size_t)(r >> 7) * (k_pad / 8) + (k >> 3)) * 128 + (r & 127)) * 8 + (k & 7)] = src[i];
    }
}
int launch_dense_pack(prism_cuda_ctx *ctx, const DenseLinear &l, const bf16 *src, uint32_t rows, uint32_t cols, uint32_t row0,
                      uint32_t k0) {
    const size_t n = (size_t)rows * cols;
    dense_pack_kernel<<<(unsigned)std::min<size_t>((n + 255) / 256, 65535), 256, 0, ctx->stream>>>(src, rows, cols, l.w, l.k_pad, row0, k0);
    return after_launch(ctx, "dense_pack_kernel");
}

__global__ void bf16_to_f32_kernel(const bf16 *__restrict__ src, float *__restrict__ dst, size_t n, float add, uint32_t cols, uint32_t pitch) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) dst[i % cols * pitch + i / cols] = __bfloat162float(src[i]) + add;
}
int launch_bf16_to_f32(prism_cuda_ctx *ctx, const bf16 *src, float *dst, size_t n, float add, uint32_t cols, uint32_t pitch) {
    bf16_to_f32_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(src, dst, n, add, cols, pitch);
    return after_launch(ctx, "bf16_to_f32_kernel");
}

__global__ void bf16_pitch_copy_kernel(const bf16 *__restrict__ src, bf16 *__restrict__ dst, uint32_t rows, uint32_t cols, uint32_t pitch) {
    const size_t n = (size_t)rows * pitch;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const uint32_t r = (uint32_t)(i / pitch), c = (uint32_t)(i % pitch);
        dst[i] = c < cols ? src[(size_t)r * cols + c] : __float2bfloat16_rn(0.0f);
    }
}
int launch_bf16_pitch_copy(prism_cuda_ctx *ctx, const bf16 *src, bf16 *dst, uint32_t rows, uint32_t cols, uint32_t dst_pitch) {
    const size_t n = (size_t)rows * dst_pitch;
    bf16_pitch_copy_kernel<<<(unsigned)std::min<size_t>((n + 255) / 256, 65535), 256, 0, ctx->stream>>>(src, dst, rows, cols, dst_pitch);
    return after_launch(ctx, "bf16_pitch_copy_kernel");
}

// Seeded values N(mean, sigma) of a benchmark model (Box-Muller over a counter hash).
__device__ __forceinline__ uint32_t mix32(uint64_t z) {
    z += 0x9E3779B97F4A7C15ull;
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    return (uint32_t)(z ^ (z >> 31));
}
__global__ void dense_synth_kernel(bf16 *__restrict__ dst, size_t n, uint64_t seed, float mean, float sigma) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const float u1 = ((float)mix32(seed * 0x100000001B3ull + 2 * i) + 1.0f) * 2.3283064e-10f;
        const float u2 = (float)mix32(seed * 0x100000001B3ull + 2 * i + 1) * 2.3283064e-10f;
        dst[i] = __float2bfloat16_rn(mean + sigma * sqrtf(-2.0f * logf(fminf(u1, 1.0f))) * cospif(2.0f * u2));
    }
}
int launch_dense_synth(prism_cuda_ctx *ctx, bf16 *dst, size_t n, uint64_t seed, float mean, float sigma) {
    dense_synth_kernel<<<(unsigned)std::min<size_t>((n + 255) / 256, 65535), 256, 0, ctx->stream>>>(dst, n, seed, mean, sigma);
    return after_launch(ctx, "dense_synth_kernel");
}

DenseEpi dense_epi(const DenseLinear &l, const DenseOut *outs) {
    DenseEpi e{};
    e.n = l.n_segs;
    for (uint32_t i = 0; i < l.n_segs; i++)
        e.s[i] = DenseEpiSeg{l.seg[i].row0, l.seg[i].rows, l.seg[i].act, outs[i].store, outs[i].pitch, l.seg[i].in,
                             l.seg[i].k ? l.seg[i].k : l.k_pad, l.seg[i].mul, l.seg[i].bias, outs[i].p};
    return e;
}

// ---- few rows: mma.sync straight from the weight units ----------------------------------------------
// A CTA takes 32 weight rows at a time; its eight warps share the k range in steps of 32.  In a step lane
// (g, t) = (lane / 4, lane % 4) loads the units (row g + 8 i, k/8 = 4 step + t): eight consecutive k of four
// rows, and the same eight k of token g of the input.  The order of k inside a dot product is free as long
// as both operands agree, so these registers ARE the fragments of two m16n8k16 products per 16 rows: no
// conversion, no shuffles, and any batch of 1..8 costs the same.  The sums of the warps meet in shared
// memory in a fixed order.  When there are too few row blocks for the GPU a cluster of `ks` CTAs shares the
// k range of a block; the sums of ranks 1.. travel to rank 0 through distributed shared memory.
struct GemvArgs {
    const uint4 *w;
    uint32_t k8, n_groups, rows, ks;
    const void *x;
    uint32_t pitch, f32;
    const bf16 *x2;
    uint32_t pitch2;
    const float *norm_w;
    const bf16 *gate;
    uint32_t gate_pitch, n_norm, norm_pad, norm_vec;  // norm_pad: n_norm rounded up to 64; norm_vec: rows allow 4-value accesses
    float eps;
    DenseEpi epi;
    // experts: the stack's row tiles per expert, the plan, whether input rows are pairs
    uint32_t n_tiles, by_pair;
    const uint32_t *n_active, *active;
    const int32_t *pair_of;
};
constexpr int GV_THREADS = 256, GV_WARPS = 8, GV_U = 4, GV_KS_MAX = 4;

// RMS norm (times weight, times gate) of the first n_norm entries of the one or two rows into shared memory as bf16.
// A row's threads keep their values and weights in registers (the weights requested before the dependency wait).
constexpr int GN_U = 8;
struct GemvNorm {
    float4 w[GN_U];
    uint32_t tpr, r, i0;
    bool vec;
    __device__ __forceinline__ void prefetch(const GemvArgs &a) {
        tpr = a.rows == 1 ? 256 : 128;  // threads per row
        r = threadIdx.x / tpr;
        i0 = threadIdx.x % tpr;
        vec = a.norm_vec && a.n_norm <= tpr * 4 * GN_U;
        if (vec) {
#pragma unroll
            for (int u = 0; u < GN_U; u++) {
                const uint32_t i = (i0 + u * tpr) * 4;
                w[u] = i < a.n_norm ? ld4(a.norm_w + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        }
    }
    __device__ __forceinline__ float inverse(const GemvArgs &a, float ss, float *sh) const {
        ss = warp_sum_f(ss);
        if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
        __syncthreads();
        float s = 0.0f;
        for (uint32_t k = 0; k < tpr / 32; k++) s += sh[r * (tpr / 32) + k];
        return 1.0f / sqrtf(s / (float)a.n_norm + a.eps);
    }
    __device__ __forceinline__ void stage(const GemvArgs &a, bf16 *xs, float *sh) const {
        const float *xf = reinterpret_cast<const float *>(a.x) + (size_t)r * a.pitch;
        const bf16 *xh = reinterpret_cast<const bf16 *>(a.x) + (size_t)r * a.pitch, *gr = a.gate ? a.gate + (size_t)r * a.gate_pitch : nullptr;
        bf16 *y = xs + (size_t)r * a.norm_pad;
        float ss = 0.0f;
        if (vec) {
            float4 v[GN_U];
#pragma unroll
            for (int u = 0; u < GN_U; u++) {
                const uint32_t i = (i0 + u * tpr) * 4;
                v[u] = i < a.n_norm ? a.f32 ? ld4(xf + i) : ld4(xh + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                ss += v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
            }
            const float inv = inverse(a, ss, sh);
#pragma unroll
            for (int u = 0; u < GN_U; u++) {
                const uint32_t i = (i0 + u * tpr) * 4;
                if (i >= a.norm_pad) break;
                float4 o = make_float4(v[u].x * inv * w[u].x, v[u].y * inv * w[u].y, v[u].z * inv * w[u].z, v[u].w * inv * w[u].w);
                if (gr && i < a.n_norm) {
                    const float4 g = ld4(gr + i);
                    o = make_float4(o.x * g.x, o.y * g.y, o.z * g.z, o.w * g.w);
                }
                st4(y + i, o);
            }
        } else {
            for (uint32_t i = i0; i < a.n_norm; i += tpr) {
                const float v = a.f32 ? xf[i] : __bfloat162float(xh[i]);
                ss += v * v;
            }
            const float inv = inverse(a, ss, sh);
            for (uint32_t i = i0; i < a.norm_pad; i += tpr) {
                float v = 0.0f;
                if (i < a.n_norm) {
                    v = (a.f32 ? xf[i] : __bfloat162float(xh[i])) * inv * __ldg(a.norm_w + i);
                    if (gr) v *= __bfloat162float(gr[i]);
                }
                y[i] = __float2bfloat16_rn(v);
            }
        }
        __syncthreads();
    }
};

// MOE: items are blocks of 32 rows of the experts in use; every token column is multiplied, the pairs are stored.
enum GemvKind { GV_PLAIN = 0, GV_NORM = 1, GV_MOE = 2 };
template <int KIND>
__global__ void __launch_bounds__(GV_THREADS, 2) dense_gemv_kernel(const GemvArgs a) {
    constexpr bool NORM = KIND == GV_NORM, MOE = KIND == GV_MOE;
    extern __shared__ __align__(16) uint8_t dsm[];
    __shared__ float red[GV_WARPS][8][33];
    __shared__ float peer[GV_KS_MAX][8][32];  // rank 0: sums of the other ranks
    __shared__ float sh[32];
    bf16 *xs = reinterpret_cast<bf16 *>(dsm);
    pdl_launch_dependents();
    cg::cluster_group cluster = cg::this_cluster();
    const uint32_t rank = a.ks > 1 ? cluster.block_rank() : 0;
    if (a.ks > 1) asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");  // met before the first remote store
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t norm8 = NORM ? a.norm_pad / 8 : 0;
    const uint4 *xl = reinterpret_cast<const uint4 *>(xs + (size_t)g8 * a.norm_pad);
    uint4 w[GV_U][4];
    uint32_t sg = 0, rb = 0, act = 0, first = 0, steps = 0;  // segment, block of 32 rows inside it, expert in use, this rank's k range
    auto locate = [&](uint32_t grp) -> const uint4 * {       // first unit
        uint32_t tile0 = 0;
        sg = 0;
        rb = grp;
        if (MOE) {
            act = grp / a.n_groups;
            rb = grp % a.n_groups;
            tile0 = a.active[act] * a.n_tiles;
        }
        while (sg + 1 < a.epi.n && rb >= (a.epi.s[sg].rows + 31) / 32) {
            rb -= (a.epi.s[sg].rows + 31) / 32;
            sg++;
        }
        const uint32_t row = a.epi.s[sg].row0 + rb * 32, all = a.epi.s[sg].k / 32;
        first = all * rank / a.ks;
        steps = all * (rank + 1) / a.ks;
        return a.w + (size_t)(tile0 + (row >> 7)) * a.k8 * 128 + (row & 127) + g8;
    };
    auto load = [&](const uint4 *wt, uint32_t s0) {
#pragma unroll
        for (int u = 0; u < GV_U; u++) {
            const uint32_t s = s0 + u * GV_WARPS;
            if (s < steps) {
                const uint4 *p = wt + (size_t)(4 * s + t4) * 128;
#pragma unroll
                for (int i = 0; i < 4; i++) w[u][i] = __ldg(p + 8 * i);
            }
        }
    };
    const uint32_t grp0 = blockIdx.x / a.ks;
    uint32_t n_items = a.n_groups;
    const uint4 *wt = nullptr;
    bool loaded = !MOE;
    if (!MOE) {
        wt = locate(grp0);
        load(wt, first + warp);  // weights do not depend on the previous kernel; the input does
    }
    GemvNorm norm;
    if (NORM) norm.prefetch(a);
    pdl_wait();
    if (NORM) norm.stage(a, xs, sh);
    if (MOE) n_items *= *reinterpret_cast<const volatile uint32_t *>(a.n_active);
    if (MOE && a.ks > 1 && grp0 >= n_items) asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");  // nothing to do for this cluster
    for (uint32_t grp = grp0; grp < n_items; grp += gridDim.x / a.ks) {
        if (!loaded) wt = locate(grp);
        const int32_t pair = MOE ? a.pair_of[act * DENSE_GEMV_ROWS + g8] : 0;
        const bool tok_on = MOE ? g8 < a.rows && pair >= 0 : g8 < a.rows;
        const uint32_t x_row = MOE && a.by_pair ? (uint32_t)pair : g8;
        const uint4 *xg = !MOE && a.epi.s[sg].in ? reinterpret_cast<const uint4 *>(a.x2 + (size_t)g8 * a.pitch2)
                                                 : reinterpret_cast<const uint4 *>(reinterpret_cast<const bf16 *>(a.x) + (size_t)x_row * a.pitch);
        float acc[2][4] = {};
        for (uint32_t s0 = first + warp; s0 < steps; s0 += GV_WARPS * GV_U) {
            if (!loaded) load(wt, s0);
            loaded = false;
#pragma unroll
            for (int u = 0; u < GV_U; u++) {
                const uint32_t s = s0 + u * GV_WARPS;
                if (s < steps) {
                    const uint32_t k8 = 4 * s + t4;
                    uint4 x = make_uint4(0, 0, 0, 0);
                    if (tok_on) x = NORM && k8 < norm8 ? xl[k8] : xg[k8];
#pragma unroll
                    for (int m = 0; m < 2; m++) {
                        const uint4 lo = w[u][2 * m], hi = w[u][2 * m + 1];
                        const uint32_t a0[4] = {lo.x, hi.x, lo.y, hi.y}, a1[4] = {lo.z, hi.z, lo.w, hi.w};
                        mma_bf16(acc[m], a0, x.x, x.y);
                        mma_bf16(acc[m], a1, x.z, x.w);
                    }
                }
            }
        }
        loaded = false;
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
            for (int i = 0; i < 4; i++) red[warp][2 * t4 + (i & 1)][16 * m + g8 + 8 * (i >> 1)] = acc[m][i];
        __syncthreads();
        const uint32_t t = threadIdx.x >> 5, rl = rb * 32 + lane;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < GV_WARPS; w++) v += red[w][t][lane];
        if (a.ks > 1) {  // one block per cluster (the grid is n_groups * ks)
            asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
            if (rank) *cluster.map_shared_rank(&peer[rank][t][lane], 0) = v;
            cluster.sync();
            if (rank) return;
            for (uint32_t r = 1; r < a.ks; r++) v += peer[r][t][lane];
        }
        const int32_t out_row = MOE ? a.pair_of[act * DENSE_GEMV_ROWS + t] : (int32_t)t;
        if (t < a.rows && out_row >= 0 && rl < a.epi.s[sg].rows) dense_store<bf16>(a.epi.s[sg], rl, (uint32_t)out_row, v);
        __syncthreads();
    }
}

static size_t gemv_smem(const DenseIn &in, uint32_t rows) {
    return in.norm_w ? (size_t)rows * round_up_u32(in.n_norm, 64) * 2 : 0;
}
constexpr size_t GV_SMEM_MAX = 160 * 1024;
constexpr uint32_t GV_FOLD_ROWS = 2;  // as many as GemvNorm splits the block into; more rows: every CTA norming all of them costs more than a norm kernel does

bool dense_gemv_ok(const DenseIn &in, uint32_t rows) {
    return rows <= DENSE_GEMV_ROWS && !(in.x2 && in.pitch2 % 8) && (in.norm_w ? rows <= GV_FOLD_ROWS && gemv_smem(in, rows) <= GV_SMEM_MAX : !in.f32) &&
           (in.f32 || in.pitch % 8 == 0);
}

// Few row blocks and a long k: a block's k range is shared inside a cluster, at least GV_WARPS * GV_U steps each.
static uint32_t gemv_cluster(prism_cuda_ctx *ctx, uint32_t blocks, uint32_t k8) {
    const uint32_t slots = 2u * (uint32_t)ctx->sm_count;
    uint32_t ks = 1;
    while (ks < GV_KS_MAX && blocks * ks * 2 <= slots + slots / 2 && k8 / 4 >= ks * 2 * GV_WARPS * GV_U) ks *= 2;
    return ks;
}
static GemvArgs gemv_args(const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows) {
    GemvArgs a{};
    a.w = reinterpret_cast<const uint4 *>(l.w);
    a.k8 = l.k_pad / 8;
    a.rows = rows;
    a.x = in.x; a.pitch = in.pitch; a.f32 = in.f32;
    a.x2 = reinterpret_cast<const bf16 *>(in.x2); a.pitch2 = in.pitch2;
    a.epi = dense_epi(l, outs);
    for (uint32_t s = 0; s < l.n_segs; s++) a.n_groups += (l.seg[s].rows + 31) / 32;
    return a;
}

int launch_dense_gemv(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows) {
    GemvArgs a = gemv_args(l, in, outs, rows);
    a.norm_w = in.norm_w; a.n_norm = in.n_norm; a.norm_pad = round_up_u32(in.n_norm, 64); a.eps = in.eps;
    a.gate = reinterpret_cast<const bf16 *>(in.gate); a.gate_pitch = in.gate_pitch;
    a.norm_vec = !((reinterpret_cast<uintptr_t>(in.x) | reinterpret_cast<uintptr_t>(in.gate) | reinterpret_cast<uintptr_t>(in.norm_w)) & 15) &&
                 !((in.pitch | in.n_norm | (in.gate ? in.gate_pitch : 0)) & 3);
    a.ks = gemv_cluster(ctx, a.n_groups, a.k8);
    const size_t smem = gemv_smem(in, rows);
    const uint32_t grid = a.ks > 1 ? a.n_groups * a.ks : std::min(a.n_groups, 2u * (uint32_t)ctx->sm_count);
    if (in.norm_w) {
        static bool configured[PRISM_MAX_DEVICES] = {false};
        if (!configured[ctx->device]) {
            PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(dense_gemv_kernel<GV_NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)GV_SMEM_MAX));
            configured[ctx->device] = true;
        }
        launch_cluster_pdl(ctx, dense_gemv_kernel<GV_NORM>, grid, GV_THREADS, smem, a.ks, a);
    } else {
        launch_cluster_pdl(ctx, dense_gemv_kernel<GV_PLAIN>, grid, GV_THREADS, 0, a.ks, a);
    }
    return after_launch(ctx, "dense_gemv_kernel");
}

int launch_moe_gemv(prism_cuda_ctx *ctx, const DenseLinear &l, const MoePlan &plan, const DenseIn &in, bool by_pair, const DenseOut &out, uint32_t tokens) {
    if (tokens > DENSE_GEMV_ROWS || l.n_segs != 1 || in.pitch % 8) return fail(ctx, PRISM_E_ARG, "experts: too many tokens for the small-batch kernel");
    GemvArgs a = gemv_args(l, in, &out, tokens);
    a.n_tiles = l.n_tiles; a.by_pair = by_pair;
    a.n_active = plan.n_active; a.active = plan.active; a.pair_of = plan.pair_of;
    const uint32_t items = a.n_groups * std::min(tokens * plan.top, plan.experts);  // at most
    a.ks = gemv_cluster(ctx, items, a.k8);
    const uint32_t grid = a.ks > 1 ? items * a.ks : std::min(items, 2u * (uint32_t)ctx->sm_count);
    launch_cluster_pdl(ctx, dense_gemv_kernel<GV_MOE>, grid, GV_THREADS, 0, a.ks, a);
    return after_launch(ctx, "dense_gemv_kernel");
}

// ---- 32-bit ------------------------------------------------------------------------------------------
// 64 weight rows x 64 input rows per CTA, 4 x 4 per thread, plain fp32 multiply-adds.
struct F32Args {
    const bf16 *w;
    uint32_t k_pad, rows;
    const float *x, *x2;
    uint32_t pitch, pitch2;
    DenseEpi epi;
    uint32_t n_tiles, experts;  // experts: rows are sorted by expert
    const uint32_t *count;
};
constexpr int F32_BK = 16;
template <bool MOE>
__global__ void __launch_bounds__(256) dense_f32_kernel(const F32Args a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float ws[F32_BK][68], xs[F32_BK][68];
    const uint32_t tid = threadIdx.x, row0 = blockIdx.x * 64;
    uint32_t t0 = blockIdx.y * 64, t_end = a.rows, tile0 = 0;
    if (MOE) {
        uint32_t expert, left;
        if (!moe_find_tile(a.count, a.experts, 64, blockIdx.y, expert, t0, left)) return;  // the same in every warp
        tile0 = expert * a.n_tiles;
        t_end = t0 + left;
    }
    const DenseEpiSeg &seg = dense_seg(a.epi, row0);
    if (row0 >= seg.row0 + seg.rows) return;                  // padding
    const float *x = seg.in ? a.x2 : a.x;
    const uint32_t pitch = seg.in ? a.pitch2 : a.pitch;
    const uint32_t tx = tid & 15, ty = tid >> 4;              // rows tx*4.., tokens ty*4..
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < seg.k; k0 += F32_BK) {
        for (uint32_t i = tid; i < 64 * F32_BK; i += 256) {
            const uint32_t r = i / F32_BK, k = i % F32_BK;
            const uint32_t row = row0 + r, kk = k0 + k;
            ws[k][r] = __bfloat162float(a.w[(((size_t)(tile0 + (row >> 7)) * (a.k_pad / 8) + (kk >> 3)) * 128 + (row & 127)) * 8 + (kk & 7)]);
            xs[k][r] = t0 + r < t_end && kk < pitch ? x[(size_t)(t0 + r) * pitch + kk] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < F32_BK; k++) {
            float w[4], x[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { w[i] = ws[k][tx * 4 + i]; x[i] = xs[k][ty * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(w[i], x[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (int j = 0; j < 4; j++)
        for (int i = 0; i < 4; i++) {
            const uint32_t rl = row0 + tx * 4 + i - seg.row0, t = t0 + ty * 4 + j;
            if (rl < seg.rows && t < t_end) dense_store<float>(seg, rl, t, acc[i][j]);
        }
}
int launch_dense_f32(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows) {
    F32Args a{l.w, l.k_pad, rows, (const float *)in.x, (const float *)in.x2, in.pitch, in.pitch2, dense_epi(l, outs), l.n_tiles, 1, nullptr};
    launch_pdl(ctx, "dense_f32_kernel", dense_f32_kernel<false>, dim3(l.n_tiles * 2, (rows + 63) / 64), 256, 0, a);
    return after_launch(ctx, "dense_f32_kernel");
}
int launch_moe_f32(prism_cuda_ctx *ctx, const DenseLinear &l, const MoePlan &plan, const DenseIn &in, const DenseOut &out, uint32_t pairs) {
    F32Args a{l.w, l.k_pad, pairs, (const float *)in.x, nullptr, in.pitch, 0, dense_epi(l, &out), l.n_tiles, plan.experts, plan.count};
    const uint32_t tiles = pairs / 64 + std::min(pairs, plan.experts);  // at most
    launch_pdl(ctx, "dense_f32_kernel", dense_f32_kernel<true>, dim3(l.n_tiles * 2, tiles), 256, 0, a);
    return after_launch(ctx, "dense_f32_kernel");
}

// ---- element-wise ------------------------------------------------------------------------------------
constexpr int DN_THREADS = 256, DN_U = 8;  // a row of up to 8192 values is read once and kept in registers
template <typename TX, typename TA>
__global__ void __launch_bounds__(DN_THREADS) dense_norm_kernel(const TX *__restrict__ x, uint32_t pitch, const float *__restrict__ w,
                                                                const TA *__restrict__ gate, uint32_t gate_pitch, uint32_t n, float eps, TA *y,
                                                                uint32_t y_pitch, uint32_t vec) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float sh[32];
    const uint32_t r = blockIdx.x;
    const TX *xr = x + (size_t)r * pitch;
    const TA *gr = gate ? gate + (size_t)r * gate_pitch : nullptr;
    TA *yr = y + (size_t)r * y_pitch;
    float ss = 0.0f;
    if (vec) {
        float4 v[DN_U];
#pragma unroll
        for (int u = 0; u < DN_U; u++) {
            const uint32_t i = (threadIdx.x + u * DN_THREADS) * 4;
            v[u] = i < n ? ld4(xr + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            ss += v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
        }
        ss = block_sum_f(ss, sh);
        const float inv = 1.0f / sqrtf(ss / (float)n + eps);
#pragma unroll
        for (int u = 0; u < DN_U; u++) {
            const uint32_t i = (threadIdx.x + u * DN_THREADS) * 4;
            if (i >= n) break;
            const float4 wv = ld4(w + i);
            float4 o = make_float4(v[u].x * inv * wv.x, v[u].y * inv * wv.y, v[u].z * inv * wv.z, v[u].w * inv * wv.w);
            if (gr) {
                const float4 g = ld4(gr + i);
                o = make_float4(o.x * g.x, o.y * g.y, o.z * g.z, o.w * g.w);
            }
            st4(yr + i, o);
        }
        return;
    }
    for (uint32_t i = threadIdx.x; i < n; i += DN_THREADS) {
        const float v = ld_act(xr + i);
        ss += v * v;
    }
    ss = block_sum_f(ss, sh);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
    for (uint32_t i = threadIdx.x; i < n; i += DN_THREADS) {
        float v = ld_act(xr + i) * inv * __ldg(w + i);
        if (gr) v *= ld_act(gr + i);
        st_act(yr + i, v);
    }
}
template <typename TX, typename TA>
static void run_dense_norm(prism_cuda_ctx *ctx, const DenseIn &in, void *y, uint32_t y_pitch, uint32_t rows) {
    const uintptr_t p = reinterpret_cast<uintptr_t>(in.x) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(in.gate) | reinterpret_cast<uintptr_t>(in.norm_w);
    const uint32_t vec = !(p & 15) && !((in.pitch | y_pitch | in.n_norm | (in.gate ? in.gate_pitch : 0)) & 3) && in.n_norm <= DN_THREADS * DN_U * 4;
    launch_pdl(ctx, "dense_norm_kernel", dense_norm_kernel<TX, TA>, rows, DN_THREADS, 0, (const TX *)in.x, in.pitch, in.norm_w, (const TA *)in.gate,
               in.gate_pitch, in.n_norm, in.eps, (TA *)y, y_pitch, vec);
}
int launch_dense_norm(prism_cuda_ctx *ctx, const DenseIn &in, void *y, uint32_t y_pitch, uint32_t rows, bool act32) {
    if (act32) run_dense_norm<float, float>(ctx, in, y, y_pitch, rows);
    else if (in.f32) run_dense_norm<float, bf16>(ctx, in, y, y_pitch, rows);
    else run_dense_norm<bf16, bf16>(ctx, in, y, y_pitch, rows);
    return after_launch(ctx, "dense_norm_kernel");
}

constexpr uint32_t DE_COLS = 1024;  // columns of a CTA
__global__ void dense_embed_kernel(const bf16 *__restrict__ table, uint32_t width, uint32_t vocab, const uint32_t *__restrict__ tokens,
                                   float *__restrict__ x, const bf16 *__restrict__ pos_table, uint32_t max_pos, const RowMap map, float *__restrict__ x2) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.x, tok = min(tokens[r], vocab - 1);  // the host rejects larger ids before the launch
    const uint32_t c1 = min(width, (blockIdx.y + 1) * DE_COLS);
    const bf16 *pt = pos_table ? pos_table + (size_t)min((uint32_t)map.pos_of(r), max_pos - 1) * width : nullptr;  // and later positions
    for (uint32_t i = blockIdx.y * DE_COLS + threadIdx.x; i < c1; i += blockDim.x) {
        const float v = __bfloat162float(table[(size_t)tok * width + i]) + (pt ? __bfloat162float(pt[i]) : 0.0f);
        x[(size_t)r * width + i] = v;
        if (x2) x2[(size_t)r * width + i] = v;
    }
}
int launch_dense_embed(prism_cuda_ctx *ctx, const bf16 *table, uint32_t width, uint32_t vocab, const uint32_t *tokens, uint32_t rows, float *x,
                       const bf16 *pos_table, uint32_t max_pos, const RowMap &map, float *x2) {
    launch_pdl(ctx, "dense_embed_kernel", dense_embed_kernel, dim3(rows, (width + DE_COLS - 1) / DE_COLS), 256, 0, table, width, vocab, tokens, x, pos_table, max_pos, map, x2);
    return after_launch(ctx, "dense_embed_kernel");
}

__global__ void gather_rows_f32_kernel(const float *__restrict__ x, const uint32_t *__restrict__ idx, uint32_t width, float *__restrict__ y) {
    pdl_launch_dependents();
    pdl_wait();
    const float *s = x + (size_t)idx[blockIdx.x] * width;
    for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) y[(size_t)blockIdx.x * width + i] = s[i];
}
int launch_gather_rows_f32(prism_cuda_ctx *ctx, const float *x, const uint32_t *idx, uint32_t n, uint32_t width, float *y) {
    launch_pdl(ctx, "gather_rows_f32_kernel", gather_rows_f32_kernel, n, 256, 0, x, idx, width, y);
    return after_launch(ctx, "gather_rows_f32_kernel");
}

__global__ void f32_to_f16_kernel(const float *__restrict__ x, uint32_t n, uint32_t stride, uint16_t *__restrict__ y, uint32_t y_stride) {
    const uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) y[(size_t)blockIdx.y * y_stride + i] = __half_as_ushort(__float2half_rn(x[(size_t)blockIdx.y * stride + i]));
}
int launch_f32_to_f16(prism_cuda_ctx *ctx, const float *x, uint32_t rows, uint32_t n, uint32_t stride, uint16_t *y, uint32_t y_stride) {
    f32_to_f16_kernel<<<dim3((n + 255) / 256, rows), 256, 0, ctx->stream>>>(x, n, stride, y, y_stride);
    return after_launch(ctx, "f32_to_f16_kernel");
}

}  // namespace prism
