// Softmax attention whose query heads share key/value heads, optionally under a sliding window, without
// rotation.  The cache keeps every position's key and value heads; a windowed layer's cache is a ring.
//   rows     one token of a row per cluster of CTAs that share its keys (decode, short portions, 32-bit)
//   prefill  the tiled tensor-core attention straight over the cache (prompt portions)
#include <cooperative_groups.h>

#include <algorithm>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace prism {

__device__ __forceinline__ size_t key_row(const GroupedArgs &a, int32_t slot, int32_t pos) {
    return (size_t)slot * a.ring + (uint32_t)pos % a.ring;
}

// Keys and values of a row into the cache; the padding of a head is zero from the start and stays so.
template <typename TA>
__global__ void __launch_bounds__(256) grouped_append_kernel(const GroupedArgs a, const TA *__restrict__ k, const TA *__restrict__ v, uint32_t pitch,
                                                             const RowMap rows) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.x;
    const size_t row = key_row(a, rows.slot_of(r), rows.pos_of(r)) * a.kv_heads;
    TA *kc = reinterpret_cast<TA *>(a.kc) + row * a.dp, *vc = reinterpret_cast<TA *>(a.vc) + row * a.vp;
    for (uint32_t i = threadIdx.x; i < a.kv_heads * a.dim; i += 256) kc[i / a.dim * a.dp + i % a.dim] = k[(size_t)r * pitch + i];
    for (uint32_t i = threadIdx.x; i < a.kv_heads * a.vdim; i += 256) vc[i / a.vdim * a.vp + i % a.vdim] = v[(size_t)r * pitch + i];
}
int launch_grouped_append(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *k, const void *v, uint32_t pitch, const RowMap &rows, uint32_t n_rows,
                          bool act32) {
    if (act32) launch_pdl(ctx, "grouped_append_kernel", grouped_append_kernel<float>, n_rows, 256, 0, a, (const float *)k, (const float *)v, pitch, rows);
    else launch_pdl(ctx, "grouped_append_kernel", grouped_append_kernel<bf16>, n_rows, 256, 0, a, (const bf16 *)k, (const bf16 *)v, pitch, rows);
    return after_launch(ctx, "grouped_append_kernel");
}

// Eight consecutive values.
__device__ __forceinline__ void ld8(const bf16 *p, float (&x)[8]) {
    const uint4 u = *reinterpret_cast<const uint4 *>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&w[i]));
        x[2 * i] = f.x;
        x[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void ld8(const float *p, float (&x)[8]) {
    const float4 u = reinterpret_cast<const float4 *>(p)[0], v = reinterpret_cast<const float4 *>(p)[1];
    x[0] = u.x; x[1] = u.y; x[2] = u.z; x[3] = u.w;
    x[4] = v.x; x[5] = v.y; x[6] = v.z; x[7] = v.w;
}

// Grid: (splits, key/value head x part of its query heads, row); a cluster along x shares the row's keys.  `lpk`
// lanes share a key in the scores, one thread owns eight value columns of some keys in the weighted sum; GR
// query heads go together.  The CTAs of a cluster exchange maxima, sums and partial outputs through shared memory.
constexpr int GA_THREADS = 256, GA_KT = 128;
template <typename TA, int GR>
__global__ void __launch_bounds__(GA_THREADS) grouped_rows_kernel(const GroupedArgs a, const TA *__restrict__ q, const TA *__restrict__ k,
                                                                  const TA *__restrict__ v, uint32_t pitch, TA *__restrict__ out, uint32_t out_pitch,
                                                                  const RowMap rows, uint32_t parts, uint32_t lpk) {
    extern __shared__ __align__(16) float gas[];
    __shared__ float sc[GR][GA_KT], ms[GR], ls[GR], fs[GR];
    pdl_launch_dependents();
    pdl_wait();
    cg::cluster_group cluster = cg::this_cluster();
    const uint32_t rank = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r = blockIdx.z;
    const uint32_t g = blockIdx.y / parts, group = a.heads / a.kv_heads, h0 = g * group + (blockIdx.y % parts) * GR, nh = min((uint32_t)GR, (g + 1) * group - h0);
    const int32_t pos = rows.pos_of(r), slot = rows.slot_of(r), lo = window_first(a.window, pos);
    const int32_t n = pos + 1 - lo, per = (n + (int32_t)a.splits - 1) / (int32_t)a.splits;
    const int32_t kb = lo + (int32_t)rank * per, ke = min(kb + per, pos + 1);
    TA *kc = reinterpret_cast<TA *>(a.kc), *vc = reinterpret_cast<TA *>(a.vc);
    float *qs = gas, *acs = gas + GR * a.dp, *red = acs + GR * a.vp;
    for (uint32_t i = tid; i < GR * a.dp; i += GA_THREADS) {
        const uint32_t hh = i / a.dp, d = i % a.dp;
        qs[i] = hh < nh && d < a.dim ? ld_act(q + (size_t)r * pitch + (h0 + hh) * a.dim + d) * a.scale : 0.0f;
    }
    if (k && kb <= pos && pos < ke) {  // the new position: appended by the CTA that reads it
        const size_t row = key_row(a, slot, pos) * a.kv_heads + g;
        for (uint32_t i = tid; i < a.dim; i += GA_THREADS) kc[row * a.dp + i] = k[(size_t)r * pitch + g * a.dim + i];
        for (uint32_t i = tid; i < a.vdim; i += GA_THREADS) vc[row * a.vp + i] = v[(size_t)r * pitch + g * a.vdim + i];
    }
    if (tid < GR) { ms[tid] = -INFINITY; ls[tid] = 0.0f; }
    __syncthreads();
    const uint32_t li = tid % lpk, kg = tid / lpk, nkg = GA_THREADS / lpk, d8 = a.dp / 8;
    float q0[GR][8];
    if (li < d8) {
#pragma unroll
        for (int h = 0; h < GR; h++) ld8(qs + h * a.dp + li * 8, q0[h]);
    }
    const uint32_t nvv = a.vp / 8, vgs = GA_THREADS / nvv, vv = tid % nvv, vg = tid / nvv;  // idle threads past nvv * vgs
    float acc[GR][8];
#pragma unroll
    for (int h = 0; h < GR; h++)
#pragma unroll
        for (int i = 0; i < 8; i++) acc[h][i] = 0.0f;
    for (int32_t k0 = kb; k0 < ke; k0 += GA_KT) {
        const uint32_t nk = (uint32_t)min(ke - k0, (int32_t)GA_KT);
        for (uint32_t j0 = 0; j0 < nk; j0 += nkg) {  // the same for every lane of a warp
            const uint32_t j = j0 + kg;
            float s[GR];
#pragma unroll
            for (int h = 0; h < GR; h++) s[h] = 0.0f;
            if (j < nk) {
                const TA *kr = kc + (key_row(a, slot, k0 + (int32_t)j) * a.kv_heads + g) * a.dp;
                float x[8];
                if (li < d8) {
                    ld8(kr + li * 8, x);
#pragma unroll
                    for (int h = 0; h < GR; h++)
#pragma unroll
                        for (int i = 0; i < 8; i++) s[h] = fmaf(q0[h][i], x[i], s[h]);
                }
                for (uint32_t c = li + lpk; c < d8; c += lpk) {
                    ld8(kr + c * 8, x);
#pragma unroll
                    for (int h = 0; h < GR; h++)
#pragma unroll
                        for (int i = 0; i < 8; i++) s[h] = fmaf(qs[h * a.dp + c * 8 + i], x[i], s[h]);
                }
            }
            for (uint32_t o = lpk / 2; o > 0; o >>= 1) {
#pragma unroll
                for (int h = 0; h < GR; h++) s[h] += __shfl_xor_sync(0xFFFFFFFFu, s[h], o);
            }
            if (li == 0 && j < nk) {
#pragma unroll
                for (int h = 0; h < GR; h++) sc[h][j] = s[h];
            }
        }
        __syncthreads();
        if (warp < GR) {
            float m = -INFINITY, l = 0.0f;
            for (uint32_t j = lane; j < nk; j += 32) m = fmaxf(m, sc[warp][j]);
            m = fmaxf(warp_max_f(m), ms[warp]);
            for (uint32_t j = lane; j < nk; j += 32) {
                const float p = expf(sc[warp][j] - m);
                sc[warp][j] = p;
                l += p;
            }
            l = warp_sum_f(l);
            if (lane == 0) {
                const float f = expf(ms[warp] - m);
                fs[warp] = f;
                ls[warp] = ls[warp] * f + l;
                ms[warp] = m;
            }
        }
        __syncthreads();
        if (vg < vgs) {
#pragma unroll
            for (int h = 0; h < GR; h++) {
                const float f = fs[h];
#pragma unroll
                for (int i = 0; i < 8; i++) acc[h][i] *= f;
            }
#pragma unroll 2
            for (uint32_t j = vg; j < nk; j += vgs) {
                float x[8];
                ld8(vc + (key_row(a, slot, k0 + (int32_t)j) * a.kv_heads + g) * a.vp + vv * 8, x);
#pragma unroll
                for (int h = 0; h < GR; h++) {
                    const float p = sc[h][j];
#pragma unroll
                    for (int i = 0; i < 8; i++) acc[h][i] = fmaf(p, x[i], acc[h][i]);
                }
            }
        }
        __syncthreads();
    }
    if (vg < vgs) {
#pragma unroll
        for (int h = 0; h < GR; h++)
#pragma unroll
            for (int i = 0; i < 8; i++) red[((size_t)vg * GR + h) * a.vp + vv * 8 + i] = acc[h][i];
    }
    __syncthreads();
    for (uint32_t i = tid; i < GR * a.vp; i += GA_THREADS) {
        float s = 0.0f;
        for (uint32_t e = 0; e < vgs; e++) s += red[(size_t)e * GR * a.vp + i];
        acs[i] = s;
    }
    if (a.splits > 1) cluster.sync();
    else __syncthreads();
    for (uint32_t i = rank * GA_THREADS + tid; i < nh * a.vdim; i += a.splits * GA_THREADS) {
        const uint32_t h = i / a.vdim, c = i % a.vdim;
        float m = -INFINITY, l = 0.0f, o = 0.0f;
        if (a.splits > 1) {
            for (uint32_t e = 0; e < a.splits; e++) m = fmaxf(m, *cluster.map_shared_rank(&ms[h], e));
            for (uint32_t e = 0; e < a.splits; e++) {
                const float f = expf(*cluster.map_shared_rank(&ms[h], e) - m);  // 0 for a CTA without keys
                l = fmaf(*cluster.map_shared_rank(&ls[h], e), f, l);
                o = fmaf(*cluster.map_shared_rank(acs + h * a.vp + c, e), f, o);
            }
        } else {
            l = ls[h];
            o = acs[h * a.vp + c];
        }
        st_act(out + (size_t)r * out_pitch + (h0 + h) * a.vdim + c, o / l);
    }
    if (a.splits > 1) cluster.sync();  // the peers read this CTA's shared memory
}

uint32_t grouped_splits(const GroupedArgs &a, uint32_t max_seq) {
    const uint32_t keys = a.window ? std::min(a.window, max_seq) : max_seq;
    uint32_t s = 1;
    while (s < 8 && keys > s * 64) s *= 2;
    return s;
}

constexpr size_t GA_SMEM_MAX = 200 * 1024;
template <typename TA, int GR>
static int launch_gr(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *q, const void *k, const void *v, uint32_t pitch, void *out,
                     uint32_t out_pitch, const RowMap &rows, uint32_t n_rows) {
    const uint32_t nvv = a.vp / 8, vgs = GA_THREADS / std::max(nvv, 1u);
    const size_t smem = ((size_t)GR * a.dp + (size_t)GR * a.vp * (1 + vgs)) * 4;
    if (!vgs || smem > GA_SMEM_MAX) return fail(ctx, PRISM_E_ARG, "grouped attention: heads too large");
    static bool configured[PRISM_MAX_DEVICES] = {false};
    if (!configured[ctx->device]) {
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(grouped_rows_kernel<TA, GR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)GA_SMEM_MAX));
        configured[ctx->device] = true;
    }
    uint32_t lpk = 1;
    while (lpk < 32 && lpk * 8 < a.dp) lpk *= 2;
    const uint32_t parts = (a.heads / a.kv_heads + GR - 1) / GR;
    for (uint32_t r = 0; r < n_rows; r += 32768) {  // the grid's third dimension ends at 65535
        RowMap sub = rows;
        if (sub.slot) {
            sub.slot += r;
            sub.pos += r;
        } else {
            sub.pos0 += (int32_t)r;
        }
        auto row = [&](const void *p, uint32_t pt) { return p ? (const TA *)p + (size_t)r * pt : nullptr; };
        launch_cluster_pdl(ctx, grouped_rows_kernel<TA, GR>, dim3(a.splits, a.kv_heads * parts, std::min(n_rows - r, 32768u)), GA_THREADS, smem, a.splits,
                           a, row(q, pitch), row(k, pitch), row(v, pitch), pitch, (TA *)out + (size_t)r * out_pitch, out_pitch, sub, parts, lpk);
        PRISM_TRY(after_launch(ctx, "grouped_rows_kernel"));
    }
    return PRISM_OK;
}
template <typename TA>
static int launch_rows(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *q, const void *k, const void *v, uint32_t pitch, void *out,
                       uint32_t out_pitch, const RowMap &rows, uint32_t n_rows) {
    const uint32_t group = a.heads / a.kv_heads;
    if (group <= 1) return launch_gr<TA, 1>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows);
    if (group <= 2) return launch_gr<TA, 2>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows);
    if (group <= 4) return launch_gr<TA, 4>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows);
    return launch_gr<TA, 8>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows);
}
int launch_grouped_rows(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *q, const void *k, const void *v, uint32_t pitch, void *out,
                        uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool act32) {
    return act32 ? launch_rows<float>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows)
                 : launch_rows<bf16>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows);
}

int launch_grouped_prefill(prism_cuda_ctx *ctx, const GroupedArgs &a, const bf16 *q, uint32_t pitch, bf16 *out, uint32_t out_pitch, const RowMap &rows,
                           uint32_t n_rows) {
    TiledAttn p{};
    p.heads = a.heads; p.group = a.heads / a.kv_heads; p.dim = a.dim; p.vdim = a.vdim; p.window = a.window;
    p.scale = a.scale;
    const size_t slot = (size_t)rows.slot0 * a.ring * a.kv_heads;
    p.q = q; p.kx = (const bf16 *)a.kc + slot * a.dp; p.vx = (const bf16 *)a.vc + slot * a.vp; p.out = out;
    p.q_pitch = pitch; p.kx_pitch = a.kv_heads * a.dp; p.vx_pitch = a.kv_heads * a.vp; p.out_pitch = out_pitch;
    p.kx_head = a.dp; p.vx_head = a.vp;
    p.ring = a.ring; p.pos0 = (uint32_t)rows.pos0; p.n_rows = n_rows;
    return launch_tiled_attn(ctx, p);
}

}  // namespace prism
