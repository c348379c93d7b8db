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

constexpr int GA_THREADS = 256, GA_KT = 128, GA_PRE = 4;  // value vectors a thread requests before the scores
// Eight consecutive values as they are in memory.
template <typename TA>
struct Raw8;
template <>
struct Raw8<bf16> {
    uint4 u;
    __device__ __forceinline__ void load(const bf16 *p) { u = *reinterpret_cast<const uint4 *>(p); }
    __device__ __forceinline__ void get(float (&x)[8]) const {
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&w[i]));
            x[2 * i] = f.x;
            x[2 * i + 1] = f.y;
        }
    }
};
template <>
struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float *p) {
        a = reinterpret_cast<const float4 *>(p)[0];
        b = reinterpret_cast<const float4 *>(p)[1];
    }
    __device__ __forceinline__ void get(float (&x)[8]) const {
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
        x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    }
};

// Grid: (splits, key/value head x part of its query heads, row); a cluster along x shares the row's keys.  `lpk`
// lanes share a key in the scores, one thread owns eight value columns of some keys in the weighted sum; GR
// query heads go together.  The CTAs of a cluster exchange maxima, sums and partial outputs through shared memory.
template <typename TA, int GR>
__global__ void __launch_bounds__(GA_THREADS) grouped_rows_kernel(const GroupedArgs a, const TA *__restrict__ q, const TA *__restrict__ k,
                                                                  const TA *__restrict__ v, uint32_t pitch, TA *__restrict__ out, uint32_t out_pitch,
                                                                  const RowMap rows, uint32_t parts, uint32_t lpk, uint32_t late) {
    extern __shared__ __align__(16) float gas[];
    __shared__ float sc[GR][GA_KT], ms[GR], ls[GR], fs[GR];
    if (!late) pdl_launch_dependents();
    pdl_wait();
    if (late) pdl_launch_dependents();
    cg::cluster_group cluster = cg::this_cluster();
    const uint32_t rank = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r = blockIdx.z;
    const uint32_t g = blockIdx.y / parts, group = a.heads / a.kv_heads, h0 = g * group + (blockIdx.y % parts) * GR, nh = min((uint32_t)GR, (g + 1) * group - h0);
    const int32_t pos = rows.pos_of(r), slot = rows.slot_of(r), lo = window_first(a.window, pos);
    const int32_t n = pos + 1 - lo, per = (n + (int32_t)a.splits - 1) / (int32_t)a.splits;
    const int32_t kb = lo + (int32_t)rank * per, ke = min(kb + per, pos + 1);
    TA *kc = reinterpret_cast<TA *>(a.kc), *vc = reinterpret_cast<TA *>(a.vc);
    float *qs = gas, *acs = gas + GR * a.dp, *red = acs + GR * a.vp;
    const bool fresh = k && kb <= pos && pos < ke;  // the new position: appended by the CTA that reads it
    if (fresh) {
        const size_t row = key_row(a, slot, pos) * a.kv_heads + g;
        for (uint32_t i = tid; i < a.dim; i += GA_THREADS) kc[row * a.dp + i] = k[(size_t)r * pitch + g * a.dim + i];
        for (uint32_t i = tid; i < a.vdim; i += GA_THREADS) vc[row * a.vp + i] = v[(size_t)r * pitch + g * a.vdim + i];
        __syncthreads();
    }
    // rows of the ring behind key kb + j, j < per
    const uint32_t ring0 = kb > pos ? 0 : (uint32_t)kb % a.ring;
    auto row_of = [&](uint32_t j) {
        const uint32_t x = ring0 + j;
        return ((size_t)slot * a.ring + (x >= a.ring ? x - a.ring : x)) * a.kv_heads + g;
    };
    const uint32_t nvv = a.vp / 8, vgs = GA_THREADS / nvv, vv = tid % nvv, vg = tid / nvv;  // idle threads past nvv * vgs
    const uint32_t li = tid % lpk, kg = tid / lpk, nkg = GA_THREADS / lpk, d8 = a.dp / 8;
    for (uint32_t i = tid; i < GR * a.dp; i += GA_THREADS) {
        const uint32_t hh = i / a.dp, d = i % a.dp;
        qs[i] = hh < nh && d < a.dim ? ld_act(q + (size_t)r * pitch + (h0 + hh) * a.dim + d) * a.scale : 0.0f;
    }
    if (tid < GR) { ms[tid] = -INFINITY; ls[tid] = 0.0f; }
    __syncthreads();
    float acc[GR][8];
#pragma unroll
    for (int h = 0; h < GR; h++)
#pragma unroll
        for (int i = 0; i < 8; i++) acc[h][i] = 0.0f;
    for (int32_t k0 = kb; k0 < ke; k0 += GA_KT) {
        const uint32_t nk = (uint32_t)min(ke - k0, (int32_t)GA_KT), j_tile = (uint32_t)(k0 - kb);
        Raw8<TA> pre[GA_PRE];
#pragma unroll
        for (int i = 0; i < GA_PRE; i++)
            if (vg < vgs && vg + i * vgs < nk) pre[i].load(vc + row_of(j_tile + vg + i * vgs) * a.vp + vv * 8);
        for (uint32_t j0 = 0; j0 < nk; j0 += 2 * nkg) {  // the same for every lane of a warp; two keys at a time
            Raw8<TA> kx[2];
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const uint32_t j = j0 + e * nkg + kg;
                if (j < nk && li < d8) kx[e].load(kc + row_of(j_tile + j) * a.dp + li * 8);
            }
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const uint32_t j = j0 + e * nkg + kg;
                float s[GR];
#pragma unroll
                for (int h = 0; h < GR; h++) s[h] = 0.0f;
                if (j < nk) {
                    float x[8];
                    if (li < d8) {
                        kx[e].get(x);
#pragma unroll
                        for (int h = 0; h < GR; h++) {
                            const float4 u = *reinterpret_cast<const float4 *>(qs + h * a.dp + li * 8), w = *reinterpret_cast<const float4 *>(qs + h * a.dp + li * 8 + 4);
                            s[h] = u.x * x[0] + u.y * x[1] + u.z * x[2] + u.w * x[3] + w.x * x[4] + w.y * x[5] + w.z * x[6] + w.w * x[7];
                        }
                    }
                    for (uint32_t c = li + lpk; c < d8; c += lpk) {
                        Raw8<TA> y;
                        y.load(kc + row_of(j_tile + j) * a.dp + c * 8);
                        y.get(x);
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
            if (k0 != kb) {
#pragma unroll
                for (int h = 0; h < GR; h++) {
                    const float f = fs[h];
#pragma unroll
                    for (int i = 0; i < 8; i++) acc[h][i] *= f;
                }
            }
            auto add = [&](const Raw8<TA> &y, uint32_t j) {
                float x[8];
                y.get(x);
#pragma unroll
                for (int h = 0; h < GR; h++) {
                    const float p = sc[h][j];
#pragma unroll
                    for (int i = 0; i < 8; i++) acc[h][i] = fmaf(p, x[i], acc[h][i]);
                }
            };
#pragma unroll
            for (int i = 0; i < GA_PRE; i++)
                if (vg + i * vgs < nk) add(pre[i], vg + i * vgs);
#pragma unroll 2
            for (uint32_t j = vg + GA_PRE * vgs; j < nk; j += vgs) {
                Raw8<TA> y;
                y.load(vc + row_of(j_tile + j) * a.vp + vv * 8);
                add(y, j);
            }
        }
        __syncthreads();
    }
    if (vg < vgs) {
#pragma unroll
        for (int h = 0; h < GR; h++)
#pragma unroll
            for (int i = 0; i < 8; i += 4)
                *reinterpret_cast<float4 *>(red + ((size_t)vg * GR + h) * a.vp + vv * 8 + i) = make_float4(acc[h][i], acc[h][i + 1], acc[h][i + 2], acc[h][i + 3]);
    }
    __syncthreads();
    for (uint32_t i = tid; i < GR * a.vp; i += GA_THREADS) {
        float s = 0.0f;
#pragma unroll 8
        for (uint32_t e = 0; e < vgs; e++) s += red[(size_t)e * GR * a.vp + i];
        acs[i] = s;
    }
    if (a.splits > 1) cluster.sync();
    else __syncthreads();
    for (uint32_t i = rank * GA_THREADS + tid; i < nh * a.vdim; i += a.splits * GA_THREADS) {
        const uint32_t h = i / a.vdim, c = i % a.vdim;
        float o = acs[h * a.vp + c], l = ls[h];
        if (a.splits > 1) {
            float pm[8], pl[8], po[8], m = -INFINITY;  // of the CTAs of the cluster
#pragma unroll
            for (int e = 0; e < 8; e++) {
                const bool on = e < (int)a.splits;
                const int peer = on ? e : 0;
                pm[e] = on ? *cluster.map_shared_rank(&ms[h], peer) : -INFINITY;
                pl[e] = *cluster.map_shared_rank(&ls[h], peer);
                po[e] = *cluster.map_shared_rank(acs + h * a.vp + c, peer);
            }
#pragma unroll
            for (int e = 0; e < 8; e++) m = fmaxf(m, pm[e]);
            l = o = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; e++) {
                const float f = expf(pm[e] - m);  // 0 for a CTA without keys
                l = fmaf(pl[e], f, l);
                o = fmaf(po[e], f, o);
            }
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
                     uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool late) {
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
                           a, row(q, pitch), row(k, pitch), row(v, pitch), pitch, (TA *)out + (size_t)r * out_pitch, out_pitch, sub, parts, lpk, (uint32_t)late);
        PRISM_TRY(after_launch(ctx, "grouped_rows_kernel"));
    }
    return PRISM_OK;
}
template <typename TA>
static int launch_rows(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *q, const void *k, const void *v, uint32_t pitch, void *out,
                       uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool late) {
    const uint32_t group = a.heads / a.kv_heads;
    if (group <= 1) return launch_gr<TA, 1>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows, late);
    if (group <= 2) return launch_gr<TA, 2>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows, late);
    if (group <= 4) return launch_gr<TA, 4>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows, late);
    return launch_gr<TA, 8>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows, late);
}
int launch_grouped_rows(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *q, const void *k, const void *v, uint32_t pitch, void *out,
                        uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool act32, bool late) {
    return act32 ? launch_rows<float>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows, late)
                 : launch_rows<bf16>(ctx, a, q, k, v, pitch, out, out_pitch, rows, n_rows, late);
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
