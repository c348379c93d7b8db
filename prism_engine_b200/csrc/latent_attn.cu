// Latent attention: keys and values are expanded from one cached latent per token (plus one rotated key
// part shared by all heads), optionally under a sliding window.  Two ways to the same sums:
//   rows     W_uk is folded into the query and W_uv applied to the weighted latent, so the cached latents
//            themselves are scored and weighed (all heads share them): decode, short portions, and 32-bit;
//   expanded a prompt portion expands keys and values of the positions it can see once (two stacked
//            linears) and runs a tiled tensor-core attention over them (tiled_attn_kernel, which the
//            grouped attention runs over its cache too).
// The cache keeps [latent | rotated key] per position; a windowed layer's cache is a ring.
#include <algorithm>
#include <cmath>

#include "dense.cuh"

namespace prism {

__device__ __forceinline__ size_t cache_row(const LatentCache &c, int32_t slot, int32_t pos) {
    return ((size_t)slot * c.ring + (uint32_t)pos % c.ring) * c.pitch;
}
__device__ __forceinline__ int32_t first_key(const LatentArgs &a, int32_t pos) { return window_first(a.window, pos); }
// Rotate-half of the pair (u, v) with index i at position pos.
__device__ __forceinline__ void rotate_pair(const float *__restrict__ freq, float mul, int32_t pos, uint32_t i, float &u, float &v) {
    float s, c;
    sincosf((float)pos * __ldg(freq + i), &s, &c);
    s *= mul;
    c *= mul;
    const float x = u * c - v * s, y = v * c + u * s;
    u = x;
    v = y;
}

// ---- append ------------------------------------------------------------------------------------------
// By a whole block: row r of W_dkv h, its latent normed, its rotated part turned, into the cache.  sh: 32 floats.
template <typename TA>
__device__ __forceinline__ void append_row(const LatentArgs &a, const TA *__restrict__ dkv, uint32_t pitch, const RowMap &rows, uint32_t r, float *sh) {
    const int32_t pos = rows.pos_of(r);
    const TA *x = dkv + (size_t)r * pitch;
    TA *y = reinterpret_cast<TA *>(a.cache.rows) + cache_row(a.cache, rows.slot_of(r), pos);
    float ss = 0.0f;
    for (uint32_t i = threadIdx.x; i < a.kv_rank; i += blockDim.x) {
        const float v = ld_act(x + i);
        ss += v * v;
    }
    ss = block_sum_f(ss, sh);
    const float inv = 1.0f / sqrtf(ss / (float)a.kv_rank + a.eps);
    for (uint32_t i = threadIdx.x; i < a.kv_rank; i += blockDim.x) st_act(y + i, ld_act(x + i) * inv * __ldg(a.dkv_norm + i));
    x += a.kv_rank;
    y += a.kv_rank;
    for (uint32_t i = threadIdx.x; i < a.rot_pairs; i += blockDim.x) {
        float u = ld_act(x + i), v = ld_act(x + a.rot_pairs + i);
        rotate_pair(a.rot_freq, a.rot_mul, pos, i, u, v);
        st_act(y + i, u);
        st_act(y + a.rot_pairs + i, v);
    }
    for (uint32_t i = 2 * a.rot_pairs + threadIdx.x; i < a.rot_dim; i += blockDim.x) y[i] = x[i];
}
template <typename TA>
__global__ void __launch_bounds__(128) latent_append_kernel(const LatentArgs a, const TA *__restrict__ dkv, uint32_t pitch, const RowMap rows) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float sh[32];
    append_row(a, dkv, pitch, rows, blockIdx.x, sh);
}
int launch_latent_append(prism_cuda_ctx *ctx, const LatentArgs &a, const void *dkv, uint32_t pitch, const RowMap &rows, uint32_t n_rows, bool act32) {
    if (act32) launch_pdl(ctx, "latent_append_kernel", latent_append_kernel<float>, n_rows, 128, 0, a, (const float *)dkv, pitch, rows);
    else launch_pdl(ctx, "latent_append_kernel", latent_append_kernel<bf16>, n_rows, 128, 0, a, (const bf16 *)dkv, pitch, rows);
    return after_launch(ctx, "latent_append_kernel");
}

// ---- rows: query against the latents -------------------------------------------------------------------
// qa[r][h] = [W_uk[h]^T q_unrotated | rotated q | zeros], fp32.  Grid: (head, 128 latent columns, 4 rows).  One
// more block along x appends the rows to the cache meanwhile.
constexpr int LQ_ROWS = 4, LQ_PRE = 8;  // weight units a thread requests before the dependency wait
template <typename TA>
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentArgs a, const TA *__restrict__ q, uint32_t q_pitch,
                                                           const TA *__restrict__ dkv, uint32_t dkv_pitch, const RowMap rows, uint32_t n_rows,
                                                           float *__restrict__ qa) {
    __shared__ float red[16][LQ_ROWS][130];
    pdl_launch_dependents();
    const uint32_t h = blockIdx.x, c8 = threadIdx.x & 15, dg = threadIdx.x >> 4, col = blockIdx.y * 128 + c8 * 8, r0 = blockIdx.z * LQ_ROWS;
    const uint32_t hq = a.dim + a.rot_dim, L = a.cache.pitch;
    if (h == a.heads) {
        pdl_wait();
        if (blockIdx.y == 0)
            for (uint32_t r = r0; r < min(n_rows, r0 + LQ_ROWS); r++) append_row(a, dkv, dkv_pitch, rows, r, &red[0][0][0]);
        return;
    }
    const bool on = col < a.uk_pitch;
    const bf16 *wk = a.uk + (size_t)h * a.dim * a.uk_pitch + col;
    uint4 pre[LQ_PRE];
#pragma unroll
    for (int i = 0; i < LQ_PRE; i++) {
        pre[i] = make_uint4(0, 0, 0, 0);
        if (on && dg + 16 * i < a.dim) pre[i] = __ldg(reinterpret_cast<const uint4 *>(wk + (size_t)(dg + 16 * i) * a.uk_pitch));
    }
    pdl_wait();
    float acc[LQ_ROWS][8] = {};
    auto add = [&](uint32_t d, const uint4 &w4) {
        const bf16 *w = reinterpret_cast<const bf16 *>(&w4);
#pragma unroll
        for (int r = 0; r < LQ_ROWS; r++) {
            const float x = r0 + r < n_rows ? ld_act(q + (size_t)(r0 + r) * q_pitch + h * hq + d) : 0.0f;
#pragma unroll
            for (int i = 0; i < 8; i++) acc[r][i] = fmaf(__bfloat162float(w[i]), x, acc[r][i]);
        }
    };
#pragma unroll
    for (int i = 0; i < LQ_PRE; i++)
        if (dg + 16 * i < a.dim) add(dg + 16 * i, pre[i]);
    for (uint32_t d = dg + 16 * LQ_PRE; d < a.dim; d += 16)
        add(d, on ? __ldg(reinterpret_cast<const uint4 *>(wk + (size_t)d * a.uk_pitch)) : make_uint4(0, 0, 0, 0));
#pragma unroll
    for (int r = 0; r < LQ_ROWS; r++)
#pragma unroll
        for (int i = 0; i < 8; i++) red[dg][r][c8 * 8 + i] = acc[r][i];
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < LQ_ROWS * 128; i += 256) {
        const uint32_t r = i >> 7, c = i & 127, j = blockIdx.y * 128 + c;
        if (r0 + r >= n_rows || j >= a.kv_rank) continue;
        float s = 0.0f;
#pragma unroll
        for (int g = 0; g < 16; g++) s += red[g][r][c];
        qa[((size_t)(r0 + r) * a.heads + h) * L + j] = s;
    }
    if (blockIdx.y == 0) {
        for (uint32_t i = threadIdx.x; i < LQ_ROWS * (L - a.kv_rank); i += 256) {
            const uint32_t r = i / (L - a.kv_rank), c = i % (L - a.kv_rank);
            if (r0 + r >= n_rows) continue;
            const TA *x = q + (size_t)(r0 + r) * q_pitch + h * hq + a.dim;
            float v = 0.0f;
            if (c < 2 * a.rot_pairs) {
                const uint32_t p = c < a.rot_pairs ? c : c - a.rot_pairs;
                float u = ld_act(x + p), w = ld_act(x + a.rot_pairs + p);
                rotate_pair(a.rot_freq, a.rot_mul, rows.pos_of(r0 + r), p, u, w);
                v = c < a.rot_pairs ? u : w;
            } else if (c < a.rot_dim) {
                v = ld_act(x + c);
            }
            qa[((size_t)(r0 + r) * a.heads + h) * L + a.kv_rank + c] = v;
        }
    }
}

// Partial sums of LR_KT keys: for every head the maximum, the sum of exponentials and the weighted latent.
constexpr int LR_KT = 64;
struct LatentPart { float *part, *ml; uint32_t splits; };  // [row][head][split][uk_pitch], [row][head][split][2]

template <typename TA>
__global__ void __launch_bounds__(128) latent_rows_kernel(const LatentArgs a, const float *__restrict__ qa, const RowMap rows, const LatentPart o) {
    __shared__ float sc[LR_KT];
    __shared__ float sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t split = blockIdx.x, h = blockIdx.y, r = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, L = a.kv_rank + a.rot_dim;
    const int32_t pos = rows.pos_of(r), slot = rows.slot_of(r), k0 = first_key(a, pos) + (int32_t)split * LR_KT, n = min(pos + 1 - k0, LR_KT);
    float *ml = o.ml + (((size_t)r * a.heads + h) * o.splits + split) * 2;
    if (n <= 0) return;  // the merge knows how many splits a row has
    const TA *c = reinterpret_cast<const TA *>(a.cache.rows);
    const float *qr = qa + ((size_t)r * a.heads + h) * a.cache.pitch;
    for (int32_t i = warp; i < n; i += 4) {
        const TA *kr = c + cache_row(a.cache, slot, k0 + i);
        float s = 0.0f;
        for (uint32_t j = lane; j < L; j += 32) s = fmaf(qr[j], ld_act(kr + j), s);
        s = warp_sum_f(s);
        if (lane == 0) sc[i] = s * a.scale;
    }
    __syncthreads();
    float m = -INFINITY;
    for (int32_t i = 0; i < n; i++) m = fmaxf(m, sc[i]);
    const float e = (int32_t)threadIdx.x < n ? expf(sc[threadIdx.x] - m) : 0.0f;
    const float l = block_sum_f(e, sh);
    __syncthreads();
    if ((int32_t)threadIdx.x < n) sc[threadIdx.x] = e;
    __syncthreads();
    float *po = o.part + (((size_t)r * a.heads + h) * o.splits + split) * a.uk_pitch;
    for (uint32_t j = threadIdx.x; j < a.kv_rank; j += blockDim.x) {
        float s = 0.0f;
        for (int32_t i = 0; i < n; i++) s = fmaf(sc[i], ld_act(c + cache_row(a.cache, slot, k0 + i) + j), s);
        po[j] = s;
    }
    if (threadIdx.x == 0) {
        ml[0] = m;
        ml[1] = l;
    }
}

// The same on the tensor cores (bf16 cache): 16 heads x 64 keys per CTA.  The fp32 query and the fp32 weights
// enter the products as two bf16 parts each.
__global__ void __launch_bounds__(128) latent_rows_mma_kernel(const LatentArgs a, const float *__restrict__ qa, const RowMap rows, const LatentPart o) {
    extern __shared__ __align__(16) uint8_t lrs[];
    __shared__ float Ss[16][LR_KT + 4];
    __shared__ __align__(16) bf16 Ph[16][LR_KT + 8], Pl[16][LR_KT + 8];
    const uint32_t split = blockIdx.x, h0 = blockIdx.y * 16, r = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t L = a.cache.pitch, P = L + 8, g8 = lane >> 2, t4 = lane & 3;
    bf16 *Cs = reinterpret_cast<bf16 *>(lrs), *Qh = Cs + LR_KT * P, *Ql = Qh + 16 * P;
    pdl_launch_dependents();
    pdl_wait();
    const int32_t pos = rows.pos_of(r), slot = rows.slot_of(r), k0 = first_key(a, pos) + (int32_t)split * LR_KT, n = min(pos + 1 - k0, LR_KT);
    if (n <= 0) return;
    const uint32_t sC = (uint32_t)__cvta_generic_to_shared(Cs), sQh = (uint32_t)__cvta_generic_to_shared(Qh), sQl = (uint32_t)__cvta_generic_to_shared(Ql);
    const bf16 *c = reinterpret_cast<const bf16 *>(a.cache.rows);
    for (uint32_t k = warp; k < LR_KT; k += 4) {  // a warp per cached row
        const bf16 *src = c + cache_row(a.cache, slot, k0 + (int32_t)k);
        for (uint32_t j = lane * 8; j < L; j += 256) {
            if ((int32_t)k < n) cp_async16(sC + (k * P + j) * 2, src + j);
            else *reinterpret_cast<uint4 *>(Cs + k * P + j) = make_uint4(0, 0, 0, 0);
        }
    }
    cp_async_commit();
    for (uint32_t h = warp; h < 16; h += 4) {
        const float *src = qa + ((size_t)r * a.heads + h0 + h) * L;
#pragma unroll 4
        for (uint32_t j = lane * 4; j < L; j += 128) {
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (h0 + h < a.heads) x = *reinterpret_cast<const float4 *>(src + j);
            uint2 hi, lo;
            split_bf16(x.x, x.y, hi.x, lo.x);
            split_bf16(x.z, x.w, hi.y, lo.y);
            *reinterpret_cast<uint2 *>(Qh + h * P + j) = hi;
            *reinterpret_cast<uint2 *>(Ql + h * P + j) = lo;
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    {
        float s[2][4] = {};
        for (uint32_t kk = 0; kk < L; kk += 16) {
            uint32_t qh[4], ql[4], b[4];
            ldsm_x4(qh, sQh + ((lane & 15) * P + kk + (lane >> 4) * 8) * 2);
            ldsm_x4(ql, sQl + ((lane & 15) * P + kk + (lane >> 4) * 8) * 2);
            ldsm_x4(b, sC + ((warp * 16 + (lane & 7) + (lane >> 4) * 8) * P + kk + ((lane >> 3) & 1) * 8) * 2);
            mma_bf16(s[0], qh, b[0], b[1]);
            mma_bf16(s[1], qh, b[2], b[3]);
            mma_bf16(s[0], ql, b[0], b[1]);
            mma_bf16(s[1], ql, b[2], b[3]);
        }
#pragma unroll
        for (int t = 0; t < 2; t++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t k = warp * 16 + t * 8 + 2 * t4 + (i & 1);
                Ss[g8 + 8 * (i >> 1)][k] = (int32_t)k < n ? s[t][i] * a.scale : -INFINITY;
            }
    }
    __syncthreads();
    {  // eight threads per head
        const uint32_t h = tid >> 3, j0 = (tid & 7) * 8;
        float m = -INFINITY, l = 0.0f, e[8];
#pragma unroll
        for (int j = 0; j < 8; j++) m = fmaxf(m, Ss[h][j0 + j]);
#pragma unroll
        for (int of = 4; of > 0; of >>= 1) m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, of));
#pragma unroll
        for (int j = 0; j < 8; j++) l += e[j] = expf(Ss[h][j0 + j] - m);
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
            uint32_t hi, lo;
            split_bf16(e[j], e[j + 1], hi, lo);
            *reinterpret_cast<uint32_t *>(&Ph[h][j0 + j]) = hi;
            *reinterpret_cast<uint32_t *>(&Pl[h][j0 + j]) = lo;
        }
#pragma unroll
        for (int of = 4; of > 0; of >>= 1) l += __shfl_xor_sync(0xFFFFFFFFu, l, of);
        if ((tid & 7) == 0 && h0 + h < a.heads) {
            float *ml = o.ml + (((size_t)r * a.heads + h0 + h) * o.splits + split) * 2;
            ml[0] = m;
            ml[1] = l;
        }
    }
    __syncthreads();
    const uint32_t sPh = (uint32_t)__cvta_generic_to_shared(&Ph[0][0]), sPl = (uint32_t)__cvta_generic_to_shared(&Pl[0][0]);
    uint32_t ph[LR_KT / 16][4], pl[LR_KT / 16][4];
#pragma unroll
    for (int kk = 0; kk < LR_KT / 16; kk++) {
        ldsm_x4(ph[kk], sPh + ((lane & 15) * (LR_KT + 8) + kk * 16 + (lane >> 4) * 8) * 2);
        ldsm_x4(pl[kk], sPl + ((lane & 15) * (LR_KT + 8) + kk * 16 + (lane >> 4) * 8) * 2);
    }
    for (uint32_t c0 = warp * 16; c0 < a.kv_rank; c0 += 64) {  // a row of Cs is a multiple of 16 wide
        float acc[2][4] = {};
#pragma unroll
        for (int kk = 0; kk < LR_KT / 16; kk++) {
            uint32_t b[4];
            ldsm_x4_t(b, sC + ((kk * 16 + (lane & 15)) * P + c0 + (lane >> 4) * 8) * 2);
            mma_bf16(acc[0], ph[kk], b[0], b[1]);
            mma_bf16(acc[1], ph[kk], b[2], b[3]);
            mma_bf16(acc[0], pl[kk], b[0], b[1]);
            mma_bf16(acc[1], pl[kk], b[2], b[3]);
        }
#pragma unroll
        for (int t = 0; t < 2; t++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t h = h0 + g8 + 8 * (i >> 1), j = c0 + t * 8 + 2 * t4 + (i & 1);
                if (h < a.heads && j < a.kv_rank) o.part[(((size_t)r * a.heads + h) * o.splits + split) * a.uk_pitch + j] = acc[t][i];
            }
    }
}

// Merges a head's splits, applies W_uv and the gate.  Grid: (head, 32 value columns, row).
constexpr int LO_PRE = 2;  // 256-column pieces of W_uv rows requested before the dependency wait
template <typename TA>
__global__ void __launch_bounds__(128) latent_out_kernel(const LatentArgs a, const LatentPart o, const RowMap rows, const TA *__restrict__ gate,
                                                         uint32_t gate_pitch, TA *__restrict__ out, uint32_t out_pitch) {
    extern __shared__ float los[];  // [uk_pitch] weighted latent, then maxima and sums of the splits
    pdl_launch_dependents();
    const uint32_t h = blockIdx.x, v0 = blockIdx.y * 32, r = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const bf16 *wv = a.uv + ((size_t)h * a.vdim + v0 + warp) * a.uk_pitch + lane * 8;  // this warp: value columns v0 + warp + 4 i
    uint4 pre[8][LO_PRE];
#pragma unroll
    for (int i = 0; i < 8; i++)
#pragma unroll
        for (int k = 0; k < LO_PRE; k++) {
            pre[i][k] = make_uint4(0, 0, 0, 0);
            if (v0 + warp + 4 * i < a.vdim && lane * 8 + 256 * k < a.uk_pitch)
                pre[i][k] = __ldg(reinterpret_cast<const uint4 *>(wv + (size_t)4 * i * a.uk_pitch + 256 * k));
        }
    pdl_wait();
    const int32_t pos = rows.pos_of(r);
    const uint32_t n = (uint32_t)(pos + 1 - first_key(a, pos) + LR_KT - 1) / LR_KT;
    const float *ml = o.ml + ((size_t)r * a.heads + h) * o.splits * 2, *part = o.part + ((size_t)r * a.heads + h) * o.splits * a.uk_pitch;
    float *ol = los, *mls = los + a.uk_pitch;
    for (uint32_t i = threadIdx.x; i < 2 * n; i += blockDim.x) mls[i] = ml[i];
    __syncthreads();
    float m = -INFINITY, l = 0.0f;
    for (uint32_t s = 0; s < n; s++) m = fmaxf(m, mls[2 * s]);
    for (uint32_t s = 0; s < n; s++) l = fmaf(mls[2 * s + 1], expf(mls[2 * s] - m), l);
    const float inv = 1.0f / l;
    for (uint32_t j = threadIdx.x; j < a.uk_pitch; j += blockDim.x) {
        float x = 0.0f;
        if (j < a.kv_rank) {
#pragma unroll 4
            for (uint32_t s = 0; s < n; s++) x = fmaf(expf(mls[2 * s] - m) * inv, part[(size_t)s * a.uk_pitch + j], x);
        }
        ol[j] = x;
    }
    __syncthreads();
    auto dot = [&](const uint4 &w4, uint32_t j) {
        const bf16 *e = reinterpret_cast<const bf16 *>(&w4);
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) s = fmaf(__bfloat162float(e[i]), ol[j + i], s);
        return s;
    };
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const uint32_t v = v0 + warp + 4 * i;
        if (v >= a.vdim) break;
        float s = 0.0f;
#pragma unroll
        for (int k = 0; k < LO_PRE; k++)
            if (lane * 8 + 256 * k < a.uk_pitch) s += dot(pre[i][k], lane * 8 + 256 * k);
        for (uint32_t j = lane * 8 + 256 * LO_PRE; j < a.uk_pitch; j += 256)
            s += dot(__ldg(reinterpret_cast<const uint4 *>(a.uv + ((size_t)h * a.vdim + v) * a.uk_pitch + j)), j);
        s = warp_sum_f(s);
        if (lane == 0) {
            const uint32_t c = h * a.vdim + v;
            st_act(out + (size_t)r * out_pitch + c, s * ld_act(gate + (size_t)r * gate_pitch + c));
        }
    }
}

uint32_t latent_rows_splits(const LatentArgs &a, uint32_t max_seq) {
    const uint32_t keys = a.window ? std::min(a.window, max_seq) : max_seq;
    return (keys + LR_KT - 1) / LR_KT;
}
size_t latent_rows_scratch_floats(const LatentArgs &a, uint32_t splits, size_t *qa, size_t *part, size_t *ml) {
    *qa = round_up_u32(a.heads * a.cache.pitch, 4);
    *part = round_up_u32(a.heads * splits * a.uk_pitch, 4);
    *ml = round_up_u32(a.heads * splits * 2, 4);
    return *qa + *part + *ml;
}
constexpr size_t LR_SMEM_MAX = 200 * 1024;

int launch_latent_rows(prism_cuda_ctx *ctx, const LatentArgs &a, const LatentRowsScratch &s, const void *q, uint32_t q_pitch, const void *dkv,
                       uint32_t dkv_pitch, const void *gate, uint32_t gate_pitch, void *out, uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool act32) {
    const LatentPart p{s.part, s.ml, s.splits};
    const dim3 gq(a.heads + 1, (a.uk_pitch + 127) / 128, (n_rows + LQ_ROWS - 1) / LQ_ROWS), gout(a.heads, (a.vdim + 31) / 32, n_rows);
    const size_t osm = ((size_t)a.uk_pitch + 2 * s.splits) * 4;
    if (osm > 48 * 1024 || n_rows > s.rows_cap) return fail(ctx, PRISM_E_ARG, "latent attention: sizes beyond the kernel's scratch");
    if (act32) {
        launch_pdl(ctx, "latent_query_kernel", latent_query_kernel<float>, gq, 256, 0, a, (const float *)q, q_pitch, (const float *)dkv, dkv_pitch, rows, n_rows, s.qa);
        PRISM_TRY(after_launch(ctx, "latent_query_kernel"));
        launch_pdl(ctx, "latent_rows_kernel", latent_rows_kernel<float>, dim3(s.splits, a.heads, n_rows), 128, 0, a, (const float *)s.qa, rows, p);
        PRISM_TRY(after_launch(ctx, "latent_rows_kernel"));
        launch_pdl(ctx, "latent_out_kernel", latent_out_kernel<float>, gout, 128, osm, a, p, rows, (const float *)gate, gate_pitch, (float *)out, out_pitch);
        return after_launch(ctx, "latent_out_kernel");
    }
    launch_pdl(ctx, "latent_query_kernel", latent_query_kernel<bf16>, gq, 256, 0, a, (const bf16 *)q, q_pitch, (const bf16 *)dkv, dkv_pitch, rows, n_rows, s.qa);
    PRISM_TRY(after_launch(ctx, "latent_query_kernel"));
    const size_t msm = (size_t)(LR_KT + 32) * (a.cache.pitch + 8) * 2;
    if (msm <= LR_SMEM_MAX) {
        static bool configured[PRISM_MAX_DEVICES] = {false};
        if (!configured[ctx->device]) {
            PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(latent_rows_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LR_SMEM_MAX));
            configured[ctx->device] = true;
        }
        launch_pdl(ctx, "latent_rows_mma_kernel", latent_rows_mma_kernel, dim3(s.splits, (a.heads + 15) / 16, n_rows), 128, msm, a, (const float *)s.qa, rows, p);
        PRISM_TRY(after_launch(ctx, "latent_rows_mma_kernel"));
    } else {
        launch_pdl(ctx, "latent_rows_kernel", latent_rows_kernel<bf16>, dim3(s.splits, a.heads, n_rows), 128, 0, a, (const float *)s.qa, rows, p);
        PRISM_TRY(after_launch(ctx, "latent_rows_kernel"));
    }
    launch_pdl(ctx, "latent_out_kernel", latent_out_kernel<bf16>, gout, 128, osm, a, p, rows, (const bf16 *)gate, gate_pitch, (bf16 *)out, out_pitch);
    return after_launch(ctx, "latent_out_kernel");
}

// ---- expanded: prompt portions -------------------------------------------------------------------------
// Cache rows of positions lo .. lo+n-1 as contiguous latents (the input of the expansion) and rotated keys.
__global__ void __launch_bounds__(128) latent_gather_kernel(const LatentArgs a, int32_t slot, uint32_t lo, bf16 *__restrict__ lat, uint32_t lat_pitch,
                                                            bf16 *__restrict__ krot) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.x;
    const bf16 *c = reinterpret_cast<const bf16 *>(a.cache.rows) + cache_row(a.cache, slot, (int32_t)(lo + r));
    for (uint32_t i = threadIdx.x; i < lat_pitch; i += blockDim.x) lat[(size_t)r * lat_pitch + i] = i < a.kv_rank ? c[i] : __float2bfloat16_rn(0.0f);
    for (uint32_t i = threadIdx.x; i < a.rot_dim; i += blockDim.x) krot[(size_t)r * a.rot_dim + i] = c[a.kv_rank + i];
}
int launch_latent_gather(prism_cuda_ctx *ctx, const LatentArgs &a, int32_t slot, uint32_t lo, uint32_t n, bf16 *lat, uint32_t lat_pitch, bf16 *krot) {
    launch_pdl(ctx, "latent_gather_kernel", latent_gather_kernel, n, 128, 0, a, slot, lo, lat, lat_pitch, krot);
    return after_launch(ctx, "latent_gather_kernel");
}

constexpr int LP_Q = 128, LP_THREADS = 256;
static size_t tiled_attn_smem(const TiledAttn &a, uint32_t vd, uint32_t kt) {
    const uint32_t dq = round_up_u32(a.dim + a.rot_dim, 16);
    return ((size_t)(LP_Q + 2 * kt) * (dq + 8) + (size_t)2 * kt * (vd + 8)) * 2;
}

// 128 queries of one head per CTA (16 per warp), key tiles of LP_K in two buffers, online softmax in fp32; the
// weights enter the second product as two bf16 parts.  Key and value heads start at multiples of 8 and may be
// shared by a group of query heads; rows of a ring are taken by position.  The last queries, which see most, go first.
template <int VD, int LP_K, int MIN_CTAS>
__global__ void __launch_bounds__(LP_THREADS, MIN_CTAS) tiled_attn_kernel(const TiledAttn a) {
    extern __shared__ __align__(16) uint8_t lps[];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t h = blockIdx.x, kh = h / a.group, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t dq = a.dim + a.rot_dim, dqp = round_up_u32(dq, 16), PQ = dqp + 8;
    constexpr uint32_t PV = VD + 8;
    bf16 *Qs = reinterpret_cast<bf16 *>(lps), *Ks = Qs + LP_Q * PQ, *Vs = Ks + 2 * LP_K * PQ;
    const uint32_t sQ = (uint32_t)__cvta_generic_to_shared(Qs), sK = (uint32_t)__cvta_generic_to_shared(Ks), sV = (uint32_t)__cvta_generic_to_shared(Vs);
    const uint32_t q0 = (gridDim.y - 1 - blockIdx.y) * LP_Q, nq = min((uint32_t)LP_Q, a.n_rows - q0);
    const int32_t first = max((int32_t)a.lo, window_first(a.window, (int32_t)(a.pos0 + q0)));
    const int32_t end = (int32_t)(a.pos0 + q0 + nq);  // keys first .. end-1
    const uint32_t n_kt = ((uint32_t)(end - first) + LP_K - 1) / LP_K;
    const uint4 z4 = make_uint4(0, 0, 0, 0);
    const uint32_t d8 = (a.dim + 7) / 8, r8 = a.rot_dim / 8, q8 = dqp / 8, v8 = (a.vdim + 7) / 8;
    const bool q_vec = !((a.dim | a.q_pitch) & 7) && !(reinterpret_cast<uintptr_t>(a.q) & 15);

    auto load_keys = [&](uint32_t kt, uint32_t buf) {
        const int32_t k0 = first + (int32_t)(kt * LP_K);
        const uint32_t row0 = a.ring ? (uint32_t)k0 % a.ring : (uint32_t)k0 - a.lo;
        auto row_of = [&](uint32_t r) { return a.ring && row0 + r >= a.ring ? row0 + r - a.ring : row0 + r; };  // the visible keys fit into the ring
        for (uint32_t r = tid >> a.shift; r < LP_K; r += LP_THREADS >> a.shift) {
            const bool on = k0 + (int32_t)r < end;
            const size_t row = row_of(r);
            for (uint32_t c = tid & ((1u << a.shift) - 1); c < q8; c += 1u << a.shift) {
                const uint32_t at = (buf * LP_K + r) * PQ + c * 8;
                if (on && c < d8) cp_async16(sK + at * 2, a.kx + row * a.kx_pitch + kh * a.kx_head + c * 8);
                else if (on && c < d8 + r8) cp_async16(sK + at * 2, a.krot + row * a.rot_dim + (c - d8) * 8);
                else *reinterpret_cast<uint4 *>(Ks + at) = z4;
            }
        }
        for (uint32_t i = tid; i < LP_K * (VD / 8); i += LP_THREADS) {
            const uint32_t r = i / (VD / 8), c = i % (VD / 8), at = (buf * LP_K + r) * PV + c * 8;
            const int32_t key = k0 + (int32_t)r;
            if (key < end && c < v8) cp_async16(sV + at * 2, a.vx + (size_t)row_of(r) * a.vx_pitch + kh * a.vx_head + c * 8);
            else *reinterpret_cast<uint4 *>(Vs + at) = z4;
        }
        cp_async_commit();
    };
    load_keys(0, 0);
    for (uint32_t i = tid; i < LP_Q * q8; i += LP_THREADS) {
        const uint32_t r = i / q8, c = i % q8;
        const bf16 *src = a.q + (size_t)(q0 + r) * a.q_pitch + h * dq + c * 8;
        uint4 x = z4;
        if (r < nq && q_vec) {
            if (c < d8 + r8) x = *reinterpret_cast<const uint4 *>(src);
        } else if (r < nq) {
#pragma unroll
            for (uint32_t j = 0; j < 8; j++)
                if (c * 8 + j < dq) reinterpret_cast<bf16 *>(&x)[j] = src[j];
        }
        *reinterpret_cast<uint4 *>(Qs + r * PQ + c * 8) = x;
    }
    __syncthreads();
    for (uint32_t i = tid; i < nq * a.rot_pairs; i += LP_THREADS) {
        const uint32_t r = i / a.rot_pairs, j = i % a.rot_pairs;
        bf16 *u = Qs + r * PQ + a.dim + j, *v = u + a.rot_pairs;
        float x = __bfloat162float(*u), y = __bfloat162float(*v);
        rotate_pair(a.rot_freq, a.rot_mul, (int32_t)(a.pos0 + q0 + r), j, x, y);
        *u = __float2bfloat16_rn(x);
        *v = __float2bfloat16_rn(y);
    }
    float acc[VD / 8][4];
#pragma unroll
    for (int n = 0; n < VD / 8; n++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[n][i] = 0.0f;
    float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.0f, 0.0f};
    const float sc2 = a.scale * 1.4426950408889634f;
    const int32_t wq0 = (int32_t)(a.pos0 + q0 + warp * 16);  // positions of this warp's queries: wq0 .. wq0+15
    for (uint32_t kt = 0; kt < n_kt; kt++) {
        const uint32_t buf = kt & 1;
        if (kt + 1 < n_kt) {
            load_keys(kt + 1, buf ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int32_t k0 = first + (int32_t)(kt * LP_K);
        const bool none = k0 > wq0 + 15 || k0 + LP_K - 1 < window_first(a.window, wq0) || warp * 16 >= nq;
        if (!none) {
            float s[LP_K / 8][4];
#pragma unroll
            for (int n = 0; n < LP_K / 8; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) s[n][i] = 0.0f;
            for (uint32_t kk = 0; kk < dqp; kk += 16) {
                uint32_t aq[4];
                ldsm_x4(aq, sQ + ((warp * 16 + (lane & 15)) * PQ + kk + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int n = 0; n < LP_K / 16; n++) {
                    uint32_t b[4];
                    ldsm_x4(b, sK + ((buf * LP_K + n * 16 + (lane & 7) + (lane >> 4) * 8) * PQ + kk + ((lane >> 3) & 1) * 8) * 2);
                    mma_bf16(s[2 * n], aq, b[0], b[1]);
                    mma_bf16(s[2 * n + 1], aq, b[2], b[3]);
                }
            }
            const bool edge = k0 + LP_K - 1 > wq0 || (a.window && k0 < window_first(a.window, wq0 + 15));
            float mx[2] = {mrow[0], mrow[1]};
#pragma unroll
            for (int n = 0; n < LP_K / 8; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    s[n][i] *= sc2;
                    if (edge) {
                        const int32_t key = k0 + n * 8 + (int32_t)(2 * t4) + (i & 1), qp = wq0 + (int32_t)g8 + 8 * (i >> 1);
                        if (key > qp || (a.window && qp - key >= (int32_t)a.window)) s[n][i] = -INFINITY;
                    }
                    mx[i >> 1] = fmaxf(mx[i >> 1], s[n][i]);
                }
#pragma unroll
            for (int i = 0; i < 2; i++) {
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xFFFFFFFFu, mx[i], 1));
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xFFFFFFFFu, mx[i], 2));
                const float ref = mx[i] == -INFINITY ? 0.0f : mx[i];  // no key of this row so far
                const float f = exp2f(mrow[i] - ref);
                mrow[i] = mx[i];
                mx[i] = ref;
                lrow[i] *= f;
#pragma unroll
                for (int n = 0; n < VD / 8; n++) {
                    acc[n][2 * i] *= f;
                    acc[n][2 * i + 1] *= f;
                }
            }
#pragma unroll
            for (int n = 0; n < LP_K / 8; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    s[n][i] = exp2f(s[n][i] - mx[i >> 1]);
                    lrow[i >> 1] += s[n][i];
                }
#pragma unroll
            for (int kk = 0; kk < LP_K / 16; kk++) {
                uint32_t ph[4], pl[4];
                split_bf16(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
                split_bf16(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
                split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
                split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
                for (int n = 0; n < VD / 16; n++) {
                    uint32_t b[4];
                    ldsm_x4_t(b, sV + ((buf * LP_K + kk * 16 + (lane & 15)) * PV + n * 16 + (lane >> 4) * 8) * 2);
                    mma_bf16(acc[2 * n], ph, b[0], b[1]);
                    mma_bf16(acc[2 * n + 1], ph, b[2], b[3]);
                    mma_bf16(acc[2 * n], pl, b[0], b[1]);
                    mma_bf16(acc[2 * n + 1], pl, b[2], b[3]);
                }
            }
        }
        __syncthreads();  // this buffer is filled again in the next round
    }
#pragma unroll
    for (int i = 0; i < 2; i++) {
        lrow[i] += __shfl_xor_sync(0xFFFFFFFFu, lrow[i], 1);
        lrow[i] += __shfl_xor_sync(0xFFFFFFFFu, lrow[i], 2);
        const uint32_t r = warp * 16 + g8 + 8 * i;
        if (r >= nq) continue;
        const float inv = 1.0f / lrow[i];
        const size_t row = q0 + r;
#pragma unroll
        for (int n = 0; n < VD / 8; n++) {
            const uint32_t c = n * 8 + 2 * t4;
            const uint32_t at = h * a.vdim + c;
            float o0 = acc[n][2 * i] * inv, o1 = acc[n][2 * i + 1] * inv;
            if (a.vdim & 1) {  // no gate
                if (c < a.vdim) st_act(a.out + row * a.out_pitch + at, o0);
                if (c + 1 < a.vdim) st_act(a.out + row * a.out_pitch + at + 1, o1);
            } else if (c < a.vdim) {
                if (a.gate) {
                    const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(a.gate + row * a.gate_pitch + at));
                    o0 *= g.x;
                    o1 *= g.y;
                }
                *reinterpret_cast<uint32_t *>(a.out + row * a.out_pitch + at) = pack_bf16(o0, o1);
            }
        }
    }
}

template <int VD, int KT, int MIN_CTAS>
static int launch_ta(prism_cuda_ctx *ctx, const TiledAttn &p) {
    static bool configured[PRISM_MAX_DEVICES] = {false};
    if (!configured[ctx->device]) {
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(tiled_attn_kernel<VD, KT, MIN_CTAS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 208 * 1024));
        configured[ctx->device] = true;
    }
    launch_pdl(ctx, "tiled_attn_kernel", tiled_attn_kernel<VD, KT, MIN_CTAS>, dim3(p.heads, (p.n_rows + LP_Q - 1) / LP_Q), LP_THREADS, tiled_attn_smem(p, VD, KT), p);
    return after_launch(ctx, "tiled_attn_kernel");
}
bool tiled_attn_ok(uint32_t dim, uint32_t vdim) { return dim <= 256 && vdim <= 256; }
int launch_tiled_attn(prism_cuda_ctx *ctx, const TiledAttn &args) {
    TiledAttn p = args;
    p.shift = row_shift(round_up_u32(p.dim + p.rot_dim, 16) / 8);
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(p.kx) | reinterpret_cast<uintptr_t>(p.vx) | reinterpret_cast<uintptr_t>(p.krot);
    if (!tiled_attn_ok(p.dim + p.rot_dim, p.vdim) || (ptrs & 15) || p.kx_pitch % 8 || p.vx_pitch % 8 || p.kx_head % 8 || p.vx_head % 8 || p.rot_dim % 8 ||
        (p.rot_dim && p.dim % 8) || p.out_pitch % 2 || (p.gate && (p.gate_pitch % 2 || p.vdim % 2)))
        return fail(ctx, PRISM_E_ARG, "tiled attention: keys and values need 16-byte rows and heads of at most 256");
    if (p.vdim <= 64) return launch_ta<64, 64, 2>(ctx, p);
    if (p.vdim <= 128) return launch_ta<128, 32, 2>(ctx, p);
    return launch_ta<256, 64, 1>(ctx, p);
}

bool latent_expand_ok(const LatentArgs &a) {
    return a.dim % 8 == 0 && a.rot_dim % 8 == 0 && a.vdim % 8 == 0 && tiled_attn_ok(a.dim + a.rot_dim, a.vdim);
}

int launch_latent_prefill(prism_cuda_ctx *ctx, const LatentArgs &a, const bf16 *q, uint32_t q_pitch, const bf16 *kx, uint32_t kx_pitch,
                          const bf16 *vx, uint32_t vx_pitch, const bf16 *krot, uint32_t lo, const bf16 *gate, uint32_t gate_pitch, bf16 *out,
                          uint32_t out_pitch, uint32_t pos0, uint32_t n_rows) {
    TiledAttn p{};
    p.heads = a.heads; p.group = 1; p.dim = a.dim; p.rot_dim = a.rot_dim; p.rot_pairs = a.rot_pairs; p.vdim = a.vdim; p.window = a.window;
    p.scale = a.scale; p.rot_mul = a.rot_mul; p.rot_freq = a.rot_freq;
    p.q = q; p.kx = kx; p.vx = vx; p.krot = krot; p.gate = gate; p.out = out;
    p.q_pitch = q_pitch; p.kx_pitch = kx_pitch; p.vx_pitch = vx_pitch; p.gate_pitch = gate_pitch; p.out_pitch = out_pitch;
    p.kx_head = a.dim; p.vx_head = a.vdim;
    p.lo = lo; p.pos0 = pos0; p.n_rows = n_rows;
    return launch_tiled_attn(ctx, p);
}

}  // namespace prism
