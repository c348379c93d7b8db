// Gated delta rule: one decay g and one step size beta per head and token, the state S in fp32,
//   S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q,
// q, k, v after a short convolution and silu, q and k as unit vectors (q times dim^-1/2), o normed per head,
// weighted and gated.
//   step   one token of every row: convolution, recurrence, norm and gate in one kernel (a cluster per head)
//   seq    consecutive tokens one by one: short portions, 32-bit runs, unusual sizes
//   chunk  prompts: per chunk of 64 tokens the triangular system of the u is solved for all value columns at once
//          (delta_prep_kernel, every chunk in parallel), then the chunks run one after the other on the tensor cores
#include <cooperative_groups.h>

#include <algorithm>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace prism {

constexpr int DL_THREADS = 256, DL_VS = 32;  // value columns of a slice
constexpr float DL_UNIT_EPS = 1e-6f;

__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float log_decay(const DeltaArgs &a, const float *ba, uint32_t h) {
    return -expf(a.a_log[h]) * softplus_f(ba[a.heads + h] + a.dt_bias[h]);
}

// ---- decode ----------------------------------------------------------------------------------------------
// silu(conv) of channel c at position pos as the activation type holds it; cur: its projection at pos.
template <typename TA>
__device__ __forceinline__ float short_conv(const DeltaArgs &a, const TA *ring, uint32_t c, int32_t pos, float cur) {
    const uint32_t C = a.channels;
    const int32_t T = (int32_t)a.taps - 1;
    float s = a.conv_w[(size_t)T * C + c] * cur;
    for (int32_t j = max(0, T - pos); j < T; j++) s = fmaf(a.conv_w[(size_t)j * C + c], ld_act(ring + (size_t)((uint32_t)(pos - T + j) % a.taps) * C + c), s);
    TA y;
    st_act(&y, s * sigmoid_f(s));
    return ld_act(&y);
}

// Grid: (CTAs of a cluster, head, row).  A CTA takes every cs-th slice of 32 value columns; thread (d group, column)
// holds NJ state values of its column in registers (NJ 0: reads them twice).
template <typename TA, int NJ>
__global__ void __launch_bounds__(DL_THREADS) delta_step_kernel(const DeltaArgs a, const RowMap rows, uint32_t cs) {
    extern __shared__ float dsm[];
    __shared__ float red[2][8][DL_VS + 1], sh[32], part;
    pdl_launch_dependents();
    if (!a.beside) pdl_wait();
    const uint32_t rank = blockIdx.x, h = blockIdx.y, r = blockIdx.z, tid = threadIdx.x, vl = tid & 31, dg = tid >> 5;
    const uint32_t group = a.heads / a.kv_heads, kh = h / group, C = a.channels, qk = a.kv_heads * a.dim;
    const int32_t pos = rows.pos_of(r), slot = rows.slot_of(r);
    TA *ring = reinterpret_cast<TA *>(a.ring) + (size_t)slot * a.taps * C, *now = ring + (size_t)((uint32_t)pos % a.taps) * C;
    float *qs = dsm, *ks = dsm + a.dim, *os = ks + a.dim;
    const uint32_t n_slices = (a.vdim + DL_VS - 1) / DL_VS;
    float *S0 = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim;
    float s[NJ ? NJ : 1];
    auto load_state = [&](uint32_t v) {
#pragma unroll
        for (int j = 0; j < NJ; j++) {
            const uint32_t d = dg + 8 * j;
            s[j] = d < a.dim && v < a.vdim ? S0[(size_t)d * a.vdim + v] : 0.0f;
        }
    };
    load_state(rank * DL_VS + vl);
    const float *ba = a.ba + (size_t)r * a.ba_pitch;
    const float beta = sigmoid_f(ba[h]), g = expf(log_decay(a, ba, h));
    float sq = 0.0f, sk = 0.0f;
    for (uint32_t d = tid; d < a.dim; d += DL_THREADS) {
        const uint32_t c = kh * a.dim + d;
        const TA qc = reinterpret_cast<const TA *>(a.q)[(size_t)r * a.pitch + c], kc = reinterpret_cast<const TA *>(a.k)[(size_t)r * a.pitch + c];
        const float q = short_conv(a, ring, c, pos, ld_act(&qc)), k = short_conv(a, ring, qk + c, pos, ld_act(&kc));
        qs[d] = q;
        ks[d] = k;
        sq = fmaf(q, q, sq);
        sk = fmaf(k, k, sk);
        if (rank == 0 && h % group == 0) {  // the row of `pos` is none of those that are read
            now[c] = qc;
            now[qk + c] = kc;
        }
    }
    sq = warp_sum_f(sq);
    sk = warp_sum_f(sk);
    if (vl == 0) {
        sh[dg] = sq;
        sh[8 + dg] = sk;
    }
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int e = 0; e < 8; e++) {
        sq += sh[e];
        sk += sh[8 + e];
    }
    const float rq = 1.0f / (sqrtf(sq + DL_UNIT_EPS) * sqrtf((float)a.dim)), rk = 1.0f / sqrtf(sk + DL_UNIT_EPS);
    float ss = 0.0f;
    for (uint32_t sl = rank, i = 0; sl < n_slices; sl += cs, i++) {
        const uint32_t v = sl * DL_VS + vl, c = 2 * qk + h * a.vdim + v;
        const bool on = v < a.vdim;
        float *S = S0 + v, vv = 0.0f, acc = 0.0f;
        if (i) load_state(v);
        if (on) {
            const TA vc = reinterpret_cast<const TA *>(a.v)[(size_t)r * a.pitch + h * a.vdim + v];
            vv = short_conv(a, ring, c, pos, ld_act(&vc));
            if (dg == 0) now[c] = vc;
        }
        if (NJ) {
#pragma unroll
            for (int j = 0; j < NJ; j++)
                if (dg + 8 * j < a.dim) acc = fmaf(ks[dg + 8 * j], s[j], acc);
        } else if (on) {
            for (uint32_t d = dg; d < a.dim; d += 8) acc = fmaf(ks[d], S[(size_t)d * a.vdim], acc);
        }
        red[0][dg][vl] = acc;
        __syncthreads();
        float kS = 0.0f;
#pragma unroll
        for (int e = 0; e < 8; e++) kS += red[0][e][vl];
        const float u = beta * (vv - g * kS * rk) * rk;  // times k's factor, once
        acc = 0.0f;
        if (NJ) {
#pragma unroll
            for (int j = 0; j < NJ; j++) {
                const uint32_t d = dg + 8 * j;
                if (d < a.dim) {
                    const float x = fmaf(g, s[j], ks[d] * u);
                    if (on) S[(size_t)d * a.vdim] = x;
                    acc = fmaf(qs[d], x, acc);
                }
            }
        } else if (on) {
            for (uint32_t d = dg; d < a.dim; d += 8) {
                const float x = fmaf(g, S[(size_t)d * a.vdim], ks[d] * u);
                S[(size_t)d * a.vdim] = x;
                acc = fmaf(qs[d], x, acc);
            }
        }
        red[1][dg][vl] = acc;
        __syncthreads();
        if (dg == 0) {
            float o = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; e++) o += red[1][e][vl];
            o = on ? o * rq : 0.0f;
            os[i * DL_VS + vl] = o;
            ss = fmaf(o, o, ss);
        }
    }
    ss = block_sum_f(ss, sh);
    if (cs > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        if (tid == 0) part = ss;
        cluster.sync();
        ss = 0.0f;
        for (uint32_t e = 0; e < cs; e++) ss += *cluster.map_shared_rank(&part, e);
    }
    const float inv = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
    for (uint32_t sl = rank + dg * cs, i = dg; sl < n_slices; sl += 8 * cs, i += 8) {
        const uint32_t v = sl * DL_VS + vl;
        if (v < a.vdim)
            st_act(reinterpret_cast<TA *>(a.o) + (size_t)r * a.o_pitch + h * a.vdim + v,
                   os[i * DL_VS + vl] * inv * a.norm[v] * ld_act(reinterpret_cast<const TA *>(a.gate) + (size_t)r * a.gate_pitch + h * a.vdim + v));
    }
    if (cs > 1) cg::this_cluster().sync();  // the peers read this CTA's sum
    if (a.beside) pdl_wait();  // the kernel after this one relies on the one before it too
}

template <typename TA>
static int run_step(prism_cuda_ctx *ctx, const DeltaArgs &a, const RowMap &rows) {
    const uint32_t n_slices = (a.vdim + DL_VS - 1) / DL_VS, cs = std::min(n_slices, 8u);
    const size_t smem = ((size_t)2 * a.dim + (size_t)((n_slices + cs - 1) / cs) * DL_VS) * 4;
    if (smem > 48 * 1024) return fail(ctx, PRISM_E_ARG, "gated delta: head too large");
    const dim3 grid(cs, a.heads, a.rows);
    if (a.dim <= 64) launch_cluster_pdl(ctx, delta_step_kernel<TA, 8>, grid, DL_THREADS, smem, cs, a, rows, cs);
    else if (a.dim <= 128) launch_cluster_pdl(ctx, delta_step_kernel<TA, 16>, grid, DL_THREADS, smem, cs, a, rows, cs);
    else if (a.dim <= 256) launch_cluster_pdl(ctx, delta_step_kernel<TA, 32>, grid, DL_THREADS, smem, cs, a, rows, cs);
    else launch_cluster_pdl(ctx, delta_step_kernel<TA, 0>, grid, DL_THREADS, smem, cs, a, rows, cs);
    return after_launch(ctx, "delta_step_kernel");
}
int launch_delta_step(prism_cuda_ctx *ctx, const DeltaArgs &a, const RowMap &rows, bool act32) {
    return act32 ? run_step<float>(ctx, a, rows) : run_step<bf16>(ctx, a, rows);
}

// ---- consecutive tokens, one by one ------------------------------------------------------------------------
// Grid: (slice of 32 value columns, head); the slice of the state in shared memory.  q, k, v are convolved already.
template <typename TA>
__global__ void __launch_bounds__(DL_THREADS) delta_seq_kernel(const DeltaArgs a, int32_t slot) {
    extern __shared__ float dsm[];
    __shared__ float red[2][8][DL_VS + 1], sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t h = blockIdx.y, kh = h / (a.heads / a.kv_heads), tid = threadIdx.x, vl = tid & 31, v = blockIdx.x * DL_VS + vl, dg = tid >> 5;
    float *qs = dsm, *ks = qs + a.dim, *ss = ks + a.dim;
    float *S = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim;
    const bool on = v < a.vdim;
    for (uint32_t d = dg; d < a.dim; d += 8) ss[d * DL_VS + vl] = on ? S[(size_t)d * a.vdim + v] : 0.0f;
    for (uint32_t r = 0; r < a.rows; r++) {
        const float *ba = a.ba + (size_t)r * a.ba_pitch;
        float sq = 0.0f, sk = 0.0f;
        __syncthreads();
        for (uint32_t d = tid; d < a.dim; d += DL_THREADS) {
            const float q = ld_act(reinterpret_cast<const TA *>(a.q) + (size_t)r * a.pitch + kh * a.dim + d);
            const float k = ld_act(reinterpret_cast<const TA *>(a.k) + (size_t)r * a.pitch + kh * a.dim + d);
            qs[d] = q;
            ks[d] = k;
            sq = fmaf(q, q, sq);
            sk = fmaf(k, k, sk);
        }
        const float vv = on ? ld_act(reinterpret_cast<const TA *>(a.v) + (size_t)r * a.pitch + h * a.vdim + v) : 0.0f;
        const float beta = sigmoid_f(ba[h]), g = expf(log_decay(a, ba, h));
        const float rq = 1.0f / (sqrtf(block_sum_f(sq, sh) + DL_UNIT_EPS) * sqrtf((float)a.dim)), rk = 1.0f / sqrtf(block_sum_f(sk, sh) + DL_UNIT_EPS);
        float acc = 0.0f;
        for (uint32_t d = dg; d < a.dim; d += 8) acc = fmaf(ks[d], ss[d * DL_VS + vl], acc);
        red[0][dg][vl] = acc;
        __syncthreads();
        float kS = 0.0f;
#pragma unroll
        for (int e = 0; e < 8; e++) kS += red[0][e][vl];
        const float u = beta * (vv - g * kS * rk) * rk;
        acc = 0.0f;
        for (uint32_t d = dg; d < a.dim; d += 8) {
            const float x = fmaf(g, ss[d * DL_VS + vl], ks[d] * u);
            ss[d * DL_VS + vl] = x;
            acc = fmaf(qs[d], x, acc);
        }
        red[1][dg][vl] = acc;
        __syncthreads();
        if (dg == 0 && on) {
            float o = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; e++) o += red[1][e][vl];
            a.o32[(size_t)r * a.heads * a.vdim + h * a.vdim + v] = o * rq;
        }
    }
    for (uint32_t d = dg; d < a.dim; d += 8)
        if (on) S[(size_t)d * a.vdim + v] = ss[d * DL_VS + vl];
}

// One warp per row and head: the output's norm over its head, weight and gate.  vec: four values of a lane at a time,
// kept in registers.
constexpr int DG_U = 2;  // vectors of a lane: heads of up to 256 values
template <typename TA>
__global__ void __launch_bounds__(DL_THREADS) delta_gate_kernel(const DeltaArgs a, uint32_t vec) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31, i = blockIdx.x * (DL_THREADS / 32) + (threadIdx.x >> 5);
    if (i >= a.rows * a.heads) return;
    const uint32_t r = i / a.heads, h = i % a.heads;
    const float *o = a.o32 + (size_t)i * a.vdim;
    const TA *gate = reinterpret_cast<const TA *>(a.gate) + (size_t)r * a.gate_pitch + h * a.vdim;
    TA *to = reinterpret_cast<TA *>(a.o) + (size_t)r * a.o_pitch + h * a.vdim;
    float ss = 0.0f;
    if (vec) {
        float4 x[DG_U], g[DG_U];
#pragma unroll
        for (int u = 0; u < DG_U; u++) {
            const uint32_t v = (lane + 32 * u) * 4;
            x[u] = v < a.vdim ? ld4(o + v) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (v < a.vdim) g[u] = ld4(gate + v);
            ss += x[u].x * x[u].x + x[u].y * x[u].y + x[u].z * x[u].z + x[u].w * x[u].w;
        }
        const float inv = 1.0f / sqrtf(warp_sum_f(ss) / (float)a.vdim + a.eps);
#pragma unroll
        for (int u = 0; u < DG_U; u++) {
            const uint32_t v = (lane + 32 * u) * 4;
            if (v >= a.vdim) break;
            const float4 w = ld4(a.norm + v);
            st4(to + v, make_float4(x[u].x * inv * w.x * g[u].x, x[u].y * inv * w.y * g[u].y, x[u].z * inv * w.z * g[u].z, x[u].w * inv * w.w * g[u].w));
        }
        return;
    }
    for (uint32_t v = lane; v < a.vdim; v += 32) ss = fmaf(o[v], o[v], ss);
    const float inv = 1.0f / sqrtf(warp_sum_f(ss) / (float)a.vdim + a.eps);
    for (uint32_t v = lane; v < a.vdim; v += 32) st_act(to + v, o[v] * inv * a.norm[v] * ld_act(gate + v));
}

// ---- prompts in chunks -------------------------------------------------------------------------------------
// Let L_i = log g_0 + .. + log g_i inside a chunk that starts with state S0, and k, q be unit vectors.  Then
//   u_i + sum_{j<i} beta_i e^(L_i-L_j) (k_i.k_j) u_j = beta_i (v_i - e^(L_i) S0^T k_i)        or  U = T (V - E K S0),
//   o_i = e^(L_i) S0^T q_i + sum_{j<=i} e^(L_i-L_j) (q_i.k_j) u_j                             or  O = F Q S0 + P U,
//   S   = e^(L_last) S0 + sum_j e^(L_last-L_j) k_j u_j^T,
// with T = (I + A)^-1 diag(beta).  The unit factors are scalars per row, so q and k themselves stay the bf16 values
// they are; everything else enters the tensor cores as two bf16 parts.
constexpr int DC_C = 64, DC_PV = DL_VS + 8, DC_PT = DC_C + 8, DC_PA = DC_C + 4, DC_PY = 36;
constexpr uint32_t DC_SCALARS = 256;                              // floats: e[64] f[64] w[64], last: e^(L_last)
constexpr size_t DC_ITEM = 4 * DC_C * DC_C * 2 + DC_SCALARS * 4;  // T hi, T lo, P hi, P lo, scalars

// Rows of a chunk into shared memory, zeros past row nt and column `valid`; 2^sh threads take a row.
template <int THREADS>
__device__ __forceinline__ void load_rows(bf16 *dst, uint32_t pitch, uint32_t cols, const bf16 *src, uint32_t src_pitch, uint32_t nt, uint32_t valid,
                                          bool vec, uint32_t sh) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(dst);
    if (vec) {
        for (uint32_t r = threadIdx.x >> sh; r < DC_C; r += THREADS >> sh)
            for (uint32_t c = (threadIdx.x & ((1u << sh) - 1)) * 8; c < cols; c += 8u << sh) {
                if (r < nt && c < valid) cp_async16(s + (r * pitch + c) * 2, src + (size_t)r * src_pitch + c);
                else *reinterpret_cast<uint4 *>(dst + r * pitch + c) = make_uint4(0, 0, 0, 0);
            }
    } else {
        for (uint32_t i = threadIdx.x; i < DC_C * cols; i += THREADS) {
            const uint32_t r = i / cols, c = i % cols;
            dst[r * pitch + c] = r < nt && c < valid ? src[(size_t)r * src_pitch + c] : __float2bfloat16_rn(0.0f);
        }
    }
}

__global__ void __launch_bounds__(DL_THREADS) delta_prep_kernel(const DeltaArgs a, uint32_t dpad, uint32_t vec, uint32_t sh) {
    extern __shared__ __align__(16) uint8_t dps[];
    __shared__ float L[DC_C], rq[DC_C], rk[DC_C], bt[DC_C];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t PD = dpad + 8, ch = blockIdx.x, h = blockIdx.y, kh = h / (a.heads / a.kv_heads), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t g8 = lane >> 2, t4 = lane & 3, r0 = ch * DC_C, nt = min((uint32_t)DC_C, a.rows - r0);
    constexpr uint32_t PA = DC_PA, PY = DC_PY;
    float *A = reinterpret_cast<float *>(dps), *X = A + DC_C * PA, *Y = X + DC_C * PA;  // X and Y share their place with Q and K
    bf16 *Q = reinterpret_cast<bf16 *>(X), *K = Q + DC_C * PD;
    const uint32_t sQ = (uint32_t)__cvta_generic_to_shared(Q), sK = (uint32_t)__cvta_generic_to_shared(K);
    load_rows<DL_THREADS>(Q, PD, dpad, reinterpret_cast<const bf16 *>(a.q) + (size_t)r0 * a.pitch + kh * a.dim, a.pitch, nt, a.dim, vec, sh);
    load_rows<DL_THREADS>(K, PD, dpad, reinterpret_cast<const bf16 *>(a.k) + (size_t)r0 * a.pitch + kh * a.dim, a.pitch, nt, a.dim, vec, sh);
    cp_async_commit();
    if (warp == 0) {  // running sums of the logarithms
        float carry = 0.0f;
#pragma unroll
        for (uint32_t i = lane; i < DC_C; i += 32) {
            const float *ba = a.ba + (size_t)(r0 + i) * a.ba_pitch;
            float x = i < nt ? fmaxf(log_decay(a, ba, h), -100.0f) : 0.0f;  // e^-100 is nothing; bounded, the sums keep their precision
            bt[i] = i < nt ? sigmoid_f(ba[h]) : 0.0f;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float y = __shfl_up_sync(0xFFFFFFFFu, x, o);
                if ((int)lane >= o) x += y;
            }
            L[i] = x + carry;
            carry += __shfl_sync(0xFFFFFFFFu, x, 31);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    {
        const uint32_t r = tid >> 2, s = tid & 3;
        float sq = 0.0f, sk = 0.0f;
        for (uint32_t d = s * 2; d < dpad; d += 8) {
            const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(Q + r * PD + d));
            const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(K + r * PD + d));
            sq += q.x * q.x + q.y * q.y;
            sk += k.x * k.x + k.y * k.y;
        }
        sq += __shfl_xor_sync(0xFFFFFFFFu, sq, 1);
        sk += __shfl_xor_sync(0xFFFFFFFFu, sk, 1);
        sq += __shfl_xor_sync(0xFFFFFFFFu, sq, 2);
        sk += __shfl_xor_sync(0xFFFFFFFFu, sk, 2);
        if (s == 0) {
            rq[r] = 1.0f / (sqrtf(sq + DL_UNIT_EPS) * sqrtf((float)a.dim));
            rk[r] = 1.0f / sqrtf(sk + DL_UNIT_EPS);
        }
    }
    __syncthreads();
    uint8_t *item = reinterpret_cast<uint8_t *>(a.chunk_scratch) + ((size_t)ch * a.heads + h) * DC_ITEM;
    bf16 *Th = reinterpret_cast<bf16 *>(item), *Tl = Th + DC_C * DC_C, *Ph = Tl + DC_C * DC_C, *Pl = Ph + DC_C * DC_C;
    float *sc = reinterpret_cast<float *>(Pl + DC_C * DC_C);
    {
        const uint32_t i0 = (warp & 3) * 16, j0 = (warp >> 2) * 32;
        float qk[4][4] = {}, kk[4][4] = {};
        if (j0 <= i0 + 15) {
            for (uint32_t d = 0; d < dpad; d += 16) {
                uint32_t aq[4], ak[4], b[4];
                ldsm_x4(aq, sQ + ((i0 + (lane & 15)) * PD + d + (lane >> 4) * 8) * 2);
                ldsm_x4(ak, sK + ((i0 + (lane & 15)) * PD + d + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    ldsm_x4(b, sK + ((j0 + n * 16 + (lane & 7) + (lane >> 4) * 8) * PD + d + ((lane >> 3) & 1) * 8) * 2);
                    mma_bf16(qk[2 * n], aq, b[0], b[1]);
                    mma_bf16(qk[2 * n + 1], aq, b[2], b[3]);
                    mma_bf16(kk[2 * n], ak, b[0], b[1]);
                    mma_bf16(kk[2 * n + 1], ak, b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < 4; n++)
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const uint32_t row = i0 + g8 + 8 * i, col = j0 + n * 8 + 2 * t4;
                float p[2], t[2];
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const uint32_t c = col + e;
                    const float f = c <= row ? expf(L[row] - L[c]) * rk[c] : 0.0f;
                    p[e] = qk[n][2 * i + e] * f * rq[row];
                    t[e] = c < row ? kk[n][2 * i + e] * f * rk[row] * bt[row] : 0.0f;
                }
                uint32_t hi, lo;
                split_bf16(p[0], p[1], hi, lo);
                *reinterpret_cast<uint32_t *>(Ph + row * DC_C + col) = hi;
                *reinterpret_cast<uint32_t *>(Pl + row * DC_C + col) = lo;
                *reinterpret_cast<float2 *>(A + row * PA + col) = make_float2(t[0], t[1]);
            }
    }
    if (tid < DC_C) {
        const float e = expf(L[tid]);
        sc[tid] = e * rk[tid];
        sc[DC_C + tid] = e * rq[tid];
        sc[2 * DC_C + tid] = expf(L[DC_C - 1] - L[tid]) * rk[tid];
        if (tid == 0) sc[3 * DC_C] = expf(L[DC_C - 1]);
    }
    __syncthreads();
    // X = (I + A)^-1: the diagonal blocks of 16 by substitution, then X21 = -X22 A21 X11 for blocks of 16 and of 32
    for (uint32_t i = tid; i < DC_C * DC_C; i += DL_THREADS) X[(i / DC_C) * PA + i % DC_C] = 0.0f;
    __syncthreads();
    if (tid < DC_C) {
        const uint32_t d = tid & ~15u, c = tid & 15;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; i++) {
            float p0 = i == (int)c ? 1.0f : 0.0f, p1 = 0.0f;
#pragma unroll
            for (int j = 0; j < i; j++) {
                const float t = A[(d + i) * PA + d + j] * x[j];
                if (j & 1) p1 -= t;
                else p0 -= t;
            }
            x[i] = p0 + p1;
            X[(d + i) * PA + d + c] = x[i];
        }
    }
    __syncthreads();
    {
        const uint32_t d = (tid >> 7) * 32, r = (tid & 127) >> 3, c = (tid & 7) * 2;
        float2 y = make_float2(0.0f, 0.0f);
#pragma unroll
        for (uint32_t k = 0; k < 16; k++) {
            const float t = A[(d + 16 + r) * PA + d + k];
            const float2 x = *reinterpret_cast<const float2 *>(X + (d + k) * PA + d + c);
            y = make_float2(fmaf(t, x.x, y.x), fmaf(t, x.y, y.y));
        }
        *reinterpret_cast<float2 *>(Y + (d / 2 + r) * PY + c) = y;
        __syncthreads();
        float2 z = make_float2(0.0f, 0.0f);
#pragma unroll
        for (uint32_t k = 0; k < 16; k++) {
            const float t = -X[(d + 16 + r) * PA + d + 16 + k];
            const float2 x = *reinterpret_cast<const float2 *>(Y + (d / 2 + k) * PY + c);
            z = make_float2(fmaf(t, x.x, z.x), fmaf(t, x.y, z.y));
        }
        *reinterpret_cast<float2 *>(X + (d + 16 + r) * PA + d + c) = z;
    }
    __syncthreads();
    {
        const uint32_t r = tid >> 3, c = (tid & 7) * 4;
        auto mul = [&](const float *m, const float *q, uint32_t pitch) {
            float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
            for (uint32_t k = 0; k < 32; k++) {
                const float t = m[k];
                const float4 x = *reinterpret_cast<const float4 *>(q + k * pitch + c);
                y = make_float4(fmaf(t, x.x, y.x), fmaf(t, x.y, y.y), fmaf(t, x.z, y.z), fmaf(t, x.w, y.w));
            }
            return y;
        };
        const float4 y = mul(A + (32 + r) * PA, X, PA);
        *reinterpret_cast<float4 *>(Y + r * PY + c) = y;
        __syncthreads();
        const float4 z = mul(X + (32 + r) * PA + 32, Y, PY);
        *reinterpret_cast<float4 *>(X + (32 + r) * PA + c) = make_float4(-z.x, -z.y, -z.z, -z.w);
    }
    __syncthreads();
    for (uint32_t i = tid; i < DC_C * DC_C / 2; i += DL_THREADS) {
        const uint32_t r = i / (DC_C / 2), c = (i % (DC_C / 2)) * 2;
        uint32_t hi, lo;
        split_bf16(X[r * PA + c] * bt[c], X[r * PA + c + 1] * bt[c + 1], hi, lo);
        *reinterpret_cast<uint32_t *>(Th + r * DC_C + c) = hi;
        *reinterpret_cast<uint32_t *>(Tl + r * DC_C + c) = lo;
    }
}

// Grid: (slice of 32 value columns, head).  The slice of the state lives in mma accumulators from the first chunk to
// the last; nbuf 2: the next chunk loads under this one.  Sixteen warps: 16 tokens x 8 value columns each, and of the
// state 16 (for more than 128 rows 2 x 16) rows x 16 columns.
constexpr int DC_THREADS = 512;
// DP: the padded key size when it is a usual one, else 0.
template <int DP>
__global__ void __launch_bounds__(DC_THREADS) delta_chunk_kernel(const DeltaArgs a, int32_t slot, uint32_t dpad_, uint32_t vec, uint32_t nbuf, uint32_t sh) {
    const uint32_t dpad = DP ? DP : dpad_;
    extern __shared__ __align__(16) uint8_t dcs[];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t PD = dpad + 8, h = blockIdx.y, kh = h / (a.heads / a.kv_heads), v0 = blockIdx.x * DL_VS, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t g8 = lane >> 2, t4 = lane & 3;
    const uint32_t TILE = 2 * DC_C * PD + DC_C * DC_PV + 4 * DC_C * DC_PT + 2 * DC_SCALARS;  // bf16 units: Q, K, V, T and P, scalars
    bf16 *tiles = reinterpret_cast<bf16 *>(dcs), *Sh = tiles + nbuf * TILE, *Sl = Sh + dpad * DC_PV, *Wh = Sl + dpad * DC_PV, *Wl = Wh + DC_C * DC_PV,
         *Uh = Wl + DC_C * DC_PV, *Ul = Uh + DC_C * DC_PV, *Hh = Ul + DC_C * DC_PV, *Hl = Hh + DC_C * DC_PV;
    auto sm = [](const bf16 *p) { return (uint32_t)__cvta_generic_to_shared(p); };
    const uint32_t sSh = sm(Sh), sSl = sm(Sl), sWh = sm(Wh), sWl = sm(Wl), sUh = sm(Uh), sUl = sm(Ul), sHh = sm(Hh), sHl = sm(Hl);
    float *S = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim;
    const uint32_t sw = warp & 7, s0 = (warp >> 3) * 16;
    float st[2][2][4];  // rows 16 (sw + 8 m) .. +16 of the key dimension, value columns s0 .. +16
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t d = (sw + 8 * m) * 16 + g8 + 8 * (i >> 1), c = v0 + s0 + n * 8 + 2 * t4 + (i & 1);
                st[m][n][i] = d < a.dim && c < a.vdim ? S[(size_t)d * a.vdim + c] : 0.0f;
            }
    const uint32_t n_mt = dpad / 16;
    auto load_chunk = [&](uint32_t r0, uint32_t buf) {
        const uint32_t nt = min((uint32_t)DC_C, a.rows - r0);
        bf16 *Q = tiles + buf * TILE, *K = Q + DC_C * PD, *V = K + DC_C * PD, *TP = V + DC_C * DC_PV, *sc = TP + 4 * DC_C * DC_PT;
        load_rows<DC_THREADS>(Q, PD, dpad, reinterpret_cast<const bf16 *>(a.q) + (size_t)r0 * a.pitch + kh * a.dim, a.pitch, nt, a.dim, vec, sh);
        load_rows<DC_THREADS>(K, PD, dpad, reinterpret_cast<const bf16 *>(a.k) + (size_t)r0 * a.pitch + kh * a.dim, a.pitch, nt, a.dim, vec, sh);
        load_rows<DC_THREADS>(V, DC_PV, DL_VS, reinterpret_cast<const bf16 *>(a.v) + (size_t)r0 * a.pitch + h * a.vdim + v0, a.pitch, nt, a.vdim - v0, vec, 2);
        const uint8_t *item = reinterpret_cast<const uint8_t *>(a.chunk_scratch) + ((size_t)(r0 / DC_C) * a.heads + h) * DC_ITEM;
        for (uint32_t i = tid; i < 4 * DC_C * 8; i += DC_THREADS)
            cp_async16(sm(TP) + ((i >> 3) * DC_PT + (i & 7) * 8) * 2, item + (size_t)i * 16);
        if (tid < DC_SCALARS / 4) cp_async16(sm(sc) + tid * 16, item + 4 * DC_C * DC_C * 2 + tid * 16);
        cp_async_commit();
    };
    load_chunk(0, 0);
    uint32_t buf = 0;
    for (uint32_t r0 = 0; r0 < a.rows; r0 += DC_C) {
        const uint32_t nt = min((uint32_t)DC_C, a.rows - r0);
        if (nbuf == 1 && r0) {
            __syncthreads();
            load_chunk(r0, 0);
        }
        const bf16 *Q = tiles + buf * TILE, *K = Q + DC_C * PD, *V = K + DC_C * PD, *T = V + DC_C * DC_PV, *P = T + 2 * DC_C * DC_PT;
        const float *sc = reinterpret_cast<const float *>(P + 2 * DC_C * DC_PT);
        const uint32_t sQ = sm(Q), sK = sm(K), sT = sm(T), sP = sm(P);
        constexpr uint32_t LO = DC_C * DC_PT * 2;  // bytes from the high to the low part
#pragma unroll
        for (int m = 0; m < 2; m++)
            if (sw + 8 * m < n_mt) {
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int i = 0; i < 2; i++) {
                        uint32_t hi, lo;
                        split_bf16(st[m][n][2 * i], st[m][n][2 * i + 1], hi, lo);
                        const uint32_t at = ((sw + 8 * m) * 16 + g8 + 8 * i) * DC_PV + s0 + n * 8 + 2 * t4;
                        *reinterpret_cast<uint32_t *>(Sh + at) = hi;
                        *reinterpret_cast<uint32_t *>(Sl + at) = lo;
                    }
            }
        cp_async_wait<0>();
        __syncthreads();  // this chunk and the state are there; every warp is done with the previous chunk
        if (nbuf == 2 && r0 + DC_C < a.rows) load_chunk(r0 + DC_C, buf ^ 1);
        const uint32_t i0 = (warp & 3) * 16, c0 = (warp >> 2) * 8;  // rows and value columns of this warp
        float ks[4] = {}, qs[4] = {}, kl[4] = {}, ql[4] = {};       // products with the state's high and low parts
#pragma unroll(DP ? DP / 16 : 2)
        for (uint32_t d = 0; d < dpad; d += 16) {
            uint32_t ak[4], aq[4], bh[2], bl[2];
            const uint32_t at = ((i0 + (lane & 15)) * PD + d + (lane >> 4) * 8) * 2, bt = ((d + (lane & 15)) * DC_PV + c0) * 2;
            ldsm_x4(ak, sK + at);
            ldsm_x4(aq, sQ + at);
            ldsm_x2_t(bh, sSh + bt);
            ldsm_x2_t(bl, sSl + bt);
            mma_bf16(ks, ak, bh[0], bh[1]);
            mma_bf16(qs, aq, bh[0], bh[1]);
            mma_bf16(kl, ak, bl[0], bl[1]);
            mma_bf16(ql, aq, bl[0], bl[1]);
        }
        const uint32_t row = i0 + g8, at0 = row * DC_PV + c0 + 2 * t4, at1 = at0 + 8 * DC_PV;  // this lane's two rows
        {
            const float2 va = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(V + at0)), vb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(V + at1));
            const float ea = sc[row], eb = sc[row + 8];
            uint32_t hi, lo;
            split_bf16(fmaf(-ea, ks[0] + kl[0], va.x), fmaf(-ea, ks[1] + kl[1], va.y), hi, lo);
            *reinterpret_cast<uint32_t *>(Wh + at0) = hi;
            *reinterpret_cast<uint32_t *>(Wl + at0) = lo;
            split_bf16(fmaf(-eb, ks[2] + kl[2], vb.x), fmaf(-eb, ks[3] + kl[3], vb.y), hi, lo);
            *reinterpret_cast<uint32_t *>(Wh + at1) = hi;
            *reinterpret_cast<uint32_t *>(Wl + at1) = lo;
        }
        __syncthreads();
        // a lower triangular matrix (high and low parts at m) times columns c0 .. +8 of a right-hand side
        auto tri = [&](float (&o)[4], uint32_t m, uint32_t bh, uint32_t bl) {
            float p[4] = {}, q[4] = {};
            for (uint32_t j = 0; j <= i0; j += 16) {
                uint32_t xh[4], xl[4], yh[2], yl[2];
                const uint32_t at = ((i0 + (lane & 15)) * DC_PT + j + (lane >> 4) * 8) * 2, bt = ((j + (lane & 15)) * DC_PV + c0) * 2;
                ldsm_x4(xh, m + at);
                ldsm_x4(xl, m + LO + at);
                ldsm_x2_t(yh, bh + bt);
                ldsm_x2_t(yl, bl + bt);
                mma_bf16(o, xh, yh[0], yh[1]);
                mma_bf16(p, xl, yh[0], yh[1]);
                mma_bf16(q, xh, yl[0], yl[1]);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) o[i] += p[i] + q[i];
        };
        float u[4] = {};
        tri(u, sT, sWh, sWl);
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const uint32_t at = i ? at1 : at0;
            const float w = sc[2 * DC_C + row + 8 * i];
            uint32_t hi, lo;
            split_bf16(u[2 * i], u[2 * i + 1], hi, lo);
            *reinterpret_cast<uint32_t *>(Uh + at) = hi;
            *reinterpret_cast<uint32_t *>(Ul + at) = lo;
            split_bf16(u[2 * i] * w, u[2 * i + 1] * w, hi, lo);
            *reinterpret_cast<uint32_t *>(Hh + at) = hi;
            *reinterpret_cast<uint32_t *>(Hl + at) = lo;
        }
        __syncthreads();
        float o[4] = {};
        tri(o, sP, sUh, sUl);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const uint32_t t = row + 8 * (i >> 1), c = v0 + c0 + 2 * t4 + (i & 1);
            if (t < nt && c < a.vdim) a.o32[(size_t)(r0 + t) * a.heads * a.vdim + h * a.vdim + c] = fmaf(sc[DC_C + t], qs[i] + ql[i], o[i]);
        }
        const float gc = sc[3 * DC_C];
#pragma unroll
        for (int m = 0; m < 2; m++)
            if (sw + 8 * m < n_mt) {
                float low[2][4] = {};
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int i = 0; i < 4; i++) st[m][n][i] *= gc;
#pragma unroll
                for (uint32_t j = 0; j < DC_C; j += 16) {
                    uint32_t ak[4], b[4];
                    const uint32_t bt = ((j + (lane & 15)) * DC_PV + s0 + (lane >> 4) * 8) * 2;
                    ldsm_x4_t(ak, sK + ((j + (lane >> 4) * 8 + (lane & 7)) * PD + (sw + 8 * m) * 16 + ((lane >> 3) & 1) * 8) * 2);
                    ldsm_x4_t(b, sHh + bt);
                    mma_bf16(st[m][0], ak, b[0], b[1]);
                    mma_bf16(st[m][1], ak, b[2], b[3]);
                    ldsm_x4_t(b, sHl + bt);
                    mma_bf16(low[0], ak, b[0], b[1]);
                    mma_bf16(low[1], ak, b[2], b[3]);
                }
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int i = 0; i < 4; i++) st[m][n][i] += low[n][i];
            }
        if (nbuf == 2) buf ^= 1;
    }
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t d = (sw + 8 * m) * 16 + g8 + 8 * (i >> 1), c = v0 + s0 + n * 8 + 2 * t4 + (i & 1);
                if (d < a.dim && c < a.vdim) S[(size_t)d * a.vdim + c] = st[m][n][i];
            }
}

// ---- host side -----------------------------------------------------------------------------------------------
constexpr size_t DL_SMEM_MAX = 224 * 1024;

size_t delta_scratch_bytes(const DeltaArgs &a, uint32_t rows) { return (size_t)((rows + DC_C - 1) / DC_C) * a.heads * DC_ITEM; }

static int configure(prism_cuda_ctx *ctx) {
    static bool configured[PRISM_MAX_DEVICES] = {false};
    if (configured[ctx->device]) return PRISM_OK;
    PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(delta_seq_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DL_SMEM_MAX));
    PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(delta_seq_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DL_SMEM_MAX));
    PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(delta_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DL_SMEM_MAX));
    PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(delta_chunk_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DL_SMEM_MAX));
    PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(delta_chunk_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DL_SMEM_MAX));
    PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(delta_chunk_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DL_SMEM_MAX));
    configured[ctx->device] = true;
    return PRISM_OK;
}

int launch_delta_seq(prism_cuda_ctx *ctx, const DeltaArgs &a, const RowMap &rows, bool act32) {
    PRISM_TRY(configure(ctx));
    const dim3 grid((a.vdim + DL_VS - 1) / DL_VS, a.heads);
    const uint32_t dpad = round_up_u32(a.dim, 16);
    if (!act32 && dpad <= 256 && a.rows > DENSE_GEMV_ROWS) {
        const uint32_t vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.pitch % 8 == 0 &&
                             !((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) | reinterpret_cast<uintptr_t>(a.v)) & 15);
        const uint32_t sh = row_shift(dpad / 8);
        const size_t qk = (size_t)2 * DC_C * (dpad + 8) * 2;
        const size_t prep = (size_t)DC_C * DC_PA * 4 + std::max(qk, (size_t)(DC_C * DC_PA + 32 * DC_PY) * 4);
        launch_pdl(ctx, "delta_prep_kernel", delta_prep_kernel, dim3((a.rows + DC_C - 1) / DC_C, a.heads), DL_THREADS, prep, a, dpad, vec, sh);
        PRISM_TRY(after_launch(ctx, "delta_prep_kernel"));
        const size_t tile = qk + (size_t)(DC_C * DC_PV + 4 * DC_C * DC_PT) * 2 + DC_SCALARS * 4, rest = (size_t)(2 * dpad + 6 * DC_C) * DC_PV * 2;
        const uint32_t nbuf = 2 * tile + rest <= DL_SMEM_MAX ? 2 : 1;
        auto chunk = [&](auto kernel) { launch_pdl(ctx, "delta_chunk_kernel", kernel, grid, DC_THREADS, nbuf * tile + rest, a, rows.slot0, dpad, vec, nbuf, sh); };
        if (dpad == 64) chunk(delta_chunk_kernel<64>);
        else if (dpad == 128) chunk(delta_chunk_kernel<128>);
        else chunk(delta_chunk_kernel<0>);
        PRISM_TRY(after_launch(ctx, "delta_chunk_kernel"));
    } else {
        const size_t smem = (size_t)a.dim * (2 + DL_VS) * 4;
        if (smem > DL_SMEM_MAX) return fail(ctx, PRISM_E_ARG, "gated delta: key dimension too large");
        if (act32) launch_pdl(ctx, "delta_seq_kernel", delta_seq_kernel<float>, grid, DL_THREADS, smem, a, rows.slot0);
        else launch_pdl(ctx, "delta_seq_kernel", delta_seq_kernel<bf16>, grid, DL_THREADS, smem, a, rows.slot0);
        PRISM_TRY(after_launch(ctx, "delta_seq_kernel"));
    }
    const uint32_t blocks = (uint32_t)(((uint64_t)a.rows * a.heads + DL_THREADS / 32 - 1) / (DL_THREADS / 32));
    const uint32_t vec = a.vdim <= 128 * DG_U && !((a.vdim | a.gate_pitch | a.o_pitch) & 3) &&
                         !((reinterpret_cast<uintptr_t>(a.gate) | reinterpret_cast<uintptr_t>(a.o) | reinterpret_cast<uintptr_t>(a.norm)) & 15);
    if (act32) launch_pdl(ctx, "delta_gate_kernel", delta_gate_kernel<float>, blocks, DL_THREADS, 0, a, vec);
    else launch_pdl(ctx, "delta_gate_kernel", delta_gate_kernel<bf16>, blocks, DL_THREADS, 0, a, vec);
    return after_launch(ctx, "delta_gate_kernel");
}

}  // namespace prism
