// Linear attention with one decay per head, S_t = d S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, the state in
// fp32:  a decode kernel (one token of every sequence), a token-by-token kernel for short portions, for
// 32-bit runs and for unusual sizes, and a chunked form for prompts on the tensor cores.
#include <algorithm>

#include "dense.cuh"

namespace prism {

constexpr int LT_THREADS = 256, LT_VS = 32;  // value columns of a CTA

// One token per sequence.  Grid: (value slice, head, row).  Thread (d group, v): the state is streamed once.
template <typename TA>
__global__ void __launch_bounds__(LT_THREADS) lightning_step_kernel(const LightningArgs a, const RowMap rows) {
    extern __shared__ float lsm[];
    __shared__ float red[8][LT_VS + 1];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.z, h = blockIdx.y, v = blockIdx.x * LT_VS + (threadIdx.x & 31), dg = threadIdx.x >> 5;
    const TA *q = reinterpret_cast<const TA *>(a.q) + (size_t)r * a.pitch + h * a.dim;
    const TA *k = reinterpret_cast<const TA *>(a.k) + (size_t)r * a.pitch + h * a.dim;
    float *qs = lsm, *ks = lsm + a.dim;
    for (uint32_t d = threadIdx.x; d < a.dim; d += LT_THREADS) {
        qs[d] = ld_act(q + d);
        ks[d] = ld_act(k + d);
    }
    __syncthreads();
    float acc = 0.0f;
    if (v < a.vdim) {
        const float vv = ld_act(reinterpret_cast<const TA *>(a.v) + (size_t)r * a.pitch + h * a.vdim + v), dec = a.decay[h];
        float *S = a.state + ((size_t)rows.slot_of(r) * a.heads + h) * a.dim * a.vdim + v;
#pragma unroll 8
        for (uint32_t d = dg; d < a.dim; d += 8) {
            const float s = fmaf(dec, S[(size_t)d * a.vdim], ks[d] * vv);
            S[(size_t)d * a.vdim] = s;
            acc = fmaf(qs[d], s, acc);
        }
    }
    red[dg][threadIdx.x & 31] = acc;
    __syncthreads();
    if (dg == 0 && v < a.vdim) {
        float o = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) o += red[i][threadIdx.x];
        st_act(reinterpret_cast<TA *>(a.o) + (size_t)r * a.o_pitch + h * a.vdim + v, o);
    }
}

// Consecutive tokens of one sequence, token by token, the state slice in shared memory.
template <typename TA>
__global__ void __launch_bounds__(LT_THREADS) lightning_seq_kernel(const LightningArgs a, int32_t slot) {
    extern __shared__ float lsm[];
    __shared__ float red[8][LT_VS + 1];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t h = blockIdx.y, vl = threadIdx.x & 31, v = blockIdx.x * LT_VS + vl, dg = threadIdx.x >> 5;
    float *qs = lsm, *ks = lsm + a.dim, *ss = ks + a.dim;
    float *S = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim;
    const float dec = a.decay[h];
    const bool on = v < a.vdim;
    for (uint32_t d = dg; d < a.dim; d += 8) ss[d * LT_VS + vl] = on ? S[(size_t)d * a.vdim + v] : 0.0f;
    for (uint32_t r = 0; r < a.rows; r++) {
        __syncthreads();
        for (uint32_t d = threadIdx.x; d < a.dim; d += LT_THREADS) {
            qs[d] = ld_act(reinterpret_cast<const TA *>(a.q) + (size_t)r * a.pitch + h * a.dim + d);
            ks[d] = ld_act(reinterpret_cast<const TA *>(a.k) + (size_t)r * a.pitch + h * a.dim + d);
        }
        const float vv = on ? ld_act(reinterpret_cast<const TA *>(a.v) + (size_t)r * a.pitch + h * a.vdim + v) : 0.0f;
        __syncthreads();
        float acc = 0.0f;
        for (uint32_t d = dg; d < a.dim; d += 8) {
            const float s = fmaf(dec, ss[d * LT_VS + vl], ks[d] * vv);
            ss[d * LT_VS + vl] = s;
            acc = fmaf(qs[d], s, acc);
        }
        red[dg][vl] = acc;
        __syncthreads();
        if (dg == 0 && on) {
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; i++) o += red[i][vl];
            st_act(reinterpret_cast<TA *>(a.o) + (size_t)r * a.o_pitch + h * a.vdim + v, o);
        }
    }
    for (uint32_t d = dg; d < a.dim; d += 8)
        if (on) S[(size_t)d * a.vdim + v] = ss[d * LT_VS + vl];
}

// Prompt portions of one sequence in chunks of 64 tokens.  A CTA owns 32 value columns of a head and walks
// the chunks; its slice of the state lives in mma accumulators (fp32) from the first chunk to the last.
//   o_i = sum_{j <= i} (q_i . k_j) d^(i-j) v_j  +  d^(i+1) S^T q_i,     S <- d^n S + sum_j d^(n-1-j) k_j v_j^T
// q, k and v are bf16; what is not (the decayed scores, the decayed values, the state as an operand) enters
// the products as a sum of two bf16 parts, so no factor of the recurrence is rounded to bf16.
constexpr int LC_C = 64, LC_PV = LT_VS + 8, LC_PA = LC_C + 8;
__global__ void __launch_bounds__(LT_THREADS) lightning_chunk_kernel(const LightningArgs a, int32_t slot, uint32_t dpad, uint32_t vec) {
    extern __shared__ __align__(16) uint8_t lcs[];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t PD = dpad + 8, h = blockIdx.y, v0 = blockIdx.x * LT_VS, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t g8 = lane >> 2, t4 = lane & 3;
    const uint32_t TILE = 2 * LC_C * PD + LC_C * LC_PV;  // q, k and v of a chunk; two of them, the next chunk loads under this one
    bf16 *tiles = reinterpret_cast<bf16 *>(lcs), *Vh = tiles + 2 * TILE, *Vl = Vh + LC_C * LC_PV,
         *Ah = Vl + LC_C * LC_PV, *Al = Ah + LC_C * LC_PA, *Sh = Al + LC_C * LC_PA, *Sl = Sh + dpad * LC_PV;
    float *pw = reinterpret_cast<float *>(Sl + dpad * LC_PV);  // d^0 .. d^64
    const uint32_t sT = (uint32_t)__cvta_generic_to_shared(tiles), sVh = (uint32_t)__cvta_generic_to_shared(Vh), sVl = (uint32_t)__cvta_generic_to_shared(Vl), sAh = (uint32_t)__cvta_generic_to_shared(Ah),
                   sAl = (uint32_t)__cvta_generic_to_shared(Al), sSh = (uint32_t)__cvta_generic_to_shared(Sh), sSl = (uint32_t)__cvta_generic_to_shared(Sl);
    const bf16 zero = __float2bfloat16_rn(0.0f);
    const bf16 *q = reinterpret_cast<const bf16 *>(a.q) + h * a.dim, *k = reinterpret_cast<const bf16 *>(a.k) + h * a.dim,
               *v = reinterpret_cast<const bf16 *>(a.v) + h * a.vdim;
    float *S = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim;
    if (tid <= LC_C) {
        double p = 1.0;
        const double d = a.decay[h];
        for (uint32_t i = 0; i < tid; i++) p *= d;
        pw[tid] = (float)p;
    }
    // state slice: warp w holds rows 16 (w + 8 m) .. +16 of the key dimension
    float st[2][4][4];
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
        for (int n = 0; n < 4; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t d = (warp + 8 * m) * 16 + g8 + 8 * (i >> 1), c = v0 + n * 8 + 2 * t4 + (i & 1);
                st[m][n][i] = d < a.dim && c < a.vdim ? S[(size_t)d * a.vdim + c] : 0.0f;
            }
    const uint32_t n_mt = dpad / 16;
    auto load_chunk = [&](uint32_t r0, uint32_t buf) {
        const uint32_t nt = min((uint32_t)LC_C, a.rows - r0), sq = sT + buf * TILE * 2, sk = sq + LC_C * PD * 2, sv = sk + LC_C * PD * 2;
        bf16 *Q = tiles + buf * TILE, *K = Q + LC_C * PD, *V = K + LC_C * PD;
        if (vec) {
            const uint4 z = make_uint4(0, 0, 0, 0);
            const uint32_t d8 = dpad / 8, n8 = a.dim / 8;
            for (uint32_t i = tid; i < LC_C * d8; i += LT_THREADS) {
                const uint32_t r = i / d8, c = i % d8, at = r * PD + c * 8;
                if (r < nt && c < n8) {
                    cp_async16(sq + at * 2, q + (size_t)(r0 + r) * a.pitch + c * 8);
                    cp_async16(sk + at * 2, k + (size_t)(r0 + r) * a.pitch + c * 8);
                } else {
                    *reinterpret_cast<uint4 *>(Q + at) = z;
                    *reinterpret_cast<uint4 *>(K + at) = z;
                }
            }
            {
                const uint32_t r = tid / (LT_VS / 8), c = (tid % (LT_VS / 8)) * 8, at = r * LC_PV + c;  // 64 x 4 pieces: one per thread
                if (r < nt && v0 + c < a.vdim) cp_async16(sv + at * 2, v + (size_t)(r0 + r) * a.pitch + v0 + c);
                else *reinterpret_cast<uint4 *>(V + at) = z;
            }
        } else {
            for (uint32_t i = tid; i < LC_C * dpad; i += LT_THREADS) {
                const uint32_t r = i / dpad, c = i % dpad;
                const bool on = r < nt && c < a.dim;
                Q[r * PD + c] = on ? q[(size_t)(r0 + r) * a.pitch + c] : zero;
                K[r * PD + c] = on ? k[(size_t)(r0 + r) * a.pitch + c] : zero;
            }
            for (uint32_t i = tid; i < LC_C * LT_VS; i += LT_THREADS) {
                const uint32_t r = i / LT_VS, c = i % LT_VS;
                V[r * LC_PV + c] = r < nt && v0 + c < a.vdim ? v[(size_t)(r0 + r) * a.pitch + v0 + c] : zero;
            }
        }
        cp_async_commit();
    };
    static_assert(LC_C * LT_VS / 8 == LT_THREADS, "one piece of v per thread");
    load_chunk(0, 0);
    uint32_t buf = 0;
    for (uint32_t r0 = 0; r0 < a.rows; r0 += LC_C, buf ^= 1) {
        const uint32_t nt = min((uint32_t)LC_C, a.rows - r0);
        const uint32_t sQ = sT + buf * TILE * 2, sK = sQ + LC_C * PD * 2, sV = sK + LC_C * PD * 2;
        const bf16 *Vs = tiles + buf * TILE + 2 * LC_C * PD;
        cp_async_wait<0>();
        __syncthreads();  // this chunk has arrived, and every warp is done with the previous one
        if (r0 + LC_C < a.rows) load_chunk(r0 + LC_C, buf ^ 1);
        for (uint32_t i = tid; i < LC_C * LT_VS / 2; i += LT_THREADS) {
            const uint32_t r = i / (LT_VS / 2), c = (i % (LT_VS / 2)) * 2;
            const float f = r < nt ? pw[nt - 1 - r] : 0.0f;
            uint32_t hi, lo;
            split_bf16(__bfloat162float(Vs[r * LC_PV + c]) * f, __bfloat162float(Vs[r * LC_PV + c + 1]) * f, hi, lo);
            *reinterpret_cast<uint32_t *>(Vh + r * LC_PV + c) = hi;
            *reinterpret_cast<uint32_t *>(Vl + r * LC_PV + c) = lo;
        }
        // the state before this chunk, as two bf16 parts
#pragma unroll
        for (int m = 0; m < 2; m++)
            if (warp + 8 * m < n_mt) {
#pragma unroll
                for (int n = 0; n < 4; n++)
#pragma unroll
                    for (int i = 0; i < 2; i++) {
                        uint32_t hi, lo;
                        split_bf16(st[m][n][2 * i], st[m][n][2 * i + 1], hi, lo);
                        const uint32_t at = ((warp + 8 * m) * 16 + g8 + 8 * i) * LC_PV + n * 8 + 2 * t4;
                        *reinterpret_cast<uint32_t *>(Sh + at) = hi;
                        *reinterpret_cast<uint32_t *>(Sl + at) = lo;
                    }
            }
        const uint32_t i0 = (warp & 3) * 16;
        // decayed scores: rows i0 .. +16, columns (warp / 4) * 32 .. +32
        {
            const uint32_t j0 = (warp >> 2) * 32;
            float sc[4][4] = {};
            if (j0 <= i0 + 15) {
                for (uint32_t kk = 0; kk < dpad; kk += 16) {
                    uint32_t aq[4], b[4];
                    ldsm_x4(aq, sQ + ((i0 + (lane & 15)) * PD + kk + (lane >> 4) * 8) * 2);
#pragma unroll
                    for (int n = 0; n < 2; n++) {
                        ldsm_x4(b, sK + ((j0 + n * 16 + (lane & 7) + (lane >> 4) * 8) * PD + kk + ((lane >> 3) & 1) * 8) * 2);
                        mma_bf16(sc[2 * n], aq, b[0], b[1]);
                        mma_bf16(sc[2 * n + 1], aq, b[2], b[3]);
                    }
                }
            }
#pragma unroll
            for (int n = 0; n < 4; n++)
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    const uint32_t row = i0 + g8 + 8 * i, col = j0 + n * 8 + 2 * t4;
                    const float x = col <= row ? sc[n][2 * i] * pw[row - col] : 0.0f;
                    const float y = col + 1 <= row ? sc[n][2 * i + 1] * pw[row - col - 1] : 0.0f;
                    uint32_t hi, lo;
                    split_bf16(x, y, hi, lo);
                    *reinterpret_cast<uint32_t *>(Ah + row * LC_PA + col) = hi;
                    *reinterpret_cast<uint32_t *>(Al + row * LC_PA + col) = lo;
                }
        }
        __syncthreads();
        // outputs: rows i0 .. +16, columns (warp / 4) * 16 .. +16
        {
            const uint32_t c0 = (warp >> 2) * 16;
            float o1[2][4] = {}, o2[2][4] = {};
            for (uint32_t kk = 0; kk <= i0; kk += 16) {  // later tokens have zero scores
                uint32_t ah[4], al[4], b[4];
                ldsm_x4(ah, sAh + ((i0 + (lane & 15)) * LC_PA + kk + (lane >> 4) * 8) * 2);
                ldsm_x4(al, sAl + ((i0 + (lane & 15)) * LC_PA + kk + (lane >> 4) * 8) * 2);
                ldsm_x4_t(b, sV + ((kk + (lane & 15)) * LC_PV + c0 + (lane >> 4) * 8) * 2);
                mma_bf16(o1[0], ah, b[0], b[1]);
                mma_bf16(o1[1], ah, b[2], b[3]);
                mma_bf16(o1[0], al, b[0], b[1]);
                mma_bf16(o1[1], al, b[2], b[3]);
            }
            for (uint32_t kk = 0; kk < dpad; kk += 16) {
                uint32_t aq[4], b[4];
                ldsm_x4(aq, sQ + ((i0 + (lane & 15)) * PD + kk + (lane >> 4) * 8) * 2);
                ldsm_x4_t(b, sSh + ((kk + (lane & 15)) * LC_PV + c0 + (lane >> 4) * 8) * 2);
                mma_bf16(o2[0], aq, b[0], b[1]);
                mma_bf16(o2[1], aq, b[2], b[3]);
                ldsm_x4_t(b, sSl + ((kk + (lane & 15)) * LC_PV + c0 + (lane >> 4) * 8) * 2);
                mma_bf16(o2[0], aq, b[0], b[1]);
                mma_bf16(o2[1], aq, b[2], b[3]);
            }
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const uint32_t row = i0 + g8 + 8 * (i >> 1), c = v0 + c0 + n * 8 + 2 * t4 + (i & 1);
                    if (row < nt && c < a.vdim)
                        st_act(reinterpret_cast<bf16 *>(a.o) + (size_t)(r0 + row) * a.o_pitch + h * a.vdim + c, fmaf(pw[row + 1], o2[n][i], o1[n][i]));
                }
        }
        // state after this chunk
        const float pn = pw[nt];
#pragma unroll
        for (int m = 0; m < 2; m++)
            if (warp + 8 * m < n_mt) {
#pragma unroll
                for (int n = 0; n < 4; n++)
#pragma unroll
                    for (int i = 0; i < 4; i++) st[m][n][i] *= pn;
                for (uint32_t kk = 0; kk < LC_C; kk += 16) {
                    uint32_t ak[4], b[4];
                    ldsm_x4_t(ak, sK + ((kk + (lane >> 4) * 8 + (lane & 7)) * PD + (warp + 8 * m) * 16 + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
                    for (int n = 0; n < 2; n++) {
                        ldsm_x4_t(b, sVh + ((kk + (lane & 15)) * LC_PV + n * 16 + (lane >> 4) * 8) * 2);
                        mma_bf16(st[m][2 * n], ak, b[0], b[1]);
                        mma_bf16(st[m][2 * n + 1], ak, b[2], b[3]);
                        ldsm_x4_t(b, sVl + ((kk + (lane & 15)) * LC_PV + n * 16 + (lane >> 4) * 8) * 2);
                        mma_bf16(st[m][2 * n], ak, b[0], b[1]);
                        mma_bf16(st[m][2 * n + 1], ak, b[2], b[3]);
                    }
                }
            }
    }
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
        for (int n = 0; n < 4; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const uint32_t d = (warp + 8 * m) * 16 + g8 + 8 * (i >> 1), c = v0 + n * 8 + 2 * t4 + (i & 1);
                if (d < a.dim && c < a.vdim) S[(size_t)d * a.vdim + c] = st[m][n][i];
            }
}

// ---- host side ---------------------------------------------------------------------------------
constexpr size_t LT_SMEM_MAX = 224 * 1024;

int launch_lightning_step(prism_cuda_ctx *ctx, const LightningArgs &a, const RowMap &rows, bool act32) {
    const dim3 grid((a.vdim + LT_VS - 1) / LT_VS, a.heads, a.rows);
    const size_t smem = 2 * (size_t)a.dim * 4;
    if (smem > 48 * 1024) return fail(ctx, PRISM_E_ARG, "lightning: key dimension too large");
    if (act32) launch_pdl(ctx, "lightning_step_kernel", lightning_step_kernel<float>, grid, LT_THREADS, smem, a, rows);
    else launch_pdl(ctx, "lightning_step_kernel", lightning_step_kernel<bf16>, grid, LT_THREADS, smem, a, rows);
    return after_launch(ctx, "lightning_step_kernel");
}

int launch_lightning_seq(prism_cuda_ctx *ctx, const LightningArgs &a, const RowMap &rows, bool act32) {
    static bool configured[PRISM_MAX_DEVICES] = {false};
    if (!configured[ctx->device]) {
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(lightning_seq_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LT_SMEM_MAX));
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(lightning_seq_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LT_SMEM_MAX));
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(lightning_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LT_SMEM_MAX));
        configured[ctx->device] = true;
    }
    const dim3 grid((a.vdim + LT_VS - 1) / LT_VS, a.heads);
    const uint32_t dpad = round_up_u32(a.dim, 16);
    const size_t csm = ((size_t)4 * LC_C * (dpad + 8) + 4 * LC_C * LC_PV + 2 * LC_C * LC_PA + 2 * (size_t)dpad * LC_PV) * 2 + (LC_C + 1) * 4;
    if (!act32 && dpad <= 256 && a.rows > DENSE_GEMV_ROWS && csm <= LT_SMEM_MAX) {
        const uint32_t vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.pitch % 8 == 0 &&
                             !((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) | reinterpret_cast<uintptr_t>(a.v)) & 15);
        launch_pdl(ctx, "lightning_chunk_kernel", lightning_chunk_kernel, grid, LT_THREADS, csm, a, rows.slot0, dpad, vec);
        return after_launch(ctx, "lightning_chunk_kernel");
    }
    const size_t smem = (size_t)a.dim * (2 + LT_VS) * 4;
    if (smem > LT_SMEM_MAX) return fail(ctx, PRISM_E_ARG, "lightning: key dimension too large");
    if (act32) launch_pdl(ctx, "lightning_seq_kernel", lightning_seq_kernel<float>, grid, LT_THREADS, smem, a, rows.slot0);
    else launch_pdl(ctx, "lightning_seq_kernel", lightning_seq_kernel<bf16>, grid, LT_THREADS, smem, a, rows.slot0);
    return after_launch(ctx, "lightning_seq_kernel");
}

}  // namespace prism
