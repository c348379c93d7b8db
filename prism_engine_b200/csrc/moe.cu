// Routing of a mixture-of-experts layer: sigmoid scores, a correction that takes part in the choice only, choice
// inside the best groups, and the plan by which the expert linears find their rows.
#include <algorithm>

#include "dense.cuh"

namespace prism {

// Index of the largest of n values in shared memory (the first of equals), by one warp.
__device__ __forceinline__ uint32_t warp_argmax(const float *v, uint32_t n, uint32_t lane) {
    float best = -INFINITY;
    uint32_t at = 0xFFFFFFFFu;
    for (uint32_t i = lane; i < n; i += 32)
        if (at == 0xFFFFFFFFu || v[i] > best) { best = v[i]; at = i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float b = __shfl_xor_sync(0xFFFFFFFFu, best, o);
        const uint32_t i = __shfl_xor_sync(0xFFFFFFFFu, at, o);
        if (i < at ? b >= best : b > best) { best = b; at = i; }
    }
    return at;
}

// One warp per token.  few: the whole batch is one block, which also writes the experts in use and their pairs.
constexpr int MR_WARPS = 8;
__global__ void __launch_bounds__(MR_WARPS * 32) moe_route_kernel(const MoeRouter m, const MoePlan plan, uint32_t tokens, uint32_t few) {
    extern __shared__ float mrs[];  // per warp: choice scores, group scores
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * MR_WARPS + warp, E = plan.experts;
    float *ch = mrs + (size_t)warp * (E + m.groups), *gs = ch + E;
    if (t < tokens) {
        const float *z = m.logits + (size_t)t * m.pitch;
        for (uint32_t e = lane; e < E; e += 32) {
            const float c = sigmoid_f(z[e]) + m.correction[e];
            ch[e] = c > -3.0e38f ? c : -3.0e38f;  // never below what a left-out group counts as, nor a NaN
        }
        __syncwarp();
        if (m.keep < m.groups) {
            const uint32_t per = E / m.groups;
            for (uint32_t g = lane; g < m.groups; g += 32) {
                float a = -INFINITY, b = -INFINITY;  // the two largest
                for (uint32_t e = g * per; e < (g + 1) * per; e++) {
                    const float c = ch[e];
                    b = fmaxf(b, fminf(a, c));
                    a = fmaxf(a, c);
                }
                gs[g] = per > 1 ? a + b : a;
            }
            __syncwarp();
            for (uint32_t g = lane; g < m.groups; g += 32) {
                uint32_t before = 0;
                for (uint32_t i = 0; i < m.groups; i++) before += gs[i] > gs[g] || (gs[i] == gs[g] && i < g);
                if (before >= m.keep)
                    for (uint32_t e = g * per; e < (g + 1) * per; e++) ch[e] = -INFINITY;
            }
            __syncwarp();
        }
        for (uint32_t k = 0; k < plan.top; k++) {
            const uint32_t e = min(warp_argmax(ch, E, lane), E - 1);
            if (lane == 0) {
                plan.idx[t * plan.top + k] = e;
                plan.wgt[t * plan.top + k] = sigmoid_f(z[e]);
                ch[e] = -INFINITY;
            }
            __syncwarp();
        }
    }
    if (!few) return;
    __syncthreads();
    const uint32_t pairs = tokens * plan.top;
    uint32_t *si = reinterpret_cast<uint32_t *>(mrs + (size_t)MR_WARPS * (E + m.groups)), *first = si + pairs;  // experts of the pairs; no earlier pair has it
    for (uint32_t p = threadIdx.x; p < pairs; p += blockDim.x) si[p] = plan.idx[p];
    __syncthreads();
    for (uint32_t p = threadIdx.x; p < pairs; p += blockDim.x) {
        uint32_t f = 1;
        for (uint32_t i = 0; i < p; i++) f &= si[i] != si[p];
        first[p] = f;
    }
    __syncthreads();
    for (uint32_t p = threadIdx.x; p < pairs; p += blockDim.x) {
        uint32_t at = 0;
        for (uint32_t i = 0; i < p; i++) at += first[i];
        if (p + 1 == pairs) *plan.n_active = at + first[p];
        if (!first[p]) continue;
        plan.active[at] = si[p];
        for (uint32_t j = 0; j < DENSE_GEMV_ROWS; j++) {
            int32_t row = -1;
            for (uint32_t i = j * plan.top; j < tokens && i < (j + 1) * plan.top; i++)
                if (si[i] == si[p]) row = (int32_t)i;
            plan.pair_of[at * DENSE_GEMV_ROWS + j] = row;
        }
    }
}

// Block e: the pairs of expert e, in order, after those of the experts before it.
constexpr int MS_THREADS = 256;
__global__ void __launch_bounds__(MS_THREADS) moe_sort_kernel(const MoePlan plan, uint32_t pairs) {
    __shared__ uint32_t sh[MS_THREADS / 32];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t e = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    uint32_t less = 0;
    for (uint32_t p = threadIdx.x; p < pairs; p += MS_THREADS) less += plan.idx[p] < e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) less += __shfl_xor_sync(0xFFFFFFFFu, less, o);
    if (lane == 0) sh[warp] = less;
    __syncthreads();
    uint32_t base = 0;
    for (uint32_t i = 0; i < MS_THREADS / 32; i++) base += sh[i];
    uint32_t n = 0;
    for (uint32_t p0 = 0; p0 < pairs; p0 += MS_THREADS) {
        const uint32_t p = p0 + threadIdx.x;
        const bool mine = p < pairs && plan.idx[p] == e;
        const uint32_t b = __ballot_sync(0xFFFFFFFFu, mine);
        __syncthreads();
        if (lane == 0) sh[warp] = __popc(b);
        __syncthreads();
        uint32_t before = 0, all = 0;
        for (uint32_t i = 0; i < MS_THREADS / 32; i++) {
            if (i < warp) before += sh[i];
            all += sh[i];
        }
        if (mine) {
            const uint32_t row = base + n + before + __popc(b & ((1u << lane) - 1));
            plan.order[row] = p;
            plan.inv[p] = row;
        }
        n += all;
    }
    if (threadIdx.x == 0) plan.count[e] = n;
}

int launch_moe_route(prism_cuda_ctx *ctx, const MoeRouter &r, const MoePlan &plan, uint32_t tokens, bool sorted) {
    if (!sorted && tokens > DENSE_GEMV_ROWS) return fail(ctx, PRISM_E_ARG, "experts: too many tokens for the small-batch plan");
    const size_t smem = (size_t)MR_WARPS * (plan.experts + r.groups) * 4 + (sorted ? 0 : (size_t)tokens * plan.top * 8);
    if (smem > 96 * 1024) return fail(ctx, PRISM_E_ARG, "experts: too many of them");
    if (smem > 48 * 1024) PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    launch_pdl(ctx, "moe_route_kernel", moe_route_kernel, (tokens + MR_WARPS - 1) / MR_WARPS, MR_WARPS * 32, smem, r, plan, tokens, (uint32_t)!sorted);
    PRISM_TRY(after_launch(ctx, "moe_route_kernel"));
    if (!sorted) return PRISM_OK;
    launch_pdl(ctx, "moe_sort_kernel", moe_sort_kernel, plan.experts, MS_THREADS, 0, plan, tokens * plan.top);
    return after_launch(ctx, "moe_sort_kernel");
}

template <typename T16>
__global__ void __launch_bounds__(128) moe_gather_kernel(const MoePlan plan, const T16 *__restrict__ x, uint32_t x_pitch, T16 *__restrict__ y,
                                                         uint32_t y_pitch, uint32_t n) {
    pdl_launch_dependents();
    pdl_wait();
    const T16 *s = x + (size_t)(plan.order[blockIdx.x] / plan.top) * x_pitch;
    for (uint32_t i = threadIdx.x; i < n; i += 128) y[(size_t)blockIdx.x * y_pitch + i] = s[i];
}
int launch_moe_gather(prism_cuda_ctx *ctx, const MoePlan &plan, const void *x, uint32_t x_pitch, void *y, uint32_t y_pitch, uint32_t width, uint32_t pairs,
                      bool act32) {
    const uint32_t per = act32 ? 4 : 8;  // values in 16 bytes; rows are padded to them
    if (x_pitch % per || y_pitch % per || ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y)) & 15))
        return fail(ctx, PRISM_E_ARG, "experts: rows must be 16-byte aligned");
    launch_pdl(ctx, "moe_gather_kernel", moe_gather_kernel<uint4>, pairs, 128, 0, plan, (const uint4 *)x, x_pitch / per, (uint4 *)y, y_pitch / per,
               (width + per - 1) / per);
    return after_launch(ctx, "moe_gather_kernel");
}

}  // namespace prism
