// Dense bf16 GEMM on tcgen05 / TMEM with the segment epilogues of dense.cuh:
//   y[t][n] = epilogue( sum_k x[t][k] * W[n][k] ),  fp32 accumulate.
//
// A persistent CTA computes tiles of RT x 128 weight rows x NT rows of x (RT = 2 reads x once for two row tiles:
// a 128-row tile needs more operand bytes per cycle than L2 delivers to all SMs).  One warp loads: the weights of a
// 64-k stage are one contiguous 16 KB run (dense.cuh), fetched by a 1-D bulk copy straight into the
// unswizzled core-matrix order of the A operand; the rows of x come through a tensor map with the
// 128-byte swizzle of the B operand (rows past the end are filled with zeros).  One thread issues the
// tcgen05.mma; four warps per accumulator read it back, apply the epilogue of the tile's segment and store.
// Two accumulators in TMEM: successive tiles alternate between them (RT = 1) or each row tile has its own
// (RT = 2), so that an epilogue overlaps the loads and, for RT = 1, the products of the next tile.
// Every mbarrier wait is bounded; one that gives up raises the context's device error word.
#include <cuda.h>

#include <algorithm>

#include "dense.cuh"
#include "tc5_ptx.cuh"

namespace prism {

constexpr int DG_A_BYTES = 128 * 64 * 2;      // weights of a stage and row tile
template <int NT, int RT>
struct DgCfg {
    static constexpr int THREADS = 64 + 128 * RT;  // loader warp, MMA warp, four epilogue warps per row tile
    static constexpr int A_BYTES = RT * DG_A_BYTES, B_BYTES = NT * 128;
    static constexpr int STAGE = A_BYTES + B_BYTES;
    static constexpr int S = (200 * 1024 / STAGE) < 8 ? (200 * 1024 / STAGE) : 8;
    static constexpr int TMEM_COLS = 2 * NT < 32 ? 32 : 2 * NT;
    static constexpr int BAR_OFF = S * STAGE;
    static constexpr int TAB_OFF = BAR_OFF + 8 * (2 * S + 4) + 64;
    static constexpr size_t SMEM = TAB_OFF + 1024;  // + slack for the 1 KB alignment of the stages; experts: + their table
};

struct DgArgs {
    const uint8_t *w;
    uint32_t kb;              // 64-k stages per row
    uint32_t n_rt, n_tt, rt_group;  // row tiles (of RT x 128), token tiles, row tiles per group of the walk
    uint32_t rows;            // rows of x
    unsigned int *err;
    DenseEpi epi;
    uint32_t experts;         // 0: plain; else rows of x are sorted by expert and a token tile belongs to one
    const uint32_t *count;    // [experts] rows
};
constexpr uint32_t DG_MAX_EXPERTS = 1024;

__device__ __forceinline__ void tma_2d(uint32_t dst, const CUtensorMap *map, int32_t x, int32_t y, uint32_t mbar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];\n" ::"r"(dst),
                 "l"(map), "r"(x), "r"(y), "r"(mbar)
                 : "memory");
}
__device__ __forceinline__ void mma_ss(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}\n" ::"r"(d_tmem),
        "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
        : "memory");
}
// K-major operand with the 128-byte swizzle: rows of 128 bytes, eight-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t desc_sw128(uint32_t addr) {
    return (uint64_t)((addr & 0x3FFFFu) >> 4) | (uint64_t)1 << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}

// Walk of the tiles: groups of rt_group row tiles over all token tiles, so that the CTAs of one wave share a
// few weights and a few rows of x in L2.
__device__ __forceinline__ void dg_item(const DgArgs &a, uint32_t w, uint32_t &rt, uint32_t &tt) {
    const uint32_t per = a.rt_group * a.n_tt, g = w / per, rem = w % per;
    const uint32_t gr = min(a.rt_group, a.n_rt - g * a.rt_group);
    rt = g * a.rt_group + rem % gr;
    tt = rem / gr;
}

// The epilogue of dense_store for one weight row (a lane) over the NT tokens of a tile, with what does not change
// along the way decided once: sixteen accumulators are read, the residual's old values requested together, and
// the activation of a bf16 result takes the fast exponential and reciprocal.
template <uint32_t ACT>
__device__ __forceinline__ float act_fast(float z) {
    if (ACT == ACT_NONE) return z;
    if (ACT == ACT_RELU2) return z > 0.0f ? z * z : 0.0f;
    const float u = ACT == ACT_GELU_TANH ? 1.5957691216057308f * (z + 0.044715f * z * z * z) : z;  // (1 + tanh(u / 2)) / 2 = sigmoid(u)
    const float g = __fdividef(1.0f, 1.0f + __expf(-u));
    return ACT == ACT_SIGMOID ? g : z * g;
}
template <int NT, uint32_t ACT, uint32_t STORE>
__device__ __forceinline__ void epilogue_row(const DenseEpiSeg &seg, uint32_t row, bool row_ok, uint32_t taddr, uint32_t t0, uint32_t rows) {
    const float bias = seg.bias && row_ok ? __ldg(seg.bias + row) : 0.0f, mul = seg.mul;
    const uint32_t pitch = seg.pitch;
    bf16 *yh = reinterpret_cast<bf16 *>(seg.p) + (size_t)t0 * pitch + row;
    float *yf = reinterpret_cast<float *>(seg.p) + (size_t)t0 * pitch + row;
    const uint32_t n = rows > t0 ? min(rows - t0, (uint32_t)NT) : 0;
#pragma unroll 1
    for (uint32_t g = 0; g < n; g += 16) {
        uint32_t v[16];
        float old[16];
        t5::ld16(taddr + g, v);
        if (STORE == ST_RESID) {
#pragma unroll
            for (uint32_t i = 0; i < 16; i++) old[i] = row_ok && g + i < n ? yf[(size_t)(g + i) * pitch] : 0.0f;
        }
        t5::wait_ld();
#pragma unroll
        for (uint32_t i = 0; i < 16; i++) {
            const float y = act_fast<ACT>(__uint_as_float(v[i]) + bias) * mul;
            if (row_ok && g + i < n) {
                if (STORE == ST_ACT) yh[(size_t)(g + i) * pitch] = __float2bfloat16_rn(y);
                else yf[(size_t)(g + i) * pitch] = STORE == ST_RESID ? old[i] + y : y;
            }
        }
        __syncwarp();  // the next TMEM read takes the whole warp
    }
}

template <int NT, int RT, bool MOE>
__global__ void __launch_bounds__(DgCfg<NT, RT>::THREADS, 1) dense_gemm_tc5_kernel(const DgArgs a, const __grid_constant__ CUtensorMap xmap,
                                                                                   const __grid_constant__ CUtensorMap xmap2) {
    using C = DgCfg<NT, RT>;
    extern __shared__ uint8_t dg_smem_raw[];
    uint8_t *smem = dg_smem_raw + (1024 - ((uint32_t)__cvta_generic_to_shared(dg_smem_raw) & 1023u)) % 1024;
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
    pdl_launch_dependents();
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t b_full = base + C::BAR_OFF, b_empty = b_full + 8 * C::S, b_dfull = b_empty + 8 * C::S, b_dempty = b_dfull + 16;
    const uint32_t state = C::BAR_OFF + 8 * (2 * C::S + 4);
    volatile uint32_t *err_flag = reinterpret_cast<volatile uint32_t *>(smem + state);
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(smem + state + 8);
    uint32_t n_items = a.n_rt * a.n_tt;
    uint32_t *tile_end = reinterpret_cast<uint32_t *>(smem + C::TAB_OFF), *row_end = tile_end + a.experts;  // experts: running sums of tiles and rows
    if (tid == 0) {
        for (int s = 0; s < C::S; s++) { t5::mbar_init(b_full + 8 * s, 1); t5::mbar_init(b_empty + 8 * s, 1); }
        for (int b = 0; b < 2; b++) { t5::mbar_init(b_dfull + 8 * b, 1); t5::mbar_init(b_dempty + 8 * b, 4); }
        *err_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) t5::tmem_alloc(base + state + 8, C::TMEM_COLS);
    t5::fence_before();
    __syncthreads();
    t5::fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_wait();  // before any bounded wait: the kernel before this one may still be at work
    if (MOE) {
        if (warp == 2) {
            uint32_t tiles = 0, rows = 0;
            for (uint32_t e0 = 0; e0 < a.experts; e0 += 32) {
                uint32_t r = e0 + lane < a.experts ? a.count[e0 + lane] : 0, t = (r + NT - 1) / NT;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const uint32_t x = __shfl_up_sync(0xFFFFFFFFu, t, o), y = __shfl_up_sync(0xFFFFFFFFu, r, o);
                    if ((int)lane >= o) { t += x; r += y; }
                }
                if (e0 + lane < a.experts) { tile_end[e0 + lane] = tiles + t; row_end[e0 + lane] = rows + r; }
                tiles += __shfl_sync(0xFFFFFFFFu, t, 31);
                rows += __shfl_sync(0xFFFFFFFFu, r, 31);
            }
        }
        __syncthreads();
        n_items = a.n_rt * tile_end[a.experts - 1];
    }
    // An item's weights (row tile, counted over all experts), first row of x and the row of x it ends before.
    auto item = [&](uint32_t w, uint32_t &rt, uint32_t &wt, uint32_t &t0, uint32_t &t_end) {
        if (!MOE) {
            uint32_t tt;
            dg_item(a, w, rt, tt);
            wt = rt * RT;
            t0 = tt * NT;
            t_end = a.rows;
        } else {
            const uint32_t tt = w / a.n_rt;
            rt = w % a.n_rt;
            uint32_t lo = 0, hi = a.experts - 1;  // first expert with tile_end > tt
            while (lo < hi) {
                const uint32_t mid = (lo + hi) / 2;
                if (tile_end[mid] > tt) hi = mid; else lo = mid + 1;
            }
            const uint32_t first = lo ? tile_end[lo - 1] : 0, r0 = lo ? row_end[lo - 1] : 0;
            wt = lo * a.n_rt * RT + rt * RT;
            t0 = r0 + (tt - first) * NT;
            t_end = row_end[lo];
        }
    };

    if (warp == 0) {
        if (lane == 0) {
            uint32_t n = 0;
            for (uint32_t w = blockIdx.x; w < n_items; w += gridDim.x) {
                uint32_t rt, wt, t0, t_end;
                item(w, rt, wt, t0, t_end);
                const DenseEpiSeg &seg = dense_seg(a.epi, rt * RT * 128);
                const uint32_t kb = seg.k / 64;
                const CUtensorMap *map = seg.in ? &xmap2 : &xmap;
                const uint8_t *wsrc = a.w + (size_t)wt * a.kb * DG_A_BYTES;
                for (uint32_t k = 0; k < kb; k++, n++) {
                    const uint32_t s = n % C::S, ph = (n / C::S) & 1, dst = base + s * C::STAGE;
                    t5::mbar_wait_bounded(b_empty + 8 * s, ph ^ 1, err_flag);
                    t5::mbar_arrive_expect_tx(b_full + 8 * s, C::STAGE);
#pragma unroll
                    for (int r = 0; r < RT; r++)
                        t5::bulk_g2s(dst + r * DG_A_BYTES, wsrc + ((size_t)r * a.kb + k) * DG_A_BYTES, DG_A_BYTES, b_full + 8 * s);
                    tma_2d(dst + C::A_BYTES, map, (int32_t)(k * 64), (int32_t)t0, b_full + 8 * s);
                }
            }
            // every copy in flight lands before the CTA leaves (a stage's last use is committed to its empty barrier)
            for (uint32_t i = 0; i < (uint32_t)C::S && i < n; i++) {
                const uint32_t m = n - 1 - i, s = m % C::S;
                t5::mbar_wait_bounded(b_full + 8 * s, (m / C::S) & 1, err_flag);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = t5::idesc_f16(128, NT) | (1u << 7) | (1u << 10);  // A and B bf16
            uint32_t n = 0, ti = 0;
            for (uint32_t w = blockIdx.x; w < n_items; w += gridDim.x, ti++) {
                uint32_t rt, wt, t0, t_end;
                item(w, rt, wt, t0, t_end);
                const uint32_t kb = dense_seg(a.epi, rt * RT * 128).k / 64;
                if (RT == 1) {
                    t5::mbar_wait_bounded(b_dempty + 8 * (ti & 1), ((ti >> 1) & 1) ^ 1, err_flag);
                    t5::fence_after();
                }
                for (uint32_t k = 0; k < kb; k++, n++) {
                    const uint32_t s = n % C::S, ph = (n / C::S) & 1, sa = base + s * C::STAGE, sb = sa + C::A_BYTES;
                    t5::mbar_wait_bounded(b_full + 8 * s, ph, err_flag);
                    t5::fence_after();
#pragma unroll
                    for (int r = 0; r < RT; r++) {
                        if (RT == 2 && k == 0) {
                            t5::mbar_wait_bounded(b_dempty + 8 * r, (ti & 1) ^ 1, err_flag);
                            t5::fence_after();
                        }
                        const uint32_t d = tmem + (RT == 1 ? ti & 1 : r) * NT;
#pragma unroll
                        for (int j = 0; j < 4; j++)  // 16 k each: two k/8 slabs of 2 KB in A, 32 bytes inside the swizzled rows of B
                            mma_ss(d, t5::smem_desc(sa + r * DG_A_BYTES + j * 4096, 2048, 128), desc_sw128(sb + j * 32), idesc, (k | j) != 0);
                    }
                    t5::commit(b_empty + 8 * s);
                }
                if (RT == 1) {
                    t5::commit(b_dfull + 8 * (ti & 1));
                } else {
                    t5::commit(b_dfull);
                    t5::commit(b_dfull + 8);
                }
            }
        }
    } else {
        const uint32_t q = warp & 3, er = (warp - 2) >> 2;  // the TMEM lanes a warp may read; its row tile
        uint32_t ti = 0;
        for (uint32_t w = blockIdx.x; w < n_items; w += gridDim.x, ti++) {
            uint32_t rt, wt, t0, t_end;
            item(w, rt, wt, t0, t_end);
            const uint32_t b = RT == 1 ? ti & 1 : er, ph = RT == 1 ? (ti >> 1) & 1 : ti & 1, row0 = (rt * RT + er) * 128;
            const DenseEpiSeg &seg = dense_seg(a.epi, row0);
            const uint32_t row = row0 + q * 32 + lane - seg.row0;
            const bool row_ok = row < seg.rows;
            t5::mbar_wait_warp(b_dfull + 8 * b, ph, err_flag);
            t5::fence_after();
            const uint32_t taddr = tmem + ((q * 32) << 16) + b * NT;
            switch (seg.store * 8 + seg.act) {
            case ST_ACT * 8 + ACT_NONE: epilogue_row<NT, ACT_NONE, ST_ACT>(seg, row, row_ok, taddr, t0, t_end); break;
            case ST_ACT * 8 + ACT_SILU: epilogue_row<NT, ACT_SILU, ST_ACT>(seg, row, row_ok, taddr, t0, t_end); break;
            case ST_ACT * 8 + ACT_SIGMOID: epilogue_row<NT, ACT_SIGMOID, ST_ACT>(seg, row, row_ok, taddr, t0, t_end); break;
            case ST_ACT * 8 + ACT_GELU_TANH: epilogue_row<NT, ACT_GELU_TANH, ST_ACT>(seg, row, row_ok, taddr, t0, t_end); break;
            case ST_ACT * 8 + ACT_RELU2: epilogue_row<NT, ACT_RELU2, ST_ACT>(seg, row, row_ok, taddr, t0, t_end); break;
            case ST_F32 * 8 + ACT_NONE: epilogue_row<NT, ACT_NONE, ST_F32>(seg, row, row_ok, taddr, t0, t_end); break;
            default: epilogue_row<NT, ACT_NONE, ST_RESID>(seg, row, row_ok, taddr, t0, t_end); break;  // the launcher rejects the rest
            }
            t5::fence_before();
            __syncwarp();
            if (lane == 0) t5::mbar_arrive(b_dempty + 8 * b);
        }
    }
    t5::fence_before();
    __syncthreads();
    t5::fence_after();
    if (warp == 1) t5::tmem_dealloc(tmem, C::TMEM_COLS);
    if (tid == 0 && *err_flag) atomicExch(a.err, 5u);
}

// ---- host side ---------------------------------------------------------------------------------
typedef CUresult (*TensorMapEncode)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                    const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                                    CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static TensorMapEncode tensor_map_encode() {
    static TensorMapEncode fn = [] {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult st;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &st) != cudaSuccess || st != cudaDriverEntryPointSuccess)
            p = nullptr;
        return reinterpret_cast<TensorMapEncode>(p);
    }();
    return fn;
}

static int encode_x(prism_cuda_ctx *ctx, CUtensorMap *map, const void *x, uint32_t pitch, uint32_t k, uint32_t rows, uint32_t nt) {
    TensorMapEncode enc = tensor_map_encode();
    if (!enc) return fail(ctx, PRISM_E_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t dims[2] = {k, rows}, strides[1] = {(cuuint64_t)pitch * 2};
    const cuuint32_t box[2] = {64, nt}, estr[2] = {1, 1};
    const CUresult rc = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(x), dims, strides, box, estr,
                            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return rc == CUDA_SUCCESS ? PRISM_OK : fail(ctx, PRISM_E_CUDA, "cuTensorMapEncodeTiled failed: " + std::to_string((int)rc));
}

template <int NT, int RT, bool MOE>
static int launch_dg(prism_cuda_ctx *ctx, const DenseLinear &l, DgArgs &a, const DenseIn &in) {
    using C = DgCfg<NT, RT>;
    const size_t smem = C::SMEM + (MOE ? 8 * DG_MAX_EXPERTS : 0);
    static bool configured[PRISM_MAX_DEVICES] = {false};
    if (!configured[ctx->device]) {
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(dense_gemm_tc5_kernel<NT, RT, MOE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured[ctx->device] = true;
    }
    CUtensorMap map, map2;
    uint32_t k[2] = {0, 0};  // columns of each input that a segment reads
    for (uint32_t i = 0; i < a.epi.n; i++) k[a.epi.s[i].in] = std::max(k[a.epi.s[i].in], a.epi.s[i].k);
    PRISM_TRY(encode_x(ctx, &map, in.x, in.pitch, std::max(k[0], 64u), a.rows, NT));
    if (k[1]) PRISM_TRY(encode_x(ctx, &map2, in.x2, in.pitch2, k[1], a.rows, NT));
    else map2 = map;
    const uint32_t G = (uint32_t)ctx->sm_count;
    a.n_rt = (l.n_tiles + RT - 1) / RT;
    if (MOE) {
        a.n_tt = a.rows / NT + std::min(a.rows, a.experts);  // at most
    } else {
        a.n_tt = (a.rows + NT - 1) / NT;
        a.rt_group = std::min(a.n_rt, std::max(1u, (G + a.n_tt - 1) / a.n_tt));
    }
    const uint32_t grid = std::min(G, a.n_rt * a.n_tt);
    launch_pdl(ctx, "dense_gemm_tc5_kernel", dense_gemm_tc5_kernel<NT, RT, MOE>, dim3(grid), dim3(C::THREADS), smem, a, map, map2);
    return after_launch(ctx, "dense_gemm_tc5_kernel");
}

// Tile shape with the least estimated time: waves x cycles of a 64-k stage, which the tensor core bounds by
// 2 NT RT and the loads by what L2 delivers to the CTAs at work (about 6000 bytes per cycle in all).
// `tt(nt)`: token tiles of nt rows.
template <bool MOE, typename F>
static int launch_best(prism_cuda_ctx *ctx, const DenseLinear &l, DgArgs &a, const DenseIn &in, F &&tt) {
    struct Shape { uint32_t nt, rt; };
    static const Shape shapes[] = {{256, 2}, {128, 2}, {64, 2}, {256, 1}, {128, 1}, {64, 1}, {32, 1}, {16, 1}};
    const uint32_t G = (uint32_t)ctx->sm_count;
    Shape best{16, 1};
    double best_t = 1e30;
    for (const Shape &s : shapes) {
        if (MOE && s.rt == 2 && l.n_tiles % 2) continue;  // a pair of row tiles lies inside an expert
        const uint64_t items = (uint64_t)((l.n_tiles + s.rt - 1) / s.rt) * tt(s.nt);
        const double bytes = s.rt * DG_A_BYTES + s.nt * 128.0, act = (double)std::min<uint64_t>(items, G);
        const double t = (double)((items + G - 1) / G) * std::max({2.0 * s.nt * s.rt, bytes * act / 6000.0, bytes / 100.0});
        if (t < best_t * 0.999) {
            best_t = t;
            best = s;
        }
    }
    switch (best.nt * 4 + best.rt) {
    case 256 * 4 + 2: return launch_dg<256, 2, MOE>(ctx, l, a, in);
    case 128 * 4 + 2: return launch_dg<128, 2, MOE>(ctx, l, a, in);
    case 64 * 4 + 2: return launch_dg<64, 2, MOE>(ctx, l, a, in);
    case 256 * 4 + 1: return launch_dg<256, 1, MOE>(ctx, l, a, in);
    case 128 * 4 + 1: return launch_dg<128, 1, MOE>(ctx, l, a, in);
    case 64 * 4 + 1: return launch_dg<64, 1, MOE>(ctx, l, a, in);
    case 32 * 4 + 1: return launch_dg<32, 1, MOE>(ctx, l, a, in);
    default: return launch_dg<16, 1, MOE>(ctx, l, a, in);
    }
}

static int dg_args(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows, DgArgs &a) {
    a.w = reinterpret_cast<const uint8_t *>(l.w);
    a.kb = l.k_pad / 64;
    a.rows = rows;
    a.err = ctx->dev_err;
    a.epi = dense_epi(l, outs);
    for (uint32_t i = 0; i < l.n_segs; i++) {
        const DenseEpiSeg &s = a.epi.s[i];
        const void *x = s.in ? in.x2 : in.x;
        const uint32_t pitch = s.in ? in.pitch2 : in.pitch;
        if (!x || (reinterpret_cast<uintptr_t>(x) & 15) || pitch % 8 || pitch < s.k || s.k % 64)
            return fail(ctx, PRISM_E_ARG, "dense gemm: input rows must be 16-byte aligned and hold the padded k range");
        if (i && (s.in != a.epi.s[i - 1].in || s.k != a.epi.s[i - 1].k) && s.row0 % 256)
            return fail(ctx, PRISM_E_ARG, "dense gemm: a segment with another input must start on an even row tile");
        if (s.store != ST_ACT && s.act != ACT_NONE) return fail(ctx, PRISM_E_ARG, "dense gemm: fp32 outputs take no activation");
    }
    return PRISM_OK;
}

int launch_dense_gemm_tc5(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows) {
    DgArgs a{};
    PRISM_TRY(dg_args(ctx, l, in, outs, rows, a));
    return launch_best<false>(ctx, l, a, in, [&](uint32_t nt) { return (rows + nt - 1) / nt; });
}

int launch_moe_gemm_tc5(prism_cuda_ctx *ctx, const DenseLinear &l, const MoePlan &plan, const DenseIn &in, const DenseOut &out, uint32_t pairs) {
    if (plan.experts > DG_MAX_EXPERTS || l.n_segs != 1) return fail(ctx, PRISM_E_ARG, "experts: at most 1024 of them");
    DgArgs a{};
    PRISM_TRY(dg_args(ctx, l, in, &out, pairs, a));
    a.experts = plan.experts;
    a.count = plan.count;
    // as if the rows were spread evenly over the experts, plus half a tile each for the ragged ends
    return launch_best<true>(ctx, l, a, in, [&](uint32_t nt) {
        const uint32_t used = std::min(pairs, plan.experts), each = (pairs + used - 1) / used;
        return used * ((each + each / 4 + nt - 1) / nt);
    });
}

}  // namespace prism
