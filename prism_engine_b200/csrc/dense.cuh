// Dense bf16 linears and the element-wise pieces of the layer-list models: weight layout, epilogue
// (shared by the tensor-core GEMM, the small-batch kernel and the 32-bit kernel) and launchers.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace prism {

using bf16 = __nv_bfloat16;

// ---------------------------------------------------------------------------
// Device layout of a dense weight: bf16, rows padded to 128 and k to 64 with zeros,
//   w : [row tile of 128][k/8][128 rows][8 k]
// i.e. 16-byte units of eight consecutive k of one row.  64 k of a row tile are one contiguous 16 KB
// run that already has the K-major core-matrix order of a tcgen05 shared-memory operand (one bulk copy
// per pipeline stage), and eight rows of one k/8 are one contiguous 128-byte line for the small-batch
// kernel, whose lanes hold mma fragments straight from these units.
//
// Several linears of the same input are stacked along the rows (each "segment" starts on a row tile and
// has its own epilogue); two linears that are added together can be stacked along k instead.  A segment may
// read a second input, or only the first columns of its input (a segment that differs in this from the one
// before it starts on an even row tile, so that a pair of row tiles shares its input).
//
// A stack of experts is one such layout repeated `experts` times; a MoePlan says which rows go through which.
// ---------------------------------------------------------------------------
enum DenseAct : uint32_t { ACT_NONE = 0, ACT_SILU = 1, ACT_SIGMOID = 2, ACT_GELU_TANH = 3, ACT_RELU2 = 4 };
enum DenseStore : uint32_t { ST_ACT = 0, ST_F32 = 1, ST_RESID = 2 };  // activation type, fp32, fp32 +=
constexpr uint32_t DENSE_MAX_SEGS = 12;

struct DenseSeg {
    uint32_t row0 = 0, rows = 0;  // first row in the stacked weight (multiple of 128), valid rows
    uint32_t in = 0, k = 0;       // which input it reads; columns of it (multiple of 64), 0: all
    uint32_t act = ACT_NONE;
    float mul = 1.0f;             // y = act(W x + bias) * mul
    const float *bias = nullptr;  // fp32 [rows] or null
};
struct DenseLinear {
    bf16 *w = nullptr;
    uint32_t k_pad = 0, n_tiles = 0, n_segs = 0;  // row tiles (of one expert)
    uint32_t experts = 1;
    DenseSeg seg[DENSE_MAX_SEGS];
    size_t bytes() const { return ((size_t)n_tiles * experts + 1) / 2 * 2 * 128 * k_pad * 2; }  // whole pairs of row tiles
    uint64_t valid_rows() const {
        uint64_t r = 0;
        for (uint32_t s = 0; s < n_segs; s++) r += seg[s].rows;
        return r;
    }
};
// Where a segment's output goes: rows `pitch` elements apart.
struct DenseOut {
    void *p = nullptr;
    uint32_t pitch = 0;
    uint32_t store = ST_ACT;
};

// Input rows of a linear.  With norm_w the first n_norm entries of a row are RMS-normalised together (times
// norm_w, and times gate when given); the rest of the row is taken as it is.
struct DenseIn {
    const void *x = nullptr;      // activation type, or fp32 when f32 is set
    uint32_t pitch = 0;           // elements between rows
    uint32_t f32 = 0;
    const float *norm_w = nullptr;
    uint32_t n_norm = 0;
    float eps = 0.0f;
    const void *gate = nullptr;   // activation type
    uint32_t gate_pitch = 0;
    const void *x2 = nullptr;     // second input (activation type, plain)
    uint32_t pitch2 = 0;
};

// Which (token, choice) pairs of a mixture-of-experts layer go through which expert; pair p = token * top + choice.
// Written on the device by launch_moe_route, so a captured step serves any routing.
struct MoePlan {
    uint32_t experts = 0, top = 0;
    uint32_t *idx = nullptr;      // [pairs] chosen expert
    float *wgt = nullptr;         // [pairs] its weight
    // few tokens (at most DENSE_GEMV_ROWS): the experts in use and, for each, the pair of every token (-1: none)
    uint32_t *n_active = nullptr, *active = nullptr;
    int32_t *pair_of = nullptr;   // [active][DENSE_GEMV_ROWS]
    // more tokens: pairs sorted by expert
    uint32_t *count = nullptr;    // [experts]
    uint32_t *order = nullptr;    // [row] pair
    uint32_t *inv = nullptr;      // [pair] row
};

struct DenseEpiSeg {
    uint32_t row0, rows, act, store, pitch, in, k;
    float mul;
    const float *bias;
    void *p;
};
struct DenseEpi {
    uint32_t n;
    DenseEpiSeg s[DENSE_MAX_SEGS];
};

#ifdef __CUDACC__
__device__ __forceinline__ float ld_act(const bf16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float ld_act(const float *p) { return *p; }
__device__ __forceinline__ void st_act(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void st_act(float *p, float v) { *p = v; }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dense_act(uint32_t act, float z) {
    switch (act) {
    case ACT_SILU: return z * sigmoid_f(z);
    case ACT_SIGMOID: return sigmoid_f(z);
    case ACT_GELU_TANH: return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    case ACT_RELU2: return z > 0.0f ? z * z : 0.0f;
    default: return z;
    }
}
// Segment that holds row `row` of a stacked weight.
__device__ __forceinline__ const DenseEpiSeg &dense_seg(const DenseEpi &e, uint32_t row) {
    uint32_t s = 0;
    while (s + 1 < e.n && row >= e.s[s + 1].row0) s++;
    return e.s[s];
}
// By one warp: the tile `tile` (of nt rows) of the rows sorted by expert -- its expert, first row, and rows of that
// expert from there on; false past the last tile.
__device__ __forceinline__ bool moe_find_tile(const uint32_t *__restrict__ count, uint32_t experts, uint32_t nt, uint32_t tile, uint32_t &expert,
                                              uint32_t &row0, uint32_t &left) {
    const uint32_t lane = threadIdx.x & 31;
    uint32_t tiles = 0, rows = 0;  // before this group of 32 experts
    for (uint32_t e0 = 0; e0 < experts; e0 += 32) {
        const uint32_t c = e0 + lane < experts ? count[e0 + lane] : 0;
        uint32_t t = (c + nt - 1) / nt, r = c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const uint32_t a = __shfl_up_sync(0xFFFFFFFFu, t, o), b = __shfl_up_sync(0xFFFFFFFFu, r, o);
            if ((int)lane >= o) { t += a; r += b; }
        }
        const uint32_t hit = __ballot_sync(0xFFFFFFFFu, tile < tiles + t);
        if (hit) {
            const int l = __ffs(hit) - 1;
            const uint32_t ct = __shfl_sync(0xFFFFFFFFu, c, l), te = tiles + __shfl_sync(0xFFFFFFFFu, t, l), re = rows + __shfl_sync(0xFFFFFFFFu, r, l);
            const uint32_t first = te - (ct + nt - 1) / nt, skip = (tile - first) * nt;
            expert = e0 + l;
            row0 = re - ct + skip;
            left = ct - skip;
            return true;
        }
        tiles += __shfl_sync(0xFFFFFFFFu, t, 31);
        rows += __shfl_sync(0xFFFFFFFFu, r, 31);
    }
    return false;
}
// Stores output `row` (inside the segment) of token t.
template <typename TA>
__device__ __forceinline__ void dense_store(const DenseEpiSeg &s, uint32_t row, uint32_t t, float acc) {
    const float v = dense_act(s.act, acc + (s.bias ? __ldg(s.bias + row) : 0.0f)) * s.mul;
    const size_t at = (size_t)t * s.pitch + row;
    if (s.store == ST_ACT) st_act(reinterpret_cast<TA *>(s.p) + at, v);
    else if (s.store == ST_F32) reinterpret_cast<float *>(s.p)[at] = v;
    else reinterpret_cast<float *>(s.p)[at] += v;
}
__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max_f(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, o));
    return v;
}
// Block-wide sum of a value per thread; sh holds 32 floats; every thread gets the result, summed in a fixed order.
__device__ __forceinline__ float block_sum_f(float v, float *sh) {
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum_f(v);
    __syncthreads();
    if (lane == 0) sh[warp] = v;
    __syncthreads();
    float r = 0.0f;
    for (uint32_t i = 0; i < nw; i++) r += sh[i];
    return r;
}
// D += A * B, m16n8k16, bf16 operands, fp32 accumulate.
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x2(uint32_t (&r)[2], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x2_t(uint32_t (&r)[2], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}
// Two floats as a bf16 pair (first in the low half), and what that rounding left over as another pair:
// hi + lo carries 16 bits of each value, so a product with a bf16 operand keeps fp32-like accuracy.
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t *>(&p);
}
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t &hi, uint32_t &lo) {
    const float ah = __bfloat162float(__float2bfloat16_rn(a)), bh = __bfloat162float(__float2bfloat16_rn(b));
    hi = pack_bf16(ah, bh);
    lo = pack_bf16(a - ah, b - bh);
}
// Four consecutive values of a row.
__device__ __forceinline__ float4 ld4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 ld4(const bf16 *p) {
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void st4(bf16 *p, float4 v) { *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }
#endif
// Rows of `n8` 16-byte pieces copied by the threads of a block: 2^row_shift(n8) neighbours take a row.
inline uint32_t row_shift(uint32_t n8) {
    uint32_t s = 0;
    while (s < 5 && (1u << s) < n8) s++;
    return s;
}

// First position that position pos sees under a window (0: none).
#ifdef __CUDACC__
__device__ __forceinline__ int32_t window_first(uint32_t window, int32_t pos) {
    return window && pos + 1 > (int32_t)window ? pos + 1 - (int32_t)window : 0;
}
#endif

// The rows of a step: (state slot, position) of each row.  Device arrays in a decode step (a captured graph
// reads them at every replay); slot == nullptr: consecutive tokens of one slot from position pos0.
struct RowMap {
    const int32_t *slot = nullptr, *pos = nullptr;
    int32_t slot0 = 0, pos0 = 0;
#ifdef __CUDACC__
    __device__ __forceinline__ int32_t slot_of(uint32_t r) const { return slot ? slot[r] : slot0; }
    __device__ __forceinline__ int32_t pos_of(uint32_t r) const { return slot ? pos[r] : pos0 + (int32_t)r; }
#endif
};

// dense.cu
int dense_alloc(prism_cuda_ctx *ctx, DenseLinear &l, uint32_t k_pad, uint32_t n_tiles);
// rows x cols bf16 (row-major, device) into rows row0.., columns k0.. of the stacked layout
int launch_dense_pack(prism_cuda_ctx *ctx, const DenseLinear &l, const bf16 *src, uint32_t rows, uint32_t cols, uint32_t row0,
                      uint32_t k0);  // expert e's rows start at e * n_tiles * 128
// dst = (n / cols rows of src)^T + add, the rows of dst `pitch` apart
int launch_bf16_to_f32(prism_cuda_ctx *ctx, const bf16 *src, float *dst, size_t n, float add, uint32_t cols, uint32_t pitch);
// dst rows `dst_pitch` apart, columns cols..dst_pitch-1 zero
int launch_bf16_pitch_copy(prism_cuda_ctx *ctx, const bf16 *src, bf16 *dst, uint32_t rows, uint32_t cols, uint32_t dst_pitch);
int launch_dense_synth(prism_cuda_ctx *ctx, bf16 *dst, size_t n, uint64_t seed, float mean, float sigma);
DenseEpi dense_epi(const DenseLinear &l, const DenseOut *outs);
// Small batch (bf16, at most DENSE_GEMV_ROWS rows): mma.sync straight from the weight units, the input's norm folded in.
constexpr uint32_t DENSE_GEMV_ROWS = 8;
bool dense_gemv_ok(const DenseIn &in, uint32_t rows);
int launch_dense_gemv(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows);
// 32-bit activations and fp32 products (the weights are exact in fp32): any number of rows, plain inputs
int launch_dense_f32(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows);
// dense_gemm_tc5.cu: tcgen05/TMEM GEMM, bf16 activations, plain inputs, pitches a multiple of 8
int launch_dense_gemm_tc5(prism_cuda_ctx *ctx, const DenseLinear &l, const DenseIn &in, const DenseOut *outs, uint32_t rows);
// Experts.  Few tokens (bf16): output row p = pair p; the input row of a pair is its token's or, by_pair, its own.
int launch_moe_gemv(prism_cuda_ctx *ctx, const DenseLinear &l, const MoePlan &plan, const DenseIn &in, bool by_pair, const DenseOut &out, uint32_t tokens);
// Rows sorted by expert, in and out; `pairs` of them.
int launch_moe_f32(prism_cuda_ctx *ctx, const DenseLinear &l, const MoePlan &plan, const DenseIn &in, const DenseOut &out, uint32_t pairs);
int launch_moe_gemm_tc5(prism_cuda_ctx *ctx, const DenseLinear &l, const MoePlan &plan, const DenseIn &in, const DenseOut &out, uint32_t pairs);
// y[r][0..n) = rms(x[r][0..n)) * w (* gate); y may be x.  f32 says whether x is fp32; act32 whether the activation type is fp32.
int launch_dense_norm(prism_cuda_ctx *ctx, const DenseIn &in, void *y, uint32_t y_pitch, uint32_t rows, bool act32);
// x[r] = table[token r] (+ pos_table[position of r]); x2 (optional): a second copy
int launch_dense_embed(prism_cuda_ctx *ctx, const bf16 *table, uint32_t width, uint32_t vocab, const uint32_t *tokens, uint32_t rows, float *x,
                       const bf16 *pos_table, uint32_t max_pos, const RowMap &map, float *x2);
int launch_gather_rows_f32(prism_cuda_ctx *ctx, const float *x, const uint32_t *idx, uint32_t n, uint32_t width, float *y);
int launch_f32_to_f16(prism_cuda_ctx *ctx, const float *x, uint32_t rows, uint32_t n, uint32_t stride, uint16_t *y, uint32_t y_stride);

// lightning.cu
struct LightningArgs {
    const void *q, *k, *v;        // activation type, rows `pitch` apart, head-major
    uint32_t pitch;
    void *o;                      // [rows] o_pitch apart, heads * vdim
    uint32_t o_pitch;
    float *state;                 // [slot][heads][dim][vdim]
    const float *decay;           // [heads]
    uint32_t heads, dim, vdim, rows;
};
// One token per row, every row another sequence (decode).
int launch_lightning_step(prism_cuda_ctx *ctx, const LightningArgs &a, const RowMap &rows, bool act32);
// The rows are consecutive tokens of one sequence (rows.slot0).
int launch_lightning_seq(prism_cuda_ctx *ctx, const LightningArgs &a, const RowMap &rows, bool act32);

// latent_attn.cu
struct LatentCache {
    void *rows = nullptr;         // activation type: [slot][ring][pitch], a row = kv_rank latent | rot_dim rotated key | zeros
    uint32_t ring = 0, pitch = 0; // position p lives in row p % ring
};
struct LatentArgs {
    uint32_t heads, dim, rot_dim, rot_pairs, vdim, kv_rank, window;  // window 0: every earlier position
    float scale, eps, rot_mul;
    const float *rot_freq;        // [rot_pairs] angle per position
    const float *dkv_norm;        // [kv_rank]
    const bf16 *uk, *uv;          // row-major [heads*dim][uk_pitch] / [heads*vdim][uk_pitch]
    uint32_t uk_pitch;
    LatentCache cache;
};
// Normalises and rotates the rows of W_dkv h and appends them to the cache.
int launch_latent_append(prism_cuda_ctx *ctx, const LatentArgs &a, const void *dkv, uint32_t pitch, const RowMap &rows, uint32_t n_rows, bool act32);
// Rows against the cached latents themselves (W_uk folded into the query, W_uv applied to the weighted latent):
// decode, short portions, and everything in 32-bit.  Appends the rows' latents (dkv) to the cache first.
struct LatentRowsScratch { float *qa; float *part; float *ml; size_t rows_cap; uint32_t splits; };
size_t latent_rows_scratch_floats(const LatentArgs &a, uint32_t splits, size_t *qa, size_t *part, size_t *ml);
uint32_t latent_rows_splits(const LatentArgs &a, uint32_t max_seq);
int launch_latent_rows(prism_cuda_ctx *ctx, const LatentArgs &a, const LatentRowsScratch &s, const void *q, uint32_t q_pitch, const void *dkv,
                       uint32_t dkv_pitch, const void *gate, uint32_t gate_pitch, void *out, uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool act32);
// Prompt portion of one sequence (bf16): keys and values expanded for positions [lo, pos0 + n_rows).
bool latent_expand_ok(const LatentArgs &a);
int launch_latent_gather(prism_cuda_ctx *ctx, const LatentArgs &a, int32_t slot, uint32_t lo, uint32_t n, bf16 *lat, uint32_t lat_pitch, bf16 *krot);
int launch_latent_prefill(prism_cuda_ctx *ctx, const LatentArgs &a, const bf16 *q, uint32_t q_pitch, const bf16 *kx, uint32_t kx_pitch,
                          const bf16 *vx, uint32_t vx_pitch, const bf16 *krot, uint32_t lo, const bf16 *gate, uint32_t gate_pitch, bf16 *out,
                          uint32_t out_pitch, uint32_t pos0, uint32_t n_rows);


// latent_attn.cu: a prompt portion's queries against keys and values laid out per position.
struct TiledAttn {
    uint32_t heads, group;            // query heads; query heads per key/value head
    uint32_t dim, rot_dim, rot_pairs, vdim, window;
    float scale, rot_mul;
    const float *rot_freq;
    const bf16 *q, *kx, *vx, *krot, *gate;  // krot (shared by the heads) and gate may be null
    bf16 *out;
    uint32_t q_pitch, kx_pitch, vx_pitch, gate_pitch, out_pitch;
    uint32_t kx_head, vx_head;        // elements between the key (value) heads of a position, multiples of 8
    uint32_t lo, ring;                // ring 0: position p is row p - lo; else row p % ring
    uint32_t pos0, n_rows;            // first query position, queries
    uint32_t shift;                   // set by the launcher: row_shift of a key's pieces
};
bool tiled_attn_ok(uint32_t dim, uint32_t vdim);
int launch_tiled_attn(prism_cuda_ctx *ctx, const TiledAttn &p);

// grouped_attn.cu: softmax attention whose query heads share key/value heads, no rotation
struct GroupedArgs {
    uint32_t heads, kv_heads, dim, vdim, window;  // window 0: every earlier position
    float scale;
    void *kc, *vc;                    // activation type: [slot][ring][kv_heads][dp] / [..][vp], zero padded
    uint32_t ring, dp, vp;            // position p lives in row p % ring; dim and vdim rounded up to 8
    uint32_t splits;                  // CTAs that share the keys of a row
};
uint32_t grouped_splits(const GroupedArgs &a, uint32_t max_seq);
int launch_grouped_append(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *k, const void *v, uint32_t pitch, const RowMap &rows, uint32_t n_rows,
                          bool act32);
// k, v: null when the rows' keys are in the cache already, else they are appended (rows of different sequences).
// late: the next kernel of the stream is released only once what this one waits for is complete (DeltaArgs::beside).
int launch_grouped_rows(prism_cuda_ctx *ctx, const GroupedArgs &a, const void *q, const void *k, const void *v, uint32_t pitch, void *out,
                        uint32_t out_pitch, const RowMap &rows, uint32_t n_rows, bool act32, bool late = false);
int launch_grouped_prefill(prism_cuda_ctx *ctx, const GroupedArgs &a, const bf16 *q, uint32_t pitch, bf16 *out, uint32_t out_pitch, const RowMap &rows,
                           uint32_t n_rows);

// rowwise.cu
// Causal convolution over the consecutive tokens of one sequence, per channel: y_t = x_t + conv or silu(conv).
// The ring [slot][taps][channels] keeps the inputs of the last positions (position p in row p % taps).
struct ConvPiece { const void *x; void *y; uint32_t channels, c0; };  // c0: first channel in weights and ring
struct ConvArgs {
    ConvPiece piece[3];
    uint32_t pieces, x_pitch, y_pitch, taps, channels;
    const float *w;                   // [taps][channels], the last row meets the current token
    void *ring;
    uint32_t silu;                    // else the input is added
};
int launch_conv_seq(prism_cuda_ctx *ctx, const ConvArgs &a, const RowMap &rows, uint32_t n_rows, bool act32);

// The row-wise end of a sublayer and beginning of the next:
//   x <- x + gate * mul * y,   y = a row | the mean of two RMS-normed rows | the weighted sum of a token's expert outputs
//   history[n] <- x,  x <- sum_j avg[j] history[j]        (depth average)
//   h <- rms(x) * norm,  hc <- h + conv(h)                (input convolution of rows of different sequences)
enum RowAdd : uint32_t { ROW_ADD_NONE = 0, ROW_ADD_ONE = 1, ROW_ADD_PAIR = 2, ROW_ADD_EXPERTS = 3 };
struct RowUpdate {
    const float *x;
    float *x_out;
    uint32_t width, add;
    float eps, mul;
    const void *y, *y2;               // activation type
    uint32_t y_pitch, y2_pitch;
    const float *w, *w2;              // weights of the two norms
    const float *wgt;                 // experts: weight of a pair
    const uint32_t *inv;              // experts: row of a pair (null: the pair itself)
    uint32_t top;
    const void *gate;                 // activation type or null
    uint32_t gate_pitch;
    float *history;                   // null: no depth average
    size_t history_stride;
    const float *avg;
    uint32_t n_history;               // this row becomes history[n_history]
    const float *norm;                // null: no norm
    void *h;
    uint32_t h_pitch;
    const float *conv_w;              // null: no convolution here
    uint32_t taps;
    void *ring, *hc;                  // ring as in ConvArgs; hc rows h_pitch apart
};
int launch_row_update(prism_cuda_ctx *ctx, const RowUpdate &u, const RowMap &rows, uint32_t n_rows, bool act32);

// moe.cu
struct MoeRouter {
    uint32_t groups, keep;            // groups of neighbouring experts, how many of them may be chosen from
    const float *logits, *correction; // fp32 [token][pitch]; added to the score for the choice only
    uint32_t pitch;
};
// plan.idx and plan.wgt of every token; then the few-token part of the plan, or the rows sorted by expert.
int launch_moe_route(prism_cuda_ctx *ctx, const MoeRouter &r, const MoePlan &plan, uint32_t tokens, bool sorted);
// y[row] = x[token of the pair at row]
int launch_moe_gather(prism_cuda_ctx *ctx, const MoePlan &plan, const void *x, uint32_t x_pitch, void *y, uint32_t y_pitch, uint32_t width, uint32_t pairs,
                      bool act32);

// delta.cu: gated delta rule, S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
struct DeltaArgs {
    uint32_t heads, kv_heads, dim, vdim, taps, rows;
    float eps;
    const void *q, *k, *v;            // activation type, rows `pitch` apart: projections (step) or convolved (sequence)
    uint32_t pitch;
    const float *ba;                  // fp32 [rows] ba_pitch apart: step size | decay projections, heads each
    uint32_t ba_pitch;
    const void *gate;                 // activation type: silu of the gate projection
    uint32_t gate_pitch;
    const float *a_log, *dt_bias, *norm;
    const float *conv_w;              // [taps][channels]: q | k | v channels
    void *ring;                       // [slot][taps][channels]
    float *state;                     // [slot][heads][dim][vdim]
    void *o;                          // [rows] o_pitch apart, heads * vdim
    uint32_t o_pitch;
    float *o32;                       // sequence: outputs before their norm, [rows][heads * vdim]
    void *chunk_scratch;              // sequence: delta_scratch_bytes
    uint32_t channels;                // 2 * kv_heads * dim + heads * vdim
    // step: runs beside the kernel launched before it, which has released its dependents only after its own
    // dependency wait: what this one reads is there when it starts, and it waits for that kernel at its end
    uint32_t beside;
};
size_t delta_scratch_bytes(const DeltaArgs &a, uint32_t rows);
int launch_delta_step(prism_cuda_ctx *ctx, const DeltaArgs &a, const RowMap &rows, bool act32);
int launch_delta_seq(prism_cuda_ctx *ctx, const DeltaArgs &a, const RowMap &rows, bool act32);

}  // namespace prism
