// Row-wise work between the linears of the layer-list models: causal convolutions over time per channel, and the
// kernel that ends a sublayer and begins the next (residual, gate, depth average, norm, input convolution).
#include <cooperative_groups.h>

#include <algorithm>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace prism {

// V consecutive values of a row, fp32.
template <int V>
struct Vals { float v[V]; };
template <int V>
__device__ __forceinline__ Vals<V> ldv(const float *p) {
    Vals<V> r;
    if constexpr (V == 4) {
        const float4 u = *reinterpret_cast<const float4 *>(p);
        r.v[0] = u.x; r.v[1] = u.y; r.v[2] = u.z; r.v[3] = u.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V>
__device__ __forceinline__ Vals<V> ldv(const bf16 *p) {
    Vals<V> r;
    if constexpr (V == 4) {
        const uint2 u = *reinterpret_cast<const uint2 *>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&u.y));
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
    } else {
        r.v[0] = __bfloat162float(*p);
    }
    return r;
}
template <int V>
__device__ __forceinline__ void stv(float *p, const Vals<V> &x) {
    if constexpr (V == 4) *reinterpret_cast<float4 *>(p) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
    else *p = x.v[0];
}
template <int V>
__device__ __forceinline__ void stv(bf16 *p, const Vals<V> &x) {
    if constexpr (V == 4) *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16(x.v[0], x.v[1]), pack_bf16(x.v[2], x.v[3]));
    else *p = __float2bfloat16_rn(x.v[0]);
}
// As the activation type holds it.
__device__ __forceinline__ float as_act(float v, const float *) { return v; }
__device__ __forceinline__ float as_act(float v, const bf16 *) { return __bfloat162float(__float2bfloat16_rn(v)); }

// ---- convolution along a portion ---------------------------------------------------------------------------
// Thread: V channels of a strip of tokens; with TAPS the last inputs stay in registers.  Only the first strip reaches
// back before the portion, and the same threads leave the portion's last inputs in the ring after they have read what
// was there.
constexpr int CV_THREADS = 128, CV_STRIP = 16, CV_U = 4;
template <typename TA, int V, int TAPS>
__global__ void __launch_bounds__(CV_THREADS) conv_seq_kernel(const ConvArgs a, const RowMap rows, uint32_t n, uint32_t strip) {
    pdl_launch_dependents();
    uint32_t b = blockIdx.x, pc = 0;
    while (pc + 1 < a.pieces && b >= (a.piece[pc].channels + CV_THREADS * V - 1) / (CV_THREADS * V)) {
        b -= (a.piece[pc].channels + CV_THREADS * V - 1) / (CV_THREADS * V);
        pc++;
    }
    const ConvPiece &p = a.piece[pc];
    const uint32_t c = (b * CV_THREADS + threadIdx.x) * V;
    if (c >= p.channels) return;
    const TA *x = reinterpret_cast<const TA *>(p.x) + c;
    TA *y = reinterpret_cast<TA *>(p.y) + c, *ring = reinterpret_cast<TA *>(a.ring) + (size_t)rows.slot0 * a.taps * a.channels + p.c0 + c;
    const float *w = a.w + p.c0 + c;
    const int32_t T = (int32_t)a.taps - 1, t0 = (int32_t)(blockIdx.y * strip), t1 = min((int32_t)n, t0 + (int32_t)strip);
    auto earlier = [&](int32_t u) {  // the input of the portion's token u, u < t0
        const int32_t pos = rows.pos0 + u;
        if (pos < 0) return Vals<V>{};
        return u >= 0 ? ldv<V>(x + (size_t)u * a.x_pitch) : ldv<V>(ring + (size_t)((uint32_t)pos % a.taps) * a.channels);
    };
    auto finish = [&](TA *to, const Vals<V> &s, const Vals<V> &cur) {
        Vals<V> o;
#pragma unroll
        for (int i = 0; i < V; i++) {
            if (!a.silu) o.v[i] = cur.v[i] + s.v[i];
            else if (sizeof(TA) == 2) o.v[i] = s.v[i] * __fdividef(1.0f, 1.0f + __expf(-s.v[i]));  // rounded to 16 bits
            else o.v[i] = s.v[i] * sigmoid_f(s.v[i]);
        }
        stv<V>(to, o);
    };
    if constexpr (TAPS > 0) {
        Vals<V> wr[TAPS], h[TAPS];  // h[j]: the input TAPS - 1 - j tokens ago
#pragma unroll
        for (int j = 0; j < TAPS; j++) wr[j] = ldv<V>(w + (size_t)j * a.channels);
        pdl_wait();
#pragma unroll
        for (int j = 1; j < TAPS; j++) h[j] = earlier(t0 - TAPS + j);
        const TA *xt = x + (size_t)t0 * a.x_pitch;
        TA *yt = y + (size_t)t0 * a.y_pitch;
        for (int32_t t = t0; t < t1; t += CV_U) {
            Vals<V> in[CV_U];
#pragma unroll
            for (int k = 0; k < CV_U; k++, xt += a.x_pitch)
                if (t + k < t1) in[k] = ldv<V>(xt);
#pragma unroll
            for (int k = 0; k < CV_U; k++, yt += a.y_pitch) {
                if (t + k >= t1) break;
#pragma unroll
                for (int j = 0; j + 1 < TAPS; j++) h[j] = h[j + 1];
                h[TAPS - 1] = in[k];
                Vals<V> s{};
#pragma unroll
                for (int j = 0; j < TAPS; j++)
#pragma unroll
                    for (int i = 0; i < V; i++) s.v[i] = fmaf(wr[j].v[i], h[j].v[i], s.v[i]);
                finish(yt, s, in[k]);
            }
        }
    } else {
        pdl_wait();
        for (int32_t t = t0; t < t1; t++) {
            Vals<V> s{};
            for (int32_t j = 0; j <= T; j++) {
                const Vals<V> h = earlier(t - T + j), wj = ldv<V>(w + (size_t)j * a.channels);
#pragma unroll
                for (int i = 0; i < V; i++) s.v[i] = fmaf(wj.v[i], h.v[i], s.v[i]);
            }
            finish(y + (size_t)t * a.y_pitch, s, ldv<V>(x + (size_t)t * a.x_pitch));
        }
    }
    if (blockIdx.y == 0)
        for (int32_t t = max(0, (int32_t)n - T); t < (int32_t)n; t++)
            stv<V>(ring + (size_t)((uint32_t)(rows.pos0 + t) % a.taps) * a.channels, ldv<V>(x + (size_t)t * a.x_pitch));
}
template <typename TA>
static int run_conv(prism_cuda_ctx *ctx, const ConvArgs &a, const RowMap &rows, uint32_t n) {
    uintptr_t at = reinterpret_cast<uintptr_t>(a.ring) | reinterpret_cast<uintptr_t>(a.w);
    uint32_t odd = a.x_pitch | a.y_pitch | a.channels;
    for (uint32_t i = 0; i < a.pieces; i++) {
        at |= reinterpret_cast<uintptr_t>(a.piece[i].x) | reinterpret_cast<uintptr_t>(a.piece[i].y);
        odd |= a.piece[i].channels | a.piece[i].c0;
    }
    const uint32_t v = (at & 15) || (odd & 3) ? 1 : 4;
    uint32_t blocks = 0;
    for (uint32_t i = 0; i < a.pieces; i++) blocks += (a.piece[i].channels + CV_THREADS * v - 1) / (CV_THREADS * v);
    const uint32_t strip = std::max((uint32_t)CV_STRIP, a.taps);
    const dim3 grid(blocks, (n + strip - 1) / strip);
    auto run = [&](auto kernel) { launch_pdl(ctx, "conv_seq_kernel", kernel, grid, dim3(CV_THREADS), 0, a, rows, n, strip); };
    if (v == 1) run(conv_seq_kernel<TA, 1, 0>);
    else if (a.taps == 2) run(conv_seq_kernel<TA, 4, 2>);
    else if (a.taps == 3) run(conv_seq_kernel<TA, 4, 3>);
    else if (a.taps == 4) run(conv_seq_kernel<TA, 4, 4>);
    else run(conv_seq_kernel<TA, 4, 0>);
    return after_launch(ctx, "conv_seq_kernel");
}
int launch_conv_seq(prism_cuda_ctx *ctx, const ConvArgs &a, const RowMap &rows, uint32_t n_rows, bool act32) {
    return act32 ? run_conv<float>(ctx, a, rows, n_rows) : run_conv<bf16>(ctx, a, rows, n_rows);
}

// ---- end of a sublayer, beginning of the next ----------------------------------------------------------------
// A cluster of CTAs takes a row, each a run of its columns; the updated run waits in shared memory for its norm.
constexpr int RU_THREADS = 256;

// Sum over the cluster of a value per thread; every thread gets it.  slot: one per use.
__device__ __forceinline__ float cluster_sum_f(float v, float *sh, float *slot, uint32_t cs) {
    v = block_sum_f(v, sh);
    if (cs == 1) return v;
    cg::cluster_group cluster = cg::this_cluster();
    if (threadIdx.x == 0) *slot = v;
    cluster.sync();
    float s = 0.0f;
    for (uint32_t r = 0; r < cs; r++) s += *cluster.map_shared_rank(slot, r);
    return s;
}

// Two sums at once (the block's part: sh holds 32 floats, slot two).
__device__ __forceinline__ float2 cluster_sum2_f(float a, float b, float *sh, float *slot, uint32_t cs) {
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum_f(a);
    b = warp_sum_f(b);
    if (lane == 0) {
        sh[warp] = a;
        sh[16 + warp] = b;
    }
    __syncthreads();
    a = b = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < RU_THREADS / 32; i++) {
        a += sh[i];
        b += sh[16 + i];
    }
    if (cs == 1) return make_float2(a, b);
    cg::cluster_group cluster = cg::this_cluster();
    if (threadIdx.x == 0) {
        slot[0] = a;
        slot[1] = b;
    }
    cluster.sync();
    a = b = 0.0f;
    for (uint32_t r = 0; r < cs; r++) {
        a += *cluster.map_shared_rank(slot, r);
        b += *cluster.map_shared_rank(slot + 1, r);
    }
    return make_float2(a, b);
}

template <typename TA, int V>
__global__ void __launch_bounds__(RU_THREADS) row_update_kernel(const RowUpdate u, const RowMap rows, uint32_t cs, uint32_t per) {
    extern __shared__ __align__(16) float xs[];  // [per]
    __shared__ float sh[32], slot[3];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r = blockIdx.y, c_lo = blockIdx.x * per, c_hi = min(c_lo + per, u.width), D = u.width;
    const float *x = u.x + (size_t)r * D;
    const TA *y = reinterpret_cast<const TA *>(u.y) + (size_t)r * u.y_pitch, *y2 = reinterpret_cast<const TA *>(u.y2) + (size_t)r * u.y2_pitch;
    const TA *gate = reinterpret_cast<const TA *>(u.gate) + (size_t)r * u.gate_pitch;
    float inv1 = 0.0f, inv2 = 0.0f;
    if (u.add == ROW_ADD_PAIR) {
        float s1 = 0.0f, s2 = 0.0f;
        for (uint32_t c = c_lo + threadIdx.x * V; c < c_hi; c += RU_THREADS * V) {
            const Vals<V> p = ldv<V>(y + c), q = ldv<V>(y2 + c);
#pragma unroll
            for (int i = 0; i < V; i++) {
                s1 = fmaf(p.v[i], p.v[i], s1);
                s2 = fmaf(q.v[i], q.v[i], s2);
            }
        }
        const float2 q = cluster_sum2_f(s1, s2, sh, slot, cs);
        inv1 = 0.5f / sqrtf(q.x / (float)D + u.eps);
        inv2 = 0.5f / sqrtf(q.y / (float)D + u.eps);
    }
    float ss = 0.0f;
    for (uint32_t c = c_lo + threadIdx.x * V; c < c_hi; c += RU_THREADS * V) {
        Vals<V> v = ldv<V>(x + c), d;
        if (u.add != ROW_ADD_NONE) {
            if (u.add == ROW_ADD_ONE) {
                d = ldv<V>(y + c);
            } else if (u.add == ROW_ADD_PAIR) {
                const Vals<V> p = ldv<V>(y + c), q = ldv<V>(y2 + c), w1 = ldv<V>(u.w + c), w2 = ldv<V>(u.w2 + c);
#pragma unroll
                for (int i = 0; i < V; i++) d.v[i] = p.v[i] * inv1 * w1.v[i] + q.v[i] * inv2 * w2.v[i];
            } else {
#pragma unroll
                for (int i = 0; i < V; i++) d.v[i] = 0.0f;
#pragma unroll 4
                for (uint32_t k = 0; k < u.top; k++) {
                    const uint32_t pair = r * u.top + k, row = u.inv ? u.inv[pair] : pair;
                    const Vals<V> e = ldv<V>(reinterpret_cast<const TA *>(u.y) + (size_t)row * u.y_pitch + c);
                    const float w = u.wgt[pair];
#pragma unroll
                    for (int i = 0; i < V; i++) d.v[i] = fmaf(w, e.v[i], d.v[i]);
                }
            }
            if (u.gate) {
                const Vals<V> g = ldv<V>(gate + c);
#pragma unroll
                for (int i = 0; i < V; i++) d.v[i] *= g.v[i];
            }
#pragma unroll
            for (int i = 0; i < V; i++) v.v[i] = fmaf(u.mul, d.v[i], v.v[i]);
        }
        if (u.history) {
            float *h = u.history + (size_t)r * D + c;
            stv<V>(h + u.n_history * u.history_stride, v);
            const float a = u.avg[u.n_history];
#pragma unroll
            for (int i = 0; i < V; i++) v.v[i] *= a;
#pragma unroll 4
            for (uint32_t j = 0; j < u.n_history; j++) {
                const Vals<V> o = ldv<V>(h + j * u.history_stride);
                const float aj = u.avg[j];
#pragma unroll
                for (int i = 0; i < V; i++) v.v[i] = fmaf(aj, o.v[i], v.v[i]);
            }
        }
        if (u.x_out) stv<V>(u.x_out + (size_t)r * D + c, v);
        stv<V>(xs + c - c_lo, v);
#pragma unroll
        for (int i = 0; i < V; i++) ss = fmaf(v.v[i], v.v[i], ss);
    }
    if (u.norm) {
        const float inv = 1.0f / sqrtf(cluster_sum_f(ss, sh, slot + 2, cs) / (float)D + u.eps);
        TA *h = reinterpret_cast<TA *>(u.h) + (size_t)r * u.h_pitch, *hc = reinterpret_cast<TA *>(u.hc) + (size_t)r * u.h_pitch;
        const int32_t pos = u.conv_w ? rows.pos_of(r) : 0, T = (int32_t)u.taps - 1;
        TA *ring = u.conv_w ? reinterpret_cast<TA *>(u.ring) + (size_t)rows.slot_of(r) * u.taps * D : nullptr;
        for (uint32_t c = c_lo + threadIdx.x * V; c < c_hi; c += RU_THREADS * V) {
            Vals<V> v = ldv<V>(xs + c - c_lo), w = ldv<V>(u.norm + c);
#pragma unroll
            for (int i = 0; i < V; i++) v.v[i] = as_act(v.v[i] * inv * w.v[i], h);
            stv<V>(h + c, v);
            if (u.conv_w) {
                Vals<V> s = ldv<V>(u.conv_w + (size_t)T * D + c);
#pragma unroll
                for (int i = 0; i < V; i++) s.v[i] = fmaf(s.v[i], v.v[i], v.v[i]);
                for (int32_t j = max(0, T - pos); j < T; j++) {
                    const Vals<V> o = ldv<V>(ring + (size_t)((uint32_t)(pos - T + j) % u.taps) * D + c), wj = ldv<V>(u.conv_w + (size_t)j * D + c);
#pragma unroll
                    for (int i = 0; i < V; i++) s.v[i] = fmaf(wj.v[i], o.v[i], s.v[i]);
                }
                stv<V>(ring + (size_t)((uint32_t)pos % u.taps) * D + c, v);
                stv<V>(hc + c, s);
            }
        }
    }
    if (cs > 1) cg::this_cluster().sync();  // the peers read this CTA's sums
}

// The same for rows whose run of columns is at most one vector per thread (narrow, or few rows with a cluster each):
// everything is requested before the first sum, weights before the dependency wait.
template <typename TA, int V>
__global__ void __launch_bounds__(RU_THREADS) row_update_few_kernel(const RowUpdate u, const RowMap rows, uint32_t cs, uint32_t per) {
    __shared__ float sh[32], slot[3];
    pdl_launch_dependents();
    const uint32_t r = blockIdx.y, D = u.width, c_lo = blockIdx.x * per, c = c_lo + threadIdx.x * V;
    const bool on = c < min(c_lo + per, D);
    constexpr int RU_TAPS = 4;  // weights of the convolution requested early
    Vals<V> w1{}, w2{}, nw{}, cw[RU_TAPS] = {};
    if (on) {
        if (u.add == ROW_ADD_PAIR) {
            w1 = ldv<V>(u.w + c);
            w2 = ldv<V>(u.w2 + c);
        }
        if (u.norm) nw = ldv<V>(u.norm + c);
#pragma unroll
        for (int j = 0; j < RU_TAPS; j++)
            if (u.conv_w && j < (int)u.taps) cw[j] = ldv<V>(u.conv_w + (size_t)j * D + c);
    }
    pdl_wait();
    const int32_t pos = u.conv_w ? rows.pos_of(r) : 0, T = (int32_t)u.taps - 1;
    TA *ring = u.conv_w ? reinterpret_cast<TA *>(u.ring) + (size_t)rows.slot_of(r) * u.taps * D + c : nullptr;
    Vals<V> v{}, d{}, d2{}, g, old{}, past[RU_TAPS - 1] = {};
#pragma unroll
    for (int i = 0; i < V; i++) g.v[i] = 1.0f;
    float own = 1.0f;
    if (on) {
        v = ldv<V>(u.x + (size_t)r * D + c);
        if (u.add == ROW_ADD_ONE || u.add == ROW_ADD_PAIR) d = ldv<V>(reinterpret_cast<const TA *>(u.y) + (size_t)r * u.y_pitch + c);
        if (u.add == ROW_ADD_PAIR) d2 = ldv<V>(reinterpret_cast<const TA *>(u.y2) + (size_t)r * u.y2_pitch + c);
        if (u.gate) g = ldv<V>(reinterpret_cast<const TA *>(u.gate) + (size_t)r * u.gate_pitch + c);
#pragma unroll
        for (int j = 0; j < RU_TAPS - 1; j++)
            if (u.conv_w && j < T && pos - T + j >= 0) past[j] = ldv<V>(ring + (size_t)((uint32_t)(pos - T + j) % u.taps) * D);
        if (u.history) {
            own = u.avg[u.n_history];
            const float *h = u.history + (size_t)r * D + c;
#pragma unroll 8
            for (uint32_t j = 0; j < u.n_history; j++) {
                const Vals<V> o = ldv<V>(h + j * u.history_stride);
                const float aj = u.avg[j];
#pragma unroll
                for (int i = 0; i < V; i++) old.v[i] = fmaf(aj, o.v[i], old.v[i]);
            }
        }
        if (u.add == ROW_ADD_EXPERTS) {
#pragma unroll 8
            for (uint32_t k = 0; k < u.top; k++) {
                const uint32_t pair = r * u.top + k, row = u.inv ? u.inv[pair] : pair;
                const Vals<V> e = ldv<V>(reinterpret_cast<const TA *>(u.y) + (size_t)row * u.y_pitch + c);
                const float w = u.wgt[pair];
#pragma unroll
                for (int i = 0; i < V; i++) d.v[i] = fmaf(w, e.v[i], d.v[i]);
            }
        }
    }
    if (u.add == ROW_ADD_PAIR) {
        float s1 = 0.0f, s2 = 0.0f;
#pragma unroll
        for (int i = 0; i < V; i++) {
            s1 = fmaf(d.v[i], d.v[i], s1);
            s2 = fmaf(d2.v[i], d2.v[i], s2);
        }
        const float2 q = cluster_sum2_f(s1, s2, sh, slot, cs);
        const float inv1 = 0.5f / sqrtf(q.x / (float)D + u.eps), inv2 = 0.5f / sqrtf(q.y / (float)D + u.eps);
#pragma unroll
        for (int i = 0; i < V; i++) d.v[i] = d.v[i] * inv1 * w1.v[i] + d2.v[i] * inv2 * w2.v[i];
    }
    float ss = 0.0f;
    if (on) {
#pragma unroll
        for (int i = 0; i < V; i++) v.v[i] = fmaf(u.mul, d.v[i] * g.v[i], v.v[i]);
        if (u.history) {
            stv<V>(u.history + u.n_history * u.history_stride + (size_t)r * D + c, v);
#pragma unroll
            for (int i = 0; i < V; i++) v.v[i] = fmaf(own, v.v[i], old.v[i]);
        }
        if (u.x_out) stv<V>(u.x_out + (size_t)r * D + c, v);
#pragma unroll
        for (int i = 0; i < V; i++) ss = fmaf(v.v[i], v.v[i], ss);
    }
    if (u.norm) {
        const float inv = 1.0f / sqrtf(cluster_sum_f(ss, sh, slot + 2, cs) / (float)D + u.eps);
        if (on) {
            TA *h = reinterpret_cast<TA *>(u.h) + (size_t)r * u.h_pitch + c;
#pragma unroll
            for (int i = 0; i < V; i++) v.v[i] = as_act(v.v[i] * inv * nw.v[i], h);
            stv<V>(h, v);
            if (u.conv_w) {
                Vals<V> s = v;
                for (int32_t j = max(0, T - pos); j <= T; j++) {
                    Vals<V> o = v, wj;
                    if (T < RU_TAPS) {
#pragma unroll
                        for (int e = 0; e < RU_TAPS; e++)
                            if (e == j) {
                                wj = cw[e];
                                if (e < RU_TAPS - 1 && e < T) o = past[e];
                            }
                    } else {
                        wj = ldv<V>(u.conv_w + (size_t)j * D + c);
                        if (j < T) o = ldv<V>(ring + (size_t)((uint32_t)(pos - T + j) % u.taps) * D);
                    }
#pragma unroll
                    for (int i = 0; i < V; i++) s.v[i] = fmaf(wj.v[i], o.v[i], s.v[i]);
                }
                stv<V>(ring + (size_t)((uint32_t)pos % u.taps) * D, v);
                stv<V>(reinterpret_cast<TA *>(u.hc) + (size_t)r * u.h_pitch + c, s);
            }
        }
    }
    if (cs > 1) cg::this_cluster().sync();  // the peers read this CTA's sums
}

template <typename TA>
static int run_row_update(prism_cuda_ctx *ctx, const RowUpdate &u, const RowMap &rows, uint32_t n) {
    uintptr_t at = 0;
    for (const void *p : {(const void *)u.x, (const void *)u.x_out, u.y, u.y2, (const void *)u.w, (const void *)u.w2, u.gate, (const void *)u.history,
                          (const void *)u.norm, (const void *)u.h, (const void *)u.conv_w, (const void *)u.ring, (const void *)u.hc})
        at |= reinterpret_cast<uintptr_t>(p);
    const uint32_t odd = u.width | (u.add ? u.y_pitch : 0) | (u.add == ROW_ADD_PAIR ? u.y2_pitch : 0) | (u.gate ? u.gate_pitch : 0) | (u.norm ? u.h_pitch : 0);
    const bool vec = !(at & 15) && !(odd & 3);
    uint32_t cs = 1;  // a cluster shares a row when the rows alone leave most of the GPU idle
    while (cs < 8 && n * cs * 2 <= (uint32_t)ctx->sm_count && u.width >= cs * 512) cs *= 2;
    uint32_t per = (u.width + cs - 1) / cs;
    per = round_up_u32(per, 4);
    if ((size_t)per * 4 > 48 * 1024) {
        if ((size_t)per * 4 > 200 * 1024) return fail(ctx, PRISM_E_ARG, "row update: the model is too wide");
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(row_update_kernel<TA, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        PRISM_CUDA_TRY(ctx, cudaFuncSetAttribute(row_update_kernel<TA, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    if (n > 65535) return fail(ctx, PRISM_E_ARG, "row update: too many rows");
    if (per <= RU_THREADS * (vec ? 4u : 1u)) {
        if (vec) launch_cluster_pdl(ctx, row_update_few_kernel<TA, 4>, dim3(cs, n), RU_THREADS, 0, cs, u, rows, cs, per);
        else launch_cluster_pdl(ctx, row_update_few_kernel<TA, 1>, dim3(cs, n), RU_THREADS, 0, cs, u, rows, cs, per);
        return after_launch(ctx, "row_update_few_kernel");
    }
    if (vec) launch_cluster_pdl(ctx, row_update_kernel<TA, 4>, dim3(cs, n), RU_THREADS, (size_t)per * 4, cs, u, rows, cs, per);
    else launch_cluster_pdl(ctx, row_update_kernel<TA, 1>, dim3(cs, n), RU_THREADS, (size_t)per * 4, cs, u, rows, cs, per);
    return after_launch(ctx, "row_update_kernel");
}
int launch_row_update(prism_cuda_ctx *ctx, const RowUpdate &u, const RowMap &rows, uint32_t n_rows, bool act32) {
    return act32 ? run_row_update<float>(ctx, u, rows, n_rows) : run_row_update<bf16>(ctx, u, rows, n_rows);
}

}  // namespace prism
