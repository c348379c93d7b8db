// The engine object behind the C ABI: what a decode loop needs whatever the model family -- batch,
// positions, tokens in and out, the captured step -- plus the weights and caches of the palettized
// Llama/Qwen2 step, or a LayeredModel in their place.
#pragma once

#include "common.cuh"

namespace prism {
struct LayeredModel;
}

struct prism_cuda_engine {
    prism_cuda_ctx *ctx = nullptr;
    prism_model_config cfg{};
    int T = 1, rank = 0;
    // local (per-rank) dimensions
    uint32_t H = 0, nh_l = 0, nkv_l = 0, hd = 0, qd_l = 0, kvd_l = 0, I_l = 0, V_l = 0;
    uint32_t head0 = 0, kvhead0 = 0, i0 = 0, v0 = 0;  // first local q head / kv head / inter row / vocab row
    std::vector<int32_t> wq, wk, wv, wo, wg, wu, wd;
    std::vector<int32_t> wqkv;   // q, k, v rows stacked into one tensor (one launch instead of three)
    bool fused_ready = false;
    uint16_t *gu = nullptr;      // [2][B][max(I_l, H)] scratch of the batched (GEMM) path
    uint16_t *qkv = nullptr;     // [B][qkv_stride]: q | k | v of a sequence side by side
    uint32_t qkv_stride = 0;
    int32_t embed = -1, lm_head = -1;
    // activations
    uint16_t *h = nullptr, *xn = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *att = nullptr,
             *act = nullptr, *logits = nullptr;
    float *part = nullptr;       // [B][H] fp32 partial sums of row-parallel matmuls (TP)
    uint32_t *tok = nullptr, *next = nullptr, *out_tokens = nullptr, *prompts = nullptr;
    uint64_t *pairs_send = nullptr, *pairs_recv = nullptr;  // TP argmax: (value bits << 32 | ~index)
    int32_t *scalars = nullptr;  // [0] pos, [1] step, [2] record
    size_t prompts_cap = 0;
    uint32_t act_stride = 0, out_cap = 0;
    void *kc = nullptr, *vc = nullptr;
    size_t kv_layer_bytes = 0;
    uint64_t kv_seq_stride = 0;  // fp16: elements, int8: bytes
    uint32_t kv_slots = 0;       // positions a layer slot can hold
    uint32_t batch = 0, pos = 0;
    bool guard_skip = false;     // down_guard && inter != hidden
    // paged KV cache (cfg.kv_page_size > 0): page table on the device and its host mirror, free pages
    int32_t *page_tbl = nullptr;             // [max_batch][pages_per_seq]
    std::vector<int32_t> page_tbl_host, free_pages;
    std::vector<uint32_t> seq_pages;         // pages each sequence holds
    uint32_t page_shift = 0, pages_per_seq = 0, pool_pages = 0;
    // batched prefill scratch (one chunk of prompt tokens of one sequence), grown on demand
    uint16_t *pf_x = nullptr, *pf_xn = nullptr, *pf_qkv = nullptr, *pf_att = nullptr, *pf_g = nullptr, *pf_u = nullptr,
             *pf_act = nullptr;
    uint32_t *pf_tok = nullptr;
    uint32_t pf_cap = 0;         // tokens the buffers hold
    cudaGraphExec_t graph = nullptr;
    uint32_t graph_batch = 0;
    uint64_t graph_epoch = ~0ull;  // option epoch of the context when the graph (or its eager warm-up) was made
    cudaEvent_t ev0 = nullptr, ev1 = nullptr, ev2 = nullptr, ev3 = nullptr;
    double last_ms = 0.0, last_device_ms = 0.0;
    uint32_t kernels_per_step = 0;
    prism::LayeredModel *lm = nullptr;  // set: a model described layer by layer (layered.cu); the palettized fields above are unused
};

namespace prism {

// layered.cu: what the engine's shared loop needs from a model described layer by layer
int layered_check_bound(prism_cuda_engine *e);             // every tensor has been set
int layered_enqueue_step(prism_cuda_engine *e);            // one token of every row of the batch (capturable)
int layered_set_rows(prism_cuda_engine *e, uint32_t pos);  // rows 0..batch-1 = slots 0..batch-1, all at `pos`
int layered_reset(prism_cuda_engine *e, uint32_t batch);   // slots 0..batch-1 open and empty, the others free
int layered_prefill(prism_cuda_engine *e, uint32_t slot, const uint32_t *tokens, uint32_t n);  // host tokens, appended to the slot
void layered_advance(prism_cuda_engine *e, uint32_t n);    // host mirror: rows 0..batch-1 took n tokens
int layered_logits_f16(prism_cuda_engine *e, uint16_t *host);
uint64_t layered_step_bytes(const prism_cuda_engine *e);
int layered_synth(prism_cuda_engine *e, uint64_t seed, float sigma);
void layered_destroy(prism_cuda_engine *e);
// engine.cu: runs, captures or replays the step of e->batch rows
int run_step(prism_cuda_engine *e);
int set_scalars(prism_cuda_engine *e, int32_t pos, int32_t step, int32_t record);
int enqueue_advance(prism_cuda_engine *e, int32_t *row_pos);
int engine_alloc_common(prism_cuda_engine *e, uint32_t max_batch);
void engine_drop_graph(prism_cuda_engine *e);

}  // namespace prism
