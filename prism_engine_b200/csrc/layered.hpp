// A model described layer by layer: weights, state and scratch behind prism_cuda_engine::lm.
#pragma once

#include <string>
#include <unordered_map>
#include <vector>

#include "dense.cuh"
#include "engine.hpp"

namespace prism {

struct LayeredLayer {
    prism_layer_config c{};
    DenseLinear in;      // everything that reads the layer's normed input: the mixer's projections, gate, feed-forward up
    DenseLinear out;     // [W_o | W_down] along k: both sublayers' outputs, added into the residual
    DenseLinear uq;      // latent: queries from the query latent
    DenseLinear ukv;     // latent: keys | values from latents (prompt portions)
    uint32_t seg_up = 0; // index of the feed-forward segment of `in`
    uint32_t k_mix = 0;  // columns of the out input before the feed-forward part (mixer width rounded up to 64)
    float *norm1 = nullptr, *mix_norm = nullptr, *dq_norm = nullptr, *up_b = nullptr, *down_b = nullptr, *decay = nullptr;
    float *state = nullptr;   // lightning: [slot][heads][dim][vdim]
    LatentArgs la{};          // latent: sizes, cache, row-major W_uk / W_uv
    uint32_t splits = 0;
};

// Where a checkpoint tensor goes.
struct LayeredDst {
    uint64_t rows = 0, cols = 0;
    DenseLinear *lin = nullptr;                    // packed at (row0, k0)
    uint32_t row0 = 0, k0 = 0;
    bf16 *rowmajor = nullptr;                      // also (or only) kept row-major, rows `pitch` apart
    uint32_t pitch = 0;
    float *vec = nullptr;                          // fp32 copy of a vector
    bool is_norm = false, bound = false;
};

struct LayeredModel {
    prism_layered_config c{};
    std::vector<LayeredLayer> layers;
    bool act32 = false;
    uint32_t width_pad = 0, vocab_pad = 0;
    bf16 *embed = nullptr;
    DenseLinear head;
    float *final_norm = nullptr;
    std::unordered_map<std::string, LayeredDst> names;
    std::vector<std::string> order;                // names in layer order
    // scratch for `cap` rows
    uint32_t cap = 0, chunk = 0, lg_cap = 0;
    float *x = nullptr, *xw = nullptr, *logits = nullptr;
    void *xn = nullptr, *proj = nullptr, *cat = nullptr, *q = nullptr, *cq = nullptr;
    uint32_t proj_pitch = 0, cat_pitch = 0, q_pitch = 0, cq_pitch = 0;
    uint32_t *want_idx = nullptr, *pf_tok = nullptr;
    LatentRowsScratch rows_scratch{};
    // expanded keys and values of a prompt portion, grown on demand
    bf16 *ex_lat = nullptr, *ex_krot = nullptr, *ex_kv = nullptr;
    size_t ex_lat_n = 0, ex_krot_n = 0, ex_kv_n = 0;
    int32_t *row_slot = nullptr, *row_pos = nullptr;
    std::vector<int64_t> slot_pos;                 // tokens a slot holds; -1: free
    std::vector<void *> allocs;                    // everything above that lives as long as the model
    bool bound_ok = false;
};

}  // namespace prism
