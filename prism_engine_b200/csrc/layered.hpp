// A model described layer by layer: weights, state and scratch behind prism_cuda_engine::lm.
#pragma once

#include <string>
#include <unordered_map>
#include <vector>

#include "dense.cuh"
#include "engine.hpp"

namespace prism {

// One mixer of a layer.
struct LayeredMixer {
    prism_layer_config c{};
    std::string name;         // prefix of its tensors
    uint32_t seg0 = 0;        // its first segment of the layer's `in`
    uint32_t col = 0;         // its first column in the rows of `cat`
    DenseLinear uq;           // latent: queries from the query latent
    DenseLinear ukv;          // latent: keys | values from latents (prompt portions)
    float *mix_norm = nullptr, *dq_norm = nullptr, *decay = nullptr;
    float *state = nullptr;   // lightning: [slot][heads][dim][vdim]
    LatentArgs la{};          // latent: sizes, cache, row-major W_uk / W_uv
    uint32_t splits = 0;
    GroupedArgs ga{};         // attention: sizes, cache
    DeltaArgs da{};           // gated delta: sizes, small weights, state, ring
    uint32_t conv_col[3] = {0, 0, 0};  // gated delta: columns of q, k, v in the convolved rows
    float *out_norm = nullptr;         // pair: norm of its result
    uint32_t width() const { return c.heads * c.vdim; }
};

struct LayeredLayer {
    prism_layer_config c{};
    std::vector<LayeredMixer> mix;  // two in a pair
    DenseLinear in;      // everything that reads the first norm (sequential: convolved or not)
    DenseLinear out;     // parallel: [W_o | W_down] along k, added into the residual; sequential: the mixers' W_o, each from its own columns
    uint32_t seg_up = 0; // index of the feed-forward segment of `in` (sequential: of `in2`)
    uint32_t k_mix = 0;  // columns of the out input before the feed-forward part (mixer width rounded up to 64)
    float *norm1 = nullptr, *up_b = nullptr, *down_b = nullptr;
    // sequential
    DenseLinear in2;     // what reads the second norm: router or feed-forward up, gate
    DenseLinear up, down;  // experts; dense: down alone
    uint32_t seg_gate1 = 0, seg_gate2 = 0;
    float *norm2 = nullptr, *canon1 = nullptr, *canon2 = nullptr, *gate1_b = nullptr, *gate2_b = nullptr, *correction = nullptr, *avg = nullptr;
    void *ring1 = nullptr, *ring2 = nullptr;  // inputs of the two input convolutions, [slot][taps][width]
};

// Where a checkpoint tensor goes.
struct LayeredDst {
    uint64_t rows = 0, cols = 0;
    DenseLinear *lin = nullptr;                    // packed at (row0, k0)
    uint32_t row0 = 0, k0 = 0;
    bf16 *rowmajor = nullptr;                      // also (or only) kept row-major, rows `pitch` apart
    uint32_t pitch = 0;
    float *vec = nullptr;                          // fp32 copy of a vector, or of a matrix transposed
    uint32_t vec_pitch = 0;                        // between the rows of the transposed copy
    float add = 0.0f;                              // added to the copy
    float mean = 0.0f;                             // of synthetic values
    bool bound = false;
};

struct LayeredModel {
    prism_layered_config c{};
    std::vector<LayeredLayer> layers;
    bool act32 = false;
    uint32_t width_pad = 0, vocab_pad = 0;
    bf16 *embed = nullptr, *pos = nullptr;
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
    // sequential arrangement
    void *xc = nullptr, *y = nullptr, *moe_x = nullptr, *act = nullptr, *conv = nullptr, *delta = nullptr;  // convolved norm, results, experts' rows
    float *aux = nullptr, *history = nullptr, *o32 = nullptr;  // fp32 projections, residual stream after every layer, outputs before their norm
    uint32_t aux_pitch = 0, y_pitch = 0, act_pitch = 0, conv_pitch = 0, o32_width = 0;
    size_t pairs_cap = 0;                          // rows of the experts' buffers
    MoePlan plan{};                                // buffers; experts and top are the layer's
    cudaStream_t side = nullptr;                   // the second mixer of a pair, in prompt portions
    cudaEvent_t fork = nullptr, join = nullptr;
    // expanded keys and values of a prompt portion, grown on demand
    bf16 *ex_lat = nullptr, *ex_krot = nullptr, *ex_kv = nullptr;
    size_t ex_lat_n = 0, ex_krot_n = 0, ex_kv_n = 0;
    int32_t *row_slot = nullptr, *row_pos = nullptr;
    std::vector<int64_t> slot_pos;                 // tokens a slot holds; -1: free
    std::vector<void *> allocs;                    // everything above that lives as long as the model
    bool bound_ok = false;
};

}  // namespace prism
