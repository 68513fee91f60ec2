// What a resident plan of a layered model holds besides the parts every plan has (model.cuh): bf16 matrices, folded
// norm gains, the scratch of its passes and of its prompt chunks.  The schedules are methods of Model (layered.cu).
#pragma once

#include "architecture.hpp"
#include "dense.cuh"
#include "latent.cuh"

#include <map>
#include <string>
#include <vector>

namespace gf {

struct LayeredLayer {
    // Gains as the kernels use them: offset + stored weight, times the layer scale behind a sublayer.
    float *gain1 = nullptr, *gain1b = nullptr, *gain2 = nullptr, *gain2b = nullptr;
    float *latent_gain = nullptr, *sink = nullptr;
    DenseMatrix q, latent_down, o;
    DenseMatrix up_key, up_value;             // per head: [rank x dim] and [vdim x rank]
    DenseMatrix expand_key;                   // [heads * dim x rank]: the same weights as up_key for chunks that expand their keys
    DenseMatrix up, down;                     // dense feed-forward
    DenseMatrix expert_up, expert_down;       // per expert, gate and up paired
    DenseMatrix router, shared_up, shared_down, shared_weight;
};

// Where the rows of a pass live: one sequence (the plan's own, a chain of rows) or one sequence per row.
struct LayeredRows {
    const StreamRings* rings;                 // [layer * layer_stride + row * ring_stride]
    uint32_t layer_stride, ring_stride;
    const uint32_t* positions;
    float* logits;
};

struct LayeredPlan {
    ArchitectureDescription description;
    bool f32 = false;
    std::vector<LayeredLayer> layers;
    DenseMatrix table;                        // token table and output head
    float* final_gain = nullptr;
    std::map<std::string, const TensorSlot*> slots;
    std::map<std::string, bool> bound;
    std::map<std::string, std::vector<float>> vectors;      // until the gains are formed

    // ---- passes of a few rows
    float *residual[2] = {nullptr, nullptr}, *normed = nullptr, *raw_q = nullptr, *raw_latent = nullptr, *heads_out = nullptr, *projected = nullptr;
    float *hidden = nullptr, *expert_hidden = nullptr, *shared_hidden = nullptr, *parts = nullptr, *router_logits = nullptr, *shared_logit = nullptr;
    uint32_t* route_ids = nullptr;
    float* route_scores = nullptr;
    void* latent_q = nullptr;
    float *partial_out = nullptr, *partial_ml = nullptr;
    StreamRings* rings_dev = nullptr;         // [layer]: the rings the plan's own passes use

    // ---- prompt chunks
    struct Chunk {
        bool ready = false;
        uint32_t rows = 0;                    // at most, per chunk
        uint32_t grouped = 0;                 // rows of the grouped operands
        uint32_t partial_rows = 0;            // (row, head, partition) triples the partial buffers hold
        Operand normed, query, latent_out, heads_out, hidden, shared_hidden, group, group_hidden;
        float *residual = nullptr, *raw_latent = nullptr, *y = nullptr, *shared_y = nullptr, *group_y = nullptr, *router_logits = nullptr, *shared_logit = nullptr;
        float *final_rows = nullptr, *partial_out = nullptr, *partial_ml = nullptr, *slot_scores = nullptr, *row_scale = nullptr;
        void* latent_q = nullptr;
        // Keys and values of a chunk that expands its latents (16-bit plans): up to expand_keys positions.
        uint32_t expand_keys = 0;
        void *latent_rows = nullptr;          // a bf16 operand of that many rows
        __half *keys = nullptr, *values = nullptr, *head_q = nullptr;
        uint32_t *group_start = nullptr, *group_rows = nullptr, *slot_rows = nullptr, *slot_experts = nullptr, *tokens = nullptr, *wanted = nullptr;
        std::vector<void*> private_rows;
        KvPublishLayer* publish_layers = nullptr;
    } chunk;
    uint32_t chunk_limit = 1024;              // rows of a chunk, at most

    const LayeredSpec& spec() const { return description.spec; }
    size_t cache_row_bytes(uint32_t layer) const { return (size_t)latent_row_elements(spec().layers[layer].mixer.rank) * (f32 ? 4u : 2u); }
};

}  // namespace gf
