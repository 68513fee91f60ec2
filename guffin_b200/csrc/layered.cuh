// What a resident plan of a layered model holds besides the parts every plan has (model.cuh): bf16 matrices, folded
// norm gains, the scratch of its passes and of its prompt chunks.  The schedules are methods of Model (layered.cu).
#pragma once

#include "architecture.hpp"
#include "dense.cuh"
#include "grouped.cuh"
#include "latent.cuh"
#include "state_space.cuh"

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
    DenseMatrix k, head_gate;                 // grouped-query attention
    float *q_gain = nullptr, *k_gain = nullptr;
    DenseMatrix state_in;                     // state space
    float *taps = nullptr, *tap_bias = nullptr, *step_bias = nullptr, *decay = nullptr, *skip = nullptr, *mixer_gain = nullptr;
    DenseMatrix up, down;                     // dense feed-forward; up and its gate paired where it has one
    DenseMatrix expert_up, expert_down;       // per expert, gate and up paired
    DenseMatrix router, shared_up, shared_down, shared_weight;
};

// Where the rows of a pass live: one sequence (the plan's own, a chain of rows) or one sequence per row.
struct LayeredRows {
    const StreamRings* rings;                 // [layer * layer_stride + row * ring_stride]
    uint32_t layer_stride, ring_stride;
    const uint32_t* positions;
    float* logits;
    const uint32_t* slots;                    // states a sequence's recurrent layers hold
};

struct LayeredPlan {
    ArchitectureDescription description;
    bool f32 = false;
    std::vector<LayeredLayer> layers;
    DenseMatrix table, output_head;           // token table; the output head where it is a matrix of its own
    float* final_gain = nullptr;
    std::map<std::string, const TensorSlot*> slots;
    std::map<std::string, bool> bound;
    std::map<std::pair<TensorRole, uint32_t>, std::vector<float>> vectors;      // by role and layer, until finalized
    std::vector<std::pair<const float2*, const float2*>> turns;      // [layer]: the tables of its rotation

    // ---- passes of a few rows
    float *residual[2] = {nullptr, nullptr}, *normed = nullptr, *raw_q = nullptr, *raw_latent = nullptr, *heads_out = nullptr, *projected = nullptr;
    float *hidden = nullptr, *expert_hidden = nullptr, *shared_hidden = nullptr, *parts = nullptr, *router_logits = nullptr, *shared_logit = nullptr;
    uint32_t* route_ids = nullptr;
    float* route_scores = nullptr;
    void* latent_q = nullptr;
    float *partial_out = nullptr, *partial_ml = nullptr;
    StreamRings* rings_dev = nullptr;         // [layer]: the rings the plan's own passes use
    float *raw_k = nullptr, *raw_gate = nullptr;
    void* query = nullptr;                    // prepared queries
    uint32_t* counters = nullptr;             // arrivals of attention partitions, zero between launches
    uint32_t* slots_dev = nullptr;            // states per sequence of the rings in rings_dev

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
        std::vector<void*> private_rows, private_values;
        float *raw_q = nullptr, *raw_k = nullptr, *raw_gate = nullptr;
        void* prepared_q = nullptr;
        float *state_x = nullptr, *state_b = nullptr, *state_c = nullptr, *state_factors = nullptr, *state_y = nullptr;
        float2* state_steps = nullptr;
        KvPublishLayer* publish_layers = nullptr;
    } chunk;
    uint32_t chunk_limit = 1024;              // rows of a chunk, at most

    const LayeredSpec& spec() const { return description.spec; }
    const LayeredLayer& weights(uint32_t layer) const { return layers[spec().layers[layer].source]; }
    const DenseMatrix& head() const { return spec().tied_head ? table : output_head; }

    // ---- the caches.  A layer that attends holds a row per position in one tensor (latents) or two (keys, values); a
    // recurrent layer holds `slots` states and a ring of the convolution's inputs in their places.
    static constexpr uint32_t kStreamSlots = 2;        // a stream's passes are always published whole
    uint32_t own_slots = 0;                            // the plan's own: the states of a pass's rows and the one behind them
    bool recurrent(uint32_t layer) const { return spec().layers[layer].mixer.kind == MixerKind::kStateSpace; }
    bool any_recurrent() const {
        for (uint32_t l = 0; l < spec().layers.size(); ++l) if (recurrent(l)) return true;
        return false;
    }
    uint32_t cache_tensors(uint32_t layer) const {
        const MixerKind kind = spec().layers[layer].mixer.kind;
        return kind == MixerKind::kStateSpace ? 0u : kind == MixerKind::kGroupedAttention ? 2u : 1u;
    }
    size_t cache_row_bytes(uint32_t layer) const {
        const MixerSpec& m = spec().layers[layer].mixer;
        const size_t element = f32 ? 4u : 2u;
        if (m.kind == MixerKind::kStateSpace) return 0u;
        return (m.kind == MixerKind::kGroupedAttention ? (size_t)m.kv_heads * grouped_row_head(m.dim, m.vdim) : latent_row_elements(m.rank)) * element;
    }
    StateSpace state_space(uint32_t layer) const {     // the shapes of a recurrent layer
        const MixerSpec& m = spec().layers[layer].mixer;
        StateSpace p;
        p.heads = m.heads; p.vdim = m.vdim; p.state = m.state; p.groups = m.groups; p.tap_count = m.taps;
        return p;
    }
    size_t state_bytes(uint32_t layer) const { return recurrent(layer) ? state_space(layer).slot_elements() * 4u : 0u; }
    // Bytes of a sequence's first and second cache tensor.
    size_t ring_bytes(uint32_t layer, uint32_t which, uint32_t ring_rows, uint32_t slots) const {
        if (recurrent(layer)) return which ? (size_t)ring_rows * state_space(layer).input_row() * 4u : state_bytes(layer) * slots;
        return which < cache_tensors(layer) ? cache_row_bytes(layer) * ring_rows : 0u;
    }
};
inline uint32_t state_inputs_ld(const MixerSpec& m) { return (m.state_inputs() + 7u) & ~7u; }

}  // namespace gf
