// Model registry: config.json -> a description the resident plan is built from.
//
// Two kinds of description exist.  The quantised Gemma families are a gf_model_config (their block schedule is
// Model::encode_blocks).  A layered decoder is a list of layers, each naming its token mixer and its feed-forward
// with their sizes and constants; its schedule is Model::encode_layers.  An architecture is an entry of the table
// in architecture.cpp: a name and a function that turns its config.json into one of the two.
#pragma once

#include "common.cuh"

#include <string>
#include <vector>

namespace gf {

struct Json;

// ---- mixers
enum class MixerKind {
    kLatentAttention,      // every head attends the same cached latents
    kGroupedAttention,     // keys and values per key/value head, rotated and normalised
    kStateSpace,           // a recurrent state per head behind a short convolution (state-space duality)
};
struct MixerSpec {
    MixerKind kind = MixerKind::kLatentAttention;
    uint32_t heads = 0, dim = 0, vdim = 0;     // query/key and value size of a head
    float scale = 1.0f;                        // of the scores
    bool sink = true;                          // a learned logit per head in the softmax's denominator
    // kLatentAttention
    uint32_t rank = 0;                         // size of the cached latent
    // kGroupedAttention: the values are the projected keys, ahead of norm and rotation; queries and keys are normalised
    // over the whole projection
    uint32_t kv_heads = 0;
    uint32_t rotated = 0;                      // leading dimensions of a head that turn with the position, in pairs (i, i + rotated / 2)
    double rotation_base = 0.0;
    float softcap = 0.0f;                      // of the scores; 0: none
    bool head_gate = false;                    // a sigmoid per head on its output
    // kStateSpace: heads of vdim channels, a state of [state][vdim] each
    uint32_t state = 0, groups = 0;            // heads of a group share the input and output vectors
    uint32_t taps = 0;                         // of the convolution
    uint32_t norm_parts = 0;                   // parts of the gated output that are normalised by themselves

    uint32_t inner() const { return heads * vdim; }
    uint32_t channels() const { return inner() + 2u * groups * state; }      // of the convolution
    uint32_t state_inputs() const { return inner() + channels() + heads; }   // of the input projection
};

// ---- feed-forward layers
enum class Activation { kSquaredRelu, kClampedGate, kGeluGate };
struct FeedForwardSpec {
    enum Kind { kNone, kDense, kExperts } kind = kNone;
    Activation activation = Activation::kSquaredRelu;      // of the dense layer, or of every expert
    uint32_t ff = 0;                                       // of the dense layer, or of an expert
    float limit = 0.0f;                                    // kClampedGate: the clamp of gate and up
    uint32_t experts = 0, top = 0;
    bool shared = false;
    uint32_t shared_ff = 0;
    float shared_limit = 0.0f;
};

struct LayerSpec {
    MixerSpec mixer;
    FeedForwardSpec mlp;
    uint32_t source = 0;                       // the layer whose tensors it uses: itself, or an earlier or later one
};

struct LayeredSpec {
    uint32_t width = 0, vocab = 0;
    float embedding_scale = 1.0f, eps = 1e-6f;
    float norm_offset = 0.0f;                  // gain = offset + stored weight
    bool pre_norm = true;                      // norms ahead of the sublayers besides the ones behind them
    bool tied_head = true;                     // the token table is the output head
    std::vector<LayerSpec> layers;
};

// Where a tensor of a layered model goes.
enum class TensorRole {
    kEmbedding, kHead, kFinalNorm, kNorm1, kNorm1b, kNorm2, kNorm2b, kScale1, kScale2,      // norms 1, 2 ahead of the sublayers, 1b, 2b behind
    kQuery, kLatentDown, kLatentNorm, kLatentUpKey, kLatentUpValue, kSink, kMixerOut,
    kKey, kQueryNorm, kKeyNorm, kHeadGate,
    kStateIn, kTaps, kTapBias, kStepBias, kDecayLog, kSkip, kMixerNorm,
    kGate, kUp, kDown, kExpertGate, kExpertUp, kExpertDown, kRouter,
    kSharedGate, kSharedUp, kSharedDown, kSharedWeight,
};
struct TensorSlot {
    std::string name;
    TensorRole role;
    uint32_t layer, index;                     // index: the expert
    uint32_t rows, columns;                    // [rows, columns] as stored, [out, in]; vectors have rows = 0
    bool table = false;                        // a table of f32 constants rather than a matrix of a product
    size_t values() const { return (size_t)(rows ? rows : 1u) * columns; }
};

struct ArchitectureDescription {
    std::string name;
    bool layered = false;
    LayeredSpec spec;                          // layered
    std::vector<TensorSlot> tensors;
    gf_model_config config {};                 // quantised families
};

int describe_architecture(const char* text, size_t size, ArchitectureDescription& out);
const char* architecture_names();              // one name per line

}  // namespace gf
