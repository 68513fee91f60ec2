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
enum class MixerKind { kLatentAttention };
struct MixerSpec {
    MixerKind kind = MixerKind::kLatentAttention;
    uint32_t heads = 0, dim = 0, vdim = 0;     // query/key and value size of a head
    uint32_t rank = 0;                         // size of the cached latent
    float scale = 1.0f;                        // of the scores
    bool sink = true;                          // a learned logit per head in the softmax's denominator
};

// ---- feed-forward layers
enum class Activation { kSquaredRelu, kClampedGate };
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
};

struct LayeredSpec {
    uint32_t width = 0, vocab = 0;
    float embedding_scale = 1.0f, eps = 1e-6f;
    float norm_offset = 0.0f;                  // gain = offset + stored weight
    std::vector<LayerSpec> layers;
};

// Where a tensor of a layered model goes.
enum class TensorRole {
    kEmbedding, kFinalNorm, kNorm1, kNorm1b, kNorm2, kNorm2b, kScale1, kScale2,
    kQuery, kLatentDown, kLatentNorm, kLatentUpKey, kLatentUpValue, kSink, kMixerOut,
    kUp, kDown, kExpertGate, kExpertUp, kExpertDown, kRouter,
    kSharedGate, kSharedUp, kSharedDown, kSharedWeight,
};
struct TensorSlot {
    std::string name;
    TensorRole role;
    uint32_t layer, index;                     // index: the expert
    uint32_t rows, columns;                    // [rows, columns] as stored, [out, in]; vectors have rows = 0
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
