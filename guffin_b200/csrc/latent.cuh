// Attention over cached latents: every head of a token attends the same cache rows, which serve as keys (against
// queries already carried into the latent space) and as values (carried out of it behind the attention).
#pragma once

#include "dense.cuh"

namespace gf {

constexpr uint32_t kLatentMaxParts = 128;

// Elements of a cache row: the rank rounded up so that a row is whole 32-byte pieces.
__host__ __device__ inline uint32_t latent_row_elements(uint32_t rank) { return (rank + 15u) / 16u * 16u; }

struct LatentAttention {
    const void* q = nullptr;             // [rows * heads][row_elements], scaled; f16, or f32 with cache_f32
    const StreamRings* rings = nullptr;  // the cache rows before the pass: rings[row * ring_stride].ring_k
    uint32_t ring_stride = 0;            // 0: the rows are a chain of one sequence; 1: every row has a sequence of its own
    const void* private_rows = nullptr;  // [rows][row_elements]: the pass's own cache rows
    const uint32_t* positions = nullptr; // chain: position of row 0; else the position of every row
    uint32_t rows = 0, heads = 0, row_elements = 0, ring_mask = 0;
    uint32_t cache_f32 = 0;
    // Partial results: [rows * heads][parts][row_elements] unnormalised outputs and (maximum, sum) pairs.
    float *partial_out = nullptr, *partial_ml = nullptr;
    uint32_t parts = 1;
    // With `result` set (parts must be 1) the normalised output of (row, head) goes to columns head * result_stride
    // of the operand instead.
    const float* sink = nullptr;         // per head, or null
    Operand result;
    uint32_t result_stride = 0;
    uint32_t block_keys = 0;             // filled by the launcher
};
// Whether the tensor-core kernel takes this shape (binary16 cache, rank up to 512); else a plain f32 kernel runs.
bool latent_attention_on_tensor_cores(const LatentAttention& p);
// Partitions of the keys worth launching for a pass of `rows` rows over up to `positions` cached rows.
uint32_t latent_attention_parts(uint32_t rows, uint32_t heads, uint32_t positions, bool chain);
int launch_latent_attention(LatentAttention p, cudaStream_t stream, bool pdl);
// Merges partial results (and the sink) into the operand `result`.
int launch_latent_merge(const LatentAttention& p, cudaStream_t stream);

// ---- attention of a chunk over keys and values per head.  For latents: the same attention with the latents expanded,
// fewer operations once a chunk has many rows for the keys it sees, since a score then costs a head's `dim` instead of
// the latent's rank.  For grouped-query attention: over the cache rows themselves.
constexpr uint32_t kHeadAttentionMaxDim = 256;
struct HeadAttention {
    const __half* q = nullptr;           // [rows][heads][dim_pad], scaled
    const __half* k = nullptr;           // [positions][kv_heads][dim_pad], positions from 0; with rings: the chunk's own rows
    const __half* v = nullptr;           // [positions][kv_heads][vdim_pad]
    const StreamRings* rings = nullptr;  // the rows before the chunk, or null
    uint32_t ring_mask = 0;
    const uint32_t* position = nullptr;  // of row 0
    const float* sink = nullptr;         // per head, or null
    const float* gate = nullptr;         // [rows][heads], ahead of the sigmoid, or null
    float softcap = 0.0f;                // of the scores; 0: none
    uint32_t rows = 0, heads = 0, kv_heads = 0, dim_pad = 0, vdim = 0, vdim_pad = 0;      // pads: multiples of 16
    Operand result;                      // (row, head * vdim + d), bf16 or f32
};
int launch_head_attention(const HeadAttention& p, cudaStream_t stream);
// The first `positions` cache rows of a sequence as a bf16 operand.
int launch_latent_operand(const StreamRings* rings, const void* own, const uint32_t* position, uint32_t positions, uint32_t row_elements, uint32_t ring_mask,
                          const Operand& result, cudaStream_t stream);
// Rows of a chunk from which expanding pays: expansion costs every key rank x (dim + vdim) per head, and saves every
// (row, key) pair 2 x rank - (dim + vdim).
inline bool latent_expansion_pays(uint32_t rows, uint32_t rank, uint32_t dim, uint32_t vdim) {
    return 2u * rank > dim + vdim && (uint64_t)rows * (2u * rank - dim - vdim) > (uint64_t)rank * (dim + vdim);
}

}  // namespace gf
