// Grouped-query attention over cached keys and values of any head size: queries and keys normalised over their whole
// projection and rotated, scores capped, a sink in the softmax's denominator, a gate per head.
//
// A cache row is [kv heads][row_head] for keys and the same for values, binary16 or f32, zeros behind a head's values.
#pragma once

#include "dense.cuh"

namespace gf {

// Elements of a head in a cache row and in a prepared query: whole 32-byte pieces.
__host__ __device__ inline uint32_t grouped_row_head(uint32_t dim, uint32_t vdim) { return ((dim > vdim ? dim : vdim) + 15u) / 16u * 16u; }

// Projected rows to queries and cache rows: rmsnorm over the whole row, times the gain, then the first `rotated`
// dimensions of every head turned by an angle that grows with the position, in pairs (i, i + rotated / 2); queries times
// `scale`; values as projected.  A position's turn is the product of two tabulated ones.
constexpr uint32_t kTurnSpan = 1024;
struct QueryKey {
    const float *raw_q = nullptr, *raw_k = nullptr, *raw_v = nullptr;      // [rows][ld]; without raw_q the cache rows alone
    uint32_t q_ld = 0, k_ld = 0, v_ld = 0;
    const float *q_gain = nullptr, *k_gain = nullptr;
    const float2 *turns = nullptr, *spans = nullptr;       // cosine and sine of positions 0 .. kTurnSpan - 1, and of multiples of it: [..][rotated / 2]
    const uint32_t* positions = nullptr;           // chain: position of row 0; else the position of every row
    bool chain = true;
    void *q = nullptr, *keys = nullptr, *values = nullptr;                 // [rows][heads][row_head], [rows][kv heads][row_head]
    uint32_t rows = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0, row_head = 0, rotated = 0, f32 = 0;
    float eps = 0.0f, scale = 1.0f;
    uint32_t* status = nullptr;
    uint32_t pairs = 0;                            // filled by the launcher: every row and head starts on an even value
};
int launch_query_key(QueryKey p, cudaStream_t stream, bool pdl);

constexpr uint32_t kGroupedMaxParts = 64;
struct GroupedAttention {
    const void* q = nullptr;             // [rows][heads][row_head], scaled; f16, or f32 with f32
    const StreamRings* rings = nullptr;  // the cache rows before the pass: rings[row * ring_stride]
    uint32_t ring_stride = 0;            // 0: the rows are a chain of one sequence; 1: every row has a sequence of its own
    const void *own_k = nullptr, *own_v = nullptr;       // [rows]: the pass's own cache rows
    const uint32_t* positions = nullptr; // chain: position of row 0; else the position of every row
    uint32_t rows = 0, heads = 0, kv_heads = 0, row_head = 0, vdim = 0, ring_mask = 0, f32 = 0;
    float softcap = 0.0f;                // 0: none
    const float* sink = nullptr;         // per head, or null
    const float* gate = nullptr;         // [rows][heads], ahead of the sigmoid, or null
    // Keys in `parts` partitions: unnormalised outputs [rows * heads][parts][row_head] and (maximum, sum) pairs; the block
    // that arrives last merges a group's partitions.  `counters` [rows * heads] are zero between launches.
    float *partial_out = nullptr, *partial_ml = nullptr;
    uint32_t* counters = nullptr;
    uint32_t parts = 1;
    Operand result;                      // (row, head * vdim + d)
    // With `fused` the blocks prepare their queries and the pass's own cache rows from the projections themselves (q is
    // not read; own_k and own_v are written): passes of the tensor-core kernel alone.
    uint32_t fused = 0;
    QueryKey prepare;
};
// Whether the tensor-core kernel takes this shape (binary16, heads of up to 256); else a plain f32 kernel runs.
inline bool grouped_attention_on_tensor_cores(uint32_t row_head, bool f32) { return !f32 && row_head <= 256u; }
constexpr uint32_t kGroupedFusedRows = GF_MAX_ROWS;
// Partitions of the keys worth launching for a pass of `rows` rows over up to `positions` cached rows.
uint32_t grouped_attention_parts(uint32_t rows, uint32_t heads, uint32_t kv_heads, uint32_t positions, bool chain);
int launch_grouped_attention(const GroupedAttention& p, cudaStream_t stream, bool pdl);

#ifdef __CUDACC__
// cap * tanh(score / cap) = cap - 2 cap / (exp(2 score / cap) + 1), off by a few 1e-7 cap at most.
__device__ __forceinline__ float soft_cap(float score, float cap, float inverse_cap) {
    const float e = __expf(2.0f * fminf(score * inverse_cap, 20.0f));
    return cap - __fdividef(2.0f * cap, e + 1.0f);
}
__device__ __forceinline__ float soft_cap_exact(float score, float cap) { return cap * tanhf(score / cap); }
#endif

}  // namespace gf
