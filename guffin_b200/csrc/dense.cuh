// bf16 matrices of layered models and the products with them.
//
// A matrix [n][k] is stored once, in the order the fifth-generation tensor core reads a K-major operand: tiles of
// 128 output columns x 64 K elements (16 KB), inside a tile groups of eight columns (1 KB), inside a group eight
// core matrices of 8 columns x 8 K elements (128 bytes).  Missing columns and K elements are zero.  A chunk's
// product copies whole tiles to shared memory; a row product reads a group's 512-byte halves, 16 bytes per lane:
// lane = (K piece of eight) * 8 + column.  A gate matrix and an up matrix whose products are combined are stored
// as one matrix with their groups alternating, so that the two halves of a pair are eight columns apart.
//
// Products over a few rows (decode) take f32 activations and accumulate in f32, whatever the plan's precision.
// Products over a chunk of prompt rows are bf16 tcgen05 products, or f32 ones in a plan built for 32-bit.
#pragma once

#include "ops.cuh"

namespace gf {

constexpr uint32_t kDenseTile = 128, kDenseBlockK = 64, kDenseTileBytes = kDenseTile * kDenseBlockK * 2u;

struct DenseMatrix {
    uint8_t* data = nullptr;
    uint32_t k = 0, n = 0;              // n counts stored columns: gate and up together for a paired matrix
    uint32_t k_blocks() const { return (k + kDenseBlockK - 1u) / kDenseBlockK; }
    uint32_t tiles() const { return (n + kDenseTile - 1u) / kDenseTile; }
    size_t bytes() const { return (size_t)tiles() * k_blocks() * kDenseTileBytes; }
};

// Byte offset of element (column n, k).
__host__ __device__ inline size_t dense_offset(uint32_t k_blocks, uint32_t n, uint32_t k) {
    return ((size_t)(n / kDenseTile) * k_blocks + k / kDenseBlockK) * kDenseTileBytes + (size_t)((n % kDenseTile) / 8u) * 1024u
           + ((k % kDenseBlockK) / 8u) * 128u + (n % 8u) * 16u + (k % 8u) * 2u;
}

// Columns of a pair of matrices of `ff` columns each, stored as one.
__host__ __device__ inline uint32_t dense_paired_columns(uint32_t ff) { return (ff + 7u) / 8u * 16u; }

// Packs `count` matrices of [n][k] elements: matrix i's element (n, k) is src[i * count_stride + n * n_stride + k * k_stride].
// Column n goes to group (n / 8) * group_step + group_first of the destination (step 2 for one half of a pair).
struct DensePack {
    const uint16_t* src;
    uint8_t* dst;
    size_t count_stride, n_stride, k_stride, dst_stride;      // dst_stride: bytes between packed matrices
    uint32_t count, n, k, k_blocks, group_step, group_first;
};
int launch_dense_pack(const DensePack& pack, cudaStream_t stream);

int launch_dense_embedding(const uint8_t* packed, uint32_t k_blocks, uint32_t width, uint32_t vocab, const uint32_t* tokens, uint32_t rows,
                           float scale, float* out, uint32_t* status, cudaStream_t stream, bool pdl);

// ---- a mixture's routing of one token: the `top` largest sigmoid scores, lower index first among equals.
constexpr uint32_t kMaxExperts = 1024;

// ---- row products ----

enum RowInput : uint32_t {
    kRowPlain = 0,        // in[row * in_ld + batch * in_batch + k]
    kRowNorm = 1,         // rmsnorm(in) * gain1
    kRowAddNorm = 2,      // residual + rmsnorm(sum of the parts of in) * gain0 -> residual_out; rmsnorm(that) * gain1 (that alone without gain1)
    kRowLatent = 3,       // batch = head: merge of the attention partitions of (row, head)
    kRowRouted = 4,       // batch = row * top + slot: row `batch / top` of in, plain; the product is multiplied by the slot's score
    kRowExperts = 5,      // batch < rows * top: in[batch * in_ld + k]; the batches behind them: row `batch - rows * top` of in2
    kRowPartNorm = 6,     // rmsnorm(in) * gain1, every one of norm_parts equal parts of the row by its own root mean square
};
enum RowOutput : uint32_t {
    kOutF32 = 0,          // out[row * ld + batch * out_batch + n]
    kOutSquaredRelu = 1,
    kOutClampedGate = 2,  // paired matrix: n halves
    kOutLatentQuery = 3,  // out[(row * heads + batch) * ld + n] = product * scale, f16 or f32
    kOutGeluGate = 4,     // paired matrix: gelu(gate) * up
};
__host__ __device__ inline bool paired_output(uint32_t output) { return output == kOutClampedGate || output == kOutGeluGate; }

struct RowMatrix {
    const uint8_t* weight = nullptr;
    size_t weight_batch = 0;            // bytes between the matrices of consecutive batches (or experts)
    void* out = nullptr;
    uint32_t k = 0, n = 0, k_blocks = 0;
    uint32_t out_ld = 0, out_batch = 0;
    uint32_t output = kOutF32;
    float limit = 0.0f;
    uint32_t groups_per_cta = 1, first_set = 0, sets = 0;      // filled by the launcher
};

struct RowProduct {
    RowMatrix m[3];
    uint32_t count = 1, batches = 1, rows = 1;
    uint32_t input = kRowPlain;
    const float* in = nullptr;
    uint32_t in_ld = 0, in_batch = 0;
    const uint32_t* in_rows = nullptr;  // kRowPlain: optional row indices
    // norms
    uint32_t width = 0, parts = 1, norm_parts = 1;
    size_t part_stride = 0;             // floats between parts
    const float *residual = nullptr, *gain0 = nullptr, *gain1 = nullptr;
    float *residual_out = nullptr, *normed_out = nullptr;
    float eps = 0.0f;
    // kRowLatent: partial outputs [row * heads + head][attention_parts][latent_ld] and (maximum, sum) pairs
    const float *latent_ml = nullptr, *sink = nullptr;
    uint32_t latent_ld = 0, attention_parts = 0, heads = 0;
    // kOutLatentQuery
    float scale = 1.0f;
    uint32_t query_f16 = 0;
    // kRowRouted / kRowExperts
    const float *router_logits = nullptr, *shared_logit = nullptr;
    uint32_t experts = 0, top = 0;
    uint32_t *route_ids = nullptr;      // [row * top + slot], written by kRowRouted and read by kRowExperts
    float *route_scores = nullptr;
    const float* in2 = nullptr;
    uint32_t in2_ld = 0;
    // a batch of its own behind the last: cache rows = rmsnorm(raw) * gain (launches of the absorbed query product)
    const float *latent_raw = nullptr, *latent_gain = nullptr;
    uint32_t latent_rank = 0, latent_raw_ld = 0;
    void* latent_rows = nullptr;
    uint32_t latent_row_elements = 0, latent_f16 = 0;
    uint32_t* status = nullptr;
    // filled by the launcher
    uint32_t k_pad = 0, vector_rows = 0;
};
// Any number of rows; launches as many kernels as the rows need (`launches` is increased by their number).
int launch_row_product(RowProduct product, cudaStream_t stream, bool pdl, uint32_t& launches);

// ---- chunk products ----

// The activations of a chunk as the next product reads them: bf16 in the tensor core's order with all rows of the
// chunk in one K block (a block is capacity x 128 bytes), or f32 rows.
struct Operand {
    void* data = nullptr;
    uint32_t capacity = 0;              // rows, a multiple of 8
    uint32_t k_pad = 0;                 // K rounded up to whole blocks
    uint32_t f32 = 0;
    __host__ __device__ size_t bytes() const { return (size_t)capacity * k_pad * (f32 ? 4u : 2u); }
};

enum ChunkOutput : uint32_t {
    kChunkF32 = 0,            // out[row * out_ld + n] = product * row scale
    kChunkOperand = 1,        // operand(row, column(n)) = product
    kChunkSquaredRelu = 2,    // operand(row, n) = max(product, 0)^2
    kChunkClampedGate = 3,    // paired matrix: operand(row, n) = clamped gate of (gate, up) * row scale
    kChunkLatentQuery = 4,    // out[(row * heads + index) * out_ld + n] = product * scale, f16 or f32
    kChunkHalfRows = 5,       // f16 out[row * out_ld + column(n)] = product * scale
    kChunkGeluGate = 6,       // paired matrix: operand(row, n) = gelu(gate) * up
};
__host__ __device__ inline bool paired_chunk(uint32_t output) { return output == kChunkClampedGate || output == kChunkGeluGate; }
constexpr uint32_t kMaxNormParts = 1024;           // of kRowPartNorm and launch_chunk_part_norm

// `count` products of the same shape: heads of one matrix, or experts.
struct ChunkProblem {
    const uint8_t* weight = nullptr;
    size_t weight_stride = 0;           // bytes between the matrices of consecutive indices
    uint32_t k = 0, n = 0, k_blocks = 0, count = 1;
    Operand a;
    uint32_t a_block0 = 0, a_block_stride = 0;     // K block of the operand at which index 0 starts, and the step per index
    uint32_t output = kChunkF32;
    float* out = nullptr;
    uint32_t out_ld = 0;
    Operand result;
    uint32_t segment = 0, segment_pad = 0;         // column(n) = (n / segment) * segment_pad + n % segment (0: n), plus
    uint32_t column_stride = 0;                    // index * column_stride
    float limit = 0.0f, scale = 1.0f;
    uint32_t heads = 0, query_f16 = 0;
    const float* row_scale = nullptr;              // per output row; sigmoid applied first if row_scale_sigmoid
    uint32_t row_scale_ld = 1, row_scale_sigmoid = 0;
    // Experts: rows [group_start[index], + group_rows[index]) of the operand and of the result; null: rows [0, rows).
    const uint32_t *group_start = nullptr, *group_rows = nullptr;
    uint32_t first_tile = 0, tiles = 0;            // filled by the launcher
};

struct ChunkProduct {
    ChunkProblem p[3];
    uint32_t problems = 1, rows = 0;
    uint32_t window = 0, stage_budget = 0;      // filled by the launcher
    int* error_flag = nullptr;
};
int launch_chunk_product(ChunkProduct product, bool f32, cudaStream_t stream);
// f32 rows [rows][k] into an operand.
int launch_chunk_operand(const float* x, uint32_t rows, uint32_t k, const Operand& result, cudaStream_t stream);

// Rows of a chunk between products: residual + rmsnorm(y) * gain0 -> residual (in place), rmsnorm(that) * gain1 ->
// operand and / or f32 rows.  y null: only the second norm.  gain1 null: the residual itself instead of its norm.  y is
// [row][width], or with `slots` set the sum over a token's slots of y[slot_rows[row * slots + slot]] and of shared[row].
struct ChunkNorm {
    float* residual = nullptr;
    const float *y = nullptr, *shared = nullptr, *gain0 = nullptr, *gain1 = nullptr;
    const uint32_t* slot_rows = nullptr;
    uint32_t slots = 0, width = 0, rows = 0;
    float eps = 0.0f;
    Operand result;
    float* normed = nullptr;
};
int launch_chunk_norm(const ChunkNorm& norm, cudaStream_t stream);
// rmsnorm(x * silu(gate)) * gain into an operand, every one of `parts` equal parts of a row by its own root mean square.
int launch_chunk_part_norm(const float* x, uint32_t x_ld, const float* gate, uint32_t gate_ld, uint32_t width, uint32_t parts, const float* gain, float eps, const Operand& result, uint32_t rows,
                           cudaStream_t stream);

// Routing of a chunk: rows grouped by expert.  Expert e's rows are [start[e], start[e] + count[e]) of the grouped
// operand, every start a multiple of eight; slot_rows maps (token, slot) to its grouped row.
struct ChunkRoute {
    const float* logits = nullptr;      // [rows][logits_ld]
    uint32_t logits_ld = 0, rows = 0, experts = 0, top = 0;
    uint32_t *group_start = nullptr, *group_rows = nullptr;      // [experts]
    uint32_t *slot_rows = nullptr, *slot_experts = nullptr;      // [rows * top]
    float *slot_scores = nullptr, *row_scale = nullptr;          // [rows * top], [grouped rows]
    Operand from, to;                   // the normalised rows, and the grouped operand
};
inline uint32_t grouped_rows(uint32_t rows, uint32_t top, uint32_t experts) { return (rows * top + 8u * experts + 31u) / 16u * 16u; }
int launch_route(const ChunkRoute& route, cudaStream_t stream);      // the choices alone
int launch_chunk_route(const ChunkRoute& route, cudaStream_t stream);

// Cache rows of a chunk: rmsnorm(raw) * gain.
int launch_chunk_latents(const float* raw, uint32_t raw_ld, const float* gain, uint32_t rank, float eps, void* cache_rows, uint32_t row_elements,
                         bool f16, uint32_t rows, uint32_t* status, cudaStream_t stream);

#ifdef __CUDACC__
__device__ __forceinline__ size_t operand_offset(const Operand& o, uint32_t row, uint32_t k) {      // bf16 form, bytes
    return (size_t)(k / kDenseBlockK) * o.capacity * 128u + (size_t)(row / 8u) * 1024u + ((k % kDenseBlockK) / 8u) * 128u + (row % 8u) * 16u + (k % 8u) * 2u;
}
__device__ __forceinline__ void store_operand(const Operand& o, uint32_t row, uint32_t k, float v) {
    if (o.f32) static_cast<float*>(o.data)[(size_t)row * o.k_pad + k] = v;
    else {
        const uint32_t bits = __float_as_uint(v);      // round to nearest even; NaN stays NaN
        const uint16_t r = (bits & 0x7fffffffu) > 0x7f800000u ? (uint16_t)((bits >> 16) | 0x40u) : (uint16_t)((bits + 0x7fffu + ((bits >> 16) & 1u)) >> 16);
        *reinterpret_cast<uint16_t*>(static_cast<uint8_t*>(o.data) + operand_offset(o, row, k)) = r;
    }
}
__device__ __forceinline__ float squared_relu(float z) { const float r = fmaxf(z, 0.0f); return r * r; }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(1.702 g) * (u + 1)
__device__ __forceinline__ float clamped_gate(float gate, float up, float limit) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g * sigmoid(1.702f * g) * (u + 1.0f);
}
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }      // to a few 1e-7
__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z))); }
// One warp turns the (maximum, sum) pairs of a query's key partitions, and its sink, into the factors of the merge.
__device__ __forceinline__ void merge_factors(const float* ml, uint32_t parts, float sink, float* factors) {
    const uint32_t lane = threadIdx.x & 31u;
    float top = sink;
    for (uint32_t part = lane; part < parts; part += 32u) top = fmaxf(top, ml[part * 2u]);
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, offset));
    float total = 0.0f;
    for (uint32_t part = lane; part < parts; part += 32u) {
        const float f = ml[part * 2u + 1u] > 0.0f ? expf(ml[part * 2u] - top) : 0.0f;      // an empty partition has no maximum
        factors[part] = f;
        total += f * ml[part * 2u + 1u];
    }
    total = warp_sum(total) + (sink == -INFINITY ? 0.0f : expf(sink - top));
    for (uint32_t part = lane; part < parts; part += 32u) factors[part] /= total;
}
// One warp picks the `slots` best experts of a row of router logits in order; `scores` is a warp's scratch of
// `experts` floats in shared memory.  pick(slot, expert, score) is called on every lane.
template <typename Pick>
__device__ __forceinline__ void route_row(const float* logits, uint32_t experts, uint32_t slots, float* scores, Pick pick) {
    const uint32_t lane = threadIdx.x & 31u;
    for (uint32_t e = lane; e < experts; e += 32u) scores[e] = sigmoid(logits[e]);
    __syncwarp();
    for (uint32_t slot = 0; slot < slots; ++slot) {
        float best = -1.0f;                            // below every score; chosen experts are marked with -2
        uint32_t at = experts;
        for (uint32_t e = lane; e < experts; e += 32u)
            if (scores[e] > best) { best = scores[e]; at = e; }
#pragma unroll
        for (int offset = 16; offset > 0; offset >>= 1) {
            const float other = __shfl_xor_sync(0xffffffffu, best, offset);
            const uint32_t index = __shfl_xor_sync(0xffffffffu, at, offset);
            if (other > best || (other == best && index < at)) { best = other; at = index; }
        }
        if (at >= experts) { at = 0; best = __int_as_float(0x7fc00000); }      // scores that are not numbers
        pick(slot, at, best);
        __syncwarp();
        if (lane == 0) scores[at] = -2.0f;
        __syncwarp();
    }
}
#endif

}  // namespace gf
