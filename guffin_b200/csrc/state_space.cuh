// State-space mixer (state-space duality): per head a state S [N][vdim] that decays and takes in an outer product at
// every token, read out by a vector; the inputs pass a short causal convolution first.
//
//   x, B, C = silu(convolution(raw))        dt = softplus(raw + step bias)
//   S_t = exp(decay * dt) S_(t-1) + dt * B_t x_t^T        y_t = S_t^T C_t + skip * x_t
//
// All of it is f32.  A sequence's state after q tokens lies in slot q modulo *slots of its states, each slot
// [heads][vdim][N rounded up to 4]; a pass over rows at position p reads the state after p tokens and leaves those after
// p + 1 .. p + rows.  With more slots than rows, rows that are never published change nothing that is committed; with
// fewer only the last states are left, and such a pass must be published whole.  The convolution's inputs lie in a ring of
// rows by position, as a cache's rows do.
#pragma once

#include "dense.cuh"

namespace gf {

struct StateSpace {
    const float* raw = nullptr;          // [rows][raw_ld]: gate | x | B | C (channels of the convolution) | step, as projected
    uint32_t raw_ld = 0;
    const float *taps = nullptr, *tap_bias = nullptr;      // [channels][tap_count], the last one the current token's; [channels]
    const float *step_bias = nullptr, *decay = nullptr, *skip = nullptr;      // [heads]; decay = -exp(A_log)
    const StreamRings* rings = nullptr;  // rings[row * ring_stride]: ring_k the states, ring_v the convolution's inputs
    uint32_t ring_stride = 0;            // 0: the rows are a chain of one sequence; 1: every row has a sequence of its own
    const uint32_t* positions = nullptr; // chain: position of row 0; else the position of every row
    const uint32_t* slots = nullptr;
    uint32_t rows = 0, heads = 0, vdim = 0, state = 0, groups = 0, tap_count = 0, input_mask = 0;
    float* out = nullptr;                // [rows][heads * vdim]: passes: y * silu(gate); chunks: y
    // Chunks (StateChunk k, the rows rounded up to eight): the convolved inputs, x [heads][blocks of columns][rows][x_ld], B
    // and C [groups][rows][n_ld]; (dt, decay * dt) [rows][heads]; what a head's rows within their eight owe one another
    // [heads][rows][kStateFactors].
    float *x = nullptr, *b = nullptr, *c = nullptr, *factors = nullptr;
    float2* steps = nullptr;
    int* error_flag = nullptr;           // set when a bounded wait for a copy gives up

    __host__ __device__ uint32_t inner() const { return heads * vdim; }
    __host__ __device__ uint32_t channels() const { return inner() + 2u * groups * state; }
    __host__ __device__ uint32_t state_row() const { return (state + 3u) & ~3u; }
    __host__ __device__ uint32_t input_row() const { return (channels() + 3u) & ~3u; }
    __host__ __device__ size_t slot_elements() const { return (size_t)heads * vdim * state_row(); }
};
constexpr uint32_t kMaxStateSize = 1024, kStateFactors = 12;

// How a chunk is cut up: a block takes `columns` of vdim of a head, `splits` warps share N by `per_warp` values, and `tile`
// tokens are in shared memory at a time, in rows of n_ld and x_ld values.
struct StateChunk { uint32_t columns = 0, splits = 0, per_warp = 0, tile = 0, n_ld = 0, x_ld = 0; };
StateChunk state_space_chunk(const StateSpace& p);

// Rows of a pass, convolution included.
int launch_state_space_rows(const StateSpace& p, cudaStream_t stream, bool pdl);
// A chunk of one sequence: the convolution, then the recurrence (two launches).
int launch_state_space_chunk(const StateSpace& p, cudaStream_t stream);

}  // namespace gf
