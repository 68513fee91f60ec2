// Products over a chunk of prompt rows and the elementwise steps between them (see dense.cuh).
#include "dense.cuh"
#include "tcgen05.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

namespace {

// ------------------------------------------------------------------ outputs

// Column n of the result of product `index` for output row `row`.
__device__ __forceinline__ void chunk_store(const ChunkProblem& p, uint32_t index, uint32_t row, uint32_t n, float v) {
    if (p.output == kChunkF32) {
        if (p.row_scale) {
            const float s = p.row_scale[(size_t)row * p.row_scale_ld];
            v *= p.row_scale_sigmoid ? sigmoid(s) : s;
        }
        p.out[(size_t)row * p.out_ld + n] = v;
    } else if (p.output == kChunkLatentQuery) {
        const size_t at = ((size_t)row * p.heads + index) * p.out_ld + n;
        if (p.query_f16) reinterpret_cast<__half*>(p.out)[at] = __float2half_rn(v * p.scale);
        else p.out[at] = v * p.scale;
    } else if (p.output == kChunkHalfRows) {
        const uint32_t column = (p.segment ? n / p.segment * p.segment_pad + n % p.segment : n) + index * p.column_stride;
        __half* out = reinterpret_cast<__half*>(p.out) + (size_t)row * p.out_ld + column;
        *out = __float2half_rn(v * p.scale);
        if (p.segment && n % p.segment + 1u == p.segment)               // the padding takes part in scores
            for (uint32_t i = 1; i <= p.segment_pad - p.segment; ++i) out[i] = __float2half_rn(0.0f);
    } else {
        const uint32_t column = (p.segment ? n / p.segment * p.segment_pad + n % p.segment : n) + index * p.column_stride;
        store_operand(p.result, row, column, p.output == kChunkSquaredRelu ? squared_relu(v) : v);
    }
}
// Column n of a paired product.
__device__ __forceinline__ float chunk_gate(const ChunkProblem& p, float gate, float up) {
    return p.output == kChunkGeluGate ? gelu_tanh(gate) * up : clamped_gate(gate, up, p.limit);
}
__device__ __forceinline__ void chunk_store_gate(const ChunkProblem& p, uint32_t row, uint32_t n, float gate, float up) {
    const float s = p.row_scale ? p.row_scale[(size_t)row * p.row_scale_ld] : 1.0f;
    store_operand(p.result, row, n, chunk_gate(p, gate * s, up * s));
}

__device__ __forceinline__ uint4 bf16_octet(const float (&v)[8]) {
    uint4 r;
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r.x) : "f"(v[1]), "f"(v[0]));
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r.y) : "f"(v[3]), "f"(v[2]));
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r.z) : "f"(v[5]), "f"(v[4]));
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r.w) : "f"(v[7]), "f"(v[6]));
    return r;
}
__device__ __forceinline__ uint4 half_octet(const float (&v)[8], float scale) {
    uint4 r;
    uint32_t* w = &r.x;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __half2 h = __floats2half2_rn(v[2 * i] * scale, v[2 * i + 1] * scale);
        w[i] = *reinterpret_cast<const uint32_t*>(&h);
    }
    return r;
}

// Columns n .. n + 7 (n a multiple of eight) of an output row at once where they stay together in the result and start
// on a 16-byte boundary; one by one otherwise.
__device__ __forceinline__ void chunk_store8(const ChunkProblem& p, uint32_t index, uint32_t row, uint32_t n, float (&v)[8]) {
    const bool whole = n + 8u <= p.n && p.segment % 8u == 0u;
    const uint32_t column = (p.segment ? n / p.segment * p.segment_pad + n % p.segment : n) + index * p.column_stride;
    if (whole && p.output == kChunkF32 && p.out_ld % 4u == 0u) {
        float s = 1.0f;
        if (p.row_scale) {
            s = p.row_scale[(size_t)row * p.row_scale_ld];
            if (p.row_scale_sigmoid) s = sigmoid(s);
        }
        float* out = p.out + (size_t)row * p.out_ld + n;
        *reinterpret_cast<float4*>(out) = make_float4(v[0] * s, v[1] * s, v[2] * s, v[3] * s);
        *reinterpret_cast<float4*>(out + 4) = make_float4(v[4] * s, v[5] * s, v[6] * s, v[7] * s);
        return;
    }
    if (whole && column % 8u == 0u && (p.output == kChunkOperand || p.output == kChunkSquaredRelu)) {
        if (p.output == kChunkSquaredRelu)
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = squared_relu(v[i]);
        *reinterpret_cast<uint4*>(static_cast<uint8_t*>(p.result.data) + operand_offset(p.result, row, column)) = bf16_octet(v);
        return;
    }
    if (whole && p.out_ld % 8u == 0u && p.output == kChunkLatentQuery && p.query_f16) {
        *reinterpret_cast<uint4*>(reinterpret_cast<__half*>(p.out) + ((size_t)row * p.heads + index) * p.out_ld + n) = half_octet(v, p.scale);
        return;
    }
    if (whole && p.out_ld % 8u == 0u && column % 8u == 0u && p.output == kChunkHalfRows && p.segment == p.segment_pad) {
        *reinterpret_cast<uint4*>(reinterpret_cast<__half*>(p.out) + (size_t)row * p.out_ld + column) = half_octet(v, p.scale);
        return;
    }
#pragma unroll 1
    for (uint32_t i = 0; i < 8u && n + i < p.n; ++i) chunk_store(p, index, row, n + i, v[i]);
}

// ------------------------------------------------------------------ bf16 products on tcgen05

constexpr uint32_t kWindowMax = 256;                                   // token rows of a tile: the product's N
constexpr uint32_t kMaxStages = 8;                                     // a stage: 128 weight columns, then the window's token rows, x 64 K
constexpr uint32_t kEpilogueWarps = 8;
constexpr uint32_t kStagedLd = kDenseTile + 4u;                        // floats between staged output rows
constexpr uint32_t kChunkThreads = (kEpilogueWarps + 2u) * 32u;        // the copying and the issuing warp behind them
constexpr uint32_t kSmemAlone = 208u * 1024u, kSmemPaired = 104u * 1024u;      // stages of a CTA that has its SM alone, or shares it with another

// The tensor core's A operand is a tile of 128 weight columns and its B operand a window of up to 256 token rows, so
// the product's N follows the rows there are (an expert may have few) and accumulator lanes are output columns.
__global__ void __launch_bounds__(kChunkThreads, 1) chunk_product_kernel(const __grid_constant__ ChunkProduct p) {
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ uint32_t tmem_slot, abort_flag;
    __shared__ __align__(8) uint64_t full[kMaxStages];                  // copies landed (bytes)
    __shared__ __align__(8) uint64_t free_bar[kMaxStages];              // the stage's products have finished
    __shared__ __align__(8) uint64_t done_bar[1];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const volatile uint32_t* abort = &abort_flag;

    uint32_t which = 0;
    while (which + 1u < p.problems && blockIdx.x >= p.p[which + 1u].first_tile) ++which;
    const ChunkProblem& m = p.p[which];
    const uint32_t index = (blockIdx.x - m.first_tile) / m.tiles, tile = (blockIdx.x - m.first_tile) % m.tiles;
    const uint32_t start = m.group_start ? m.group_start[index] : 0u, rows = m.group_rows ? m.group_rows[index] : p.rows;
    const uint32_t first_row = blockIdx.y * p.window;
    if (first_row >= rows) return;
    const uint32_t live = min(p.window, rows - first_row), n_rows = (live + 15u) & ~15u, row0 = start + first_row;
    const uint8_t* weight = m.weight + index * m.weight_stride + (size_t)tile * m.k_blocks * kDenseTileBytes;
    const uint8_t* rows_at = static_cast<const uint8_t*>(m.a.data) + (size_t)(m.a_block0 + index * m.a_block_stride) * m.a.capacity * 128u + (size_t)row0 * 128u;

    const uint32_t stage_bytes = kDenseTileBytes + n_rows * 128u, stages = min(kMaxStages, p.stage_budget / stage_bytes);
    uint32_t tmem_columns = 32u;
    while (tmem_columns < n_rows) tmem_columns *= 2u;
    if (tid == 0) {
        abort_flag = 0u;
        for (uint32_t i = 0; i < kMaxStages; ++i) { mbar_init(&full[i], 1); mbar_init(&free_bar[i], 1); }
        mbar_init(done_bar, 1);
        fence_barrier_init();
    }
    if (warp == 0) tmem_alloc(&tmem_slot, tmem_columns);
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem = tmem_slot, steps = m.k_blocks;
    bool ok = true;

    if (warp == kEpilogueWarps) {
        if (lane == 0) {
            uint32_t requested = 0;
            for (uint32_t step = 0; step < steps; ++step) {
                const uint32_t stage = step % stages, use = step / stages;
                if (use > 0u && !wait_or_abort(&free_bar[stage], (use - 1u) & 1u, abort)) { ok = false; break; }
                uint8_t* at = smem + stage * stage_bytes;
                mbar_expect_tx(&full[stage], kDenseTileBytes + n_rows * 128u);
                bulk_load(at, weight + (size_t)step * kDenseTileBytes, kDenseTileBytes, &full[stage]);
                bulk_load(at + kDenseTileBytes, rows_at + (size_t)step * m.a.capacity * 128u, n_rows * 128u, &full[stage]);
                requested = step + 1u;
            }
            if (!ok || !wait_or_abort(done_bar, 0u, abort)) {
                // Copies already requested get a bounded chance to land before the shared memory is released.
                ok = false;
                abort_flag = 1u;
                for (uint32_t step = requested > stages ? requested - stages : 0u; step < requested; ++step)
                    mbar_wait(&full[step % stages], (step / stages) & 1u, 1u << 16);
            }
        }
    } else if (warp == kEpilogueWarps + 1u) {
        if (lane == 0) {
            const uint32_t instruction = mma_instruction(kDenseTile, n_rows);
            for (uint32_t step = 0; step < steps; ++step) {
                const uint32_t stage = step % stages;
                if (!wait_or_abort(&full[stage], (step / stages) & 1u, abort)) { ok = false; break; }
                tc_fence_after_sync();
                const uint32_t at = smem_u32(smem + stage * stage_bytes);
#pragma unroll
                for (uint32_t kk = 0; kk < kDenseBlockK / 16u; ++kk)
                    mma_bf16(tmem, operand_descriptor(at + kk * 256u), operand_descriptor(at + kDenseTileBytes + kk * 256u), instruction, (step | kk) != 0u ? 1u : 0u);
                mma_commit(&free_bar[stage]);
            }
            if (ok) mma_commit(done_bar);
            else abort_flag = 1u;
        }
    } else {
        if (!wait_or_abort(done_bar, 0u, abort)) { ok = false; if (lane == 0) abort_flag = 1u; }
    }
    const bool failed = __syncthreads_or(ok ? 0 : 1) != 0;
    // Output, 64 token rows at a time: the accumulators go through shared memory (the stages are free again), so that a
    // thread holds eight neighbouring columns of a row.
    float* staged = reinterpret_cast<float*>(smem);                     // [64][kStagedLd]
    for (uint32_t c0 = 0; c0 < live && !failed; c0 += 64u) {
        if (warp < kEpilogueWarps) {
            // Warp w reads accumulator lanes 32 (w % 4) .. + 31, i.e. output columns; a warp's accumulator columns are token rows.
            tc_fence_after_sync();
            const uint32_t quarter = warp & 3u, c = c0 + (warp >> 2) * 32u;
            if (c < live) {
                float v[32];
                tmem_load_32(tmem + ((quarter * 32u) << 16) + c, v);
#pragma unroll
                for (uint32_t i = 0; i < 32u; ++i) staged[((warp >> 2) * 32u + i) * kStagedLd + quarter * 32u + lane] = v[i];
            }
            tc_fence_before_sync();
        }
        __syncthreads();
        const bool paired = paired_chunk(m.output);
        const uint32_t octets = paired ? 8u : 16u, count = min(64u, live - c0) * octets;
#pragma unroll 1
        for (uint32_t i = tid; i < count; i += kChunkThreads) {
            const uint32_t r = i / octets, octet = i % octets, row = row0 + c0 + r;
            const float* src = staged + r * kStagedLd + octet * (paired ? 16u : 8u);
            float v[8];
#pragma unroll
            for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4*>(v + j) = *reinterpret_cast<const float4*>(src + j);
            if (!paired) {
                const uint32_t n = tile * kDenseTile + octet * 8u;
                if (n < m.n) chunk_store8(m, index, row, n, v);
                continue;
            }
            const uint32_t n = tile * (kDenseTile / 2u) + octet * 8u;
            if (n >= m.n / 2u) continue;
            const float s = m.row_scale ? m.row_scale[(size_t)row * m.row_scale_ld] : 1.0f;
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = chunk_gate(m, v[j] * s, src[8 + j] * s);
            *reinterpret_cast<uint4*>(static_cast<uint8_t*>(m.result.data) + operand_offset(m.result, row, n)) = bf16_octet(v);
        }
        __syncthreads();
    }
    if (failed && tid == 0) atomicExch(p.error_flag, 1);
    __syncthreads();
    if (warp == 0) tmem_dealloc(tmem, tmem_columns);
}

// ------------------------------------------------------------------ f32 products

// 64 rows x 64 columns per CTA, 4 x 4 per thread; a thread's columns are two (gate, up) pairs of a paired matrix.
__global__ void __launch_bounds__(256) chunk_product_f32_kernel(const __grid_constant__ ChunkProduct p) {
    __shared__ float a_tile[32][65], w_tile[32][65];
    const uint32_t tid = threadIdx.x;
    uint32_t which = 0;
    while (which + 1u < p.problems && blockIdx.x >= p.p[which + 1u].first_tile) ++which;
    const ChunkProblem& m = p.p[which];
    const uint32_t index = (blockIdx.x - m.first_tile) / m.tiles, tile = (blockIdx.x - m.first_tile) % m.tiles;
    const uint32_t start = m.group_start ? m.group_start[index] : 0u, rows = m.group_rows ? m.group_rows[index] : p.rows;
    const uint32_t first_row = blockIdx.y * 64u;
    if (first_row >= rows) return;
    const uint32_t live = min(64u, rows - first_row), row0 = start + first_row;
    const uint8_t* weight = m.weight + index * m.weight_stride;
    const float* a = static_cast<const float*>(m.a.data) + (size_t)(m.a_block0 + index * m.a_block_stride) * kDenseBlockK;
    const uint32_t tx = tid & 15u, ty = tid >> 4, column0 = (tx >> 3) * 16u + (tx & 7u);
    const uint32_t columns[4] = {column0, column0 + 8u, column0 + 32u, column0 + 40u};
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < m.k; k0 += 32u) {
        for (uint32_t i = tid; i < 64u * 32u; i += 256u) {
            const uint32_t r = i >> 5, k = i & 31u;
            a_tile[k][r] = r < live && k0 + k < m.k ? a[(size_t)(row0 + r) * m.a.k_pad + k0 + k] : 0.0f;
        }
        {
            const uint32_t n = tid & 63u, piece = tid >> 6;            // 64 columns x four pieces of eight
            const uint4 v = *reinterpret_cast<const uint4*>(weight + dense_offset(m.k_blocks, tile * 64u + n, k0 + piece * 8u));
            const uint32_t words[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (uint32_t j = 0; j < 4u; ++j) {
                w_tile[piece * 8u + 2u * j][n] = __uint_as_float(words[j] << 16);
                w_tile[piece * 8u + 2u * j + 1u][n] = __uint_as_float(words[j] & 0xffff0000u);
            }
        }
        __syncthreads();
#pragma unroll 8
        for (uint32_t k = 0; k < 32u; ++k) {
            float x[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { x[i] = a_tile[k][ty * 4u + i]; w[i] = w_tile[k][columns[i]]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (int i = 0; i < 4; ++i) {
        const uint32_t r = ty * 4u + i;
        if (r >= live) continue;
        if (paired_chunk(m.output)) {
            for (int j = 0; j < 4; j += 2) {
                const uint32_t n = tile * 32u + (columns[j] >> 4) * 8u + (columns[j] & 7u);
                if (n < m.n / 2u) chunk_store_gate(m, row0 + r, n, acc[i][j], acc[i][j + 1]);
            }
        } else {
            for (int j = 0; j < 4; ++j)
                if (tile * 64u + columns[j] < m.n) chunk_store(m, index, row0 + r, tile * 64u + columns[j], acc[i][j]);
        }
    }
}

// ------------------------------------------------------------------ norms, routing, cache rows

__device__ __forceinline__ float block_total(float v, float* scratch) {
    v = warp_sum(v);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float total = 0.0f;
    for (uint32_t w = 0; w < blockDim.x / 32u; ++w) total += scratch[w];
    __syncthreads();
    return total;
}

__global__ void __launch_bounds__(256) chunk_norm_kernel(const ChunkNorm p) {
    extern __shared__ __align__(16) float row_values[];
    __shared__ float scratch[8];
    const uint32_t row = blockIdx.x;
    float* residual = p.residual + (size_t)row * p.width;
    float sum = 0.0f;
    if (p.width % 8u == 0u && !p.slots && !p.result.f32) {             // whole 16-byte pieces
        auto octet = [](float* to, const float* from) {
#pragma unroll
            for (int j = 0; j < 8; j += 4) *reinterpret_cast<float4*>(to + j) = *reinterpret_cast<const float4*>(from + j);
        };
        float v[8], g[8];
        if (p.y) {
            for (uint32_t i = threadIdx.x * 8u; i < p.width; i += blockDim.x * 8u) {
                octet(v, p.y + (size_t)row * p.width + i);
                octet(row_values + i, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) sum = fmaf(v[j], v[j], sum);
            }
            const float inv = 1.0f / sqrtf(block_total(sum, scratch) / (float)p.width + p.eps);
            sum = 0.0f;
            for (uint32_t i = threadIdx.x * 8u; i < p.width; i += blockDim.x * 8u) {
                float x[8];
                octet(v, residual + i);
                octet(x, row_values + i);
                octet(g, p.gain0 + i);
#pragma unroll
                for (int j = 0; j < 8; ++j) { v[j] += x[j] * inv * g[j]; sum = fmaf(v[j], v[j], sum); }
                octet(residual + i, v);
                octet(row_values + i, v);
            }
        } else {
            for (uint32_t i = threadIdx.x * 8u; i < p.width; i += blockDim.x * 8u) {
                octet(v, residual + i);
                octet(row_values + i, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) sum = fmaf(v[j], v[j], sum);
            }
        }
        const float inv = p.gain1 ? 1.0f / sqrtf(block_total(sum, scratch) / (float)p.width + p.eps) : 1.0f;
        for (uint32_t i = threadIdx.x * 8u; i < p.width; i += blockDim.x * 8u) {
            octet(v, row_values + i);
            if (p.gain1) {
                octet(g, p.gain1 + i);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] = v[j] * inv * g[j];
            }
            if (p.result.data) *reinterpret_cast<uint4*>(static_cast<uint8_t*>(p.result.data) + operand_offset(p.result, row, i)) = bf16_octet(v);
            if (p.normed) octet(p.normed + (size_t)row * p.width + i, v);
        }
        return;
    }
    if (p.y) {
        for (uint32_t i = threadIdx.x; i < p.width; i += blockDim.x) {
            float v;
            if (p.slots) {
                v = 0.0f;
                for (uint32_t s = 0; s < p.slots; ++s) v += p.y[(size_t)p.slot_rows[row * p.slots + s] * p.width + i];
                if (p.shared) v += p.shared[(size_t)row * p.width + i];
            } else v = p.y[(size_t)row * p.width + i];
            row_values[i] = v;
            sum = fmaf(v, v, sum);
        }
        const float inv = 1.0f / sqrtf(block_total(sum, scratch) / (float)p.width + p.eps);
        sum = 0.0f;
        for (uint32_t i = threadIdx.x; i < p.width; i += blockDim.x) {
            const float v = residual[i] + row_values[i] * inv * p.gain0[i];
            residual[i] = v;
            row_values[i] = v;
            sum = fmaf(v, v, sum);
        }
    } else {
        for (uint32_t i = threadIdx.x; i < p.width; i += blockDim.x) {
            const float v = residual[i];
            row_values[i] = v;
            sum = fmaf(v, v, sum);
        }
    }
    const float inv = p.gain1 ? 1.0f / sqrtf(block_total(sum, scratch) / (float)p.width + p.eps) : 1.0f;
    for (uint32_t i = threadIdx.x; i < p.width; i += blockDim.x) {
        const float v = p.gain1 ? row_values[i] * inv * p.gain1[i] : row_values[i];
        if (p.result.data) store_operand(p.result, row, i, v);
        if (p.normed) p.normed[(size_t)row * p.width + i] = v;
    }
}

// Block = (row, part): the part by its own root mean square.
__global__ void __launch_bounds__(256) chunk_part_norm_kernel(const float* __restrict__ x, uint32_t x_ld, const float* __restrict__ gate, uint32_t gate_ld, uint32_t part, const float* __restrict__ gain, float eps,
                                                              const Operand result) {
    extern __shared__ __align__(16) float row_values[];
    __shared__ float scratch[8];
    const uint32_t row = blockIdx.x, first = blockIdx.y * part;
    const float *in = x + (size_t)row * x_ld + first, *z = gate + (size_t)row * gate_ld + first;
    float sum = 0.0f;
    for (uint32_t i = threadIdx.x; i < part; i += blockDim.x) {
        const float v = in[i] * silu(z[i]);
        row_values[i] = v;
        sum = fmaf(v, v, sum);
    }
    const float inv = 1.0f / sqrtf(block_total(sum, scratch) / (float)part + eps);
    for (uint32_t i = threadIdx.x; i < part; i += blockDim.x) store_operand(result, row, first + i, row_values[i] * inv * gain[first + i]);
}

// The same for parts of whole 256 values, bf16: block = row, a thread takes eight values at a time.
__global__ void __launch_bounds__(256) chunk_part_norm_octets_kernel(const float* __restrict__ x, uint32_t x_ld, const float* __restrict__ gate, uint32_t gate_ld,
                                                                     uint32_t width, uint32_t part, const float* __restrict__ gain, float eps, const Operand result) {
    extern __shared__ __align__(16) float row_values[];                // [width], then a sum per 256 values
    float* sums = row_values + width;
    const uint32_t row = blockIdx.x;
    for (uint32_t i = threadIdx.x * 8u; i < width; i += blockDim.x * 8u) {
        float sum = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; j += 4) {
            const float4 v = *reinterpret_cast<const float4*>(x + (size_t)row * x_ld + i + j), z = *reinterpret_cast<const float4*>(gate + (size_t)row * gate_ld + i + j);
            const float4 y = make_float4(v.x * silu(z.x), v.y * silu(z.y), v.z * silu(z.z), v.w * silu(z.w));
            *reinterpret_cast<float4*>(row_values + i + j) = y;
            sum = fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, fmaf(y.w, y.w, sum))));
        }
        sum = warp_sum(sum);
        if ((threadIdx.x & 31u) == 0u) sums[i / 256u] = sum;
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x * 8u; i < width; i += blockDim.x * 8u) {
        const uint32_t first = i / part * (part / 256u);
        float sum = 0.0f, v[8];
        for (uint32_t s = 0; s < part / 256u; ++s) sum += sums[first + s];
        const float inv = 1.0f / sqrtf(sum / (float)part + eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = row_values[i + j] * inv * gain[i + j];
        *reinterpret_cast<uint4*>(static_cast<uint8_t*>(result.data) + operand_offset(result, row, i)) = bf16_octet(v);
    }
}

// A warp per row chooses its experts.
__global__ void __launch_bounds__(128) chunk_route_kernel(const ChunkRoute p) {
    extern __shared__ float scores[];                                  // [warps][experts]
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, row = blockIdx.x * 4u + warp;
    if (row >= p.rows) return;
    route_row(p.logits + (size_t)row * p.logits_ld, p.experts, p.top, scores + warp * p.experts, [&](uint32_t slot, uint32_t e, float score) {
        if (lane != 0) return;
        p.slot_experts[row * p.top + slot] = e;
        p.slot_scores[row * p.top + slot] = score;
    });
}

// One block: the experts' counts, their starts, and every choice's grouped row.
__global__ void __launch_bounds__(1024) chunk_starts_kernel(const ChunkRoute p) {
    __shared__ uint32_t counts[kMaxExperts], starts[kMaxExperts];
    for (uint32_t e = threadIdx.x; e < p.experts; e += blockDim.x) counts[e] = 0;
    __syncthreads();
    for (uint32_t at = threadIdx.x; at < p.rows * p.top; at += blockDim.x) p.slot_rows[at] = atomicAdd(&counts[p.slot_experts[at]], 1u);
    __syncthreads();
    if (threadIdx.x < 32u) {                                           // prefix sums of the counts, rounded up to eight
        uint32_t before = 0;
        for (uint32_t first = 0; first < p.experts; first += 32u) {
            const uint32_t e = first + threadIdx.x, padded = e < p.experts ? (counts[e] + 7u) & ~7u : 0u;
            uint32_t sum = padded;
#pragma unroll
            for (int offset = 1; offset < 32; offset <<= 1) {
                const uint32_t other = __shfl_up_sync(0xffffffffu, sum, offset);
                if (threadIdx.x >= (uint32_t)offset) sum += other;
            }
            if (e < p.experts) starts[e] = before + sum - padded;
            before += __shfl_sync(0xffffffffu, sum, 31);
        }
    }
    __syncthreads();
    for (uint32_t e = threadIdx.x; e < p.experts; e += blockDim.x) { p.group_start[e] = starts[e]; p.group_rows[e] = counts[e]; }
    for (uint32_t at = threadIdx.x; at < p.rows * p.top; at += blockDim.x) {
        const uint32_t grouped = starts[p.slot_experts[at]] + p.slot_rows[at];
        p.slot_rows[at] = grouped;
        p.row_scale[grouped] = p.slot_scores[at];
    }
}

// Copies a token's normalised row to its grouped rows, 16 bytes at a time.
__global__ void __launch_bounds__(256) chunk_group_kernel(const ChunkRoute p) {
    const uint32_t at = blockIdx.x, row = at / p.top, grouped = p.slot_rows[at];
    if (p.from.f32) {
        const float4* src = reinterpret_cast<const float4*>(static_cast<const float*>(p.from.data) + (size_t)row * p.from.k_pad);
        float4* dst = reinterpret_cast<float4*>(static_cast<float*>(p.to.data) + (size_t)grouped * p.to.k_pad);
        for (uint32_t i = threadIdx.x; i < p.from.k_pad / 4u; i += blockDim.x) dst[i] = src[i];
        return;
    }
    for (uint32_t i = threadIdx.x; i < p.from.k_pad / 8u; i += blockDim.x)
        *reinterpret_cast<uint4*>(static_cast<uint8_t*>(p.to.data) + operand_offset(p.to, grouped, i * 8u)) =
            *reinterpret_cast<const uint4*>(static_cast<const uint8_t*>(p.from.data) + operand_offset(p.from, row, i * 8u));
}

__global__ void __launch_bounds__(256) chunk_operand_kernel(const float* __restrict__ x, uint32_t k, const Operand result) {
    for (uint32_t i = threadIdx.x; i < result.k_pad; i += blockDim.x) store_operand(result, blockIdx.x, i, i < k ? x[(size_t)blockIdx.x * k + i] : 0.0f);
}

__global__ void __launch_bounds__(128) chunk_latents_kernel(const float* __restrict__ raw, uint32_t raw_ld, const float* __restrict__ gain, uint32_t rank,
                                                            float eps, void* cache_rows, uint32_t row_elements, bool f16, uint32_t* status) {
    __shared__ float scratch[8];
    const uint32_t row = blockIdx.x;
    const float* x = raw + (size_t)row * raw_ld;
    float sum = 0.0f;
    for (uint32_t i = threadIdx.x; i < rank; i += blockDim.x) sum = fmaf(x[i], x[i], sum);
    const float inv = 1.0f / sqrtf(block_total(sum, scratch) / (float)rank + eps);
    for (uint32_t i = threadIdx.x; i < row_elements; i += blockDim.x) {
        const float v = i < rank ? x[i] * inv * gain[i] : 0.0f;
        const size_t at = (size_t)row * row_elements + i;
        if (f16) {
            const __half h = __float2half_rn(v);
            if (__hisinf(h) || __hisnan(h)) atomicOr(status, kStatusKvNonFinite);
            static_cast<__half*>(cache_rows)[at] = h;
        } else static_cast<float*>(cache_rows)[at] = v;
    }
}

template <typename Kernel>
int allow_smem(Kernel kernel, std::once_flag* once, uint32_t bytes) {
    int device = 0;
    cudaGetDevice(&device);
    cudaError_t error = cudaSuccess;
    std::call_once(once[device & 63], [&] { error = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes); });
    GF_CUDA(error);
    return GF_OK;
}

}  // namespace

int launch_chunk_product(ChunkProduct p, bool f32, cudaStream_t stream) {
    if (p.problems == 0 || p.problems > 3 || p.rows == 0 || !p.error_flag) return fail(GF_ERR_INVALID, "chunk product: bad launch");
    const uint32_t tile_columns = f32 ? 64u : kDenseTile;
    uint32_t total = 0;
    for (uint32_t i = 0; i < p.problems; ++i) {
        ChunkProblem& m = p.p[i];
        if (!m.weight || !m.a.data || m.n == 0 || m.k == 0 || m.count == 0 || m.a.f32 != (f32 ? 1u : 0u)) return fail(GF_ERR_INVALID, "chunk product: bad problem");
        m.k_blocks = (m.k + kDenseBlockK - 1u) / kDenseBlockK;
        if ((m.a_block0 + (m.count - 1u) * m.a_block_stride + m.k_blocks) * kDenseBlockK > m.a.k_pad) return fail(GF_ERR_INVALID, "chunk product: the operand is narrower than K");
        if (!m.group_rows && p.rows > m.a.capacity) return fail(GF_ERR_INVALID, "chunk product: more rows than the operand holds");
        m.first_tile = total;
        m.tiles = (m.n + tile_columns - 1u) / tile_columns;
        total += m.tiles * m.count;
    }
    if (f32) {
        p.window = 64u;
        chunk_product_f32_kernel<<<dim3(total, (p.rows + 63u) / 64u), 256, 0, stream>>>(p);
    } else {
        // The widest window of rows that still gives most SMs a tile.
        p.window = kWindowMax;
        while (p.window > 64u && (uint64_t)total * ((p.rows + p.window - 1u) / p.window) * 5u < (uint64_t)sm_count() * 4u) p.window /= 2u;
        static std::once_flag once[64];
        const int status = allow_smem(chunk_product_kernel, once, kSmemAlone);
        if (status != GF_OK) return status;
        // Many tiles: two CTAs share an SM, so that one's start and output overlap the other's products.
        p.stage_budget = (uint64_t)total * ((p.rows + p.window - 1u) / p.window) > 3u * (uint64_t)sm_count() ? kSmemPaired : kSmemAlone;
        chunk_product_kernel<<<dim3(total, (p.rows + p.window - 1u) / p.window), kChunkThreads, p.stage_budget, stream>>>(p);
    }
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

int launch_chunk_norm(const ChunkNorm& p, cudaStream_t stream) {
    if (!p.residual || p.rows == 0 || p.width == 0 || p.width > 48u * 1024u) return fail(GF_ERR_INVALID, "chunk norm: bad arguments");
    static std::once_flag once[64];
    const int status = allow_smem(chunk_norm_kernel, once, 200u * 1024u);
    if (status != GF_OK) return status;
    chunk_norm_kernel<<<p.rows, 256, p.width * 4u, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

int launch_chunk_part_norm(const float* x, uint32_t x_ld, const float* gate, uint32_t gate_ld, uint32_t width, uint32_t parts, const float* gain, float eps, const Operand& result, uint32_t rows,
                           cudaStream_t stream) {
    if (!x || !gate || !gain || !result.data || rows == 0 || rows > result.capacity || parts == 0 || parts > kMaxNormParts || width % parts || width > result.k_pad
        || width / parts > 48u * 1024u)
        return fail(GF_ERR_INVALID, "chunk part norm: bad arguments");
    const uint32_t part = width / parts;
    static std::once_flag once[2][64];
    int status = allow_smem(chunk_part_norm_kernel, once[0], 200u * 1024u);
    if (status == GF_OK) status = allow_smem(chunk_part_norm_octets_kernel, once[1], 200u * 1024u);
    if (status != GF_OK) return status;
    if (part % 256u == 0u && x_ld % 4u == 0u && gate_ld % 4u == 0u && width <= 40u * 1024u && !result.f32) {
        chunk_part_norm_octets_kernel<<<rows, 256, (width + width / 256u) * 4u, stream>>>(x, x_ld, gate, gate_ld, width, part, gain, eps, result);
        GF_CUDA(cudaGetLastError());
        return GF_OK;
    }
    chunk_part_norm_kernel<<<dim3(rows, parts), part >= 256u ? 256u : (part + 31u) / 32u * 32u, part * 4u, stream>>>(x, x_ld, gate, gate_ld, part, gain, eps, result);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

int launch_route(const ChunkRoute& p, cudaStream_t stream) {
    if (p.rows == 0 || p.experts == 0 || p.experts > kMaxExperts || p.top == 0 || p.top > p.experts) return fail(GF_ERR_INVALID, "route: bad arguments");
    chunk_route_kernel<<<(p.rows + 3u) / 4u, 128, 4u * p.experts * 4u, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

int launch_chunk_route(const ChunkRoute& p, cudaStream_t stream) {
    if (grouped_rows(p.rows, p.top, p.experts) > p.to.capacity) return fail(GF_ERR_INVALID, "chunk route: the grouped operand is too small");
    const int status = launch_route(p, stream);
    if (status != GF_OK) return status;
    chunk_starts_kernel<<<1, 1024, 0, stream>>>(p);
    chunk_group_kernel<<<p.rows * p.top, 256, 0, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

int launch_chunk_operand(const float* x, uint32_t rows, uint32_t k, const Operand& result, cudaStream_t stream) {
    if (!x || !result.data || rows == 0 || rows > result.capacity || k > result.k_pad) return fail(GF_ERR_INVALID, "chunk operand: bad arguments");
    chunk_operand_kernel<<<rows, 256, 0, stream>>>(x, k, result);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

int launch_chunk_latents(const float* raw, uint32_t raw_ld, const float* gain, uint32_t rank, float eps, void* cache_rows, uint32_t row_elements,
                         bool f16, uint32_t rows, uint32_t* status, cudaStream_t stream) {
    chunk_latents_kernel<<<rows, 128, 0, stream>>>(raw, raw_ld, gain, rank, eps, cache_rows, row_elements, f16, status);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

}  // namespace gf
