// Attention over cached latents (see latent.cuh).
#include "latent.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

namespace {

constexpr uint32_t kKeys = 64;                       // cache rows per tile
constexpr uint32_t kNarrowKeys = 32;                 // of the kernel for up to sixteen queries
constexpr uint32_t kThreads = 256;
constexpr uint32_t kSmemLimit = 226u * 1024u;

__device__ __forceinline__ void copy16(void* dst_smem, const void* src, bool valid) {      // zero-fills when not valid
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst_smem)), "l"(src), "r"(valid ? 16u : 0u) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix4_transposed(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LatentSmem { uint32_t q, cache, scores, weights, stats, bytes; };
template <int MT>
__host__ __device__ inline LatentSmem latent_smem(uint32_t row_elements) {
    constexpr uint32_t queries = 16u * MT, keys = MT == 1 ? kNarrowKeys : kKeys, slots = MT == 1 ? 4u : 2u, planes = MT == 1 ? 2u : 1u;
    const uint32_t stride = (row_elements + 8u) * 2u;
    LatentSmem s;
    s.q = 0;
    s.cache = queries * stride;
    s.scores = s.cache + slots * keys * stride;
    s.weights = s.scores + planes * queries * (keys + 4u) * 4u;
    s.stats = s.weights + queries * (keys + 8u) * 2u;
    s.bytes = s.stats + queries * 3u * 4u;
    return s;
}

// A block serves 16 * MT queries -- (row, head) pairs in order, heads fastest -- against one partition of the cache
// rows they see.  Per tile of cache rows: scores on the tensor cores, an online softmax over shared-memory scores, then
// the outputs, warp w accumulating the dimension groups w, w + 8, .. of sixteen; later tiles' rows are copied meanwhile.
// MT = 4 (prompts): tiles of 64 rows, the eight warps split the queries and the tile's rows.  MT = 1 (decoding, bound
// by the cache): tiles of 32 rows, three of them in flight, the warps split the rows and the dimensions of a score.
template <int MT, int NP>
__global__ void __launch_bounds__(kThreads, 1) latent_attention_kernel(const __grid_constant__ LatentAttention p) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr uint32_t kQueries = 16u * MT, kTile = MT == 1 ? kNarrowKeys : kKeys, kSlots = MT == 1 ? 4u : 2u;
    const LatentSmem at = latent_smem<MT>(p.row_elements);
    const uint32_t stride = p.row_elements + 8u;                     // halves; rows land in different banks
    __half* q_tile = reinterpret_cast<__half*>(smem + at.q);
    __half* cache_tiles = reinterpret_cast<__half*>(smem + at.cache);
    float* scores = reinterpret_cast<float*>(smem + at.scores);      // [queries][kTile + 4], two of them for MT = 1
    __half* weights = reinterpret_cast<__half*>(smem + at.weights);  // [queries][kTile + 8]
    float* run_max = reinterpret_cast<float*>(smem + at.stats);
    float* run_sum = run_max + kQueries;
    float* correction = run_sum + kQueries;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, g = lane >> 2, t = lane & 3u;

    pdl_wait();
    pdl_launch_dependents();
    const bool chain = p.ring_stride == 0u;
    const uint32_t z = blockIdx.z, queries = chain ? p.rows * p.heads : p.heads;      // this sequence's queries
    const uint32_t first_query = blockIdx.x * kQueries, part = blockIdx.y;
    const uint32_t base = p.positions[chain ? 0u : z];
    const __half* ring = static_cast<const __half*>(p.rings[(size_t)z * p.ring_stride].ring_k);
    const __half* own = static_cast<const __half*>(p.private_rows) + (chain ? 0u : (size_t)z * p.row_elements);
    const __half* q = static_cast<const __half*>(p.q) + (size_t)z * p.heads * p.row_elements * (chain ? 0u : 1u);
    const uint32_t out_query = chain ? 0u : z * p.heads;
    const uint32_t last_query = min(first_query + kQueries, queries) - 1u;
    const uint32_t end = base + last_query / p.heads + 1u;           // cache rows the block's last query sees
    const uint32_t tiles = (end + kTile - 1u) / kTile;
    const uint32_t tile_begin = (uint32_t)((uint64_t)tiles * part / p.parts), tile_end = (uint32_t)((uint64_t)tiles * (part + 1u) / p.parts);

    const uint32_t pieces = p.row_elements / 8u;
    auto load_tile = [&](uint32_t tile, uint32_t slot) {
        constexpr uint32_t kPerRow = kThreads / kTile;                // threads that share a row, alternating pieces
        const uint32_t r = tid / kPerRow, position = tile * kTile + r;
        const bool valid = position < end;
        const __half* src = !valid ? own : position < base ? ring + (size_t)(position & p.ring_mask) * p.row_elements
                                                          : own + (size_t)(position - base) * p.row_elements;
        __half* dst = cache_tiles + (size_t)slot * kTile * stride + r * stride;
#pragma unroll 4
        for (uint32_t piece = tid % kPerRow; piece < pieces; piece += kPerRow) copy16(dst + piece * 8u, src + piece * 8u, valid);
    };
    for (uint32_t i = tid; i < kQueries * pieces; i += kThreads) {
        const uint32_t m = i / pieces, piece = i % pieces;
        const bool valid = first_query + m < queries;
        copy16(q_tile + m * stride + piece * 8u, q + (size_t)(valid ? first_query + m : 0u) * p.row_elements + piece * 8u, valid);
    }
#pragma unroll
    for (uint32_t i = 0; i + 1u < kSlots; ++i) {                      // one copy group per tile, the queries with the first
        if (tile_begin + i < tile_end) load_tile(tile_begin + i, i);
        copies_commit();
    }
    for (uint32_t m = tid; m < kQueries; m += kThreads) { run_max[m] = -INFINITY; run_sum[m] = 0.0f; correction[m] = 1.0f; }

    float acc[MT][NP][2][4];
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int b = 0; b < NP; ++b)
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int d = 0; d < 4; ++d) acc[a][b][c][d] = 0.0f;

    const uint32_t steps = p.row_elements / 16u;
    for (uint32_t tile = tile_begin; tile < tile_end; ++tile) {
        const uint32_t slot = (tile - tile_begin) % kSlots;
        if (tile + kSlots - 1u < tile_end) load_tile(tile + kSlots - 1u, (slot + kSlots - 1u) % kSlots);
        copies_commit();
        copies_wait<(int)kSlots - 1>();
        __syncthreads();
        const __half* cache = cache_tiles + (size_t)slot * kTile * stride;
        // ---- scores: MT = 4: two query tiles x sixteen keys per warp; MT = 1: sixteen queries x eight keys x half of the
        // dimensions.
        if (MT == 4) {
            const uint32_t m0 = (warp & 1u) * 32u, n0 = (warp >> 1) * 16u;
            float s[2][2][4] = {};
            const __half* a_row = q_tile + (m0 + (lane & 15u)) * stride + (lane >> 4) * 8u;
            const __half* b_row = cache + (n0 + (lane & 7u) + (lane >> 4) * 8u) * stride + ((lane >> 3) & 1u) * 8u;
#pragma unroll 4
            for (uint32_t k = 0; k < steps; ++k) {
                uint32_t a0[4], a1[4], b[4];
                ldmatrix4(a0, a_row + k * 16u);
                ldmatrix4(a1, a_row + 16u * stride + k * 16u);
                ldmatrix4(b, b_row + k * 16u);
                mma_f16(s[0][0], a0, b[0], b[1]);
                mma_f16(s[0][1], a0, b[2], b[3]);
                mma_f16(s[1][0], a1, b[0], b[1]);
                mma_f16(s[1][1], a1, b[2], b[3]);
            }
#pragma unroll
            for (int a = 0; a < 2; ++a)
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    float* out = scores + (m0 + 16u * a + g) * (kTile + 4u) + n0 + 8u * b + 2u * t;
                    *reinterpret_cast<float2*>(out) = make_float2(s[a][b][0], s[a][b][1]);
                    *reinterpret_cast<float2*>(out + 8u * (kTile + 4u)) = make_float2(s[a][b][2], s[a][b][3]);
                }
        } else {
            const uint32_t n0 = (warp & 3u) * 8u, half = warp >> 2, k_end = steps * (half + 1u) / 2u;
            float s[2][4] = {};
            const __half* a_row = q_tile + (lane & 15u) * stride + (lane >> 4) * 8u;
            const __half* b_row = cache + (n0 + (lane & 7u)) * stride + (lane >> 3) * 8u;      // 32 dimensions of eight keys
            uint32_t k = steps * half / 2u;
#pragma unroll 4
            for (; k + 2u <= k_end; k += 2u) {
                uint32_t a0[4], a1[4], b[4];
                ldmatrix4(a0, a_row + k * 16u);
                ldmatrix4(a1, a_row + k * 16u + 16u);
                ldmatrix4(b, b_row + k * 16u);
                mma_f16(s[0], a0, b[0], b[1]);
                mma_f16(s[1], a1, b[2], b[3]);
            }
            if (k < k_end) {
                uint32_t a0[4], b[4];
                ldmatrix4(a0, a_row + k * 16u);
                ldmatrix4(b, cache + (n0 + (lane & 7u)) * stride + ((lane >> 3) & 1u) * 8u + k * 16u);
                mma_f16(s[0], a0, b[0], b[1]);
            }
            float* out = scores + (half * kQueries + g) * (kTile + 4u) + n0 + 2u * t;
            *reinterpret_cast<float2*>(out) = make_float2(s[0][0] + s[1][0], s[0][1] + s[1][1]);
            *reinterpret_cast<float2*>(out + 8u * (kTile + 4u)) = make_float2(s[0][2] + s[1][2], s[0][3] + s[1][3]);
        }
        __syncthreads();
        // ---- softmax: 16 / MT threads per query.
        {
            constexpr uint32_t kPer = kThreads / kQueries, kEach = kTile / kPer;
            const uint32_t m = tid / kPer, sub = tid % kPer;
            const uint32_t sees = base + min(first_query + m, queries - 1u) / p.heads;      // last visible position
            const float* row = scores + m * (kTile + 4u);
            float v[kEach], top = -INFINITY;
#pragma unroll
            for (uint32_t j = 0; j < kEach; ++j) {
                const uint32_t key = j * kPer + sub;
                const float score = MT == 1 ? row[key] + row[kQueries * (kTile + 4u) + key] : row[key];
                v[j] = tile * kTile + key <= sees ? score : -INFINITY;
                top = fmaxf(top, v[j]);
            }
#pragma unroll
            for (uint32_t o = kPer / 2u; o > 0u; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
            const float before = run_max[m], now = fmaxf(before, top);
            float sum = 0.0f;
#pragma unroll
            for (uint32_t j = 0; j < kEach; ++j) {
                const float w = v[j] == -INFINITY ? 0.0f : expf(v[j] - now);
                sum += w;
                weights[m * (kTile + 8u) + j * kPer + sub] = __float2half_rn(w);
            }
#pragma unroll
            for (uint32_t o = kPer / 2u; o > 0u; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            __syncwarp();                                             // every lane has read run_max
            if (sub == 0u) {
                const float c = before == -INFINITY ? 0.0f : expf(before - now);
                run_max[m] = now;
                run_sum[m] = run_sum[m] * c + sum;
                correction[m] = c;
            }
        }
        __syncthreads();
        // ---- outputs
#pragma unroll
        for (int a = 0; a < MT; ++a) {
            const float c0 = correction[16 * a + g], c1 = correction[16 * a + g + 8];
#pragma unroll
            for (int b = 0; b < NP; ++b)
#pragma unroll
                for (int c = 0; c < 2; ++c) { acc[a][b][c][0] *= c0; acc[a][b][c][1] *= c0; acc[a][b][c][2] *= c1; acc[a][b][c][3] *= c1; }
        }
#pragma unroll
        for (uint32_t k = 0; k < kTile / 16u; ++k) {
            uint32_t w[MT][4];
#pragma unroll
            for (int a = 0; a < MT; ++a) ldmatrix4(w[a], weights + (16u * a + (lane & 15u)) * (kTile + 8u) + k * 16u + (lane >> 4) * 8u);
#pragma unroll
            for (int b = 0; b < NP; ++b) {
                const uint32_t d0 = (b * 8u + warp) * 16u;
                if (d0 >= p.row_elements) break;
                uint32_t v[4];
                ldmatrix4_transposed(v, cache + (k * 16u + (lane & 15u)) * stride + d0 + (lane >> 4) * 8u);
#pragma unroll
                for (int a = 0; a < MT; ++a) {
                    mma_f16(acc[a][b][0], w[a], v[0], v[1]);
                    mma_f16(acc[a][b][1], w[a], v[2], v[3]);
                }
            }
        }
        __syncthreads();                                              // the tile and the weights are free again
    }
    copies_wait<0>();
    __syncthreads();

    const bool direct = p.result.data != nullptr;
    if (!direct)
        for (uint32_t m = tid; m < kQueries; m += kThreads)
            if (first_query + m < queries)
                *reinterpret_cast<float2*>(p.partial_ml + ((size_t)(out_query + first_query + m) * p.parts + part) * 2u) = make_float2(run_max[m], run_sum[m]);
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t m = 16u * a + g + 8u * i, query = first_query + m;
            if (query >= queries) continue;
            const uint32_t row = query / p.heads, head = query % p.heads;
            float factor = 1.0f;
            if (direct) {
                const float top = p.sink ? fmaxf(run_max[m], p.sink[head]) : run_max[m];
                const float total = run_sum[m] * expf(run_max[m] - top) + (p.sink ? expf(p.sink[head] - top) : 0.0f);
                factor = expf(run_max[m] - top) / total;
            }
#pragma unroll
            for (int b = 0; b < NP; ++b) {
                const uint32_t d0 = (b * 8u + warp) * 16u;
                if (d0 >= p.row_elements) break;
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const uint32_t d = d0 + 8u * c + 2u * t;
                    const float x = acc[a][b][c][2 * i], y = acc[a][b][c][2 * i + 1];
                    if (direct) {
                        store_operand(p.result, row, head * p.result_stride + d, x * factor);
                        store_operand(p.result, row, head * p.result_stride + d + 1u, y * factor);
                    } else {
                        *reinterpret_cast<float2*>(p.partial_out + ((size_t)(out_query + query) * p.parts + part) * p.row_elements + d) = make_float2(x, y);
                    }
                }
            }
        }
}

// Any shape, f32 arithmetic, f32 or binary16 cache: one block per (query, partition); warps take the keys of a tile in turn for the
// scores, threads the dimensions for the outputs (kept in shared memory).
template <typename Cache>
__global__ void __launch_bounds__(kThreads) latent_attention_plain_kernel(const __grid_constant__ LatentAttention p) {
    extern __shared__ __align__(16) float plain[];                   // query, output: [row_elements] each
    __shared__ float scores[kKeys];
    float* query = plain;
    float* out = plain + p.row_elements;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    pdl_wait();
    pdl_launch_dependents();
    const bool chain = p.ring_stride == 0u;
    const uint32_t m = blockIdx.x, row = m / p.heads, head = m % p.heads, part = blockIdx.y;
    const uint32_t base = p.positions[chain ? 0u : row], end = chain ? base + row + 1u : base + 1u;
    const Cache* ring = static_cast<const Cache*>(p.rings[(size_t)row * p.ring_stride].ring_k);
    const Cache* own = static_cast<const Cache*>(p.private_rows) + (chain ? 0u : (size_t)row * p.row_elements);
    for (uint32_t i = tid; i < p.row_elements; i += kThreads) {
        query[i] = (float)static_cast<const Cache*>(p.q)[(size_t)m * p.row_elements + i];
        out[i] = 0.0f;
    }
    __syncthreads();
    float top = -INFINITY, sum = 0.0f;
    const uint32_t tiles = (end + kKeys - 1u) / kKeys;
    const uint32_t tile_begin = (uint32_t)((uint64_t)tiles * part / p.parts), tile_end = (uint32_t)((uint64_t)tiles * (part + 1u) / p.parts);
    auto cache_row = [&](uint32_t position) { return position < base ? ring + (size_t)(position & p.ring_mask) * p.row_elements : own + (size_t)(position - base) * p.row_elements; };
    for (uint32_t tile = tile_begin; tile < tile_end; ++tile) {
        const uint32_t keys = min(kKeys, end - tile * kKeys);
        for (uint32_t key = warp; key < keys; key += kThreads / 32u) {
            const Cache* c = cache_row(tile * kKeys + key);
            float s = 0.0f;
            for (uint32_t i = lane; i < p.row_elements; i += 32u) s = fmaf(query[i], (float)c[i], s);
            s = warp_sum(s);
            if (lane == 0) scores[key] = s;
        }
        __syncthreads();
        float now = top;
        for (uint32_t key = 0; key < keys; ++key) now = fmaxf(now, scores[key]);
        const float factor = top == -INFINITY ? 0.0f : expf(top - now);
        sum *= factor;
        __syncthreads();
        if (tid < keys) scores[tid] = expf(scores[tid] - now);
        __syncthreads();
        for (uint32_t key = 0; key < keys; ++key) sum += scores[key];
        for (uint32_t i = tid; i < p.row_elements; i += kThreads) {
            float v = out[i] * factor;
            for (uint32_t key = 0; key < keys; ++key) v = fmaf(scores[key], (float)cache_row(tile * kKeys + key)[i], v);
            out[i] = v;
        }
        top = now;
        __syncthreads();
    }
    if (p.result.data) {
        const float most = p.sink ? fmaxf(top, p.sink[head]) : top;
        const float factor = expf(top - most) / (sum * expf(top - most) + (p.sink ? expf(p.sink[head] - most) : 0.0f));
        for (uint32_t i = tid; i < p.row_elements; i += kThreads) store_operand(p.result, row, head * p.result_stride + i, out[i] * factor);
        return;
    }
    if (tid == 0) *reinterpret_cast<float2*>(p.partial_ml + ((size_t)m * p.parts + part) * 2u) = make_float2(top, sum);
    for (uint32_t i = tid; i < p.row_elements; i += kThreads) p.partial_out[((size_t)m * p.parts + part) * p.row_elements + i] = out[i];
}

__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttention p) {
    __shared__ float factors[kLatentMaxParts];
    const uint32_t m = blockIdx.x, row = m / p.heads, head = m % p.heads;
    if (threadIdx.x < 32u) merge_factors(p.partial_ml + (size_t)m * p.parts * 2u, p.parts, p.sink ? p.sink[head] : -INFINITY, factors);
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < p.row_elements; i += blockDim.x) {
        float v = 0.0f;
#pragma unroll 8
        for (uint32_t part = 0; part < p.parts; ++part) v = fmaf(p.partial_out[((size_t)m * p.parts + part) * p.row_elements + i], factors[part], v);
        store_operand(p.result, row, head * p.result_stride + i, v);
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

template <int MT, int NP>
int launch_tensor(const LatentAttention& p, cudaStream_t stream, bool pdl) {
    constexpr uint32_t kQueries = 16u * MT;
    static std::once_flag once[64];
    const int status = allow_smem(latent_attention_kernel<MT, NP>, once, kSmemLimit);
    if (status != GF_OK) return status;
    const bool chain = p.ring_stride == 0u;
    const uint32_t queries = chain ? p.rows * p.heads : p.heads;
    return launch_kernel(latent_attention_kernel<MT, NP>, dim3((queries + kQueries - 1u) / kQueries, p.parts, chain ? 1u : p.rows), dim3(kThreads),
                         latent_smem<MT>(p.row_elements).bytes, stream, pdl, p);
}

}  // namespace

bool latent_attention_on_tensor_cores(const LatentAttention& p) { return !p.cache_f32 && p.row_elements <= 512u; }

uint32_t latent_attention_parts(uint32_t rows, uint32_t heads, uint32_t positions, bool chain) {
    const uint32_t queries = chain ? rows * heads : heads, wide = queries > 16u ? 64u : 16u;
    const uint32_t blocks = (queries + wide - 1u) / wide * (chain ? 1u : rows);
    const uint32_t keys = wide > 16u ? kKeys : kNarrowKeys, tiles = (positions + keys - 1u) / keys;
    // Every partition is read again by the merge: more than 64 only where each has several tiles.
    const uint32_t most = std::min(kLatentMaxParts, std::max(64u, tiles / 4u));
    return std::max(1u, std::min(std::min(tiles, most), (uint32_t)sm_count() / std::max(1u, blocks)));
}

int launch_latent_attention(LatentAttention p, cudaStream_t stream, bool pdl) {
    if (!p.q || !p.rings || !p.private_rows || !p.positions || p.rows == 0 || p.heads == 0 || p.row_elements == 0 || p.row_elements % 16u
        || p.parts == 0 || p.parts > kLatentMaxParts || (p.result.data ? p.parts != 1u : (!p.partial_out || !p.partial_ml)))
        return fail(GF_ERR_INVALID, "latent attention: bad arguments");
    if (latent_attention_on_tensor_cores(p)) {
        const bool narrow = (p.ring_stride == 0u ? p.rows * p.heads : p.heads) <= 16u;
        const uint32_t groups = (p.row_elements + 127u) / 128u;
        if (narrow) return groups == 1u ? launch_tensor<1, 1>(p, stream, pdl) : groups == 2u ? launch_tensor<1, 2>(p, stream, pdl) : launch_tensor<1, 4>(p, stream, pdl);
        return groups == 1u ? launch_tensor<4, 1>(p, stream, pdl) : groups == 2u ? launch_tensor<4, 2>(p, stream, pdl) : launch_tensor<4, 4>(p, stream, pdl);
    }
    const uint32_t smem = p.row_elements * 8u;
    if (smem > 200u * 1024u) return fail(GF_ERR_INVALID, "latent attention: a latent of %u elements is too wide", p.row_elements);
    const dim3 grid(p.rows * p.heads, p.parts);
    static std::once_flag once32[64], once16[64];
    if (p.cache_f32) {
        const int status = allow_smem(latent_attention_plain_kernel<float>, once32, 200u * 1024u);
        if (status != GF_OK) return status;
        return launch_kernel(latent_attention_plain_kernel<float>, grid, dim3(kThreads), smem, stream, pdl, p);
    }
    const int status = allow_smem(latent_attention_plain_kernel<__half>, once16, 200u * 1024u);
    if (status != GF_OK) return status;
    return launch_kernel(latent_attention_plain_kernel<__half>, grid, dim3(kThreads), smem, stream, pdl, p);
}

int launch_latent_merge(const LatentAttention& p, cudaStream_t stream) {
    if (!p.result.data || !p.partial_out || !p.partial_ml || p.parts == 0 || p.parts > kLatentMaxParts) return fail(GF_ERR_INVALID, "latent merge: bad arguments");
    latent_merge_kernel<<<p.rows * p.heads, 128, 0, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

}  // namespace gf
