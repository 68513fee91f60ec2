// Grouped-query attention of passes and of 32-bit chunks (see grouped.cuh; 16-bit chunks run head_attention.cu).
#include "grouped.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

namespace {

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
__device__ __forceinline__ uint32_t half_pair(float lo, float hi) {
    const __half2 h = __floats2half2_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}

// ------------------------------------------------------------------ queries and cache rows

constexpr uint32_t kPrepareThreads = 256;

// Cosine and sine of a position's angle in pair i.
__device__ __forceinline__ float2 rotation(const QueryKey& p, uint32_t position, uint32_t i) {
    const uint32_t half = p.rotated / 2u;
    const float2 a = p.turns[(size_t)(position % kTurnSpan) * half + i], b = p.spans[(size_t)(position / kTurnSpan) * half + i];
    return make_float2(a.x * b.x - a.y * b.y, a.y * b.x + a.x * b.y);
}

// Dimension d of a head that starts at `first` of a projected row: normalised, turned.
__device__ __forceinline__ float turned(const QueryKey& p, const float* x, const float* gain, float inv, const float2* turn, uint32_t first, uint32_t d) {
    const float here = x[first + d] * inv * gain[first + d];
    if (d >= p.rotated) return here;
    const uint32_t half = p.rotated / 2u, i = d < half ? d : d - half, other = first + (d < half ? d + half : i);
    const float there = x[other] * inv * gain[other];
    return d < half ? here * turn[i].x - there * turn[i].y : here * turn[i].x + there * turn[i].y;
}
__device__ __forceinline__ __half cache_half(const QueryKey& p, float value) {
    const __half h = __float2half_rn(value);
    if (__hisinf(h) || __hisnan(h)) atomicOr(p.status, kStatusKvNonFinite);
    return h;
}
__device__ __forceinline__ void store_cache(const QueryKey& p, void* to, size_t at, float value) {
    if (p.f32) static_cast<float*>(to)[at] = value;
    else static_cast<__half*>(to)[at] = cache_half(p, value);
}

__global__ void __launch_bounds__(kPrepareThreads) query_key_kernel(const __grid_constant__ QueryKey p) {
    extern __shared__ float2 turn[];                                   // [rotated / 2]
    __shared__ float sums[kPrepareThreads / 32u][2];
    const uint32_t row = blockIdx.x, tid = threadIdx.x, half = p.rotated / 2u;
    const uint32_t q_width = p.heads * p.dim, k_width = p.kv_heads * p.dim;
    const uint32_t position = p.chain ? p.positions[0] + row : p.positions[row];
    for (uint32_t i = tid; i < half; i += kPrepareThreads) turn[i] = rotation(p, position, i);
    pdl_wait();
    pdl_launch_dependents();
    const float *q = p.raw_q ? p.raw_q + (size_t)row * p.q_ld : nullptr, *k = p.raw_k + (size_t)row * p.k_ld, *v = p.raw_v + (size_t)row * p.v_ld;
    float q_sum = 0.0f, k_sum = 0.0f;
    if (q)
#pragma unroll 4
        for (uint32_t i = tid; i < q_width; i += kPrepareThreads) q_sum = fmaf(q[i], q[i], q_sum);
#pragma unroll 4
    for (uint32_t i = tid; i < k_width; i += kPrepareThreads) k_sum = fmaf(k[i], k[i], k_sum);
    q_sum = warp_sum(q_sum);
    k_sum = warp_sum(k_sum);
    if ((tid & 31u) == 0u) { sums[tid >> 5][0] = q_sum; sums[tid >> 5][1] = k_sum; }
    __syncthreads();
    q_sum = k_sum = 0.0f;
    for (uint32_t w = 0; w < kPrepareThreads / 32u; ++w) { q_sum += sums[w][0]; k_sum += sums[w][1]; }
    const float q_inv = 1.0f / sqrtf(q_sum / (float)q_width + p.eps), k_inv = 1.0f / sqrtf(k_sum / (float)k_width + p.eps);
    // Dimensions d and d + 1 of a head that starts at `first`.
    auto turned2 = [&](const float* x, const float* gain, float inv, uint32_t first, uint32_t d) {
        const float2 v = *reinterpret_cast<const float2*>(x + first + d), w = *reinterpret_cast<const float2*>(gain + first + d);
        const float2 here = make_float2(v.x * inv * w.x, v.y * inv * w.y);
        if (d >= p.rotated) return here;
        const bool lower = d < half;
        const uint32_t i = lower ? d : d - half, other = first + (lower ? d + half : i);
        const float2 ov = *reinterpret_cast<const float2*>(x + other), ow = *reinterpret_cast<const float2*>(gain + other);
        const float2 there = make_float2(ov.x * inv * ow.x, ov.y * inv * ow.y), a = turn[i], c = turn[i + 1u];
        return lower ? make_float2(here.x * a.x - there.x * a.y, here.y * c.x - there.y * c.y) : make_float2(here.x * a.x + there.x * a.y, here.y * c.x + there.y * c.y);
    };
    if (!p.f32 && p.pairs) {
        auto store2 = [&](void* to, size_t at, float2 v) {
            const __half2 h = __floats2half2_rn(v.x, v.y);
            if (__hisinf(h.x) || __hisnan(h.x) || __hisinf(h.y) || __hisnan(h.y)) atomicOr(p.status, kStatusKvNonFinite);
            *reinterpret_cast<__half2*>(static_cast<__half*>(to) + at) = h;
        };
        const float2 zero = make_float2(0.0f, 0.0f);
        if (q)
#pragma unroll 4
            for (uint32_t i = tid * 2u; i < p.heads * p.row_head; i += kPrepareThreads * 2u) {
                const uint32_t head = i / p.row_head, d = i % p.row_head;
                float2 v = d < p.dim ? turned2(q, p.q_gain, q_inv, head * p.dim, d) : zero;
                store2(p.q, (size_t)row * p.heads * p.row_head + i, make_float2(v.x * p.scale, v.y * p.scale));
            }
        for (uint32_t i = tid * 2u; i < p.kv_heads * p.row_head; i += kPrepareThreads * 2u) {
            const uint32_t head = i / p.row_head, d = i % p.row_head;
            const size_t at = (size_t)row * p.kv_heads * p.row_head + i;
            store2(p.keys, at, d < p.dim ? turned2(k, p.k_gain, k_inv, head * p.dim, d) : zero);
            store2(p.values, at, d < p.vdim ? *reinterpret_cast<const float2*>(v + head * p.vdim + d) : zero);
        }
        return;
    }
    if (q)
        for (uint32_t i = tid; i < p.heads * p.row_head; i += kPrepareThreads) {
            const uint32_t head = i / p.row_head, d = i % p.row_head;
            store_cache(p, p.q, (size_t)row * p.heads * p.row_head + i, d < p.dim ? turned(p, q, p.q_gain, q_inv, turn, head * p.dim, d) * p.scale : 0.0f);
        }
    for (uint32_t i = tid; i < p.kv_heads * p.row_head; i += kPrepareThreads) {
        const uint32_t head = i / p.row_head, d = i % p.row_head;
        const size_t at = (size_t)row * p.kv_heads * p.row_head + i;
        store_cache(p, p.keys, at, d < p.dim ? turned(p, k, p.k_gain, k_inv, turn, head * p.dim, d) : 0.0f);
        store_cache(p, p.values, at, d < p.vdim ? v[head * p.vdim + d] : 0.0f);
    }
}

// ------------------------------------------------------------------ attention

// What a group of blocks shares: whether this block is the last of them to arrive.  All threads; the partial results
// are visible to the last block.
__device__ __forceinline__ bool last_to_arrive(uint32_t* counter, uint32_t parts) {
    __shared__ uint32_t last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        last = atomicAdd(counter, 1u) + 1u == parts ? 1u : 0u;
        if (last) *counter = 0u;
    }
    __syncthreads();
    if (last) __threadfence();
    return last != 0u;
}

__device__ __forceinline__ float head_gate(const GroupedAttention& p, uint32_t row, uint32_t head) {
    return p.gate ? sigmoid(p.gate[(size_t)row * p.heads + head]) : 1.0f;
}

// A warp merges the partitions of (row, head) into the result; `factors` is its scratch of kGroupedMaxParts * 3 floats.
__device__ __forceinline__ void merge_query(const GroupedAttention& p, uint32_t row, uint32_t head, float* factors) {
    const uint32_t lane = threadIdx.x & 31u;
    const size_t query = (size_t)row * p.heads + head;
    float* pairs = factors + kGroupedMaxParts;
    for (uint32_t i = lane; i < p.parts * 2u; i += 32u) pairs[i] = __ldcg(p.partial_ml + query * p.parts * 2u + i);
    __syncwarp();
    merge_factors(pairs, p.parts, p.sink ? p.sink[head] : -INFINITY, factors);
    __syncwarp();
    const float gate = head_gate(p, row, head);
#pragma unroll 1
    for (uint32_t d = lane * 4u; d < p.vdim; d += 128u) {              // a row's head is whole 16-byte pieces
        const float4* from = reinterpret_cast<const float4*>(p.partial_out + query * p.parts * p.row_head + d);
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 1
        for (uint32_t first = 0; first < p.parts; first += 16u) {
            float4 x[16];
#pragma unroll
            for (uint32_t i = 0; i < 16u; ++i) x[i] = first + i < p.parts ? __ldcg(from + (first + i) * (p.row_head / 4u)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (uint32_t i = 0; i < 16u; ++i) {
                const float f = first + i < p.parts ? factors[first + i] : 0.0f;
                v = make_float4(fmaf(x[i].x, f, v.x), fmaf(x[i].y, f, v.y), fmaf(x[i].z, f, v.z), fmaf(x[i].w, f, v.w));
            }
        }
        const float four[4] = {v.x * gate, v.y * gate, v.z * gate, v.w * gate};
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j)
            if (d + j < p.vdim) store_operand(p.result, row, head * p.vdim + d + j, four[j]);
    }
    __syncwarp();
}

// The prologue of a fused pass: the block's queries and the pass's own keys and values of key/value head `kv`, prepared
// from the projections.  Rows [first_row, first_row + query_rows) have queries here; with `own` all of `rows` leave their
// cache rows in own_k and own_v, and with `publish` in the private rows too.  Loops stay rolled: every block runs this
// once, and instructions have to be fetched as well.
struct FusedRows { uint32_t first_row, query_rows, rows, row0; bool own, publish; };
template <int kThreads>
__device__ __forceinline__ void prepare_fused(const GroupedAttention& p, const FusedRows& f, const float2* turns, uint32_t kv, uint32_t first_query, uint32_t queries,
                                              __half* q_tile, __half* own_k, __half* own_v, uint32_t stride) {
    constexpr uint32_t kWarps = kThreads / 32u, kItems = 16u + kGroupedFusedRows;
    __shared__ float sums[kItems][kWarps], factors[kItems];
    const QueryKey& in = p.prepare;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, group = p.heads / p.kv_heads, half = in.rotated / 2u, couples = p.row_head / 2u;
    const uint32_t q_width = in.heads * in.dim, k_width = in.kv_heads * in.dim, items = f.query_rows + (f.own ? f.rows : 0u);
#pragma unroll 1
    for (uint32_t item = 0; item < items; ++item) {
        const bool query = item < f.query_rows;
        const uint32_t row = f.row0 + (query ? f.first_row + item : item - f.query_rows), width = query ? q_width : k_width;
        const float* x = query ? in.raw_q + (size_t)row * in.q_ld : in.raw_k + (size_t)row * in.k_ld;
        float sum = 0.0f;
        if ((width | in.q_ld | in.k_ld) % 4u == 0u) {
#pragma unroll 1
            for (uint32_t i = tid * 4u; i < width; i += kThreads * 16u) {
                float4 v[4];
#pragma unroll
                for (uint32_t j = 0; j < 4u; ++j)
                    v[j] = i + j * kThreads * 4u < width ? *reinterpret_cast<const float4*>(x + i + j * kThreads * 4u) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                for (uint32_t j = 0; j < 4u; ++j) sum = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, sum))));
            }
        } else {
#pragma unroll 4
            for (uint32_t i = tid; i < width; i += kThreads) sum = fmaf(x[i], x[i], sum);
        }
        sum = warp_sum(sum);
        if (lane == 0) sums[item][warp] = sum;
    }
    __syncthreads();
    if (tid < items) {
        float sum = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < kWarps; ++w) sum += sums[tid][w];
        factors[tid] = 1.0f / sqrtf(sum / (float)(tid < f.query_rows ? q_width : k_width) + in.eps);
    }
    __syncthreads();
    // Couples of dimensions: those that turn together, then neighbours.
    const uint32_t tile_queries = min(16u, queries - first_query), lines = tile_queries + (f.own ? f.rows : 0u);
#pragma unroll 2
    for (uint32_t i = tid; i < lines * couples; i += kThreads) {
        const uint32_t line = i / couples, j = i % couples;
        const bool query = line < tile_queries;
        const uint32_t r = query ? (first_query + line) / group : line - tile_queries;
        const uint32_t first = (query ? kv * group + (first_query + line) % group : kv) * in.dim;
        const uint32_t d0 = j < half ? j : 2u * j, d1 = j < half ? j + half : 2u * j + 1u;       // 2 j = rotated + 2 (j - half)
        const float* x = (query ? in.raw_q + (size_t)(f.row0 + r) * in.q_ld : in.raw_k + (size_t)(f.row0 + r) * in.k_ld) + first;
        const float* gain = (query ? in.q_gain : in.k_gain) + first;
        const float inv = factors[query ? r - f.first_row : f.query_rows + r];
        float u = d0 < in.dim ? x[d0] * inv * gain[d0] : 0.0f, v = d1 < in.dim ? x[d1] * inv * gain[d1] : 0.0f;
        if (j < half) {
            const float2 turn = turns[r * half + j];
            const float turned_u = u * turn.x - v * turn.y;
            v = v * turn.x + u * turn.y;
            u = turned_u;
        }
        const float scale = query ? in.scale : 1.0f;
        const __half hu = cache_half(in, u * scale), hv = cache_half(in, v * scale);
        __half* to = query ? q_tile + line * stride : own_k + r * stride;
        to[d0] = hu;
        to[d1] = hv;
        if (!query && f.publish) {
            __half* row = static_cast<__half*>(in.keys) + ((size_t)(f.row0 + r) * p.kv_heads + kv) * p.row_head;
            row[d0] = hu;
            row[d1] = hv;
        }
    }
    if (!f.own) return;
#pragma unroll 1
    for (uint32_t i = tid; i < f.rows * p.row_head; i += kThreads) {
        const uint32_t r = i / p.row_head, d = i % p.row_head;
        const __half value = cache_half(in, d < in.vdim ? in.raw_v[(size_t)(f.row0 + r) * in.v_ld + kv * in.vdim + d] : 0.0f);
        own_v[r * stride + d] = value;
        if (f.publish) static_cast<__half*>(in.values)[((size_t)(f.row0 + r) * p.kv_heads + kv) * p.row_head + d] = value;
    }
}

constexpr uint32_t kRowsTile = 16;
template <int G> constexpr uint32_t rows_warps() { return G <= 8 ? 8u : 4u; }      // as many as have room for two tiles each

// A block serves sixteen queries of one key/value head -- (row, head of the group) pairs, heads fastest -- against one
// partition of the keys; its warps take tiles of keys in turn, the next one copied while this one is used, and keep
// scores, weights and outputs in registers.  G = groups of sixteen dimensions a head has at most.
template <int G>
__global__ void __launch_bounds__(rows_warps<G>() * 32) grouped_attention_kernel(const __grid_constant__ GroupedAttention p) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr uint32_t kWarps = rows_warps<G>();
    __shared__ float warp_top[kWarps][16], warp_sum_of[kWarps][16], scratch[kWarps][kGroupedMaxParts * 3u];
    constexpr uint32_t kTile = kRowsTile;
    const uint32_t stride = p.row_head + 8u, pieces = p.row_head / 8u;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, g = lane >> 2, t = lane & 3u;
    __half* q_tile = reinterpret_cast<__half*>(smem);
    __half* tiles = q_tile + 16u * stride;                             // [warps][2][keys, values][kTile][stride]
    __half* mine = tiles + (size_t)warp * 4u * kTile * stride;
    __half* own_rows = tiles + (size_t)kWarps * 4u * kTile * stride;           // fused: [keys, values][rows][stride], then the turns
    const bool chain = p.ring_stride == 0u;
    const uint32_t kv = blockIdx.z % p.kv_heads, z = blockIdx.z / p.kv_heads, part = blockIdx.y;
    const uint32_t group = p.heads / p.kv_heads, queries = (chain ? p.rows : 1u) * group, first_query = blockIdx.x * 16u;
    const uint32_t base = p.positions[z], cache_row = p.kv_heads * p.row_head;
    const StreamRings rings = p.rings[(size_t)z * p.ring_stride];
    const uint32_t end = base + min(first_query + 15u, queries - 1u) / group + 1u;      // keys the block's last query sees
    const uint32_t all = (end + kTile - 1u) / kTile;
    constexpr uint32_t step = kWarps;
    const uint32_t tile_begin = (uint32_t)((uint64_t)all * part / p.parts), tile_end = (uint32_t)((uint64_t)all * (part + 1u) / p.parts);
    const __half *ring_k = static_cast<const __half*>(rings.ring_k) + kv * p.row_head, *ring_v = static_cast<const __half*>(rings.ring_v) + kv * p.row_head;
    const size_t own_at = (size_t)(chain ? 0u : z) * cache_row + kv * p.row_head;
    const __half *own_k = static_cast<const __half*>(p.own_k) + own_at, *own_v = static_cast<const __half*>(p.own_v) + own_at;

    const uint32_t copied = p.fused ? base : end;                      // a fused pass has its own rows in shared memory
    auto load_tile = [&](uint32_t tile, uint32_t slot) {
        __half *kd = mine + slot * 2u * kTile * stride, *vd = kd + kTile * stride;
#pragma unroll
        for (uint32_t r0 = 0; r0 < kTile; r0 += 4u) {                  // four rows at a time, eight lanes each
            const uint32_t r = r0 + (lane >> 3), position = tile * kTile + r;
            const bool valid = position < copied, cached = position < base;
            const size_t at = valid ? (size_t)(cached ? position & p.ring_mask : position - base) * cache_row : 0u;
            const __half *ks = (cached ? ring_k : own_k) + at, *vs = (cached ? ring_v : own_v) + at;
            for (uint32_t piece = lane & 7u; piece < pieces; piece += 8u) {
                copy16(kd + r * stride + piece * 8u, ks + piece * 8u, valid);
                copy16(vd + r * stride + piece * 8u, vs + piece * 8u, valid);
            }
        }
    };
    const uint32_t rows = chain ? p.rows : 1u;
    __half *my_k = own_rows, *my_v = own_rows + rows * stride;
    if (p.fused) {
        // Cached rows and positions were written at least two launches back: read ahead of the wait.
        if (tile_begin + warp < tile_end) load_tile(tile_begin + warp, 0u);
        copies_commit();
        float2* turns = reinterpret_cast<float2*>(own_rows + 2u * rows * stride);
        const uint32_t half = p.prepare.rotated / 2u;
        for (uint32_t i = tid; i < rows * half; i += kWarps * 32u) turns[i] = rotation(p.prepare, base + i / half, i % half);
        const uint32_t last_query = min(first_query + 15u, queries - 1u);
        FusedRows f;
        f.first_row = first_query / group; f.query_rows = last_query / group - f.first_row + 1u; f.rows = rows; f.row0 = chain ? 0u : z;
        f.publish = part + 1u == p.parts && blockIdx.x + 1u == gridDim.x;
        f.own = tile_end * kTile > base;
        pdl_wait();
        pdl_launch_dependents();
        prepare_fused<kWarps * 32>(p, f, turns, kv, first_query, queries, q_tile, my_k, my_v, stride);
    } else {
        pdl_wait();
        pdl_launch_dependents();
        if (tile_begin + warp < tile_end) load_tile(tile_begin + warp, 0u);
        copies_commit();
        const __half* q = static_cast<const __half*>(p.q);
        for (uint32_t m = tid >> 3; m < 16u; m += kWarps * 4u) {
            const uint32_t query = first_query + m;
            const bool valid = query < queries;
            const size_t row = chain ? query / group : z;
            const __half* src = q + (valid ? (row * p.heads + kv * group + query % group) * p.row_head : 0u);
            for (uint32_t piece = tid & 7u; piece < pieces; piece += 8u)
                *reinterpret_cast<uint4*>(q_tile + m * stride + piece * 8u) = valid ? *reinterpret_cast<const uint4*>(src + piece * 8u) : make_uint4(0u, 0u, 0u, 0u);
        }
    }
    __syncthreads();
    float acc[2 * G][4];
#pragma unroll
    for (int i = 0; i < 2 * G; ++i) { acc[i][0] = 0.0f; acc[i][1] = 0.0f; acc[i][2] = 0.0f; acc[i][3] = 0.0f; }
    float top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
    const uint32_t steps = p.row_head / 16u;
    const uint32_t sees[2] = {base + min(first_query + g, queries - 1u) / group, base + min(first_query + g + 8u, queries - 1u) / group};
    const __half* a_row = q_tile + (lane & 15u) * stride + (lane >> 4) * 8u;
    constexpr float kLog2e = 1.4426950408889634f;
    const float inverse_cap = p.softcap > 0.0f ? 1.0f / p.softcap : 0.0f;

    uint32_t slot = 0;
    for (uint32_t tile = tile_begin + warp; tile < tile_end; tile += step, slot ^= 1u) {
        if (tile + step < tile_end) load_tile(tile + step, slot ^ 1u);
        copies_commit();
        copies_wait<1>();
        __syncwarp();
        __half *k_tile = mine + slot * 2u * kTile * stride, *v_tile = k_tile + kTile * stride;
        if (p.fused && (tile + 1u) * kTile > base) {
            for (uint32_t r = max(base, tile * kTile); r < min(end, (tile + 1u) * kTile); ++r)
                for (uint32_t piece = lane; piece < pieces; piece += 32u) {
                    *reinterpret_cast<uint4*>(k_tile + (r - tile * kTile) * stride + piece * 8u) = *reinterpret_cast<const uint4*>(my_k + (r - base) * stride + piece * 8u);
                    *reinterpret_cast<uint4*>(v_tile + (r - tile * kTile) * stride + piece * 8u) = *reinterpret_cast<const uint4*>(my_v + (r - base) * stride + piece * 8u);
                }
            __syncwarp();
        }
        float s[kTile / 8u][4];
#pragma unroll
        for (uint32_t n = 0; n < kTile / 8u; ++n) { s[n][0] = 0.0f; s[n][1] = 0.0f; s[n][2] = 0.0f; s[n][3] = 0.0f; }
        const __half* b_row = k_tile + ((lane & 7u) + (lane >> 4) * 8u) * stride + ((lane >> 3) & 1u) * 8u;
#pragma unroll
        for (int k = 0; k < G; ++k) {
            if ((uint32_t)k >= steps) break;
            uint32_t a[4];
            ldmatrix4(a, a_row + k * 16u);
#pragma unroll
            for (uint32_t n = 0; n < kTile / 16u; ++n) {
                uint32_t b[4];
                ldmatrix4(b, b_row + n * 16u * stride + k * 16u);
                mma_f16(s[2 * n], a, b[0], b[1]);
                mma_f16(s[2 * n + 1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (uint32_t n = 0; n < kTile / 8u; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if (p.softcap > 0.0f) s[n][e] = soft_cap(s[n][e], p.softcap, inverse_cap);
                if (tile * kTile + 8u * n + 2u * t + (e & 1) > sees[e >> 1]) s[n][e] = -INFINITY;
            }
        uint32_t w[kTile / 16u][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float now = top[i];
#pragma unroll
            for (uint32_t n = 0; n < kTile / 8u; ++n) now = fmaxf(now, fmaxf(s[n][2 * i], s[n][2 * i + 1]));
            now = fmaxf(now, __shfl_xor_sync(0xffffffffu, now, 1));
            now = fmaxf(now, __shfl_xor_sync(0xffffffffu, now, 2));
            const float shift = now == -INFINITY ? 0.0f : now * kLog2e;
            const float correction = exp2f(fmaf(top[i], kLog2e, -shift));
            float total = 0.0f;
#pragma unroll
            for (uint32_t n = 0; n < kTile / 8u; ++n) {
                const float x = exp2f(fmaf(s[n][2 * i], kLog2e, -shift)), y = exp2f(fmaf(s[n][2 * i + 1], kLog2e, -shift));
                total += x + y;
                w[n >> 1][(n & 1) * 2 + i] = half_pair(x, y);
            }
            sum[i] = sum[i] * correction + total;
            top[i] = now;
#pragma unroll
            for (int o = 0; o < 2 * G; ++o) { acc[o][2 * i] *= correction; acc[o][2 * i + 1] *= correction; }
        }
        const __half* v_row = v_tile + (lane & 15u) * stride + (lane >> 4) * 8u;
#pragma unroll
        for (uint32_t k = 0; k < kTile / 16u; ++k)
#pragma unroll
            for (int d = 0; d < G; ++d) {
                if ((uint32_t)d >= steps) break;
                uint32_t b[4];
                ldmatrix4_transposed(b, v_row + k * 16u * stride + d * 16u);
                mma_f16(acc[2 * d], w[k], b[0], b[1]);
                mma_f16(acc[2 * d + 1], w[k], b[2], b[3]);
            }
        __syncwarp();                                                  // the tile's buffer is free again
    }
    copies_wait<0>();
    // ---- the warps' results meet in shared memory
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
        if (t == 0u) { warp_top[warp][g + 8 * i] = top[i]; warp_sum_of[warp][g + 8 * i] = sum[i]; }
    }
    __syncthreads();
    float* parked = reinterpret_cast<float*>(tiles);                   // [warps][16][row_head + 4]
    const uint32_t parked_ld = p.row_head + 4u;
#pragma unroll
    for (int o = 0; o < 2 * G; ++o) {
        if ((uint32_t)o * 8u >= p.row_head) break;
#pragma unroll
        for (int i = 0; i < 2; ++i)
            if (first_query + g + 8u * i < queries)
                *reinterpret_cast<float2*>(parked + (warp * 16u + g + 8u * i) * parked_ld + o * 8u + 2u * t) = make_float2(acc[o][2 * i], acc[o][2 * i + 1]);
    }
    __syncthreads();
#pragma unroll 1
    for (uint32_t m = warp; m < 16u; m += kWarps) {
        const uint32_t query = first_query + m;
        if (query >= queries) break;
        const uint32_t row = chain ? query / group : z, head = kv * group + query % group;
        float most = warp_top[0][m], factor[kWarps], total = 0.0f;
#pragma unroll
        for (uint32_t w = 1; w < kWarps; ++w) most = fmaxf(most, warp_top[w][m]);
#pragma unroll
        for (uint32_t w = 0; w < kWarps; ++w) {
            factor[w] = warp_top[w][m] == -INFINITY ? 0.0f : expf(warp_top[w][m] - most);
            total += factor[w] * warp_sum_of[w][m];
        }
        float scale = 1.0f;
        if (p.parts == 1u) {
            const float sink = p.sink ? p.sink[head] : -INFINITY, high = fmaxf(most, sink), shrink = expf(most - high);
            scale = shrink / (total * shrink + (p.sink ? expf(sink - high) : 0.0f)) * head_gate(p, row, head);
        } else if (lane == 0u) {
            *reinterpret_cast<float2*>(p.partial_ml + (((size_t)row * p.heads + head) * p.parts + part) * 2u) = make_float2(most, total);
        }
#pragma unroll 1
        for (uint32_t d = lane; d < p.vdim; d += 32u) {
            float v = 0.0f;
#pragma unroll
            for (uint32_t w = 0; w < kWarps; ++w) v = fmaf(parked[(w * 16u + m) * parked_ld + d], factor[w], v);
            if (p.parts == 1u) store_operand(p.result, row, head * p.vdim + d, v * scale);
            else p.partial_out[(((size_t)row * p.heads + head) * p.parts + part) * p.row_head + d] = v;
        }
    }
    if (p.parts == 1u || !last_to_arrive(p.counters + (size_t)blockIdx.z * gridDim.x + blockIdx.x, p.parts)) return;
#pragma unroll 1
    for (uint32_t m = warp; m < 16u; m += kWarps) {
        const uint32_t query = first_query + m;
        if (query >= queries) break;
        merge_query(p, chain ? query / group : z, kv * group + query % group, scratch[warp]);
    }
}

// Any shape, f32 arithmetic, f32 or binary16 cache: one block per (query, partition); warps take the keys of a tile in
// turn for the scores, threads the dimensions for the outputs (kept in shared memory).
constexpr uint32_t kPlainKeys = 64, kPlainThreads = 256;
template <typename Cache>
__global__ void __launch_bounds__(kPlainThreads) grouped_attention_plain_kernel(const __grid_constant__ GroupedAttention p) {
    extern __shared__ __align__(16) float plain[];                     // query, output: [row_head] each
    __shared__ float scores[kPlainKeys], scratch[kGroupedMaxParts * 3u];
    float *query = plain, *out = plain + p.row_head;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    pdl_wait();
    pdl_launch_dependents();
    const bool chain = p.ring_stride == 0u;
    const uint32_t m = blockIdx.x, row = m / p.heads, head = m % p.heads, kv = head / (p.heads / p.kv_heads), part = blockIdx.y;
    const uint32_t base = p.positions[chain ? 0u : row], end = chain ? base + row + 1u : base + 1u, cache_row = p.kv_heads * p.row_head;
    const StreamRings rings = p.rings[(size_t)row * p.ring_stride];
    const Cache *ring_k = static_cast<const Cache*>(rings.ring_k) + kv * p.row_head, *ring_v = static_cast<const Cache*>(rings.ring_v) + kv * p.row_head;
    const size_t own_at = (size_t)(chain ? 0u : row) * cache_row + kv * p.row_head;
    const Cache *own_k = static_cast<const Cache*>(p.own_k) + own_at, *own_v = static_cast<const Cache*>(p.own_v) + own_at;
    for (uint32_t i = tid; i < p.row_head; i += kPlainThreads) {
        query[i] = (float)static_cast<const Cache*>(p.q)[(size_t)m * p.row_head + i];
        out[i] = 0.0f;
    }
    __syncthreads();
    float top = -INFINITY, sum = 0.0f;
    const uint32_t tiles = (end + kPlainKeys - 1u) / kPlainKeys;
    const uint32_t tile_begin = (uint32_t)((uint64_t)tiles * part / p.parts), tile_end = (uint32_t)((uint64_t)tiles * (part + 1u) / p.parts);
    auto cached = [&](const Cache* ring, const Cache* own, uint32_t position) {
        return position < base ? ring + (size_t)(position & p.ring_mask) * cache_row : own + (size_t)(position - base) * cache_row;
    };
    for (uint32_t tile = tile_begin; tile < tile_end; ++tile) {
        const uint32_t keys = min(kPlainKeys, end - tile * kPlainKeys);
        for (uint32_t key = warp; key < keys; key += kPlainThreads / 32u) {
            const Cache* c = cached(ring_k, own_k, tile * kPlainKeys + key);
            float s = 0.0f;
            for (uint32_t i = lane; i < p.row_head; i += 32u) s = fmaf(query[i], (float)c[i], s);
            s = warp_sum(s);
            if (lane == 0) scores[key] = p.softcap > 0.0f ? soft_cap_exact(s, p.softcap) : s;
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
        for (uint32_t i = tid; i < p.vdim; i += kPlainThreads) {
            float v = out[i] * factor;
            for (uint32_t key = 0; key < keys; ++key) v = fmaf(scores[key], (float)cached(ring_v, own_v, tile * kPlainKeys + key)[i], v);
            out[i] = v;
        }
        top = now;
        __syncthreads();
    }
    if (p.parts == 1u) {
        const float sink = p.sink ? p.sink[head] : -INFINITY, most = fmaxf(top, sink), shrink = expf(top - most);
        const float factor = shrink / (sum * shrink + (p.sink ? expf(sink - most) : 0.0f)) * head_gate(p, row, head);
        for (uint32_t i = tid; i < p.vdim; i += kPlainThreads) store_operand(p.result, row, head * p.vdim + i, out[i] * factor);
        return;
    }
    if (tid == 0) *reinterpret_cast<float2*>(p.partial_ml + ((size_t)m * p.parts + part) * 2u) = make_float2(top, sum);
    for (uint32_t i = tid; i < p.vdim; i += kPlainThreads) p.partial_out[((size_t)m * p.parts + part) * p.row_head + i] = out[i];
    if (last_to_arrive(p.counters + m, p.parts) && warp == 0) merge_query(p, row, head, scratch);
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

template <int G>
int launch_rows(const GroupedAttention& p, cudaStream_t stream, bool pdl) {
    constexpr uint32_t kTile = kRowsTile;
    static std::once_flag once[64];
    const int status = allow_smem(grouped_attention_kernel<G>, once, 200u * 1024u);
    if (status != GF_OK) return status;
    const bool chain = p.ring_stride == 0u;
    const uint32_t rows = chain ? p.rows : 1u, queries = rows * (p.heads / p.kv_heads);
    const uint32_t smem = (16u + rows_warps<G>() * 4u * kTile + (p.fused ? 2u * rows : 0u)) * (p.row_head + 8u) * 2u + (p.fused ? rows * p.prepare.rotated * 4u : 0u);
    return launch_kernel(grouped_attention_kernel<G>, dim3((queries + 15u) / 16u, p.parts, p.kv_heads * (chain ? 1u : p.rows)), dim3(rows_warps<G>() * 32u), smem, stream, pdl, p);
}

}  // namespace

int launch_query_key(QueryKey p, cudaStream_t stream, bool pdl) {
    if (!p.raw_k || !p.raw_v || (p.raw_q && (!p.q_gain || !p.q)) || !p.k_gain || !p.positions || !p.keys || !p.values || p.rows == 0 || p.heads == 0 || p.kv_heads == 0
        || p.dim == 0 || p.vdim == 0 || p.row_head < p.dim || p.row_head < p.vdim || p.rotated > p.dim || p.rotated % 2u || (p.rotated && (!p.turns || !p.spans)))
        return fail(GF_ERR_INVALID, "query and key preparation: bad arguments");
    p.pairs = p.dim % 2u == 0u && p.vdim % 2u == 0u && p.rotated % 4u == 0u && p.q_ld % 2u == 0u && p.k_ld % 2u == 0u && p.v_ld % 2u == 0u ? 1u : 0u;
    return launch_kernel(query_key_kernel, dim3(p.rows), dim3(kPrepareThreads), p.rotated / 2u * sizeof(float2), stream, pdl, p);
}

uint32_t grouped_attention_parts(uint32_t rows, uint32_t heads, uint32_t kv_heads, uint32_t positions, bool chain) {
    const uint32_t queries = (chain ? rows : 1u) * (heads / kv_heads), blocks = (queries + 15u) / 16u * kv_heads * (chain ? 1u : rows);
    // Two tiles for every warp of a partition, and few partitions where they are short: the last block reads all of them.
    const uint32_t most = std::max(1u, std::min((positions + 127u) / 128u, std::max(16u, positions / 512u)));
    return std::max(1u, std::min({most, kGroupedMaxParts, (uint32_t)sm_count() / std::max(1u, blocks)}));
}

int launch_grouped_attention(const GroupedAttention& p, cudaStream_t stream, bool pdl) {
    if (p.fused ? (!grouped_attention_on_tensor_cores(p.row_head, p.f32 != 0u) || p.rows > kGroupedFusedRows || !p.prepare.raw_q || !p.prepare.raw_k || !p.prepare.raw_v
                   || !p.prepare.keys || !p.prepare.values || p.prepare.row_head != p.row_head || p.prepare.vdim != p.vdim || (p.prepare.rotated && (!p.prepare.turns || !p.prepare.spans)))
                : !p.q)
        return fail(GF_ERR_INVALID, "grouped attention: bad arguments");
    if (!p.rings || !p.own_k || !p.own_v || !p.positions || !p.result.data || p.rows == 0 || p.heads == 0 || p.kv_heads == 0 || p.heads % p.kv_heads
        || p.row_head == 0 || p.row_head % 16u || p.vdim > p.row_head || p.parts == 0 || p.parts > kGroupedMaxParts
        || (p.parts > 1u && (!p.partial_out || !p.partial_ml || !p.counters)))
        return fail(GF_ERR_INVALID, "grouped attention: bad arguments");
    if (grouped_attention_on_tensor_cores(p.row_head, p.f32 != 0u)) {
        const uint32_t groups = p.row_head / 16u;
        if (groups <= 2u) return launch_rows<2>(p, stream, pdl);
        if (groups <= 4u) return launch_rows<4>(p, stream, pdl);
        if (groups <= 8u) return launch_rows<8>(p, stream, pdl);
        return launch_rows<16>(p, stream, pdl);
    }
    const dim3 grid(p.rows * p.heads, p.parts);
    const uint32_t smem = p.row_head * 8u;
    if (p.f32) return launch_kernel(grouped_attention_plain_kernel<float>, grid, dim3(kPlainThreads), smem, stream, pdl, p);
    return launch_kernel(grouped_attention_plain_kernel<__half>, grid, dim3(kPlainThreads), smem, stream, pdl, p);
}

}  // namespace gf
