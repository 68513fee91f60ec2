// Packing of bf16 matrices, the embedding gather from them, and row products (see dense.cuh).
#include "dense.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

// ------------------------------------------------------------------ packing, embedding

__global__ void __launch_bounds__(256) dense_pack_kernel(const DensePack p) {
    const uint32_t pieces = p.k_blocks * 8u;
    const uint64_t total = (uint64_t)p.count * p.n * pieces;
    for (uint64_t i = blockIdx.x * (uint64_t)blockDim.x + threadIdx.x; i < total; i += (uint64_t)gridDim.x * blockDim.x) {
        const uint32_t piece = (uint32_t)(i % pieces), n = (uint32_t)(i / pieces % p.n), matrix = (uint32_t)(i / pieces / p.n);
        const uint16_t* src = p.src + matrix * p.count_stride + n * p.n_stride;
        uint16_t v[8];
#pragma unroll
        for (uint32_t j = 0; j < 8u; ++j) {
            const uint32_t k = piece * 8u + j;
            v[j] = k < p.k ? src[k * p.k_stride] : (uint16_t)0;
        }
        const uint32_t column = ((n / 8u) * p.group_step + p.group_first) * 8u + n % 8u;
        *reinterpret_cast<uint4*>(p.dst + matrix * p.dst_stride + dense_offset(p.k_blocks, column, piece * 8u)) =
            make_uint4(v[0] | (uint32_t)v[1] << 16, v[2] | (uint32_t)v[3] << 16, v[4] | (uint32_t)v[5] << 16, v[6] | (uint32_t)v[7] << 16);
    }
}

int launch_dense_pack(const DensePack& p, cudaStream_t stream) {
    if (!p.src || !p.dst || p.count == 0 || p.n == 0 || p.k == 0) return fail(GF_ERR_INVALID, "dense pack: bad arguments");
    const uint64_t total = (uint64_t)p.count * p.n * p.k_blocks * 8u;
    dense_pack_kernel<<<(uint32_t)std::min<uint64_t>((total + 255u) / 256u, 8192u), 256, 0, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

__global__ void __launch_bounds__(256) dense_embedding_kernel(const uint8_t* __restrict__ packed, uint32_t k_blocks, uint32_t width, uint32_t vocab,
                                                              const uint32_t* __restrict__ tokens, float scale, float* __restrict__ out, uint32_t* status) {
    pdl_wait();
    pdl_launch_dependents();
    const uint32_t row = blockIdx.x, token = tokens[row];
    for (uint32_t k = threadIdx.x; k < width; k += blockDim.x) {
        float v = __int_as_float(0x7fc00000);
        if (token < vocab) v = __uint_as_float((uint32_t)*reinterpret_cast<const uint16_t*>(packed + dense_offset(k_blocks, token, k)) << 16) * scale;
        out[(size_t)row * width + k] = v;
    }
    if (token >= vocab && threadIdx.x == 0) atomicOr(status, kStatusBadToken);
}

int launch_dense_embedding(const uint8_t* packed, uint32_t k_blocks, uint32_t width, uint32_t vocab, const uint32_t* tokens, uint32_t rows,
                           float scale, float* out, uint32_t* status, cudaStream_t stream, bool pdl) {
    return launch_kernel(dense_embedding_kernel, dim3(rows), dim3(256), 0, stream, pdl, packed, k_blocks, width, vocab, tokens, scale, out, status);
}

// ------------------------------------------------------------------ row products

namespace {

constexpr uint32_t kRowThreads = 256, kRowWarps = kRowThreads / 32u;
constexpr uint32_t kRowAhead = 8;                    // 512-byte loads a warp keeps in flight
constexpr uint32_t kRowSmemLimit = 200u * 1024u;     // activations of a launch
constexpr uint32_t kRowMaxRows = 8;
constexpr uint32_t kNormQuads = 4;                   // 16-byte pieces of a row a thread holds: rows of up to 4096 values

__device__ __forceinline__ uint4 load_weight(const uint8_t* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ float low_half(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float high_half(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

// Sums over the block of `count` <= kRowMaxRows values per thread; every thread gets all of them.
template <int R>
__device__ __forceinline__ void block_sums(float (&v)[R], float* scratch) {
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const float s = warp_sum(v[r]);
        if (lane == 0) scratch[warp * R + r] = s;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < R; ++r) {
        v[r] = 0.0f;
        for (uint32_t w = 0; w < kRowWarps; ++w) v[r] += scratch[w * R + r];      // the same order in every thread
    }
    __syncthreads();
}

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float dot4(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }

__device__ __forceinline__ float norm_factor(float sum, uint32_t width, float eps) { return 1.0f / sqrtf(sum / (float)width + eps); }

// Cache row of one token: the latent's RMS norm.
__device__ void store_latent(const RowProduct& p, uint32_t row, float* scratch) {
    const float* raw = p.latent_raw + (size_t)row * p.latent_raw_ld;
    float sum[1] = {0.0f};
    for (uint32_t i = threadIdx.x; i < p.latent_rank; i += kRowThreads) sum[0] = fmaf(raw[i], raw[i], sum[0]);
    block_sums<1>(sum, scratch);
    const float inv = norm_factor(sum[0], p.latent_rank, p.eps);
    for (uint32_t i = threadIdx.x; i < p.latent_row_elements; i += kRowThreads) {
        const float v = i < p.latent_rank ? raw[i] * inv * p.latent_gain[i] : 0.0f;
        const size_t at = (size_t)row * p.latent_row_elements + i;
        if (p.latent_f16) {
            const __half h = __float2half_rn(v);
            if (__hisinf(h) || __hisnan(h)) atomicOr(p.status, kStatusKvNonFinite);
            static_cast<__half*>(p.latent_rows)[at] = h;
        } else static_cast<float*>(p.latent_rows)[at] = v;
    }
}

// One CTA: sets of `groups_per_cta` groups of eight output columns; the eight warps share a set, 8 / groups_per_cta
// of them splitting a group's K.  The first loads of the first set are in flight before the dependency wait.
template <int R>
__global__ void __launch_bounds__(kRowThreads) row_product_kernel(const __grid_constant__ RowProduct p) {
    extern __shared__ __align__(16) float act[];                   // [R][k_pad]
    __shared__ float partial[kRowWarps][R][8];
    __shared__ float scratch[kRowWarps * R];
    __shared__ float route_scratch[kMaxExperts];
    __shared__ uint32_t route_id;
    __shared__ float route_score;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, batch = blockIdx.y;
    if (batch >= p.batches) {                                      // the cache rows of this pass
        pdl_wait();
        pdl_launch_dependents();
        if (blockIdx.x < p.rows) store_latent(p, blockIdx.x, scratch);
        return;
    }
    const bool routed = p.input == kRowRouted || (p.input == kRowExperts && batch < p.rows * p.top);
    const bool behind = p.input == kRowExperts && !routed;         // the shared expert's batches use matrix 1
    const uint32_t first_matrix = behind ? 1u : 0u, end_matrix = p.input == kRowExperts ? first_matrix + 1u : p.count;
    const uint32_t set_base = p.m[first_matrix].first_set, set_end = p.m[end_matrix - 1u].first_set + p.m[end_matrix - 1u].sets;

    uint4 w[kRowAhead];
    uint32_t unit_begin = 0, unit_end = 0, group = 0, which = 0;
    const uint8_t* base = nullptr;
    auto locate = [&](uint32_t set) {
        which = first_matrix;
        while (which + 1u < end_matrix && set >= p.m[which + 1u].first_set) ++which;
        const RowMatrix& m = p.m[which];
        const uint32_t split = kRowWarps / m.groups_per_cta, units = (m.k + 31u) / 32u;
        group = (set - m.first_set) * m.groups_per_cta + warp / split;
        const uint32_t slice = warp % split;
        unit_begin = units * slice / split;
        unit_end = group * 8u < m.n ? units * (slice + 1u) / split : unit_begin;
        const uint32_t index = routed ? route_id : behind ? 0u : batch;
        base = m.weight + index * m.weight_batch + (size_t)(group / 16u) * m.k_blocks * kDenseTileBytes + (group % 16u) * 1024u + lane * 16u;
    };
    auto fetch = [&](uint32_t unit) { return load_weight(base + (size_t)(unit >> 1) * kDenseTileBytes + (unit & 1u) * 512u); };
    auto prefetch = [&]() {
#pragma unroll
        for (uint32_t i = 0; i < kRowAhead; ++i)
            if (unit_begin + i < unit_end) w[i] = fetch(unit_begin + i);
    };

    uint32_t set = set_base + blockIdx.x;
    if (set >= set_end) return;
    if (!routed) { locate(set); prefetch(); }
    const bool quads = p.vector_rows != 0u;                        // widths and strides are whole 16-byte pieces
    // The residual rows and the gains were written at least two launches back: read ahead of the wait.
    float4 early_residual[kNormQuads], early_gain0[kNormQuads], early_gain1[kNormQuads];
    const bool early = R == 1 && quads && (p.input == kRowNorm || p.input == kRowAddNorm) && p.width <= kNormQuads * kRowThreads * 4u;
    if (early)
#pragma unroll
        for (uint32_t j = 0; j < kNormQuads; ++j) {
            const uint32_t i = (j * kRowThreads + tid) * 4u;
            if (i >= p.width) continue;
            if (p.gain1) early_gain1[j] = *reinterpret_cast<const float4*>(p.gain1 + i);
            if (p.input == kRowAddNorm) {
                early_residual[j] = *reinterpret_cast<const float4*>(p.residual + i);
                early_gain0[j] = *reinterpret_cast<const float4*>(p.gain0 + i);
            }
        }
    pdl_wait();
    pdl_launch_dependents();

    // ---- the activations
    if (routed) {
        if (p.input == kRowRouted) {
            const uint32_t row = batch / p.top, slot = batch % p.top;
            if (warp == 0)
                route_row(p.router_logits + (size_t)row * p.experts, p.experts, slot + 1u, route_scratch, [&](uint32_t s, uint32_t e, float score) {
                    if (s != slot || lane != 0) return;
                    route_id = e;
                    route_score = score;
                    if (blockIdx.x == 0) { p.route_ids[batch] = e; p.route_scores[batch] = score; }
                });
        } else if (tid == 0) {
            route_id = p.route_ids[batch];
        }
        __syncthreads();
        locate(set);
        prefetch();
    }
    const uint32_t k_used = p.m[which].k, k_pad = p.k_pad;
    if (early) {
        // One row held in registers: both norms without a pass through shared memory in between.
        const bool writer = blockIdx.x == 0 && batch == 0;
        float4 v[kNormQuads];
        float sum[1] = {0.0f};
#pragma unroll
        for (uint32_t j = 0; j < kNormQuads; ++j) {
            const uint32_t i = (j * kRowThreads + tid) * 4u;
            v[j] = i < p.width ? *reinterpret_cast<const float4*>(p.in + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
#pragma unroll 4
        for (uint32_t part = 1; part < p.parts; ++part)
#pragma unroll
            for (uint32_t j = 0; j < kNormQuads; ++j) {
                const uint32_t i = (j * kRowThreads + tid) * 4u;
                if (i < p.width) v[j] = add4(v[j], *reinterpret_cast<const float4*>(p.in + part * p.part_stride + i));
            }
#pragma unroll
        for (uint32_t j = 0; j < kNormQuads; ++j) sum[0] += dot4(v[j], v[j]);
        block_sums<1>(sum, scratch);
        float inv = norm_factor(sum[0], p.width, p.eps);
        if (p.input == kRowAddNorm) {
            sum[0] = 0.0f;
#pragma unroll
            for (uint32_t j = 0; j < kNormQuads; ++j) {
                const uint32_t i = (j * kRowThreads + tid) * 4u;
                if (i >= p.width) continue;
                const float4 r = early_residual[j], g = early_gain0[j];
                v[j] = make_float4(r.x + v[j].x * inv * g.x, r.y + v[j].y * inv * g.y, r.z + v[j].z * inv * g.z, r.w + v[j].w * inv * g.w);
                if (writer && p.residual_out) *reinterpret_cast<float4*>(p.residual_out + i) = v[j];
                sum[0] += dot4(v[j], v[j]);
            }
            if (p.gain1) {
                block_sums<1>(sum, scratch);
                inv = norm_factor(sum[0], p.width, p.eps);
            }
        }
#pragma unroll
        for (uint32_t j = 0; j < kNormQuads; ++j) {
            const uint32_t i = (j * kRowThreads + tid) * 4u;
            if (i >= p.width) continue;
            float4 n = v[j];
            if (p.gain1) {
                const float4 g = early_gain1[j];
                n = make_float4(n.x * inv * g.x, n.y * inv * g.y, n.z * inv * g.z, n.w * inv * g.w);
            }
            *reinterpret_cast<float4*>(act + i) = n;
            if (writer && p.normed_out) *reinterpret_cast<float4*>(p.normed_out + i) = n;
        }
        for (uint32_t i = p.width + tid; i < k_pad; i += kRowThreads) act[i] = 0.0f;
    } else if (p.input == kRowNorm || p.input == kRowAddNorm) {
        const bool writer = blockIdx.x == 0 && batch == 0;
        float sum[R];
#pragma unroll
        for (int r = 0; r < R; ++r) sum[r] = 0.0f;
        for (uint32_t i = tid; i < p.width; i += kRowThreads)
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float* x = p.in + (size_t)r * p.in_ld + i;
                float v = *x;
                for (uint32_t part = 1; part < p.parts; ++part) v += x[part * p.part_stride];
                act[r * k_pad + i] = v;
                sum[r] = fmaf(v, v, sum[r]);
            }
        block_sums<R>(sum, scratch);
        if (p.input == kRowAddNorm) {
#pragma unroll
            for (int r = 0; r < R; ++r) { sum[r] = norm_factor(sum[r], p.width, p.eps); }
            float next[R];
#pragma unroll
            for (int r = 0; r < R; ++r) next[r] = 0.0f;
            for (uint32_t i = tid; i < p.width; i += kRowThreads) {
                const float gain = p.gain0[i];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const size_t at = (size_t)r * p.width + i;
                    const float v = p.residual[at] + act[r * k_pad + i] * sum[r] * gain;
                    act[r * k_pad + i] = v;
                    if (writer && p.residual_out) p.residual_out[at] = v;
                    next[r] = fmaf(v, v, next[r]);
                }
            }
            if (p.gain1) block_sums<R>(next, scratch);
#pragma unroll
            for (int r = 0; r < R; ++r) sum[r] = next[r];
        }
#pragma unroll
        for (int r = 0; r < R; ++r) sum[r] = p.gain1 ? norm_factor(sum[r], p.width, p.eps) : 1.0f;
        for (uint32_t i = tid; i < k_pad; i += kRowThreads) {
            const float gain = i >= p.width ? 0.0f : p.gain1 ? p.gain1[i] : 1.0f;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float v = i < p.width ? act[r * k_pad + i] * sum[r] * gain : 0.0f;
                act[r * k_pad + i] = v;
                if (writer && p.normed_out && i < p.width) p.normed_out[(size_t)r * p.width + i] = v;
            }
        }
    } else if (p.input == kRowPartNorm) {
        const uint32_t part = p.width / p.norm_parts;
        if (quads && part % 128u == 0u && p.norm_parts <= kRowThreads && p.width <= kMaxExperts * 128u) {
            // Sums of 128 values at a time, a warp's 16-byte pieces.
            for (int r = 0; r < R; ++r) {
                const float* x = p.in + (size_t)r * p.in_ld;
#pragma unroll 8
                for (uint32_t i = tid * 4u; i < p.width; i += kRowThreads * 4u) {
                    const float4 v = *reinterpret_cast<const float4*>(x + i);
                    *reinterpret_cast<float4*>(act + r * k_pad + i) = v;
                    const float sum = warp_sum(dot4(v, v));
                    if (lane == 0) route_scratch[i / 128u] = sum;
                }
                __syncthreads();
                float inv = 0.0f;
                if (tid < p.norm_parts) {
                    for (uint32_t s = 0; s < part / 128u; ++s) inv += route_scratch[tid * (part / 128u) + s];
                    inv = norm_factor(inv, part, p.eps);
                }
                __syncthreads();
                if (tid < p.norm_parts) route_scratch[tid] = inv;
                __syncthreads();
#pragma unroll 4
                for (uint32_t i = tid * 4u; i < p.width; i += kRowThreads * 4u) {
                    const float4 g = *reinterpret_cast<const float4*>(p.gain1 + i);
                    float4* at = reinterpret_cast<float4*>(act + r * k_pad + i);
                    const float f = route_scratch[i / part];
                    *at = make_float4(at->x * f * g.x, at->y * f * g.y, at->z * f * g.z, at->w * f * g.w);
                }
                for (uint32_t i = p.width + tid; i < k_pad; i += kRowThreads) act[r * k_pad + i] = 0.0f;
                __syncthreads();
            }
        } else {
            // Warps share the parts: several to a part where there are fewer parts than warps.
            uint32_t per = kRowWarps;
            while (per > 1u && per * p.norm_parts > kRowWarps) per /= 2u;
            for (int r = 0; r < R; ++r) {
                const float* x = p.in + (size_t)r * p.in_ld;
                for (uint32_t unit = warp; unit < per * p.norm_parts; unit += kRowWarps) {
                    const uint32_t first = unit / per * part;
                    float sum = 0.0f;
                    for (uint32_t i = (unit % per) * 32u + lane; i < part; i += per * 32u) {
                        const float v = x[first + i];
                        act[r * k_pad + first + i] = v;
                        sum = fmaf(v, v, sum);
                    }
                    sum = warp_sum(sum);
                    if (lane == 0) route_scratch[unit] = sum;
                }
                __syncthreads();
                for (uint32_t i = tid; i < k_pad; i += kRowThreads) {
                    float v = 0.0f;
                    if (i < p.width) {
                        float sum = 0.0f;
                        for (uint32_t s = 0; s < per; ++s) sum += route_scratch[i / part * per + s];
                        v = act[r * k_pad + i] * norm_factor(sum, part, p.eps) * p.gain1[i];
                    }
                    act[r * k_pad + i] = v;
                }
                __syncthreads();
            }
        }
    } else if (p.input == kRowLatent) {
        for (int r = 0; r < R; ++r) {
            const uint32_t m = r * p.heads + batch, parts = p.attention_parts;
            if (warp == 0) merge_factors(p.latent_ml + (size_t)m * parts * 2u, parts, p.sink ? p.sink[batch] : -INFINITY, route_scratch);
            __syncthreads();
            // Two halves of the block take the even and the odd partitions, a thread four dimensions at a time.
            const float* rows_in = p.in + (size_t)m * parts * p.latent_ld;
            const uint32_t odd = tid / (kRowThreads / 2u), first = (tid % (kRowThreads / 2u)) * 4u;
            for (uint32_t i0 = 0; i0 < k_pad; i0 += kRowThreads * 2u) {
                const uint32_t i = i0 + first;
                float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (i < p.latent_ld) {
#pragma unroll 8
                    for (uint32_t part = odd; part < parts; part += 2u) {
                        const float4 o = *reinterpret_cast<const float4*>(rows_in + (size_t)part * p.latent_ld + i);
                        const float f = route_scratch[part];
                        v.x = fmaf(o.x, f, v.x); v.y = fmaf(o.y, f, v.y); v.z = fmaf(o.z, f, v.z); v.w = fmaf(o.w, f, v.w);
                    }
                }
                float4* dst = reinterpret_cast<float4*>(act + r * k_pad + i);
                if (odd && i < k_pad) *dst = v;
                __syncthreads();
                if (!odd && i < k_pad) *dst = add4(*dst, v);
            }
            __syncthreads();
        }
    } else {
        for (int r = 0; r < R; ++r) {
            const float* x;
            if (p.input == kRowRouted) x = p.in + (size_t)(batch / p.top) * p.in_ld;
            else if (p.input == kRowExperts) x = behind ? p.in2 + (size_t)(batch - p.rows * p.top) * p.in2_ld : p.in + (size_t)batch * p.in_ld;
            else x = p.in + (size_t)(p.in_rows ? p.in_rows[r] : (uint32_t)r) * p.in_ld + (size_t)batch * p.in_batch;
            if (quads) {
#pragma unroll 4
                for (uint32_t i = tid * 4u; i < k_pad; i += kRowThreads * 4u)
                    *reinterpret_cast<float4*>(act + r * k_pad + i) = i < k_used ? *reinterpret_cast<const float4*>(x + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            } else {
                for (uint32_t i = tid; i < k_pad; i += kRowThreads) act[r * k_pad + i] = i < k_used ? x[i] : 0.0f;
            }
        }
    }
    __syncthreads();

    // ---- the products
    const float* lane_act = act + (lane >> 3) * 8u;
    for (; set < set_end; ) {
        float acc[R][2];
#pragma unroll
        for (int r = 0; r < R; ++r) { acc[r][0] = 0.0f; acc[r][1] = 0.0f; }
        auto consume = [&](const uint4& v, uint32_t unit) {
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float4 x = *reinterpret_cast<const float4*>(lane_act + r * k_pad + unit * 32u);
                const float4 y = *reinterpret_cast<const float4*>(lane_act + r * k_pad + unit * 32u + 4u);
                float a = acc[r][0], b = acc[r][1];
                a = fmaf(low_half(v.x), x.x, a); b = fmaf(high_half(v.x), x.y, b);
                a = fmaf(low_half(v.y), x.z, a); b = fmaf(high_half(v.y), x.w, b);
                a = fmaf(low_half(v.z), y.x, a); b = fmaf(high_half(v.z), y.y, b);
                a = fmaf(low_half(v.w), y.z, a); b = fmaf(high_half(v.w), y.w, b);
                acc[r][0] = a; acc[r][1] = b;
            }
        };
        uint32_t unit = unit_begin;
        for (; unit + 2u * kRowAhead <= unit_end; unit += kRowAhead)      // whole rounds with a whole round behind them
#pragma unroll
            for (uint32_t i = 0; i < kRowAhead; ++i) {
                consume(w[i], unit + i);
                w[i] = fetch(unit + kRowAhead + i);
            }
        for (; unit < unit_end; unit += kRowAhead)
#pragma unroll
            for (uint32_t i = 0; i < kRowAhead; ++i)
                if (unit + i < unit_end) {
                    consume(w[i], unit + i);
                    if (unit + kRowAhead + i < unit_end) w[i] = fetch(unit + kRowAhead + i);
                }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            float v = acc[r][0] + acc[r][1];
            v += __shfl_xor_sync(0xffffffffu, v, 8);
            v += __shfl_xor_sync(0xffffffffu, v, 16);
            if (lane < 8u) partial[warp][r][lane] = v;
        }
        const RowMatrix& m = p.m[which];
        const uint32_t here = set, split = kRowWarps / m.groups_per_cta;
        set += gridDim.x;
        if (set < set_end) { locate(set); prefetch(); }            // the next set's loads overlap the hand-over
        __syncthreads();
        // ---- K slices summed in order, then the output
        const bool paired = paired_output(m.output);
        const uint32_t outputs = m.groups_per_cta * 8u / (paired ? 2u : 1u);
        for (uint32_t i = tid; i < outputs * R; i += kRowThreads) {
            const uint32_t column = i % outputs, r = i / outputs;
            auto sum_group = [&](uint32_t g) {
                float v = 0.0f;
                for (uint32_t s = 0; s < split; ++s) v += partial[g * split + s][r][column & 7u];
                return v;
            };
            const uint32_t first_column = (here - m.first_set) * m.groups_per_cta * 8u;
            if (paired) {
                const uint32_t n = first_column / 2u + column;
                if (n >= m.n / 2u) continue;
                const float score = p.input == kRowRouted ? route_score : 1.0f;
                const uint32_t pair = column >> 3;
                const float gate = sum_group(2u * pair) * score, up = sum_group(2u * pair + 1u) * score;
                const float v = m.output == kOutGeluGate ? gelu_tanh(gate) * up : clamped_gate(gate, up, m.limit);
                static_cast<float*>(m.out)[(size_t)r * m.out_ld + (size_t)batch * m.out_batch + n] = v;
                continue;
            }
            const uint32_t n = first_column + column;
            if (n >= m.n) continue;
            float v = sum_group(column >> 3);
            if (m.output == kOutLatentQuery) {
                const size_t at = (size_t)(r * p.heads + batch) * m.out_ld + n;
                v *= p.scale;
                if (p.query_f16) {
                    const __half h = __float2half_rn(v);
                    if (__hisinf(h) || __hisnan(h)) atomicOr(p.status, kStatusKvNonFinite);
                    static_cast<__half*>(m.out)[at] = h;
                } else static_cast<float*>(m.out)[at] = v;
                continue;
            }
            if (m.output == kOutSquaredRelu) v = squared_relu(v);
            float* out = static_cast<float*>(m.out);
            if (p.input == kRowExperts) {
                // Parts of the mixture: [slot][row][width], the shared expert behind the routed ones.
                const uint32_t row = behind ? batch - p.rows * p.top : batch / p.top, part = behind ? p.top : batch % p.top;
                if (behind) v *= sigmoid(p.shared_logit[row]);
                out[part * p.part_stride + (size_t)row * m.out_ld + n] = v;
            } else {
                out[(size_t)r * m.out_ld + (size_t)batch * m.out_batch + n] = v;
            }
        }
        __syncthreads();
    }
}

template <int R>
int launch_rows(const RowProduct& p, dim3 grid, uint32_t smem, cudaStream_t stream, bool pdl) {
    static std::once_flag once[64];
    int device = 0;
    cudaGetDevice(&device);
    cudaError_t error = cudaSuccess;
    std::call_once(once[device & 63], [&] {
        error = cudaFuncSetAttribute(row_product_kernel<R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kRowSmemLimit);
    });
    GF_CUDA(error);
    return launch_kernel(row_product_kernel<R>, grid, dim3(kRowThreads), smem, stream, pdl, p);
}

}  // namespace

int launch_row_product(RowProduct p, cudaStream_t stream, bool pdl, uint32_t& launches) {
    if (p.count == 0 || p.count > 3 || p.rows == 0 || p.batches == 0) return fail(GF_ERR_INVALID, "row product: bad launch");
    const bool single = p.input == kRowRouted || p.input == kRowExperts;
    uint32_t k_max = 0, sets = 0, widest = 0;
    // Groups per CTA from the shapes alone, so that a row's sums are added in the same order whatever the row count.
    const uint32_t wanted = 2u * (uint32_t)sm_count();              // what is resident at once
    for (uint32_t i = 0; i < p.count; ++i) {
        RowMatrix& m = p.m[i];
        if (!m.weight || !m.out || m.k == 0 || m.n == 0) return fail(GF_ERR_INVALID, "row product: bad matrix");
        m.k_blocks = (m.k + kDenseBlockK - 1u) / kDenseBlockK;
        const uint32_t groups = (m.n + 7u) / 8u, batches = single ? 4u : p.batches;
        uint32_t per = paired_output(m.output) ? 2u : 1u;
        while (per < kRowWarps && (uint64_t)(groups + per - 1u) / per * batches > wanted) per *= 2u;
        // A warp's slice of K should not fall below two of its 512-byte loads.
        while (per < kRowWarps && (m.k + 31u) / 32u < 2u * (kRowWarps / per)) per *= 2u;
        // Every CTA of a head merges all of its attention partitions: few CTAs per head.
        if (p.input == kRowLatent) while (per < kRowWarps && (groups + per - 1u) / per > 4u) per *= 2u;
        m.groups_per_cta = per;
        m.first_set = sets;
        m.sets = (groups + per - 1u) / per;
        sets += m.sets;
        widest = std::max(widest, m.sets);
        k_max = std::max(k_max, m.k);
    }
    p.k_pad = (k_max + 31u) / 32u * 32u;
    if ((p.input == kRowNorm || p.input == kRowAddNorm || p.input == kRowPartNorm) && k_max != p.width) return fail(GF_ERR_INVALID, "row product: a normalised input has the matrices' K");
    if (p.input == kRowPartNorm && (p.norm_parts == 0 || p.norm_parts > kMaxNormParts || p.width % p.norm_parts)) return fail(GF_ERR_INVALID, "row product: %u norm parts of %u", p.norm_parts, p.width);
    auto whole = [](const void* pointer) { return (reinterpret_cast<uintptr_t>(pointer) & 15u) == 0u; };
    p.vector_rows = p.in_ld % 4u == 0u && p.in_batch % 4u == 0u && p.in2_ld % 4u == 0u && p.part_stride % 4u == 0u && whole(p.in) && whole(p.in2);
    if (p.input == kRowNorm || p.input == kRowAddNorm || p.input == kRowPartNorm)
        p.vector_rows = p.vector_rows && p.width % 4u == 0u && whole(p.residual) && whole(p.residual_out) && whole(p.gain0) && whole(p.gain1) && whole(p.normed_out);
    for (uint32_t i = 0; i < p.count; ++i) p.vector_rows = p.vector_rows && p.m[i].k % 4u == 0u;
    const uint32_t row_bytes = p.k_pad * 4u;
    if (row_bytes > kRowSmemLimit) return fail(GF_ERR_INVALID, "row product: K = %u is too wide", k_max);
    const uint32_t per_launch = single ? 1u : std::max(1u, std::min<uint32_t>(kRowMaxRows, kRowSmemLimit / row_bytes));
    const uint32_t all_rows = p.rows;
    const uint32_t cta_sets = p.input == kRowExperts ? widest : sets;
    const uint32_t cap = std::max(1u, (4u * (uint32_t)sm_count() + p.batches - 1u) / p.batches);
    for (uint32_t row = 0; row < all_rows; row += single ? all_rows : per_launch) {
        RowProduct q = p;
        const uint32_t rows = single ? 1u : std::min(per_launch, all_rows - row);
        q.rows = single ? all_rows : rows;
        if (!single && row) {
            if (q.in_rows) q.in_rows += row;
            else if (q.input == kRowLatent) q.in += (size_t)row * p.heads * p.attention_parts * p.latent_ld;
            else q.in += (size_t)row * p.in_ld;
            if (q.latent_ml) q.latent_ml += (size_t)row * p.heads * p.attention_parts * 2u;
            if (q.residual) q.residual += (size_t)row * p.width;
            if (q.residual_out) q.residual_out += (size_t)row * p.width;
            if (q.normed_out) q.normed_out += (size_t)row * p.width;
            if (q.latent_raw) {
                q.latent_raw += (size_t)row * p.latent_raw_ld;
                q.latent_rows = static_cast<uint8_t*>(p.latent_rows) + (size_t)row * p.latent_row_elements * (p.latent_f16 ? 2u : 4u);
            }
            for (uint32_t i = 0; i < q.count; ++i) {
                const size_t element = q.m[i].output == kOutLatentQuery && p.query_f16 ? 2u : 4u;
                const size_t rows_before = q.m[i].output == kOutLatentQuery ? (size_t)row * p.heads : row;
                q.m[i].out = static_cast<uint8_t*>(q.m[i].out) + rows_before * q.m[i].out_ld * element;
            }
        }
        dim3 grid(std::min(cta_sets, cap), p.batches + (p.latent_raw ? 1u : 0u));
        if (p.latent_raw) grid.x = std::max(grid.x, rows);
        const uint32_t smem = rows * row_bytes;
        int status = GF_ERR_INVALID;
        switch (rows) {
            case 1: status = launch_rows<1>(q, grid, smem, stream, pdl); break;
            case 2: status = launch_rows<2>(q, grid, smem, stream, pdl); break;
            case 3: status = launch_rows<3>(q, grid, smem, stream, pdl); break;
            case 4: status = launch_rows<4>(q, grid, smem, stream, pdl); break;
            case 5: status = launch_rows<5>(q, grid, smem, stream, pdl); break;
            case 6: status = launch_rows<6>(q, grid, smem, stream, pdl); break;
            case 7: status = launch_rows<7>(q, grid, smem, stream, pdl); break;
            case 8: status = launch_rows<8>(q, grid, smem, stream, pdl); break;
        }
        if (status != GF_OK) return status;
        ++launches;
    }
    return GF_OK;
}

}  // namespace gf
