// Causal attention of a prompt chunk over keys and values per head or per group of heads, binary16 (see latent.cuh).
#include "grouped.cuh"
#include "latent.cuh"

#include <mutex>

namespace gf {

namespace {

constexpr uint32_t kRows = 64, kKeys = 64, kThreads = 128;      // a warp owns sixteen query rows

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

// Block = (64 chunk rows, head).  Tiles of 64 keys and values, the next one copied while this one is used; a warp's
// scores, weights and outputs stay in its registers.  G = groups of sixteen dimensions a head has at most.
// kCap: capped scores.
template <int G, bool kCap>
__global__ void __launch_bounds__(kThreads) head_attention_kernel(const __grid_constant__ HeadAttention p) {
    extern __shared__ __align__(16) uint8_t smem[];
    const uint32_t q_stride = p.dim_pad + 8u, v_stride = p.vdim_pad + 8u;
    __half* q_tile = reinterpret_cast<__half*>(smem);
    __half* k_tiles = q_tile + kRows * q_stride;
    __half* v_tiles = k_tiles + 2u * kKeys * q_stride;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, g = lane >> 2, t = lane & 3u;
    const uint32_t head = blockIdx.y, first_row = (gridDim.x - 1u - blockIdx.x) * kRows;      // the longest blocks first
    const uint32_t base = *p.position, end = base + min(first_row + kRows, p.rows), tiles = (end + kKeys - 1u) / kKeys;
    const __half* q = p.q + (size_t)head * p.dim_pad;
    const uint32_t kv = head / (p.heads / p.kv_heads);
    const __half* keys = p.k + (size_t)kv * p.dim_pad;
    const __half* values = p.v + (size_t)kv * p.vdim_pad;
    const size_t q_ld = (size_t)p.heads * p.dim_pad, k_ld = (size_t)p.kv_heads * p.dim_pad, v_ld = (size_t)p.kv_heads * p.vdim_pad;
    // Keys before the chunk lie in the rings, or ahead of the chunk's own where there are none.
    const uint32_t own_from = p.rings ? base : 0u;
    const __half *ring_k = nullptr, *ring_v = nullptr;
    if (p.rings) {
        ring_k = static_cast<const __half*>(p.rings->ring_k) + (size_t)kv * p.dim_pad;
        ring_v = static_cast<const __half*>(p.rings->ring_v) + (size_t)kv * p.vdim_pad;
    }
    const uint32_t k_pieces = p.dim_pad / 8u, v_pieces = p.vdim_pad / 8u;

    auto load_tile = [&](uint32_t tile, uint32_t slot) {
        __half* kd = k_tiles + slot * kKeys * q_stride;
        __half* vd = v_tiles + slot * kKeys * v_stride;
        // Two threads per key, alternating pieces.
        const uint32_t r = tid >> 1, position = tile * kKeys + r;
        const bool valid = position < end, cached = position < own_from;
        const size_t at = !valid ? 0u : cached ? position & p.ring_mask : position - own_from;
        const __half* ks = (cached ? ring_k : keys) + at * k_ld;
        const __half* vs = (cached ? ring_v : values) + at * v_ld;
        for (uint32_t piece = tid & 1u; piece < k_pieces; piece += 2u) copy16(kd + r * q_stride + piece * 8u, ks + piece * 8u, valid);
        for (uint32_t piece = tid & 1u; piece < v_pieces; piece += 2u) copy16(vd + r * v_stride + piece * 8u, vs + piece * 8u, valid);
    };
    {
        const uint32_t r = tid >> 1, row = first_row + r;
        const bool valid = row < p.rows;
        const __half* src = q + (valid ? row : 0u) * q_ld;
        for (uint32_t piece = tid & 1u; piece < k_pieces; piece += 2u) copy16(q_tile + r * q_stride + piece * 8u, src + piece * 8u, valid);
    }
    load_tile(0u, 0u);
    copies_commit();

    float acc[2 * G][4];
#pragma unroll
    for (int i = 0; i < 2 * G; ++i) { acc[i][0] = 0.0f; acc[i][1] = 0.0f; acc[i][2] = 0.0f; acc[i][3] = 0.0f; }
    float top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
    uint32_t qa[G <= 8 ? G : 1][4];
    const uint32_t steps = p.dim_pad / 16u, groups = p.vdim_pad / 16u;
    const uint32_t sees[2] = {base + first_row + warp * 16u + g, base + first_row + warp * 16u + g + 8u};      // last visible position
    const __half* a_row = q_tile + (warp * 16u + (lane & 15u)) * q_stride + (lane >> 4) * 8u;
    constexpr float kLog2e = 1.4426950408889634f;
    const float inverse_cap = kCap ? 1.0f / p.softcap : 0.0f;

    for (uint32_t tile = 0; tile < tiles; ++tile) {
        if (tile + 1u < tiles) load_tile(tile + 1u, (tile + 1u) & 1u);
        copies_commit();
        copies_wait<1>();
        __syncthreads();
        if (G <= 8 && tile == 0u)
#pragma unroll
            for (int k = 0; k < G; ++k)
                if ((uint32_t)k < steps) ldmatrix4(qa[k < (G <= 8 ? G : 1) ? k : 0], a_row + k * 16u);
        const __half* k_tile = k_tiles + (tile & 1u) * kKeys * q_stride;
        const __half* v_tile = v_tiles + (tile & 1u) * kKeys * v_stride;
        // ---- scores of sixteen rows x 64 keys
        float s[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n) { s[n][0] = 0.0f; s[n][1] = 0.0f; s[n][2] = 0.0f; s[n][3] = 0.0f; }
        const __half* b_row = k_tile + ((lane & 7u) + (lane >> 4) * 8u) * q_stride + ((lane >> 3) & 1u) * 8u;
#pragma unroll
        for (int k = 0; k < G; ++k) {
            if ((uint32_t)k >= steps) break;
            uint32_t a[4];
            if (G <= 8) {
#pragma unroll
                for (int i = 0; i < 4; ++i) a[i] = qa[k < (G <= 8 ? G : 1) ? k : 0][i];
            } else ldmatrix4(a, a_row + k * 16u);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                uint32_t b[4];
                ldmatrix4(b, b_row + n * 16u * q_stride + k * 16u);
                mma_f16(s[2 * n], a, b[0], b[1]);
                mma_f16(s[2 * n + 1], a, b[2], b[3]);
            }
        }
        if (kCap)
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[n][e] = soft_cap(s[n][e], p.softcap, inverse_cap);
        if (tile * kKeys + kKeys > base + first_row + warp * 16u + 1u)      // some key of the tile lies behind some row
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (tile * kKeys + 8u * n + 2u * t + (e & 1) > sees[e >> 1]) s[n][e] = -INFINITY;
        // ---- softmax
        uint32_t w[4][4];                                                    // A operands of the outputs
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float now = top[i];
#pragma unroll
            for (int n = 0; n < 8; ++n) now = fmaxf(now, fmaxf(s[n][2 * i], s[n][2 * i + 1]));
            now = fmaxf(now, __shfl_xor_sync(0xffffffffu, now, 1));
            now = fmaxf(now, __shfl_xor_sync(0xffffffffu, now, 2));
            const float shift = now == -INFINITY ? 0.0f : now * kLog2e;
            const float correction = exp2f(fmaf(top[i], kLog2e, -shift));
            float part = 0.0f;
#pragma unroll
            for (int n = 0; n < 8; ++n) {
                const float x = exp2f(fmaf(s[n][2 * i], kLog2e, -shift)), y = exp2f(fmaf(s[n][2 * i + 1], kLog2e, -shift));
                part += x + y;
                w[n >> 1][(n & 1) * 2 + i] = half_pair(x, y);
            }
            sum[i] = sum[i] * correction + part;
            top[i] = now;
#pragma unroll
            for (int o = 0; o < 2 * G; ++o) { acc[o][2 * i] *= correction; acc[o][2 * i + 1] *= correction; }
        }
        // ---- outputs
        const __half* v_row = v_tile + (lane & 15u) * v_stride + (lane >> 4) * 8u;
#pragma unroll
        for (int k = 0; k < 4; ++k)
#pragma unroll
            for (int d = 0; d < G; ++d) {
                if ((uint32_t)d >= groups) break;
                uint32_t b[4];
                ldmatrix4_transposed(b, v_row + k * 16u * v_stride + d * 16u);
                mma_f16(acc[2 * d], w[k], b[0], b[1]);
                mma_f16(acc[2 * d + 1], w[k], b[2], b[3]);
            }
        __syncthreads();                                                      // the tile's buffer is free again
    }
    copies_wait<0>();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
        const uint32_t row = first_row + warp * 16u + g + 8u * i;
        if (row >= p.rows) continue;
        float factor = 1.0f / sum[i];
        if (p.sink) {
            const float sink = p.sink[head], most = fmaxf(top[i], sink);
            factor = expf(top[i] - most) / (sum[i] * expf(top[i] - most) + expf(sink - most));
        }
        if (p.gate) factor *= sigmoid(p.gate[(size_t)row * p.heads + head]);
#pragma unroll
        for (int o = 0; o < 2 * G; ++o) {
            const uint32_t d = o * 8u + 2u * t;
            if (d < p.vdim) store_operand(p.result, row, head * p.vdim + d, acc[o][2 * i] * factor);
            if (d + 1u < p.vdim) store_operand(p.result, row, head * p.vdim + d + 1u, acc[o][2 * i + 1] * factor);
        }
    }
}

// Cache rows [0, positions) -- the ring's, then the chunk's own -- as a bf16 operand.
__global__ void __launch_bounds__(64) latent_operand_kernel(const StreamRings* rings, const __half* __restrict__ own, const uint32_t* __restrict__ base_position,
                                                            uint32_t row_elements, uint32_t ring_mask, const Operand result) {
    const uint32_t position = blockIdx.x, base = *base_position;
    const __half* ring = static_cast<const __half*>(rings->ring_k);
    const __half* src = position < base ? ring + (size_t)(position & ring_mask) * row_elements : own + (size_t)(position - base) * row_elements;
    for (uint32_t piece = threadIdx.x; piece < result.k_pad / 8u; piece += blockDim.x) {
        uint4 out = make_uint4(0u, 0u, 0u, 0u);
        if (piece * 8u < row_elements) {
            const uint4 in = *reinterpret_cast<const uint4*>(src + piece * 8u);
            const __half2* h = reinterpret_cast<const __half2*>(&in);
            uint32_t* o = reinterpret_cast<uint32_t*>(&out);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f = __half22float2(h[i]);
                asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(o[i]) : "f"(f.y), "f"(f.x));
            }
        }
        *reinterpret_cast<uint4*>(static_cast<uint8_t*>(result.data) + operand_offset(result, position, piece * 8u)) = out;
    }
}

template <int G, bool kCap>
int launch_groups(const HeadAttention& p, cudaStream_t stream) {
    const uint32_t smem = (kRows + 2u * kKeys) * (p.dim_pad + 8u) * 2u + 2u * kKeys * (p.vdim_pad + 8u) * 2u;
    static std::once_flag once[64];
    int device = 0;
    cudaGetDevice(&device);
    cudaError_t error = cudaSuccess;
    std::call_once(once[device & 63], [&] { error = cudaFuncSetAttribute(head_attention_kernel<G, kCap>, cudaFuncAttributeMaxDynamicSharedMemorySize, 180 * 1024); });
    GF_CUDA(error);
    head_attention_kernel<G, kCap><<<dim3((p.rows + kRows - 1u) / kRows, p.heads), kThreads, smem, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

template <bool kCap>
int launch_by_dim(const HeadAttention& p, cudaStream_t stream) {
    const uint32_t groups = (p.dim_pad > p.vdim_pad ? p.dim_pad : p.vdim_pad) / 16u;
    if (groups <= 2u) return launch_groups<2, kCap>(p, stream);
    if (groups <= 4u) return launch_groups<4, kCap>(p, stream);
    if (groups <= 8u) return launch_groups<8, kCap>(p, stream);
    return launch_groups<16, kCap>(p, stream);
}

}  // namespace

int launch_head_attention(const HeadAttention& p, cudaStream_t stream) {
    if (!p.q || !p.k || !p.v || !p.position || !p.result.data || p.rows == 0 || p.heads == 0 || p.kv_heads == 0 || p.heads % p.kv_heads || p.dim_pad % 16u || p.vdim_pad % 16u || p.dim_pad == 0
        || p.vdim_pad == 0 || p.dim_pad > kHeadAttentionMaxDim || p.vdim_pad > kHeadAttentionMaxDim || p.vdim > p.vdim_pad)
        return fail(GF_ERR_INVALID, "head attention: bad arguments");
    return p.softcap > 0.0f ? launch_by_dim<true>(p, stream) : launch_by_dim<false>(p, stream);
}

int launch_latent_operand(const StreamRings* rings, const void* own, const uint32_t* position, uint32_t positions, uint32_t row_elements, uint32_t ring_mask,
                          const Operand& result, cudaStream_t stream) {
    if (!rings || !own || !position || positions == 0 || positions > result.capacity || row_elements > result.k_pad || result.f32)
        return fail(GF_ERR_INVALID, "latent operand: bad arguments");
    latent_operand_kernel<<<positions, 64, 0, stream>>>(rings, static_cast<const __half*>(own), position, row_elements, ring_mask, result);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

}  // namespace gf
