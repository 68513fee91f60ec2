// State-space mixer (see state_space.cuh).
#include "state_space.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

namespace {

constexpr uint32_t kMaxWarps = 4;
constexpr uint32_t kSmemLimit = 160u * 1024u;

__device__ __forceinline__ void copy16(void* dst_smem, const void* src, bool valid) {      // zero-fills when not valid
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst_smem)), "l"(src), "r"(valid ? 16u : 0u) : "memory");
}
__device__ __forceinline__ void copy8(void* dst_smem, const void* src, bool valid) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(smem_u32(dst_smem)), "l"(src), "r"(valid ? 8u : 0u) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Two f32 values side by side in a register pair.
using Pair = unsigned long long;
__device__ __forceinline__ Pair pair_of(float lo, float hi) {
    Pair r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float pair_sum(Pair v) {
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}
__device__ __forceinline__ Pair pair_fma(Pair a, Pair b, Pair c) {
    Pair r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ Pair pair_mul(Pair a, Pair b) {
    Pair r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// The convolution of one channel at row r of a portion that starts at `base`: rows of the portion come from `raw`,
// earlier ones from the ring.
__device__ __forceinline__ float convolve(const StateSpace& p, const float* raw, const float* ring, uint32_t base, uint32_t r, uint32_t channel) {
    const float* taps = p.taps + (size_t)channel * p.tap_count;
    const uint32_t inner = p.inner(), row = p.input_row();
    float sum = 0.0f;
    for (uint32_t j = 0; j < p.tap_count; ++j) {
        const uint32_t back = p.tap_count - 1u - j;                    // rows behind row r
        if (base + r < back) continue;
        const float v = back <= r ? raw[(size_t)(r - back) * p.raw_ld + inner + channel] : ring[(size_t)((base + r - back) & p.input_mask) * row + channel];
        sum = fmaf(taps[j], v, sum);
    }
    return silu(sum + p.tap_bias[channel]);
}
__device__ __forceinline__ float2 step_of(const StateSpace& p, const float* raw, uint32_t r, uint32_t head) {
    const float dt = softplus(raw[(size_t)r * p.raw_ld + p.inner() + p.channels() + head] + p.step_bias[head]);
    return make_float2(dt, expf(p.decay[head] * dt));
}

struct TileLayout { uint32_t b, c, x, steps, stage, doubled, gate, bytes; };
// Offsets in bytes: `stages` stages of B, C, x and steps for `tile` tokens, then (x * dt) twice and the gates.
__host__ __device__ inline TileLayout tile_layout(uint32_t tile, uint32_t wide, uint32_t columns, uint32_t stages) {
    TileLayout t;
    t.b = 0;
    t.c = t.b + tile * wide * 4u;
    t.x = t.c + tile * wide * 4u;
    t.steps = t.x + tile * columns * 4u;
    t.stage = (t.steps + tile * 8u + 15u) & ~15u;
    t.doubled = stages * t.stage;
    t.gate = t.doubled + tile * columns * 8u;
    t.bytes = t.gate + (stages == 1u ? tile * columns * 4u : 0u);
    return t;
}
template <int NL> constexpr uint32_t tile_tokens() { return NL <= 256 ? 16u : NL <= 512 ? 8u : 4u; }

// A block holds some columns (of vdim) of one head's state in registers while it walks the tokens: L lanes share a
// column's N values, four apart in turn, NQ fours each; a lane holds V columns.  kPass: the convolution is computed here and the gate
// applied (rows of a pass); else the inputs come convolved.
template <int L, int NQ, int V, bool kPass>
__global__ void __launch_bounds__(kMaxWarps * 32) state_space_kernel(const __grid_constant__ StateSpace p) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr uint32_t kWide = L * NQ * 4, kTile = tile_tokens<(int)kWide>(), kStages = kPass ? 1u : 2u, kThreadsPer = 32u / L;
    const uint32_t tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31u, ln = lane % L;
    const uint32_t columns = threads / L * V, c0 = blockIdx.y * columns, local = (warp * kThreadsPer + lane / L) * V, column = c0 + local;
    const TileLayout at = tile_layout(kTile, kWide, columns, kStages);
    const bool chain = p.ring_stride == 0u;
    const uint32_t head = blockIdx.x, z = blockIdx.z, rows = chain ? p.rows : 1u, row0 = chain ? 0u : z;
    const uint32_t group = head / (p.heads / p.groups), np = p.state_row(), inner = p.inner(), input_row = p.input_row();
    // The state, the position and the ring were written at least two launches back: read ahead of the wait.
    const uint32_t base = p.positions[chain ? 0u : z], slots = *p.slots;
    const StreamRings rings = p.rings[(size_t)z * p.ring_stride];
    float* states = static_cast<float*>(const_cast<void*>(rings.ring_k)) + (size_t)head * p.vdim * np;
    float* ring = static_cast<float*>(const_cast<void*>(rings.ring_v));
    const size_t slot_elements = p.slot_elements();
    Pair s[V][2 * NQ];
    {
        const float* from = states + (base % slots) * slot_elements;
#pragma unroll
        for (int v = 0; v < V; ++v)
#pragma unroll
            for (int j = 0; j < NQ; ++j) {
                const uint32_t n = (j * L + ln) * 4u;
                float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (base > 0u && column + v < p.vdim && n < np) q = *reinterpret_cast<const float4*>(from + (size_t)(column + v) * np + n);
                s[v][2 * j] = pair_of(q.x, q.y);
                s[v][2 * j + 1] = pair_of(q.z, q.w);
            }
    }
    if (kPass) {
        pdl_wait();
        pdl_launch_dependents();
    }
    const float* raw = p.raw + (size_t)row0 * p.raw_ld;
    const float skip = p.skip[head];

    auto fill = [&](uint32_t tile, uint32_t stage) {
        uint8_t* to = smem + stage * at.stage;
        float *b = reinterpret_cast<float*>(to + at.b), *c = reinterpret_cast<float*>(to + at.c), *x = reinterpret_cast<float*>(to + at.x);
        float2* steps = reinterpret_cast<float2*>(to + at.steps);
        const uint32_t first = tile * kTile;
        if (kPass) {
            float* gate = reinterpret_cast<float*>(smem + at.gate);
            const uint32_t live = min(kTile, rows - first);
            for (uint32_t i = tid; i < live * kWide; i += threads) {
                const uint32_t t = i / kWide, n = i % kWide;
                const uint32_t channel = inner + group * p.state + n;
                b[i] = n < p.state ? convolve(p, raw, ring, base, first + t, channel) : 0.0f;
                c[i] = n < p.state ? convolve(p, raw, ring, base, first + t, channel + p.groups * p.state) : 0.0f;
            }
            for (uint32_t t = 0; t < live; ++t)
                for (uint32_t i = tid; i < columns; i += threads) {
                    const bool valid = c0 + i < p.vdim;
                    x[t * columns + i] = valid ? convolve(p, raw, ring, base, first + t, head * p.vdim + c0 + i) : 0.0f;
                    gate[t * columns + i] = valid ? raw[(size_t)(first + t) * p.raw_ld + head * p.vdim + c0 + i] : 0.0f;
                }
            if (tid < live) steps[tid] = step_of(p, raw, first + tid, head);
            return;
        }
        const uint32_t x_row = p.x_row();
        for (uint32_t i = tid; i < kTile * (kWide / 4u); i += threads) {
            const uint32_t t = i / (kWide / 4u), n = i % (kWide / 4u) * 4u, row = first + t;
            const bool valid = row < rows && n < np;
            const size_t from = valid ? ((size_t)row * p.groups + group) * np + n : 0u;
            copy16(b + t * kWide + n, p.b + from, valid);
            copy16(c + t * kWide + n, p.c + from, valid);
        }
        for (uint32_t i = tid; i < kTile * (columns / 4u); i += threads) {
            const uint32_t t = i / (columns / 4u), k = i % (columns / 4u) * 4u, row = first + t;
            const bool valid = row < rows && c0 + k < x_row;
            copy16(x + t * columns + k, p.x + (valid ? ((size_t)row * p.heads + head) * x_row + c0 + k : 0u), valid);
        }
        if (tid < kTile) copy8(steps + tid, p.steps + (first + tid < rows ? (size_t)(first + tid) * p.heads + head : 0u), first + tid < rows);
    };

    const uint32_t tiles = (rows + kTile - 1u) / kTile;
    // States kept: all of them where the slots hold them besides the one that was read, else the last.
    const uint32_t kept = kPass ? rows - min(rows, slots - 1u) : rows - 1u;
    if (!kPass) { fill(0u, 0u); copies_commit(); }
    for (uint32_t tile = 0; tile < tiles; ++tile) {
        const uint32_t stage = kPass ? 0u : tile & 1u, first = tile * kTile;
        if (kPass) fill(tile, 0u);
        else {
            if (tile + 1u < tiles) fill(tile + 1u, stage ^ 1u);
            copies_commit();
            copies_wait<1>();
        }
        __syncthreads();
        const uint8_t* from = smem + stage * at.stage;
        const float *b = reinterpret_cast<const float*>(from + at.b), *c = reinterpret_cast<const float*>(from + at.c), *x = reinterpret_cast<const float*>(from + at.x);
        const float2* steps = reinterpret_cast<const float2*>(from + at.steps);
        Pair* doubled = reinterpret_cast<Pair*>(smem + at.doubled);
        for (uint32_t i = tid; i < kTile * columns; i += threads) {
            const float v = x[i] * steps[i / columns].x;
            doubled[i] = pair_of(v, v);
        }
        __syncthreads();
#pragma unroll 1
        for (uint32_t t4 = 0; t4 < kTile && first + t4 < rows; t4 += 4u) {
            float part[4 * V];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const uint32_t t = t4 + q;
                const float decay = steps[t].y;
                const Pair a = pair_of(decay, decay);
                Pair xd[V], sum[V];
#pragma unroll
                for (int v = 0; v < V; v += 2) {
                    const ulonglong2 two = *reinterpret_cast<const ulonglong2*>(doubled + t * columns + local + v);
                    xd[v] = two.x;
                    xd[v + 1] = two.y;
                }
#pragma unroll
                for (int j = 0; j < NQ; ++j) {
                    const ulonglong2 bq = *reinterpret_cast<const ulonglong2*>(b + t * kWide + (j * L + ln) * 4u);
                    const ulonglong2 cq = *reinterpret_cast<const ulonglong2*>(c + t * kWide + (j * L + ln) * 4u);
#pragma unroll
                    for (int v = 0; v < V; ++v) {
                        s[v][2 * j] = pair_fma(bq.x, xd[v], pair_mul(s[v][2 * j], a));
                        s[v][2 * j + 1] = pair_fma(bq.y, xd[v], pair_mul(s[v][2 * j + 1], a));
                        sum[v] = j == 0 ? pair_mul(s[v][0], cq.x) : pair_fma(s[v][2 * j], cq.x, sum[v]);
                        sum[v] = pair_fma(s[v][2 * j + 1], cq.y, sum[v]);
                    }
                }
#pragma unroll
                for (int v = 0; v < V; ++v) part[q * V + v] = pair_sum(sum[v]);
                const uint32_t row = first + t;
                if (row >= kept && row < rows) {
                    float* to = states + ((base + row + 1u) % slots) * slot_elements;
#pragma unroll
                    for (int v = 0; v < V; ++v)
#pragma unroll
                        for (int j = 0; j < NQ; ++j) {
                            const uint32_t n = (j * L + ln) * 4u;
                            if (column + v < p.vdim && n < np) *reinterpret_cast<ulonglong2*>(to + (size_t)(column + v) * np + n) = make_ulonglong2(s[v][2 * j], s[v][2 * j + 1]);
                        }
                }
            }
            // Sums over the L lanes: every round halves the values a lane is left with.
            uint32_t count = 4u * V, index = 0;
#pragma unroll
            for (uint32_t o = L / 2u; o > 0u; o >>= 1) {
                const bool upper = (lane & o) != 0u;
                if (count > 1u) {
                    count /= 2u;
                    if (upper) index += count;
#pragma unroll
                    for (uint32_t i = 0; i < 2u * V; ++i) {
                        if (i >= count) break;
                        const float keep = upper ? part[i + count] : part[i], send = upper ? part[i] : part[i + count];
                        part[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                    }
                } else part[0] += __shfl_xor_sync(0xffffffffu, part[0], o);
            }
            const bool writer = (uint32_t)L <= 4u * V || ln % (L / (4u * V) > 0u ? L / (4u * V) : 1u) == 0u;
#pragma unroll
            for (uint32_t i = 0; i < 4u * V; ++i) {
                if (i >= count) break;
                const uint32_t t = t4 + (index + i) / V, k = local + (index + i) % V, row = first + t;
                if (!writer || row >= rows || c0 + k >= p.vdim) continue;
                float y = fmaf(skip, x[t * columns + k], part[i]);
                if (kPass) y *= silu(reinterpret_cast<const float*>(smem + at.gate)[t * columns + k]);
                p.out[(size_t)(row0 + row) * inner + head * p.vdim + c0 + k] = y;
            }
        }
        __syncthreads();                                               // the tile's buffers are free again
    }
    // The convolution's inputs of the rows that later tokens look back at: every block its own columns, the first one
    // of a group the shared channels.
    const uint32_t first_kept = kPass ? 0u : rows - min(rows, p.tap_count - 1u);
    const bool shared = head % (p.heads / p.groups) == 0u && blockIdx.y == 0u;
    for (uint32_t r = first_kept; r < rows; ++r) {
        const float* from = raw + (size_t)r * p.raw_ld + inner;
        float* to = ring + (size_t)((base + r) & p.input_mask) * input_row;
        for (uint32_t i = tid; i < columns; i += threads)
            if (c0 + i < p.vdim) to[head * p.vdim + c0 + i] = from[head * p.vdim + c0 + i];
        if (shared)
            for (uint32_t i = tid; i < p.state; i += threads) {
                const uint32_t channel = inner + group * p.state + i;
                to[channel] = from[channel];
                to[channel + p.groups * p.state] = from[channel + p.groups * p.state];
            }
    }
}

// The convolved inputs of a chunk, padding included.
constexpr uint32_t kConvolveRows = 8;
__global__ void __launch_bounds__(128) convolve_chunk_kernel(const __grid_constant__ StateSpace p) {
    const uint32_t np = p.state_row(), x_row = p.x_row(), all_x = p.heads * x_row, all_n = p.groups * np;
    const uint32_t base = p.positions[0], end = min(p.rows, (blockIdx.y + 1u) * kConvolveRows);
    const float* ring = static_cast<const float*>(p.rings->ring_v);
    uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    float* out = nullptr;
    uint32_t ld = 0, channel = 0;
    bool valid = false;
    if (i < all_x) {
        const uint32_t k = i % x_row;
        out = p.x + i; ld = all_x; channel = i / x_row * p.vdim + k; valid = k < p.vdim;
    } else if (i - all_x < 2u * all_n) {
        i -= all_x;
        const uint32_t which = i / all_n, j = i % all_n, n = j % np;
        out = (which ? p.c : p.b) + j; ld = all_n; channel = p.inner() + (which * p.groups + j / np) * p.state + n; valid = n < p.state;
    } else if (i - all_x - 2u * all_n < p.heads) {
        const uint32_t head = i - all_x - 2u * all_n;
        for (uint32_t r = blockIdx.y * kConvolveRows; r < end; ++r) p.steps[(size_t)r * p.heads + head] = step_of(p, p.raw, r, head);
        return;
    } else return;
    for (uint32_t r = blockIdx.y * kConvolveRows; r < end; ++r) out[(size_t)r * ld] = valid ? convolve(p, p.raw, ring, base, r, channel) : 0.0f;
}

template <int L, int NQ, int V, bool kPass>
int launch_recurrence(const StateSpace& p, cudaStream_t stream, bool pdl) {
    constexpr uint32_t kWide = L * NQ * 4, per_warp = 32u / L * V;
    static std::once_flag once[64];
    int device = 0;
    cudaGetDevice(&device);
    cudaError_t error = cudaSuccess;
    std::call_once(once[device & 63], [&] {
        error = cudaFuncSetAttribute(state_space_kernel<L, NQ, V, kPass>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit);
    });
    GF_CUDA(error);
    // As many warps per block as still give every SM a block; the block's columns are whole 16-byte pieces.
    const uint32_t sequences = p.ring_stride ? p.rows : 1u;
    uint32_t warps = kMaxWarps;
    while (warps > 1u && (warps / 2u) * per_warp % 4u == 0u
           && ((uint64_t)p.heads * sequences * ((p.vdim + warps * per_warp - 1u) / (warps * per_warp)) < (uint64_t)sm_count() || (warps / 2u) * per_warp >= p.vdim))
        warps /= 2u;
    const uint32_t columns = warps * per_warp;
    const TileLayout layout = tile_layout(tile_tokens<(int)kWide>(), kWide, columns, kPass ? 1u : 2u);
    return launch_kernel(state_space_kernel<L, NQ, V, kPass>, dim3(p.heads, (p.vdim + columns - 1u) / columns, sequences), dim3(warps * 32u), layout.bytes, stream, pdl, p);
}

template <bool kPass>
int launch_by_state(const StateSpace& p, cudaStream_t stream, bool pdl) {
    const uint32_t fours = p.state_row() / 4u;
    if (fours <= 1u) return launch_recurrence<1, 1, 4, kPass>(p, stream, pdl);
    if (fours <= 2u) return launch_recurrence<1, 2, 4, kPass>(p, stream, pdl);
    if (fours <= 4u) return launch_recurrence<2, 2, 4, kPass>(p, stream, pdl);
    if (fours <= 8u) return launch_recurrence<4, 2, 4, kPass>(p, stream, pdl);
    if (fours <= 16u) return launch_recurrence<8, 2, 4, kPass>(p, stream, pdl);
    if (fours <= 32u) return launch_recurrence<16, 2, 4, kPass>(p, stream, pdl);
    if (fours <= 64u) return launch_recurrence<32, 2, 4, kPass>(p, stream, pdl);
    if (fours <= 128u) return launch_recurrence<32, 4, 4, kPass>(p, stream, pdl);
    return launch_recurrence<32, 8, 2, kPass>(p, stream, pdl);
}

bool usable(const StateSpace& p) {
    return p.raw && p.taps && p.tap_bias && p.step_bias && p.decay && p.skip && p.rings && p.positions && p.slots && p.out && p.rows && p.heads && p.vdim
           && p.state && p.state <= kMaxStateSize && p.groups && p.heads % p.groups == 0u && p.tap_count && (p.input_mask & (p.input_mask + 1u)) == 0u
           && p.raw_ld >= p.inner() + p.channels() + p.heads;
}

}  // namespace

int launch_state_space_rows(const StateSpace& p, cudaStream_t stream, bool pdl) {
    // Rows of the pass and the rows they look back at share the ring.
    if (!usable(p) || p.input_mask + 1u < p.tap_count - 1u + (p.ring_stride ? 1u : p.rows)) return fail(GF_ERR_INVALID, "state space: bad arguments");
    return launch_by_state<true>(p, stream, pdl);
}

int launch_state_space_chunk(const StateSpace& p, cudaStream_t stream) {
    if (!usable(p) || p.ring_stride || !p.x || !p.b || !p.c || !p.steps || p.input_mask + 1u < p.tap_count - 1u) return fail(GF_ERR_INVALID, "state space: bad arguments");
    const uint32_t items = p.heads * p.x_row() + 2u * p.groups * p.state_row() + p.heads;
    convolve_chunk_kernel<<<dim3((items + 127u) / 128u, (p.rows + kConvolveRows - 1u) / kConvolveRows), 128, 0, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return launch_by_state<false>(p, stream, false);
}

}  // namespace gf
