// State-space mixer (see state_space.cuh).
#include "state_space.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

namespace {

constexpr uint32_t kMaxWarps = 4, kChunkWarps = 8;
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
// earlier ones from the ring.  kFew: up to four taps, whose reads are issued together.
template <bool kFew>
__device__ __forceinline__ float convolve(const StateSpace& p, const float* raw, const float* ring, uint32_t base, uint32_t r, uint32_t channel) {
    const float* taps = p.taps + (size_t)channel * p.tap_count;
    const uint32_t inner = p.inner(), row = p.input_row();
    auto value = [&](uint32_t back) {                                  // `back` rows behind row r
        if (base + r < back) return 0.0f;
        return back <= r ? raw[(size_t)(r - back) * p.raw_ld + inner + channel] : ring[(size_t)((base + r - back) & p.input_mask) * row + channel];
    };
    float sum = 0.0f;
    if constexpr (kFew) {
        float v[4], w[4];
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j) {                            // j taps before the last one
            v[j] = j < p.tap_count ? value(j) : 0.0f;
            w[j] = j < p.tap_count ? taps[p.tap_count - 1u - j] : 0.0f;
        }
        const float bias = p.tap_bias[channel];
#pragma unroll
        for (int j = 3; j >= 0; --j) sum = fmaf(w[j], v[j], sum);
        return silu(sum + bias);
    } else {
        for (uint32_t j = 0; j < p.tap_count; ++j) sum = fmaf(taps[j], value(p.tap_count - 1u - j), sum);
        return silu(sum + p.tap_bias[channel]);
    }
}
// dt and the logarithm of the decay.
__device__ __forceinline__ float2 step_of(const StateSpace& p, const float* raw, uint32_t r, uint32_t head) {
    const float dt = softplus(raw[(size_t)r * p.raw_ld + p.inner() + p.channels() + head] + p.step_bias[head]);
    return make_float2(dt, p.decay[head] * dt);
}

// Sums part[0 .. 4 V) over the L lanes that share a column: every round halves the values a lane is left with, so that
// part[0 .. lane_values()) hold the sums of values lane_first(lane) on.  Lanes left with the same value: the first writes.
template <int L, int V> constexpr uint32_t lane_values() { return L >= 4 * V ? 1u : 4u * V / L; }
template <int L, int V> constexpr uint32_t lane_copies() { return L > 4 * V ? L / (4u * V) : 1u; }
template <int L, int V>
__device__ __forceinline__ uint32_t lane_first(uint32_t lane) { return lane % L / lane_copies<L, V>() * lane_values<L, V>(); }
template <int L, int V>
__device__ __forceinline__ void lane_sums(float (&part)[4 * V], uint32_t lane) {
    uint32_t count = 4u * V;
#pragma unroll
    for (uint32_t o = L / 2u; o > 0u; o >>= 1) {
        const bool upper = (lane & o) != 0u;
        if (count > 1u) {
            count /= 2u;
#pragma unroll
            for (uint32_t i = 0; i < 2u * V; ++i) {
                if (i >= count) break;
                const float keep = upper ? part[i + count] : part[i], send = upper ? part[i] : part[i + count];
                part[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        } else part[0] += __shfl_xor_sync(0xffffffffu, part[0], o);
    }
}

// A block holds some columns (of vdim) of one head's state in registers while it walks the tokens: L lanes share a
// column's N values, four apart in turn, NQ fours each; a lane holds V columns.
template <int L, int NQ, int V>
struct Columns {
    static constexpr uint32_t kWide = L * NQ * 4;                      // N with its padding
    uint32_t count, first, local, ln, np, vdim;                        // count columns from `first` on; this lane's from first + local on
    __device__ Columns(const StateSpace& p) {
        const uint32_t lane = threadIdx.x & 31u;
        count = blockDim.x / L * V; first = blockIdx.y * count;
        ln = lane % L; local = ((threadIdx.x >> 5) * (32u / L) + lane / L) * V;
        np = p.state_row(); vdim = p.vdim;
    }
    __device__ uint32_t column(int v) const { return first + local + v; }
    __device__ uint32_t n(int j) const { return (j * L + ln) * 4u; }
    __device__ void load(Pair (&s)[V][2 * NQ], const float* head_state, bool any) const {
#pragma unroll
        for (int v = 0; v < V; ++v)
#pragma unroll
            for (int j = 0; j < NQ; ++j) {
                float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (any && column(v) < vdim && n(j) < np) q = *reinterpret_cast<const float4*>(head_state + (size_t)column(v) * np + n(j));
                s[v][2 * j] = pair_of(q.x, q.y);
                s[v][2 * j + 1] = pair_of(q.z, q.w);
            }
    }
    __device__ void store(const Pair (&s)[V][2 * NQ], float* head_state) const {
#pragma unroll
        for (int v = 0; v < V; ++v)
#pragma unroll
            for (int j = 0; j < NQ; ++j)
                if (column(v) < vdim && n(j) < np) *reinterpret_cast<ulonglong2*>(head_state + (size_t)column(v) * np + n(j)) = make_ulonglong2(s[v][2 * j], s[v][2 * j + 1]);
    }
};

// The convolution's inputs of the rows from `first` on, which later tokens look back at: every block its own columns,
// the first one of a group the shared channels.
__device__ __forceinline__ void keep_inputs(const StateSpace& p, const float* raw, float* ring, uint32_t base, uint32_t first, uint32_t rows, uint32_t head,
                                            uint32_t first_column, uint32_t columns) {
    const uint32_t per_group = p.heads / p.groups, inner = p.inner();
    const bool shared = head % per_group == 0u && blockIdx.y == 0u;
    for (uint32_t r = first; r < rows; ++r) {
        const float* from = raw + (size_t)r * p.raw_ld + inner;
        float* to = ring + (size_t)((base + r) & p.input_mask) * p.input_row();
        for (uint32_t i = threadIdx.x; i < columns; i += blockDim.x)
            if (first_column + i < p.vdim) to[head * p.vdim + first_column + i] = from[head * p.vdim + first_column + i];
        if (shared)
            for (uint32_t i = threadIdx.x; i < p.state; i += blockDim.x) {
                const uint32_t channel = inner + head / per_group * p.state + i;
                to[channel] = from[channel];
                to[channel + p.groups * p.state] = from[channel + p.groups * p.state];
            }
    }
}

// ------------------------------------------------------------------ rows of a pass

constexpr uint32_t kPassTile = 4;
__host__ __device__ inline uint32_t pass_smem(uint32_t wide, uint32_t columns) { return kPassTile * (2u * wide + 4u * columns) * 4u + kPassTile * 8u; }

// Token by token, the convolution computed here and the gate applied.
template <int L, int NQ, int V>
__global__ void __launch_bounds__(kMaxWarps * 32, 3) state_space_rows_kernel(const __grid_constant__ StateSpace p) {
    extern __shared__ __align__(16) uint8_t smem[];
    const Columns<L, NQ, V> mine(p);
    constexpr uint32_t kWide = Columns<L, NQ, V>::kWide;
    const uint32_t tid = threadIdx.x, threads = blockDim.x, lane = tid & 31u, columns = mine.count, c0 = mine.first;
    Pair* doubled = reinterpret_cast<Pair*>(smem);                     // [tile][columns]: x * dt, twice
    float* b = reinterpret_cast<float*>(doubled + kPassTile * columns);            // [tile][kWide]
    float *c = b + kPassTile * kWide, *x = c + kPassTile * kWide, *gate = x + kPassTile * columns;
    float2* steps = reinterpret_cast<float2*>(gate + kPassTile * columns);         // dt, decay
    const bool chain = p.ring_stride == 0u;
    const uint32_t head = blockIdx.x, z = blockIdx.z, rows = chain ? p.rows : 1u, row0 = chain ? 0u : z, inner = p.inner(), group = head / (p.heads / p.groups);
    // The state, the position and the ring were written at least two launches back: read ahead of the wait.
    const uint32_t base = p.positions[chain ? 0u : z], slots = *p.slots;
    const StreamRings rings = p.rings[(size_t)z * p.ring_stride];
    const size_t slot_elements = p.slot_elements();
    float* states = static_cast<float*>(const_cast<void*>(rings.ring_k)) + (size_t)head * p.vdim * mine.np;
    float* ring = static_cast<float*>(const_cast<void*>(rings.ring_v));
    Pair s[V][2 * NQ];
    mine.load(s, states + (base % slots) * slot_elements, base > 0u);
    pdl_wait();
    pdl_launch_dependents();
    const float* raw = p.raw + (size_t)row0 * p.raw_ld;
    const float skip = p.skip[head];

    auto fill = [&](uint32_t first, uint32_t live, auto convolved) {
        for (uint32_t t = 0; t < live; ++t) {
            const uint32_t r = first + t, all = 2u * kWide + columns;
#pragma unroll 3
            for (uint32_t i = tid; i < all; i += threads) {
                const uint32_t n = i % kWide, k = i - 2u * kWide;
                const bool vectors = i < 2u * kWide, valid = vectors ? n < p.state : c0 + k < p.vdim;
                const uint32_t channel = vectors ? inner + (i < kWide ? 0u : p.groups * p.state) + group * p.state + n : head * p.vdim + c0 + k;
                const float v = valid ? convolved(r, channel) : 0.0f;
                if (vectors) (i < kWide ? b : c)[t * kWide + n] = v;
                else x[t * columns + k] = v;
            }
            for (uint32_t i = tid; i < columns; i += threads) gate[t * columns + i] = c0 + i < p.vdim ? raw[(size_t)r * p.raw_ld + head * p.vdim + c0 + i] : 0.0f;
        }
        if (tid < live) {
            const float2 step = step_of(p, raw, first + tid, head);
            steps[tid] = make_float2(step.x, expf(step.y));
        }
    };
    // States kept: all of them where the slots hold them besides the one that was read, else the last.
    const uint32_t kept = rows - min(rows, slots - 1u);
    for (uint32_t first = 0; first < rows; first += kPassTile) {
        const uint32_t live = min(kPassTile, rows - first);
        if (p.tap_count <= 4u) fill(first, live, [&](uint32_t r, uint32_t channel) { return convolve<true>(p, raw, ring, base, r, channel); });
        else fill(first, live, [&](uint32_t r, uint32_t channel) { return convolve<false>(p, raw, ring, base, r, channel); });
        __syncthreads();
        for (uint32_t i = tid; i < live * columns; i += threads) {
            const float v = x[i] * steps[i / columns].x;
            doubled[i] = pair_of(v, v);
        }
        __syncthreads();
        float part[4 * V];
#pragma unroll
        for (int i = 0; i < 4 * V; ++i) part[i] = 0.0f;
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            if ((uint32_t)t >= live) break;
            const float decay = steps[t].y;
            const Pair a = pair_of(decay, decay);
            Pair sum[V];
#pragma unroll
            for (int j = 0; j < NQ; ++j) {
                const ulonglong2 bq = *reinterpret_cast<const ulonglong2*>(b + t * kWide + mine.n(j)), cq = *reinterpret_cast<const ulonglong2*>(c + t * kWide + mine.n(j));
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    const Pair xd = doubled[t * columns + mine.local + v];
                    s[v][2 * j] = pair_fma(bq.x, xd, pair_mul(s[v][2 * j], a));
                    s[v][2 * j + 1] = pair_fma(bq.y, xd, pair_mul(s[v][2 * j + 1], a));
                    sum[v] = j == 0 ? pair_mul(s[v][0], cq.x) : pair_fma(s[v][2 * j], cq.x, sum[v]);
                    sum[v] = pair_fma(s[v][2 * j + 1], cq.y, sum[v]);
                }
            }
#pragma unroll
            for (int v = 0; v < V; ++v) part[t * V + v] = pair_sum(sum[v]);
            const uint32_t row = first + t;
            if (row >= kept) mine.store(s, states + ((base + row + 1u) % slots) * slot_elements);
        }
        lane_sums<L, V>(part, lane);
#pragma unroll
        for (uint32_t i = 0; i < lane_values<L, V>(); ++i) {
            const uint32_t at = lane_first<L, V>(lane) + i, t = at / V, k = mine.local + at % V;
            if (mine.ln % lane_copies<L, V>() || t >= live || c0 + k >= p.vdim) continue;
            p.out[(size_t)(row0 + first + t) * inner + head * p.vdim + c0 + k] = fmaf(skip, x[t * columns + k], part[i]) * silu(gate[t * columns + k]);
        }
        __syncthreads();                                               // the tile's buffers are free again
    }
    keep_inputs(p, raw, ring, base, 0u, rows, head, c0, columns);
}

// ------------------------------------------------------------------ chunks

// Four tokens at a time.  With a_t the logarithm of token t's decay and A_t their sums within the four,
//   y_t = exp(A_t) C_t . S + sum over s <= t of exp(A_t - A_s) dt_s (C_t . B_s) x_s + skip x_t
//   S  <- exp(A_3) S + sum over s of exp(A_3 - A_s) dt_s B_s x_s^T
// so that a state's element costs nine multiply-adds per four tokens; the products C_t . B_s come with the inputs.
template <int NL> constexpr uint32_t chunk_tile() { return NL <= 128 ? 32u : NL <= 256 ? 16u : NL <= 512 ? 8u : 4u; }
struct ChunkLayout { uint32_t c, x, steps, cb, stage, doubled, m, u, w, whole, bytes; };
__host__ __device__ inline ChunkLayout chunk_layout(uint32_t tile, uint32_t wide, uint32_t columns) {      // bytes; two stages, then one of each
    ChunkLayout t;
    t.c = tile * wide * 4u;
    t.x = 2u * t.c;
    t.cb = t.x + tile * columns * 4u;
    t.steps = t.cb + tile * 16u;
    t.stage = t.steps + tile * 8u;
    t.doubled = 2u * t.stage;
    t.m = t.doubled + tile * columns * 8u;
    t.u = t.m + tile * 16u;
    t.w = t.u + tile * 4u;
    t.whole = t.w + tile * 4u;
    t.bytes = t.whole + tile * 4u;
    return t;
}

template <int L, int NQ, int V>
__global__ void __launch_bounds__(kChunkWarps * 32) state_space_chunk_kernel(const __grid_constant__ StateSpace p) {
    extern __shared__ __align__(16) uint8_t smem[];
    const Columns<L, NQ, V> mine(p);
    constexpr uint32_t kWide = Columns<L, NQ, V>::kWide, kTile = chunk_tile<(int)kWide>();
    const uint32_t tid = threadIdx.x, threads = blockDim.x, lane = tid & 31u, columns = mine.count, c0 = mine.first, rows = p.rows;
    const ChunkLayout at = chunk_layout(kTile, kWide, columns);
    const uint32_t head = blockIdx.x, group = head / (p.heads / p.groups), np = mine.np, inner = p.inner(), x_row = p.x_row();
    const uint32_t base = *p.positions, slots = *p.slots;
    const size_t slot_elements = p.slot_elements();
    float* states = static_cast<float*>(const_cast<void*>(p.rings->ring_k)) + (size_t)head * p.vdim * np;
    Pair s[V][2 * NQ];
    mine.load(s, states + (base % slots) * slot_elements, base > 0u);
    const float skip = p.skip[head];

    auto fill = [&](uint32_t tile, uint32_t stage) {                   // zeros behind the chunk's rows
        uint8_t* to = smem + stage * at.stage;
        const uint32_t first = tile * kTile;
        for (uint32_t i = tid; i < kTile * (kWide / 4u); i += threads) {
            const uint32_t t = i / (kWide / 4u), n = i % (kWide / 4u) * 4u, row = first + t;
            const bool valid = row < rows && n < np;
            const size_t from = valid ? ((size_t)row * p.groups + group) * np + n : 0u;
            copy16(to + (t * kWide + n) * 4u, p.b + from, valid);
            copy16(to + at.c + (t * kWide + n) * 4u, p.c + from, valid);
        }
        for (uint32_t i = tid; i < kTile * (columns / 4u); i += threads) {
            const uint32_t t = i / (columns / 4u), k = i % (columns / 4u) * 4u, row = first + t;
            const bool valid = row < rows && c0 + k < x_row;
            copy16(to + at.x + (t * columns + k) * 4u, p.x + (valid ? ((size_t)row * p.heads + head) * x_row + c0 + k : 0u), valid);
        }
        if (tid < kTile) {
            const bool valid = first + tid < rows;
            const size_t row = valid ? first + tid : 0u;
            copy16(to + at.cb + tid * 16u, p.cb + (row * p.groups + group) * 4u, valid);
            copy8(to + at.steps + tid * 8u, p.steps + row * p.heads + head, valid);
        }
        copies_commit();
    };
    const uint32_t tiles = (rows + kTile - 1u) / kTile;
    const uint32_t lane_at = lane_first<L, V>(lane);                   // the values of every four tokens that this lane writes
    const bool writes = mine.ln % lane_copies<L, V>() == 0u;
    float* out = p.out + (size_t)(lane_at / V) * inner + head * p.vdim + c0 + mine.local + lane_at % V;
    fill(0u, 0u);
    for (uint32_t tile = 0; tile < tiles; ++tile) {
        const uint32_t first = tile * kTile;
        if (tile + 1u < tiles) fill(tile + 1u, (tile + 1u) & 1u);
        else copies_commit();
        copies_wait<1>();
        __syncthreads();
        const uint8_t* from = smem + (tile & 1u) * at.stage;
        const float *b = reinterpret_cast<const float*>(from), *c = reinterpret_cast<const float*>(from + at.c), *x = reinterpret_cast<const float*>(from + at.x);
        float4* m = reinterpret_cast<float4*>(smem + at.m);            // of x_0 .. x_3 of the four tokens, in y_t
        float *u = reinterpret_cast<float*>(smem + at.u), *w = reinterpret_cast<float*>(smem + at.w), *whole = reinterpret_cast<float*>(smem + at.whole);
        Pair* doubled = reinterpret_cast<Pair*>(smem + at.doubled);    // w_t x_t, twice
        if (tid < kTile) {
            const float2* steps = reinterpret_cast<const float2*>(from + at.steps) + (tid & ~3u);
            const float* cb = reinterpret_cast<const float*>(from + at.cb) + tid * 4u;
            const uint32_t q = tid & 3u;
            float factors[4], behind = 0.0f, rest = 0.0f;              // sums of logarithms: (s, q], and (q, 3]
#pragma unroll
            for (int i = 3; i >= 0; --i) {
                factors[i] = 0.0f;
                if ((uint32_t)i > q) { rest += steps[i].y; continue; }
                factors[i] = cb[i] * expf(behind) * steps[i].x;
                if ((uint32_t)i == q) factors[i] += skip;
                behind += steps[i].y;
            }
            m[tid] = make_float4(factors[0], factors[1], factors[2], factors[3]);
            u[tid] = expf(behind);
            w[tid] = expf(rest) * steps[q].x;
            whole[tid] = expf(behind + rest);
        }
        __syncthreads();
        for (uint32_t i = tid; i < kTile * columns; i += threads) {
            const float v = x[i] * w[i / columns];
            doubled[i] = pair_of(v, v);
        }
        __syncthreads();
#pragma unroll 1
        for (uint32_t t4 = 0; t4 < kTile && first + t4 < rows; t4 += 4u) {
            Pair xw[4][V], sum[4][V];
#pragma unroll
            for (int q = 0; q < 4; ++q)
#pragma unroll
                for (int v = 0; v < V; v += 2) {
                    const ulonglong2 two = *reinterpret_cast<const ulonglong2*>(doubled + (t4 + q) * columns + mine.local + v);
                    xw[q][v] = two.x;
                    xw[q][v + 1] = two.y;
                }
            const float decay = whole[t4 + 3u];
            const Pair a = pair_of(decay, decay);
#pragma unroll
            for (int j = 0; j < NQ; ++j) {
                ulonglong2 bq[4], cq[4];
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    cq[q] = *reinterpret_cast<const ulonglong2*>(c + (t4 + q) * kWide + mine.n(j));
                    bq[q] = *reinterpret_cast<const ulonglong2*>(b + (t4 + q) * kWide + mine.n(j));
                }
#pragma unroll
                for (int v = 0; v < V; ++v) {
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        sum[q][v] = j == 0 ? pair_mul(s[v][0], cq[q].x) : pair_fma(s[v][2 * j], cq[q].x, sum[q][v]);
                        sum[q][v] = pair_fma(s[v][2 * j + 1], cq[q].y, sum[q][v]);
                    }
                    s[v][2 * j] = pair_mul(s[v][2 * j], a);
                    s[v][2 * j + 1] = pair_mul(s[v][2 * j + 1], a);
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        s[v][2 * j] = pair_fma(bq[q].x, xw[q][v], s[v][2 * j]);
                        s[v][2 * j + 1] = pair_fma(bq[q].y, xw[q][v], s[v][2 * j + 1]);
                    }
                }
            }
            float part[4 * V];
#pragma unroll
            for (int i = 0; i < 4 * V; ++i) part[i] = pair_sum(sum[i / V][i % V]);
            lane_sums<L, V>(part, lane);
#pragma unroll
            for (uint32_t i = 0; i < lane_values<L, V>(); ++i) {
                const uint32_t t = t4 + (lane_at + i) / V, k = mine.local + (lane_at + i) % V;
                if (!writes || first + t >= rows || c0 + k >= p.vdim) continue;
                const float4 f = m[t];
                const float* x4 = x + t4 * columns + k;
                float y = u[t] * part[i];
                y = fmaf(f.x, x4[0], y);
                y = fmaf(f.y, x4[columns], y);
                y = fmaf(f.z, x4[2u * columns], y);
                out[((t4 + i / V) * inner) + i % V] = fmaf(f.w, x4[3u * columns], y);
            }
        }
        out += (size_t)kTile * inner;
        __syncthreads();                                               // the tile's buffers are free again
    }
    mine.store(s, states + ((base + rows) % slots) * slot_elements);
    keep_inputs(p, p.raw, static_cast<float*>(const_cast<void*>(p.rings->ring_v)), base, rows - min(rows, p.tap_count - 1u), rows, head, c0, columns);
}

// The convolved inputs of eight rows, padding included: the first blocks take a group's B and C, its heads' steps, and
// the products C_t . B_s within every four tokens; the others columns of x.
constexpr uint32_t kConvolveRows = 8, kConvolveThreads = 256;

// Eight rows of one channel: emit(row, value).  T: taps at most (0: any number).
template <int T, typename Emit>
__device__ __forceinline__ void convolve_rows(const StateSpace& p, const float* ring, uint32_t base, uint32_t row, uint32_t live, uint32_t channel, Emit emit) {
    if constexpr (T == 0) {
        for (uint32_t r = 0; r < live; ++r) emit(r, convolve<false>(p, p.raw, ring, base, row + r, channel));
    } else {
    constexpr int kBack = T - 1;
    float v[kBack + (int)kConvolveRows], w[T];
    const float* raw = p.raw + p.inner() + channel;
    if (row >= (uint32_t)kBack && live == kConvolveRows) {
        const float* from = raw + (size_t)(row - kBack) * p.raw_ld;
#pragma unroll
        for (int i = 0; i < kBack + (int)kConvolveRows; ++i) v[i] = from[(size_t)i * p.raw_ld];
    } else
#pragma unroll
    for (int i = 0; i < kBack + (int)kConvolveRows; ++i) {
        const int r = (int)row + i - kBack;                            // a row of the chunk, or behind it
        v[i] = 0.0f;
        if (i < kBack && (uint32_t)(kBack - i) >= p.tap_count) continue;
        if (r >= 0) { if ((uint32_t)r < row + live) v[i] = raw[(size_t)r * p.raw_ld]; }
        else if (base >= (uint32_t)-r) v[i] = ring[(size_t)((base + (uint32_t)r) & p.input_mask) * p.input_row() + channel];
    }
#pragma unroll
    for (int j = 0; j < T; ++j) w[j] = (uint32_t)j < p.tap_count ? p.taps[(size_t)channel * p.tap_count + p.tap_count - 1u - j] : 0.0f;
    const float bias = p.tap_bias[channel];
#pragma unroll
    for (int r = 0; r < (int)kConvolveRows; ++r) {
        if ((uint32_t)r >= live) break;
        float sum = 0.0f;
#pragma unroll
        for (int j = T - 1; j >= 0; --j) sum = fmaf(w[j], v[kBack + r - j], sum);
        emit((uint32_t)r, silu(sum + bias));
    }
    }
}

template <int T>
__global__ void __launch_bounds__(kConvolveThreads) convolve_chunk_kernel(const __grid_constant__ StateSpace p) {
    extern __shared__ float vectors[];                                 // [2][8][np]: B, C
    const uint32_t np = p.state_row(), x_row = p.x_row(), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t base = p.positions[0], row = blockIdx.y * kConvolveRows, live = min(kConvolveRows, p.rows - row);
    const float* ring = static_cast<const float*>(p.rings->ring_v);
    if (blockIdx.x >= p.groups) {
        const uint32_t i = (blockIdx.x - p.groups) * kConvolveThreads + tid, all = p.heads * x_row, k = i % x_row;
        if (i >= all) return;
        float* out = p.x + (size_t)row * all + i;
        if (k >= p.vdim) {
            for (uint32_t r = 0; r < live; ++r) out[(size_t)r * all] = 0.0f;
            return;
        }
        convolve_rows<T>(p, ring, base, row, live, i / x_row * p.vdim + k, [&](uint32_t r, float v) { out[(size_t)r * all] = v; });
        return;
    }
    const uint32_t group = blockIdx.x, per_group = p.heads / p.groups;
    for (uint32_t i = tid; i < 2u * np; i += kConvolveThreads) {
        const uint32_t which = i / np, n = i % np;
        float *out = (which ? p.c : p.b) + ((size_t)row * p.groups + group) * np + n, *here = vectors + which * kConvolveRows * np + n;
        if (n >= p.state) {
            for (uint32_t r = 0; r < kConvolveRows; ++r) { here[r * np] = 0.0f; if (r < live) out[(size_t)r * p.groups * np] = 0.0f; }
            continue;
        }
        for (uint32_t r = live; r < kConvolveRows; ++r) here[r * np] = 0.0f;
        convolve_rows<T>(p, ring, base, row, live, p.inner() + (which * p.groups + group) * p.state + n, [&](uint32_t r, float v) {
            here[r * np] = v;
            out[(size_t)r * p.groups * np] = v;
        });
    }
    for (uint32_t i = tid; i < live * per_group; i += kConvolveThreads) {
        const uint32_t r = row + i / per_group, head = group * per_group + i % per_group;
        p.steps[(size_t)r * p.heads + head] = step_of(p, p.raw, r, head);
    }
    __syncthreads();
    for (uint32_t i = warp; i < kConvolveRows * 4u; i += kConvolveThreads / 32u) {
        const uint32_t t = i / 4u, s = i % 4u;
        if (t >= live) break;
        const float *b = vectors + ((t & ~3u) + s) * np, *c = vectors + (kConvolveRows + t) * np;
        float sum = 0.0f;
        if (s <= (t & 3u))
            for (uint32_t n = lane; n < np; n += 32u) sum = fmaf(c[n], b[n], sum);
        sum = warp_sum(sum);
        if (lane == 0) p.cb[((size_t)(row + t) * p.groups + group) * 4u + s] = sum;
    }
}

// ------------------------------------------------------------------ launches

template <typename Kernel>
int allow_smem(Kernel kernel, std::once_flag* once, uint32_t bytes) {
    int device = 0;
    cudaGetDevice(&device);
    cudaError_t error = cudaSuccess;
    std::call_once(once[device & 63], [&] { error = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes); });
    GF_CUDA(error);
    return GF_OK;
}

template <int L, int NQ, int V, bool kPass>
int launch_recurrence(const StateSpace& p, cudaStream_t stream, bool pdl) {
    constexpr uint32_t kWide = L * NQ * 4, per_warp = 32u / L * V;
    static std::once_flag once[64];
    int status = GF_OK;
    if constexpr (kPass) status = allow_smem(state_space_rows_kernel<L, NQ, V>, once, kSmemLimit);
    else status = allow_smem(state_space_chunk_kernel<L, NQ, V>, once, kSmemLimit);
    if (status != GF_OK) return status;
    // As many warps per block as still give most SMs a block; the block's columns are whole 16-byte pieces.
    const uint32_t sequences = p.ring_stride ? p.rows : 1u;
    uint32_t warps = kPass ? kMaxWarps : kChunkWarps;
    while (warps > 1u && (warps / 2u) * per_warp % 4u == 0u
           && ((uint64_t)p.heads * sequences * ((p.vdim + warps * per_warp - 1u) / (warps * per_warp)) * 5u < (uint64_t)sm_count() * 4u
               || (warps / 2u) * per_warp >= p.vdim))
        warps /= 2u;
    while (!kPass && warps > 1u && chunk_layout(chunk_tile<(int)kWide>(), kWide, warps * per_warp).bytes > kSmemLimit) warps /= 2u;
    const uint32_t columns = warps * per_warp;
    const dim3 grid(p.heads, (p.vdim + columns - 1u) / columns, sequences);
    if constexpr (kPass) return launch_kernel(state_space_rows_kernel<L, NQ, V>, grid, dim3(warps * 32u), pass_smem(kWide, columns), stream, pdl, p);
    else return launch_kernel(state_space_chunk_kernel<L, NQ, V>, grid, dim3(warps * 32u), chunk_layout(chunk_tile<(int)kWide>(), kWide, columns).bytes, stream, pdl, p);
}

// Chunks hold half the columns a lane: twice the warps hide more of one another's waits.
template <bool kPass>
int launch_by_state(const StateSpace& p, cudaStream_t stream, bool pdl) {
    constexpr int V = kPass ? 4 : 2;
    const uint32_t fours = p.state_row() / 4u;
    if (fours <= 1u) return launch_recurrence<1, 1, V, kPass>(p, stream, pdl);
    if (fours <= 2u) return launch_recurrence<1, 2, V, kPass>(p, stream, pdl);
    if (fours <= 4u) return launch_recurrence<2, 2, V, kPass>(p, stream, pdl);
    if (fours <= 8u) return launch_recurrence<4, 2, V, kPass>(p, stream, pdl);
    if (fours <= 16u) return launch_recurrence<8, 2, V, kPass>(p, stream, pdl);
    if (fours <= 32u) return launch_recurrence<16, 2, V, kPass>(p, stream, pdl);
    if (fours <= 64u) return launch_recurrence<32, 2, V, kPass>(p, stream, pdl);
    if (fours <= 128u) return launch_recurrence<32, 4, V, kPass>(p, stream, pdl);
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
    if (!usable(p) || p.ring_stride || !p.x || !p.b || !p.c || !p.steps || !p.cb || p.input_mask + 1u < p.tap_count - 1u) return fail(GF_ERR_INVALID, "state space: bad arguments");
    const dim3 grid(p.groups + (p.heads * p.x_row() + kConvolveThreads - 1u) / kConvolveThreads, (p.rows + kConvolveRows - 1u) / kConvolveRows);
    const uint32_t smem = 2u * kConvolveRows * p.state_row() * 4u;
    static std::once_flag once[3][64];
    int status = allow_smem(convolve_chunk_kernel<4>, once[0], 2u * kConvolveRows * kMaxStateSize * 4u);
    if (status == GF_OK) status = allow_smem(convolve_chunk_kernel<8>, once[1], 2u * kConvolveRows * kMaxStateSize * 4u);
    if (status == GF_OK) status = allow_smem(convolve_chunk_kernel<0>, once[2], 2u * kConvolveRows * kMaxStateSize * 4u);
    if (status != GF_OK) return status;
    if (p.tap_count <= 4u) convolve_chunk_kernel<4><<<grid, kConvolveThreads, smem, stream>>>(p);
    else if (p.tap_count <= 8u) convolve_chunk_kernel<8><<<grid, kConvolveThreads, smem, stream>>>(p);
    else convolve_chunk_kernel<0><<<grid, kConvolveThreads, smem, stream>>>(p);
    GF_CUDA(cudaGetLastError());
    return launch_by_state<false>(p, stream, false);
}

}  // namespace gf
