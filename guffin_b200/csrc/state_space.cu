// State-space mixer (see state_space.cuh).
#include "state_space.cuh"
#include "tcgen05.cuh"

#include <algorithm>
#include <mutex>

namespace gf {

namespace {

constexpr uint32_t kMaxWarps = 4, kChunkWarps = 16;
constexpr uint32_t kSmemLimit = 160u * 1024u, kChunkSmem = 200u * 1024u;

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

// Sums part[0 .. M) over the L lanes that share a column: every round halves the values a lane is left with, so that
// part[0 .. lane_values()) hold the sums of values lane_first(lane) on.  Lanes left with the same value: the first writes.
template <int L, int M> constexpr uint32_t lane_values() { return L >= M ? 1u : (uint32_t)(M / L); }
template <int L, int M> constexpr uint32_t lane_copies() { return L > M ? (uint32_t)(L / M) : 1u; }
template <int L, int M>
__device__ __forceinline__ uint32_t lane_first(uint32_t lane) { return lane % L / lane_copies<L, M>() * lane_values<L, M>(); }
template <int L, int M>
__device__ __forceinline__ void lane_sums(float (&part)[M], uint32_t lane) {
    uint32_t count = M;
#pragma unroll
    for (uint32_t o = L / 2u; o > 0u; o >>= 1) {
        const bool upper = (lane & o) != 0u;
        if (count > 1u) {
            count /= 2u;
#pragma unroll
            for (uint32_t i = 0; i < M / 2u; ++i) {
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
        lane_sums<L, 4 * V>(part, lane);
#pragma unroll
        for (uint32_t i = 0; i < lane_values<L, 4 * V>(); ++i) {
            const uint32_t at = lane_first<L, 4 * V>(lane) + i, t = at / V, k = mine.local + at % V;
            if (mine.ln % lane_copies<L, 4 * V>() || t >= live || c0 + k >= p.vdim) continue;
            p.out[(size_t)(row0 + first + t) * inner + head * p.vdim + c0 + k] = fmaf(skip, x[t * columns + k], part[i]) * silu(gate[t * columns + k]);
        }
        __syncthreads();                                               // the tile's buffers are free again
    }
    keep_inputs(p, raw, ring, base, 0u, rows, head, c0, columns);
}

// ------------------------------------------------------------------ chunks

// Eight tokens at a time.  With a_t the logarithm of token t's decay and A_t their sums within the eight,
//   y_t = exp(A_t) S . C_t + sum over s <= t of M_ts x_s        M_ts = exp(A_t - A_s) dt_s (C_t . B_s), plus skip for s = t
//   S  <- exp(A_7) S + sum over s of exp(A_7 - A_s) dt_s x_s B_s^T
// as products on the tensor cores, in pairs of tf32 values (a value's leading bits and what they leave out) so that they
// are as exact as f32 ones.  A warp keeps 16 columns (of vdim) x 8 NT values (of N) of the state in accumulators, which
// are the first operand of the read-out as they lie: an accumulator's neighbouring columns 2 t and 2 t + 1 count as the
// operand's t and t + 4.  Helper warps have the next
// tile's inputs and factors copied and write the last tile's outputs meanwhile.
constexpr uint32_t kHelpers = 4;
struct ChunkLayout { uint32_t c, x, factors, stage, y, y_stage, bytes; };
__host__ __device__ inline ChunkLayout chunk_layout(const StateChunk& k) {      // bytes; two stages each of inputs and of outputs
    ChunkLayout t;
    t.c = k.tile * k.n_ld * 4u;
    t.x = 2u * t.c;
    t.factors = t.x + k.tile * k.x_ld * 4u;
    t.stage = t.factors + k.tile * kStateFactors * 4u;
    t.y = 2u * t.stage;
    t.y_stage = k.splits * k.tile * k.x_ld * 4u;
    t.bytes = t.y + 2u * t.y_stage;
    return t;
}

__device__ __forceinline__ void mma_tf32(float (&d)[4], const float (&a)[4], float b0, float b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])), "r"(__float_as_uint(b0)), "r"(__float_as_uint(b1)));
}
// The bits of a value that tf32 holds, and the rest.
__device__ __forceinline__ float leading(float v) { return __uint_as_float(__float_as_uint(v) & 0xffffe000u); }
struct Split4 {
    float hi[4], lo[4];
    __device__ __forceinline__ Split4(float a, float b, float c, float d) {
        const float v[4] = {a, b, c, d};
#pragma unroll
        for (int i = 0; i < 4; ++i) { hi[i] = leading(v[i]); lo[i] = v[i] - hi[i]; }
    }
};

template <int NT>
__global__ void __launch_bounds__((kChunkWarps + kHelpers) * 32) state_space_chunk_kernel(const __grid_constant__ StateSpace p, const __grid_constant__ StateChunk k) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ __align__(8) uint64_t full[2];                          // a stage's copies have landed
    __shared__ volatile uint32_t abort_flag;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, g = lane >> 2, t = lane & 3u, rows = p.rows;
    const ChunkLayout at = chunk_layout(k);
    const uint32_t head = blockIdx.x, c0 = blockIdx.y * k.columns, np = p.state_row(), inner = p.inner();
    const uint32_t workers = k.columns / 16u * k.splits, tiles = (rows + k.tile - 1u) / k.tile;
    const bool helper = warp >= workers;
    const uint32_t split = warp % k.splits, own = warp / k.splits * 16u;      // a worker's part of N, and its columns from c0 + own on
    const uint32_t base = *p.positions, slots = *p.slots;
    const size_t slot_elements = p.slot_elements();
    float* states = static_cast<float*>(const_cast<void*>(p.rings->ring_k)) + (size_t)head * p.vdim * np;
    float s[NT][4];
    auto state_at = [&](int j, int i) { return (size_t)(c0 + own + g + 8u * i) * np + (split * NT + j) * 8u + 2u * t; };
    auto state_valid = [&](int j, int i) { return !helper && c0 + own + g + 8u * i < p.vdim && (split * NT + j) * 8u + 2u * t < np; };
    {
        const float* from = states + (base % slots) * slot_elements;
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float2 v = base > 0u && state_valid(j, i) ? *reinterpret_cast<const float2*>(from + state_at(j, i)) : make_float2(0.0f, 0.0f);
                s[j][2 * i] = v.x;
                s[j][2 * i + 1] = v.y;
            }
    }
    const uint32_t all_rows = (rows + 7u) & ~7u;                        // the inputs have whole eights
    if (threadIdx.x == 0) {
        abort_flag = 0u;
        mbar_init(&full[0], 1);
        mbar_init(&full[1], 1);
        fence_barrier_init();
    }
    __syncthreads();
    // ---- helpers
    auto fill = [&](uint32_t tile) {                                   // one thread: a tile's rows follow one another
        uint8_t* to = smem + (tile & 1u) * at.stage;
        uint64_t* bar = &full[tile & 1u];
        const uint32_t first = tile * k.tile, count = min(k.tile, all_rows - first), group = head / (p.heads / p.groups);
        const size_t vectors = ((size_t)group * all_rows + first) * k.n_ld, columns = (((size_t)head * gridDim.y + blockIdx.y) * all_rows + first) * k.x_ld;
        mbar_expect_tx(bar, count * (2u * k.n_ld + k.x_ld + kStateFactors) * 4u);
        bulk_load(to, p.b + vectors, count * k.n_ld * 4u, bar);
        bulk_load(to + at.c, p.c + vectors, count * k.n_ld * 4u, bar);
        bulk_load(to + at.x, p.x + columns, count * k.x_ld * 4u, bar);
        bulk_load(to + at.factors, p.factors + ((size_t)head * all_rows + first) * kStateFactors, count * kStateFactors * 4u, bar);
    };
    auto write = [&](uint32_t tile) {
        const float* y = reinterpret_cast<const float*>(smem + at.y + (tile & 1u) * at.y_stage);
        const uint32_t first = tile * k.tile, count = min(k.tile, rows - first), quads = k.columns / 4u, part_step = k.tile * k.x_ld;
        for (uint32_t i = threadIdx.x - workers * 32u; i < count * quads; i += kHelpers * 32u) {
            const uint32_t r = i / quads, column = i % quads * 4u;
            const float* from = y + r * k.x_ld + column;
            float4 v = *reinterpret_cast<const float4*>(from);
#pragma unroll 4
            for (uint32_t part = 1; part < k.splits; ++part) {
                const float4 o = *reinterpret_cast<const float4*>(from + part * part_step);
                v = make_float4(v.x + o.x, v.y + o.y, v.z + o.z, v.w + o.w);
            }
            float* out = p.out + (size_t)(first + r) * inner + head * p.vdim + c0 + column;
            if (p.vdim % 4u == 0u) {
                if (c0 + column < p.vdim) *reinterpret_cast<float4*>(out) = v;
                continue;
            }
            const float four[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (uint32_t j = 0; j < 4u; ++j)
                if (c0 + column + j < p.vdim) out[j] = four[j];
        }
    };
    // ---- workers
    auto work = [&](uint32_t tile) {
        const uint8_t* from = smem + (tile & 1u) * at.stage;
        const float *b = reinterpret_cast<const float*>(from), *c = reinterpret_cast<const float*>(from + at.c), *x = reinterpret_cast<const float*>(from + at.x);
        const float* factors = reinterpret_cast<const float*>(from + at.factors);      // a row: M, exp(A_t), dt exp(A_7 - A_t), exp(A_7)
        float* y = reinterpret_cast<float*>(smem + at.y + (tile & 1u) * at.y_stage);
#pragma unroll 2
        for (uint32_t t0 = 0; t0 < k.tile && tile * k.tile + t0 < rows; t0 += 8u) {
            const float* x_at = x + (t0 + t) * k.x_ld + own + g;
            const float x0 = x_at[0], x1 = x_at[8], x2 = x_at[4u * k.x_ld], x3 = x_at[4u * k.x_ld + 8u];
            const float* eight = factors + t0 * kStateFactors;
            const float w0 = eight[t * kStateFactors + 9u], w1 = eight[(t + 4u) * kStateFactors + 9u], decay = eight[10];
            const Split4 xw(x0 * w0, x1 * w0, x2 * w1, x3 * w1);
            float y0[4] = {}, y1[4] = {}, y2[4] = {};
            const float *c_at = c + (t0 + g) * k.n_ld + split * NT * 8u + 2u * t, *b_at = b + (t0 + t) * k.n_ld + split * NT * 8u + g;
            float bh[NT][2], bl[NT][2];
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const float2 cv = *reinterpret_cast<const float2*>(c_at + j * 8);
                const float ch0 = leading(cv.x), ch1 = leading(cv.y);
                const Split4 state(s[j][0], s[j][2], s[j][1], s[j][3]);
                mma_tf32(y0, state.hi, ch0, ch1);
                mma_tf32(y1, state.hi, cv.x - ch0, cv.y - ch1);
                mma_tf32(y2, state.lo, ch0, ch1);
#pragma unroll
                for (int i = 0; i < 4; ++i) s[j][i] *= decay;
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const float v = b_at[j * 8 + i * 4u * k.n_ld];
                    bh[j][i] = leading(v);
                    bl[j][i] = v - bh[j][i];
                }
            }
            // Products into the same accumulators as far apart as there are accumulators.
#pragma unroll
            for (int j = 0; j < NT; ++j) mma_tf32(s[j], xw.hi, bh[j][0], bh[j][1]);
#pragma unroll
            for (int j = 0; j < NT; ++j) mma_tf32(s[j], xw.hi, bl[j][0], bl[j][1]);
#pragma unroll
            for (int j = 0; j < NT; ++j) mma_tf32(s[j], xw.lo, bh[j][0], bh[j][1]);
            const float u0 = eight[2u * t * kStateFactors + 8u], u1 = eight[(2u * t + 1u) * kStateFactors + 8u];
#pragma unroll
            for (int i = 0; i < 4; ++i) y0[i] = (y0[i] + (y1[i] + y2[i])) * (i & 1 ? u1 : u0);
            if (split < 3u) {                                          // the three terms, one a warp where there are as many
                const Split4 xs(x0, x1, x2, x3);
                const float m0 = eight[g * kStateFactors + t], m1 = eight[g * kStateFactors + t + 4u], mh0 = leading(m0), mh1 = leading(m1);
                if (split == 0u) mma_tf32(y0, xs.hi, mh0, mh1);
                if (k.splits < 3u ? split == 0u : split == 1u) mma_tf32(y0, xs.hi, m0 - mh0, m1 - mh1);
                if (k.splits < 3u ? split == 0u : split == 2u) mma_tf32(y0, xs.lo, mh0, mh1);
            }
            float* y_at = y + (split * k.tile + t0 + 2u * t) * k.x_ld + own + g;
            y_at[0] = y0[0];
            y_at[k.x_ld] = y0[1];
            y_at[8] = y0[2];
            y_at[k.x_ld + 8u] = y0[3];
        }
    };
    const bool copier = warp == workers && lane == 0u;
    if (copier) fill(0u);
    bool ok = true;
    for (uint32_t tile = 0; tile < tiles; ++tile) {
        if (helper) {
            if (copier && tile + 1u < tiles && abort_flag == 0u) fill(tile + 1u);
            __syncwarp();
            if (tile > 0u) write(tile - 1u);
        } else {
            if (ok && !wait_or_abort(&full[tile & 1u], (tile >> 1) & 1u, &abort_flag)) {
                ok = false;
                if (lane == 0) { abort_flag = 1u; atomicExch(p.error_flag, 1); }
            }
            work(tile);
        }
        __syncthreads();
    }
    if (abort_flag != 0u && copier)                                    // copies already requested get a bounded chance to land
        for (uint32_t tile = tiles > 2u ? tiles - 2u : 0u; tile < tiles; ++tile) mbar_wait(&full[tile & 1u], (tile >> 1) & 1u, 1u << 16);
    if (helper) {
        write(tiles - 1u);
    } else {
        float* to = states + ((base + rows) % slots) * slot_elements;
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int i = 0; i < 2; ++i)
                if (state_valid(j, i)) *reinterpret_cast<float2*>(to + state_at(j, i)) = make_float2(s[j][2 * i], s[j][2 * i + 1]);
    }
    keep_inputs(p, p.raw, static_cast<float*>(const_cast<void*>(p.rings->ring_v)), base, rows - min(rows, p.tap_count - 1u), rows, head, c0, k.columns);
}

// The convolved inputs of eight rows, padding and rows behind the chunk included (zeros): the first blocks take a group's B
// and C and the factors of its heads, the others columns of x.
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
        } else {
#pragma unroll
            for (int i = 0; i < kBack + (int)kConvolveRows; ++i) {
                const int r = (int)row + i - kBack;                    // a row of the chunk, or behind it
                v[i] = 0.0f;
                if (i < kBack && (uint32_t)(kBack - i) >= p.tap_count) continue;
                if (r >= 0) { if ((uint32_t)r < row + live) v[i] = raw[(size_t)r * p.raw_ld]; }
                else if (base >= (uint32_t)-r) v[i] = ring[(size_t)((base + (uint32_t)r) & p.input_mask) * p.input_row() + channel];
            }
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
__global__ void __launch_bounds__(kConvolveThreads) convolve_chunk_kernel(const __grid_constant__ StateSpace p, const __grid_constant__ StateChunk k) {
    extern __shared__ float vectors[];                                 // [2][8][n_ld]: B, C
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t base = p.positions[0], row = blockIdx.y * kConvolveRows, live = min(kConvolveRows, p.rows - row), all_rows = (p.rows + 7u) & ~7u;
    const float* ring = static_cast<const float*>(p.rings->ring_v);
    if (blockIdx.x >= p.groups) {
        const uint32_t i = (blockIdx.x - p.groups) * kConvolveThreads + tid, blocks = (p.vdim + k.columns - 1u) / k.columns;
        const uint32_t head_block = i / k.x_ld, c = i % k.x_ld, head = head_block / blocks, column = head_block % blocks * k.columns + c;
        if (head >= p.heads) return;
        float* out = p.x + ((size_t)head_block * all_rows + row) * k.x_ld + c;
        const bool valid = c < k.columns && column < p.vdim;
        for (uint32_t r = valid ? live : 0u; r < kConvolveRows; ++r) out[r * k.x_ld] = 0.0f;
        if (valid) convolve_rows<T>(p, ring, base, row, live, head * p.vdim + column, [&](uint32_t r, float v) { out[r * k.x_ld] = v; });
        return;
    }
    const uint32_t group = blockIdx.x, per_group = p.heads / p.groups, np = k.n_ld;
    // The steps of the first heads stay in shared memory.
    constexpr uint32_t kNear = 64;
    __shared__ float2 near[kConvolveRows * kNear];
    for (uint32_t i = tid; i < kConvolveRows * per_group; i += kConvolveThreads) {
        const uint32_t r = i / per_group, h = i % per_group;
        const float2 step = r < live ? step_of(p, p.raw, row + r, group * per_group + h) : make_float2(0.0f, 0.0f);
        if (h < kNear) near[r * kNear + h] = step;
        else p.steps[(size_t)(row + r) * p.heads + group * per_group + h] = step;
    }
    for (uint32_t i = tid; i < 2u * np; i += kConvolveThreads) {
        const uint32_t which = i / np, n = i % np;
        float *out = (which ? p.c : p.b) + ((size_t)group * all_rows + row) * np + n, *here = vectors + which * kConvolveRows * np + n;
        const bool valid = n < p.state;
        for (uint32_t r = valid ? live : 0u; r < kConvolveRows; ++r) { here[r * np] = 0.0f; out[r * np] = 0.0f; }
        if (!valid) continue;
        convolve_rows<T>(p, ring, base, row, live, p.inner() + (which * p.groups + group) * p.state + n, [&](uint32_t r, float v) {
            here[r * np] = v;
            out[r * np] = v;
        });
    }
    __shared__ float cb[kConvolveRows * 8u];
    __syncthreads();
    for (uint32_t i = warp; i < kConvolveRows * 8u; i += kConvolveThreads / 32u) {
        const uint32_t t = i / 8u, other = i % 8u;
        if (other > t) continue;
        const float *b = vectors + other * np, *c = vectors + (kConvolveRows + t) * np;
        float sum = 0.0f;
        for (uint32_t n = lane; n < np; n += 32u) sum = fmaf(c[n], b[n], sum);
        sum = warp_sum(sum);
        if (lane == 0) cb[i] = sum;
    }
    __syncthreads();
    // The factors of every head: element (t, s) of M, and with s = t the row's exponentials.
    for (uint32_t i = tid; i < per_group * kConvolveRows * 8u; i += kConvolveThreads) {
        const uint32_t h = i / (kConvolveRows * 8u), head = group * per_group + h, t = i / 8u % kConvolveRows, s = i % 8u;
        float between = 0.0f, before = 0.0f, behind = 0.0f, dt = 0.0f;
#pragma unroll
        for (uint32_t l = 0; l < 8u; ++l) {
            const float2 step = h < kNear ? near[l * kNear + h] : p.steps[(size_t)(row + l) * p.heads + head];
            if (l > s && l <= t) between += step.y;
            (l <= t ? before : behind) += step.y;
            if (l == s) dt = step.x;
        }
        float* out = p.factors + ((size_t)head * all_rows + row + t) * kStateFactors;
        out[s] = s > t ? 0.0f : fmaf(cb[t * 8u + s] * dt, expf(between), s == t ? p.skip[head] : 0.0f);
        if (s != t) continue;
        *reinterpret_cast<float4*>(out + 8) = make_float4(expf(before), expf(behind) * dt, expf(before + behind), 0.0f);
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

template <int L, int NQ, int V>
int launch_rows(const StateSpace& p, cudaStream_t stream, bool pdl) {
    constexpr uint32_t kWide = L * NQ * 4, per_warp = 32u / L * V;
    static std::once_flag once[64];
    const int status = allow_smem(state_space_rows_kernel<L, NQ, V>, once, kSmemLimit);
    if (status != GF_OK) return status;
    // As many warps per block as still give most SMs a block; the block's columns are whole 16-byte pieces.
    const uint32_t sequences = p.ring_stride ? p.rows : 1u;
    uint32_t warps = kMaxWarps;
    while (warps > 1u && (warps / 2u) * per_warp % 4u == 0u
           && ((uint64_t)p.heads * sequences * ((p.vdim + warps * per_warp - 1u) / (warps * per_warp)) * 5u < (uint64_t)sm_count() * 4u
               || (warps / 2u) * per_warp >= p.vdim))
        warps /= 2u;
    const uint32_t columns = warps * per_warp;
    return launch_kernel(state_space_rows_kernel<L, NQ, V>, dim3(p.heads, (p.vdim + columns - 1u) / columns, sequences), dim3(warps * 32u), pass_smem(kWide, columns),
                         stream, pdl, p);
}

template <int NT>
int launch_chunk(const StateSpace& p, const StateChunk& k, cudaStream_t stream) {
    static std::once_flag once[64];
    const int status = allow_smem(state_space_chunk_kernel<NT>, once, kChunkSmem);
    if (status != GF_OK) return status;
    state_space_chunk_kernel<NT><<<dim3(p.heads, (p.vdim + k.columns - 1u) / k.columns), (k.columns / 16u * k.splits + kHelpers) * 32u, chunk_layout(k).bytes, stream>>>(p, k);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
}

template <int T>
int launch_convolution(const StateSpace& p, const StateChunk& k, cudaStream_t stream) {
    static std::once_flag once[64];
    const int status = allow_smem(convolve_chunk_kernel<T>, once, kChunkSmem);
    if (status != GF_OK) return status;
    const uint32_t x_all = p.heads * ((p.vdim + k.columns - 1u) / k.columns) * k.x_ld;
    convolve_chunk_kernel<T><<<dim3(p.groups + (x_all + kConvolveThreads - 1u) / kConvolveThreads, (p.rows + kConvolveRows - 1u) / kConvolveRows), kConvolveThreads,
                               2u * kConvolveRows * k.n_ld * 4u, stream>>>(p, k);
    GF_CUDA(cudaGetLastError());
    return GF_OK;
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
    const uint32_t fours = p.state_row() / 4u;
    if (fours <= 1u) return launch_rows<1, 1, 4>(p, stream, pdl);
    if (fours <= 2u) return launch_rows<1, 2, 4>(p, stream, pdl);
    if (fours <= 4u) return launch_rows<2, 2, 4>(p, stream, pdl);
    if (fours <= 8u) return launch_rows<4, 2, 4>(p, stream, pdl);
    if (fours <= 16u) return launch_rows<8, 2, 4>(p, stream, pdl);
    if (fours <= 32u) return launch_rows<16, 2, 4>(p, stream, pdl);
    if (fours <= 64u) return launch_rows<32, 2, 4>(p, stream, pdl);
    if (fours <= 128u) return launch_rows<32, 4, 4>(p, stream, pdl);
    return launch_rows<32, 8, 2>(p, stream, pdl);
}

StateChunk state_space_chunk(const StateSpace& p) {
    StateChunk k;
    k.per_warp = p.state <= 8u ? 8u : p.state <= 16u ? 16u : p.state <= 256u ? 32u : 64u;
    k.splits = (p.state + k.per_warp - 1u) / k.per_warp;
    uint32_t sixteens = std::max(1u, std::min((p.vdim + 15u) / 16u, kChunkWarps / k.splits));
    while (sixteens > 1u && (uint64_t)p.heads * ((p.vdim + sixteens * 16u - 1u) / (sixteens * 16u)) * 5u < (uint64_t)sm_count() * 4u) sixteens = (sixteens + 1u) / 2u;
    k.columns = sixteens * 16u;
    // Row lengths that put a fragment's lanes into different banks.
    k.n_ld = k.splits * k.per_warp + 8u;
    k.x_ld = k.columns + 8u;
    k.tile = 32u;
    while (k.tile > 8u && chunk_layout(k).bytes > kChunkSmem) k.tile /= 2u;
    return k;
}

int launch_state_space_chunk(const StateSpace& p, cudaStream_t stream) {
    if (!usable(p) || p.ring_stride || !p.x || !p.b || !p.c || !p.steps || !p.factors || !p.error_flag || p.input_mask + 1u < p.tap_count - 1u)
        return fail(GF_ERR_INVALID, "state space: bad arguments");
    const StateChunk k = state_space_chunk(p);
    const int status = p.tap_count <= 4u ? launch_convolution<4>(p, k, stream) : p.tap_count <= 8u ? launch_convolution<8>(p, k, stream) : launch_convolution<0>(p, k, stream);
    if (status != GF_OK) return status;
    switch (k.per_warp) {
        case 8u: return launch_chunk<1>(p, k, stream);
        case 16u: return launch_chunk<2>(p, k, stream);
        case 32u: return launch_chunk<4>(p, k, stream);
        default: return launch_chunk<8>(p, k, stream);
    }
}

}  // namespace gf
