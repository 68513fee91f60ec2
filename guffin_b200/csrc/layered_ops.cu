// C entry points of the layered models' operators (tests, single-kernel measurements, hosts with schedules of their own).
#include "latent.cuh"

#include <algorithm>

using namespace gf;

namespace {

// A launch's give-up word, one per device.
int device_flag(int** out) {
    static int* flags[64] = {nullptr};
    int device = 0;
    GF_CUDA(cudaGetDevice(&device));
    device &= 63;
    if (!flags[device]) {
        GF_CUDA(cudaMalloc(&flags[device], sizeof(int)));
        GF_CUDA(cudaMemset(flags[device], 0, sizeof(int)));
    }
    *out = flags[device];
    return GF_OK;
}

Operand chunk_operand(uint32_t rows, uint32_t k, int precision, void* data) {
    Operand o;
    o.capacity = (rows + 15u) / 16u * 16u;
    o.k_pad = (k + kDenseBlockK - 1u) / kDenseBlockK * kDenseBlockK;
    o.f32 = precision == GF_PRECISION_F32 ? 1u : 0u;
    o.data = data;
    return o;
}

}  // namespace

#define GF_TRY(expr) do { const int gf_s_ = (expr); if (gf_s_ != GF_OK) return gf_s_; } while (0)

extern "C" {

size_t gf_dense_packed_bytes(uint32_t k, uint32_t n) {
    DenseMatrix m;
    m.k = k; m.n = n;
    return m.bytes();
}

int gf_dense_pack(const uint16_t* bf16_dev, uint32_t k, uint32_t n, void* packed_dev, void* stream) {
    if (!bf16_dev || !packed_dev || k == 0 || n == 0) return fail(GF_ERR_INVALID, "gf_dense_pack: bad arguments");
    GF_CUDA(cudaMemsetAsync(packed_dev, 0, gf_dense_packed_bytes(k, n), as_stream(stream)));
    DensePack p {};
    p.src = bf16_dev; p.dst = static_cast<uint8_t*>(packed_dev);
    p.n_stride = k; p.k_stride = 1; p.count = 1; p.n = n; p.k = k; p.k_blocks = (k + kDenseBlockK - 1u) / kDenseBlockK; p.group_step = 1;
    return launch_dense_pack(p, as_stream(stream));
}

int gf_dense_matmul(const void* packed_dev, const float* x_dev, float* y_dev, uint32_t rows, uint32_t k, uint32_t n, void* stream) {
    if (!packed_dev || !x_dev || !y_dev || rows == 0) return fail(GF_ERR_INVALID, "gf_dense_matmul: bad arguments");
    RowProduct p;
    p.rows = rows; p.in = x_dev; p.in_ld = k;
    p.m[0].weight = static_cast<const uint8_t*>(packed_dev); p.m[0].k = k; p.m[0].n = n; p.m[0].out = y_dev; p.m[0].out_ld = n;
    uint32_t launches = 0;
    return launch_row_product(p, as_stream(stream), false, launches);
}

size_t gf_dense_chunk_workspace_bytes(uint32_t rows, uint32_t k, int precision) { return chunk_operand(rows, k, precision, nullptr).bytes(); }

int gf_dense_chunk_matmul(const void* packed_dev, const float* x_dev, float* y_dev, uint32_t rows, uint32_t k, uint32_t n, int precision,
                          void* workspace_dev, void* stream) {
    if (!packed_dev || !x_dev || !y_dev || !workspace_dev || rows == 0 || k == 0 || n == 0) return fail(GF_ERR_INVALID, "gf_dense_chunk_matmul: bad arguments");
    int* flag = nullptr;
    GF_TRY(device_flag(&flag));
    ChunkProduct product;
    product.rows = rows; product.error_flag = flag;
    ChunkProblem& m = product.p[0];
    m.weight = static_cast<const uint8_t*>(packed_dev); m.k = k; m.n = n; m.out = y_dev; m.out_ld = n;
    m.a = chunk_operand(rows, k, precision, workspace_dev);
    GF_TRY(launch_chunk_operand(x_dev, rows, k, m.a, as_stream(stream)));
    GF_TRY(launch_chunk_product(product, precision == GF_PRECISION_F32, as_stream(stream)));
    int value = 0;
    GF_CUDA(cudaMemcpyAsync(&value, flag, sizeof(int), cudaMemcpyDeviceToHost, as_stream(stream)));
    GF_CUDA(cudaStreamSynchronize(as_stream(stream)));
    if (value == 0) return GF_OK;
    cudaMemsetAsync(flag, 0, sizeof(int), as_stream(stream));
    return fail(GF_ERR_TIMEOUT, "gf_dense_chunk_matmul: a bounded wait gave up");
}

size_t gf_latent_attention_workspace_bytes(uint32_t rows, uint32_t heads, uint32_t rank, uint32_t parts) {
    return (size_t)rows * heads * parts * (latent_row_elements(rank) + 2u) * sizeof(float) + 256u;
}

int gf_latent_attention(const void* q_dev, const void* ring_dev, const void* private_dev, const uint32_t* position_dev, const float* sink_dev,
                        float* out_dev, uint32_t rows, uint32_t heads, uint32_t rank, uint32_t ring_rows, uint32_t parts, int precision,
                        void* workspace_dev, void* stream) {
    if (!q_dev || !ring_dev || !private_dev || !position_dev || !out_dev || !workspace_dev || rows == 0 || heads == 0 || rank == 0 || ring_rows == 0
        || (ring_rows & (ring_rows - 1u)) || parts == 0 || parts > kLatentMaxParts)
        return fail(GF_ERR_INVALID, "gf_latent_attention: bad arguments (ring rows must be a power of two, parts at most %u)", kLatentMaxParts);
    cudaStream_t s = as_stream(stream);
    StreamRings* rings = static_cast<StreamRings*>(workspace_dev);          // its first 256 bytes
    const StreamRings host{ring_dev, nullptr};
    GF_CUDA(cudaMemcpyAsync(rings, &host, sizeof host, cudaMemcpyHostToDevice, s));
    LatentAttention p;
    p.q = q_dev; p.rings = rings; p.private_rows = private_dev; p.positions = position_dev; p.rows = rows; p.heads = heads;
    p.row_elements = latent_row_elements(rank); p.ring_mask = ring_rows - 1u; p.cache_f32 = precision == GF_PRECISION_F32 ? 1u : 0u;
    p.partial_out = reinterpret_cast<float*>(static_cast<uint8_t*>(workspace_dev) + 256u);
    p.partial_ml = p.partial_out + (size_t)rows * heads * parts * p.row_elements;
    p.parts = parts; p.sink = sink_dev;
    GF_TRY(launch_latent_attention(p, s, false));
    p.result.data = out_dev; p.result.capacity = rows; p.result.k_pad = heads * p.row_elements; p.result.f32 = 1; p.result_stride = p.row_elements;
    return launch_latent_merge(p, s);
}

int gf_route(const float* logits_dev, uint32_t rows, uint32_t experts, uint32_t top, uint32_t* ids_dev, float* scores_dev, void* stream) {
    if (!logits_dev || !ids_dev || !scores_dev) return fail(GF_ERR_INVALID, "gf_route: null argument");
    ChunkRoute p;
    p.logits = logits_dev; p.logits_ld = experts; p.rows = rows; p.experts = experts; p.top = top; p.slot_experts = ids_dev; p.slot_scores = scores_dev;
    return launch_route(p, as_stream(stream));
}

}  // extern "C"
