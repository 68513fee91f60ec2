// Layered models: weight binding and the schedules of a pass and of a prompt chunk (see layered.cuh).
//
// A pass of up to GF_MAX_ROWS rows, per layer (row_product launches unless said otherwise).  Latent attention:
//   q, latent     <- prologue: [residual + norm(previous sublayer)]; norm
//   latent query  <- per head, with the new cache rows stored beside it
//   attention over the cached latents (split over the keys)
//   values        <- per head; prologue: merge of the attention partitions and the sink
//   mixer output
// Grouped-query attention:
//   q, k, gates of the heads <- the same prologue
//   norm, rotation and the new cache rows; attention over the cached keys and values (split over the keys; the last block
//   merges, with sink and gate) -- one launch, two in 32-bit plans
//   mixer output
// State space:
//   input projection <- the same prologue
//   convolution, recurrence, gate
//   mixer output  <- prologue: norm in parts
// Feed-forward:
//   dense:   up (squared relu, or gate and up) <- prologue: residual + norm(mixer); norm          down
//   mixture: router, shared gate / up <- the same prologue     routed gate / up     routed and shared down
// A chunk of prompt rows runs the same steps as products over all its rows with small kernels between them.
#include "layered.cuh"
#include "model.cuh"

#include <algorithm>
#include <cmath>
#include <cstring>

#define GF_TRY(expr) do { const int gf_s_ = (expr); if (gf_s_ != GF_OK) return gf_s_; } while (0)

namespace gf {

template <typename T>
static int plan_alloc(std::vector<void*>& owner, T** out, size_t count) {
    void* p = nullptr;
    const size_t bytes = std::max<size_t>(count * sizeof(T), 256);
    GF_CUDA(cudaMalloc(&p, bytes));
    owner.push_back(p);
    GF_CUDA(cudaMemset(p, 0, bytes));          // padding of operands and rows is read and must be finite
    *out = static_cast<T*>(p);
    return GF_OK;
}
static int bytes_alloc(std::vector<void*>& owner, void** out, size_t bytes) {
    uint8_t* p = nullptr;
    GF_TRY(plan_alloc(owner, &p, bytes));
    *out = p;
    return GF_OK;
}

static uint32_t next_pow2(uint32_t v) {
    uint32_t p = 1;
    while (p < v) p <<= 1;
    return p;
}
static uint32_t round_up(uint32_t v, uint32_t to) { return (v + to - 1u) / to * to; }

// ------------------------------------------------------------------ binding

Model::Model(const ArchitectureDescription& description, uint32_t context, uint32_t row_capacity, bool f32) : config_ {} {
    layered_.reset(new LayeredPlan());
    LayeredPlan& p = *layered_;
    p.description = description;
    p.f32 = f32;
    const LayeredSpec& s = p.spec();
    p.layers.resize(s.layers.size());
    for (const TensorSlot& slot : p.description.tensors) p.slots[slot.name] = &slot;
    config_.hidden = s.width; config_.vocab = s.vocab; config_.layers = (uint32_t)s.layers.size();
    config_.heads = s.layers[0].mixer.heads; config_.kv_heads = 1;
    p.own_slots = row_capacity + 1u;
    config_.rms_eps = s.eps; config_.kv_f16 = f32 ? 0 : 1; config_.attention_scale = s.layers[0].mixer.scale;
    config_.context = context; config_.row_capacity = row_capacity;
    layers_.resize(config_.layers);
    caches_.resize(config_.layers);
}

// Allocates `count` packed matrices of [n][k] once; later tensors of the family find them.
static int ensure_matrix(std::vector<void*>& owner, DenseMatrix& m, uint32_t k, uint32_t n, uint32_t count, size_t& total) {
    if (m.data) return GF_OK;
    m.k = k; m.n = n;
    GF_TRY(plan_alloc(owner, &m.data, m.bytes() * count));
    total += m.bytes() * count;
    return GF_OK;
}

int Model::set_tensor(const char* name, int dtype, const void* host, const uint64_t* dims, uint32_t rank) {
    if (!layered_) return fail(GF_ERR_STATE, "gf_model_set_tensor: this plan's tensors are bound by kind (gf_model_set_matrix)");
    if (finalized_) return fail(GF_ERR_STATE, "gf_model_set_tensor: the plan is already finalized");
    if (!name || !host || !dims || rank == 0 || rank > 2) return fail(GF_ERR_INVALID, "gf_model_set_tensor: bad arguments");
    LayeredPlan& p = *layered_;
    const auto found = p.slots.find(name);
    if (found == p.slots.end()) return fail(GF_ERR_INVALID, "gf_model_set_tensor: this model has no tensor '%s'", name);
    const TensorSlot& slot = *found->second;
    if (p.bound[name]) return fail(GF_ERR_STATE, "gf_model_set_tensor: tensor '%s' bound twice", name);
    const bool vector = slot.rows == 0, constants = vector || slot.table;
    if (rank != (vector ? 1u : 2u) || dims[rank - 1u] != slot.columns || (!vector && dims[0] != slot.rows))
        return fail(GF_ERR_INVALID, "gf_model_set_tensor: tensor '%s' should have shape [%s%u]", name,
                    vector ? "" : (std::to_string(slot.rows) + ", ").c_str(), slot.columns);
    if (constants) {
        if (dtype != GF_BF16 && dtype != GF_F32) return fail(GF_ERR_INVALID, "gf_model_set_tensor: vector '%s' must be bf16 or f32", name);
        std::vector<float> values(slot.values());
        if (dtype == GF_F32) std::memcpy(values.data(), host, values.size() * 4u);
        else
            for (size_t i = 0; i < values.size(); ++i) {
                const uint32_t bits = (uint32_t)static_cast<const uint16_t*>(host)[i] << 16;
                std::memcpy(&values[i], &bits, 4u);
            }
        native_weight_bytes_ += values.size() * 4u;
        p.vectors[{slot.role, slot.layer}] = std::move(values);
        p.bound[name] = true;
        return GF_OK;
    }
    if (dtype != GF_BF16) return fail(GF_ERR_INVALID, "gf_model_set_tensor: matrix '%s' must be bf16", name);
    if (!stream_) GF_CUDA(cudaStreamCreateWithFlags(&stream_, cudaStreamNonBlocking));
    const LayeredSpec& s = p.spec();
    LayeredLayer& l = p.layers[slot.layer];
    const MixerSpec& m = s.layers[slot.layer].mixer;
    const FeedForwardSpec& f = s.layers[slot.layer].mlp;
    DensePack pack {};
    pack.n_stride = slot.columns; pack.k_stride = 1; pack.count = 1; pack.n = slot.rows; pack.k = slot.columns; pack.group_step = 1;
    DenseMatrix* dst = nullptr;
    uint32_t index = 0, columns = slot.rows, k = slot.columns, count = 1;
    const uint32_t paired = dense_paired_columns(f.ff), shared_paired = dense_paired_columns(f.shared_ff);
    auto half = [&](uint32_t stored, uint32_t first) { columns = stored; pack.group_step = 2; pack.group_first = first; };
    switch (slot.role) {
        case TensorRole::kEmbedding: dst = &p.table; break;
        case TensorRole::kHead: dst = &p.output_head; break;
        case TensorRole::kQuery: dst = &l.q; break;
        case TensorRole::kKey: dst = &l.k; break;
        case TensorRole::kHeadGate: dst = &l.head_gate; break;
        case TensorRole::kStateIn: dst = &l.state_in; break;
        case TensorRole::kLatentDown: dst = &l.latent_down; break;
        case TensorRole::kLatentUpKey:        // per head the transposed matrix: latent from query
            dst = &l.up_key; count = m.heads; k = m.dim; columns = m.rank;
            pack.count = m.heads; pack.n = m.rank; pack.k = m.dim; pack.count_stride = (size_t)m.dim * m.rank; pack.n_stride = 1; pack.k_stride = m.rank;
            break;
        case TensorRole::kLatentUpValue:
            dst = &l.up_value; count = m.heads; k = m.rank; columns = m.vdim;
            pack.count = m.heads; pack.n = m.vdim; pack.count_stride = (size_t)m.vdim * m.rank;
            break;
        case TensorRole::kMixerOut: dst = &l.o; break;
        case TensorRole::kGate: dst = &l.up; half(paired, 0); break;
        case TensorRole::kUp: dst = &l.up; if (f.activation == Activation::kGeluGate) half(paired, 1); break;
        case TensorRole::kDown: dst = &l.down; break;
        case TensorRole::kExpertGate: dst = &l.expert_up; index = slot.index; count = f.experts; half(paired, 0); break;
        case TensorRole::kExpertUp: dst = &l.expert_up; index = slot.index; count = f.experts; half(paired, 1); break;
        case TensorRole::kExpertDown: dst = &l.expert_down; index = slot.index; count = f.experts; break;
        case TensorRole::kRouter: dst = &l.router; break;
        case TensorRole::kSharedGate: dst = &l.shared_up; half(shared_paired, 0); break;
        case TensorRole::kSharedUp: dst = &l.shared_up; half(shared_paired, 1); break;
        case TensorRole::kSharedDown: dst = &l.shared_down; break;
        case TensorRole::kSharedWeight: dst = &l.shared_weight; break;
        default: return fail(GF_ERR_INVALID, "gf_model_set_tensor: '%s' is a vector", name);
    }
    GF_TRY(ensure_matrix(allocations_, *dst, k, columns, count, weight_bytes_));
    const size_t bytes = (size_t)slot.rows * slot.columns * 2u;
    uint8_t* staged = nullptr;
    uint32_t staging = 0;
    GF_TRY(stage_upload(host, bytes, &staged, &staging));
    pack.src = reinterpret_cast<const uint16_t*>(staged);
    pack.dst = dst->data + index * dst->bytes();
    pack.dst_stride = dst->bytes();
    pack.k_blocks = dst->k_blocks();
    GF_TRY(launch_dense_pack(pack, stream_));
    if (slot.role == TensorRole::kLatentUpKey && !p.f32) {
        GF_TRY(ensure_matrix(allocations_, l.expand_key, m.rank, m.heads * m.dim, 1, weight_bytes_));
        DensePack plain = pack;
        plain.dst = l.expand_key.data; plain.count = 1; plain.count_stride = 0; plain.n = m.heads * m.dim; plain.k = m.rank;
        plain.n_stride = m.rank; plain.k_stride = 1; plain.k_blocks = l.expand_key.k_blocks();
        GF_TRY(launch_dense_pack(plain, stream_));
    }
    GF_CUDA(cudaEventRecord(stager_.packed[staging], stream_));
    native_weight_bytes_ += bytes;
    p.bound[name] = true;
    return GF_OK;
}

int Model::finalize_layered() {
    LayeredPlan& p = *layered_;
    const LayeredSpec& s = p.spec();
    const gf_model_config& c = config_;
    for (const auto& slot : p.slots)
        if (!p.bound[slot.first]) return fail(GF_ERR_STATE, "tensor '%s' is not bound", slot.first.c_str());
    auto upload = [&](const std::vector<float>& v, float** out) -> int {
        GF_TRY(plan_alloc(allocations_, out, v.size()));
        GF_CUDA(cudaMemcpy(*out, v.data(), v.size() * 4u, cudaMemcpyHostToDevice));
        return GF_OK;
    };
    // offset + stored weight, times the layer scale where there is one; tensors the design does not have stay null.
    auto gain = [&](TensorRole norm, uint32_t l, float offset, float** out, TensorRole scale = TensorRole::kFinalNorm) -> int {
        const auto found = p.vectors.find({norm, l});
        if (found == p.vectors.end()) return GF_OK;
        std::vector<float> v = found->second;
        const auto scales = p.vectors.find({scale, l});
        for (size_t i = 0; i < v.size(); ++i) {
            v[i] = offset + v[i];
            if (scale != TensorRole::kFinalNorm && scales != p.vectors.end()) v[i] *= scales->second[i];
        }
        return upload(v, out);
    };
    auto plain = [&](TensorRole role, uint32_t l, float** out) { return gain(role, l, 0.0f, out); };
    GF_TRY(gain(TensorRole::kFinalNorm, 0, s.norm_offset, &p.final_gain));
    uint32_t q_width = 0, latent = 0, heads = 0, values = 0, ff = 0, top = 0, experts = 0, expert_ff = 0, shared_ff = 0, query_elements = 0;
    uint32_t k_width = 0, prepared = 0;
    size_t partial = 0, partial_pairs = 0;             // elements per row
    p.turns.assign(s.layers.size(), {nullptr, nullptr});
    std::map<std::pair<uint32_t, double>, std::pair<const float2*, const float2*>> rotations;
    for (uint32_t l = 0; l < s.layers.size(); ++l) {
        LayeredLayer& w = p.layers[l];
        const MixerSpec& m = s.layers[l].mixer;
        const FeedForwardSpec& f = s.layers[l].mlp;
        if (s.layers[l].source == l) {
            GF_TRY(gain(TensorRole::kNorm1, l, s.norm_offset, &w.gain1));
            GF_TRY(gain(TensorRole::kNorm1b, l, s.norm_offset, &w.gain1b, TensorRole::kScale1));
            GF_TRY(gain(TensorRole::kNorm2, l, s.norm_offset, &w.gain2));
            GF_TRY(gain(TensorRole::kNorm2b, l, s.norm_offset, &w.gain2b, TensorRole::kScale2));
            GF_TRY(plain(TensorRole::kLatentNorm, l, &w.latent_gain));
            GF_TRY(plain(TensorRole::kSink, l, &w.sink));
            GF_TRY(plain(TensorRole::kQueryNorm, l, &w.q_gain));
            GF_TRY(plain(TensorRole::kKeyNorm, l, &w.k_gain));
            GF_TRY(plain(TensorRole::kTaps, l, &w.taps));
            GF_TRY(plain(TensorRole::kTapBias, l, &w.tap_bias));
            GF_TRY(plain(TensorRole::kStepBias, l, &w.step_bias));
            GF_TRY(plain(TensorRole::kSkip, l, &w.skip));
            GF_TRY(plain(TensorRole::kMixerNorm, l, &w.mixer_gain));
            const auto logs = p.vectors.find({TensorRole::kDecayLog, l});
            if (logs != p.vectors.end()) {
                for (float& v : logs->second) v = -std::exp(v);
                GF_TRY(plain(TensorRole::kDecayLog, l, &w.decay));
            }
        }
        values = std::max(values, m.inner());
        if (m.kind == MixerKind::kLatentAttention) {
            const size_t row_elements = latent_row_elements(m.rank);
            q_width = std::max(q_width, m.heads * m.dim); latent = std::max(latent, m.rank);
            query_elements = std::max(query_elements, m.heads * latent_row_elements(m.rank));
            partial = std::max(partial, m.heads * kLatentMaxParts * row_elements);
            partial_pairs = std::max<size_t>(partial_pairs, m.heads * kLatentMaxParts * 2u);
        } else if (m.kind == MixerKind::kGroupedAttention) {
            const uint32_t row_head = grouped_row_head(m.dim, m.vdim);
            q_width = std::max(q_width, m.heads * m.dim); k_width = std::max(k_width, m.kv_heads * m.dim); heads = std::max(heads, m.heads);
            prepared = std::max(prepared, m.heads * row_head);
            partial = std::max(partial, (size_t)m.heads * kGroupedMaxParts * row_head);
            partial_pairs = std::max<size_t>(partial_pairs, m.heads * kGroupedMaxParts * 2u);
            // Angles in double; one pair of tables per (dimensions, base).
            const uint32_t half = m.rotated / 2u, spans = c.context / kTurnSpan + 1u;
            auto& tables = rotations[{m.rotated, m.rotation_base}];
            if (half && !tables.first) {
                auto tabulate = [&](uint32_t count, uint32_t step, const float2** out) -> int {
                    std::vector<float2> host((size_t)count * half);
                    for (uint32_t i = 0; i < half; ++i) {
                        const double frequency = std::pow(m.rotation_base, -2.0 * (double)i / (double)m.rotated);
                        for (uint32_t n = 0; n < count; ++n) {
                            const double angle = (double)n * (double)step * frequency;
                            host[(size_t)n * half + i] = make_float2((float)std::cos(angle), (float)std::sin(angle));
                        }
                    }
                    float2* dev = nullptr;
                    GF_TRY(plan_alloc(allocations_, &dev, host.size()));
                    GF_CUDA(cudaMemcpy(dev, host.data(), host.size() * sizeof(float2), cudaMemcpyHostToDevice));
                    *out = dev;
                    return GF_OK;
                };
                GF_TRY(tabulate(kTurnSpan, 1u, &tables.first));
                GF_TRY(tabulate(spans, kTurnSpan, &tables.second));
            }
            p.turns[l] = tables;
        } else {
            q_width = std::max(q_width, state_inputs_ld(m));
        }
        if (f.kind == FeedForwardSpec::kNone) continue;
        if (f.kind == FeedForwardSpec::kDense) ff = std::max(ff, round_up(f.ff, 8u));
        else {
            top = std::max(top, f.top); experts = std::max(experts, f.experts);
            expert_ff = std::max(expert_ff, f.top * round_up(f.ff, 8u)); shared_ff = std::max(shared_ff, round_up(f.shared_ff, 8u));
        }
    }
    p.vectors.clear();
    const uint32_t R = c.row_capacity, ring_rows = next_pow2(c.context);
    std::vector<KvPublishLayer> table(c.layers);
    std::vector<StreamRings> rings(c.layers);
    for (uint32_t l = 0; l < c.layers; ++l) {
        LayerCache& cache = caches_[l];
        const size_t row = p.cache_row_bytes(l);
        cache.window = 0;
        // A recurrent layer's ring holds the rows a convolution looks back at, those of a pass, and as many again to go
        // back to.
        cache.ring_rows = p.recurrent(l) ? next_pow2(s.layers[l].mixer.taps - 1u + 2u * R) : ring_rows;
        void** ring[2] = {&cache.ring_k, &cache.ring_v};
        void** own[2] = {&cache.private_k, &cache.private_v};
        for (uint32_t which = 0; which < 2u; ++which) {
            const size_t bytes = p.ring_bytes(l, which, cache.ring_rows, p.own_slots);
            if (bytes) GF_TRY(bytes_alloc(allocations_, ring[which], bytes));
            if (which < p.cache_tensors(l)) GF_TRY(bytes_alloc(allocations_, own[which], row * R));
        }
        table[l] = publish_layer(l, cache.ring_k, cache.ring_v, cache.private_k, cache.private_v);
        rings[l] = StreamRings{cache.ring_k, cache.ring_v};
    }
    GF_TRY(plan_alloc(allocations_, &publish_layers_, c.layers));
    GF_CUDA(cudaMemcpy(publish_layers_, table.data(), sizeof(KvPublishLayer) * c.layers, cudaMemcpyHostToDevice));
    GF_TRY(plan_alloc(allocations_, &p.rings_dev, c.layers));
    GF_CUDA(cudaMemcpy(p.rings_dev, rings.data(), sizeof(StreamRings) * c.layers, cudaMemcpyHostToDevice));
    for (float*& r : p.residual) GF_TRY(plan_alloc(allocations_, &r, (size_t)R * s.width));
    GF_TRY(plan_alloc(allocations_, &p.normed, (size_t)R * s.width));
    GF_TRY(plan_alloc(allocations_, &p.raw_q, (size_t)R * q_width));
    GF_TRY(plan_alloc(allocations_, &p.raw_latent, (size_t)R * latent));
    GF_TRY(plan_alloc(allocations_, &p.heads_out, (size_t)R * values));
    GF_TRY(plan_alloc(allocations_, &p.projected, (size_t)R * s.width));
    GF_TRY(bytes_alloc(allocations_, &p.latent_q, (size_t)R * query_elements * 4u));
    GF_TRY(plan_alloc(allocations_, &p.partial_out, R * partial));
    GF_TRY(plan_alloc(allocations_, &p.partial_ml, R * partial_pairs));
    if (heads) {
        GF_TRY(plan_alloc(allocations_, &p.raw_k, (size_t)R * k_width));
        GF_TRY(plan_alloc(allocations_, &p.raw_gate, (size_t)R * heads));
        GF_TRY(bytes_alloc(allocations_, &p.query, (size_t)R * prepared * 4u));
        GF_TRY(plan_alloc(allocations_, &p.counters, (size_t)R * heads));
    }
    GF_TRY(plan_alloc(allocations_, &p.slots_dev, 2u));
    const uint32_t slots[2] = {p.own_slots, LayeredPlan::kStreamSlots};
    GF_CUDA(cudaMemcpy(p.slots_dev, slots, sizeof slots, cudaMemcpyHostToDevice));
    if (ff) GF_TRY(plan_alloc(allocations_, &p.hidden, (size_t)R * ff));
    if (top) {
        GF_TRY(plan_alloc(allocations_, &p.expert_hidden, (size_t)R * expert_ff));
        GF_TRY(plan_alloc(allocations_, &p.shared_hidden, (size_t)R * shared_ff));
        GF_TRY(plan_alloc(allocations_, &p.parts, (size_t)(top + 1u) * R * s.width));
        GF_TRY(plan_alloc(allocations_, &p.router_logits, (size_t)R * experts));
        GF_TRY(plan_alloc(allocations_, &p.shared_logit, R));
        GF_TRY(plan_alloc(allocations_, &p.route_ids, (size_t)R * top));
        GF_TRY(plan_alloc(allocations_, &p.route_scores, (size_t)R * top));
    }
    return finalize_shared();
}

// A layer's entry of a publication table: its cache rows, or nothing to publish (recurrent layers).
KvPublishLayer Model::publish_layer(uint32_t l, void* ring_k, void* ring_v, const void* own_k, const void* own_v) const {
    const uint32_t tensors = layered_->cache_tensors(l);
    KvPublishLayer entry {};
    entry.ring_mask = caches_[l].ring_rows - 1u;
    entry.row_bytes = (uint32_t)layered_->cache_row_bytes(l);
    if (tensors > 0u) { entry.ring_k = static_cast<uint8_t*>(ring_k); entry.private_k = static_cast<const uint8_t*>(own_k); }
    if (tensors > 1u) { entry.ring_v = static_cast<uint8_t*>(ring_v); entry.private_v = static_cast<const uint8_t*>(own_v); }
    return entry;
}

// ------------------------------------------------------------------ a pass of a few rows

static RowMatrix row_matrix(const DenseMatrix& w, void* out, uint32_t out_ld, uint32_t output = kOutF32) {
    RowMatrix m;
    m.weight = w.data; m.k = w.k; m.n = w.n; m.out = out; m.out_ld = out_ld; m.output = output;
    return m;
}

int Model::encode_layers(uint32_t rows, bool logits, const LayeredRows& where) {
    LayeredPlan& p = *layered_;
    const LayeredSpec& s = p.spec();
    const uint32_t R = config_.row_capacity;
    ++launches_;
    GF_TRY(launch_dense_embedding(p.table.data, p.table.k_blocks(), s.width, s.vocab, tokens_dev_, rows, s.embedding_scale, p.residual[0], status_dev_, stream_, false));
    float *x = p.residual[0], *other = p.residual[1];
    struct { const float *y = nullptr, *gain = nullptr; uint32_t parts = 1; size_t stride = 0; } pending;      // a sublayer's output not yet in the residual
    auto run = [&](RowProduct& r) { r.rows = rows; r.eps = s.eps; r.status = status_dev_; return launch_row_product(r, stream_, true, launches_); };
    auto normalised = [&](RowProduct& r, const float* gain) {
        r.width = s.width; r.in_ld = s.width; r.gain1 = gain;      // without a gain the residual itself
        if (!pending.y) { r.input = gain ? kRowNorm : kRowPlain; r.in = x; return; }
        r.input = kRowAddNorm; r.in = pending.y; r.parts = pending.parts; r.part_stride = pending.stride; r.gain0 = pending.gain;
        r.residual = x; r.residual_out = other;
        std::swap(x, other);
        pending = {};
    };
    auto latent_attention = [&](uint32_t l, const LayeredLayer& w, const MixerSpec& m) -> int {
        const uint32_t row_elements = latent_row_elements(m.rank);
        RowProduct down;
        down.count = 2;
        down.m[0] = row_matrix(w.q, p.raw_q, m.heads * m.dim);
        down.m[1] = row_matrix(w.latent_down, p.raw_latent, m.rank);
        normalised(down, w.gain1);
        GF_TRY(run(down));
        RowProduct query;
        query.batches = m.heads; query.heads = m.heads;
        query.in = p.raw_q; query.in_ld = m.heads * m.dim; query.in_batch = m.dim;
        query.m[0] = row_matrix(w.up_key, p.latent_q, row_elements, kOutLatentQuery);
        query.m[0].weight_batch = w.up_key.bytes();
        query.scale = m.scale; query.query_f16 = p.f32 ? 0u : 1u;
        query.latent_raw = p.raw_latent; query.latent_raw_ld = m.rank; query.latent_rank = m.rank; query.latent_gain = w.latent_gain;
        query.latent_rows = caches_[l].private_k; query.latent_row_elements = row_elements; query.latent_f16 = p.f32 ? 0u : 1u;
        GF_TRY(run(query));
        LatentAttention attention;
        attention.q = p.latent_q;
        attention.rings = where.rings + (size_t)l * where.layer_stride; attention.ring_stride = where.ring_stride;
        attention.private_rows = caches_[l].private_k; attention.positions = where.positions;
        attention.rows = rows; attention.heads = m.heads; attention.row_elements = row_elements; attention.ring_mask = caches_[l].ring_rows - 1u;
        attention.cache_f32 = p.f32 ? 1u : 0u;
        attention.partial_out = p.partial_out; attention.partial_ml = p.partial_ml;
        attention.parts = latent_attention_parts(rows, m.heads, config_.context, where.ring_stride == 0u);
        ++launches_;
        GF_TRY(launch_latent_attention(attention, stream_, true));
        RowProduct value;
        value.batches = m.heads; value.heads = m.heads; value.input = kRowLatent;
        value.in = p.partial_out; value.latent_ml = p.partial_ml; value.sink = w.sink; value.latent_ld = row_elements; value.attention_parts = attention.parts;
        value.m[0] = row_matrix(w.up_value, p.heads_out, m.heads * m.vdim);
        value.m[0].weight_batch = w.up_value.bytes(); value.m[0].out_batch = m.vdim;
        GF_TRY(run(value));
        return GF_OK;
    };
    auto grouped_attention = [&](uint32_t l, const LayeredLayer& w, const MixerSpec& m) -> int {
        const uint32_t row_head = grouped_row_head(m.dim, m.vdim);
        RowProduct in;
        in.count = 3;
        in.m[0] = row_matrix(w.q, p.raw_q, m.heads * m.dim);
        in.m[1] = row_matrix(w.k, p.raw_k, m.kv_heads * m.dim);
        in.m[2] = row_matrix(w.head_gate, p.raw_gate, m.heads);
        normalised(in, w.gain1);
        GF_TRY(run(in));
        QueryKey prepare;
        prepare.raw_q = p.raw_q; prepare.raw_k = prepare.raw_v = p.raw_k;
        prepare.q_ld = m.heads * m.dim; prepare.k_ld = prepare.v_ld = m.kv_heads * m.dim;
        prepare.q_gain = w.q_gain; prepare.k_gain = w.k_gain; prepare.turns = p.turns[l].first; prepare.spans = p.turns[l].second;
        prepare.positions = where.positions; prepare.chain = where.ring_stride == 0u;
        prepare.q = p.query; prepare.keys = caches_[l].private_k; prepare.values = caches_[l].private_v;
        prepare.rows = rows; prepare.heads = m.heads; prepare.kv_heads = m.kv_heads; prepare.dim = m.dim; prepare.vdim = m.vdim;
        prepare.row_head = row_head; prepare.rotated = m.rotated; prepare.f32 = p.f32 ? 1u : 0u;
        prepare.eps = s.eps; prepare.scale = m.scale; prepare.status = status_dev_;
        GroupedAttention attention;
        attention.q = p.query; attention.prepare = prepare;
        attention.fused = grouped_attention_on_tensor_cores(row_head, p.f32) ? 1u : 0u;
        if (!attention.fused) { ++launches_; GF_TRY(launch_query_key(prepare, stream_, true)); }
        attention.rings = where.rings + (size_t)l * where.layer_stride; attention.ring_stride = where.ring_stride;
        attention.own_k = caches_[l].private_k; attention.own_v = caches_[l].private_v; attention.positions = where.positions;
        attention.rows = rows; attention.heads = m.heads; attention.kv_heads = m.kv_heads; attention.row_head = row_head; attention.vdim = m.vdim;
        attention.ring_mask = caches_[l].ring_rows - 1u; attention.f32 = p.f32 ? 1u : 0u;
        attention.softcap = m.softcap; attention.sink = w.sink; attention.gate = p.raw_gate;
        attention.partial_out = p.partial_out; attention.partial_ml = p.partial_ml; attention.counters = p.counters;
        attention.parts = grouped_attention_parts(rows, m.heads, m.kv_heads, config_.context, where.ring_stride == 0u);
        attention.result.data = p.heads_out; attention.result.capacity = R; attention.result.k_pad = m.inner(); attention.result.f32 = 1u;
        ++launches_;
        return launch_grouped_attention(attention, stream_, true);
    };
    auto state_space = [&](uint32_t l, const LayeredLayer& w, const MixerSpec& m) -> int {
        RowProduct in;
        in.m[0] = row_matrix(w.state_in, p.raw_q, state_inputs_ld(m));
        normalised(in, w.gain1);
        GF_TRY(run(in));
        StateSpace step = p.state_space(l);
        step.raw = p.raw_q; step.raw_ld = state_inputs_ld(m);
        step.taps = w.taps; step.tap_bias = w.tap_bias; step.step_bias = w.step_bias; step.decay = w.decay; step.skip = w.skip;
        step.rings = where.rings + (size_t)l * where.layer_stride; step.ring_stride = where.ring_stride;
        step.positions = where.positions; step.slots = where.slots; step.rows = rows; step.input_mask = caches_[l].ring_rows - 1u;
        step.out = p.heads_out;
        ++launches_;
        return launch_state_space_rows(step, stream_, true);
    };
    for (uint32_t l = 0; l < s.layers.size(); ++l) {
        const LayeredLayer& w = p.weights(l);
        const MixerSpec& m = s.layers[l].mixer;
        const FeedForwardSpec& f = s.layers[l].mlp;
        if (m.kind == MixerKind::kLatentAttention) GF_TRY(latent_attention(l, w, m));
        else if (m.kind == MixerKind::kGroupedAttention) GF_TRY(grouped_attention(l, w, m));
        else GF_TRY(state_space(l, w, m));
        RowProduct out;
        out.in = p.heads_out; out.in_ld = m.inner();
        if (m.kind == MixerKind::kStateSpace) { out.input = kRowPartNorm; out.width = m.inner(); out.norm_parts = m.norm_parts; out.gain1 = w.mixer_gain; }
        out.m[0] = row_matrix(w.o, p.projected, s.width);
        GF_TRY(run(out));
        pending.y = p.projected; pending.gain = w.gain1b;
        if (f.kind == FeedForwardSpec::kNone) continue;
        if (f.kind == FeedForwardSpec::kDense) {
            RowProduct up;
            const uint32_t ff = round_up(f.ff, 8u);
            up.m[0] = row_matrix(w.up, p.hidden, ff, f.activation == Activation::kGeluGate ? kOutGeluGate : kOutSquaredRelu);
            normalised(up, w.gain2);
            GF_TRY(run(up));
            RowProduct d;
            d.in = p.hidden; d.in_ld = ff;
            d.m[0] = row_matrix(w.down, p.projected, s.width);
            GF_TRY(run(d));
            pending.y = p.projected; pending.gain = w.gain2b;
            continue;
        }
        const uint32_t ff = round_up(f.ff, 8u), shared_ff = round_up(f.shared_ff, 8u);
        RowProduct route;
        route.m[0] = row_matrix(w.router, p.router_logits, f.experts);
        if (f.shared) {
            route.count = 3;
            route.m[1] = row_matrix(w.shared_weight, p.shared_logit, 1);
            route.m[2] = row_matrix(w.shared_up, p.shared_hidden, shared_ff, kOutClampedGate);
            route.m[2].limit = f.shared_limit;
        }
        normalised(route, w.gain2);
        route.normed_out = p.normed;
        GF_TRY(run(route));
        RowProduct up;
        up.input = kRowRouted; up.batches = rows * f.top; up.in = p.normed; up.in_ld = s.width;
        up.router_logits = p.router_logits; up.experts = f.experts; up.top = f.top; up.route_ids = p.route_ids; up.route_scores = p.route_scores;
        up.m[0] = row_matrix(w.expert_up, p.expert_hidden, ff, kOutClampedGate);
        up.m[0].weight_batch = w.expert_up.bytes(); up.m[0].out_batch = ff; up.m[0].limit = f.limit;
        GF_TRY(run(up));
        RowProduct d;
        d.input = kRowExperts; d.batches = rows * f.top + (f.shared ? rows : 0u); d.top = f.top; d.experts = f.experts;
        d.in = p.expert_hidden; d.in_ld = ff; d.in2 = p.shared_hidden; d.in2_ld = shared_ff; d.route_ids = p.route_ids; d.shared_logit = p.shared_logit;
        d.part_stride = (size_t)R * s.width;
        d.m[0] = row_matrix(w.expert_down, p.parts, s.width);
        d.m[0].weight_batch = w.expert_down.bytes();
        if (f.shared) { d.count = 2; d.m[1] = row_matrix(w.shared_down, p.parts, s.width); }
        GF_TRY(run(d));
        pending.y = p.parts; pending.gain = w.gain2b; pending.parts = f.top + (f.shared ? 1u : 0u); pending.stride = (size_t)R * s.width;
    }
    if (logits) {
        RowProduct head;
        head.m[0] = row_matrix(p.head(), where.logits, s.vocab);
        normalised(head, p.final_gain);
        GF_TRY(run(head));
    }
    return GF_OK;
}

// ------------------------------------------------------------------ a chunk of prompt rows

int Model::ensure_chunk_arena() {
    LayeredPlan& p = *layered_;
    LayeredPlan::Chunk& a = p.chunk;
    if (a.ready) return GF_OK;
    const LayeredSpec& s = p.spec();
    const gf_model_config& c = config_;
    a.rows = std::min(p.chunk_limit, round_up(c.context, 16u));
    const uint32_t rows = round_up(a.rows, 16u), f32 = p.f32 ? 1u : 0u;
    auto operand = [&](Operand& o, uint32_t k, uint32_t capacity) -> int {
        o.capacity = capacity; o.f32 = f32; o.k_pad = round_up(std::max(k, 1u), kDenseBlockK);
        return bytes_alloc(allocations_, &o.data, o.bytes());
    };
    uint32_t query = 0, latent_out = 0, values = 0, latent = 0, query_elements = 0, row_elements = 0, ff = 0, shared_ff = 0, expert_ff = 0, experts = 0, top = 0, heads = 0;
    size_t raw_q = 0, raw_k = 0, gates = 0, prepared = 0, x_elements = 0, bc_elements = 0, step_elements = 0, y_elements = 0;      // per row
    for (const LayerSpec& l : s.layers) {
        const MixerSpec& m = l.mixer;
        values = std::max(values, m.inner());
        if (m.kind == MixerKind::kLatentAttention) {
            query = std::max(query, m.heads * round_up(m.dim, kDenseBlockK)); latent_out = std::max(latent_out, m.heads * round_up(m.rank, kDenseBlockK));
            latent = std::max(latent, m.rank); heads = std::max(heads, m.heads);
            query_elements = std::max(query_elements, m.heads * latent_row_elements(m.rank)); row_elements = std::max(row_elements, latent_row_elements(m.rank));
        } else if (m.kind == MixerKind::kGroupedAttention) {
            raw_q = std::max<size_t>(raw_q, m.heads * m.dim); raw_k = std::max<size_t>(raw_k, m.kv_heads * m.dim); gates = std::max<size_t>(gates, m.heads);
            prepared = std::max<size_t>(prepared, m.heads * grouped_row_head(m.dim, m.vdim));
        } else {
            const StateSpace shape = p.state_space((uint32_t)(&l - s.layers.data()));
            raw_q = std::max<size_t>(raw_q, state_inputs_ld(m)); y_elements = std::max<size_t>(y_elements, m.inner());
            const StateChunk cut = state_space_chunk(shape);
            x_elements = std::max<size_t>(x_elements, m.heads * ((m.vdim + cut.columns - 1u) / cut.columns) * cut.x_ld);
            bc_elements = std::max<size_t>(bc_elements, m.groups * cut.n_ld);
            step_elements = std::max<size_t>(step_elements, m.heads);
        }
        const FeedForwardSpec& f = l.mlp;
        if (f.kind == FeedForwardSpec::kDense) ff = std::max(ff, f.ff);
        if (f.kind == FeedForwardSpec::kExperts) {
            shared_ff = std::max(shared_ff, f.shared_ff); expert_ff = std::max(expert_ff, f.ff); experts = std::max(experts, f.experts); top = std::max(top, f.top);
            a.grouped = std::max(a.grouped, grouped_rows(a.rows, f.top, f.experts));
        }
    }
    GF_TRY(operand(a.normed, s.width, rows));
    GF_TRY(operand(a.heads_out, values, rows));
    if (raw_q) GF_TRY(plan_alloc(allocations_, &a.raw_q, rows * raw_q));
    if (raw_k) {
        GF_TRY(plan_alloc(allocations_, &a.raw_k, rows * raw_k));
        GF_TRY(plan_alloc(allocations_, &a.raw_gate, rows * gates));
        GF_TRY(bytes_alloc(allocations_, &a.prepared_q, rows * prepared * (p.f32 ? 4u : 2u)));
    }
    if (y_elements) {
        GF_TRY(plan_alloc(allocations_, &a.state_x, rows * x_elements));
        GF_TRY(plan_alloc(allocations_, &a.state_b, rows * bc_elements));
        GF_TRY(plan_alloc(allocations_, &a.state_c, rows * bc_elements));
        GF_TRY(plan_alloc(allocations_, &a.state_factors, rows * step_elements * kStateFactors));
        GF_TRY(plan_alloc(allocations_, &a.state_steps, rows * step_elements));
        GF_TRY(plan_alloc(allocations_, &a.state_y, rows * y_elements));
    }
    if (ff) GF_TRY(operand(a.hidden, ff, rows));
    if (experts) {
        if (shared_ff) GF_TRY(operand(a.shared_hidden, shared_ff, rows));
        GF_TRY(operand(a.group, s.width, a.grouped));
        GF_TRY(operand(a.group_hidden, expert_ff, a.grouped));
        GF_TRY(plan_alloc(allocations_, &a.group_y, (size_t)a.grouped * s.width));
        GF_TRY(plan_alloc(allocations_, &a.shared_y, (size_t)rows * s.width));
        GF_TRY(plan_alloc(allocations_, &a.router_logits, (size_t)rows * experts));
        GF_TRY(plan_alloc(allocations_, &a.shared_logit, rows));
        GF_TRY(plan_alloc(allocations_, &a.row_scale, a.grouped));
        GF_TRY(plan_alloc(allocations_, &a.slot_scores, (size_t)rows * top));
        GF_TRY(plan_alloc(allocations_, &a.slot_rows, (size_t)rows * top));
        GF_TRY(plan_alloc(allocations_, &a.slot_experts, (size_t)rows * top));
        GF_TRY(plan_alloc(allocations_, &a.group_start, experts));
        GF_TRY(plan_alloc(allocations_, &a.group_rows, experts));
    }
    GF_TRY(plan_alloc(allocations_, &a.residual, (size_t)rows * s.width));
    GF_TRY(plan_alloc(allocations_, &a.y, (size_t)rows * s.width));
    GF_TRY(plan_alloc(allocations_, &a.final_rows, (size_t)rows * s.width));
    if (latent) {
        GF_TRY(operand(a.query, query, rows));
        GF_TRY(operand(a.latent_out, latent_out, rows));
        GF_TRY(plan_alloc(allocations_, &a.raw_latent, (size_t)rows * latent));
        GF_TRY(bytes_alloc(allocations_, &a.latent_q, (size_t)rows * query_elements * (p.f32 ? 4u : 2u)));
        a.partial_rows = std::max((uint32_t)sm_count() * 64u, heads * 16u);
        GF_TRY(plan_alloc(allocations_, &a.partial_out, (size_t)a.partial_rows * row_elements));
        GF_TRY(plan_alloc(allocations_, &a.partial_ml, (size_t)a.partial_rows * 2u));
    }
    if (latent && !p.f32) {
        size_t per_key = 0, q_elements = 0;
        for (const LayerSpec& l : s.layers) {
            if (l.mixer.kind != MixerKind::kLatentAttention) continue;
            const size_t dims = round_up(l.mixer.dim, 16u), vdims = round_up(l.mixer.vdim, 16u);
            per_key = std::max(per_key, l.mixer.heads * std::max(dims, vdims));
            q_elements = std::max(q_elements, l.mixer.heads * dims);
        }
        // At most 1 GiB for either; chunks that see more positions than fit attend the latents themselves.
        a.expand_keys = (uint32_t)std::min<size_t>(round_up(c.context, 16u), ((size_t)1 << 30) / (per_key * 2u) / 16u * 16u);
        GF_TRY(bytes_alloc(allocations_, &a.latent_rows, (size_t)a.expand_keys * round_up(latent, kDenseBlockK) * 2u));
        GF_TRY(plan_alloc(allocations_, &a.keys, a.expand_keys * per_key));
        GF_TRY(plan_alloc(allocations_, &a.values, a.expand_keys * per_key));
        GF_TRY(plan_alloc(allocations_, &a.head_q, rows * q_elements));
    }
    GF_TRY(plan_alloc(allocations_, &a.tokens, rows));
    GF_TRY(plan_alloc(allocations_, &a.wanted, rows));
    std::vector<KvPublishLayer> table(c.layers);
    a.private_rows.assign(c.layers, nullptr);
    a.private_values.assign(c.layers, nullptr);
    for (uint32_t l = 0; l < c.layers; ++l) {
        if (p.cache_tensors(l) > 0u) GF_TRY(bytes_alloc(allocations_, &a.private_rows[l], p.cache_row_bytes(l) * rows));
        if (p.cache_tensors(l) > 1u) GF_TRY(bytes_alloc(allocations_, &a.private_values[l], p.cache_row_bytes(l) * rows));
        table[l] = publish_layer(l, caches_[l].ring_k, caches_[l].ring_v, a.private_rows[l], a.private_values[l]);
    }
    GF_TRY(plan_alloc(allocations_, &a.publish_layers, c.layers));
    GF_CUDA(cudaMemcpy(a.publish_layers, table.data(), sizeof(KvPublishLayer) * c.layers, cudaMemcpyHostToDevice));
    a.ready = true;
    return GF_OK;
}

static Operand operand_view(const Operand& buffer, uint32_t k) {
    Operand o = buffer;
    o.k_pad = round_up(k, kDenseBlockK);
    return o;
}
static ChunkProblem chunk_problem(const DenseMatrix& w, const Operand& a) {
    ChunkProblem m;
    m.weight = w.data; m.k = w.k; m.n = w.n; m.a = a; m.weight_stride = w.bytes();
    return m;
}

// One chunk: its cache rows are published at the end.  With `logits` every row's final norm is left in final_rows.
int Model::chunk_layers(const uint32_t* tokens_host, uint32_t rows, bool logits) {
    LayeredPlan& p = *layered_;
    LayeredPlan::Chunk& a = p.chunk;
    const LayeredSpec& s = p.spec();
    const bool f32 = p.f32;
    GF_CUDA(cudaMemcpyAsync(a.tokens, tokens_host, rows * sizeof(uint32_t), cudaMemcpyHostToDevice, stream_));
    ++launches_;
    GF_TRY(launch_dense_embedding(p.table.data, p.table.k_blocks(), s.width, s.vocab, a.tokens, rows, s.embedding_scale, a.residual, status_dev_, stream_, false));
    ChunkNorm pending;          // the norm step that takes the last sublayer's output into the residual
    pending.residual = a.residual; pending.width = s.width; pending.rows = rows; pending.eps = s.eps;
    auto normalise = [&](const float* gain, bool final_rows) -> int {
        ChunkNorm n = pending;
        n.gain1 = gain;
        if (final_rows) n.normed = a.final_rows;
        else n.result = operand_view(a.normed, s.width);
        pending.y = nullptr; pending.slots = 0; pending.shared = nullptr;
        ++launches_;
        return launch_chunk_norm(n, stream_);
    };
    auto run = [&](ChunkProduct& product) -> int {
        if (product.rows == 0) product.rows = rows;
        product.error_flag = error_flag_;
        ++launches_;
        return launch_chunk_product(product, f32, stream_);
    };
    const Operand normed = operand_view(a.normed, s.width);
    auto latent_attention = [&](uint32_t l, const LayeredLayer& w, const MixerSpec& m, const Operand& heads_out, bool last) -> int {
        const uint32_t row_elements = latent_row_elements(m.rank), dim_pad = round_up(m.dim, kDenseBlockK), rank_pad = round_up(m.rank, kDenseBlockK);
        ChunkProduct down;
        down.p[0] = chunk_problem(w.latent_down, normed);
        down.p[0].out = a.raw_latent; down.p[0].out_ld = m.rank;
        const Operand query = operand_view(a.query, m.heads * dim_pad);
        const uint32_t positions = position_ + rows, head_pad = round_up(m.dim, 16u), value_pad = round_up(m.vdim, 16u);
        const bool expand = !f32 && positions <= a.expand_keys && head_pad <= kHeadAttentionMaxDim && value_pad <= kHeadAttentionMaxDim
                            && latent_expansion_pays(rows, m.rank, m.dim, m.vdim);
        if (!last && expand) {
            down.problems = 2;
            down.p[1] = chunk_problem(w.q, normed);
            down.p[1].output = kChunkHalfRows; down.p[1].out = reinterpret_cast<float*>(a.head_q); down.p[1].out_ld = m.heads * head_pad;
            down.p[1].segment = m.dim; down.p[1].segment_pad = head_pad; down.p[1].scale = m.scale;
        } else if (!last) {
            down.problems = 2;
            down.p[1] = chunk_problem(w.q, normed);
            down.p[1].output = kChunkOperand; down.p[1].result = query; down.p[1].segment = m.dim; down.p[1].segment_pad = dim_pad;
        }
        GF_TRY(run(down));
        ++launches_;
        GF_TRY(launch_chunk_latents(a.raw_latent, m.rank, w.latent_gain, m.rank, s.eps, a.private_rows[l], row_elements, !f32, rows, status_dev_, stream_));
        if (last) return GF_OK;
        if (expand) {
            Operand latents;
            latents.data = a.latent_rows; latents.capacity = round_up(positions, 16u); latents.k_pad = rank_pad;
            ++launches_;
            GF_TRY(launch_latent_operand(p.rings_dev + l, a.private_rows[l], state_dev_, positions, row_elements, caches_[l].ring_rows - 1u, latents, stream_));
            ChunkProduct expansion;
            expansion.problems = 2;
            expansion.p[0] = chunk_problem(w.expand_key, latents);
            expansion.p[0].output = kChunkHalfRows; expansion.p[0].out = reinterpret_cast<float*>(a.keys); expansion.p[0].out_ld = m.heads * head_pad;
            expansion.p[0].segment = m.dim; expansion.p[0].segment_pad = head_pad;
            expansion.p[1] = chunk_problem(w.up_value, latents);
            expansion.p[1].count = m.heads; expansion.p[1].output = kChunkHalfRows; expansion.p[1].out = reinterpret_cast<float*>(a.values);
            expansion.p[1].out_ld = m.heads * value_pad; expansion.p[1].column_stride = value_pad;
            expansion.rows = positions;
            GF_TRY(run(expansion));
            HeadAttention attention;
            attention.q = a.head_q; attention.k = a.keys; attention.v = a.values; attention.position = state_dev_; attention.sink = w.sink;
            attention.rows = rows; attention.heads = attention.kv_heads = m.heads; attention.dim_pad = head_pad; attention.vdim = m.vdim; attention.vdim_pad = value_pad;
            attention.result = heads_out;
            ++launches_;
            GF_TRY(launch_head_attention(attention, stream_));
        } else {
            ChunkProduct absorb;
            absorb.p[0] = chunk_problem(w.up_key, query);
            absorb.p[0].count = m.heads; absorb.p[0].a_block_stride = dim_pad / kDenseBlockK;
            absorb.p[0].output = kChunkLatentQuery; absorb.p[0].out = static_cast<float*>(a.latent_q); absorb.p[0].out_ld = row_elements;
            absorb.p[0].heads = m.heads; absorb.p[0].scale = m.scale; absorb.p[0].query_f16 = f32 ? 0u : 1u;
            GF_TRY(run(absorb));
            LatentAttention attention;
            attention.q = a.latent_q; attention.rings = p.rings_dev + l; attention.ring_stride = 0;
            attention.private_rows = a.private_rows[l]; attention.positions = state_dev_;
            attention.rows = rows; attention.heads = m.heads; attention.row_elements = row_elements; attention.ring_mask = caches_[l].ring_rows - 1u;
            attention.cache_f32 = f32 ? 1u : 0u; attention.sink = w.sink;
            attention.partial_out = a.partial_out; attention.partial_ml = a.partial_ml;
            attention.parts = std::max(1u, std::min(latent_attention_parts(rows, m.heads, position_ + rows, true), a.partial_rows / (rows * m.heads)));
            const Operand latent_out = operand_view(a.latent_out, m.heads * rank_pad);
            const bool merge = attention.parts > 1u;
            LatentAttention merged = attention;
            merged.result = latent_out; merged.result_stride = rank_pad;
            ++launches_;
            GF_TRY(launch_latent_attention(merge ? attention : merged, stream_, false));
            if (merge) { ++launches_; GF_TRY(launch_latent_merge(merged, stream_)); }
            ChunkProduct value;
            value.p[0] = chunk_problem(w.up_value, latent_out);
            value.p[0].count = m.heads; value.p[0].a_block_stride = rank_pad / kDenseBlockK;
            value.p[0].output = kChunkOperand; value.p[0].result = heads_out; value.p[0].column_stride = m.vdim;
            GF_TRY(run(value));
        }
        return GF_OK;
    };
    auto grouped_attention = [&](uint32_t l, const LayeredLayer& w, const MixerSpec& m, const Operand& heads_out, bool last) -> int {
        const uint32_t row_head = grouped_row_head(m.dim, m.vdim);
        ChunkProduct in;
        in.p[0] = chunk_problem(w.k, normed);
        in.p[0].out = a.raw_k; in.p[0].out_ld = m.kv_heads * m.dim;
        if (!last) {
            in.problems = 3;
            in.p[1] = chunk_problem(w.q, normed);
            in.p[1].out = a.raw_q; in.p[1].out_ld = m.heads * m.dim;
            in.p[2] = chunk_problem(w.head_gate, normed);
            in.p[2].out = a.raw_gate; in.p[2].out_ld = m.heads;
        }
        GF_TRY(run(in));
        QueryKey prepare;
        prepare.raw_q = last ? nullptr : a.raw_q; prepare.raw_k = prepare.raw_v = a.raw_k;
        prepare.q_ld = m.heads * m.dim; prepare.k_ld = prepare.v_ld = m.kv_heads * m.dim;
        prepare.q_gain = w.q_gain; prepare.k_gain = w.k_gain; prepare.turns = p.turns[l].first; prepare.spans = p.turns[l].second; prepare.positions = state_dev_;
        prepare.q = a.prepared_q; prepare.keys = a.private_rows[l]; prepare.values = a.private_values[l];
        prepare.rows = rows; prepare.heads = m.heads; prepare.kv_heads = m.kv_heads; prepare.dim = m.dim; prepare.vdim = m.vdim;
        prepare.row_head = row_head; prepare.rotated = m.rotated; prepare.f32 = f32 ? 1u : 0u;
        prepare.eps = s.eps; prepare.scale = m.scale; prepare.status = status_dev_;
        ++launches_;
        GF_TRY(launch_query_key(prepare, stream_, false));
        if (last) return GF_OK;
        ++launches_;
        if (!f32 && row_head <= kHeadAttentionMaxDim) {
            HeadAttention attention;
            attention.q = static_cast<const __half*>(a.prepared_q);
            attention.k = static_cast<const __half*>(a.private_rows[l]); attention.v = static_cast<const __half*>(a.private_values[l]);
            attention.rings = p.rings_dev + l; attention.ring_mask = caches_[l].ring_rows - 1u; attention.position = state_dev_;
            attention.sink = w.sink; attention.gate = a.raw_gate; attention.softcap = m.softcap;
            attention.rows = rows; attention.heads = m.heads; attention.kv_heads = m.kv_heads;
            attention.dim_pad = attention.vdim_pad = row_head; attention.vdim = m.vdim; attention.result = heads_out;
            return launch_head_attention(attention, stream_);
        }
        GroupedAttention attention;
        attention.q = a.prepared_q; attention.rings = p.rings_dev + l;
        attention.own_k = a.private_rows[l]; attention.own_v = a.private_values[l]; attention.positions = state_dev_;
        attention.rows = rows; attention.heads = m.heads; attention.kv_heads = m.kv_heads; attention.row_head = row_head; attention.vdim = m.vdim;
        attention.ring_mask = caches_[l].ring_rows - 1u; attention.f32 = f32 ? 1u : 0u;
        attention.softcap = m.softcap; attention.sink = w.sink; attention.gate = a.raw_gate; attention.result = heads_out;
        return launch_grouped_attention(attention, stream_, false);
    };
    auto state_space = [&](uint32_t l, const LayeredLayer& w, const MixerSpec& m, const Operand& heads_out, bool last) -> int {
        ChunkProduct in;
        in.p[0] = chunk_problem(w.state_in, normed);
        in.p[0].out = a.raw_q; in.p[0].out_ld = state_inputs_ld(m);
        GF_TRY(run(in));
        StateSpace step = p.state_space(l);
        step.raw = a.raw_q; step.raw_ld = state_inputs_ld(m);
        step.taps = w.taps; step.tap_bias = w.tap_bias; step.step_bias = w.step_bias; step.decay = w.decay; step.skip = w.skip;
        step.rings = p.rings_dev + l; step.positions = state_dev_; step.slots = p.slots_dev; step.rows = rows; step.input_mask = caches_[l].ring_rows - 1u;
        step.out = a.state_y; step.x = a.state_x; step.b = a.state_b; step.c = a.state_c; step.factors = a.state_factors; step.error_flag = error_flag_; step.steps = a.state_steps;
        launches_ += 2;
        GF_TRY(launch_state_space_chunk(step, stream_));
        if (last) return GF_OK;
        ++launches_;
        return launch_chunk_part_norm(a.state_y, m.inner(), a.raw_q, state_inputs_ld(m), m.inner(), m.norm_parts, w.mixer_gain, s.eps, heads_out, rows, stream_);
    };
    for (uint32_t l = 0; l < s.layers.size(); ++l) {
        const LayeredLayer& w = p.weights(l);
        const MixerSpec& m = s.layers[l].mixer;
        const FeedForwardSpec& f = s.layers[l].mlp;
        const bool last = l + 1u == s.layers.size() && !logits;      // nothing downstream of the last layer's cache rows and state is needed
        const Operand heads_out = operand_view(a.heads_out, m.inner());
        GF_TRY(normalise(w.gain1, false));
        if (m.kind == MixerKind::kLatentAttention) GF_TRY(latent_attention(l, w, m, heads_out, last));
        else if (m.kind == MixerKind::kGroupedAttention) GF_TRY(grouped_attention(l, w, m, heads_out, last));
        else GF_TRY(state_space(l, w, m, heads_out, last));
        if (last) break;
        ChunkProduct out;
        out.p[0] = chunk_problem(w.o, heads_out);
        out.p[0].out = a.y; out.p[0].out_ld = s.width;
        GF_TRY(run(out));
        pending.y = a.y; pending.gain0 = w.gain1b;
        if (f.kind == FeedForwardSpec::kNone) continue;
        GF_TRY(normalise(w.gain2, false));
        if (f.kind == FeedForwardSpec::kDense) {
            const Operand hidden = operand_view(a.hidden, f.ff);
            ChunkProduct up;
            up.p[0] = chunk_problem(w.up, normed);
            up.p[0].output = f.activation == Activation::kGeluGate ? kChunkGeluGate : kChunkSquaredRelu; up.p[0].result = hidden;
            GF_TRY(run(up));
            ChunkProduct d;
            d.p[0] = chunk_problem(w.down, hidden);
            d.p[0].out = a.y; d.p[0].out_ld = s.width;
            GF_TRY(run(d));
            pending.y = a.y; pending.gain0 = w.gain2b;
            continue;
        }
        const Operand shared_hidden = f.shared ? operand_view(a.shared_hidden, f.shared_ff) : Operand();
        ChunkProduct route;
        route.p[0] = chunk_problem(w.router, normed);
        route.p[0].out = a.router_logits; route.p[0].out_ld = f.experts;
        if (f.shared) {
            route.problems = 3;
            route.p[1] = chunk_problem(w.shared_weight, normed);
            route.p[1].out = a.shared_logit; route.p[1].out_ld = 1;
            route.p[2] = chunk_problem(w.shared_up, normed);
            route.p[2].output = kChunkClampedGate; route.p[2].result = shared_hidden; route.p[2].limit = f.shared_limit;
        }
        GF_TRY(run(route));
        Operand group = operand_view(a.group, s.width), group_hidden = operand_view(a.group_hidden, f.ff);
        ChunkRoute groups;
        groups.logits = a.router_logits; groups.logits_ld = f.experts; groups.rows = rows; groups.experts = f.experts; groups.top = f.top;
        groups.group_start = a.group_start; groups.group_rows = a.group_rows; groups.slot_rows = a.slot_rows; groups.slot_experts = a.slot_experts;
        groups.slot_scores = a.slot_scores; groups.row_scale = a.row_scale; groups.from = normed; groups.to = group;
        launches_ += 3;
        GF_TRY(launch_chunk_route(groups, stream_));
        ChunkProduct up;
        up.p[0] = chunk_problem(w.expert_up, group);
        up.p[0].count = f.experts; up.p[0].group_start = a.group_start; up.p[0].group_rows = a.group_rows;
        up.p[0].output = kChunkClampedGate; up.p[0].result = group_hidden; up.p[0].limit = f.limit; up.p[0].row_scale = a.row_scale;
        GF_TRY(run(up));
        ChunkProduct d;
        d.p[0] = chunk_problem(w.expert_down, group_hidden);
        d.p[0].count = f.experts; d.p[0].group_start = a.group_start; d.p[0].group_rows = a.group_rows;
        d.p[0].out = a.group_y; d.p[0].out_ld = s.width;
        if (f.shared) {
            d.problems = 2;
            d.p[1] = chunk_problem(w.shared_down, shared_hidden);
            d.p[1].out = a.shared_y; d.p[1].out_ld = s.width;
            d.p[1].row_scale = a.shared_logit; d.p[1].row_scale_sigmoid = 1;
        }
        GF_TRY(run(d));
        pending.y = a.group_y; pending.gain0 = w.gain2b; pending.slots = f.top; pending.slot_rows = a.slot_rows; pending.shared = f.shared ? a.shared_y : nullptr;
    }
    if (logits) GF_TRY(normalise(p.final_gain, true));
    GF_TRY(launch_kv_publish(a.publish_layers, config_.layers, state_dev_, rows, stream_));
    launches_ += 2;
    position_ += rows;
    state_floor_ = state_frontier_ = position_;          // a chunk leaves its last state alone
    return GF_OK;
}

// ------------------------------------------------------------------ portions of a prompt

int Model::extend(const uint32_t* tokens_host, uint32_t count, const uint32_t* want, uint32_t want_count, float* logits_host) {
    if (!finalized_) return fail(GF_ERR_STATE, "plan is not finalized");
    if (poisoned_) return fail(GF_ERR_STATE, "plan is poisoned after an unknown GPU outcome; reset it");
    if (!tokens_host || count == 0 || (want_count && !want)) return fail(GF_ERR_INVALID, "empty portion");
    if (position_ > config_.context || count > config_.context - position_)
        return fail(GF_ERR_INVALID, "portion exceeds the bound context (%u + %u > %u)", position_, count, config_.context);
    for (uint32_t i = 0; i < count; ++i)
        if (tokens_host[i] >= token_vocab()) return fail(GF_ERR_INVALID, "token id %u outside the vocabulary", tokens_host[i]);
    for (uint32_t i = 0; i < want_count; ++i)
        if (want[i] >= count || (i && want[i] <= want[i - 1u])) return fail(GF_ERR_INVALID, "wanted places must rise and lie inside the portion");
    const size_t row_bytes = (size_t)config_.vocab * sizeof(float);
    uint32_t done = 0, next = 0;             // tokens taken, wanted places answered
    auto keep = [&](uint32_t row) -> int {
        prefill_logits_row_ = row;
        if (logits_host)
            GF_CUDA(cudaMemcpyAsync(logits_host + (size_t)next * config_.vocab, logits_ + (size_t)row * config_.vocab, row_bytes, cudaMemcpyDeviceToHost, stream_));
        ++next;
        return GF_OK;
    };
    while (done < count) {
        const uint32_t left = count - done;
        if (layered_ && tensor_prefill_ && left > 2u * config_.row_capacity) {
            GF_TRY(ensure_chunk_arena());
            LayeredPlan& p = *layered_;
            const uint32_t rows = std::min(p.chunk.rows, left);
            std::vector<uint32_t> places;
            for (uint32_t i = next; i < want_count && want[i] < done + rows; ++i) places.push_back(want[i] - done);
            GF_TRY(chunk_layers(tokens_host + done, rows, !places.empty()));
            if (!places.empty()) {
                GF_CUDA(cudaMemcpyAsync(p.chunk.wanted, places.data(), places.size() * 4u, cudaMemcpyHostToDevice, stream_));      // pageable: staged by the driver
                for (uint32_t i = 0; i < places.size(); i += config_.row_capacity) {
                    RowProduct head;
                    head.rows = std::min(config_.row_capacity, (uint32_t)places.size() - i);
                    head.in = p.chunk.final_rows; head.in_ld = config_.hidden; head.in_rows = p.chunk.wanted + i;
                    head.m[0] = row_matrix(p.head(), logits_, config_.vocab);
                    GF_TRY(launch_row_product(head, stream_, false, launches_));
                    for (uint32_t r = 0; r < head.rows; ++r) GF_TRY(keep(r));
                }
            }
            done += rows;
            continue;
        }
        const uint32_t rows = std::min(config_.row_capacity, left);
        const bool logits = next < want_count && want[next] < done + rows;
        GF_TRY(forward(tokens_host + done, rows, logits ? kForwardLogits : 0u));
        GF_TRY(publish(rows));
        while (next < want_count && want[next] < done + rows) GF_TRY(keep(want[next] - done));
        done += rows;
    }
    if (!logits_host) return GF_OK;
    return status_word(nullptr);
}

}  // namespace gf
