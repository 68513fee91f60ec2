// The model registry (see architecture.hpp).
#include "architecture.hpp"
#include "json.hpp"

#include <cmath>
#include <cstdio>

namespace gf {
namespace {

// Typed access to a configuration's values; the first missing or ill-typed one is remembered by its path.
struct ConfigReader {
    std::string problem;
    bool ok() const { return problem.empty(); }
    void complain(const std::string& path, const char* what) { if (problem.empty()) problem = path + " " + what; }
    const Json* member(const Json* from, const std::string& path, const char* key, Json::Kind kind, bool required = true) {
        const Json* v = from ? from->find(key) : nullptr;
        if (v && v->is_null() && !required) return nullptr;
        if (!v) { if (required) complain(path + key, "is missing"); return nullptr; }
        if (v->kind != kind) { complain(path + key, "has the wrong type"); return nullptr; }
        return v;
    }
    uint32_t count(const Json* from, const std::string& path, const char* key, uint32_t least = 1u, uint32_t most = 1u << 24) {
        const Json* v = member(from, path, key, Json::kNumber);
        if (!v) return 0;
        if (!(v->number >= (double)least && v->number <= (double)most) || v->number != std::floor(v->number)) {
            complain(path + key, "is out of range");
            return 0;
        }
        return (uint32_t)v->number;
    }
    double number(const Json* from, const std::string& path, const char* key) {
        const Json* v = member(from, path, key, Json::kNumber);
        return v ? v->number : 0.0;
    }
    float real(const Json* from, const std::string& path, const char* key) { return (float)number(from, path, key); }
};

// ---- Zasevik: every layer attends cached latents (no rotation), its feed-forward is dense, routed or absent; each
// sublayer has a pre-norm, a post-norm and a per-channel scale; the token table is also the output head.

bool read_mixer(ConfigReader& r, const Json* layer, const std::string& path, MixerSpec& out) {
    const Json* type = r.member(layer, path, "type", Json::kString);
    if (type && type->text != "latent_attention") r.complain(path + "type", ("names the unknown mixer '" + type->text + "'").c_str());
    const Json* m = r.member(layer, path, "mixer", Json::kObject);
    const std::string at = path + "mixer.";
    out.kind = MixerKind::kLatentAttention;
    out.heads = r.count(m, at, "heads", 1, 4096);
    out.dim = r.count(m, at, "dim", 1, 65536);
    out.vdim = r.count(m, at, "vdim", 1, 65536);
    out.rank = r.count(m, at, "kv_rank", 1, 65536);
    out.scale = r.real(m, at, "scale");
    out.sink = true;
    return r.ok();
}

bool read_feed_forward(ConfigReader& r, const Json* layer, const std::string& path, FeedForwardSpec& out) {
    const Json* m = r.member(layer, path, "mlp", Json::kObject, false);
    if (!m) return r.ok();
    const std::string at = path + "mlp.";
    const Json* kind = r.member(m, at, "kind", Json::kString);
    if (!kind) return false;
    if (kind->text == "dense") {
        out.kind = FeedForwardSpec::kDense;
        out.activation = Activation::kSquaredRelu;
        out.ff = r.count(m, at, "ff");
    } else if (kind->text == "moe") {
        out.kind = FeedForwardSpec::kExperts;
        out.activation = Activation::kClampedGate;
        const Json* router = r.member(m, at, "router", Json::kObject);
        out.experts = r.count(router, at + "router.", "experts", 1, 1024);
        out.top = r.count(router, at + "router.", "top", 1, 64);
        if (r.ok() && out.top > out.experts) r.complain(at + "router.top", "exceeds the number of experts");
        const Json* expert = r.member(m, at, "expert", Json::kObject);
        out.ff = r.count(expert, at + "expert.", "ff");
        out.limit = r.real(expert, at + "expert.", "limit");
        if (const Json* shared = r.member(m, at, "shared", Json::kObject, false)) {
            out.shared = true;
            out.shared_ff = r.count(shared, at + "shared.", "ff");
            out.shared_limit = r.real(shared, at + "shared.", "limit");
        }
    } else {
        r.complain(at + "kind", ("names the unknown feed-forward '" + kind->text + "'").c_str());
    }
    return r.ok();
}

void list_tensors(const LayeredSpec& s, std::vector<TensorSlot>& out) {
    auto add = [&](const std::string& name, TensorRole role, uint32_t layer, uint32_t index, uint32_t rows, uint32_t columns) {
        out.push_back(TensorSlot{name, role, layer, index, rows, columns, false});
    };
    add("embed", TensorRole::kEmbedding, 0, 0, s.vocab, s.width);
    add("final.norm", TensorRole::kFinalNorm, 0, 0, 0, s.width);
    for (uint32_t l = 0; l < s.layers.size(); ++l) {
        const MixerSpec& m = s.layers[l].mixer;
        const FeedForwardSpec& f = s.layers[l].mlp;
        const std::string p = "l" + std::to_string(l) + ".";
        add(p + "norm1", TensorRole::kNorm1, l, 0, 0, s.width);
        add(p + "norm1b", TensorRole::kNorm1b, l, 0, 0, s.width);
        add(p + "ls1", TensorRole::kScale1, l, 0, 0, s.width);
        add(p + "mix.q", TensorRole::kQuery, l, 0, m.heads * m.dim, s.width);
        add(p + "mix.dkv", TensorRole::kLatentDown, l, 0, m.rank, s.width);
        add(p + "mix.dkv.norm", TensorRole::kLatentNorm, l, 0, 0, m.rank);
        add(p + "mix.uk", TensorRole::kLatentUpKey, l, 0, m.heads * m.dim, m.rank);
        add(p + "mix.uv", TensorRole::kLatentUpValue, l, 0, m.heads * m.vdim, m.rank);
        if (m.sink) add(p + "mix.sink", TensorRole::kSink, l, 0, 0, m.heads);
        add(p + "mix.o", TensorRole::kMixerOut, l, 0, s.width, m.heads * m.vdim);
        if (f.kind == FeedForwardSpec::kNone) continue;
        add(p + "norm2", TensorRole::kNorm2, l, 0, 0, s.width);
        add(p + "norm2b", TensorRole::kNorm2b, l, 0, 0, s.width);
        add(p + "ls2", TensorRole::kScale2, l, 0, 0, s.width);
        if (f.kind == FeedForwardSpec::kDense) {
            add(p + "mlp.up", TensorRole::kUp, l, 0, f.ff, s.width);
            add(p + "mlp.down", TensorRole::kDown, l, 0, s.width, f.ff);
            continue;
        }
        for (uint32_t e = 0; e < f.experts; ++e) {
            const std::string q = p + "mlp.e" + std::to_string(e);
            add(q + ".gate", TensorRole::kExpertGate, l, e, f.ff, s.width);
            add(q + ".up", TensorRole::kExpertUp, l, e, f.ff, s.width);
            add(q + ".down", TensorRole::kExpertDown, l, e, s.width, f.ff);
        }
        add(p + "mlp.router", TensorRole::kRouter, l, 0, f.experts, s.width);
        if (f.shared) {
            add(p + "mlp.shared.gate", TensorRole::kSharedGate, l, 0, f.shared_ff, s.width);
            add(p + "mlp.shared.up", TensorRole::kSharedUp, l, 0, f.shared_ff, s.width);
            add(p + "mlp.shared.down", TensorRole::kSharedDown, l, 0, s.width, f.shared_ff);
            add(p + "mlp.shared.sg", TensorRole::kSharedWeight, l, 0, 1, s.width);
        }
    }
}

// Follows every layer's source to the layer that has the tensors, which must be a layer of the same shape.
void resolve_sources(ConfigReader& r, LayeredSpec& s) {
    for (uint32_t l = 0; l < s.layers.size(); ++l) {
        uint32_t at = s.layers[l].source;
        for (size_t steps = 0; s.layers[at].source != at; at = s.layers[at].source)
            if (++steps > s.layers.size()) { r.complain("layers[" + std::to_string(l) + "].weights_of", "leads round in a circle"); return; }
        const MixerSpec &a = s.layers[l].mixer, &b = s.layers[at].mixer;
        const FeedForwardSpec &f = s.layers[l].mlp, &g = s.layers[at].mlp;
        if (a.kind != b.kind || a.heads != b.heads || a.dim != b.dim || a.vdim != b.vdim || a.kv_heads != b.kv_heads || a.rank != b.rank || a.state != b.state
            || a.groups != b.groups || a.taps != b.taps || a.norm_parts != b.norm_parts || f.kind != g.kind || f.ff != g.ff)
            r.complain("layers[" + std::to_string(l) + "].weights_of", "names a layer of another shape");
    }
    std::vector<uint32_t> owners(s.layers.size());
    for (uint32_t l = 0; l < s.layers.size(); ++l)
        for (owners[l] = l; s.layers[owners[l]].source != owners[l];) owners[l] = s.layers[owners[l]].source;
    for (uint32_t l = 0; l < s.layers.size(); ++l) s.layers[l].source = owners[l];
}

void describe_zasevik(ConfigReader& r, const Json& config, ArchitectureDescription& out) {
    LayeredSpec& s = out.spec;
    out.layered = true;
    s.width = r.count(&config, "", "width", 1, 1u << 20);
    s.vocab = r.count(&config, "", "vocab");
    s.embedding_scale = r.real(r.member(&config, "", "embedding", Json::kObject), "embedding.", "scale");
    s.eps = r.real(r.member(&config, "", "norm", Json::kObject), "norm.", "eps");
    s.norm_offset = 1.0f;
    const Json* layers = r.member(&config, "", "layers", Json::kArray);
    if (!layers) return;
    if (layers->items.empty()) { r.complain("layers", "is empty"); return; }
    for (size_t i = 0; i < layers->items.size(); ++i) {
        LayerSpec layer;
        const std::string path = "layers[" + std::to_string(i) + "].";
        layer.source = (uint32_t)i;
        if (!read_mixer(r, &layers->items[i], path, layer.mixer) || !read_feed_forward(r, &layers->items[i], path, layer.mlp)) return;
        s.layers.push_back(layer);
    }
    list_tensors(s, out.tensors);
}

// ---- Tufirax: layers of grouped-query attention (rotated, capped scores, sinks, a gate per head, values that are the
// projected keys) and of state-space mixers, dense gated feed-forward layers or none; sublayers read the residual stream
// itself and are normalised behind; layers may use another layer's tensors; the output head is a matrix of its own.

void read_grouped_attention(ConfigReader& r, const Json* m, const std::string& at, MixerSpec& out) {
    out.kind = MixerKind::kGroupedAttention;
    out.heads = r.count(m, at, "heads", 1, 4096);
    out.kv_heads = r.count(m, at, "kv_heads", 1, 4096);
    out.dim = r.count(m, at, "dim", 1, 4096);
    out.vdim = r.count(m, at, "vdim", 1, 4096);
    out.scale = r.real(m, at, "scale");
    out.softcap = r.real(m, at, "softcap");
    out.sink = out.head_gate = true;
    const Json* rotation = r.member(m, at, "rot", Json::kObject);
    out.rotated = r.count(rotation, at + "rot.", "dims", 0, 4096);
    out.rotation_base = r.number(rotation, at + "rot.", "base");
    if (!r.ok()) return;
    if (out.heads % out.kv_heads) r.complain(at + "kv_heads", "does not divide heads");
    if (out.vdim != out.dim) r.complain(at + "vdim", "differs from dim, but the values are the keys");
    if (out.rotated % 2u || out.rotated > out.dim) r.complain(at + "rot.dims", "must be even and at most dim");
    if (out.rotated && !(out.rotation_base > 0.0)) r.complain(at + "rot.base", "must be positive");
    if (!(out.softcap > 0.0f)) r.complain(at + "softcap", "must be positive");
}

void read_state_space(ConfigReader& r, const Json* m, const std::string& at, MixerSpec& out) {
    out.kind = MixerKind::kStateSpace;
    out.heads = r.count(m, at, "heads", 1, 4096);
    out.vdim = r.count(m, at, "vdim", 1, 4096);
    out.state = r.count(m, at, "state", 1, 1024);
    out.groups = r.count(m, at, "groups", 1, 4096);
    out.taps = r.count(m, at, "conv", 1, 256);
    out.norm_parts = r.count(m, at, "norm_groups", 1, 1024);
    if (!r.ok()) return;
    if (out.heads % out.groups) r.complain(at + "groups", "does not divide heads");
    if (out.inner() % out.norm_parts) r.complain(at + "norm_groups", "does not divide heads * vdim");
}

void list_tufirax_tensors(const LayeredSpec& s, std::vector<TensorSlot>& out) {
    auto add = [&](const std::string& name, TensorRole role, uint32_t layer, uint32_t rows, uint32_t columns, bool table = false) {
        out.push_back(TensorSlot{name, role, layer, 0, rows, columns, table});
    };
    add("embed", TensorRole::kEmbedding, 0, s.vocab, s.width);
    add("head", TensorRole::kHead, 0, s.vocab, s.width);
    add("final.norm", TensorRole::kFinalNorm, 0, 0, s.width);
    for (uint32_t l = 0; l < s.layers.size(); ++l) {
        if (s.layers[l].source != l) continue;
        const MixerSpec& m = s.layers[l].mixer;
        const FeedForwardSpec& f = s.layers[l].mlp;
        const std::string p = "l" + std::to_string(l) + ".";
        add(p + "norm1", TensorRole::kNorm1b, l, 0, s.width);
        if (m.kind == MixerKind::kGroupedAttention) {
            add(p + "mix.q", TensorRole::kQuery, l, m.heads * m.dim, s.width);
            add(p + "mix.k", TensorRole::kKey, l, m.kv_heads * m.dim, s.width);
            add(p + "mix.q.norm", TensorRole::kQueryNorm, l, 0, m.heads * m.dim);
            add(p + "mix.k.norm", TensorRole::kKeyNorm, l, 0, m.kv_heads * m.dim);
            add(p + "mix.sink", TensorRole::kSink, l, 0, m.heads);
            add(p + "mix.g", TensorRole::kHeadGate, l, m.heads, s.width);
        } else {
            add(p + "mix.in", TensorRole::kStateIn, l, m.state_inputs(), s.width);
            add(p + "mix.conv", TensorRole::kTaps, l, m.channels(), m.taps, true);
            add(p + "mix.conv.b", TensorRole::kTapBias, l, 0, m.channels());
            add(p + "mix.dt_bias", TensorRole::kStepBias, l, 0, m.heads);
            add(p + "mix.A_log", TensorRole::kDecayLog, l, 0, m.heads);
            add(p + "mix.D", TensorRole::kSkip, l, 0, m.heads);
            add(p + "mix.norm", TensorRole::kMixerNorm, l, 0, m.inner());
        }
        add(p + "mix.o", TensorRole::kMixerOut, l, s.width, m.inner());
        if (f.kind == FeedForwardSpec::kNone) continue;
        add(p + "norm2", TensorRole::kNorm2b, l, 0, s.width);
        add(p + "mlp.gate", TensorRole::kGate, l, f.ff, s.width);
        add(p + "mlp.up", TensorRole::kUp, l, f.ff, s.width);
        add(p + "mlp.down", TensorRole::kDown, l, s.width, f.ff);
    }
}

void describe_tufirax(ConfigReader& r, const Json& config, ArchitectureDescription& out) {
    LayeredSpec& s = out.spec;
    out.layered = true;
    s.width = r.count(&config, "", "width", 1, 1u << 20);
    s.vocab = r.count(&config, "", "vocab");
    s.eps = r.real(r.member(&config, "", "norm", Json::kObject), "norm.", "eps");
    s.pre_norm = s.tied_head = false;
    const Json* layers = r.member(&config, "", "layers", Json::kArray);
    if (!layers) return;
    if (layers->items.empty()) { r.complain("layers", "is empty"); return; }
    for (size_t i = 0; i < layers->items.size(); ++i) {
        const Json* entry = &layers->items[i];
        const std::string path = "layers[" + std::to_string(i) + "].";
        LayerSpec layer;
        layer.source = (uint32_t)i;
        if (entry->find("weights_of") && !entry->find("weights_of")->is_null()) layer.source = r.count(entry, path, "weights_of", 0, (uint32_t)layers->items.size() - 1u);
        const Json* type = r.member(entry, path, "type", Json::kString);
        const Json* m = r.member(entry, path, "mixer", Json::kObject);
        if (!r.ok()) return;
        if (type->text == "attention") read_grouped_attention(r, m, path + "mixer.", layer.mixer);
        else if (type->text == "mamba2") read_state_space(r, m, path + "mixer.", layer.mixer);
        else r.complain(path + "type", ("names the unknown mixer '" + type->text + "'").c_str());
        if (const Json* f = r.member(entry, path, "mlp", Json::kObject, false)) {
            const Json* kind = r.member(f, path + "mlp.", "kind", Json::kString);
            if (kind && kind->text != "dense") r.complain(path + "mlp.kind", ("names the unknown feed-forward '" + kind->text + "'").c_str());
            layer.mlp.kind = FeedForwardSpec::kDense;
            layer.mlp.activation = Activation::kGeluGate;
            layer.mlp.ff = r.count(f, path + "mlp.", "ff");
        }
        if (!r.ok()) return;
        s.layers.push_back(layer);
    }
    resolve_sources(r, s);
    if (r.ok()) list_tufirax_tensors(s, out.tensors);
}

// ---- the quantised Gemma families: the fields of gf_model_config under their own names (weights in model.gguf).

void describe_gemma(ConfigReader& r, const Json& config, ArchitectureDescription& out) {
    gf_model_config& c = out.config;
    c.hidden = r.count(&config, "", "hidden"); c.ffn = r.count(&config, "", "ffn");
    c.heads = r.count(&config, "", "heads"); c.kv_heads = r.count(&config, "", "kv_heads"); c.head_dim = r.count(&config, "", "head_dim");
    c.layers = r.count(&config, "", "layers"); c.vocab = r.count(&config, "", "vocab");
    c.sliding_window = r.count(&config, "", "sliding_window", 0); c.sliding_pattern = r.count(&config, "", "sliding_pattern", 0);
    c.rope_base_global = r.real(&config, "", "rope_base_global"); c.rope_scale_global = r.real(&config, "", "rope_scale_global");
    c.rope_base_local = r.real(&config, "", "rope_base_local"); c.rope_scale_local = r.real(&config, "", "rope_scale_local");
    c.rms_eps = r.real(&config, "", "rms_eps"); c.attn_softcap = r.real(&config, "", "attn_softcap");
    c.final_softcap = r.real(&config, "", "final_softcap"); c.attention_scale = r.real(&config, "", "attention_scale");
    c.uses_qk_norm = (int32_t)r.count(&config, "", "uses_qk_norm", 0, 1); c.kv_f16 = (int32_t)r.count(&config, "", "kv_f16", 0, 1);
}

struct Architecture { const char* name; void (*describe)(ConfigReader&, const Json&, ArchitectureDescription&); };
const Architecture kArchitectures[] = {
    {"Gemma2", describe_gemma},
    {"Gemma3", describe_gemma},
    {"Tufirax", describe_tufirax},
    {"Zasevik", describe_zasevik},
};

}  // namespace

int describe_architecture(const char* text, size_t size, ArchitectureDescription& out) {
    Json config;
    size_t at = 0;
    if (!Json::parse(text, size, config, &at) || config.kind != Json::kObject) return fail(GF_ERR_INVALID, "configuration: malformed JSON near byte %zu", at);
    const Json* name = config.find("architecture");
    if (!name || name->kind != Json::kString) return fail(GF_ERR_INVALID, "configuration: 'architecture' is missing");
    for (const Architecture& a : kArchitectures) {
        if (name->text != a.name) continue;
        ConfigReader reader;
        out = ArchitectureDescription();
        out.name = a.name;
        a.describe(reader, config, out);
        return reader.ok() ? GF_OK : fail(GF_ERR_INVALID, "configuration: %s", reader.problem.c_str());
    }
    return fail(GF_ERR_INVALID, "configuration: no architecture named '%s' (known:\n%s)", name->text.c_str(), architecture_names());
}

const char* architecture_names() {
    static const std::string names = [] {
        std::string all;
        for (const Architecture& a : kArchitectures) all += std::string(a.name) + "\n";
        return all;
    }();
    return names.c_str();
}

}  // namespace gf

extern "C" const char* gf_architectures(void) { return gf::architecture_names(); }
