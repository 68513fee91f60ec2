// safetensors files and model folders: binds the tensors of a checkpoint to a resident plan by name.
//
// A file is an eight-byte little-endian header length, that many bytes of JSON (name -> dtype, shape, data_offsets)
// and the data.  The file is mapped read-only; a tensor travels to the device through the plan's upload pipeline.
#include "common.cuh"
#include "json.hpp"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cmath>
#include <cstring>
#include <string>
#include <vector>

namespace gf {
namespace {

struct MappedFile {
    const uint8_t* data = nullptr;
    size_t size = 0;
    int fd = -1;
    ~MappedFile() {
        if (data) munmap(const_cast<uint8_t*>(data), size);
        if (fd >= 0) close(fd);
    }
    bool open_file(const char* path) {
        fd = open(path, O_RDONLY);
        struct stat info;
        if (fd < 0 || fstat(fd, &info) != 0 || info.st_size <= 0) return false;
        size = (size_t)info.st_size;
        void* mapped = mmap(nullptr, size, PROT_READ, MAP_PRIVATE, fd, 0);
        if (mapped == MAP_FAILED) return false;
        data = static_cast<const uint8_t*>(mapped);
        return true;
    }
};

bool exists(const std::string& path) {
    struct stat info;
    return stat(path.c_str(), &info) == 0;
}

}  // namespace
}  // namespace gf

using namespace gf;

extern "C" {

int gf_model_load_safetensors(gf_model* model, const char* path, uint32_t* out_bound_tensors) {
    if (!model || !path) return fail(GF_ERR_INVALID, "gf_model_load_safetensors: null argument");
    MappedFile file;
    if (!file.open_file(path)) return fail(GF_ERR_INVALID, "gf_model_load_safetensors: cannot read %s", path);
    uint64_t header = 0;
    if (file.size >= 8u) std::memcpy(&header, file.data, 8u);
    if (file.size < 8u || header > file.size - 8u) return fail(GF_ERR_INVALID, "gf_model_load_safetensors: %s is truncated", path);
    Json directory;
    if (!Json::parse(reinterpret_cast<const char*>(file.data) + 8u, (size_t)header, directory) || directory.kind != Json::kObject)
        return fail(GF_ERR_INVALID, "gf_model_load_safetensors: %s has a malformed header", path);
    const size_t data_bytes = file.size - 8u - (size_t)header;
    const uint8_t* data = file.data + 8u + header;
    uint32_t bound = 0;
    for (const auto& entry : directory.members) {
        if (entry.first == "__metadata__") continue;
        const Json *dtype = entry.second.find("dtype"), *shape = entry.second.find("shape"), *offsets = entry.second.find("data_offsets");
        if (!dtype || !shape || !offsets || dtype->kind != Json::kString || shape->kind != Json::kArray || offsets->kind != Json::kArray || offsets->items.size() != 2u)
            return fail(GF_ERR_INVALID, "gf_model_load_safetensors: tensor %s is malformed", entry.first.c_str());
        const size_t element = dtype->text == "BF16" || dtype->text == "F16" ? 2u : dtype->text == "F32" ? 4u : 0u;
        const int type = dtype->text == "BF16" ? GF_BF16 : dtype->text == "F16" ? GF_F16 : GF_F32;
        if (element == 0) return fail(GF_ERR_INVALID, "gf_model_load_safetensors: tensor %s has type %s", entry.first.c_str(), dtype->text.c_str());
        std::vector<uint64_t> dims;
        double elements = 1.0;
        for (const Json& d : shape->items) {
            if (d.kind != Json::kNumber || !(d.number >= 0.0 && d.number < 1e12) || d.number != std::floor(d.number))
                return fail(GF_ERR_INVALID, "gf_model_load_safetensors: tensor %s has a bad shape", entry.first.c_str());
            dims.push_back((uint64_t)d.number);
            elements *= d.number;
        }
        const double begin = offsets->items[0].number, end = offsets->items[1].number;
        if (dims.empty() || !(begin >= 0.0 && end >= begin && end <= (double)data_bytes) || end - begin != elements * (double)element)
            return fail(GF_ERR_INVALID, "gf_model_load_safetensors: tensor %s lies outside the file", entry.first.c_str());
        const int status = gf_model_set_tensor(model, entry.first.c_str(), type, data + (size_t)begin, dims.data(), (uint32_t)dims.size());
        if (status != GF_OK) return status;
        ++bound;
    }
    if (out_bound_tensors) *out_bound_tensors = bound;
    return GF_OK;
}

int gf_model_open(const char* folder, uint32_t context, uint32_t row_capacity, int precision, gf_model** out_model) {
    if (!folder || !out_model) return fail(GF_ERR_INVALID, "gf_model_open: null argument");
    const std::string base = std::string(folder) + "/";
    std::string config;
    {
        MappedFile file;
        if (!file.open_file((base + "config.json").c_str())) return fail(GF_ERR_INVALID, "gf_model_open: cannot read %sconfig.json", base.c_str());
        config.assign(reinterpret_cast<const char*>(file.data), file.size);
    }
    gf_model* model = nullptr;
    int status = gf_model_create_described(config.c_str(), context, row_capacity, precision, &model);
    if (status != GF_OK) return status;
    const std::string quantised = base + "model.gguf";
    status = exists(quantised) ? gf_model_load_gguf(model, quantised.c_str(), nullptr) : gf_model_load_safetensors(model, (base + "model.safetensors").c_str(), nullptr);
    if (status == GF_OK) status = gf_model_finalize(model);
    if (status != GF_OK) {
        const std::string why = gf_last_error();
        gf_model_destroy(model);
        return fail(status, "%s", why.c_str());
    }
    *out_model = model;
    return GF_OK;
}

}  // extern "C"
