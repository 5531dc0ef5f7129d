// A model folder: config.json and model.safetensors (an 8-byte little-endian header length, that many bytes of JSON
// name -> {dtype, shape, data_offsets}, then the data). The data stays memory-mapped; nothing is converted here.
#pragma once

#include <cstdint>
#include <map>
#include <string>
#include <vector>

#include "json_value.h"

struct TensorView {
    std::string name, dtype;          // safetensors names: "BF16", "F32", "I32", ...
    std::vector<int64_t> shape;
    const unsigned char* data = nullptr;
    size_t bytes = 0;
    int64_t elems() const {
        int64_t n = 1;
        for (int64_t d : shape) n *= d;
        return n;
    }
};

class ModelDir {
public:
    explicit ModelDir(const std::string& path);  // throws std::runtime_error
    ~ModelDir();
    ModelDir(const ModelDir&) = delete;
    ModelDir& operator=(const ModelDir&) = delete;

    const Json& config() const { return config_; }
    bool has(const std::string& name) const { return tensors_.count(name) > 0; }
    const TensorView& tensor(const std::string& name) const;  // throws if missing
    // The same, and throws unless the tensor has this shape.
    const TensorView& tensor(const std::string& name, const std::vector<int64_t>& shape) const;
    size_t n_tensors() const { return tensors_.size(); }

private:
    Json config_;
    std::map<std::string, TensorView> tensors_;
    void* map_ = nullptr;
    size_t map_bytes_ = 0;
};

// Widens a BF16 or F32 tensor to f32.
std::vector<float> tensor_f32(const TensorView& t);
