#include "model_dir.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstring>
#include <fstream>
#include <sstream>
#include <stdexcept>

static std::string read_text(const std::string& path) {
    std::ifstream f(path, std::ios::binary);
    if (!f) throw std::runtime_error("cannot open " + path);
    std::ostringstream ss;
    ss << f.rdbuf();
    return ss.str();
}

ModelDir::ModelDir(const std::string& path) {
    config_ = Json::parse(read_text(path + "/config.json"));
    const std::string file = path + "/model.safetensors";
    const int fd = open(file.c_str(), O_RDONLY);
    if (fd < 0) throw std::runtime_error("cannot open " + file);
    struct stat st;
    if (fstat(fd, &st) != 0 || st.st_size < 8) {
        close(fd);
        throw std::runtime_error(file + ": not a safetensors file");
    }
    map_bytes_ = size_t(st.st_size);
    map_ = mmap(nullptr, map_bytes_, PROT_READ, MAP_PRIVATE, fd, 0);
    close(fd);
    if (map_ == MAP_FAILED) {
        map_ = nullptr;
        throw std::runtime_error("cannot map " + file);
    }
    const unsigned char* base = static_cast<const unsigned char*>(map_);
    uint64_t header = 0;
    for (int i = 7; i >= 0; i--) header = header << 8 | base[i];
    if (header > map_bytes_ - 8) throw std::runtime_error(file + ": header longer than the file");
    const Json index = Json::parse(std::string(reinterpret_cast<const char*>(base) + 8, size_t(header)));
    const unsigned char* data = base + 8 + header;
    const uint64_t data_bytes = map_bytes_ - 8 - header;
    for (const auto& [name, entry] : index.members()) {
        if (name == "__metadata__") continue;
        TensorView t;
        t.name = name;
        t.dtype = entry.at("dtype").str();
        for (const Json& d : entry.at("shape").items()) t.shape.push_back(d.integer());
        const auto& off = entry.at("data_offsets").items();
        if (off.size() != 2) throw std::runtime_error(file + ": tensor " + name + " has bad offsets");
        const int64_t a = off[0].integer(), b = off[1].integer();
        if (a < 0 || b < a || uint64_t(b) > data_bytes) throw std::runtime_error(file + ": tensor " + name + " lies outside the file");
        t.data = data + a;
        t.bytes = size_t(b - a);
        const size_t width = t.dtype == "BF16" || t.dtype == "F16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : 0;
        if (width && size_t(t.elems()) * width != t.bytes) throw std::runtime_error(file + ": tensor " + name + " has the wrong size");
        tensors_.emplace(name, std::move(t));
    }
}

ModelDir::~ModelDir() {
    if (map_) munmap(map_, map_bytes_);
}

const TensorView& ModelDir::tensor(const std::string& name) const {
    auto it = tensors_.find(name);
    if (it == tensors_.end()) throw std::runtime_error("model: tensor " + name + " is missing");
    return it->second;
}

const TensorView& ModelDir::tensor(const std::string& name, const std::vector<int64_t>& shape) const {
    const TensorView& t = tensor(name);
    if (t.shape != shape) {
        std::string want, got;
        for (int64_t d : shape) want += (want.empty() ? "" : ", ") + std::to_string(d);
        for (int64_t d : t.shape) got += (got.empty() ? "" : ", ") + std::to_string(d);
        throw std::runtime_error("model: tensor " + name + " has shape [" + got + "], expected [" + want + "]");
    }
    return t;
}

std::vector<float> tensor_f32(const TensorView& t) {
    std::vector<float> out(static_cast<size_t>(t.elems()));
    if (t.dtype == "F32") {
        memcpy(out.data(), t.data, out.size() * 4);
    } else if (t.dtype == "BF16") {
        for (size_t i = 0; i < out.size(); i++) {
            uint16_t h;
            memcpy(&h, t.data + 2 * i, 2);
            const uint32_t u = uint32_t(h) << 16;
            memcpy(&out[i], &u, 4);
        }
    } else {
        throw std::runtime_error("model: tensor " + t.name + " has type " + t.dtype + ", expected BF16 or F32");
    }
    return out;
}
