#include "model_registry.h"

#include <map>
#include <stdexcept>

static std::map<std::string, ModelFactory>& table() {
    static std::map<std::string, ModelFactory> t;
    return t;
}

RegisterModel::RegisterModel(const char* architecture, ModelFactory factory) { table()[architecture] = factory; }

std::vector<std::string> registered_architectures() {
    std::vector<std::string> names;
    for (const auto& [name, f] : table()) names.push_back(name);
    return names;
}

std::unique_ptr<ModelBackend> open_model(const std::string& dir, const EngineOptions& options) {
    ModelDir files(dir);
    const std::string& arch = files.config().at("architecture").str();
    auto it = table().find(arch);
    if (it == table().end()) {
        std::string known;
        for (const std::string& n : registered_architectures()) known += (known.empty() ? "" : ", ") + n;
        throw std::runtime_error("no model class for architecture \"" + arch + "\" (known: " + known + ")");
    }
    return it->second(files, options);
}
