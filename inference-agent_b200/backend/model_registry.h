// Which code serves which model folder: architecture name (config.json "architecture") -> factory. A design registers
// itself from its own source file; callers only see BatchedBackend.
#pragma once

#include <memory>
#include <string>
#include <vector>

#include "batched_backend.h"
#include "model_dir.h"

struct EngineOptions {
    bool f32 = false;          // every product in 32-bit arithmetic (bf16 weights are widened), f32 caches
    int max_tokens = 4096;     // most tokens the live sequences hold together; sizes the cache pools
    int max_seqs = 4;          // sequences alive at a time (state slots)
    int max_step_tokens = 0;   // most tokens of one step; 0: max_tokens
};

// A backend of a registered architecture, with what callers outside the step function need to know about the model.
class ModelBackend : public BatchedBackend {
public:
    virtual int n_vocab() const = 0;
    virtual std::string describe() const = 0;
    // Residual stream after every layer of the next steps, [layer][n_tok][width] f32, appended to `out` (null: off). Diagnostics.
    virtual void tap_residuals(std::vector<float>* out) = 0;
    // Bytes of weights a step reads once (embedding table excluded), and device time of the last step in milliseconds.
    virtual size_t weight_bytes() const = 0;
    virtual float last_step_ms() const = 0;
};

using ModelFactory = std::unique_ptr<ModelBackend> (*)(const ModelDir&, const EngineOptions&);
struct RegisterModel {
    RegisterModel(const char* architecture, ModelFactory factory);
};
std::vector<std::string> registered_architectures();
// Opens a model folder with the class its config names; throws std::runtime_error if no class is registered for it.
std::unique_ptr<ModelBackend> open_model(const std::string& dir, const EngineOptions& options);
