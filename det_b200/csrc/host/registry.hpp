// Which model class runs a checkpoint.  An architecture is found by the name a checkpoint carries — "architecture" of a
// folder's config.json, "general.architecture" of a det GGUF — and supplies the loader.
#pragma once
#include "model.hpp"

namespace det {

struct OpenOptions {
    size_t max_ctx = 0, max_batch = 0;
    Dtype dtype = Dtype::BF16;      // activations of a floating-point model; quantized models have one form
};
struct Architecture {
    const char* name;
    bool folder;                    // config.json + model.safetensors, else a GGUF file
    std::unique_ptr<Model> (*open)(const std::string& path, Backend* backend, const OpenOptions& opt);   // throws on failure
};
const std::vector<Architecture>& architectures();

// Opens a model folder or a GGUF file; throws std::runtime_error with the reason.
std::unique_ptr<Model> open_model(const std::string& path, Backend* backend, const OpenOptions& opt);

}  // namespace det
