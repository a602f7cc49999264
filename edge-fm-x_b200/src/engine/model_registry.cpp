#include "model_registry.h"

#include <efm_b200.h>

#include <algorithm>

namespace edge_fm {

namespace {
std::vector<ModelFamily>& families() {
    static std::vector<ModelFamily> f;
    return f;
}
}  // namespace

void ModelRegistry::add(const ModelFamily& family) { families().push_back(family); }

std::vector<std::string> ModelRegistry::names() {
    std::vector<std::string> out;
    for (const ModelFamily& f : families()) out.push_back(f.name);
    std::sort(out.begin(), out.end());
    return out;
}

const ModelFamily& ModelRegistry::resolve(const EngineConfig& config) {
    const std::string name = EngineConfig::normalize_model_name(config.model_name());
    if (name.empty()) {
        const std::string arch = config.checkpoint_architecture();
        for (const ModelFamily& f : families())
            if (!arch.empty() && std::find(f.architectures.begin(), f.architectures.end(), arch) != f.architectures.end()) return f;
    }
    for (const ModelFamily& f : families())
        if (f.name == name) return f;
    std::string known;
    for (const std::string& n : names()) known += (known.empty() ? "" : ", ") + n;
    throw ConfigurationError("Unsupported or missing model_name in engine config. Supported values include: Qwen2.5, Qwen2.5-VL, Folizen, Temuvik, Vekolix, Viladra (" + known + ")");
}

void check_backend(int32_t st, const efm_b200_ctx* ctx, const char* what) {
    if (st == EFM_OK) return;
    const std::string msg = std::string(what) + ": " + efm_b200_last_error(ctx);
    switch (st) {
        case EFM_ERR_OUT_OF_MEMORY: throw OutOfMemoryError(msg);
        case EFM_ERR_INVALID_ARGUMENT: throw InvalidRequestError(msg);
        case EFM_ERR_UNSUPPORTED: throw ConfigurationError(msg);
        case EFM_ERR_STATE: throw InternalError(msg);
        default: throw DeviceError(msg);
    }
}

int32_t backend_dtype_code(const std::string& st) {
    if (st == "BF16") return EFM_BF16;
    if (st == "F16") return EFM_F16;
    if (st == "F32") return EFM_F32;
    if (st == "I32") return EFM_I32;
    if (st == "I64") return EFM_I64;
    if (st == "U8") return EFM_U8;
    if (st == "I8") return EFM_I8;
    return -1;
}

}  // namespace edge_fm
