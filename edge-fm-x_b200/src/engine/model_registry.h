// Model registry: which names (engine JSON "model_name") and which checkpoints (config.json "architecture") this build
// serves, and how a model's device context and caches are set up.  Each family registers itself from its own file.
#pragma once
#include <memory>
#include <string>
#include <vector>

#include "config.h"
#include "kv_manager.h"
#include "paged_cache.h"

struct efm_b200_ctx;

namespace edge_fm {

// What the token-generation engine needs from a freshly built model; the engine owns ctx afterwards.
struct ModelSetup {
    efm_b200_ctx* ctx = nullptr;
    int32_t device_id = 0;
    int32_t hidden = 0;
    int32_t vocab = 0;
    bool use_mrope = false;
    std::shared_ptr<KVManager> kv_manager;      // the slots declared in kvcache.requests
    std::shared_ptr<PagedCache> paged_cache;    // models on the paged cache only
    int32_t max_live_requests = 0;              // batched steps: sequences at a time (0: the model has no batched step)
    int32_t max_step_tokens = 0;
};

struct ModelFamily {
    std::string name;                           // canonical model name
    std::vector<std::string> architectures;     // config.json "architecture" values that select it
    ModelSetup (*build)(const EngineConfig&);
};

class ModelRegistry {
public:
    static void add(const ModelFamily& family);
    // By the engine JSON's model_name, else by the checkpoint's config.json; throws ConfigurationError.
    static const ModelFamily& resolve(const EngineConfig& config);
    static std::vector<std::string> names();
};

struct ModelRegistrar {
    explicit ModelRegistrar(const ModelFamily& f) { ModelRegistry::add(f); }
};

// backend status -> edge_fm exception
void check_backend(int32_t status, const efm_b200_ctx* ctx, const char* what);
int32_t backend_dtype_code(const std::string& safetensors_dtype);      // -1: not a type the backend takes

}  // namespace edge_fm
