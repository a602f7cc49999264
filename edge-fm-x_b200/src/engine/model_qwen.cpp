// The Qwen2.5 / Qwen2.5-VL family: config.json -> efm_model_desc, checkpoint tensors (optionally a second, INT4 decode
// checkpoint), tensor-parallel rendezvous, contiguous KV slots.
#include <efm_b200.h>

#include <algorithm>
#include <cstdlib>
#include <cstring>

#include "model_registry.h"
#include "safetensors.h"
#include "tp_rendezvous.h"

namespace edge_fm {

namespace {

// KV buffers live in the backend; the manager only keeps the bookkeeping and the pointers.
class BackendKVAllocator : public KVBufferAllocator {
public:
    explicit BackendKVAllocator(efm_b200_ctx* ctx) : ctx_(ctx) {}
    Device device() const override { return Device::GPU; }
    std::vector<void*> allocate_slot(int32_t request_id, int32_t max_tokens, size_t, int32_t num_layers) override {
        efm_status st = efm_b200_alloc_kv_slot(ctx_, request_id, max_tokens);
        if (st == EFM_ERR_OUT_OF_MEMORY) throw OutOfMemoryError(efm_b200_last_error(ctx_));
        if (st != EFM_OK) throw DeviceError(efm_b200_last_error(ctx_));
        std::vector<void*> out;
        for (int32_t l = 0; l < num_layers; ++l) {
            void* p = nullptr;
            if (efm_b200_kv_layer_ptr(ctx_, request_id, l, &p, nullptr) != EFM_OK) throw InternalError(efm_b200_last_error(ctx_));
            out.push_back(p);
        }
        return out;
    }

private:
    efm_b200_ctx* ctx_;
};

ModelSetup build_qwen(const EngineConfig& config) {
    ModelSetup setup;
    const std::string model = EngineConfig::normalize_model_name(config.model_name());
    const json::Value mc = config.prefill_model_config();
    setup.device_id = config.runtime_device_id();
    if (dtype_from_string(config.kvcache_dtype()) != DType::BFloat16)
        throw ConfigurationError("kvcache.dtype must be bf16 for this backend");
    const AttentionType attn = attention_type_from_string(config.kvcache_attention_type());

    efm_model_desc d;
    std::memset(&d, 0, sizeof(d));
    d.struct_size = (int32_t)sizeof(d);
    d.num_layers = (int32_t)mc.get_int("num_hidden_layers", 0);
    d.hidden = (int32_t)mc.get_int("hidden_size", 0);
    d.q_heads = (int32_t)mc.get_int("num_attention_heads", 0);
    d.kv_heads = (int32_t)mc.get_int("num_key_value_heads", d.q_heads);
    d.intermediate = (int32_t)mc.get_int("intermediate_size", 0);
    d.vocab = (int32_t)mc.get_int("vocab_size", 0);
    if (d.num_layers <= 0 || d.hidden <= 0 || d.q_heads <= 0 || d.vocab <= 0 || d.intermediate <= 0)
        throw ConfigurationError("config.json lacks num_hidden_layers / hidden_size / num_attention_heads / vocab_size / intermediate_size");
    d.head_dim = d.hidden / d.q_heads;      // as the reference derives it (kv_manager.cpp:80)
    d.rms_eps = (float)mc.get_double("rms_norm_eps", 1e-6);
    d.rope_theta = (float)mc.get_double("rope_theta", 10000.0);
    const std::string act = mc.get_string("hidden_act", "silu");
    if (act != "silu") throw ConfigurationError("hidden_act must be silu, got " + act);
    const std::string torch_dtype = mc.get_string("torch_dtype", mc.get_string("dtype", "bfloat16"));
    if (torch_dtype != "bfloat16") throw ConfigurationError("checkpoint dtype must be bfloat16, got " + torch_dtype);
    const json::Value* rs = mc.find("rope_scaling");
    if (rs != nullptr && rs->is_object()) {
        const json::Value* sec = rs->find("mrope_section");
        if (sec != nullptr && sec->is_array() && sec->arr.size() == 3) {
            d.use_mrope = 1;
            for (int i = 0; i < 3; ++i) d.mrope_section[i] = (int32_t)sec->arr[i].inum;
        }
    }
    setup.use_mrope = d.use_mrope != 0;
    setup.hidden = d.hidden;
    setup.vocab = d.vocab;
    if (model == "qwen2_5" && setup.use_mrope) throw ConfigurationError("model_name Qwen2.5 with an mrope checkpoint: use Qwen2.5-VL");

    // tied lm_head <=> the checkpoint carries no lm_head.weight (reference: src/layers/linear.cu:2244-2248)
    const std::vector<std::string> files = collect_safetensors_files(config.prefill_model_path());
    if (files.empty())
        throw ConfigurationError("No model.safetensors or model-*-of-*.safetensors found in: " + config.prefill_model_path());
    std::vector<std::unique_ptr<SafeTensorsFile>> maps;
    bool has_lm_head = false;
    const bool vlm = model == "qwen2_5_vl";
    for (const std::string& f : files) {
        maps.emplace_back(new SafeTensorsFile(f));
        for (const SafeTensorEntry& e : maps.back()->entries()) {
            std::string name = e.name;
            if (vlm && !map_vlm_weight_name(e.name, &name)) continue;
            if (name == "lm_head.weight") has_lm_head = true;
        }
    }
    d.tied_lm_head = has_lm_head ? 0 : 1;

    const std::vector<KvRequestConfig> reqs = config.kv_requests();
    int32_t max_tokens = 1;
    for (const KvRequestConfig& r : reqs) max_tokens = std::max(max_tokens, r.max_tokens);
    d.max_prefill_tokens = std::min(max_tokens, 2048);
    d.max_response_tokens = config.sampling_max_new_tokens() + 1;

    // Tensor parallel: one process per GPU, every process builds the same engine and issues the same requests.
    // Rank from the environment, device = $LOCAL_RANK (else runtime.device_id + rank), host exchange through files.
    const int32_t tp = config.tensor_parallel();
    if (tp < 1 || tp > 8) throw ConfigurationError("runtime.tensor_parallel must be between 1 and 8");
    const int32_t tp_rank = tp > 1 ? config.tp_rank() : 0;
    std::unique_ptr<TpRendezvous> meet;
    if (tp > 1) {
        if (tp_rank < 0 || tp_rank >= tp) throw ConfigurationError("tensor parallel rank (EFM_TP_RANK / RANK) must be in [0, runtime.tensor_parallel)");
        const char* local = std::getenv("LOCAL_RANK");
        setup.device_id = local != nullptr && local[0] != 0 ? std::atoi(local) : setup.device_id + tp_rank;
        meet.reset(new TpRendezvous(config.tp_rendezvous(), tp_rank, tp));
    }
    efm_status st = efm_b200_create(&d, setup.device_id, tp_rank, tp, &setup.ctx);
    if (st != EFM_OK) {
        const std::string msg = std::string("backend creation failed: ") + efm_b200_last_error(nullptr);
        if (st == EFM_ERR_OUT_OF_MEMORY) throw OutOfMemoryError(msg);
        if (st == EFM_ERR_UNSUPPORTED || st == EFM_ERR_INVALID_ARGUMENT) throw ConfigurationError(msg);
        throw DeviceError(msg);
    }
    try {
        if (tp > 1) {
            std::vector<char> id(128, 0);
            if (tp_rank == 0) check_backend(efm_b200_tp_unique_id(id.data()), setup.ctx, "communicator id");
            id = meet->broadcast_from_root("nccl_id", id);
            if (id.size() != 128) throw ConfigurationError("tensor parallel rendezvous: malformed communicator id");
            check_backend(efm_b200_tp_init(setup.ctx, id.data()), setup.ctx, "communicator initialisation");
        }
        for (const auto& m : maps) {
            for (const SafeTensorEntry& e : m->entries()) {
                std::string name = e.name;
                if (vlm && !map_vlm_weight_name(e.name, &name)) continue;
                const int32_t code = backend_dtype_code(e.dtype);
                if (code < 0) continue;
                st = efm_b200_set_weight(setup.ctx, name.c_str(), e.data, e.shape.data(), (int32_t)e.shape.size(), code, EFM_MEM_HOST);
                if (st != EFM_OK) throw ModelNotLoadedError(std::string("loading ") + name + ": " + efm_b200_last_error(setup.ctx));
            }
        }
        // Two checkpoints (reference: engine_factory.cpp:64-72): when decode_model_path names another directory, its
        // group-wise INT4 tensors (<linear>.qweight / .scaling_factors) become the decode pass's weights; prefill keeps
        // the bf16 ones.  Tensors of other kinds in that directory are ignored.
        const std::string decode_path = config.decode_model_path();
        if (!decode_path.empty() && decode_path != config.prefill_model_path()) {
            const std::vector<std::string> dfiles = collect_safetensors_files(decode_path);
            if (dfiles.empty()) throw ConfigurationError("No model.safetensors or model-*-of-*.safetensors found in decode path");
            for (const std::string& f : dfiles) {
                SafeTensorsFile dm(f);
                for (const SafeTensorEntry& e : dm.entries()) {
                    std::string name = e.name;
                    if (vlm && !map_vlm_weight_name(e.name, &name)) continue;
                    const int32_t code = backend_dtype_code(e.dtype);
                    if (code < 0) continue;
                    st = efm_b200_set_decode_weight(setup.ctx, name.c_str(), e.data, e.shape.data(), (int32_t)e.shape.size(), code, EFM_MEM_HOST);
                    if (st == EFM_ERR_UNSUPPORTED) throw ConfigurationError(std::string("decode checkpoint, ") + name + ": " + efm_b200_last_error(setup.ctx));
                    if (st != EFM_OK) throw ModelNotLoadedError(std::string("loading decode weight ") + name + ": " + efm_b200_last_error(setup.ctx));
                }
            }
        }
        st = efm_b200_finalize_weights(setup.ctx);
        if (st != EFM_OK) throw ModelNotLoadedError(std::string("checkpoint incomplete: ") + efm_b200_last_error(setup.ctx));
        maps.clear();

        KVGeometry geo;
        geo.num_layers = d.num_layers;
        geo.kv_heads = d.kv_heads;
        geo.head_dim = d.head_dim;
        geo.dtype = DType::BFloat16;
        setup.kv_manager = std::make_shared<KVManager>(reqs, geo, attn, setup.device_id, std::make_shared<BackendKVAllocator>(setup.ctx));
        if (tp > 1) {      // decode all-reduces inside the GEMVs over peer memory: exchange the buffer handles, then a barrier
            std::vector<char> mine(64, 0);
            check_backend(efm_b200_tp_peer_export(setup.ctx, mine.data()), setup.ctx, "peer buffer export");
            const std::vector<std::vector<char>> all = meet->all_gather("peer", mine);
            std::vector<char> flat;
            for (const auto& h : all) {
                if (h.size() != 64) throw ConfigurationError("tensor parallel rendezvous: malformed peer handle");
                flat.insert(flat.end(), h.begin(), h.end());
            }
            check_backend(efm_b200_tp_peer_import(setup.ctx, flat.data(), tp), setup.ctx, "peer buffer import");
            meet->barrier("ready");
        }

        const std::string pa = config.prefill_attention();
        if (pa == "int8") check_backend(efm_b200_set_prefill_attention(setup.ctx, 1), setup.ctx, "prefill attention selection");
        else if (pa != "bf16") throw ConfigurationError("runtime.prefill_attention must be \"bf16\" or \"int8\", got " + pa);
    } catch (...) {
        efm_b200_destroy(setup.ctx);
        throw;
    }
    return setup;
}

const ModelRegistrar kQwen({"qwen2_5", {}, build_qwen});
const ModelRegistrar kQwenVl({"qwen2_5_vl", {}, build_qwen});

}  // namespace

}  // namespace edge_fm
