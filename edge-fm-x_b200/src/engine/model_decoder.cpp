// Layered decoders: config.json -> efm_decoder_desc, checkpoint tensors, paged cache.  A family is a reader of its
// config.json; everything behind it (mixers, cache, steps) is shared.
//
// Folizen: "layers" lists {type, mixer, mlp}; type "attention" {heads, kv_heads, dim, vdim, scale, mask.size} or
// "general_delta" {heads, dim}; mlp null or {kind: "dense", ff}; "norm.eps", "token_side.dim", "vocab", "width".  Sizes
// the JSON does not give (rank of the decay projection) are read from the tensors' shapes.
//
// Temuvik: "layers" lists {type, mixer, mlp}; type "attention" {heads, kv_heads, dim, vdim, scale, rot {base, dims},
// mask {size, keep_first}} or "latent_attention" {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims},
// mask {size}}; mlp null or {kind: "moe", expert.ff, router {experts, top, groups {count, keep}}}; "norm.eps",
// "embedding.scale", "loop" {start, stop, times}, "vocab", "width".
//
// Vekolix: "layers" lists {type, mixer, mlp}; type "latent_attention" {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot} or
// "parallel" {left {heads, kv_heads, dim, vdim, scale, rot}, right {heads, dim, vdim, decay}, left_scale, right_scale}; rot {base,
// dims, scaling {factor, original, fast, slow}}; mlp null, {kind: "dense", ff} or {kind: "moe", expert {ff, limit}, router
// {experts, top}, shared {ff, limit}}; "norm.eps", "residual_mult", "logit_scale", "logit_softcap", "vocab", "width".
//
// Viladra: "layers" lists {type, mixer, mlp}; type "retention" {heads, dim, vdim, decay, rot {base, dims}}, "gla" {heads, dim, vdim, tau}
// or "attention" {heads, kv_heads, dim, vdim, scale, mask.size}; mlp null or {kind: "moe", expert.ff, router {experts, top, scale},
// shared.ff}; "canon.taps", "embedding.scale", "norm.eps", "logit_softcap", "vocab", "width".
#include <efm_b200.h>

#include <algorithm>
#include <cstring>
#include <map>

#include "model_registry.h"
#include "safetensors.h"

namespace edge_fm {

namespace {

struct DecoderConfig {
    efm_decoder_desc desc{};
    std::vector<efm_decoder_layer> layers;
    std::vector<std::vector<double>> decays;             // by layer; efm_decoder_layer::linear_decay points here once all are read
};
using Shapes = std::map<std::string, std::vector<int64_t>>;

const json::Value& member(const json::Value& v, const char* key, const std::string& where) {
    const json::Value* m = v.find(key);
    if (m == nullptr) throw ConfigurationError("config.json: " + where + " lacks \"" + key + "\"");
    return *m;
}
int32_t positive(const json::Value& v, const char* key, const std::string& where) {
    const json::Value& m = member(v, key, where);
    if (!m.is_number() || m.num <= 0) throw ConfigurationError("config.json: " + where + "." + key + " must be a positive number");
    return (int32_t)(m.is_int ? m.inum : (int64_t)m.num);
}

float number(const json::Value& v, const char* key, const std::string& where) {
    const json::Value& m = member(v, key, where);
    if (!m.is_number()) throw ConfigurationError("config.json: " + where + "." + key + " must be a number");
    return (float)m.num;
}
int32_t whole(const json::Value& v, const char* key, const std::string& where) {
    const json::Value& m = member(v, key, where);
    if (!m.is_number() || m.num < 0) throw ConfigurationError("config.json: " + where + "." + key + " must be a number, zero or more");
    return (int32_t)(m.is_int ? m.inum : (int64_t)m.num);
}
bool given(const json::Value* v) { return v != nullptr && v->is_object(); }

// What the layered decoders' configurations share.
void read_model(const json::Value& cfg, efm_decoder_desc& d) {
    d.struct_size = (int32_t)sizeof(d);
    d.vocab = positive(cfg, "vocab", "model");
    d.width = positive(cfg, "width", "model");
    d.norm_eps = (float)member(member(cfg, "norm", "model"), "eps", "norm").num;
    d.embed_scale = 1.0f;
    d.logit_scale = 1.0f;
}
const json::Value& layer_list(const json::Value& cfg) {
    const json::Value& layers = member(cfg, "layers", "model");
    if (!layers.is_array() || layers.arr.empty()) throw ConfigurationError("config.json: \"layers\" must be a non-empty list");
    return layers;
}

DecoderConfig folizen_config(const json::Value& cfg, const Shapes& shapes) {
    DecoderConfig out;
    efm_decoder_desc& d = out.desc;
    read_model(cfg, d);
    const json::Value* side = cfg.find("token_side");
    if (side != nullptr && side->is_object()) d.side_dim = positive(*side, "dim", "token_side");
    const json::Value& layers = layer_list(cfg);
    for (size_t i = 0; i < layers.arr.size(); ++i) {
        const json::Value& l = layers.arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]";
        const json::Value& mix = member(l, "mixer", where);
        const std::string type = l.get_string("type", "");
        efm_decoder_layer e{};
        e.heads = positive(mix, "heads", where + ".mixer");
        e.dim = positive(mix, "dim", where + ".mixer");
        if (type == "attention") {
            e.mixer = EFM_MIXER_ATTENTION;
            e.kv_heads = positive(mix, "kv_heads", where + ".mixer");
            e.vdim = positive(mix, "vdim", where + ".mixer");
            e.scale = (float)member(mix, "scale", where + ".mixer").num;
            e.distance_bias = 1;
            e.head_temp = 1;
            const json::Value* mask = mix.find("mask");
            if (mask != nullptr && mask->is_object()) e.window = positive(*mask, "size", where + ".mixer.mask");
        } else if (type == "general_delta") {
            e.mixer = EFM_MIXER_GENERAL_DELTA;
            const auto it = shapes.find("l" + std::to_string(i) + ".mix.w1");
            if (it == shapes.end() || it->second.size() != 2) throw ModelNotLoadedError("checkpoint lacks l" + std::to_string(i) + ".mix.w1");
            e.decay_rank = (int32_t)it->second[0];
        } else {
            throw ConfigurationError("config.json: " + where + " has an unknown type \"" + type + "\"");
        }
        const json::Value* mlp = l.find("mlp");
        if (mlp != nullptr && mlp->is_object()) {
            const std::string kind = mlp->get_string("kind", "");
            if (kind != "dense") throw ConfigurationError("config.json: " + where + ".mlp has an unknown kind \"" + kind + "\"");
            e.ff = positive(*mlp, "ff", where + ".mlp");
        }
        out.layers.push_back(e);
    }
    d.num_layers = (int32_t)out.layers.size();
    return out;
}

void read_rotation(const json::Value& mix, int32_t kind, const std::string& where, efm_decoder_layer& e) {
    const json::Value& rot = member(mix, "rot", where);
    e.rot_kind = kind;
    e.rot_dims = positive(rot, "dims", where + ".rot");
    e.rot_base = number(rot, "base", where + ".rot");
    const json::Value* scaling = rot.find("scaling");
    if (!given(scaling)) return;
    const std::string in = where + ".rot.scaling";
    for (const char* key : {"factor", "original", "fast", "slow"})
        if (number(*scaling, key, in) <= 0.f) throw ConfigurationError("config.json: " + in + "." + key + " must be positive");
    e.rot_factor = number(*scaling, "factor", in);
    e.rot_original = number(*scaling, "original", in);
    e.rot_fast = number(*scaling, "fast", in);
    e.rot_slow = number(*scaling, "slow", in);
}

void read_experts(const json::Value& mlp, const std::string& where, efm_decoder_layer& e) {
    const std::string kind = mlp.get_string("kind", "");
    if (kind != "moe") throw ConfigurationError("config.json: " + where + " has an unknown kind \"" + kind + "\"");
    e.expert_ff = positive(member(mlp, "expert", where), "ff", where + ".expert");
    const json::Value& router = member(mlp, "router", where);
    e.experts = positive(router, "experts", where + ".router");
    e.expert_top = positive(router, "top", where + ".router");
    e.expert_groups = e.expert_groups_kept = 1;
    const json::Value* groups = router.find("groups");
    if (given(groups)) {
        e.expert_groups = positive(*groups, "count", where + ".router.groups");
        e.expert_groups_kept = positive(*groups, "keep", where + ".router.groups");
    }
}

void read_latent(const json::Value& mix, const std::string& in, efm_decoder_layer& e) {
    e.mixer = EFM_MIXER_LATENT_ATTENTION;
    e.heads = positive(mix, "heads", in);
    e.dim = positive(mix, "dim", in);
    e.vdim = positive(mix, "vdim", in);
    e.scale = number(mix, "scale", in);
    e.q_rank = positive(mix, "q_rank", in);
    e.kv_rank = positive(mix, "kv_rank", in);
    read_rotation(mix, EFM_ROT_PAIRS, in, e);
    if (positive(mix, "rot_dim", in) != e.rot_dims) throw ConfigurationError("config.json: " + in + ".rot.dims must be rot_dim");
}

DecoderConfig temuvik_config(const json::Value& cfg, const Shapes&) {
    DecoderConfig out;
    efm_decoder_desc& d = out.desc;
    read_model(cfg, d);
    d.norm_layout = EFM_NORM_SANDWICH;
    d.embed_scale = number(member(cfg, "embedding", "model"), "scale", "embedding");
    const json::Value& layers = layer_list(cfg);
    for (size_t i = 0; i < layers.arr.size(); ++i) {
        const json::Value& l = layers.arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]", in = where + ".mixer";
        const json::Value& mix = member(l, "mixer", where);
        const std::string type = l.get_string("type", "");
        efm_decoder_layer e{};
        const json::Value* mask = mix.find("mask");
        if (given(mask)) e.window = positive(*mask, "size", in + ".mask");
        if (type == "attention") {
            e.mixer = EFM_MIXER_ATTENTION;
            e.heads = positive(mix, "heads", in);
            e.dim = positive(mix, "dim", in);
            e.vdim = positive(mix, "vdim", in);
            e.scale = number(mix, "scale", in);
            e.kv_heads = positive(mix, "kv_heads", in);
            e.qk_norm = EFM_QK_NORM_PLAIN;
            e.qkv_bias = 1;
            if (given(mask) && mask->find("keep_first") != nullptr) e.keep_first = whole(*mask, "keep_first", in + ".mask");
            read_rotation(mix, EFM_ROT_HALF, in, e);
        } else if (type == "latent_attention") {
            read_latent(mix, in, e);
            e.sink = 1;
            e.out_gate = EFM_GATE_CHANNELS;
        } else {
            throw ConfigurationError("config.json: " + where + " has an unknown type \"" + type + "\"");
        }
        const json::Value* mlp = l.find("mlp");
        if (given(mlp)) read_experts(*mlp, where + ".mlp", e);
        out.layers.push_back(e);
    }
    d.num_layers = (int32_t)out.layers.size();
    const json::Value* loop = cfg.find("loop");
    if (given(loop)) {
        d.loop_start = whole(*loop, "start", "loop");
        d.loop_stop = whole(*loop, "stop", "loop");
        d.loop_times = positive(*loop, "times", "loop");
        if (d.loop_stop <= d.loop_start || d.loop_stop > d.num_layers) throw ConfigurationError("config.json: loop.start .. loop.stop must be a span of the layers");
    }
    return out;
}

void read_decay(const json::Value& mix, int32_t heads, const std::string& in, std::vector<double>& decay) {
    const json::Value& d = member(mix, "decay", in);
    if (!d.is_array() || (int32_t)d.arr.size() != heads) throw ConfigurationError("config.json: " + in + ".decay must list one number per head");
    for (const json::Value& v : d.arr) {
        if (!v.is_number()) throw ConfigurationError("config.json: " + in + ".decay must list one number per head");
        decay.push_back(v.num);
    }
}

void read_parallel(const json::Value& mix, const std::string& in, efm_decoder_layer& e, std::vector<double>& decay) {
    e.mixer = EFM_MIXER_PARALLEL;
    const json::Value &left = member(mix, "left", in), &right = member(mix, "right", in);
    const std::string l = in + ".left", r = in + ".right";
    e.heads = positive(left, "heads", l);
    e.kv_heads = positive(left, "kv_heads", l);
    e.dim = positive(left, "dim", l);
    e.vdim = positive(left, "vdim", l);
    e.scale = number(left, "scale", l);
    e.qk_norm = EFM_QK_NORM_NONE;
    read_rotation(left, EFM_ROT_HALF, l, e);
    e.linear_heads = positive(right, "heads", r);
    e.linear_dim = positive(right, "dim", r);
    e.linear_vdim = positive(right, "vdim", r);
    e.mix_scale = number(mix, "left_scale", in);
    e.linear_scale = number(mix, "right_scale", in);
    read_decay(right, e.linear_heads, r, decay);
}

DecoderConfig vekolix_config(const json::Value& cfg, const Shapes&) {
    DecoderConfig out;
    efm_decoder_desc& d = out.desc;
    read_model(cfg, d);
    d.norm_layout = EFM_NORM_INPUT;
    d.tied_head = 1;
    d.residual_mult = number(cfg, "residual_mult", "model");
    d.logit_scale = number(cfg, "logit_scale", "model");
    d.logit_softcap = number(cfg, "logit_softcap", "model");
    const json::Value& layers = layer_list(cfg);
    out.decays.resize(layers.arr.size());
    for (size_t i = 0; i < layers.arr.size(); ++i) {
        const json::Value& l = layers.arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]", in = where + ".mixer", ff = where + ".mlp";
        const json::Value& mix = member(l, "mixer", where);
        const std::string type = l.get_string("type", "");
        efm_decoder_layer e{};
        if (type == "latent_attention") {
            read_latent(mix, in, e);
            e.out_gate = EFM_GATE_HEADS;
        } else if (type == "parallel") {
            read_parallel(mix, in, e, out.decays[i]);
        } else {
            throw ConfigurationError("config.json: " + where + " has an unknown type \"" + type + "\"");
        }
        const json::Value* mlp = l.find("mlp");
        if (given(mlp) && mlp->get_string("kind", "") == "dense") {
            e.ff = positive(*mlp, "ff", ff);
            e.ff_act = EFM_ACT_RELU2;
        } else if (given(mlp)) {
            read_experts(*mlp, ff, e);
            e.expert_glu = EFM_GLU_CLAMPED;
            e.expert_score = EFM_SCORE_SIGMOID;
            e.expert_weight_input = 1;
            e.expert_limit = number(member(*mlp, "expert", ff), "limit", ff + ".expert");
            const json::Value* shared = mlp->find("shared");
            if (given(shared)) {
                e.shared_ff = positive(*shared, "ff", ff + ".shared");
                e.shared_limit = number(*shared, "limit", ff + ".shared");
            }
        }
        out.layers.push_back(e);
    }
    d.num_layers = (int32_t)out.layers.size();
    return out;
}

DecoderConfig viladra_config(const json::Value& cfg, const Shapes& shapes) {
    DecoderConfig out;
    efm_decoder_desc& d = out.desc;
    read_model(cfg, d);
    d.norm_layout = EFM_NORM_OUTPUT;
    d.tied_head = 1;
    d.depth_average = 1;
    d.conv_taps = positive(member(cfg, "canon", "model"), "taps", "canon");
    d.embed_scale = number(member(cfg, "embedding", "model"), "scale", "embedding");
    d.logit_softcap = number(cfg, "logit_softcap", "model");
    if (!(d.logit_softcap > 0.f)) throw ConfigurationError("config.json: logit_softcap must be positive");
    const json::Value& layers = layer_list(cfg);
    out.decays.resize(layers.arr.size());
    for (size_t i = 0; i < layers.arr.size(); ++i) {
        const json::Value& l = layers.arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]", in = where + ".mixer", ff = where + ".mlp";
        const json::Value& mix = member(l, "mixer", where);
        const std::string type = l.get_string("type", "");
        efm_decoder_layer e{};
        e.heads = positive(mix, "heads", in);
        e.dim = positive(mix, "dim", in);
        e.vdim = positive(mix, "vdim", in);
        if (type == "attention") {
            e.mixer = EFM_MIXER_ATTENTION;
            e.kv_heads = positive(mix, "kv_heads", in);
            e.scale = number(mix, "scale", in);
            e.qk_norm = EFM_QK_NORM_ROW;
            e.qkv_bias = e.out_bias = 1;
            e.score_weights = EFM_WEIGHTS_SIGMOID;
            e.out_gate = EFM_GATE_HEADS;
            const json::Value* mask = mix.find("mask");
            if (given(mask)) e.window = positive(*mask, "size", in + ".mask");
        } else if (type == "retention" || type == "gla") {
            e.mixer = EFM_MIXER_LINEAR;
            e.linear_heads = e.heads;
            e.linear_dim = e.dim;
            e.linear_vdim = e.vdim;
            if (type == "retention") {
                read_rotation(mix, EFM_ROT_HALF, in, e);
                read_decay(mix, e.heads, in, out.decays[i]);
            } else {
                e.linear_norm = 1;
                e.linear_tau = number(mix, "tau", in);
                if (!(e.linear_tau > 0.f)) throw ConfigurationError("config.json: " + in + ".tau must be positive");
                const std::string a1 = "l" + std::to_string(i) + ".mix.a1";
                const auto it = shapes.find(a1);
                if (it == shapes.end() || it->second.size() != 2) throw ModelNotLoadedError("checkpoint lacks " + a1);
                e.decay_rank = (int32_t)it->second[0];
            }
        } else {
            throw ConfigurationError("config.json: " + where + " has an unknown type \"" + type + "\"");
        }
        const json::Value* mlp = l.find("mlp");
        if (given(mlp)) {
            read_experts(*mlp, ff, e);
            e.expert_glu = EFM_GLU_NONE_RELU2;
            e.expert_scale = number(member(*mlp, "router", ff), "scale", ff + ".router");
            if (!(e.expert_scale > 0.f)) throw ConfigurationError("config.json: " + ff + ".router.scale must be positive");
            e.shared_gate = EFM_SHARED_PLAIN;
            const json::Value* shared = mlp->find("shared");
            if (given(shared)) e.shared_ff = positive(*shared, "ff", ff + ".shared");
        }
        out.layers.push_back(e);
    }
    d.num_layers = (int32_t)out.layers.size();
    return out;
}

// Page lists go to the device context; declared slots get their pages once, for good.
class DevicePageMapper : public PageMapper {
public:
    explicit DevicePageMapper(efm_b200_ctx* ctx) : ctx_(ctx) {}
    void map(int32_t slot, const std::vector<int32_t>& pages, int32_t state_slot) override {
        check_backend(efm_b200_decoder_map_slot(ctx_, slot, pages.data(), (int32_t)pages.size(), state_slot), ctx_, "mapping cache pages");
    }
    void unmap(int32_t slot) override { check_backend(efm_b200_decoder_unmap_slot(ctx_, slot), ctx_, "unmapping cache pages"); }

private:
    efm_b200_ctx* ctx_;
};

// Keeps the mapper alive next to the cache that uses it.
class OwningPagedCache : public PagedCache {
public:
    OwningPagedCache(int32_t pages, int32_t states, std::unique_ptr<PageMapper> mapper)
        : PagedCache(pages, states, mapper.get()), mapper_own_(std::move(mapper)) {}

private:
    std::unique_ptr<PageMapper> mapper_own_;
};

class PagedKVAllocator : public KVBufferAllocator {
public:
    explicit PagedKVAllocator(std::shared_ptr<PagedCache> cache) : cache_(std::move(cache)) {}
    Device device() const override { return Device::GPU; }
    std::vector<void*> allocate_slot(int32_t request_id, int32_t max_tokens, size_t, int32_t) override {
        if (!cache_->reserve(request_id, max_tokens)) throw OutOfMemoryError("the cache pool has no room for request_id " + std::to_string(request_id));
        return {};
    }

private:
    std::shared_ptr<PagedCache> cache_;
};

ModelSetup build_decoder(const EngineConfig& config, DecoderConfig (*read)(const json::Value&, const Shapes&)) {
    const std::vector<std::string> files = collect_safetensors_files(config.prefill_model_path());
    if (files.empty())
        throw ConfigurationError("No model.safetensors or model-*-of-*.safetensors found in: " + config.prefill_model_path());
    std::vector<std::unique_ptr<SafeTensorsFile>> maps;
    Shapes shapes;
    for (const std::string& f : files) {
        maps.emplace_back(new SafeTensorsFile(f));
        for (const SafeTensorEntry& e : maps.back()->entries()) shapes[e.name] = e.shape;
    }
    DecoderConfig dc = read(config.prefill_model_config(), shapes);
    efm_decoder_desc& d = dc.desc;
    for (size_t i = 0; i < dc.decays.size(); ++i)
        if (!dc.decays[i].empty()) dc.layers[i].linear_decay = dc.decays[i].data();

    const std::string compute = config.compute_dtype();
    if (compute != "bf16" && compute != "fp32") throw ConfigurationError("runtime.compute_dtype must be \"bf16\" or \"fp32\", got " + compute);
    d.compute_dtype = compute == "fp32" ? EFM_F32 : EFM_BF16;
    const DType cache_dtype = dtype_from_string(config.kvcache_dtype());
    if (cache_dtype != (compute == "fp32" ? DType::Float32 : DType::BFloat16))
        throw ConfigurationError("kvcache.dtype must be " + compute + " with runtime.compute_dtype " + compute);
    if (config.tensor_parallel() != 1) throw ConfigurationError("runtime.tensor_parallel: this model runs on one GPU");
    if (config.prefill_attention() != "bf16") throw ConfigurationError("runtime.prefill_attention: this model has one form only");
    const std::string decode_path = config.decode_model_path();
    if (!decode_path.empty() && decode_path != config.prefill_model_path()) throw ConfigurationError("decode_model_path: this model takes no second checkpoint");

    const std::vector<KvRequestConfig> reqs = config.kv_requests();
    const int32_t pool = std::max(0, config.kv_pool_tokens()), live = pool > 0 ? std::max(1, config.kv_max_live_requests()) : 0;
    int64_t pages = PagedCache::pages_for(pool);
    int32_t longest = pool, states = live;
    for (const KvRequestConfig& r : reqs) {
        pages += PagedCache::pages_for(std::max(1, r.max_tokens));
        longest = std::max(longest, r.max_tokens);
        states += 1 + (r.prefix_token_ids.empty() ? 0 : 1);
    }
    if (pages <= 0) throw ConfigurationError("kvcache declares neither requests nor pool_tokens");
    const bool recurrent = d.conv_taps > 0 || std::any_of(dc.layers.begin(), dc.layers.end(), [](const efm_decoder_layer& l) {
        return l.mixer == EFM_MIXER_GENERAL_DELTA || l.mixer == EFM_MIXER_PARALLEL || l.mixer == EFM_MIXER_LINEAR;
    });
    d.cache_pages = (int32_t)pages;
    d.state_slots = recurrent ? states : 0;
    d.max_slots = (int32_t)reqs.size() + live;
    d.max_step_tokens = std::min(PagedCache::pages_for(longest) * kCachePageTokens, 2048);
    d.max_response_tokens = config.sampling_max_new_tokens() + 1;

    ModelSetup setup;
    setup.device_id = config.runtime_device_id();
    setup.hidden = d.width;
    setup.vocab = d.vocab;
    setup.max_live_requests = live;
    setup.max_step_tokens = d.max_step_tokens;
    const efm_status st = efm_b200_decoder_create(&d, dc.layers.data(), setup.device_id, &setup.ctx);
    if (st != EFM_OK) {
        const std::string msg = std::string("backend creation failed: ") + efm_b200_last_error(nullptr);
        if (st == EFM_ERR_OUT_OF_MEMORY) throw OutOfMemoryError(msg);
        if (st == EFM_ERR_UNSUPPORTED || st == EFM_ERR_INVALID_ARGUMENT) throw ConfigurationError(msg);
        throw DeviceError(msg);
    }
    try {
        for (const auto& m : maps)
            for (const SafeTensorEntry& e : m->entries()) {
                const int32_t code = backend_dtype_code(e.dtype);
                if (code < 0) continue;
                if (efm_b200_set_weight(setup.ctx, e.name.c_str(), e.data, e.shape.data(), (int32_t)e.shape.size(), code, EFM_MEM_HOST) != EFM_OK)
                    throw ModelNotLoadedError("loading " + e.name + ": " + efm_b200_last_error(setup.ctx));
            }
        if (efm_b200_finalize_weights(setup.ctx) != EFM_OK)
            throw ModelNotLoadedError(std::string("checkpoint incomplete: ") + efm_b200_last_error(setup.ctx));
        setup.paged_cache = std::make_shared<OwningPagedCache>(d.cache_pages, d.state_slots, std::unique_ptr<PageMapper>(new DevicePageMapper(setup.ctx)));
        KVGeometry geo;
        geo.paged = true;
        geo.dtype = cache_dtype;
        for (int32_t i = 0; i < d.num_layers; ++i) {
            const efm_decoder_layer& l = dc.layers[i];
            const size_t times = d.loop_times > 1 && i >= d.loop_start && i < d.loop_stop ? d.loop_times : 1;
            if (l.mixer == EFM_MIXER_ATTENTION || l.mixer == EFM_MIXER_PARALLEL) geo.token_bytes += times * l.kv_heads * (l.dim + l.vdim) * get_dtype_size(cache_dtype);
            if (l.mixer == EFM_MIXER_LATENT_ATTENTION) geo.token_bytes += times * (l.kv_rank + l.rot_dims) * get_dtype_size(cache_dtype);
        }
        setup.kv_manager = std::make_shared<KVManager>(reqs, geo, attention_type_from_string(config.kvcache_attention_type()), setup.device_id,
                                                       std::make_shared<PagedKVAllocator>(setup.paged_cache));
    } catch (...) {
        efm_b200_destroy(setup.ctx);
        throw;
    }
    return setup;
}

ModelSetup build_folizen(const EngineConfig& config) { return build_decoder(config, folizen_config); }

ModelSetup build_temuvik(const EngineConfig& config) { return build_decoder(config, temuvik_config); }

ModelSetup build_vekolix(const EngineConfig& config) { return build_decoder(config, vekolix_config); }

ModelSetup build_viladra(const EngineConfig& config) { return build_decoder(config, viladra_config); }

const ModelRegistrar kFolizen({"folizen", {"Folizen"}, build_folizen});
const ModelRegistrar kTemuvik({"temuvik", {"Temuvik"}, build_temuvik});
const ModelRegistrar kVekolix({"vekolix", {"Vekolix"}, build_vekolix});
const ModelRegistrar kViladra({"viladra", {"Viladra"}, build_viladra});

}  // namespace

}  // namespace edge_fm
