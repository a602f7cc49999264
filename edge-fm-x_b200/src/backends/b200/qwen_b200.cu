// Qwen2.5 / Qwen2.5-VL text tower behind the C ABI: context creation, tensor parallelism, weight ingestion (fusing
// q|k|v and interleaving gate/up as the kernels expect), the optional INT4 decode copies, slot layout and byte counts.
#include <cmath>
#include <cstdio>

#include "../../layers/launch.cuh"
#include "../../layers/qwen_text.h"
#include "../../operators/gemm_tc.cuh"
#define EFM_DECLARATIONS_ONLY
#include "../../operators/sample.cuh"
#undef EFM_DECLARATIONS_ONLY
#include "ctx.h"
#include "ctx_util.h"
#include "nccl_glue.h"
#include "text_device.h"

using namespace efm;

namespace {

enum : uint32_t { kQw = 1, kQb = 2, kKw = 4, kKb = 8, kVw = 16, kVb = 32, kO = 64, kGate = 128, kUp = 256,
                  kDown = 512, kInNorm = 1024, kPostNorm = 2048 };
constexpr uint32_t kRequired = kQw | kKw | kVw | kO | kGate | kUp | kDown | kInNorm | kPostNorm;

extern const ModelOps kQwenOps;
}  // namespace

extern "C" {

efm_status efm_b200_create(const efm_model_desc* desc, int32_t device_id, int32_t tp_rank, int32_t tp_size,
                           efm_b200_ctx** out) {
    if (desc == nullptr || out == nullptr) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "null argument");
    *out = nullptr;
    if (desc->struct_size != (int32_t)sizeof(efm_model_desc))
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "efm_model_desc.struct_size mismatch");
    const efm_model_desc& d = *desc;
    if (d.num_layers <= 0 || d.hidden <= 0 || d.q_heads <= 0 || d.kv_heads <= 0 || d.vocab <= 0 || d.intermediate <= 0)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "non-positive model dimension");
    if (d.head_dim != 64 && d.head_dim != 128) return fail(nullptr, EFM_ERR_UNSUPPORTED, "head_dim must be 64 or 128");
    if (d.q_heads % d.kv_heads != 0 || d.q_heads / d.kv_heads > kMaxGroup)
        return fail(nullptr, EFM_ERR_UNSUPPORTED, "q_heads / kv_heads must be an integer <= 8");
    if (d.hidden % 32 != 0 || d.intermediate % 64 != 0 || d.vocab % 2 != 0)
        return fail(nullptr, EFM_ERR_UNSUPPORTED, "hidden % 32, intermediate % 64 and vocab % 2 must be 0");
    if (d.use_mrope && d.mrope_section[0] + d.mrope_section[1] + d.mrope_section[2] != d.head_dim / 2)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "mrope_section must sum to head_dim / 2");
    if (tp_size < 1 || tp_rank < 0 || tp_rank >= tp_size) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "bad tensor-parallel coordinates");
    // heads are sharded min(tp, kv_heads) ways; beyond that, ranks pair up on a head shard and split o_proj's input
    const int att_shards = std::min(tp_size, d.kv_heads);
    if (tp_size % att_shards != 0 || d.kv_heads % att_shards != 0 || d.q_heads % att_shards != 0)
        return fail(nullptr, EFM_ERR_UNSUPPORTED, "tensor-parallel size must divide (or be a multiple of) the kv head count");
    const int att_rep = tp_size / att_shards;
    if (d.intermediate % (64 * tp_size) != 0 || d.vocab % (2 * tp_size) != 0 ||
        ((d.q_heads / att_shards) * d.head_dim) % (32 * att_rep) != 0)
        return fail(nullptr, EFM_ERR_UNSUPPORTED, "intermediate / vocab / attention width do not split evenly over the ranks");
    if (d.max_prefill_tokens <= 0 || d.max_response_tokens <= 0)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "max_prefill_tokens and max_response_tokens must be positive");
    efm_status st = require_b200(nullptr, device_id);
    if (st != EFM_OK) return st;

    efm_b200_ctx* c = new (std::nothrow) efm_b200_ctx();
    if (c == nullptr) return fail(nullptr, EFM_ERR_OUT_OF_MEMORY, "host allocation failed");
    c->ops = &kQwenOps;
    c->full = d;
    c->d = d;
    c->d.q_heads = d.q_heads / att_shards;
    c->d.kv_heads = d.kv_heads / att_shards;
    c->d.intermediate = d.intermediate / tp_size;
    c->att_shards = att_shards;
    c->att_rep = att_rep;
    c->att_shard = tp_rank / att_rep;
    c->att_rep_idx = tp_rank % att_rep;
    c->o_k = c->d.q_heads * d.head_dim / att_rep;
    c->vocab_l = d.vocab / tp_size;
    c->vocab_off = tp_rank * c->vocab_l;
    c->device = device_id;
    c->tp_rank = tp_rank;
    c->tp_size = tp_size;
    c->pdl = std::getenv("EFM_B200_NO_PDL") == nullptr;
    auto bail = [&](cudaError_t e, const char* what) {
        efm_status s = cuda_fail(nullptr, e, what);
        efm_b200_destroy(c);
        return s;
    };
#define EFM_TRY(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) return bail(e_, #call); } while (0)
    EFM_TRY(cudaDeviceGetAttribute(&c->num_sms, cudaDevAttrMultiProcessorCount, device_id));
    EFM_TRY(cudaStreamCreateWithFlags(&c->stream, cudaStreamNonBlocking));
    for (auto& ev : c->events) EFM_TRY(cudaEventCreate(&ev));

    const efm_model_desc& dl = c->d;
    const size_t H = dl.hidden, D = dl.head_dim, QD = (size_t)dl.q_heads * D, KVD = (size_t)dl.kv_heads * D, I = dl.intermediate,
                 V = dl.vocab, S = dl.max_prefill_tokens;
    EFM_TRY(dev_alloc(c, &c->embed, V * H, false));
    if (d.tied_lm_head) c->lm_head = c->embed + (size_t)c->vocab_off * H;      // this rank's rows of the shared table
    else EFM_TRY(dev_alloc(c, &c->lm_head, (size_t)c->vocab_l * H, false));
    if (tp_size > 1) {
        EFM_TRY(dev_alloc(c, &c->ybuf, S * H));
        EFM_TRY(dev_alloc(c, &c->ysum, S * H));
        EFM_TRY(dev_alloc(c, &c->logits_l, (size_t)c->vocab_l));
        // zeroed: header (counts, tickets, prefill flags) | decode {value, count} words | prefill receive slots | gather buffers
        c->tp_prefill_off = 256 + (((size_t)2 * tp_size * H * 8 + 255) & ~(size_t)255);
        c->tp_slot_floats = ((S + tp_size - 1) / tp_size) * H;
        c->tp_gather_off = c->tp_prefill_off + (((size_t)2 * tp_size * c->tp_slot_floats * sizeof(float) + 255) & ~(size_t)255);
        c->tp_sample_off = c->tp_gather_off + (((size_t)2 * S * H * sizeof(float) + 255) & ~(size_t)255);
        EFM_TRY(dev_alloc(c, &c->tp_xchg, c->tp_sample_off + 256));
        EFM_TRY(cudaHostAlloc(reinterpret_cast<void**>(&c->error_host), sizeof(int), cudaHostAllocMapped));
        *c->error_host = 0;
        if (const char* ms = std::getenv("EFM_B200_PEER_WAIT_MS")) {
            const long v = std::atol(ms);
            if (v > 0) c->peer_wait_ns = (unsigned long long)v * 1000000ull;
        }
        if (const char* ts = std::getenv("EFM_B200_TP_TIMEOUT_S")) {
            const double v = std::atof(ts);
            if (v > 0) c->tp_timeout_s = v;
        }
    }
    EFM_TRY(dev_alloc(c, &c->final_norm, H));
    c->layers.resize(d.num_layers);
    for (auto& w : c->layers) {
        EFM_TRY(dev_alloc(c, &w.in_norm, H));
        EFM_TRY(dev_alloc(c, &w.post_norm, H));
        EFM_TRY(dev_alloc(c, &w.qkv, (QD + 2 * KVD) * H, false));
        EFM_TRY(dev_alloc(c, &w.qkv_bias, QD + 2 * KVD));
        EFM_TRY(dev_alloc(c, &w.o, H * (size_t)c->o_k, false));
        EFM_TRY(dev_alloc(c, &w.gate_up, 2 * I * H, false));
        EFM_TRY(dev_alloc(c, &w.down, H * I, false));
    }
    {
        std::vector<float> f(D / 2);
        for (size_t i = 0; i < D / 2; ++i) f[i] = (float)std::pow((double)d.rope_theta, -2.0 * (double)i / (double)D);
        EFM_TRY(dev_alloc(c, &c->inv_freq, D / 2));
        EFM_TRY(cudaMemcpyAsync(c->inv_freq, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice, c->stream));
        EFM_TRY(cudaStreamSynchronize(c->stream));
    }
    c->max_s = (int)S;
    EFM_TRY(dev_alloc(c, &c->ids, S));
    EFM_TRY(dev_alloc(c, &c->pos3, 3 * S));
    EFM_TRY(dev_alloc(c, &c->resid, S * H));
    EFM_TRY(dev_alloc(c, &c->norm, S * H));
    EFM_TRY(dev_alloc(c, &c->qkv, S * (QD + 2 * KVD)));
    EFM_TRY(dev_alloc(c, &c->qbuf, S * QD));
    EFM_TRY(dev_alloc(c, &c->attn, S * QD));
    EFM_TRY(dev_alloc(c, &c->act, S * I));
    EFM_TRY(dev_alloc(c, &c->resid_d, H));
    EFM_TRY(dev_alloc(c, &c->resid_d2, H));
    EFM_TRY(dev_alloc(c, &c->q_d, QD));
    EFM_TRY(dev_alloc(c, &c->attn_d, QD));
    EFM_TRY(dev_alloc(c, &c->act_d, I));
    EFM_TRY(dev_alloc(c, &c->logits, V));
    EFM_TRY(dev_alloc(c, &c->part_val, 2 * (size_t)c->num_sms + 8));
    EFM_TRY(dev_alloc(c, &c->part_idx, 2 * (size_t)c->num_sms + 8));
    EFM_TRY(dev_alloc(c, &c->wbuf, sample_scratch_words((int)V)));
    EFM_TRY(dev_alloc(c, &c->attn_part_o, (size_t)dl.q_heads * 64 * D));
    EFM_TRY(dev_alloc(c, &c->attn_part_ml, (size_t)dl.q_heads * 64 * 2));
    EFM_TRY(dev_alloc(c, &c->attn_counters, (size_t)dl.kv_heads));
    {   // the longest GEMV input row must fit the kernel's shared memory as fp32
        int optin = 0;
        EFM_TRY(cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, device_id));
        const size_t need = gemv_w4_smem_bytes((int)std::max(H, std::max(QD, I)));
        if (need + 2048 > (size_t)optin) {
            efm_status s = fail(nullptr, EFM_ERR_UNSUPPORTED, "hidden / intermediate size exceeds what the decode GEMV stages in shared memory");
            efm_b200_destroy(c);
            return s;
        }
    }
    c->gemm_ws_floats = (size_t)c->num_sms * 128 * 256;      // splits x tiles never exceeds the SM count
    EFM_TRY(dev_alloc(c, &c->gemm_ws, c->gemm_ws_floats, false));
    EFM_TRY(dev_alloc(c, &c->state, 1));
    EFM_TRY(dev_alloc(c, &c->tokens_out, (size_t)d.max_response_tokens));
    EFM_TRY(cudaStreamSynchronize(c->stream));
#undef EFM_TRY
    *out = c;
    return EFM_OK;
}

efm_status efm_b200_tp_unique_id(void* out128) {
    if (out128 == nullptr) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "null argument");
    const NcclApi& api = nccl_api();
    if (!api.ok) return fail(nullptr, EFM_ERR_UNSUPPORTED, api.error);
    const int r = api.get_unique_id(out128);
    if (r != 0) return fail(nullptr, EFM_ERR_CUDA, std::string("ncclGetUniqueId: ") + api.error_string(r));
    return EFM_OK;
}

efm_status efm_b200_tp_init(efm_b200_ctx* c, const void* id128) {
    if (c == nullptr || id128 == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->tp_size == 1) return EFM_OK;
    if (c->nccl_comm != nullptr) return fail(c, EFM_ERR_STATE, "communicator already initialised");
    const NcclApi& api = nccl_api();
    if (!api.ok) return fail(c, EFM_ERR_UNSUPPORTED, api.error);
    EFM_CK(c, cudaSetDevice(c->device));
    // In-switch (NVLS) collectives bind this rank's buffers to an NVLink multicast object; a rank that dies while bound
    // can fault its peers' GPUs.  Off unless the caller's environment already decided.
    setenv("NCCL_NVLS_ENABLE", "0", 0);
    const int r = api.comm_init_rank(&c->nccl_comm, c->tp_size, id128, c->tp_rank);
    if (r != 0) { c->nccl_comm = nullptr; return fail(c, EFM_ERR_CUDA, std::string("ncclCommInitRank: ") + api.error_string(r)); }
    return EFM_OK;
}

efm_status efm_b200_tp_set_wait_limit(efm_b200_ctx* c, int64_t device_wait_us, double host_timeout_s) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    if (device_wait_us < 0 || host_timeout_s < 0) return fail(c, EFM_ERR_INVALID_ARGUMENT, "limits must be >= 0 (0 keeps the current value)");
    bool changed = false;
    if (device_wait_us > 0) { changed = c->peer_wait_ns != (unsigned long long)device_wait_us * 1000ull; c->peer_wait_ns = (unsigned long long)device_wait_us * 1000ull; }
    if (host_timeout_s > 0) c->tp_timeout_s = host_timeout_s;
    if (changed)     // the device limit is a kernel argument baked into the captured step
        for (auto& kv : c->slots)
            if (kv.second.graph != nullptr) { cudaGraphExecDestroy(kv.second.graph); kv.second.graph = nullptr; }
    return EFM_OK;
}

efm_status efm_b200_tp_host_wait(void* nccl_comm, int (*ready)(void*), void* arg, double timeout_s) {
    if (ready == nullptr || !(timeout_s >= 0)) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "tp_host_wait: bad arguments");
    std::string what;
    const int r = tp_host_wait(nccl_comm, ready, arg, timeout_s, &what);
    if (r == 0) return EFM_OK;
    return fail(nullptr, r == 2 ? EFM_ERR_DEVICE_WAIT : EFM_ERR_CUDA, what);
}

efm_status efm_b200_tp_peer_export(efm_b200_ctx* c, void* handle64) {
    if (c == nullptr || handle64 == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->tp_size == 1 || c->tp_xchg == nullptr) return fail(c, EFM_ERR_STATE, "peer exchange needs tp_size > 1");
    static_assert(sizeof(cudaIpcMemHandle_t) == 64, "handle size");
    EFM_CK(c, cudaSetDevice(c->device));
    EFM_CK(c, cudaStreamSynchronize(c->stream));            // the buffer's zero fill has landed
    cudaIpcMemHandle_t h;
    EFM_CK(c, cudaIpcGetMemHandle(&h, c->tp_xchg));
    std::memcpy(handle64, &h, 64);
    return EFM_OK;
}

efm_status efm_b200_tp_peer_import(efm_b200_ctx* c, const void* handles, int32_t n_handles) {
    if (c == nullptr || handles == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->tp_size == 1 || c->tp_xchg == nullptr) return fail(c, EFM_ERR_STATE, "peer exchange needs tp_size > 1");
    if (n_handles != c->tp_size || c->tp_size > 8) return fail(c, EFM_ERR_INVALID_ARGUMENT, "one handle per rank, at most 8 ranks");
    if (c->peers_ready) return fail(c, EFM_ERR_STATE, "peer buffers are already imported");
    EFM_CK(c, cudaSetDevice(c->device));
    for (int r = 0; r < c->tp_size; ++r) {
        if (r == c->tp_rank) { c->peer_base[r] = c->tp_xchg; continue; }
        cudaIpcMemHandle_t h;
        std::memcpy(&h, static_cast<const char*>(handles) + (size_t)r * 64, 64);
        void* p = nullptr;
        cudaError_t e = cudaIpcOpenMemHandle(&p, h, cudaIpcMemLazyEnablePeerAccess);
        if (e != cudaSuccess) {
            for (int q = 0; q < r; ++q)
                if (q != c->tp_rank && c->peer_base[q] != nullptr) { cudaIpcCloseMemHandle(c->peer_base[q]); c->peer_base[q] = nullptr; }
            return cuda_fail(c, e, "cudaIpcOpenMemHandle (peer exchange buffer)");
        }
        c->peer_base[r] = static_cast<char*>(p);
    }
    for (auto& kv : c->slots)       // decode graphs captured with the NCCL form are rebuilt on next use
        if (kv.second.graph != nullptr) { cudaGraphExecDestroy(kv.second.graph); kv.second.graph = nullptr; }
    drop_prefill_graphs(c);
    c->peers_ready = true;
    return EFM_OK;
}

efm_status efm_b200_set_prefill_attention(efm_b200_ctx* c, int32_t kind) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->decoder != nullptr) return kind == 0 ? EFM_OK : fail(c, EFM_ERR_UNSUPPORTED, "this model has no INT8 prefill attention");
    if (kind != 0 && kind != 1) return fail(c, EFM_ERR_INVALID_ARGUMENT, "prefill attention kind must be 0 (bf16) or 1 (int8)");
    if (kind == 1) {
        int rows = 0;
        for (auto& kv : c->slots) rows = std::max(rows, kv.second.max_tokens);
        if (rows == 0) return fail(c, EFM_ERR_STATE, "allocate the KV slots before selecting the INT8 prefill attention");
        if (c->d.head_dim != 64 && c->d.head_dim != 128) return fail(c, EFM_ERR_UNSUPPORTED, "INT8 prefill attention: head_dim 64 or 128");
        EFM_CK(c, cudaSetDevice(c->device));
        if (rows > c->sage.kv_rows) {
            EFM_CK(c, cudaStreamSynchronize(c->stream));
            free_sage(c->sage);
            cudaError_t e = alloc_sage(c->sage, c->max_s, rows, c->d.q_heads, c->d.kv_heads, c->d.head_dim);
            if (e != cudaSuccess) { free_sage(c->sage); return cuda_fail(c, e, "INT8 attention scratch"); }
        }
    }
    if (c->prefill_attention_kind != kind) drop_prefill_graphs(c);     // the INT8 scratch may have moved as well
    c->prefill_attention_kind = kind;
    return EFM_OK;
}

}  // extern "C"

namespace {

efm_status qwen_set_weight(efm_b200_ctx* c, const char* hf_name, const void* data, const int64_t* shape,
                               int32_t ndim, int32_t dtype, int32_t mem_kind) {
    // The caller always hands over the WHOLE tensor; this rank keeps its slice: q/k/v rows of its head
    // shard, its o_proj input columns, its gate/up rows and down columns, its lm_head rows.
    const efm_model_desc& d = c->d;          // local
    const efm_model_desc& F = c->full;       // whole model
    const int64_t H = d.hidden, D = d.head_dim, I = d.intermediate, V = d.vocab;
    const int64_t QD = d.q_heads * D, KVD = d.kv_heads * D;              // local widths
    const int64_t FQD = F.q_heads * D, FKVD = F.kv_heads * D, FI = F.intermediate;
    const int64_t q_off = (int64_t)c->att_shard * QD, kv_off = (int64_t)c->att_shard * KVD, i_off = (int64_t)c->tp_rank * I;
    const std::string name(hf_name);
    const char* src = static_cast<const char*>(data);
    const cudaMemcpyKind kind = mem_kind == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice;
    auto bad_shape = [&]() { return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + name); };
    auto known = [&]() -> efm_status {
        if (dtype != EFM_BF16) return fail(c, EFM_ERR_UNSUPPORTED, "weights must be bf16: " + name);
        return EFM_OK;
    };
    efm_status st = EFM_OK;
    if (name == "model.embed_tokens.weight") {
        if ((st = known()) != EFM_OK) return st;
        if (!shape_is(shape, ndim, V, H)) return bad_shape();
        st = copy_rows(c, c->embed, data, (size_t)V * H * 2, mem_kind);
        c->seen_embed = true;
    } else if (name == "lm_head.weight") {
        if ((st = known()) != EFM_OK) return st;
        if (!shape_is(shape, ndim, V, H)) return bad_shape();
        if (!d.tied_lm_head) st = copy_rows(c, c->lm_head, src + (size_t)c->vocab_off * H * 2, (size_t)c->vocab_l * H * 2, mem_kind);
        c->seen_lm_head = true;
    } else if (name == "model.norm.weight") {
        if ((st = known()) != EFM_OK) return st;
        if (!shape_is(shape, ndim, H)) return bad_shape();
        st = copy_rows(c, c->final_norm, data, (size_t)H * 2, mem_kind);
        c->seen_final_norm = true;
    } else if (name.rfind("model.layers.", 0) == 0) {
        const size_t dot = name.find('.', 13);
        if (dot == std::string::npos) return EFM_OK;
        const int l = std::atoi(name.substr(13, dot - 13).c_str());
        if (l < 0 || l >= d.num_layers) return EFM_OK;      // e.g. extra layers of a draft model: ignored
        const std::string rest = name.substr(dot + 1);
        LayerWeights& w = c->layers[l];
        if ((st = known()) != EFM_OK) return st;
        const size_t rowb = (size_t)H * 2;
        if (rest == "input_layernorm.weight") {
            if (!shape_is(shape, ndim, H)) return bad_shape();
            st = copy_rows(c, w.in_norm, data, rowb, mem_kind); w.seen |= kInNorm;
        } else if (rest == "post_attention_layernorm.weight") {
            if (!shape_is(shape, ndim, H)) return bad_shape();
            st = copy_rows(c, w.post_norm, data, rowb, mem_kind); w.seen |= kPostNorm;
        } else if (rest == "self_attn.q_proj.weight") {
            if (!shape_is(shape, ndim, FQD, H)) return bad_shape();
            st = copy_rows(c, w.qkv, src + (size_t)q_off * rowb, (size_t)QD * rowb, mem_kind); w.seen |= kQw;
        } else if (rest == "self_attn.k_proj.weight") {
            if (!shape_is(shape, ndim, FKVD, H)) return bad_shape();
            st = copy_rows(c, w.qkv + QD * H, src + (size_t)kv_off * rowb, (size_t)KVD * rowb, mem_kind); w.seen |= kKw;
        } else if (rest == "self_attn.v_proj.weight") {
            if (!shape_is(shape, ndim, FKVD, H)) return bad_shape();
            st = copy_rows(c, w.qkv + (QD + KVD) * H, src + (size_t)kv_off * rowb, (size_t)KVD * rowb, mem_kind); w.seen |= kVw;
        } else if (rest == "self_attn.q_proj.bias") {
            if (!shape_is(shape, ndim, FQD)) return bad_shape();
            st = copy_rows(c, w.qkv_bias, src + (size_t)q_off * 2, (size_t)QD * 2, mem_kind); w.seen |= kQb;
        } else if (rest == "self_attn.k_proj.bias") {
            if (!shape_is(shape, ndim, FKVD)) return bad_shape();
            st = copy_rows(c, w.qkv_bias + QD, src + (size_t)kv_off * 2, (size_t)KVD * 2, mem_kind); w.seen |= kKb;
        } else if (rest == "self_attn.v_proj.bias") {
            if (!shape_is(shape, ndim, FKVD)) return bad_shape();
            st = copy_rows(c, w.qkv_bias + QD + KVD, src + (size_t)kv_off * 2, (size_t)KVD * 2, mem_kind); w.seen |= kVb;
        } else if (rest == "self_attn.o_proj.weight") {
            if (!shape_is(shape, ndim, H, FQD)) return bad_shape();
            // this rank's input columns: its head shard, then its share of the shard when ranks pair up
            const int64_t col0 = q_off + (int64_t)c->att_rep_idx * c->o_k;
            EFM_CK(c, cudaMemcpy2DAsync(w.o, (size_t)c->o_k * 2, src + (size_t)col0 * 2, (size_t)FQD * 2, (size_t)c->o_k * 2,
                                        (size_t)H, kind, c->stream));
            w.seen |= kO;
        } else if (rest == "mlp.gate_proj.weight" || rest == "mlp.up_proj.weight") {
            if (!shape_is(shape, ndim, FI, H)) return bad_shape();
            const bool up = rest[4] == 'u';
            // 64-row blocks: gate block b -> fused rows [128b, 128b+64), up block b -> [128b+64, 128b+128)
            EFM_CK(c, cudaMemcpy2DAsync(w.gate_up + (up ? 64 * H : 0), 128 * rowb, src + (size_t)i_off * rowb, 64 * rowb, 64 * rowb,
                                        (size_t)(I / 64), kind, c->stream));
            w.seen |= up ? kUp : kGate;
        } else if (rest == "mlp.down_proj.weight") {
            if (!shape_is(shape, ndim, H, FI)) return bad_shape();
            EFM_CK(c, cudaMemcpy2DAsync(w.down, (size_t)I * 2, src + (size_t)i_off * 2, (size_t)FI * 2, (size_t)I * 2, (size_t)H, kind,
                                        c->stream));
            w.seen |= kDown;
        } else {
            return EFM_OK;
        }
    } else {
        return EFM_OK;   // visual tower etc.: not part of this path
    }
    if (st != EFM_OK) return st;
    EFM_CK(c, cudaStreamSynchronize(c->stream));   // the caller may release `data` on return
    return EFM_OK;
}

efm_status qwen_set_decode_weight(efm_b200_ctx* c, const char* hf_name, const void* data, const int64_t* shape, int32_t ndim,
                                      int32_t dtype, int32_t mem_kind) {
    if (c->tp_size > 1) return fail(c, EFM_ERR_UNSUPPORTED, "INT4 decode weights are not sharded: tensor-parallel contexts decode in bf16");
    const efm_model_desc& d = c->d;
    const int64_t H = d.hidden, D = d.head_dim, I = d.intermediate, V = d.vocab, QD = d.q_heads * D, KVD = d.kv_heads * D;
    std::string name(hf_name);
    bool is_q;
    const std::string qs = ".qweight", ss = ".scaling_factors";
    if (name.size() > qs.size() && name.compare(name.size() - qs.size(), qs.size(), qs) == 0) { is_q = true; name.resize(name.size() - qs.size()); }
    else if (name.size() > ss.size() && name.compare(name.size() - ss.size(), ss.size(), ss) == 0) { is_q = false; name.resize(name.size() - ss.size()); }
    else return EFM_OK;                                   // bf16 tensors of a decode checkpoint: the prefill copy serves
    W4Linear* lin = nullptr;
    int src = 0;
    int64_t rows = 0, K = 0;
    if (name == "lm_head") { lin = &c->w4_lm_head; rows = V; K = H; }
    else if (name.rfind("model.layers.", 0) == 0) {
        const size_t dot = name.find('.', 13);
        if (dot == std::string::npos) return EFM_OK;
        const int l = std::atoi(name.substr(13, dot - 13).c_str());
        if (l < 0 || l >= d.num_layers) return EFM_OK;
        const std::string rest = name.substr(dot + 1);
        LayerWeights& w = c->layers[l];
        if (rest == "self_attn.q_proj") { lin = &w.w4_qkv; src = 0; rows = QD; K = H; }
        else if (rest == "self_attn.k_proj") { lin = &w.w4_qkv; src = 1; rows = KVD; K = H; }
        else if (rest == "self_attn.v_proj") { lin = &w.w4_qkv; src = 2; rows = KVD; K = H; }
        else if (rest == "self_attn.o_proj") { lin = &w.w4_o; rows = H; K = QD; }
        else if (rest == "mlp.gate_proj") { lin = &w.w4_gate_up; src = 0; rows = I; K = H; }
        else if (rest == "mlp.up_proj") { lin = &w.w4_gate_up; src = 1; rows = I; K = H; }
        else if (rest == "mlp.down_proj") { lin = &w.w4_down; rows = H; K = I; }
        else return EFM_OK;
    } else {
        return EFM_OK;
    }
    if (K % kW4Group != 0 || rows % 2 != 0)
        return fail(c, EFM_ERR_UNSUPPORTED, "INT4 linear needs in_features % 128 == 0 and even out_features: " + std::string(hf_name));
    size_t bytes;
    if (is_q) {
        if (dtype != EFM_I8 && dtype != EFM_U8) return fail(c, EFM_ERR_UNSUPPORTED, "qweight must be int8 (two 4-bit values per byte): " + std::string(hf_name));
        if (!shape_is(shape, ndim, rows / 2, K)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + std::string(hf_name) + " (want [out_features / 2, in_features])");
        bytes = (size_t)(rows / 2) * K;
    } else {
        if (dtype != EFM_F16 && dtype != EFM_BF16) return fail(c, EFM_ERR_UNSUPPORTED, "scaling_factors must be fp16 or bf16: " + std::string(hf_name));
        if (!shape_is(shape, ndim, K / kW4Group, rows)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + std::string(hf_name) + " (want [in_features / 128, out_features])");
        bytes = (size_t)(K / kW4Group) * rows * 2;
        lin->src_s_bf16[src] = dtype == EFM_BF16;
    }
    void** slot = is_q ? &lin->src_q[src] : &lin->src_s[src];
    if (*slot == nullptr) {
        cudaError_t e = cudaMalloc(slot, bytes);          // released again by finalize_weights
        if (e != cudaSuccess) { *slot = nullptr; return cuda_fail(c, e, "staging an INT4 tensor"); }
    }
    EFM_CK(c, cudaMemcpyAsync(*slot, data, bytes, mem_kind == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice, c->stream));
    EFM_CK(c, cudaStreamSynchronize(c->stream));
    return EFM_OK;
}

// kind: 0 neighbours, 1 rotary partners, 2 gate / up
efm_status finish_w4_linear(efm_b200_ctx* c, W4Linear& lin, int n_src, const int rows[3], int K, int kind, const char* what) {
    if (!lin.any()) return EFM_OK;
    if (!lin.complete(n_src)) return fail(c, EFM_ERR_STATE, std::string("INT4 decode weights incomplete (qweight and scaling_factors of every part): ") + what);
    int total_rows = 0;
    for (int i = 0; i < n_src; ++i) total_rows += rows[i];
    lin.n_items = total_rows / 2;
    lin.K = K;
    if (K % kW4Group != 0) return fail(c, EFM_ERR_UNSUPPORTED, std::string("INT4 decode weights need in_features % 128 == 0: ") + what);
    const size_t padded = (size_t)((lin.n_items + 7) / 8) * 8;          // whole 16-row tiles; the padding holds zeros
    EFM_CK(c, dev_alloc(c, &lin.q, padded * K, false));
    __half2* s = nullptr;
    EFM_CK(c, dev_alloc(c, &s, padded * (K / kW4Group), false));
    lin.s = s;
    W4RepackParams p{};
    int row0 = 0;
    for (int i = 0; i < n_src; ++i) {
        p.q[i] = static_cast<const uint8_t*>(lin.src_q[i]);
        p.s[i] = lin.src_s[i];
        p.row0[i] = row0;
        p.rows[i] = rows[i];
        p.s_is_bf16[i] = lin.src_s_bf16[i];
        row0 += rows[i];
    }
    p.n_src = n_src; p.K = K; p.n_items = lin.n_items; p.kind = kind; p.head_dim = c->d.head_dim; p.half = rows[0];
    p.out_q = lin.q; p.out_s = s;
    Launcher L = make_launcher(c);
    L.counter = nullptr;
    launch_w4_repack(L, p);
    if (L.err != cudaSuccess) return cuda_fail(c, L.err, "INT4 repack launch");
    EFM_CK(c, cudaStreamSynchronize(c->stream));
    for (int i = 0; i < 3; ++i) {
        if (lin.src_q[i] != nullptr) { cudaFree(lin.src_q[i]); lin.src_q[i] = nullptr; }
        if (lin.src_s[i] != nullptr) { cudaFree(lin.src_s[i]); lin.src_s[i] = nullptr; }
    }
    lin.ready = true;
    return EFM_OK;
}

efm_status qwen_finalize(efm_b200_ctx* c) {
    if (!c->seen_embed) return fail(c, EFM_ERR_STATE, "missing model.embed_tokens.weight");
    if (!c->seen_final_norm) return fail(c, EFM_ERR_STATE, "missing model.norm.weight");
    if (!c->d.tied_lm_head && !c->seen_lm_head) return fail(c, EFM_ERR_STATE, "missing lm_head.weight (untied model)");
    for (int l = 0; l < c->d.num_layers; ++l)
        if ((c->layers[l].seen & kRequired) != kRequired)
            return fail(c, EFM_ERR_STATE, "missing weights in layer " + std::to_string(l));
    EFM_CK(c, cudaStreamSynchronize(c->stream));
    {   // INT4 copies of the decode linears, when a decode checkpoint supplied them: all layers or none
        const efm_model_desc& d = c->d;
        const int D = d.head_dim, QD = d.q_heads * D, KVD = d.kv_heads * D;
        bool all = true, any = c->w4_lm_head.any();
        for (auto& w : c->layers) any = any || w.w4_qkv.any() || w.w4_o.any() || w.w4_gate_up.any() || w.w4_down.any();
        if (any) {
            for (int l = 0; l < d.num_layers; ++l) {
                LayerWeights& w = c->layers[l];
                const int r_qkv[3] = {QD, KVD, KVD}, r_o[3] = {d.hidden, 0, 0}, r_gu[3] = {d.intermediate, d.intermediate, 0};
                efm_status st = finish_w4_linear(c, w.w4_qkv, 3, r_qkv, d.hidden, 1, "q/k/v_proj");
                if (st == EFM_OK) st = finish_w4_linear(c, w.w4_o, 1, r_o, QD, 0, "o_proj");
                if (st == EFM_OK) st = finish_w4_linear(c, w.w4_gate_up, 2, r_gu, d.hidden, 2, "gate/up_proj");
                if (st == EFM_OK) st = finish_w4_linear(c, w.w4_down, 1, r_o, d.intermediate, 0, "down_proj");
                if (st != EFM_OK) return st;
                all = all && w.w4_qkv.ready && w.w4_o.ready && w.w4_gate_up.ready && w.w4_down.ready;
            }
            const int r_lm[3] = {d.vocab, 0, 0};
            const efm_status st = finish_w4_linear(c, c->w4_lm_head, 1, r_lm, d.hidden, 0, "lm_head");
            if (st != EFM_OK) return st;
            if (!all) return fail(c, EFM_ERR_STATE, "INT4 decode weights must cover q/k/v/o/gate/up/down_proj of every layer (lm_head is optional)");
            c->decode_w4 = true;
        }
    }
    c->finalized = true;
    return EFM_OK;
}

efm_status qwen_alloc_slot(efm_b200_ctx* c, int32_t slot, int32_t max_tokens) {
    KvSlot s;
    s.max_tokens = max_tokens;
    const size_t block = (size_t)max_tokens * c->d.kv_heads * c->d.head_dim;
    for (int l = 0; l < c->d.num_layers; ++l) {
        __nv_bfloat16* base = nullptr;
        EFM_CK(c, dev_alloc(c, &base, 2 * block));
        s.k.push_back(base);
        s.v.push_back(base + block);
    }
    const AttnPlan plan = plan_decode_attention(max_tokens, c->d.kv_heads, c->num_sms);
    s.n_splits = plan.n_splits;
    s.chunk_cap = plan.chunk_cap;
    s.attn_cluster = plan.cluster;
    EFM_CK(c, cudaStreamSynchronize(c->stream));
    c->slots[slot] = s;
    return EFM_OK;
}

int64_t qwen_step_bytes(const efm_b200_ctx& ctx, int32_t kv_len) {
    const efm_b200_ctx* c = &ctx;
    const efm_model_desc& d = c->d;
    const int64_t H = d.hidden, D = d.head_dim, q = d.q_heads, kv = d.kv_heads, I = d.intermediate, V = d.vocab, L = d.num_layers;
    // what THIS rank streams: its head shard, its o_proj columns, its MLP columns, its lm_head rows
    const int64_t per_layer = (q + 2 * kv) * D * H + (q + 2 * kv) * D + (int64_t)c->o_k * H + 3 * I * H + 2 * H;
    int64_t w = 2 * (L * per_layer + H + (int64_t)c->vocab_l * H) + 2 * H;      // + final norm, lm_head rows, one embedding row
    if (c->decode_w4) {
        // INT4 linears: half a byte per weight + one fp16 scale per 128 weights; biases, norms, embedding row in bf16
        const int64_t lin = (q + 2 * kv) * D * H + q * D * H + 3 * I * H;
        const int64_t lm = V * H;
        const auto w4 = [](int64_t n) { return n / 2 + n / kW4Group * 2; };
        w = L * (w4(lin) + 2 * ((q + 2 * kv) * D + 2 * H)) + 2 * H + (c->w4_lm_head.ready ? w4(lm) : 2 * lm) + 2 * H;
    }
    return w + L * 2 * (int64_t)kv_len * kv * D * 2;
}

void qwen_gather_logits(efm_b200_ctx& c, Launcher& L) {
    if (tp_greedy_exchange(c)) tp_gather_logits(c, L);       // the step exchanged maxima only
}

const ModelOps kQwenOps = {qwen_set_weight, qwen_set_decode_weight, qwen_finalize, qwen_alloc_slot, nullptr, nullptr,
                           qwen_prefill_chunk, qwen_decode_step, qwen_gather_logits, qwen_step_bytes, nullptr};

}  // namespace
