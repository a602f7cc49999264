// Model-independent part of the C ABI declared in include/efm_b200.h: errors, context teardown, KV slots, sampling
// parameters, the prefill and decode entry points with CUDA-graph capture, read-back and timing.  What depends on the
// model (weights, slot layout, launch sequences) is behind the context's ModelOps (ctx.h); each family creates its
// contexts in its own file.
#include <algorithm>
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <cmath>
#include <new>
#include <string>

#include "../../operators/gemv_w4.cuh"
#include "ctx.h"
#include "ctx_util.h"
#include "nccl_glue.h"

using namespace efm;

namespace efm {

std::string& create_error() {
    static thread_local std::string e;
    return e;
}

efm_status require_device(efm_b200_ctx* c, int device_id) {
    int n = 0;
    cudaError_t e = cudaGetDeviceCount(&n);
    if (e != cudaSuccess || n == 0)
        return fail(c, EFM_ERR_CUDA, std::string("no CUDA device available: ") + cudaGetErrorString(e));
    if (device_id < 0 || device_id >= n) return fail(c, EFM_ERR_INVALID_ARGUMENT, "device_id out of range");
    int major = 0;
    EFM_CK(c, cudaDeviceGetAttribute(&major, cudaDevAttrComputeCapabilityMajor, device_id));
    if (major != 10) return fail(c, EFM_ERR_CUDA, "device is not sm_100 (this library carries sm_100a code only)");
    EFM_CK(c, cudaSetDevice(device_id));
    return EFM_OK;
}

Launcher make_launcher(efm_b200_ctx* c) {
    Launcher L;
    L.stream = c->stream;
    L.pdl = c->pdl;
    L.counter = &c->launches;
    L.gemm_ws = c->gemm_ws;
    L.gemm_ws_floats = c->gemm_ws_floats;
    L.num_sms = c->num_sms;
    return L;
}

// Stream synchronisation of a context.  Tensor-parallel contexts do not block inside the driver: they poll the stream
// and NCCL's asynchronous error state, and give up after tp_timeout_s (the communicator is then aborted and gone).
static int stream_ready(void* stream) { return cudaStreamQuery(static_cast<cudaStream_t>(stream)) != cudaErrorNotReady; }
efm_status ctx_sync(efm_b200_ctx* c) {
    if (c->tp_size > 1 && c->nccl_comm != nullptr) {
        std::string what;
        const int r = tp_host_wait(c->nccl_comm, stream_ready, c->stream, c->tp_timeout_s, &what);
        if (r != 0) {
            c->nccl_comm = nullptr;       // aborted
            return fail(c, r == 2 ? EFM_ERR_DEVICE_WAIT : EFM_ERR_CUDA, what);
        }
    }
    cudaError_t e = cudaStreamSynchronize(c->stream);
    if (e != cudaSuccess) return cuda_fail(c, e, "cudaStreamSynchronize");
    return EFM_OK;
}

void drop_prefill_graphs(efm_b200_ctx* c) {
    for (auto& g : c->prefill_cache)
        if (g.exec != nullptr) cudaGraphExecDestroy(g.exec);
    c->prefill_cache.clear();
}

void drop_decode_graphs(efm_b200_ctx* c) {
    for (auto& kv : c->slots)
        if (kv.second.graph != nullptr) { cudaGraphExecDestroy(kv.second.graph); kv.second.graph = nullptr; }
}

}  // namespace efm

static constexpr size_t kMaxPrefillGraphs = 8;

extern "C" {

const char* efm_b200_version(void) { return "efm_b200 0.1 (sm_100a)"; }

const char* efm_b200_last_error(const efm_b200_ctx* ctx) {
    return ctx != nullptr ? ctx->error.c_str() : create_error().c_str();
}

efm_status efm_b200_destroy(efm_b200_ctx* c) {
    if (c == nullptr) return EFM_OK;
    cudaSetDevice(c->device);
    if (c->stream != nullptr) cudaStreamSynchronize(c->stream);
    if (c->ops != nullptr && c->ops->destroy != nullptr) c->ops->destroy(c);
    drop_decode_graphs(c);         // graphs that hold collective nodes go before their communicator
    drop_prefill_graphs(c);
    for (int r = 0; r < 8; ++r)
        if (c->peers_ready && r != c->tp_rank && c->peer_base[r] != nullptr) cudaIpcCloseMemHandle(c->peer_base[r]);
    if (c->nccl_comm != nullptr && nccl_api().ok) nccl_api().comm_destroy(c->nccl_comm);
    if (c->sage.q8 != nullptr) { cudaFree(c->sage.q8); cudaFree(c->sage.k8); cudaFree(c->sage.vh); cudaFree(c->sage.sq); cudaFree(c->sage.sk); cudaFree(c->sage.kmean); }
    for (void* p : c->allocations) cudaFree(p);
    for (auto& ev : c->events)
        if (ev != nullptr) cudaEventDestroy(ev);
    if (c->stream != nullptr) cudaStreamDestroy(c->stream);
    if (c->error_host != nullptr) cudaFreeHost(c->error_host);
    delete c;
    return EFM_OK;
}

efm_status efm_b200_set_weight(efm_b200_ctx* c, const char* hf_name, const void* data, const int64_t* shape,
                               int32_t ndim, int32_t dtype, int32_t mem_kind) {
    if (c == nullptr || hf_name == nullptr || data == nullptr || (shape == nullptr && ndim != 0))
        return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->finalized) return fail(c, EFM_ERR_STATE, "weights are already finalized");
    EFM_CK(c, cudaSetDevice(c->device));
    return c->ops->set_weight(c, hf_name, data, shape, ndim, dtype, mem_kind);
}

efm_status efm_b200_set_decode_weight(efm_b200_ctx* c, const char* hf_name, const void* data, const int64_t* shape, int32_t ndim,
                                      int32_t dtype, int32_t mem_kind) {
    if (c == nullptr || hf_name == nullptr || data == nullptr || shape == nullptr)
        return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->finalized) return fail(c, EFM_ERR_STATE, "weights are already finalized");
    if (c->ops->set_decode_weight == nullptr) return fail(c, EFM_ERR_UNSUPPORTED, "this model takes no separate decode weights");
    EFM_CK(c, cudaSetDevice(c->device));
    return c->ops->set_decode_weight(c, hf_name, data, shape, ndim, dtype, mem_kind);
}

efm_status efm_b200_finalize_weights(efm_b200_ctx* c) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    return c->ops->finalize(c);
}

efm_status efm_b200_alloc_kv_slot(efm_b200_ctx* c, int32_t slot, int32_t max_tokens) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    if (max_tokens <= 0) return fail(c, EFM_ERR_INVALID_ARGUMENT, "max_tokens must be positive");
    if (c->slots.count(slot)) return fail(c, EFM_ERR_STATE, "slot already allocated");
    EFM_CK(c, cudaSetDevice(c->device));
    return c->ops->alloc_slot(c, slot, max_tokens);
}

efm_status efm_b200_kv_layer_ptr(efm_b200_ctx* c, int32_t slot, int32_t layer, void** k_base, int32_t* max_tokens) {
    if (c == nullptr || k_base == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    auto it = c->slots.find(slot);
    if (it == c->slots.end() || layer < 0 || layer >= (int)it->second.k.size()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "no such slot/layer");
    *k_base = it->second.k[layer];
    if (max_tokens != nullptr) *max_tokens = it->second.max_tokens;
    return EFM_OK;
}

efm_status efm_b200_set_sampling(efm_b200_ctx* c, const efm_sampling* s) {
    if (c == nullptr || s == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (!(s->temperature >= 0.f)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "temperature must be >= 0");
    const bool changed = std::memcmp(&c->sampling, s, sizeof(*s)) != 0;
    c->sampling = *s;
    if (changed) {   // sampling parameters are baked into the captured step
        drop_decode_graphs(c);
        drop_prefill_graphs(c);
    }
    return EFM_OK;
}

efm_status efm_b200_set_prefill_graph(efm_b200_ctx* c, int32_t enable) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    c->prefill_graphs = enable != 0;
    if (!c->prefill_graphs) drop_prefill_graphs(c);
    return EFM_OK;
}

efm_status efm_b200_prefill_graph_stats(efm_b200_ctx* c, int32_t* captured, int64_t* replays) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    int n = 0;
    for (const auto& g : c->prefill_cache) n += g.exec != nullptr ? 1 : 0;
    if (captured != nullptr) *captured = n;
    if (replays != nullptr) *replays = c->prefill_graph_replays;
    return EFM_OK;
}

efm_status efm_b200_prefill(efm_b200_ctx* c, int32_t slot, const int32_t* token_ids, int32_t n_tokens, int32_t kv_offset,
                            const void* embeds, int32_t n_embeds, int32_t embed_token_id, int32_t embeds_mem,
                            const int32_t* pos_ids3, int32_t sample) {
    if (c == nullptr || token_ids == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (!c->finalized) return fail(c, EFM_ERR_STATE, "weights not finalized");
    if (c->tp_size > 1 && c->nccl_comm == nullptr) return fail(c, EFM_ERR_STATE, "tensor-parallel context without efm_b200_tp_init");
    auto it = c->slots.find(slot);
    if (it == c->slots.end()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unknown KV slot " + std::to_string(slot));
    KvSlot& s = it->second;
    if (n_tokens <= 0 || kv_offset < 0) return fail(c, EFM_ERR_INVALID_ARGUMENT, "n_tokens must be > 0 and kv_offset >= 0");
    if ((int64_t)kv_offset + n_tokens > s.max_tokens)
        return fail(c, EFM_ERR_INVALID_ARGUMENT, "prefill exceeds the slot's max_tokens");
    if (pos_ids3 != nullptr && c->pos3 == nullptr) return fail(c, EFM_ERR_UNSUPPORTED, "this model takes no position ids");
    if (c->d.use_mrope && pos_ids3 == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "M-RoPE model needs position ids");
    EFM_CK(c, cudaSetDevice(c->device));
    if (c->ops->prefill_begin != nullptr) {
        const efm_status bs = c->ops->prefill_begin(c, slot, s, n_tokens, kv_offset, embeds != nullptr ? n_embeds : 0);
        if (bs != EFM_OK) return bs;
    }
    const size_t H = c->d.hidden;
    if (embeds != nullptr && n_embeds > 0) {
        const size_t need = (size_t)n_embeds * H;
        if (need > c->custom_embeds_cap) {
            EFM_CK(c, dev_alloc(c, &c->custom_embeds, need, false));
            c->custom_embeds_cap = need;
        }
        EFM_CK(c, cudaMemcpyAsync(c->custom_embeds, embeds, need * 2,
                                  embeds_mem == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice, c->stream));
    } else {
        n_embeds = 0;
    }
    Launcher L = make_launcher(c);
    // A sampled prefill runs its LAST token as a decode step (same arithmetic, K / V rows and logits as if it had been
    // a row of the GEMMs, but with the decode kernels' fp32 activations): every logit vector the caller sees then
    // comes from one set of kernels, and the first sample is as accurate as the later ones.  The rows before it go
    // through the tensor-core GEMMs.  Not when the last token is an injected embedding row or outside the vocabulary.
    const int32_t last_id = token_ids[n_tokens - 1];
    const bool tail = sample != 0 && last_id >= 0 && last_id < c->d.vocab &&
                      !(n_embeds > 0 && last_id >= embed_token_id && last_id < embed_token_id + n_embeds);
    const int n_gemm = tail ? n_tokens - 1 : n_tokens;
    if (sample != 0 && !tail) {
        DecodeState st{};
        st.token = -1;
        st.kv_len = (uint32_t)(kv_offset + n_tokens);
        EFM_CK(c, cudaMemcpyAsync(c->state, &st, sizeof(st), cudaMemcpyHostToDevice, c->stream));
    }
    if (tail) {
        DecodeState st{};
        st.token = last_id;
        st.kv_len = (uint32_t)(kv_offset + n_tokens);
        for (int r = 0; r < 3; ++r) st.pos[r] = pos_ids3 != nullptr ? pos_ids3[(size_t)r * n_tokens + n_tokens - 1] : 0;
        EFM_CK(c, cudaMemcpyAsync(c->state, &st, sizeof(st), cudaMemcpyHostToDevice, c->stream));
    }
    auto run_tail = [&](Launcher& LL) {
        if (!tail) return;
        const bool w4 = c->decode_w4;
        c->decode_w4 = false;            // the first token belongs to the prefill pass: bf16 weights even when decode runs on INT4
        c->ops->decode_step(*c, s, LL);
        c->decode_w4 = w4;
    };
    // ---- one chunk, graphs on: replay (or capture) the launch sequence of this shape ------------------------------
    if (c->prefill_graphs && n_gemm <= c->max_s) {
        const int S = n_gemm;
        if (S > 0) {
            EFM_CK(c, cudaMemcpyAsync(c->ids, token_ids, (size_t)S * 4, cudaMemcpyHostToDevice, c->stream));
            if (pos_ids3 != nullptr)
                for (int r = 0; r < 3; ++r)
                    EFM_CK(c, cudaMemcpyAsync(c->pos3 + (size_t)r * S, pos_ids3 + (size_t)r * n_tokens, (size_t)S * 4, cudaMemcpyHostToDevice, c->stream));
        }
        PrefillGraph key;
        key.slot = slot; key.rows = n_tokens; key.kv_offset = kv_offset; key.n_embeds = n_embeds; key.embed_token_id = embed_token_id;
        key.sample = (sample != 0 ? 1 : 0) + (tail ? 2 : 0); key.attention_kind = c->prefill_attention_kind;
        key.embeds_buf = n_embeds > 0 ? c->custom_embeds : nullptr;
        PrefillGraph* hit = nullptr;
        for (auto& g : c->prefill_cache)
            if (g.same_key(key)) { hit = &g; break; }
        auto launch_all = [&]() {
            if (S > 0) c->ops->prefill_chunk(*c, s, S, kv_offset, n_embeds, embed_token_id, sample != 0 && !tail, L);
            run_tail(L);
        };
        if (hit != nullptr && hit->exec == nullptr) {          // second sighting: capture
            cudaGraph_t g = nullptr;
            const int64_t before = c->launches;
            EFM_CK(c, cudaStreamBeginCapture(c->stream, cudaStreamCaptureModeThreadLocal));
            launch_all();
            cudaError_t e = cudaStreamEndCapture(c->stream, &g);
            hit->nodes = (int)(c->launches - before);
            c->launches = before;
            if (L.err != cudaSuccess) { if (g) cudaGraphDestroy(g); return cuda_fail(c, L.err, "prefill capture launch"); }
            if (e != cudaSuccess) return cuda_fail(c, e, "cudaStreamEndCapture (prefill)");
            e = cudaGraphInstantiate(&hit->exec, g, 0);
            cudaGraphDestroy(g);
            if (e != cudaSuccess) { hit->exec = nullptr; return cuda_fail(c, e, "cudaGraphInstantiate (prefill)"); }
        }
        if (hit != nullptr) {
            hit->last_use = ++c->prefill_clock;
            EFM_CK(c, cudaGraphLaunch(hit->exec, c->stream));
            c->launches += hit->nodes;
            ++c->prefill_graph_replays;
            return EFM_OK;
        }
        // first sighting: remember the shape (evicting the least recently used one), run kernel by kernel
        if (c->prefill_cache.size() >= kMaxPrefillGraphs) {
            size_t victim = 0;
            for (size_t i = 1; i < c->prefill_cache.size(); ++i)
                if (c->prefill_cache[i].last_use < c->prefill_cache[victim].last_use) victim = i;
            if (c->prefill_cache[victim].exec != nullptr) cudaGraphExecDestroy(c->prefill_cache[victim].exec);
            c->prefill_cache.erase(c->prefill_cache.begin() + (long)victim);
        }
        key.last_use = ++c->prefill_clock;
        c->prefill_cache.push_back(key);
        launch_all();
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "prefill launch");
        return EFM_OK;
    }
    for (int off = 0; off < n_gemm; off += c->max_s) {
        const int S = std::min(c->max_s, n_gemm - off);
        EFM_CK(c, cudaMemcpyAsync(c->ids, token_ids + off, (size_t)S * 4, cudaMemcpyHostToDevice, c->stream));
        if (pos_ids3 != nullptr)
            for (int r = 0; r < 3; ++r)
                EFM_CK(c, cudaMemcpyAsync(c->pos3 + (size_t)r * S, pos_ids3 + (size_t)r * n_tokens + off, (size_t)S * 4,
                                          cudaMemcpyHostToDevice, c->stream));
        const bool last = off + S >= n_gemm;
        c->ops->prefill_chunk(*c, s, S, kv_offset + off, n_embeds, embed_token_id, last && sample != 0 && !tail, L);
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "prefill launch");
    }
    run_tail(L);
    if (L.err != cudaSuccess) return cuda_fail(c, L.err, "prefill launch (last token)");
    return EFM_OK;
}

efm_status efm_b200_decode_begin(efm_b200_ctx* c, int32_t slot, int32_t kv_len, const int32_t mrope_pos[3], int32_t step) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    auto it = c->slots.find(slot);
    if (it == c->slots.end()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unknown KV slot " + std::to_string(slot));
    if (kv_len < 0 || kv_len >= it->second.max_tokens) return fail(c, EFM_ERR_INVALID_ARGUMENT, "kv_len leaves no room in the slot");
    if (step < 0) return fail(c, EFM_ERR_INVALID_ARGUMENT, "step must be >= 0");
    EFM_CK(c, cudaSetDevice(c->device));
    if (c->ops->decode_begin != nullptr) {
        const efm_status bs = c->ops->decode_begin(c, it->second, kv_len);
        if (bs != EFM_OK) return bs;
    }
    struct { uint32_t kv_len; int32_t pos[3]; int32_t step; int32_t error; } tail;
    tail.kv_len = (uint32_t)kv_len + 1u;      // the step appends its own K/V before attending
    for (int i = 0; i < 3; ++i) tail.pos[i] = mrope_pos != nullptr ? mrope_pos[i] : 0;
    tail.step = step;
    tail.error = 0;
    static_assert(offsetof(DecodeState, kv_len) == 4 && sizeof(tail) == 24, "DecodeState layout");
    EFM_CK(c, cudaMemcpyAsync(reinterpret_cast<char*>(c->state) + 4, &tail, sizeof(tail), cudaMemcpyHostToDevice, c->stream));
    if (c->error_host != nullptr) *reinterpret_cast<volatile int*>(c->error_host) = 0;
    c->bound_slot = slot;
    return EFM_OK;
}

efm_status efm_b200_set_token(efm_b200_ctx* c, int32_t token) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    EFM_CK(c, cudaMemcpyAsync(&c->state->token, &token, 4, cudaMemcpyHostToDevice, c->stream));
    return EFM_OK;
}

static efm_status ensure_graph(efm_b200_ctx* c, KvSlot& s) {
    if (s.graph != nullptr) return EFM_OK;
    Launcher L = make_launcher(c);
    cudaGraph_t g = nullptr;
    const int64_t before = c->launches;
    EFM_CK(c, cudaStreamBeginCapture(c->stream, cudaStreamCaptureModeThreadLocal));
    c->ops->decode_step(*c, s, L);
    cudaError_t e = cudaStreamEndCapture(c->stream, &g);
    s.graph_nodes = (int)(c->launches - before);
    c->launches = before;                 // capture records, it does not run
    if (L.err != cudaSuccess) { if (g) cudaGraphDestroy(g); return cuda_fail(c, L.err, "decode capture launch"); }
    if (e != cudaSuccess) return cuda_fail(c, e, "cudaStreamEndCapture");
    e = cudaGraphInstantiate(&s.graph, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) { s.graph = nullptr; return cuda_fail(c, e, "cudaGraphInstantiate"); }
    return EFM_OK;
}

efm_status efm_b200_capture_decode(efm_b200_ctx* c, int32_t slot) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    if (!c->finalized) return fail(c, EFM_ERR_STATE, "weights not finalized");
    auto it = c->slots.find(slot);
    if (it == c->slots.end()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unknown KV slot " + std::to_string(slot));
    EFM_CK(c, cudaSetDevice(c->device));
    return ensure_graph(c, it->second);
}

efm_status efm_b200_decode_steps(efm_b200_ctx* c, int32_t n_steps, int32_t use_graph) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    if (c->bound_slot < 0) return fail(c, EFM_ERR_STATE, "decode_begin has not been called");
    if (n_steps <= 0) return EFM_OK;
    KvSlot& s = c->slots[c->bound_slot];
    EFM_CK(c, cudaSetDevice(c->device));
    if (!use_graph) {
        Launcher L = make_launcher(c);
        for (int i = 0; i < n_steps; ++i) c->ops->decode_step(*c, s, L);
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "decode launch");
        s.len += n_steps;
        return EFM_OK;
    }
    const efm_status st = ensure_graph(c, s);
    if (st != EFM_OK) return st;
    for (int i = 0; i < n_steps; ++i) {
        // a kernel of an earlier step gave up waiting for a peer: queue nothing more behind it
        if (c->error_host != nullptr && *reinterpret_cast<volatile int*>(c->error_host) != 0)
            return fail(c, EFM_ERR_DEVICE_WAIT, "a tensor-parallel peer did not answer within the wait limit; decode stopped after " +
                                                    std::to_string(i) + " queued steps");
        EFM_CK(c, cudaGraphLaunch(s.graph, c->stream));
        c->launches += s.graph_nodes;
        ++s.len;
    }
    return EFM_OK;
}

static efm_status check_device_state(efm_b200_ctx* c) {
    DecodeState st{};
    EFM_CK(c, cudaMemcpyAsync(&st, c->state, sizeof(st), cudaMemcpyDeviceToHost, c->stream));
    { const efm_status s = ctx_sync(c); if (s != EFM_OK) return s; }
    if (st.error != 0) {
        int zero = 0;
        if (c->error_host != nullptr) *reinterpret_cast<volatile int*>(c->error_host) = 0;
        cudaMemcpyAsync(&c->state->error, &zero, 4, cudaMemcpyHostToDevice, c->stream);
        return fail(c, EFM_ERR_DEVICE_WAIT, "a kernel refused an out-of-range cache row or abandoned a bounded wait (device status " + std::to_string(st.error) + ")");
    }
    return EFM_OK;
}

efm_status efm_b200_read_tokens(efm_b200_ctx* c, int32_t* host_out, int32_t first, int32_t n) {
    if (c == nullptr || host_out == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (first < 0 || n < 0 || first + n > c->d.max_response_tokens) return fail(c, EFM_ERR_INVALID_ARGUMENT, "token range outside the response buffer");
    EFM_CK(c, cudaSetDevice(c->device));
    if (n > 0) EFM_CK(c, cudaMemcpyAsync(host_out, c->tokens_out + first, (size_t)n * 4, cudaMemcpyDeviceToHost, c->stream));
    return check_device_state(c);
}

efm_status efm_b200_read_logits(efm_b200_ctx* c, float* host_out, int32_t n) {
    if (c == nullptr || host_out == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (n < 0 || n > c->d.vocab) return fail(c, EFM_ERR_INVALID_ARGUMENT, "n exceeds vocab");
    EFM_CK(c, cudaSetDevice(c->device));
    if (c->ops->gather_logits != nullptr) {       // a collective on tensor-parallel contexts that exchanged maxima only
        Launcher L = make_launcher(c);
        L.counter = nullptr;
        c->ops->gather_logits(*c, L);
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "gathering the logits of the tensor-parallel ranks");
    }
    EFM_CK(c, cudaMemcpyAsync(host_out, c->logits, (size_t)n * 4, cudaMemcpyDeviceToHost, c->stream));
    return ctx_sync(c);
}

efm_status efm_b200_synchronize(efm_b200_ctx* c) {
    if (c == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null context");
    return ctx_sync(c);
}

efm_status efm_b200_event_record(efm_b200_ctx* c, int32_t idx) {
    if (c == nullptr || idx < 0 || idx >= 16) return fail(c, EFM_ERR_INVALID_ARGUMENT, "event index out of range");
    EFM_CK(c, cudaEventRecord(c->events[idx], c->stream));
    return EFM_OK;
}

efm_status efm_b200_event_elapsed_ms(efm_b200_ctx* c, int32_t a, int32_t b, float* ms) {
    if (c == nullptr || ms == nullptr || a < 0 || a >= 16 || b < 0 || b >= 16) return fail(c, EFM_ERR_INVALID_ARGUMENT, "bad event arguments");
    EFM_CK(c, cudaEventSynchronize(c->events[b]));
    EFM_CK(c, cudaEventElapsedTime(ms, c->events[a], c->events[b]));
    return EFM_OK;
}

efm_status efm_b200_launch_count(efm_b200_ctx* c, int64_t* count) {
    if (c == nullptr || count == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    *count = c->launches;
    return EFM_OK;
}

efm_status efm_b200_decode_breakdown(efm_b200_ctx* c, int32_t n_steps, float* ms_out) {
    if (c == nullptr || ms_out == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    if (c->decoder != nullptr) return fail(c, EFM_ERR_UNSUPPORTED, "the breakdown is laid out for the text tower's five kernels per layer");
    if (c->bound_slot < 0) return fail(c, EFM_ERR_STATE, "decode_begin has not been called");
    KvSlot& s = c->slots[c->bound_slot];
    EFM_CK(c, cudaSetDevice(c->device));
    for (int i = 0; i < 7; ++i) ms_out[i] = 0.f;
    const int per_step = 5 * c->d.num_layers + 2;
    for (int step = 0; step < n_steps; ++step) {
        std::vector<cudaEvent_t> ev;
        Launcher L = make_launcher(c);
        L.pdl = false;
        L.trace = &ev;
        cudaEvent_t first = nullptr;
        EFM_CK(c, cudaEventCreate(&first));
        EFM_CK(c, cudaEventRecord(first, c->stream));
        c->ops->decode_step(*c, s, L);
        cudaError_t e = L.err != cudaSuccess ? L.err : cudaStreamSynchronize(c->stream);
        if (e == cudaSuccess && (int)ev.size() == per_step) {
            cudaEvent_t prev = first;
            for (int i = 0; i < per_step; ++i) {
                float ms = 0.f;
                cudaEventElapsedTime(&ms, prev, ev[i]);
                const int kind = i < 5 * c->d.num_layers ? i % 5 : 5 + (i - 5 * c->d.num_layers);
                ms_out[kind] += ms;
                prev = ev[i];
            }
        }
        cudaEventDestroy(first);
        for (cudaEvent_t x : ev) cudaEventDestroy(x);
        if (e != cudaSuccess) return cuda_fail(c, e, "decode breakdown");
    }
    return EFM_OK;
}

efm_status efm_b200_decode_step_bytes(efm_b200_ctx* c, int32_t kv_len, int64_t* bytes) {
    if (c == nullptr || bytes == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "null argument");
    *bytes = c->ops->step_bytes(*c, kv_len);
    return EFM_OK;
}

}  // extern "C"
