// Layered decoders behind the C ABI: context creation, weight ingestion (fused projections, zero-padded rows), the
// paged cache and the recurrent state slots, batched steps.
#include <algorithm>
#include <cstdio>
#include <cstring>

#include "../../layers/decoder.h"
#include "../../layers/shared_launch.h"
#include "../../operators/gemv.cuh"
#define EFM_DECLARATIONS_ONLY
#include "../../operators/sample.cuh"
#undef EFM_DECLARATIONS_ONLY
#include "ctx.h"
#include "ctx_util.h"

using namespace efm;

namespace {

extern const ModelOps kDecoderOps;

size_t act_bytes(const DecoderModel& m) { return m.f32 ? 4 : 2; }

efm_status validate(const efm_decoder_desc& d, const efm_decoder_layer* layers) {
    if (d.num_layers <= 0 || d.vocab <= 0 || d.width <= 0 || d.side_dim < 0 || d.max_step_tokens <= 0 || d.max_response_tokens <= 0 ||
        d.max_slots <= 0 || d.cache_pages < 0 || d.state_slots < 0)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "non-positive decoder dimension");
    if (d.compute_dtype != EFM_BF16 && d.compute_dtype != EFM_F32) return fail(nullptr, EFM_ERR_UNSUPPORTED, "compute_dtype must be bf16 or fp32");
    for (int i = 0; i < d.num_layers; ++i) {
        const efm_decoder_layer& l = layers[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        if (l.heads <= 0 || l.dim <= 0 || l.ff < 0) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "non-positive dimension");
        if (l.dim > 256) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "dim above 256");
        if (l.mixer == EFM_MIXER_ATTENTION) {
            if (l.kv_heads <= 0 || l.heads % l.kv_heads != 0 || l.vdim <= 0 || l.window < 0)
                return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "heads must be a multiple of kv_heads, vdim positive, window >= 0");
            if (l.vdim > 256) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "vdim above 256");
        } else if (l.mixer == EFM_MIXER_GENERAL_DELTA) {
            if (l.decay_rank <= 0) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "decay_rank must be positive");
            if (l.decay_rank > 512) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "decay_rank above 512");
        } else {
            return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "unknown mixer");
        }
    }
    return EFM_OK;
}

cudaError_t alloc_linear(efm_b200_ctx* c, DecLinear& w, int N, int K) {
    w.N = N; w.K = K; w.Np = round_up(N, 8); w.Kp = round_up(K, 8);
    return dev_alloc(c, &w.w, (size_t)w.Np * w.Kp);
}

}  // namespace

extern "C" {

efm_status efm_b200_decoder_create(const efm_decoder_desc* desc, const efm_decoder_layer* layers, int32_t device_id, efm_b200_ctx** out) {
    if (desc == nullptr || layers == nullptr || out == nullptr) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "null argument");
    *out = nullptr;
    if (desc->struct_size != (int32_t)sizeof(efm_decoder_desc)) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "efm_decoder_desc.struct_size mismatch");
    efm_status st = validate(*desc, layers);
    if (st != EFM_OK) return st;
    st = require_device(nullptr, device_id);
    if (st != EFM_OK) return st;
    efm_b200_ctx* c = new (std::nothrow) efm_b200_ctx();
    DecoderModel* m = new (std::nothrow) DecoderModel();
    if (c == nullptr || m == nullptr) { delete c; delete m; return fail(nullptr, EFM_ERR_OUT_OF_MEMORY, "host allocation failed"); }
    c->ops = &kDecoderOps;
    c->decoder = m;
    c->device = device_id;
    c->pdl = std::getenv("EFM_B200_NO_PDL") == nullptr;
    m->d = *desc;
    m->f32 = desc->compute_dtype == EFM_F32;
    m->W = desc->width;
    m->Wp = round_up(desc->width, 8);
    m->side_p = round_up(std::max(desc->side_dim, 1), 8);
    const int S = desc->max_step_tokens, Wp = m->Wp;
    // what the model-independent calls read
    c->d.struct_size = (int32_t)sizeof(efm_model_desc);
    c->d.num_layers = desc->num_layers;
    c->d.hidden = Wp;
    c->d.vocab = desc->vocab;
    c->d.rms_eps = desc->norm_eps;
    c->d.max_prefill_tokens = S;
    c->d.max_response_tokens = desc->max_response_tokens;
    c->full = c->d;
    c->max_s = S;
    c->vocab_l = desc->vocab;
    auto bail = [&](cudaError_t e, const char* what) {
        efm_status s = cuda_fail(nullptr, e, what);
        efm_b200_destroy(c);
        return s;
    };
#define EFM_TRY(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) return bail(e_, #call); } while (0)
    EFM_TRY(cudaDeviceGetAttribute(&c->num_sms, cudaDevAttrMultiProcessorCount, device_id));
    EFM_TRY(cudaStreamCreateWithFlags(&c->stream, cudaStreamNonBlocking));
    for (auto& ev : c->events) EFM_TRY(cudaEventCreate(&ev));
    EFM_TRY(configure_decoder(*m));
    EFM_TRY(configure_sampler());

    const size_t rows = (size_t)std::max(desc->cache_pages, 1) * EFM_PAGE_TOKENS, es = act_bytes(*m);
    size_t w_in = 8, w_mix = 8, w_ff = 8, w_q = 8, w_delta_in = 8, n_pack = 8, w_rank = 8, k_max = Wp;
    bool any_delta = false;
    m->layers.resize(desc->num_layers);
    for (int i = 0; i < desc->num_layers; ++i) {
        DecoderLayer& l = m->layers[i];
        l.d = layers[i];
        const efm_decoder_layer& d = l.d;
        EFM_TRY(dev_alloc(c, &l.norm1, Wp));
        if (d.mixer == EFM_MIXER_ATTENTION) {
            l.Dp = round_up(d.dim, 64);
            l.Vp = round_up(d.vdim, 64);
            l.mix_w = d.heads * d.vdim;
            EFM_TRY(alloc_linear(c, l.in, (d.heads + d.kv_heads) * d.dim + d.kv_heads * d.vdim, m->W));
            EFM_TRY(dev_alloc(c, &l.q_norm, d.dim));
            EFM_TRY(dev_alloc(c, &l.k_norm, d.dim));
            EFM_TRY(dev_alloc(c, &l.temp, d.heads));
            char *k = nullptr, *v = nullptr;
            EFM_TRY(dev_alloc(c, &k, rows * d.kv_heads * l.Dp * es));
            EFM_TRY(dev_alloc(c, &v, rows * d.kv_heads * l.Vp * es));
            l.k_pool = k;
            l.v_pool = v;
            w_q = std::max(w_q, (size_t)d.heads * l.Dp);
            w_in = std::max(w_in, (size_t)l.in.Np);
        } else {
            any_delta = true;
            const int HD = d.heads * d.dim;
            l.mix_w = HD;
            EFM_TRY(alloc_linear(c, l.in, 5 * HD + d.decay_rank, m->W));
            EFM_TRY(alloc_linear(c, l.w2, HD, d.decay_rank));
            EFM_TRY(dev_alloc(c, &l.w0, HD));
            EFM_TRY(dev_alloc(c, &l.a_bias, HD));
            EFM_TRY(dev_alloc(c, &l.mix_norm, HD));
            l.state_off = m->state_stride;
            m->state_stride += (size_t)HD * d.dim;
            w_delta_in = std::max(w_delta_in, (size_t)l.in.Np);
            n_pack = std::max(n_pack, decoder_delta_pack_floats(d.heads, d.dim, S, std::min(desc->max_slots, S)));
            w_rank = std::max(w_rank, (size_t)l.w2.Kp);
        }
        l.mix_wp = round_up(l.mix_w, 8);
        w_mix = std::max(w_mix, (size_t)l.mix_wp);
        EFM_TRY(alloc_linear(c, l.out, m->W, l.mix_w));
        if (d.ff > 0) {
            EFM_TRY(alloc_linear(c, l.up, d.ff, m->W));
            EFM_TRY(alloc_linear(c, l.down, m->W, d.ff));
            EFM_TRY(dev_alloc(c, &l.act, 4));
            EFM_TRY(dev_alloc(c, &l.norm2, Wp));
            w_ff = std::max(w_ff, (size_t)l.up.Np);
        }
        if (desc->side_dim > 0) {
            EFM_TRY(alloc_linear(c, l.gate, desc->side_dim, m->W));
            EFM_TRY(alloc_linear(c, l.proj, m->W, desc->side_dim));
            EFM_TRY(dev_alloc(c, &l.side_norm, Wp));
        }
        k_max = std::max(k_max, std::max((size_t)l.out.Kp, (size_t)(d.ff > 0 ? l.down.Kp : 0)));
    }
    {   // the longest GEMV input must fit the kernel's shared memory as fp32
        int optin = 0;
        EFM_TRY(cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, device_id));
        if (std::max(gemv_smem_bytes((int)k_max), gemv_ext_smem_bytes(Wp)) + 2048 > (size_t)optin) {
            efm_status s = fail(nullptr, EFM_ERR_UNSUPPORTED, "width / feed-forward size exceeds what the decode GEMV stages in shared memory");
            efm_b200_destroy(c);
            return s;
        }
    }
    EFM_TRY(dev_alloc(c, &c->embed, (size_t)desc->vocab * Wp));
    if (desc->side_dim > 0) EFM_TRY(dev_alloc(c, &m->side_embed, (size_t)desc->vocab * desc->side_dim * desc->num_layers));
    EFM_TRY(dev_alloc(c, &m->final_norm, Wp));
    EFM_TRY(alloc_linear(c, m->head, desc->vocab, m->W));
    c->lm_head = m->head.w;
    c->final_norm = m->final_norm;

    EFM_TRY(dev_alloc(c, &m->page_table, (size_t)desc->max_slots * std::max(desc->cache_pages, 1)));
    if (m->state_stride > 0) EFM_TRY(dev_alloc(c, &m->state_pool, m->state_stride * std::max(desc->state_slots, 1)));
    for (int i = desc->max_slots - 1; i >= 0; --i) m->free_tables.push_back(i);

    auto act = [&](void** p, size_t n) {
        char* raw = nullptr;
        const cudaError_t e = dev_alloc(c, &raw, n * es);
        *p = raw;
        return e;
    };
    EFM_TRY(dev_alloc(c, &c->ids, S));
    EFM_TRY(dev_alloc(c, &c->resid, (size_t)S * Wp));
    if (!m->f32) EFM_TRY(act(&m->xa, (size_t)S * Wp));
    EFM_TRY(act(&m->proj_a, S * w_in));
    EFM_TRY(act(&m->q, S * w_q));
    EFM_TRY(act(&m->mix, S * w_mix));
    EFM_TRY(act(&m->ff, S * w_ff));
    EFM_TRY(act(&m->ff2, S * w_ff));
    EFM_TRY(act(&m->side_a, (size_t)S * m->side_p));
    EFM_TRY(dev_alloc(c, &m->side_f, (size_t)S * m->side_p));
    EFM_TRY(dev_alloc(c, &m->y, (size_t)S * Wp));
    if (any_delta) {
        EFM_TRY(dev_alloc(c, &m->proj_f, S * w_delta_in));
        EFM_TRY(dev_alloc(c, &m->pack, n_pack));
        EFM_TRY(dev_alloc(c, &m->tanh_w, S * w_rank));
        EFM_TRY(dev_alloc(c, &m->decay, S * w_mix));
        EFM_TRY(dev_alloc(c, &m->o, S * w_mix));
    }
    m->max_want = std::min(S, 256);
    EFM_TRY(act(&m->head_a, (size_t)m->max_want * Wp));
    EFM_TRY(dev_alloc(c, &m->logits_rows, (size_t)m->max_want * m->head.Np));
    // per pass: ids, row entries, wanted rows, two tile lists, entries
    m->step_words = (size_t)S * 3 + 2 * (size_t)S * 2 + (size_t)S * (sizeof(RowEntry) / 4) + 64;
    EFM_TRY(dev_alloc(c, &m->step_buf, m->step_words));

    EFM_TRY(dev_alloc(c, &c->resid_d, Wp));
    EFM_TRY(dev_alloc(c, &c->resid_d2, Wp));
    EFM_TRY(dev_alloc(c, &m->d_in, std::max(w_in, w_delta_in)));
    EFM_TRY(dev_alloc(c, &m->d_mix, w_mix));
    EFM_TRY(dev_alloc(c, &m->d_y, Wp));
    EFM_TRY(dev_alloc(c, &m->d_y2, Wp));
    EFM_TRY(dev_alloc(c, &m->d_ff, w_ff));
    EFM_TRY(dev_alloc(c, &m->d_gate, m->side_p));
    EFM_TRY(dev_alloc(c, &c->logits, m->head.Np));
    EFM_TRY(dev_alloc(c, &c->part_val, 2 * (size_t)c->num_sms + 8));
    EFM_TRY(dev_alloc(c, &c->part_idx, 2 * (size_t)c->num_sms + 8));
    EFM_TRY(dev_alloc(c, &c->wbuf, sample_scratch_words(desc->vocab)));
    c->gemm_ws_floats = (size_t)c->num_sms * 128 * 256;
    EFM_TRY(dev_alloc(c, &c->gemm_ws, c->gemm_ws_floats, false));
    EFM_TRY(dev_alloc(c, &c->state, 1));
    EFM_TRY(dev_alloc(c, &c->tokens_out, (size_t)std::max(desc->max_response_tokens, m->max_want)));
    EFM_TRY(cudaStreamSynchronize(c->stream));
#undef EFM_TRY
    *out = c;
    return EFM_OK;
}

efm_status efm_b200_decoder_map_slot(efm_b200_ctx* c, int32_t slot, const int32_t* pages, int32_t n_pages, int32_t state_slot) {
    if (c == nullptr || c->decoder == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "not a layered-decoder context");
    DecoderModel& m = *c->decoder;
    if (n_pages <= 0 || n_pages > m.d.cache_pages || pages == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "bad page list");
    for (int i = 0; i < n_pages; ++i)
        if (pages[i] < 0 || pages[i] >= m.d.cache_pages) return fail(c, EFM_ERR_INVALID_ARGUMENT, "page number outside the pool");
    if (m.state_stride > 0 && (state_slot < 0 || state_slot >= m.d.state_slots)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "state slot outside the pool");
    EFM_CK(c, cudaSetDevice(c->device));
    auto it = c->slots.find(slot);
    if (it == c->slots.end()) {
        if (m.free_tables.empty()) return fail(c, EFM_ERR_STATE, "every slot is mapped (max_slots)");
        KvSlot s;
        s.table = m.free_tables.back();
        m.free_tables.pop_back();
        it = c->slots.emplace(slot, s).first;
    }
    KvSlot& s = it->second;
    if (s.len > n_pages * EFM_PAGE_TOKENS) return fail(c, EFM_ERR_INVALID_ARGUMENT, "fewer pages than the tokens the slot holds");
    // number of pages and state address are baked into a captured decode step; the page numbers are read from the table
    if (s.graph != nullptr && (s.n_pages != n_pages || s.state_slot != state_slot)) { cudaGraphExecDestroy(s.graph); s.graph = nullptr; }
    s.n_pages = n_pages;
    s.max_tokens = n_pages * EFM_PAGE_TOKENS;
    s.state_slot = state_slot;
    EFM_CK(c, cudaMemcpyAsync(m.page_table + (size_t)s.table * m.d.cache_pages, pages, (size_t)n_pages * 4, cudaMemcpyHostToDevice, c->stream));
    return EFM_OK;
}

efm_status efm_b200_decoder_unmap_slot(efm_b200_ctx* c, int32_t slot) {
    if (c == nullptr || c->decoder == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "not a layered-decoder context");
    auto it = c->slots.find(slot);
    if (it == c->slots.end()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unknown slot " + std::to_string(slot));
    if (it->second.graph != nullptr) { EFM_CK(c, cudaStreamSynchronize(c->stream)); cudaGraphExecDestroy(it->second.graph); }
    for (size_t i = 0; i < c->prefill_cache.size();)
        if (c->prefill_cache[i].slot == slot) {
            if (c->prefill_cache[i].exec != nullptr) cudaGraphExecDestroy(c->prefill_cache[i].exec);
            c->prefill_cache.erase(c->prefill_cache.begin() + (long)i);
        } else {
            ++i;
        }
    c->decoder->free_tables.push_back(it->second.table);
    if (c->bound_slot == slot) c->bound_slot = -1;
    c->slots.erase(it);
    return EFM_OK;
}

efm_status efm_b200_decoder_pin_prefix(efm_b200_ctx* c, int32_t slot, int32_t pin_state) {
    if (c == nullptr || c->decoder == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "not a layered-decoder context");
    DecoderModel& m = *c->decoder;
    auto it = c->slots.find(slot);
    if (it == c->slots.end()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unknown slot " + std::to_string(slot));
    KvSlot& s = it->second;
    if (m.state_stride > 0) {
        if (pin_state < 0 || pin_state >= m.d.state_slots || pin_state == s.state_slot) return fail(c, EFM_ERR_INVALID_ARGUMENT, "bad state slot for the prefix");
        EFM_CK(c, cudaMemcpyAsync(m.state_pool + (size_t)pin_state * m.state_stride, m.state_pool + (size_t)s.state_slot * m.state_stride,
                                  m.state_stride * sizeof(float), cudaMemcpyDeviceToDevice, c->stream));
    }
    s.pin_state = pin_state;
    s.pin_len = s.len;
    return EFM_OK;
}

}  // extern "C"

namespace {

// The slot continues at kv_offset: where it stands, at its pinned prefix (state restored) or from the start.
efm_status position_slot(efm_b200_ctx* c, KvSlot& s, int kv_offset, int n_tokens) {
    DecoderModel& m = *c->decoder;
    if ((int64_t)kv_offset + n_tokens > (int64_t)s.n_pages * EFM_PAGE_TOKENS) return fail(c, EFM_ERR_INVALID_ARGUMENT, "tokens exceed the slot's pages");
    if (kv_offset == s.len || kv_offset == 0) return EFM_OK;
    if (s.pin_len > 0 && kv_offset == s.pin_len) {
        if (m.state_stride > 0)
            EFM_CK(c, cudaMemcpyAsync(m.state_pool + (size_t)s.state_slot * m.state_stride, m.state_pool + (size_t)s.pin_state * m.state_stride,
                                      m.state_stride * sizeof(float), cudaMemcpyDeviceToDevice, c->stream));
        return EFM_OK;
    }
    if (m.state_stride == 0 && kv_offset < s.len) return EFM_OK;          // attention alone can go back to any earlier row
    return fail(c, EFM_ERR_STATE, "kv_offset " + std::to_string(kv_offset) + " is neither what the slot holds (" + std::to_string(s.len) +
                                      "), its fixed prefix (" + std::to_string(s.pin_len) + ") nor 0");
}

}  // namespace

extern "C" {

efm_status efm_b200_decoder_step(efm_b200_ctx* c, const efm_step_entry* entries, int32_t n_entries, float* logits, int32_t* sampled) {
    if (c == nullptr || c->decoder == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "not a layered-decoder context");
    if (entries == nullptr || n_entries <= 0) return fail(c, EFM_ERR_INVALID_ARGUMENT, "a step needs entries");
    if (!c->finalized) return fail(c, EFM_ERR_STATE, "weights not finalized");
    DecoderModel& m = *c->decoder;
    EFM_CK(c, cudaSetDevice(c->device));
    int64_t total_want = 0;
    for (int e = 0; e < n_entries; ++e) {
        const efm_step_entry& en = entries[e];
        auto it = c->slots.find(en.slot);
        if (it == c->slots.end()) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unknown slot " + std::to_string(en.slot));
        if (en.n_tokens <= 0 || en.tokens == nullptr || en.kv_offset < 0 || en.n_want < 0 || (en.n_want > 0 && en.want == nullptr))
            return fail(c, EFM_ERR_INVALID_ARGUMENT, "bad step entry");
        for (int i = 0; i < en.n_tokens; ++i)
            if (en.tokens[i] < 0 || en.tokens[i] >= c->d.vocab) return fail(c, EFM_ERR_INVALID_ARGUMENT, "token id outside the vocabulary");
        for (int i = 0; i < en.n_want; ++i)
            if (en.want[i] < 0 || en.want[i] >= en.n_tokens) return fail(c, EFM_ERR_INVALID_ARGUMENT, "wanted position outside the entry");
        for (int f = 0; f < e; ++f)
            if (entries[f].slot == en.slot) return fail(c, EFM_ERR_INVALID_ARGUMENT, "a slot appears twice in one step");
        const efm_status st = position_slot(c, it->second, en.kv_offset, en.n_tokens);
        if (st != EFM_OK) return st;
        total_want += en.n_want;
    }
    if (total_want > 0 && logits == nullptr && sampled == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "logits are wanted but no buffer was given");
    Launcher L = make_launcher(c);
    auto emit_sample = [&](const float* row, int64_t idx, uint32_t rng_step) -> efm_status {
        if (sampled == nullptr) return (efm_status)EFM_OK;
        SampleParams s{};
        s.logits = row; s.vocab = c->d.vocab; s.n_part = 0;
        s.temperature = c->sampling.temperature; s.top_p = c->sampling.top_p; s.seed = c->sampling.seed; s.rng_step = rng_step;
        s.token_single = c->tokens_out; s.wbuf = c->wbuf; s.xchg = sample_xchg(c->wbuf, c->d.vocab);
        const bool pdl = L.pdl;
        L.pdl = false;
        launch_sample(L, s);
        L.pdl = pdl;
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "sampler launch");
        EFM_CK(c, cudaMemcpyAsync(sampled + idx, c->tokens_out, 4, cudaMemcpyDeviceToHost, c->stream));
        return EFM_OK;
    };
    m.tap_row0 = 0;

    if (n_entries == 1 && entries[0].n_tokens == 1) {          // one row: the decode kernels
        const efm_step_entry& en = entries[0];
        KvSlot& s = c->slots.at(en.slot);
        DecodeState st{};
        st.token = en.tokens[0];
        st.kv_len = (uint32_t)en.kv_offset + 1u;
        EFM_CK(c, cudaMemcpyAsync(c->state, &st, sizeof(st), cudaMemcpyHostToDevice, c->stream));
        decoder_decode_step(*c, s, L, /*sample=*/false, en.n_want > 0);
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "decode launch");
        s.len = en.kv_offset + 1;
        m.tap_row0 = 1;
        for (int i = 0; i < en.n_want; ++i) {
            if (logits != nullptr) EFM_CK(c, cudaMemcpyAsync(logits + (size_t)i * c->d.vocab, c->logits, (size_t)c->d.vocab * 4, cudaMemcpyDeviceToHost, c->stream));
            const efm_status ss = emit_sample(c->logits, i, en.rng_step);
            if (ss != EFM_OK) return ss;
        }
        return en.n_want > 0 ? ctx_sync(c) : EFM_OK;
    }

    // passes of at most max_step_tokens rows; an entry may be cut between passes
    std::vector<int> done((size_t)n_entries, 0);
    std::vector<int64_t> want0((size_t)n_entries, 0);
    for (int e = 1; e < n_entries; ++e) want0[e] = want0[e - 1] + entries[e - 1].n_want;
    int first = 0;
    while (first < n_entries) {
        std::vector<RowEntry> re;
        std::vector<int32_t> ids, row_entry;
        std::vector<RowTile> tc, simt;
        struct Want { int32_t row; int64_t idx; uint32_t rng_step; };
        std::vector<Want> wants;
        int rows = 0;
        for (int e = first; e < n_entries && rows < c->max_s; ++e) {
            const efm_step_entry& en = entries[e];
            const int n = std::min(en.n_tokens - done[e], c->max_s - rows);
            KvSlot& s = c->slots.at(en.slot);
            RowEntry r{rows, n, en.kv_offset + done[e], s.table, s.state_slot};
            const int idx = (int)re.size(), step = n >= kTcMinRows ? decoder_tc_tile_rows() : decoder_simt_tile_rows();
            for (int i = 0; i < n; i += step) (n >= kTcMinRows ? tc : simt).push_back(RowTile{idx, i});
            for (int i = 0; i < n; ++i) { ids.push_back(en.tokens[done[e] + i]); row_entry.push_back(idx); }
            for (int i = 0; i < en.n_want; ++i)
                if (en.want[i] >= done[e] && en.want[i] < done[e] + n) wants.push_back(Want{rows + en.want[i] - done[e], want0[e] + i, en.rng_step});
            re.push_back(r);
            rows += n;
            done[e] += n;
            s.len = en.kv_offset + done[e];
            if (done[e] == en.n_tokens && e == first) ++first;
        }
        while (first < n_entries && done[first] == entries[first].n_tokens) ++first;
        // tiles of the tensor-core form go to the CUDA-core form in layers it does not take: list them in its units too
        std::vector<RowTile> all_simt;
        for (size_t i = 0; i < re.size(); ++i)
            for (int r = 0; r < re[i].n; r += decoder_simt_tile_rows()) all_simt.push_back(RowTile{(int32_t)i, r});
        std::vector<int32_t> pk;
        auto put = [&](const void* p, size_t words) {
            const size_t at = pk.size();
            const int32_t* w = static_cast<const int32_t*>(p);
            pk.insert(pk.end(), w, w + words);
            return at;
        };
        std::vector<int32_t> want_rows;
        for (const Want& w : wants) want_rows.push_back(w.row);
        const size_t o_ids = put(ids.data(), ids.size()), o_re = put(re.data(), re.size() * sizeof(RowEntry) / 4),
                     o_row = put(row_entry.data(), row_entry.size()), o_tc = put(tc.data(), tc.size() * 2), o_simt = put(simt.data(), simt.size() * 2),
                     o_all = put(all_simt.data(), all_simt.size() * 2), o_want = put(want_rows.data(), want_rows.size());
        if (pk.size() > m.step_words) {
            EFM_CK(c, cudaStreamSynchronize(c->stream));
            EFM_CK(c, dev_alloc(c, &m.step_buf, pk.size() * 2, false));
            m.step_words = pk.size() * 2;
        }
        EFM_CK(c, cudaMemcpyAsync(m.step_buf, pk.data(), pk.size() * 4, cudaMemcpyHostToDevice, c->stream));
        RowPlan plan{};
        plan.entries = reinterpret_cast<const RowEntry*>(m.step_buf + o_re);
        plan.row_entry = m.step_buf + o_row;
        plan.page_table = m.page_table;
        plan.max_pages = m.d.cache_pages;
        plan.n_entries = (int)re.size();
        plan.rows = rows;
        RowTiles tiles;
        tiles.listed = true;
        tiles.tc = reinterpret_cast<const RowTile*>(m.step_buf + o_tc);
        tiles.n_tc = (int)tc.size();
        tiles.simt = reinterpret_cast<const RowTile*>(m.step_buf + o_simt);
        tiles.n_simt = (int)simt.size();
        tiles.all = reinterpret_cast<const RowTile*>(m.step_buf + o_all);
        tiles.n_all = (int)all_simt.size();
        decoder_rows_pass(*c, plan, m.step_buf + o_ids, tiles, L);
        m.tap_row0 += rows;
        for (size_t w0 = 0; w0 < wants.size(); w0 += (size_t)m.max_want) {
            const int n = (int)std::min(wants.size() - w0, (size_t)m.max_want);
            decoder_rows_logits(*c, m.step_buf + o_want + w0, n, L);
            if (L.err != cudaSuccess) return cuda_fail(c, L.err, "step launch");
            for (int i = 0; i < n; ++i) {
                const int64_t idx = wants[w0 + i].idx;
                const float* row = m.logits_rows + (size_t)i * m.head.Np;
                if (logits != nullptr) EFM_CK(c, cudaMemcpyAsync(logits + (size_t)idx * c->d.vocab, row, (size_t)c->d.vocab * 4, cudaMemcpyDeviceToHost, c->stream));
                const efm_status ss = emit_sample(row, idx, wants[w0 + i].rng_step);
                if (ss != EFM_OK) return ss;
            }
        }
        if (L.err != cudaSuccess) return cuda_fail(c, L.err, "step launch");
        EFM_CK(c, cudaStreamSynchronize(c->stream));           // the packed indices are host memory of this pass
    }
    int error = 0;
    EFM_CK(c, cudaMemcpyAsync(&error, &c->state->error, 4, cudaMemcpyDeviceToHost, c->stream));
    const efm_status st = ctx_sync(c);
    if (st != EFM_OK) return st;
    if (error != 0) {
        EFM_CK(c, cudaMemsetAsync(&c->state->error, 0, 4, c->stream));
        return fail(c, EFM_ERR_DEVICE_WAIT, "a kernel refused an out-of-range cache row or abandoned a bounded wait (device status " + std::to_string(error) + ")");
    }
    return EFM_OK;
}

efm_status efm_b200_decoder_set_taps(efm_b200_ctx* c, int32_t rows) {
    if (c == nullptr || c->decoder == nullptr || rows < 0) return fail(c, EFM_ERR_INVALID_ARGUMENT, "not a layered-decoder context");
    DecoderModel& m = *c->decoder;
    drop_decode_graphs(c);
    drop_prefill_graphs(c);
    m.tap = nullptr;
    m.tap_rows = rows;
    if (rows > 0) EFM_CK(c, dev_alloc(c, &m.tap, (size_t)m.d.num_layers * rows * m.Wp));
    return EFM_OK;
}

efm_status efm_b200_decoder_read_taps(efm_b200_ctx* c, float* host_out) {
    if (c == nullptr || c->decoder == nullptr || host_out == nullptr || c->decoder->tap == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "no taps are set");
    DecoderModel& m = *c->decoder;
    EFM_CK(c, cudaMemcpy2DAsync(host_out, (size_t)m.W * 4, m.tap, (size_t)m.Wp * 4, (size_t)m.W * 4, (size_t)m.d.num_layers * m.tap_rows,
                                cudaMemcpyDeviceToHost, c->stream));
    return ctx_sync(c);
}

}  // extern "C"

namespace {

// ---- weights -------------------------------------------------------------------------------------------------------
efm_status put_rows(efm_b200_ctx* c, const DecLinear& w, int row0, int rows, const void* data, const std::string& name, const int64_t* shape, int ndim,
                    int mem_kind) {
    if (!shape_is(shape, ndim, rows, w.K)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + name);
    EFM_CK(c, cudaMemcpy2DAsync(w.w + (size_t)row0 * w.Kp, (size_t)w.Kp * 2, data, (size_t)w.K * 2, (size_t)w.K * 2, (size_t)rows,
                                mem_kind == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice, c->stream));
    return EFM_OK;
}
efm_status put_vec(efm_b200_ctx* c, __nv_bfloat16* dst, int n, const void* data, const std::string& name, const int64_t* shape, int ndim, int mem_kind) {
    if (!shape_is(shape, ndim, n)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + name);
    return copy_rows(c, dst, data, (size_t)n * 2, mem_kind);
}

// Where a tensor goes: a row range of a (fused) linear or a vector.
struct Target { DecLinear* lin = nullptr; int row0 = 0, rows = 0; __nv_bfloat16* vec = nullptr; int n = 0; };

bool layer_target(DecoderModel& m, DecoderLayer& l, const std::string& rest, Target* t) {
    const efm_decoder_layer& d = l.d;
    auto lin = [&](DecLinear& w, int row0, int rows) { t->lin = &w; t->row0 = row0; t->rows = rows; return true; };
    auto vec = [&](__nv_bfloat16* v, int n) { t->vec = v; t->n = n; return v != nullptr; };
    if (rest == "norm1") return vec(l.norm1, m.W);
    if (rest == "norm2") return vec(l.norm2, m.W);
    if (rest == "mix.o") return lin(l.out, 0, m.W);
    if (d.mixer == EFM_MIXER_ATTENTION) {
        const int q = d.heads * d.dim, k = d.kv_heads * d.dim;
        if (rest == "mix.q") return lin(l.in, 0, q);
        if (rest == "mix.k") return lin(l.in, q, k);
        if (rest == "mix.v") return lin(l.in, q + k, d.kv_heads * d.vdim);
        if (rest == "mix.q.norm") return vec(l.q_norm, d.dim);
        if (rest == "mix.k.norm") return vec(l.k_norm, d.dim);
        if (rest == "mix.temp") return vec(l.temp, d.heads);
    } else {
        const int HD = d.heads * d.dim;
        static const char* seg[5] = {"mix.r", "mix.k", "mix.v", "mix.g", "mix.a"};
        for (int i = 0; i < 5; ++i)
            if (rest == seg[i]) return lin(l.in, i * HD, HD);
        if (rest == "mix.w1") return lin(l.in, 5 * HD, d.decay_rank);
        if (rest == "mix.w2") return lin(l.w2, 0, HD);
        if (rest == "mix.w0") return vec(l.w0, HD);
        if (rest == "mix.a.b") return vec(l.a_bias, HD);
        if (rest == "mix.norm") return vec(l.mix_norm, HD);
    }
    if (d.ff > 0) {
        if (rest == "mlp.up") return lin(l.up, 0, d.ff);
        if (rest == "mlp.down") return lin(l.down, 0, m.W);
        if (rest == "mlp.act") return vec(l.act, 4);
    }
    if (m.d.side_dim > 0) {
        if (rest == "side.gate") return lin(l.gate, 0, m.d.side_dim);
        if (rest == "side.proj") return lin(l.proj, 0, m.W);
        if (rest == "side.norm") return vec(l.side_norm, m.W);
    }
    return false;
}

efm_status decoder_set_weight(efm_b200_ctx* c, const char* raw, const void* data, const int64_t* shape, int32_t ndim, int32_t dtype, int32_t mem_kind) {
    DecoderModel& m = *c->decoder;
    const std::string name(raw);
    Target t;
    DecLinear table;                       // plain row tables share the padded copy
    if (name == "embed") { table.w = c->embed; table.K = m.W; table.Kp = m.Wp; t.lin = &table; t.rows = m.d.vocab; }
    else if (name == "side.embed" && m.side_embed != nullptr) {
        table.w = m.side_embed; table.K = table.Kp = m.d.side_dim * m.d.num_layers;
        t.lin = &table; t.rows = m.d.vocab;
    }
    else if (name == "head") { t.lin = &m.head; t.rows = m.d.vocab; }
    else if (name == "final.norm") { t.vec = m.final_norm; t.n = m.W; }
    else if (name.size() > 1 && name[0] == 'l' && name[1] >= '0' && name[1] <= '9') {
        const size_t dot = name.find('.');
        const int i = std::atoi(name.c_str() + 1);
        if (dot == std::string::npos || i < 0 || i >= m.d.num_layers || !layer_target(m, m.layers[i], name.substr(dot + 1), &t)) return EFM_OK;
    } else {
        return EFM_OK;                     // not part of this model
    }
    if (dtype != EFM_BF16) return fail(c, EFM_ERR_UNSUPPORTED, "weights must be bf16: " + name);
    const efm_status st = t.lin != nullptr ? put_rows(c, *t.lin, t.row0, t.rows, data, name, shape, ndim, mem_kind)
                                           : put_vec(c, t.vec, t.n, data, name, shape, ndim, mem_kind);
    if (st != EFM_OK) return st;
    EFM_CK(c, cudaStreamSynchronize(c->stream));          // the caller may release `data` on return
    m.seen.insert(name);
    return EFM_OK;
}

efm_status decoder_finalize(efm_b200_ctx* c) {
    DecoderModel& m = *c->decoder;
    std::vector<std::string> need = {"embed", "head", "final.norm"};
    if (m.d.side_dim > 0) need.push_back("side.embed");
    for (int i = 0; i < m.d.num_layers; ++i) {
        const efm_decoder_layer& d = m.layers[i].d;
        auto add = [&](std::initializer_list<const char*> names) { for (const char* n : names) need.push_back("l" + std::to_string(i) + "." + n); };
        add({"norm1", "mix.o"});
        if (d.mixer == EFM_MIXER_ATTENTION) add({"mix.q", "mix.k", "mix.v", "mix.q.norm", "mix.k.norm", "mix.temp"});
        else add({"mix.r", "mix.k", "mix.v", "mix.g", "mix.a", "mix.a.b", "mix.w1", "mix.w2", "mix.w0", "mix.norm"});
        if (d.ff > 0) add({"norm2", "mlp.up", "mlp.down", "mlp.act"});
        if (m.d.side_dim > 0) add({"side.gate", "side.proj", "side.norm"});
    }
    for (const std::string& n : need)
        if (m.seen.count(n) == 0) return fail(c, EFM_ERR_STATE, "missing " + n);
    EFM_CK(c, cudaStreamSynchronize(c->stream));
    c->finalized = true;
    return EFM_OK;
}

efm_status decoder_alloc_slot(efm_b200_ctx* c, int32_t, int32_t) {
    return fail(c, EFM_ERR_UNSUPPORTED, "slots of a layered decoder are mapped with efm_b200_decoder_map_slot");
}

// ---- the single-sequence generate path -----------------------------------------------------------------------------
efm_status decoder_prefill_begin(efm_b200_ctx* c, int32_t, KvSlot& s, int n_tokens, int kv_offset, int n_embeds) {
    if (n_embeds > 0) return fail(c, EFM_ERR_UNSUPPORTED, "this model takes no injected embeddings");
    const efm_status st = position_slot(c, s, kv_offset, n_tokens);
    if (st == EFM_OK) s.len = kv_offset + n_tokens;
    return st;
}
efm_status decoder_decode_begin(efm_b200_ctx* c, KvSlot& s, int kv_len) {
    if (kv_len != s.len && (c->decoder->state_stride > 0 || kv_len > s.len))
        return fail(c, EFM_ERR_STATE, "decode_begin: the slot holds " + std::to_string(s.len) + " tokens, not " + std::to_string(kv_len));
    s.len = kv_len;
    return EFM_OK;
}
void decoder_prefill_chunk(efm_b200_ctx& c, KvSlot& slot, int S, int kv_offset, int, int, bool sample_last, Launcher& L) {
    DecoderModel& m = *c.decoder;
    RowPlan plan{};
    plan.one = RowEntry{0, S, kv_offset, slot.table, slot.state_slot};
    plan.page_table = m.page_table;
    plan.max_pages = m.d.cache_pages;
    plan.n_entries = 1;
    plan.rows = S;
    decoder_rows_pass(c, plan, c.ids, RowTiles{}, L);
    if (sample_last && L.err == cudaSuccess) L.err = cudaErrorNotSupported;     // a sampled prefill ends with a decode step
}
void decoder_step_op(efm_b200_ctx& c, KvSlot& slot, Launcher& L) { decoder_decode_step(c, slot, L, true, true); }

int64_t decoder_step_bytes(const efm_b200_ctx& c, int32_t kv_len) {
    const DecoderModel& m = *c.decoder;
    auto lin = [](const DecLinear& w) { return (int64_t)w.N * w.K * 2; };
    int64_t b = lin(m.head) + (int64_t)m.W * 2 * 2;
    for (const DecoderLayer& l : m.layers) {
        b += lin(l.in) + lin(l.out) + lin(l.w2) + lin(l.up) + lin(l.down) + lin(l.gate) + lin(l.proj);
        if (l.d.mixer == EFM_MIXER_ATTENTION) {
            const int64_t n = l.d.window > 0 ? std::min(kv_len, l.d.window) : kv_len;
            b += n * l.d.kv_heads * (l.d.dim + l.d.vdim) * (m.f32 ? 4 : 2);
        } else {
            b += 2 * (int64_t)l.d.heads * l.d.dim * l.d.dim * 4;
        }
    }
    return b;
}

void decoder_destroy(efm_b200_ctx* c) {
    delete c->decoder;
    c->decoder = nullptr;
}

const ModelOps kDecoderOps = {decoder_set_weight, nullptr, decoder_finalize, decoder_alloc_slot, decoder_prefill_begin, decoder_decode_begin,
                              decoder_prefill_chunk, decoder_step_op, nullptr, decoder_step_bytes, decoder_destroy};

}  // namespace
