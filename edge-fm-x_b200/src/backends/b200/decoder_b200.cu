// Layered decoders behind the C ABI: context creation, weight ingestion (fused projections, zero-padded rows), the
// paged cache and the recurrent state slots, batched steps.
#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstring>

#include "../../layers/decoder.h"
#include "../../layers/shared_launch.h"
#include "../../operators/conv_limits.h"
#include "../../operators/gemv.cuh"
#include "../../operators/rotary.cuh"
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
    if (d.norm_layout < EFM_NORM_OUTPUT || d.norm_layout > EFM_NORM_INPUT) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "unknown norm_layout");
    if (d.logit_softcap < 0.f) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "logit_softcap must not be negative");
    if (d.norm_layout != EFM_NORM_INPUT && (d.logit_scale != 1.0f || (d.logit_softcap > 0.f && d.norm_layout != EFM_NORM_OUTPUT)))
        return fail(nullptr, EFM_ERR_UNSUPPORTED, "scaled logits, or capped ones behind a sandwich of norms");
    if (d.conv_taps < 0 || d.conv_taps > kMaxConvTaps) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "conv_taps must lie between 0 and 16");
    if ((d.conv_taps > 0 || d.depth_average) && (d.norm_layout != EFM_NORM_OUTPUT || d.side_dim > 0 || d.loop_times > 1))
        return fail(nullptr, EFM_ERR_UNSUPPORTED, "input convolutions and depth averages need output norms, no token input and no loop");
    if (d.norm_layout != EFM_NORM_OUTPUT && d.side_dim > 0) return fail(nullptr, EFM_ERR_UNSUPPORTED, "a token input behind normalised sublayer inputs");
    if (d.loop_times < 0 || (d.loop_times > 1 && (d.loop_start < 0 || d.loop_stop <= d.loop_start || d.loop_stop > d.num_layers)))
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "the looped layers must be a span of the layers");
    for (int i = 0; i < d.num_layers; ++i) {
        const efm_decoder_layer& l = layers[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        if (l.heads <= 0 || l.dim <= 0 || l.ff < 0 || l.experts < 0) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "non-positive dimension");
        if (l.dim > 256) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "dim above 256");
        const bool input = d.norm_layout == EFM_NORM_INPUT;
        if (l.mixer == EFM_MIXER_ATTENTION || l.mixer == EFM_MIXER_PARALLEL) {
            if (l.kv_heads <= 0 || l.heads % l.kv_heads != 0 || l.vdim <= 0 || l.window < 0)
                return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "heads must be a multiple of kv_heads, vdim positive, window >= 0");
            if (l.vdim > 256) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "vdim above 256");
            if (l.keep_first < 0 || l.qk_norm < EFM_QK_NORM_WEIGHTED || l.qk_norm > EFM_QK_NORM_ROW) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "keep_first or qk_norm");
            if (l.rot_kind != EFM_ROT_NONE && l.rot_dims > l.dim) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "more rotated channels than dim");
            if (l.sink || (l.out_gate != EFM_GATE_NONE && l.out_gate != EFM_GATE_HEADS)) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "sinks and gates per channel belong to latent attention");
            if (l.score_weights < EFM_WEIGHTS_SOFTMAX || l.score_weights > EFM_WEIGHTS_SIGMOID) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "unknown score_weights");
            if (l.score_weights == EFM_WEIGHTS_SIGMOID && l.keep_first > 0) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "kept first tokens with sigmoid weights");
            if ((l.score_weights != EFM_WEIGHTS_SOFTMAX || l.out_gate || l.out_bias || l.qk_norm == EFM_QK_NORM_ROW) && (l.mixer != EFM_MIXER_ATTENTION || d.norm_layout != EFM_NORM_OUTPUT))
                return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "sigmoid weights, gates, output biases and norms over all heads belong to attention behind output norms");
            if (l.score_weights != EFM_WEIGHTS_SOFTMAX && l.rot_kind != EFM_ROT_NONE) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "rotation with sigmoid weights");
            if (input && l.qkv_bias) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "biases behind elementwise input norms");
            if (l.mixer == EFM_MIXER_PARALLEL) {
                if (!input) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "parallel mixers need input norms");
                if (l.linear_heads <= 0 || l.linear_dim <= 0 || l.linear_vdim <= 0 || l.linear_decay == nullptr)
                    return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "linear attention needs positive sizes and a decay per head");
                if (l.linear_dim > 256 || l.linear_vdim > 256) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "linear attention heads above 256 channels");
                for (int h = 0; h < l.linear_heads; ++h)
                    if (!(l.linear_decay[h] >= 0.0 && l.linear_decay[h] <= 1.0)) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "decays must lie between 0 and 1");
            }
        } else if (l.mixer == EFM_MIXER_LATENT_ATTENTION) {
            if (l.vdim <= 0 || l.window < 0 || l.q_rank <= 0 || l.kv_rank <= 0) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "non-positive dimension");
            if (l.vdim > 256 || l.kv_rank > 1024) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "vdim above 256 or kv_rank above 1024");
            if (l.rot_kind == EFM_ROT_NONE) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "latent attention has a rotated part");
            if (l.keep_first != 0) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "keep_first belongs to attention");
            if (l.out_gate < EFM_GATE_NONE || l.out_gate > EFM_GATE_HEADS) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "unknown out_gate");
        } else if (l.mixer == EFM_MIXER_LINEAR) {
            if (d.norm_layout != EFM_NORM_OUTPUT) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "linear attention alone needs output norms");
            if (l.linear_heads <= 0 || l.linear_dim <= 0 || l.linear_vdim <= 0) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "linear attention needs positive sizes");
            if (l.linear_dim > 256 || l.linear_vdim > 256) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "linear attention heads above 256 channels");
            if (l.rot_kind != EFM_ROT_NONE && l.rot_dims > l.linear_dim) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "more rotated channels than dim");
            if (!(l.linear_tau >= 0.f)) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "linear_tau must not be negative");
            if (l.linear_tau > 0.f ? l.decay_rank <= 0 : l.linear_decay == nullptr) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "linear attention needs a decay per head, or decay_rank and linear_tau");
            if (l.decay_rank > 512) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "decay_rank above 512");
            if (l.linear_tau == 0.f)
                for (int h = 0; h < l.linear_heads; ++h)
                    if (!(l.linear_decay[h] >= 0.0 && l.linear_decay[h] <= 1.0)) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "decays must lie between 0 and 1");
        } else if (l.mixer == EFM_MIXER_GENERAL_DELTA) {
            if (l.decay_rank <= 0) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "decay_rank must be positive");
            if (l.decay_rank > 512) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "decay_rank above 512");
        } else {
            return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "unknown mixer");
        }
        if (l.rot_kind != EFM_ROT_NONE) {
            if ((l.rot_kind != EFM_ROT_HALF && l.rot_kind != EFM_ROT_PAIRS) || l.rot_dims <= 0 || l.rot_dims % 2 != 0 || !(l.rot_base > 0.f))
                return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "rotation needs a kind, an even number of channels and a base");
            if (l.rot_dims > 2 * kRotMaxPairs) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "more than 256 rotated channels");
            if (l.rot_factor < 0.f || (l.rot_factor > 0.f && !(l.rot_original > 0.f && l.rot_fast > 0.f && l.rot_slow > 0.f && l.rot_base != 1.0f)))
                return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "a scaled rotation needs a positive factor, context and limits");
        }
        if (l.ff > 0 && l.ff_act != EFM_ACT_POLYNORM && l.ff_act != EFM_ACT_RELU2) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "unknown ff_act");
        if (l.ff > 0 && (d.conv_taps > 0 || d.depth_average)) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "a dense feed-forward behind an input convolution");
        if (l.ff > 0 && l.ff_act == EFM_ACT_RELU2 && !input) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "a squared ReLU behind output norms");
        if (l.experts > 0) {
            const bool plain = l.expert_glu == EFM_GLU_NONE_RELU2;
            if (!input && (l.expert_glu == EFM_GLU_CLAMPED || l.expert_weight_input || (l.shared_ff > 0 && !plain)))
                return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "clamped, input-weighted or (with a gated unit) shared experts behind output norms");
            if (plain && d.norm_layout != EFM_NORM_OUTPUT) return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "experts without a gate need output norms");
            if (l.expert_scale < 0.f || l.shared_gate < EFM_SHARED_GATED || l.shared_gate > EFM_SHARED_PLAIN) return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "expert_scale or shared_gate");
            if (l.shared_ff < 0 || l.expert_glu < EFM_GLU_SILU || l.expert_glu > EFM_GLU_NONE_RELU2 || l.expert_score < EFM_SCORE_SOFTMAX || l.expert_score > EFM_SCORE_SIGMOID)
                return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "unknown form of the experts");
            if (l.ff > 0 || l.expert_ff <= 0 || l.expert_top <= 0 || l.expert_groups <= 0 || l.expert_groups_kept <= 0 ||
                l.expert_groups_kept > l.expert_groups || l.experts % l.expert_groups != 0 ||
                l.expert_top > l.experts / l.expert_groups * l.expert_groups_kept)
                return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, at + "experts: equal groups, some of them kept, with at least expert_top experts");
            if (l.experts > kMaxExperts || l.expert_top > kMaxExpertTop || l.expert_groups > kMaxExpertGroups)
                return fail(nullptr, EFM_ERR_UNSUPPORTED, at + "more experts, choices or groups than the router takes");
        }
    }
    return EFM_OK;
}

cudaError_t alloc_linear(efm_b200_ctx* c, DecLinear& w, int N, int K, bool bias = false, int pad_k = 8) {
    w.N = N; w.K = K; w.Np = round_up(N, 8); w.Kp = round_up(K, pad_k);
    cudaError_t e = dev_alloc(c, &w.w, (size_t)w.Np * w.Kp);
    if (e == cudaSuccess && bias) e = dev_alloc(c, &w.bias, w.Np);
    return e;
}

// base^(-2 i / dims), rounded once.  Scaled: the pairs that turn rot_fast and rot_slow times within the original context bound a
// ramp from the frequency itself to a rot_factor-th of it.
cudaError_t alloc_inv_freq(efm_b200_ctx* c, DecoderLayer& l) {
    if (l.d.rot_kind == EFM_ROT_NONE) return cudaSuccess;
    std::vector<float> f((size_t)l.d.rot_dims / 2);
    const double dims = l.d.rot_dims, base = l.d.rot_base, factor = l.d.rot_factor;
    double lo = 0.0, hi = 0.0;
    if (factor > 0.0) {
        auto pair = [&](double turns) { return dims * std::log(l.d.rot_original / (2.0 * M_PI * turns)) / (2.0 * std::log(base)); };
        lo = std::max(std::floor(pair(l.d.rot_fast)), 0.0);
        hi = std::min(std::ceil(pair(l.d.rot_slow)), dims - 1.0);
    }
    for (size_t i = 0; i < f.size(); ++i) {
        double w = std::pow(base, -2.0 * (double)i / dims);
        if (factor > 0.0) {
            const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            w = w / factor * ramp + w * (1.0 - ramp);
        }
        f[i] = (float)w;
    }
    cudaError_t e = dev_alloc(c, &l.inv_freq, f.size());
    if (e == cudaSuccess) e = cudaStreamSynchronize(c->stream);
    return e == cudaSuccess ? cudaMemcpy(l.inv_freq, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice) : e;
}

// decay^i of every head, rounded once
cudaError_t alloc_powers(efm_b200_ctx* c, DecoderLayer& l) {
    std::vector<float> f;
    for (int h = 0; h < l.d.linear_heads; ++h)
        for (int i = 0; i <= kLinearPowers; ++i) f.push_back((float)std::pow(l.d.linear_decay[h], (double)i));
    cudaError_t e = dev_alloc(c, &l.lin_powers, f.size());
    if (e == cudaSuccess) e = cudaStreamSynchronize(c->stream);
    return e == cudaSuccess ? cudaMemcpy(l.lin_powers, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice) : e;
}

cudaError_t alloc_norm(efm_b200_ctx* c, DecNorm& n, int width, bool tanh) {
    cudaError_t e = dev_alloc(c, &n.w, width);
    if (e == cudaSuccess && tanh) e = dev_alloc(c, &n.b, width);
    if (e == cudaSuccess && tanh) e = dev_alloc(c, &n.alpha, 1);
    return e;
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
    EFM_TRY(configure_sampler());
    m->extended = desc->norm_layout == EFM_NORM_OUTPUT && (desc->conv_taps > 0 || desc->depth_average || desc->logit_softcap > 0.f);
    for (int i = 0; i < desc->num_layers; ++i) {
        const efm_decoder_layer& l = layers[i];
        m->extended = m->extended || l.mixer == EFM_MIXER_LINEAR || l.out_bias || (l.experts > 0 && l.expert_glu == EFM_GLU_NONE_RELU2) ||
                      (desc->norm_layout == EFM_NORM_OUTPUT && (l.experts > 0 || l.qkv_bias));
    }
    const bool outputs = desc->norm_layout != EFM_NORM_INPUT, inputs = desc->norm_layout != EFM_NORM_OUTPUT, tanh = !outputs;
    for (int i = 0; i < desc->num_layers; ++i) {
        const int times = desc->loop_times > 1 && i == desc->loop_start ? desc->loop_times : 1;
        const int stop = times > 1 ? desc->loop_stop : i + 1;
        for (int t = 0; t < times; ++t)
            for (int k = i; k < stop; ++k) {
                DecoderRun r;
                r.layer = k;
                m->runs.push_back(r);
            }
        i = stop - 1;
    }

    const size_t rows = (size_t)std::max(desc->cache_pages, 1) * EFM_PAGE_TOKENS, es = act_bytes(*m);
    size_t w_in = 8, w_mix = 8, w_ff = 8, w_q = 8, w_delta_in = 8, n_pack = 8, w_rank = 8, w_cq = 8, k_max = Wp;
    size_t ws_c = 0, ws_kv = 0, n_experts = 0, w_route = 8, ex_ff = 0, top = 0, w_act = 8, n_lin = 0, w_lin = 0, sh_ff = 0;
    size_t w_proj_f = 0, w_decay = 0;
    bool any_delta = false, any_dense = false, ws_full = false;
    m->layers.resize(desc->num_layers);
    for (int i = 0; i < desc->num_layers; ++i) {
        DecoderLayer& l = m->layers[i];
        l.d = layers[i];
        const efm_decoder_layer& d = l.d;
        if (outputs) EFM_TRY(dev_alloc(c, &l.post1, Wp));
        if (inputs) EFM_TRY(alloc_norm(c, l.pre1, Wp, tanh));
        if (desc->conv_taps > 0) {
            EFM_TRY(dev_alloc(c, &l.canon1, (size_t)desc->conv_taps * Wp));
            if (l.mlp()) EFM_TRY(dev_alloc(c, &l.canon2, (size_t)desc->conv_taps * Wp));
        }
        if (desc->depth_average) EFM_TRY(dev_alloc(c, &l.dwa, (size_t)i + 2));
        EFM_TRY(alloc_inv_freq(c, l));
        if (l.attention()) {
            l.Dp = round_up(d.dim, 64);
            l.Vp = round_up(d.vdim, 64);
            l.mix_w = d.heads * d.vdim;
            int n_in = (d.heads + d.kv_heads) * d.dim + d.kv_heads * d.vdim;
            if (d.out_gate) n_in += d.heads;
            if (l.parallel()) {
                const int v = d.linear_heads * d.linear_vdim;
                l.lin_vp = round_up(d.linear_vdim, 4);
                l.lin_in = round_up(n_in, 8);
                n_in = l.lin_in + 2 * l.linear_qk() + 2 * l.linear_v();
                l.lin_mix = round_up(l.mix_w, 8);
                l.mix_w = l.lin_mix + v;
                EFM_TRY(dev_alloc(c, &l.mix_norm, round_up(v, 8)));
                EFM_TRY(alloc_powers(c, l));
                n_lin = std::max(n_lin, decoder_linear_ws_floats(l, S, std::min(desc->max_slots, S)));
                w_lin = std::max(w_lin, (size_t)round_up(v, 8));
            }
            l.d.linear_decay = nullptr;
            EFM_TRY(alloc_linear(c, l.in, n_in, m->W, d.qkv_bias != 0));
            if (d.qk_norm == EFM_QK_NORM_WEIGHTED || d.qk_norm == EFM_QK_NORM_ROW) {
                const bool row = d.qk_norm == EFM_QK_NORM_ROW;
                EFM_TRY(dev_alloc(c, &l.q_norm, row ? d.heads * d.dim : d.dim));
                EFM_TRY(dev_alloc(c, &l.k_norm, row ? d.kv_heads * d.dim : d.dim));
            }
            if (d.score_weights == EFM_WEIGHTS_SIGMOID) EFM_TRY(dev_alloc(c, &l.shift, d.heads));
            if (d.head_temp) EFM_TRY(dev_alloc(c, &l.temp, d.heads));
            w_q = std::max(w_q, (size_t)d.heads * l.Dp);
            w_in = std::max(w_in, (size_t)l.in.Np);
        } else if (d.mixer == EFM_MIXER_LATENT_ATTENTION) {
            l.Dp = round_up(d.dim, 8);
            l.Vp = round_up(d.vdim, 8);
            l.Qp = round_up(d.q_rank, 8);
            l.Lc = round_up(d.kv_rank, 8);
            l.Rc = round_up(d.rot_dims, 8);
            l.mix_w = d.heads * d.vdim;
            EFM_TRY(alloc_linear(c, l.in, l.Qp + l.Lc + l.Rc + (d.out_gate == EFM_GATE_HEADS ? d.heads : d.out_gate ? d.heads * d.vdim : 0), m->W));
            EFM_TRY(alloc_linear(c, l.uq, d.heads * (l.Dp + l.Rc), d.q_rank));
            EFM_TRY(alloc_linear(c, l.ukv, d.heads * (l.Dp + l.Vp), d.kv_rank));
            EFM_TRY(dev_alloc(c, &l.q_norm, l.Qp));
            EFM_TRY(dev_alloc(c, &l.k_norm, l.Lc));
            if (d.sink) EFM_TRY(dev_alloc(c, &l.sink, d.heads));
            w_q = std::max(w_q, (size_t)l.uq.Np);
            w_cq = std::max(w_cq, (size_t)l.Qp);
            w_in = std::max(w_in, (size_t)l.in.Np);
            k_max = std::max(k_max, (size_t)l.uq.Kp);
            if (decoder_layer_tc(*m, l)) {
                ws_c = std::max(ws_c, (size_t)(l.Lc + l.Rc));
                ws_kv = std::max(ws_kv, (size_t)l.ukv.Np);
                ws_full = ws_full || d.window == 0;
                m->ws_window = std::max(m->ws_window, d.window);
            }
        } else if (l.alone()) {
            const int v = d.linear_heads * d.linear_vdim, rank = l.channel_decay() ? d.decay_rank : 0;
            l.lin_vp = round_up(d.linear_vdim, 4);
            l.mix_w = v;
            EFM_TRY(alloc_linear(c, l.in, 2 * l.linear_qk() + 2 * l.linear_v() + rank, m->W));
            if (d.linear_norm) EFM_TRY(dev_alloc(c, &l.mix_norm, d.linear_vdim));
            if (rank > 0) {
                EFM_TRY(alloc_linear(c, l.w2, d.linear_heads * d.linear_dim, rank, true));
                w_decay = std::max(w_decay, (size_t)l.w2.Np);
            } else {
                EFM_TRY(alloc_powers(c, l));
            }
            l.d.linear_decay = nullptr;
            n_lin = std::max(n_lin, decoder_linear_ws_floats(l, S, std::min(desc->max_slots, S)));
            w_lin = std::max(w_lin, (size_t)l.linear_v());
            w_in = std::max(w_in, (size_t)l.in.Np);
            if (d.rot_kind != EFM_ROT_NONE && !m->f32) {
                if (d.linear_dim % 32 == 0 && d.rot_dims % 32 == 0) {
                    for (size_t k = 0; k < m->rot_tables.size() && l.rot_table < 0; ++k) {
                        const efm_decoder_layer& o = layers[m->rot_tables[k].layer];
                        if (o.rot_dims == d.rot_dims && o.rot_base == d.rot_base && o.rot_factor == d.rot_factor && o.rot_original == d.rot_original &&
                            o.rot_fast == d.rot_fast && o.rot_slow == d.rot_slow)
                            l.rot_table = (int)k;
                    }
                    if (l.rot_table < 0) {
                        DecoderModel::RotTable t;
                        t.dims = d.rot_dims;
                        t.layer = i;
                        EFM_TRY(dev_alloc(c, &t.cs, (size_t)S * (d.rot_dims / 2)));
                        l.rot_table = (int)m->rot_tables.size();
                        m->rot_tables.push_back(t);
                    }
                } else {
                    w_proj_f = std::max(w_proj_f, (size_t)l.in.Np);
                }
            }
        } else {
            any_delta = true;
            const int HD = d.heads * d.dim;
            l.mix_w = HD;
            EFM_TRY(alloc_linear(c, l.in, 5 * HD + d.decay_rank, m->W));
            EFM_TRY(alloc_linear(c, l.w2, HD, d.decay_rank));
            EFM_TRY(dev_alloc(c, &l.w0, HD));
            EFM_TRY(dev_alloc(c, &l.a_bias, HD));
            EFM_TRY(dev_alloc(c, &l.mix_norm, HD));
            w_delta_in = std::max(w_delta_in, (size_t)l.in.Np);
            n_pack = std::max(n_pack, decoder_delta_pack_floats(d.heads, d.dim, S, std::min(desc->max_slots, S)));
            w_rank = std::max(w_rank, (size_t)l.w2.Kp);
        }
        l.mix_wp = round_up(l.mix_w, 8);
        w_mix = std::max(w_mix, (size_t)l.mix_wp);
        EFM_TRY(alloc_linear(c, l.out, m->W, l.mix_w, d.out_bias != 0));
        if (l.mlp()) {
            if (outputs) EFM_TRY(dev_alloc(c, &l.post2, Wp));
            if (inputs) EFM_TRY(alloc_norm(c, l.pre2, Wp, tanh));
        }
        if (l.moe()) {
            l.ffp = round_up(d.expert_ff, 64);
            EFM_TRY(alloc_linear(c, l.router, d.experts + (d.shared_ff > 0 && d.shared_gate == EFM_SHARED_GATED ? 1 : 0), m->W));
            EFM_TRY(alloc_linear(c, l.expert_in, d.experts * l.up_rows(l.ffp), m->W));
            EFM_TRY(alloc_linear(c, l.expert_out, d.experts * Wp, d.expert_ff, false, 64));
            n_experts = std::max(n_experts, (size_t)d.experts);
            w_route = std::max(w_route, (size_t)l.router.Np);
            ex_ff = std::max(ex_ff, (size_t)l.ffp);
            top = std::max(top, (size_t)d.expert_top);
            if (d.shared_ff > 0) {
                l.sfp = round_up(d.shared_ff, 64);
                EFM_TRY(alloc_linear(c, l.shared_in, l.up_rows(l.sfp), m->W));
                EFM_TRY(alloc_linear(c, l.shared_out, m->W, d.shared_ff, false, 64));
                sh_ff = std::max(sh_ff, (size_t)l.sfp);
            }
            w_act = std::max(w_act, (size_t)d.expert_top * l.ffp + l.sfp);
            k_max = std::max(k_max, (size_t)d.expert_top * l.ffp + l.sfp);
        } else if (d.ff > 0) {
            any_dense = true;
            EFM_TRY(alloc_linear(c, l.up, d.ff, m->W));
            EFM_TRY(alloc_linear(c, l.down, m->W, d.ff));
            if (d.ff_act == EFM_ACT_POLYNORM) EFM_TRY(dev_alloc(c, &l.act, 4));
            w_ff = std::max(w_ff, (size_t)l.up.Np);
        }
        if (desc->side_dim > 0) {
            EFM_TRY(alloc_linear(c, l.gate, desc->side_dim, m->W));
            EFM_TRY(alloc_linear(c, l.proj, m->W, desc->side_dim));
            EFM_TRY(dev_alloc(c, &l.side_norm, Wp));
        }
        k_max = std::max(k_max, std::max((size_t)l.out.Kp, (size_t)(d.ff > 0 ? l.down.Kp : 0)));
    }
    EFM_TRY(configure_decoder(*m));
    for (DecoderRun& r : m->runs) {
        const DecoderLayer& l = m->layers[r.layer];
        char *k = nullptr, *v = nullptr;
        if (l.linear()) {
            r.state_off = m->state_stride;
            m->state_stride += (size_t)l.d.linear_heads * l.d.linear_dim * l.lin_vp;
        }
        if (desc->conv_taps > 0) {
            r.conv1_off = m->state_stride;
            r.conv2_off = r.conv1_off + (size_t)desc->conv_taps * Wp;
            m->state_stride = r.conv2_off + (l.mlp() ? (size_t)desc->conv_taps * Wp : 0);
        }
        if (l.attention()) {
            EFM_TRY(dev_alloc(c, &k, rows * l.d.kv_heads * l.Dp * es));
            EFM_TRY(dev_alloc(c, &v, rows * l.d.kv_heads * l.Vp * es));
        } else if (l.d.mixer == EFM_MIXER_LATENT_ATTENTION) {
            EFM_TRY(dev_alloc(c, &k, rows * (l.Lc + l.Rc) * es));
        } else if (!l.alone()) {
            r.state_off = m->state_stride;
            m->state_stride += ((size_t)l.d.heads * l.d.dim * l.d.dim + 3) / 4 * 4;
        }
        r.k_pool = k;
        r.v_pool = v;
    }
    {   // the longest GEMV input must fit the kernel's shared memory as fp32
        int optin = 0;
        EFM_TRY(cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, device_id));
        size_t need = std::max(std::max(gemv_smem_bytes((int)k_max), gemv_ext_smem_bytes(Wp)), gemv_ext_smem_bytes((int)w_cq));
        if (desc->conv_taps > 0) need = std::max(need, gemv_conv_smem_bytes(Wp));
        for (const DecoderLayer& l : m->layers)
            if (l.parallel()) need = std::max(need, gemv_ext_smem_bytes(l.out.Kp));
        if (need + 2048 > (size_t)optin) {
            efm_status s = fail(nullptr, EFM_ERR_UNSUPPORTED, "width / feed-forward size exceeds what the decode GEMV stages in shared memory");
            efm_b200_destroy(c);
            return s;
        }
    }
    EFM_TRY(alloc_linear(c, m->head, desc->vocab, m->W));
    if (desc->tied_head) c->embed = m->head.w;
    else EFM_TRY(dev_alloc(c, &c->embed, (size_t)desc->vocab * Wp));
    if (desc->side_dim > 0) EFM_TRY(dev_alloc(c, &m->side_embed, (size_t)desc->vocab * desc->side_dim * desc->num_layers));
    EFM_TRY(alloc_norm(c, m->final_norm, Wp, tanh));
    c->lm_head = m->head.w;
    c->final_norm = m->final_norm.w;

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
    if (!m->f32 || inputs || desc->conv_taps > 0) EFM_TRY(act(&m->xa, (size_t)S * Wp));
    if (desc->depth_average) {
        EFM_TRY(dev_alloc(c, &m->hist, ((size_t)desc->num_layers + 1) * S * Wp));
        EFM_TRY(dev_alloc(c, &m->d_hist, ((size_t)desc->num_layers + 1) * Wp));
        EFM_TRY(dev_alloc(c, &m->d_avg, Wp));
    }
    EFM_TRY(act(&m->cq, S * w_cq));
    if (ws_c > 0) {
        // the rows' own pages plus, for every entry long enough, those of a window
        if (ws_full) m->ws_window = 0;
        const size_t entries = std::min(desc->max_slots, std::max(1, S / kTcMinRows));
        size_t pages = (size_t)std::max(desc->cache_pages, 1);
        if (!ws_full) pages = std::min(pages, (size_t)S / EFM_PAGE_TOKENS + 1 + entries * ((size_t)m->ws_window / EFM_PAGE_TOKENS + 3));
        m->ws_pages = (int)pages;
        EFM_TRY(dev_alloc(c, &m->ws_c, pages * EFM_PAGE_TOKENS * ws_c));
        EFM_TRY(dev_alloc(c, &m->ws_kv, pages * EFM_PAGE_TOKENS * ws_kv));
    }
    if (n_experts > 0) {
        const size_t picks = (size_t)S * top;
        m->ex_rows = (int)((picks / kExpertTile + std::min(picks, n_experts)) * kExpertTile);
        EFM_TRY(act(&m->ex_in, (size_t)m->ex_rows * Wp));
        EFM_TRY(act(&m->ex_act, (size_t)m->ex_rows * ex_ff));
        if (m->f32) EFM_TRY(dev_alloc(c, &m->ex_gu, (size_t)m->ex_rows * 2 * ex_ff));
        EFM_TRY(act(&m->ex_y, (size_t)m->ex_rows * Wp));
        EFM_TRY(dev_alloc(c, &m->route_logits, S * w_route));
        EFM_TRY(dev_alloc(c, &m->ex.id, picks));
        EFM_TRY(dev_alloc(c, &m->ex.weight, picks));
        EFM_TRY(dev_alloc(c, &m->ex.place, picks));
        EFM_TRY(dev_alloc(c, &m->ex.count, n_experts));
        EFM_TRY(dev_alloc(c, &m->ex.tile, (size_t)m->ex_rows / kExpertTile));
        EFM_TRY(dev_alloc(c, &m->ex.n_tiles, 1));
        EFM_TRY(dev_alloc(c, &m->ex.shared, S));
        if (sh_ff > 0) {
            EFM_TRY(cudaStreamCreateWithFlags(&m->side, cudaStreamNonBlocking));
            EFM_TRY(cudaEventCreateWithFlags(&m->side_start, cudaEventDisableTiming));
            EFM_TRY(cudaEventCreateWithFlags(&m->side_end, cudaEventDisableTiming));
            EFM_TRY(act(&m->sh_act, S * sh_ff));
            EFM_TRY(act(&m->sh_y, (size_t)S * Wp));
            if (m->f32) EFM_TRY(dev_alloc(c, &m->sh_gu, S * 2 * sh_ff));
        }
        EFM_TRY(dev_alloc(c, &m->d_h, Wp));
        EFM_TRY(dev_alloc(c, &m->d_route, w_route));
        EFM_TRY(dev_alloc(c, &m->d_act, w_act));
        EFM_TRY(dev_alloc(c, &m->d_route_id, top));
        EFM_TRY(dev_alloc(c, &m->d_route_w, top + 1));
        EFM_TRY(dev_alloc(c, &m->d_route_ticket, 1));
    }
    if (n_lin > 0) EFM_TRY(dev_alloc(c, &m->lin_ws, n_lin));
    if (n_lin > 0 || any_delta) EFM_TRY(dev_alloc(c, &m->o, S * std::max(w_lin, any_delta ? w_mix : 0)));
    EFM_TRY(act(&m->proj_a, S * w_in));
    EFM_TRY(act(&m->q, S * w_q));
    EFM_TRY(act(&m->mix, S * w_mix));
    if (any_dense) {
        EFM_TRY(act(&m->ff, S * w_ff));
        EFM_TRY(act(&m->ff2, S * w_ff));
    }
    EFM_TRY(act(&m->side_a, (size_t)S * m->side_p));
    EFM_TRY(dev_alloc(c, &m->side_f, (size_t)S * m->side_p));
    EFM_TRY(dev_alloc(c, &m->y, (size_t)S * Wp));
    if (any_delta) {
        EFM_TRY(dev_alloc(c, &m->pack, n_pack));
        EFM_TRY(dev_alloc(c, &m->tanh_w, S * w_rank));
        w_proj_f = std::max(w_proj_f, w_delta_in);
        w_decay = std::max(w_decay, w_mix);
    }
    if (w_proj_f > 0) EFM_TRY(dev_alloc(c, &m->proj_f, S * w_proj_f));
    if (w_decay > 0) EFM_TRY(dev_alloc(c, &m->decay, S * w_decay));
    m->max_want = std::min(S, 256);
    EFM_TRY(act(&m->head_a, (size_t)m->max_want * Wp));
    EFM_TRY(dev_alloc(c, &m->logits_rows, (size_t)m->max_want * m->head.Np));
    // per pass: ids, row entries, wanted rows, short rows, tile and page lists, entries
    m->step_words = (size_t)S * 4 + 2 * (size_t)S * 2 + (size_t)m->ws_pages * 2 + (size_t)S * (sizeof(RowEntry) / 4) + 64;
    EFM_TRY(dev_alloc(c, &m->step_buf, m->step_words));

    EFM_TRY(dev_alloc(c, &c->resid_d, Wp));
    EFM_TRY(dev_alloc(c, &c->resid_d2, Wp));
    EFM_TRY(dev_alloc(c, &m->d_in, std::max(w_in, w_delta_in)));
    EFM_TRY(dev_alloc(c, &m->d_q, w_q));
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
        std::vector<RowTile> tc, simt, ws;
        std::vector<int32_t> short_rows;
        int n_ws = 0;
        struct Want { int32_t row; int64_t idx; uint32_t rng_step; };
        std::vector<Want> wants;
        int rows = 0;
        for (int e = first; e < n_entries && rows < c->max_s; ++e) {
            const efm_step_entry& en = entries[e];
            const int n = std::min(en.n_tokens - done[e], c->max_s - rows);
            KvSlot& s = c->slots.at(en.slot);
            RowEntry r{rows, n, en.kv_offset + done[e], s.table, s.state_slot, 0};
            const int idx = (int)re.size(), step = n >= kTcMinRows ? decoder_tc_tile_rows() : decoder_simt_tile_rows();
            for (int i = 0; i < n; i += step) (n >= kTcMinRows ? tc : simt).push_back(RowTile{idx, i});
            if (n < kTcMinRows)
                for (int i = 0; i < n; ++i) short_rows.push_back(rows + i);
            else if (m.ws_pages > 0) {
                const int p0 = decoder_ws_page0(m, r.pos0), p1 = (r.pos0 + n - 1) / EFM_PAGE_TOKENS;
                r.ws0 = (n_ws - p0) * EFM_PAGE_TOKENS;
                n_ws += p1 - p0 + 1;
                for (int p = p0; p * EFM_PAGE_TOKENS < r.pos0; ++p) ws.push_back(RowTile{idx, p});
            }
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
        if (n_ws > m.ws_pages) return fail(c, EFM_ERR_STATE, "the entries see more cache pages than the pool has");
        // late rows see the most keys; the kernel takes the last tiles first
        std::stable_sort(tc.begin(), tc.end(), [&](const RowTile& a, const RowTile& b) { return re[a.entry].pos0 + a.row < re[b.entry].pos0 + b.row; });
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
                     o_all = put(all_simt.data(), all_simt.size() * 2), o_want = put(want_rows.data(), want_rows.size()),
                     o_short = put(short_rows.data(), short_rows.size()), o_ws = put(ws.data(), ws.size() * 2);
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
        tiles.short_rows = m.step_buf + o_short;
        tiles.n_short = (int)short_rows.size();
        tiles.ws_pages = reinterpret_cast<const RowTile*>(m.step_buf + o_ws);
        tiles.n_ws = n_ws;
        tiles.n_gather = (int)ws.size();
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
    if (rows > 0) EFM_CK(c, dev_alloc(c, &m.tap, m.runs.size() * rows * m.Wp));
    return EFM_OK;
}

efm_status efm_b200_decoder_read_taps(efm_b200_ctx* c, float* host_out) {
    if (c == nullptr || c->decoder == nullptr || host_out == nullptr || c->decoder->tap == nullptr) return fail(c, EFM_ERR_INVALID_ARGUMENT, "no taps are set");
    DecoderModel& m = *c->decoder;
    EFM_CK(c, cudaMemcpy2DAsync(host_out, (size_t)m.W * 4, m.tap, (size_t)m.Wp * 4, (size_t)m.W * 4, m.runs.size() * m.tap_rows,
                                cudaMemcpyDeviceToHost, c->stream));
    return ctx_sync(c);
}

}  // extern "C"

namespace {

// ---- weights -------------------------------------------------------------------------------------------------------
// Rows [src, src + n) of a tensor become rows [dst, dst + n) of a (fused, padded) linear, from column `col` on.  Several tensors may
// be parts of one linear.
// step: destination rows from one to the next.
struct Piece { int dst, src, n, col = 0, step = 1; };

efm_status put_rows(efm_b200_ctx* c, const DecLinear& w, const std::vector<Piece>& pieces, const void* data, const std::string& name, const int64_t* shape,
                    int ndim, int mem_kind, int cols) {
    const int K = cols > 0 ? cols : w.K;             // a part of the linear's columns, or all
    int rows = 0;
    for (const Piece& p : pieces) rows += p.n;
    if (!shape_is(shape, ndim, rows, K)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + name);
    for (const Piece& p : pieces)
        EFM_CK(c, cudaMemcpy2DAsync(w.w + (size_t)p.dst * w.Kp + p.col, (size_t)w.Kp * 2 * p.step, static_cast<const char*>(data) + (size_t)p.src * K * 2, (size_t)K * 2,
                                    (size_t)K * 2, (size_t)p.n, mem_kind == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice, c->stream));
    return EFM_OK;
}
efm_status put_vec(efm_b200_ctx* c, __nv_bfloat16* dst, int n, const void* data, const std::string& name, const int64_t* shape, int ndim, int mem_kind) {
    if (!(n == 1 && ndim == 0) && !shape_is(shape, ndim, n)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + name);
    return copy_rows(c, dst, data, (size_t)n * 2, mem_kind);
}

// Where a tensor goes: a row range of a (fused) linear or a vector.
// taps > 0: [n, taps] into the vector, tap by tap (row stride ld).
struct Target { DecLinear* lin = nullptr; std::vector<Piece> pieces; int cols = 0; __nv_bfloat16* vec = nullptr; int n = 0, taps = 0, ld = 0; };
efm_status put_taps(efm_b200_ctx* c, const Target& t, const void* data, const std::string& name, const int64_t* shape, int ndim, int mem_kind) {
    if (!shape_is(shape, ndim, t.n, t.taps)) return fail(c, EFM_ERR_INVALID_ARGUMENT, "unexpected shape for " + name);
    for (int j = 0; j < t.taps; ++j)
        EFM_CK(c, cudaMemcpy2DAsync(t.vec + (size_t)j * t.ld, 2, static_cast<const char*>(data) + (size_t)j * 2, (size_t)t.taps * 2, 2, (size_t)t.n,
                                    mem_kind == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice, c->stream));
    return EFM_OK;
}

// `name`, `name`.b or `name`.alpha of an input norm
bool norm_target(const DecoderModel& m, const DecNorm& n, const std::string& what, const char* name, Target* t) {
    const std::string base(name);
    if (what == base) { t->vec = n.w; t->n = m.W; }
    else if (what == base + ".b") { t->vec = n.b; t->n = m.W; }
    else if (what == base + ".alpha") { t->vec = n.alpha; t->n = 1; }
    return t->vec != nullptr;
}

bool layer_target(DecoderModel& m, DecoderLayer& l, int index, const std::string& rest, Target* t) {
    const efm_decoder_layer& d = l.d;
    auto lin = [&](DecLinear& w, int row0, int rows) { t->lin = &w; t->pieces.push_back(Piece{row0, 0, rows}); return true; };
    auto vec = [&](__nv_bfloat16* v, int n) { t->vec = v; t->n = n; return v != nullptr; };
    // heads of `n` rows, laid out from row0 on with `ld` rows each, `gap` more behind the first `cut` rows
    auto heads = [&](DecLinear& w, int row0, int ld, int n, int cut, int gap) {
        t->lin = &w;
        for (int h = 0; h < d.heads; ++h) {
            t->pieces.push_back(Piece{row0 + h * ld, h * n, cut});
            if (n > cut) t->pieces.push_back(Piece{row0 + h * ld + cut + gap, h * n + cut, n - cut});
        }
        return true;
    };
    const bool sandwich = m.d.norm_layout == EFM_NORM_SANDWICH;
    if (m.d.norm_layout == EFM_NORM_OUTPUT) {
        if (rest == "norm1") return vec(l.post1, m.W);
        if (rest == "norm2") return vec(l.post2, m.W);
    } else if (norm_target(m, l.pre1, rest, "norm1", t) || norm_target(m, l.pre2, rest, "norm2", t)) {
        return true;
    }
    if (sandwich && rest == "norm1b") return vec(l.post1, m.W);
    if (sandwich && rest == "norm2b") return vec(l.post2, m.W);
    if (rest == "canon1" || rest == "canon2") {
        t->vec = rest == "canon1" ? l.canon1 : l.canon2;
        t->n = m.W;
        t->taps = m.d.conv_taps;
        t->ld = m.Wp;
        return t->vec != nullptr;
    }
    if (rest == "dwa") return vec(l.dwa, index + 2);
    if (rest == "mix.o" && !l.parallel()) return lin(l.out, 0, m.W);
    if (rest == "mix.o.b") return vec(l.out.bias, m.W);
    if (l.alone()) {
        const int qk = d.linear_heads * d.linear_dim, v = d.linear_heads * d.linear_vdim, g = 2 * l.linear_qk() + l.linear_v();
        // channels that turn with each other become neighbours: q and k alike, so that their products stay what they are
        auto turned = [&](int row0) {
            const int half = d.rot_kind == EFM_ROT_HALF ? d.rot_dims / 2 : 0, D = d.linear_dim;
            t->lin = &l.in;
            for (int h = 0; h < d.linear_heads; ++h) {
                if (half > 0) {
                    t->pieces.push_back(Piece{row0 + h * D, h * D, half, 0, 2});
                    t->pieces.push_back(Piece{row0 + h * D + 1, h * D + half, half, 0, 2});
                }
                if (D > 2 * half) t->pieces.push_back(Piece{row0 + h * D + 2 * half, h * D + 2 * half, D - 2 * half});
            }
            return true;
        };
        if (rest == "mix.q") return turned(0);
        if (rest == "mix.k") return turned(l.linear_qk());
        if (rest == "mix.v") return lin(l.in, 2 * l.linear_qk(), v);
        if (rest == "mix.g") return lin(l.in, g, v);
        if (rest == "mix.norm") return vec(l.mix_norm, d.linear_vdim);
        if (l.channel_decay()) {
            if (rest == "mix.a1") return lin(l.in, g + l.linear_v(), d.decay_rank);
            if (rest == "mix.a2") return lin(l.w2, 0, qk);
            if (rest == "mix.a2.b") return vec(l.w2.bias, qk);
        }
    } else if (l.parallel()) {                                  // the two halves share one projection and one output product
        const int q = d.heads * d.dim, k = d.kv_heads * d.dim, lv = d.linear_heads * d.linear_vdim, lq = d.linear_heads * d.linear_dim;
        auto out = [&](int col, int cols) { t->lin = &l.out; t->cols = cols; t->pieces.push_back(Piece{0, 0, m.W, col}); return true; };
        if (rest == "mix.left.q") return lin(l.in, 0, q);
        if (rest == "mix.left.k") return lin(l.in, q, k);
        if (rest == "mix.left.v") return lin(l.in, q + k, d.kv_heads * d.vdim);
        if (rest == "mix.left.o") return out(0, d.heads * d.vdim);
        const int qp = round_up(lq, 8), vp = round_up(lv, 8);
        if (rest == "mix.right.q") return lin(l.in, l.lin_in, lq);
        if (rest == "mix.right.k") return lin(l.in, l.lin_in + qp, lq);
        if (rest == "mix.right.v") return lin(l.in, l.lin_in + 2 * qp, lv);
        if (rest == "mix.right.g") return lin(l.in, l.lin_in + 2 * qp + vp, lv);
        if (rest == "mix.right.o") return out(l.lin_mix, lv);
        if (rest == "mix.right.norm") return vec(l.mix_norm, lv);
    } else if (d.mixer == EFM_MIXER_ATTENTION) {
        const int q = d.heads * d.dim, k = d.kv_heads * d.dim;
        if (rest == "mix.q") return lin(l.in, 0, q);
        if (rest == "mix.k") return lin(l.in, q, k);
        if (rest == "mix.v") return lin(l.in, q + k, d.kv_heads * d.vdim);
        const bool row = d.qk_norm == EFM_QK_NORM_ROW;
        if (rest == "mix.q.norm") return vec(l.q_norm, row ? q : d.dim);
        if (rest == "mix.k.norm") return vec(l.k_norm, row ? k : d.dim);
        if (rest == "mix.pb") return vec(l.shift, d.heads);
        if (rest == "mix.g" && d.out_gate) return lin(l.in, q + k + d.kv_heads * d.vdim, d.heads);
        if (rest == "mix.temp") return vec(l.temp, d.heads);
        if (d.qkv_bias) {
            if (rest == "mix.q.b") return vec(l.in.bias, q);
            if (rest == "mix.k.b") return vec(l.in.bias + q, k);
            if (rest == "mix.v.b") return vec(l.in.bias + q + k, d.kv_heads * d.vdim);
        }
    } else if (d.mixer == EFM_MIXER_LATENT_ATTENTION) {
        if (rest == "mix.dq") return lin(l.in, 0, d.q_rank);
        if (rest == "mix.dkv") {
            lin(l.in, l.Qp, d.kv_rank);
            t->pieces.push_back(Piece{l.Qp + l.Lc, d.kv_rank, d.rot_dims});
            return true;
        }
        if (rest == "mix.g" && d.out_gate) return lin(l.in, l.Qp + l.Lc + l.Rc, d.out_gate == EFM_GATE_HEADS ? d.heads : d.heads * d.vdim);
        if (rest == "mix.uq") return heads(l.uq, 0, l.Dp + l.Rc, d.dim + d.rot_dims, d.dim, l.Dp - d.dim);
        if (rest == "mix.uk") return heads(l.ukv, 0, l.Dp, d.dim, d.dim, 0);
        if (rest == "mix.uv") return heads(l.ukv, d.heads * l.Dp, l.Vp, d.vdim, d.vdim, 0);
        if (rest == "mix.dq.norm") return vec(l.q_norm, d.q_rank);
        if (rest == "mix.dkv.norm") return vec(l.k_norm, d.kv_rank);
        if (rest == "mix.sink") return vec(l.sink, d.heads);
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
    if (l.moe()) {
        if (rest == "mlp.router") return lin(l.router, 0, d.experts);
        auto gate_up = [&](DecLinear& w, int row0, int n, bool up) {     // 64 gate rows, the 64 matching up rows, ...
            if (!l.gated_experts()) return up && lin(w, row0, n);
            t->lin = &w;
            for (int r = 0; r < n; r += 64) t->pieces.push_back(Piece{row0 + 2 * r + (up ? 64 : 0), r, std::min(64, n - r)});
            return true;
        };
        if (d.shared_ff > 0) {
            if (rest == "mlp.shared.gate" || rest == "mlp.shared.up") return gate_up(l.shared_in, 0, d.shared_ff, rest == "mlp.shared.up");
            if (rest == "mlp.shared.down") return lin(l.shared_out, 0, m.W);
            if (rest == "mlp.shared.sg" && d.shared_gate == EFM_SHARED_GATED) return lin(l.router, d.experts, 1);
        }
        const size_t dot = rest.find('.', 5);
        if (rest.compare(0, 5, "mlp.e") == 0 && dot != std::string::npos && dot > 5) {
            const int e = std::atoi(rest.c_str() + 5);
            const std::string what = rest.substr(dot + 1);
            if (rest.substr(5, dot - 5) != std::to_string(e) || e >= d.experts) return false;
            if (what == "down") return lin(l.expert_out, e * m.Wp, m.W);
            if (what != "gate" && what != "up") return false;
            return gate_up(l.expert_in, e * l.up_rows(l.ffp), d.expert_ff, what == "up");
        }
    } else if (d.ff > 0) {
        if (rest == "mlp.up") return lin(l.up, 0, d.ff);
        if (rest == "mlp.down") return lin(l.down, 0, m.W);
        if (rest == "mlp.act" && l.act != nullptr) return vec(l.act, 4);
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
    if (name == "embed") { table.w = c->embed; table.K = m.W; table.Kp = m.Wp; t.lin = &table; t.pieces.push_back(Piece{0, 0, m.d.vocab}); }
    else if (name == "side.embed" && m.side_embed != nullptr) {
        table.w = m.side_embed; table.K = table.Kp = m.d.side_dim * m.d.num_layers;
        t.lin = &table; t.pieces.push_back(Piece{0, 0, m.d.vocab});
    }
    else if (name == "head" && !m.d.tied_head) { t.lin = &m.head; t.pieces.push_back(Piece{0, 0, m.d.vocab}); }
    else if (norm_target(m, m.final_norm, name, "final.norm", &t)) {}
    else if (name.size() > 1 && name[0] == 'l' && name[1] >= '0' && name[1] <= '9') {
        const size_t dot = name.find('.');
        const int i = std::atoi(name.c_str() + 1);
        if (dot == std::string::npos || i < 0 || i >= m.d.num_layers || !layer_target(m, m.layers[i], i, name.substr(dot + 1), &t)) return EFM_OK;
    } else {
        return EFM_OK;                     // not part of this model
    }
    if (dtype != EFM_BF16) return fail(c, EFM_ERR_UNSUPPORTED, "weights must be bf16: " + name);
    const efm_status st = t.taps > 0 ? put_taps(c, t, data, name, shape, ndim, mem_kind) : t.lin != nullptr ? put_rows(c, *t.lin, t.pieces, data, name, shape, ndim, mem_kind, t.cols)
                                           : put_vec(c, t.vec, t.n, data, name, shape, ndim, mem_kind);
    if (st != EFM_OK) return st;
    EFM_CK(c, cudaStreamSynchronize(c->stream));          // the caller may release `data` on return
    m.seen.insert(name);
    return EFM_OK;
}

efm_status decoder_finalize(efm_b200_ctx* c) {
    DecoderModel& m = *c->decoder;
    const bool tanh = m.tanh_norms();
    std::vector<std::string> need = {"embed", "final.norm"};
    if (!m.d.tied_head) need.push_back("head");
    if (tanh) for (const char* n : {"final.norm.b", "final.norm.alpha"}) need.push_back(n);
    if (m.d.side_dim > 0) need.push_back("side.embed");
    for (int i = 0; i < m.d.num_layers; ++i) {
        const efm_decoder_layer& d = m.layers[i].d;
        auto add = [&](std::initializer_list<const char*> names) { for (const char* n : names) need.push_back("l" + std::to_string(i) + "." + n); };
        add({"norm1"});
        if (m.d.conv_taps > 0) add({"canon1"});
        if (m.layers[i].canon2 != nullptr) add({"canon2"});
        if (m.d.depth_average) add({"dwa"});
        if (d.out_bias) add({"mix.o.b"});
        if (tanh) add({"norm1.b", "norm1.alpha"});
        if (d.mixer != EFM_MIXER_PARALLEL) add({"mix.o"});
        if (m.d.norm_layout == EFM_NORM_SANDWICH) add({"norm1b"});
        if (d.mixer == EFM_MIXER_ATTENTION) {
            add({"mix.q", "mix.k", "mix.v"});
            if (d.qk_norm == EFM_QK_NORM_WEIGHTED || d.qk_norm == EFM_QK_NORM_ROW) add({"mix.q.norm", "mix.k.norm"});
            if (d.score_weights == EFM_WEIGHTS_SIGMOID) add({"mix.pb"});
            if (d.out_gate) add({"mix.g"});
            if (d.head_temp) add({"mix.temp"});
            if (d.qkv_bias) add({"mix.q.b", "mix.k.b", "mix.v.b"});
        } else if (d.mixer == EFM_MIXER_PARALLEL) {
            add({"mix.left.q", "mix.left.k", "mix.left.v", "mix.left.o", "mix.right.q", "mix.right.k", "mix.right.v", "mix.right.g", "mix.right.o", "mix.right.norm"});
        } else if (d.mixer == EFM_MIXER_LATENT_ATTENTION) {
            add({"mix.dq", "mix.dq.norm", "mix.uq", "mix.dkv", "mix.dkv.norm", "mix.uk", "mix.uv"});
            if (d.sink) add({"mix.sink"});
            if (d.out_gate) add({"mix.g"});
        } else if (d.mixer == EFM_MIXER_LINEAR) {
            add({"mix.q", "mix.k", "mix.v", "mix.g"});
            if (d.linear_norm) add({"mix.norm"});
            if (d.linear_tau > 0.f) add({"mix.a1", "mix.a2", "mix.a2.b"});
        } else add({"mix.r", "mix.k", "mix.v", "mix.g", "mix.a", "mix.a.b", "mix.w1", "mix.w2", "mix.w0", "mix.norm"});
        if (d.experts > 0 || d.ff > 0) {
            add({"norm2"});
            if (tanh) add({"norm2.b", "norm2.alpha"});
            if (m.d.norm_layout == EFM_NORM_SANDWICH) add({"norm2b"});
        }
        if (d.experts > 0) {
            add({"mlp.router"});
            const bool gated = d.expert_glu != EFM_GLU_NONE_RELU2;
            if (d.shared_ff > 0) {
                add({"mlp.shared.up", "mlp.shared.down"});
                if (gated) add({"mlp.shared.gate"});
                if (d.shared_gate == EFM_SHARED_GATED) add({"mlp.shared.sg"});
            }
            for (int e = 0; e < d.experts; ++e)
                for (const char* what : {".gate", ".up", ".down"})
                    if (gated || what[1] != 'g') add({("mlp.e" + std::to_string(e) + what).c_str()});
        } else if (d.ff > 0) {
            add({"mlp.up", "mlp.down"});
            if (d.ff_act == EFM_ACT_POLYNORM) add({"mlp.act"});
        }
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
    plan.one = RowEntry{0, S, kv_offset, slot.table, slot.state_slot, 0};
    RowTiles tiles;
    if (m.ws_pages > 0) {
        tiles.ws_page0 = decoder_ws_page0(m, kv_offset);
        tiles.n_ws = (kv_offset + S - 1) / EFM_PAGE_TOKENS - tiles.ws_page0 + 1;
        tiles.n_gather = std::max(0, (kv_offset + EFM_PAGE_TOKENS - 1) / EFM_PAGE_TOKENS - tiles.ws_page0);
        plan.one.ws0 = -tiles.ws_page0 * EFM_PAGE_TOKENS;
    }
    plan.page_table = m.page_table;
    plan.max_pages = m.d.cache_pages;
    plan.n_entries = 1;
    plan.rows = S;
    decoder_rows_pass(c, plan, c.ids, tiles, L);
    if (sample_last && L.err == cudaSuccess) L.err = cudaErrorNotSupported;     // a sampled prefill ends with a decode step
}
void decoder_step_op(efm_b200_ctx& c, KvSlot& slot, Launcher& L) { decoder_decode_step(c, slot, L, true, true); }

int64_t decoder_step_bytes(const efm_b200_ctx& c, int32_t kv_len) {
    const DecoderModel& m = *c.decoder;
    auto lin = [](const DecLinear& w) { return (int64_t)w.N * w.K * 2; };
    int64_t b = lin(m.head) + (int64_t)m.W * 2 * 2;
    for (const DecoderRun& r : m.runs) {
        const DecoderLayer& l = m.layers[r.layer];
        b += lin(l.in) + lin(l.out) + lin(l.w2) + lin(l.up) + lin(l.down) + lin(l.gate) + lin(l.proj) + lin(l.uq) + lin(l.ukv) + lin(l.router) + lin(l.shared_in) + lin(l.shared_out);
        if (l.moe()) b += (int64_t)l.d.expert_top * (l.gated_experts() ? 3 : 2) * l.d.expert_ff * m.W * 2;
        if (m.d.conv_taps > 0) b += (int64_t)(l.mlp() ? 2 : 1) * m.d.conv_taps * m.W * 6;
        const int64_t n = l.d.window > 0 ? std::min(kv_len, l.d.window + l.d.keep_first) : kv_len;
        if (l.linear()) b += 2 * (int64_t)l.d.linear_heads * l.d.linear_dim * l.lin_vp * 4;
        if (l.attention()) b += n * l.d.kv_heads * (l.d.dim + l.d.vdim) * (m.f32 ? 4 : 2);
        else if (l.d.mixer == EFM_MIXER_LATENT_ATTENTION) b += n * (l.d.kv_rank + l.d.rot_dims) * (m.f32 ? 4 : 2);
        else if (!l.alone()) b += 2 * (int64_t)l.d.heads * l.d.dim * l.d.dim * 4;
    }
    return b;
}

void decoder_destroy(efm_b200_ctx* c) {
    DecoderModel& m = *c->decoder;
    if (m.side_start != nullptr) cudaEventDestroy(m.side_start);
    if (m.side_end != nullptr) cudaEventDestroy(m.side_end);
    if (m.side != nullptr) cudaStreamDestroy(m.side);
    delete c->decoder;
    c->decoder = nullptr;
}

const ModelOps kDecoderOps = {decoder_set_weight, nullptr, decoder_finalize, decoder_alloc_slot, decoder_prefill_begin, decoder_decode_begin,
                              decoder_prefill_chunk, decoder_step_op, nullptr, decoder_step_bytes, decoder_destroy};

}  // namespace
