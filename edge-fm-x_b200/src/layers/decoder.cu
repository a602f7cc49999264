// Launch sequences of the layered decoders.
//
// Decode (one row), per layer:  [pending output norm + residual add (+ input norm)] + input projections | mixer (norms,
// cache / state update, attention or recurrence) | W_o | [norm + add] + W_up | [PolyNorm] + W_down | [norm + add] + token
// input; what stands in brackets is the prologue of the kernel that follows it: three launches for a layer without a
// feed-forward and token input, two more for a dense feed-forward, one more for the token input.  Latent attention adds
// [query norm] + W_uq; routed experts are [norms + add] + router | [choice] + gate, up, gated unit | [weights] + down, a shared expert
// among them.  Linear attention runs in the launch of the attention beside it, its norm and gate are a prologue of W_o; alone it is one
// launch, norm and gate included.  Input convolutions and the average over depth are part of the prologues, too.
// Many rows: tensor-core GEMMs (bf16 operands) or fp32 FMAs (32-bit mode) between row kernels.
#include "decoder.h"

#include <cmath>
#include <cstdlib>
#include <type_traits>

#include "../operators/decoder_rows.cuh"
#include "../operators/delta_chunk.cuh"
#include "../operators/delta_rule.cuh"
#include "../operators/experts.cuh"
#include "../operators/gemm_tc.cuh"
#include "../operators/latent_attention.cuh"
#include "../operators/linear_attention.cuh"
#include "../operators/linear_attention_tc.cuh"
#include "../operators/token_side.cuh"
#include "../operators/window_attention.cuh"
#include "../operators/window_attention_tc.cuh"
#define EFM_DECLARATIONS_ONLY
#include "../operators/sample.cuh"
#undef EFM_DECLARATIONS_ONLY
#include "gemv_plan.h"
#include "launcher.h"
#include "shared_launch.h"
#include "tensor_map.h"

namespace efm {

// ---- one row -----------------------------------------------------------------------------------------------------
namespace {

// The sublayer output that has not been added to the residual stream yet.
struct Pending {
    const float* y = nullptr;
    const __nv_bfloat16* norm = nullptr;
    int flip = 0;                        // which residual buffer holds the stream
};

// The next launch starts when its predecessor is done instead of overlapping with its tail.  Small grids in front of a product
// that fills the GPU (the router, attention with rotation): launched ahead, they and the blocks of the product that find no
// room beside them end up staggered, which cost 8 to 16 % of a decode step.
struct InOrder {
    Launcher& L;
    bool pdl;
    explicit InOrder(Launcher& l) : L(l), pdl(l.pdl) { L.pdl = false; }
    ~InOrder() { L.pdl = pdl; }
};

template <Epi EPI>
void launch_gemv_ext(efm_b200_ctx& c, Launcher& L, const GemvParams& p) {
    int ks = plan_gemv_ksplit(p.n_items, p.K, c.num_sms);
    if (EPI == Epi::Router)                                            // few rows: one chunk per lane, over as many blocks as that takes
        while (ks * 2 <= kGemvWarps && ks * 32 < p.K / 8 && p.n_items * ks * 2 <= c.num_sms * kGemvWarps) ks *= 2;
    // Logits publishes one maximum per block of a full grid; the others launch no idle blocks
    const int per = kGemvWarps / ks, need = (p.n_items + per - 1) / per;
    const int grid = EPI == Epi::Logits ? c.num_sms : std::min(c.num_sms, need);
    const bool two = p.prologue == kProAddNorm || p.prologue == kProNorm || p.prologue == kProAddTanh || p.prologue == kProMerge;
    const size_t smem = p.conv_w != nullptr ? gemv_conv_smem_bytes(p.K) : two ? gemv_ext_smem_bytes(p.K) : gemv_smem_bytes(p.K);
    constexpr bool kExperts = EPI == Epi::Router || EPI == Epi::ExpertUp || EPI == Epi::ExpertDown;
    const int level = c.decoder->gemv_level();
    auto run = [&](auto kernel) { L.launch(kernel, dim3(grid), dim3(kGemvThreads), smem, p, ks); };
    if constexpr (EPI == Epi::Router) {
        if (level == 4) { run(gemv_kernel<EPI, 4>); return; }          // holds its dependents back itself
        InOrder serial(L);
        run(level == 3 ? gemv_kernel<EPI, 3> : gemv_kernel<EPI, 2>);
    } else if constexpr (kExperts) run(level == 4 ? gemv_kernel<EPI, 4> : level == 3 ? gemv_kernel<EPI, 3> : gemv_kernel<EPI, 2>);
    else if constexpr (EPI == Epi::Store32Bias) run(level == 4 ? gemv_kernel<EPI, 4> : gemv_kernel<EPI, 2>);
    else if constexpr (EPI == Epi::TokenGate) run(gemv_kernel<EPI, 1>);
    else if constexpr (EPI == Epi::Relu2) run(gemv_kernel<EPI, 3>);
    else run(level == 4 ? gemv_kernel<EPI, 4> : level == 3 ? gemv_kernel<EPI, 3> : level == 2 ? gemv_kernel<EPI, 2> : gemv_kernel<EPI, 1>);
}

template <Epi EPI>
void gemv_ext(efm_b200_ctx& c, Launcher& L, const DecLinear& w, GemvParams& p) {
    p.W = w.w;
    p.N = w.N;
    p.K = w.Kp;
    p.n_items = w.Np / 2;
    p.eps = c.decoder->d.norm_eps;
    p.state = c.state;
    p.vocab = c.d.vocab;
    p.bias = w.bias;
    launch_gemv_ext<EPI>(c, L, p);
}

// Input of a product that reads the residual stream: embedding row (first layer) or stream + pending output; with `pre` the
// product reads the norm of it.
void stream_input(efm_b200_ctx& c, GemvParams& p, Pending& pend, bool first, const DecNorm& pre) {
    float* bufs[2] = {c.resid_d, c.resid_d2};
    const bool tanh = c.decoder->tanh_norms();
    p.k_true = c.decoder->W;
    if (tanh) {
        p.norm_w = pre.w;
        p.norm_b = pre.b;
        p.norm_alpha = pre.alpha;
        p.add_mult = c.decoder->d.residual_mult;
    } else {
        p.norm2_w = pre.w;
    }
    if (first) {
        p.prologue = kProEmbed;
        p.embed_table = c.embed;
        p.embed_scale = c.decoder->d.embed_scale;
        p.resid_out = bufs[pend.flip];
        return;
    }
    if (pend.y == nullptr) { p.prologue = kProPlain; p.xf = bufs[pend.flip]; return; }
    p.prologue = tanh ? kProAddTanh : kProAddNorm;
    p.xr = bufs[pend.flip];
    p.addend = pend.y;
    if (!tanh) p.norm_w = pend.norm;
    pend.flip ^= 1;                      // other blocks still read the old row: the new one goes to the other buffer
    p.resid_out = bufs[pend.flip];
    pend.y = nullptr;
}

RotShape rot_shape(const DecoderLayer& l) {
    const int kind = l.d.rot_kind == EFM_ROT_HALF ? kRotHalf : l.d.rot_kind == EFM_ROT_PAIRS ? kRotPairs : kRotNone;
    return RotShape{kind, kind == kRotNone ? 0 : l.d.rot_dims, l.inv_freq, l.d.rot_factor > 0.f ? 0.1f * std::log(l.d.rot_factor) + 1.0f : 1.0f};
}
WindowAttnShape attn_shape(const DecoderModel& m, const DecoderLayer& l) {
    WindowAttnShape s{};
    s.H = l.d.heads; s.G = l.d.kv_heads; s.D = l.d.dim; s.Dv = l.d.vdim; s.Dp = l.Dp; s.Vp = l.Vp;
    s.window = l.d.window; s.keep = l.d.window > 0 ? l.d.keep_first : 0;
    s.bias = l.d.distance_bias; s.scale = l.d.scale; s.eps = m.d.norm_eps;
    s.qk_norm = l.d.qk_norm == EFM_QK_NORM_ROW ? 2 : l.d.qk_norm != EFM_QK_NORM_NONE; s.out_scale = l.parallel() ? l.d.mix_scale : 1.0f;
    s.shift = l.shift;
    s.q_norm = l.q_norm; s.k_norm = l.k_norm; s.temp = l.temp;
    s.rot = rot_shape(l);
    return s;
}
LatentShape latent_shape(const DecoderModel& m, const DecoderLayer& l) {
    LatentShape s{};
    s.H = l.d.heads; s.D = l.d.dim; s.R = l.d.rot_dims; s.Dv = l.d.vdim; s.L = l.d.kv_rank;
    s.Dp = l.Dp; s.Vp = l.Vp; s.Qp = l.Qp; s.Lc = l.Lc; s.Rc = l.Rc;
    s.q_rank = l.d.q_rank; s.window = l.d.window; s.scale = l.d.scale; s.eps = m.d.norm_eps;
    s.rot = rot_shape(l);
    s.q_norm = l.q_norm; s.kv_norm = l.k_norm; s.sink = l.sink;
    s.wk = l.ukv.w; s.wv = l.ukv.w + (size_t)l.d.heads * l.Dp * l.Lc;
    s.gate = l.d.out_gate;
    return s;
}
// column of the gates of an attention layer in its projections
int gate_column(const DecoderLayer& l) { return (l.d.heads + l.d.kv_heads) * l.d.dim + l.d.kv_heads * l.d.vdim; }
LinearShape linear_shape(const DecoderModel& m, const DecoderLayer& l) {
    LinearShape s{};
    s.heads = l.d.linear_heads; s.D = l.d.linear_dim; s.Dv = l.d.linear_vdim; s.Vp = l.lin_vp;
    const int qk = l.linear_qk(), v = l.linear_v();
    s.off_q = l.lin_in; s.off_k = l.lin_in + qk; s.off_v = l.lin_in + 2 * qk; s.off_g = l.lin_in + 2 * qk + v;
    s.ld = l.in.Np; s.powers = l.lin_powers; s.norm = l.mix_norm; s.eps = m.d.norm_eps; s.scale = l.d.linear_scale;
    if (l.alone()) {
        s.scale = 1.0f / std::sqrt((float)s.D);
        s.rot = rot_shape(l);
        if (s.rot.kind == kRotHalf) s.rot.kind = kRotPairs;            // the weights' rows are laid out so
        if (l.channel_decay()) {
            s.rank = l.d.decay_rank; s.off_a = s.off_g + v; s.inv_tau = 1.0f / l.d.linear_tau;
            s.a2 = l.w2.w; s.a2_bias = l.w2.bias; s.ld_a2 = l.w2.Kp;
        }
    }
    return s;
}
int glu_kind(const DecoderLayer& l) { return !l.gated_experts() ? kGluRelu2 : l.d.expert_glu == EFM_GLU_CLAMPED ? kGluClamped : kGluSilu; }
RouteShape route_shape(const DecoderLayer& l) {
    const int shared = l.d.shared_ff <= 0 ? kSharedNone : l.d.shared_gate == EFM_SHARED_PLAIN ? kSharedPlain : kSharedGated;
    return RouteShape{l.d.experts, l.d.expert_top, l.d.expert_groups, l.d.expert_groups_kept, l.d.expert_score == EFM_SCORE_SIGMOID, shared,
                      l.d.expert_scale != 0.f ? l.d.expert_scale : 1.0f};
}
DeltaShape delta_shape(const DecoderModel& m, const DecoderLayer& l) {
    DeltaShape s{};
    s.heads = l.d.heads; s.D = l.d.dim; s.Dp = round_up(l.d.dim, 32); s.rank = l.d.decay_rank; s.ld = l.in.Np;
    s.eps = m.d.norm_eps; s.w0 = l.w0; s.a_bias = l.a_bias; s.norm = l.mix_norm;
    return s;
}

template <typename TC, int VM, bool ROT>
void launch_attn_decode_v(Launcher& L, const WindowDecodeParams<TC>& p, int cluster) {
    const int hb = (p.s.H / p.s.G + wd::kHeads - 1) / wd::kHeads, lin = (p.lin.units + cluster - 1) / cluster;
    L.cluster_x = cluster;
    const bool pdl = L.pdl;
    L.pdl = pdl && (!ROT || lin > 0);                                  // see InOrder; with linear attention the grid is larger
    L.launch(lin > 0 ? window_attention_decode_kernel<TC, VM, ROT, true> : window_attention_decode_kernel<TC, VM, ROT, false>, dim3(cluster, p.s.G * hb + lin),
             dim3(wd::kThreads), sizeof(wd::Smem<VM>), p);
    L.pdl = pdl;
}
template <typename TC>
void launch_attn_decode(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const KvSlot& slot, bool early) {
    DecoderModel& m = *c.decoder;
    WindowDecodeParams<TC> p{};
    p.s = attn_shape(m, l);
    p.qkv = m.d_in;
    p.k_pool = static_cast<TC*>(run.k_pool);
    p.v_pool = static_cast<TC*>(run.v_pool);
    p.pages = m.page_table + (size_t)slot.table * m.d.cache_pages;
    p.max_pages = slot.n_pages;
    p.state = c.state;
    p.out = m.d_mix;
    p.early = early ? 1 : 0;
    if (l.d.out_gate) p.gate = m.d_in + gate_column(l);
    if (l.parallel()) {
        p.lin.s = linear_shape(m, l);
        p.lin.pool = m.state_pool + (size_t)slot.state_slot * m.state_stride + run.state_off;
        p.lin.out = m.d_mix + l.lin_mix;
        p.lin.units = ln::decode_units(p.lin.s);
    }
    // one block per 64 keys of the visible range, up to the cluster width (a power of two)
    int pages = slot.n_pages;
    if (l.d.window > 0) pages = std::min(pages, (l.d.window + p.s.keep + kPageTokens - 1) / kPageTokens);
    int cluster = 1;
    while (cluster < pages && cluster < m.attn_cluster) cluster *= 2;
    const int v = std::max(l.Dp, l.Vp);
    const bool rot = p.s.rot.kind != kRotNone;
    if (v <= 64) rot ? launch_attn_decode_v<TC, 64, true>(L, p, cluster) : launch_attn_decode_v<TC, 64, false>(L, p, cluster);
    else if (v <= 128) rot ? launch_attn_decode_v<TC, 128, true>(L, p, cluster) : launch_attn_decode_v<TC, 128, false>(L, p, cluster);
    else rot ? launch_attn_decode_v<TC, 256, true>(L, p, cluster) : launch_attn_decode_v<TC, 256, false>(L, p, cluster);
}

// ---- latent attention, absorbed form: a decode step, or rows of a pass ---------------------------------------------------
// keys per tile, at most `most`, that the block's shared memory takes next to everything else
int latent_tile(const LatentShape& s, int nh, int splits, int es, int most) {
    int kt = most;
    while (kt > 16 && la::layout(s, nh, splits, es, kt).bytes > 200u * 1024u) kt /= 2;
    return kt;
}
// blocks that share a row: one per 64 visible keys or 64 latent channels, a power of two
int latent_splits(const DecoderLayer& l, int pages, int limit) {
    if (l.d.window > 0) pages = std::min(pages, (l.d.window + kPageTokens - 1) / kPageTokens);
    const int want = std::max(pages, l.Lc / 64);
    int n = 1;
    while (n < want && n < limit) n *= 2;
    return std::min(n, limit);
}
template <typename TC, bool DECODE, typename P>
void launch_latent_kernel(Launcher& L, const DecoderLayer& l, P& p, int splits, int rows) {
    p.kt = latent_tile(p.s, l.la_heads, splits, sizeof(TC), l.la_tile);
    const size_t smem = la::layout(p.s, l.la_heads, splits, sizeof(TC), p.kt).bytes;
    const dim3 grid(splits, (l.d.heads + l.la_heads - 1) / l.la_heads, rows), block(la::kThreads);
    L.cluster_x = splits;
    InOrder serial(L);
    if (l.la_heads == 1) L.launch(latent_attention_kernel<TC, DECODE, 1>, grid, block, smem, p);
    else if (l.la_heads == 2) L.launch(latent_attention_kernel<TC, DECODE, 2>, grid, block, smem, p);
    else L.launch(latent_attention_kernel<TC, DECODE, 4>, grid, block, smem, p);
}
template <typename TC>
void launch_latent_decode(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const KvSlot& slot, bool early) {
    DecoderModel& m = *c.decoder;
    LatentParams<TC, float, float> p{};
    p.s = latent_shape(m, l);
    p.q = m.d_q;
    p.proj = m.d_in;
    p.ld = l.in.Np;
    p.pool = static_cast<TC*>(run.k_pool);
    p.out = m.d_mix;
    p.ld_out = l.mix_wp;
    p.pages = m.page_table + (size_t)slot.table * m.d.cache_pages;
    p.max_pages = slot.n_pages;
    p.early = early ? 1 : 0;
    p.state = c.state;
    launch_latent_kernel<TC, true>(L, l, p, latent_splits(l, slot.n_pages, l.la_cluster), 1);
}
template <typename TA>
void launch_latent_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const RowPlan& plan, const int32_t* list, int n) {
    DecoderModel& m = *c.decoder;
    LatentParams<TA, TA, TA> p{};
    p.s = latent_shape(m, l);
    p.q = static_cast<const TA*>(m.q);
    p.proj = static_cast<const TA*>(m.proj_a);
    p.ld = l.in.Np;
    p.pool = static_cast<TA*>(run.k_pool);
    p.out = static_cast<TA*>(m.mix);
    p.ld_out = l.mix_wp;
    p.plan = plan;
    const int groups = (l.d.heads + l.la_heads - 1) / l.la_heads;
    int splits = latent_splits(l, m.d.cache_pages, l.la_cluster);
    while (splits > 1 && (int64_t)splits * groups * n > 4 * c.num_sms) splits /= 2;       // many rows fill the GPU by themselves
    for (int r0 = 0; r0 < n; r0 += 32768) {                          // grid.z
        p.rows = list != nullptr ? list + r0 : nullptr;
        launch_latent_kernel<TA, false>(L, l, p, splits, std::min(n - r0, 32768));
    }
}

void launch_linear_decode(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const KvSlot& slot, bool early) {
    DecoderModel& m = *c.decoder;
    LinearDecodeParams p{};
    p.s = linear_shape(m, l);
    p.pool = m.state_pool + (size_t)slot.state_slot * m.state_stride + run.state_off;
    p.out = m.d_mix;
    const int slices = (p.s.Dv + ln::kCols - 1) / ln::kCols;
    L.cluster_x = slices;
    L.launch(linear_decode_kernel, dim3(slices, p.s.heads), dim3(256), 0, p, (const float*)m.d_in, c.state, slot.n_pages * kPageTokens, early ? 1 : 0);
}

void launch_delta_decode(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const KvSlot& slot, bool early) {
    DecoderModel& m = *c.decoder;
    DeltaDecodeParams p{};
    p.s = delta_shape(m, l);
    p.proj = m.d_in;
    p.w2 = l.w2.w;
    p.ld_w2 = l.w2.Kp;
    p.pool = m.state_pool + (size_t)slot.state_slot * m.state_stride + run.state_off;
    p.state = c.state;
    p.out = m.d_mix;
    p.early = early ? 1 : 0;
    const int D = l.d.dim, rpt = (D + 512 / D - 1) / (512 / D);
    const dim3 grid(l.d.heads), block(512);
    if (rpt <= 8) L.launch(delta_decode_kernel<8>, grid, block, 0, p);
    else if (rpt <= 32) L.launch(delta_decode_kernel<32>, grid, block, 0, p);
    else L.launch(delta_decode_kernel<0>, grid, block, 0, p);
}

}  // namespace

void decoder_decode_step(efm_b200_ctx& c, KvSlot& slot, Launcher& L, bool sample, bool want_logits) {
    DecoderModel& m = *c.decoder;
    Pending pend;
    auto tap = [&](int layer) {
        if (m.tap == nullptr || m.tap_row0 >= m.tap_rows) return;
        const float* src = pend.flip ? c.resid_d2 : c.resid_d;
        if (L.err == cudaSuccess)
            L.err = cudaMemcpyAsync(m.tap + ((size_t)layer * m.tap_rows + m.tap_row0) * m.Wp, src, (size_t)m.Wp * 4, cudaMemcpyDeviceToDevice, L.stream);
    };
    // the product that starts layer i closes layer i - 1
    auto end_of_layer = [&](GemvParams& p, size_t i) {
        p.hist_out = m.d_hist + i * m.Wp;
        if (i == 0) return;
        p.avg = m.d_avg;
        p.avg_w = m.layers[m.runs[i - 1].layer].dwa + i;
    };
    for (size_t i = 0; i < m.runs.size(); ++i) {
        const DecoderRun& run = m.runs[i];
        const DecoderLayer& l = m.layers[run.layer];
        // From the second layer on a mixer may read the device state and what earlier steps left in its cache before its
        // dependency wait: the mixer one layer up releases its dependents only after its own wait, so nothing of an
        // earlier step is still running.
        const bool early = i > 0;
        float* state = m.state_pool != nullptr ? m.state_pool + (size_t)slot.state_slot * m.state_stride : nullptr;
        auto convolve = [&](GemvParams& p, const __nv_bfloat16* w, size_t off, bool ready) {
            if (w == nullptr) return;
            p.conv_w = w;
            p.conv_ring = state + off;
            p.conv_taps = m.d.conv_taps;
            p.conv_early = ready ? 1 : 0;
        };
        {
            GemvParams p{};
            stream_input(c, p, pend, i == 0, l.pre1);
            if (m.d.depth_average) end_of_layer(p, i);
            convolve(p, l.canon1, run.conv1_off, early);
            p.out_f = m.d_in;
            if (l.in.bias != nullptr) gemv_ext<Epi::Store32Bias>(c, L, l.in, p);
            else gemv_ext<Epi::Store32>(c, L, l.in, p);
            if (i > 0) tap((int)i - 1);
        }
        if (l.attention()) {
            if (m.f32) launch_attn_decode<float>(c, L, l, run, slot, early);
            else launch_attn_decode<__nv_bfloat16>(c, L, l, run, slot, early);
        } else if (l.d.mixer == EFM_MIXER_LATENT_ATTENTION) {
            GemvParams p{};
            p.prologue = kProNorm;
            p.xf = m.d_in;
            p.norm_w = l.q_norm;
            p.k_true = l.d.q_rank;
            p.out_f = m.d_q;
            gemv_ext<Epi::Store32>(c, L, l.uq, p);
            if (m.f32) launch_latent_decode<float>(c, L, l, run, slot, early);
            else launch_latent_decode<__nv_bfloat16>(c, L, l, run, slot, early);
        } else if (l.alone()) {
            launch_linear_decode(c, L, l, run, slot, early);
        } else {
            launch_delta_decode(c, L, l, run, slot, early);
        }
        {
            GemvParams p{};
            p.prologue = kProPlain;
            p.xf = m.d_mix;
            if (m.d.depth_average) {                                   // what is known of the average behind this layer
                p.sum_in = m.d_hist;
                p.sum_w = l.dwa;
                p.sum_out = m.d_avg;
                p.sum_n = (int)i + 1;
                p.sum_k = m.Wp;
            }
            if (l.parallel()) {
                p.prologue = kProMerge;
                p.merge0 = l.lin_mix;
                p.merge_gate = m.d_in + linear_shape(m, l).off_g;
                p.merge_scale = l.d.linear_scale;
                p.norm_w = l.mix_norm;
                p.k_true = l.d.linear_heads * l.d.linear_vdim;
            }
            p.out_f = m.d_y;
            if (l.out.bias != nullptr) gemv_ext<Epi::Store32Bias>(c, L, l.out, p);
            else gemv_ext<Epi::Store32>(c, L, l.out, p);
            pend.y = m.d_y;
            pend.norm = l.post1;
        }
        if (l.moe()) {
            GemvParams r{};
            stream_input(c, r, pend, false, l.pre2);
            convolve(r, l.canon2, run.conv2_off, true);
            r.x_out = m.d_h;
            r.out_f = m.d_route;
            r.route = route_shape(l);
            r.route_id = m.d_route_id;
            r.route_w = m.d_route_w;
            r.route_ticket = m.d_route_ticket;
            gemv_ext<Epi::Router>(c, L, l.router, r);
            GemvParams p{};
            p.prologue = kProPlain;
            p.W = l.expert_in.w;
            p.xf = m.d_h;
            p.K = l.expert_in.Kp;
            const int pair = l.gated_experts() ? 1 : 2;                // channels of an item
            p.ff = (l.d.expert_ff + pair - 1) / pair;
            p.shared_ff = (l.d.shared_ff + pair - 1) / pair;
            p.n_items = l.d.expert_top * p.ff + p.shared_ff;
            p.glu = glu_kind(l);
            p.weight_input = l.d.expert_weight_input;
            p.limit = l.d.expert_limit;
            p.shared_limit = l.d.shared_limit;
            p.shared_ffp = l.sfp;
            p.W2 = l.shared_in.w;
            p.N = 2 * p.n_items;
            p.state = c.state;
            p.route = route_shape(l);
            p.route_id = m.d_route_id;
            p.route_w = m.d_route_w;
            p.ffp = l.ffp;
            p.expert_rows = l.up_rows(l.ffp);
            p.out_f = m.d_act;
            launch_gemv_ext<Epi::ExpertUp>(c, L, p);
            GemvParams q = p;
            q.W = l.expert_out.w;
            q.W2 = l.shared_out.w;
            q.xf = m.d_act;
            q.K = l.d.expert_top * l.ffp + l.sfp;
            q.n_items = m.Wp / 2;
            q.N = m.W;
            q.expert_rows = m.Wp;
            q.out_f = m.d_y;
            launch_gemv_ext<Epi::ExpertDown>(c, L, q);
            pend.y = m.d_y;
            pend.norm = l.post2;
        } else if (l.d.ff > 0) {
            GemvParams p{};
            stream_input(c, p, pend, false, l.pre2);
            convolve(p, l.canon2, run.conv2_off, true);
            p.out_f = m.d_ff;
            const bool poly = l.d.ff_act == EFM_ACT_POLYNORM;
            if (poly) gemv_ext<Epi::Store32>(c, L, l.up, p);
            else gemv_ext<Epi::Relu2>(c, L, l.up, p);
            GemvParams q{};
            q.prologue = poly ? kProPolyNorm : kProPlain;
            q.xf = m.d_ff;
            q.k_true = l.d.ff;
            q.poly = l.act;
            q.out_f = m.d_y;
            gemv_ext<Epi::Store32>(c, L, l.down, q);
            pend.y = m.d_y;
            pend.norm = l.post2;
        }
        if (m.d.side_dim > 0) {
            GemvParams p{};
            stream_input(c, p, pend, false, DecNorm{});
            p.out_f = m.d_gate;
            p.gate_table = m.side_embed;
            p.gate_ld = m.d.side_dim * m.d.num_layers;
            p.gate_off = run.layer * m.d.side_dim;
            if (m.side_cluster > 1 && p.prologue == kProAddNorm) {
                TokenSideParams q{};
                p.W = l.gate.w;
                p.N = l.gate.N;
                p.K = l.gate.Kp;
                p.eps = m.d.norm_eps;
                p.state = c.state;
                p.vocab = c.d.vocab;
                q.p = p;
                q.proj = l.proj.w;
                q.side_p = l.proj.Kp;
                q.n_out = l.proj.Np;
                q.y = m.d_y2;
                L.cluster_x = m.side_cluster;
                L.launch(token_side_kernel, dim3(m.side_cluster), dim3(kGemvThreads), ts::layout(p.K, q.side_p, q.n_out, m.side_cluster).bytes, q);
                pend.y = m.d_y2;
            } else {
                gemv_ext<Epi::TokenGate>(c, L, l.gate, p);
                GemvParams q{};
                q.prologue = kProPlain;
                q.xf = m.d_gate;
                q.out_f = m.d_y;
                gemv_ext<Epi::Store32>(c, L, l.proj, q);
                pend.y = m.d_y;
            }
            pend.norm = l.side_norm;
        }
    }
    if (!want_logits && !sample && m.tap == nullptr) return;
    {
        GemvParams p{};
        stream_input(c, p, pend, false, m.final_norm);
        if (m.d.depth_average) end_of_layer(p, m.runs.size());
        p.logits = c.logits;
        p.logit_scale = m.d.logit_scale;
        p.logit_softcap = m.d.logit_softcap;
        p.part_val = c.part_val;
        p.part_idx = c.part_idx;
        gemv_ext<Epi::Logits>(c, L, m.head, p);
        tap((int)m.runs.size() - 1);
    }
    if (!sample) return;
    SampleParams s{};
    s.logits = c.logits;
    s.vocab = c.d.vocab;
    s.part_val = c.part_val;
    s.part_idx = c.part_idx;
    s.n_part = c.num_sms;
    s.temperature = c.sampling.temperature;
    s.top_p = c.sampling.top_p;
    s.seed = c.sampling.seed;
    s.state = c.state;
    s.tokens_out = c.tokens_out;
    s.max_response = c.d.max_response_tokens;
    s.advance = 1;
    s.wbuf = c.wbuf;
    s.xchg = sample_xchg(c.wbuf, c.d.vocab);
    launch_sample(L, s);
}

// ---- many rows ---------------------------------------------------------------------------------------------------
int decoder_tc_tile_rows() { return wt::BM; }
int decoder_simt_tile_rows() { return wa::QT; }
// bf16 heads of at most 128 key channels whose visible pages fit the kernel's page list
bool decoder_layer_tc(const DecoderModel& m, const DecoderLayer& l) {
    static const bool off = [] { const char* e = std::getenv("EFM_B200_ATTN_TC"); return e != nullptr && e[0] == '0'; }();
    int pages = m.d.cache_pages;
    if (l.d.window > 0) pages = std::min(pages, (l.d.window + wt::BM) / kPageTokens + 2 + (l.d.keep_first + kPageTokens - 1) / kPageTokens);
    return !off && !m.f32 && l.Dp <= 128 && l.Vp <= 256 && l.Rc <= 64 && pages <= wt::kMaxTiles;
}

namespace {

// out[rows, w.Np] = a[rows, w.Kp] . w^T.  bf16 activations run on the tensor cores, fp32 ones in fp32 FMAs.
void linear_f32(efm_b200_ctx& c, Launcher& L, const DecLinear& w, const void* a, float* out, int rows) {
    if (c.decoder->f32) {
        L.launch(gemm_f32_kernel, dim3((w.Np + 63) / 64, (rows + 63) / 64), dim3(256), 0, static_cast<const float*>(a), w.Kp,
                 (const __nv_bfloat16*)w.w, w.Kp, out, w.Np, rows, w.Np, w.Kp, (const __nv_bfloat16*)w.bias, RowGroups{});
        return;
    }
    GemmParams g{static_cast<const __nv_bfloat16*>(a), w.w, w.bias, nullptr, out, rows, w.Np, w.Kp};
    launch_gemm_epi(L, GemmEpi::F32, g, &c.state->error);
}
// the same with the activation type of the pass as output
void linear_act(efm_b200_ctx& c, Launcher& L, const DecLinear& w, const void* a, void* out, int rows) {
    if (c.decoder->f32) { linear_f32(c, L, w, a, static_cast<float*>(out), rows); return; }
    GemmParams g{static_cast<const __nv_bfloat16*>(a), w.w, w.bias, static_cast<__nv_bfloat16*>(out), nullptr, rows, w.Np, w.Kp};
    launch_gemm_epi(L, GemmEpi::Bf16Bias, g, &c.state->error);
}

template <int NC>
void launch_delta_scan(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const RowPlan& plan) {
    DecoderModel& m = *c.decoder;
    const DeltaShape s = delta_shape(m, l);
    const int groups = (s.Dp + ds::kCols - 1) / ds::kCols;
    L.launch(delta_scan_kernel<NC>, dim3(l.d.heads * groups, plan.n_entries), dim3(ds::kThreads), ds::smem_bytes(s.Dp), (const float*)m.pack, m.o, l.mix_wp,
             m.state_pool, m.state_stride, run.state_off, s, plan);
}

// The maps of attention and latent attention differ; what is launched is the same.
template <int DP, int VP, int RP, bool KEEP, bool SIG>
void launch_attention_tc_v(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const WindowAttnShape& s, const WindowTcMaps& maps, const RowPlan& plan,
                           const RowTile* list, int n) {
    const int blocks = n * s.H * ((s.Vp + VP - 1) / VP), first_wave = blocks <= 2 * c.num_sms ? std::min(blocks, c.num_sms) : blocks;
    L.launch(window_attention_tc_kernel<DP, VP, RP, KEEP, SIG>, dim3(blocks), dim3(wt::kThreads), wt::Cfg<DP, VP, RP>::SMEM, maps, static_cast<__nv_bfloat16*>(c.decoder->mix),
             l.mix_wp, s, plan, list, n, first_wave, RP > 0 ? 1 : 0, &c.state->error);
}
template <int RP, bool KEEP = false, bool SIG = false>
void launch_attention_tc_r(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const WindowAttnShape& s, const WindowTcMaps& maps, const RowPlan& plan,
                           const RowTile* list, int n) {
    if (l.Dp <= 64 && l.Vp <= 64) launch_attention_tc_v<64, 64, RP, KEEP, SIG>(c, L, l, s, maps, plan, list, n);
    else if (l.Dp <= 64) launch_attention_tc_v<64, 128, RP, KEEP, SIG>(c, L, l, s, maps, plan, list, n);
    else if (l.Vp <= 64) launch_attention_tc_v<128, 64, RP, KEEP, SIG>(c, L, l, s, maps, plan, list, n);
    else launch_attention_tc_v<128, 128, RP, KEEP, SIG>(c, L, l, s, maps, plan, list, n);
}
// [rows][heads][channels] with strides in elements
bool head_map(CUtensorMap* map, const void* base, int channels, int heads, int rows, int head_stride, int row_stride, int box_rows) {
    const uint64_t d[3] = {(uint64_t)channels, (uint64_t)heads, (uint64_t)rows}, st[2] = {(uint64_t)head_stride * 2, (uint64_t)row_stride * 2};
    const uint32_t b[3] = {64, 1, (uint32_t)box_rows};
    return make_map_nd(map, base, 3, d, st, b);
}
void launch_attention_tc(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const WindowAttnShape& s, const RowPlan& plan,
                         const RowTile* list, int n) {
    if (n <= 0) return;
    DecoderModel& m = *c.decoder;
    WindowTcMaps maps;
    const int rows = m.d.cache_pages * kPageTokens;
    if (!head_map(&maps.q, m.q, s.Dp, s.H, plan.rows, s.Dp, s.H * s.Dp, wt::BM) || !head_map(&maps.k, run.k_pool, s.Dp, s.G, rows, s.Dp, s.G * s.Dp, wt::BN) ||
        !head_map(&maps.v, run.v_pool, s.Vp, s.G, rows, s.Vp, s.G * s.Vp, wt::BN)) {
        if (L.err == cudaSuccess) L.err = cudaErrorInvalidValue;
        return;
    }
    maps.qr = maps.q;
    maps.kr = maps.k;
    if (s.shift != nullptr) launch_attention_tc_r<0, false, true>(c, L, l, s, maps, plan, list, n);
    else if (s.keep > 0) launch_attention_tc_r<0, true>(c, L, l, s, maps, plan, list, n);
    else launch_attention_tc_r<0>(c, L, l, s, maps, plan, list, n);
}
// Long entries of a latent layer: visible cache rows into the workspace, keys and values of all heads by one product,
// attention over those.
void launch_latent_tc(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const RowPlan& plan, const RowTiles& tiles,
                      const RowTile* list, int n) {
    DecoderModel& m = *c.decoder;
    const LatentShape z = latent_shape(m, l);
    const int LR = z.Lc + z.Rc, n_ws = tiles.n_ws * kPageTokens, ld = l.ukv.Np;
    if (tiles.n_gather > 0)
        L.launch(latent_gather_rows_kernel<__nv_bfloat16>, dim3(tiles.n_gather, 4), dim3(256), 0, static_cast<const __nv_bfloat16*>(run.k_pool), m.ws_c, LR, plan,
                 tiles.ws_pages, tiles.ws_page0);
    GemmParams g{m.ws_c, l.ukv.w, nullptr, m.ws_kv, nullptr, n_ws, l.ukv.Np, l.ukv.Kp};
    g.lda = LR;
    launch_gemm_epi(L, GemmEpi::Bf16Bias, g, &c.state->error);
    WindowAttnShape s{};
    s.H = s.G = z.H; s.D = z.D; s.Dv = z.Dv; s.Dp = z.Dp; s.Vp = z.Vp;
    s.window = z.window; s.scale = z.scale; s.eps = z.eps; s.sink = z.sink; s.out_scale = 1.0f;
    if (z.gate) { s.gate = static_cast<const __nv_bfloat16*>(m.proj_a) + z.off_gate(); s.gate_ld = l.in.Np; s.gate_heads = z.gate == EFM_GATE_HEADS; }
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(m.q);
    WindowTcMaps maps;
    const int qh = z.Dp + z.Rc;
    if (!head_map(&maps.q, q, z.Dp, z.H, plan.rows, qh, z.q_ld(), wt::BM) || !head_map(&maps.qr, q + z.Dp, z.Rc, z.H, plan.rows, qh, z.q_ld(), wt::BM) ||
        !head_map(&maps.k, m.ws_kv, z.Dp, z.H, n_ws, z.Dp, ld, wt::BN) || !head_map(&maps.v, m.ws_kv + (size_t)z.H * z.Dp, z.Vp, z.H, n_ws, z.Vp, ld, wt::BN) ||
        !head_map(&maps.kr, m.ws_c + z.Lc, z.Rc, 1, n_ws, LR, LR, wt::BN)) {
        if (L.err == cudaSuccess) L.err = cudaErrorInvalidValue;
        return;
    }
    launch_attention_tc_r<64>(c, L, l, s, maps, plan, list, n);
}

// Chunked recurrence: every chunk's state-independent part at once, then the chunks in sequence.
template <int DP>
void launch_delta_chunks(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const RowPlan& plan) {
    DecoderModel& m = *c.decoder;
    const DeltaShape s = delta_shape(m, l);
    const int chunks = plan.n_entries == 1 ? (plan.rows + dc::C - 1) / dc::C : plan.rows / dc::C + plan.n_entries;     // at most
    L.launch(delta_prepare_kernel<DP>, dim3(chunks, l.d.heads), dim3(dc::kThreads), sizeof(dc::PrepSmem<DP>), (const float*)m.proj_f, (const float*)m.decay,
             l.w2.Np, m.pack, s, plan);
    L.launch(delta_chunk_scan_kernel<DP>, dim3(l.d.heads * (DP / dc::kCols), plan.n_entries), dim3(dc::kScanThreads), sizeof(dc::ScanSmem<DP>), (const float*)m.pack,
             m.o, l.mix_wp, m.state_pool, m.state_stride, run.state_off, s, plan);
}

// Linear attention of rows whose projections are in proj_a, into its columns of the mixer output.
template <typename TA>
void linear_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const RowPlan& plan) {
    DecoderModel& m = *c.decoder;
    const LinearShape s = linear_shape(m, l);
    const TA* proj = static_cast<const TA*>(m.proj_a);
    const int ld_o = round_up(s.width(), 8);
    bool tensor_cores = false;
    if constexpr (std::is_same<TA, __nv_bfloat16>::value) tensor_cores = s.D <= 128 && plan.rows >= kLinearChunk;      // short passes: CUDA cores
    const int chunks = max_chunks(plan, tensor_cores ? kLinearChunkTc : kLinearChunk);
    const int ld_sums = l.w2.Np;
    auto chain = [&](auto kernel) {
        L.launch(kernel, dim3((unsigned)((s.heads * s.head_floats() + 1023) / 1024), plan.n_entries), dim3(256), 0, m.lin_ws, m.state_pool, m.state_stride, run.state_off,
                 s, plan, (const float*)m.decay, ld_sums);
    };
    auto output = [&] {
        if (l.alone()) {
            L.launch(linear_head_output_rows_kernel<TA>, dim3((plan.rows * s.heads + 7) / 8), dim3(256), 0, (const float*)m.o, ld_o, proj, static_cast<TA*>(m.mix), l.mix_wp,
                     plan.rows, s);
            return;
        }
        L.launch(linear_output_rows_kernel<TA>, dim3(plan.rows), dim3(256), 0, (const float*)m.o, ld_o, proj, static_cast<TA*>(m.mix) + l.lin_mix, l.mix_wp,
                 l.mix_wp - l.lin_mix, s);
    };
    auto decay_product = [&](auto rank) {
        constexpr int RANK = decltype(rank)::value;
        L.launch(linear_decay_product_sums_kernel<kLinearChunkTc, RANK>, dim3((ld_sums + 63) / 64, chunks), dim3(512), 0, reinterpret_cast<const __nv_bfloat16*>(proj),
                 m.decay, ld_sums, s, plan);
    };
    if (s.rank > 0 && s.rank <= 32 && tensor_cores) {
        if (s.rank <= 16) decay_product(std::integral_constant<int, 16>{});
        else decay_product(std::integral_constant<int, 32>{});
    } else if (s.rank > 0) {                                           // W_a2 W_a1 x + b, then the decays it stands for
        if (m.f32) {
            L.launch(gemm_f32_kernel, dim3((l.w2.Np + 63) / 64, (plan.rows + 63) / 64), dim3(256), 0, reinterpret_cast<const float*>(proj) + s.off_a, s.ld,
                     (const __nv_bfloat16*)l.w2.w, l.w2.Kp, m.decay, l.w2.Np, plan.rows, l.w2.Np, l.w2.Kp, (const __nv_bfloat16*)l.w2.bias, RowGroups{});
        } else {
            GemmParams g{reinterpret_cast<const __nv_bfloat16*>(proj) + s.off_a, l.w2.w, l.w2.bias, nullptr, m.decay, plan.rows, l.w2.Np, l.w2.Kp};
            g.lda = s.ld;
            launch_gemm_epi(L, GemmEpi::F32, g, &c.state->error);
        }
        if (tensor_cores)
            L.launch(linear_decay_sums_kernel<kLinearChunkTc>, dim3((ld_sums + 127) / 128, chunks), dim3(128), 0, m.decay, ld_sums, s.inv_tau, plan);
        else
            L.launch(linear_decay_rows_kernel, dim3((ld_sums + 255) / 256, plan.rows), dim3(256), 0, m.decay, ld_sums, s.inv_tau);
    }
    if constexpr (std::is_same<TA, __nv_bfloat16>::value) {
        if (tensor_cores) {
            auto products = [&](auto vp) {
                constexpr int VP = decltype(vp)::value;
                using Cf = lt::Cfg<VP>;
                const dim3 grid(chunks, s.heads, (s.Dv + VP - 1) / VP), block(lt::kThreads);
                const float *sums = m.decay, *ws = m.lin_ws;
                const bool whole = l.alone() && s.Dv <= VP;             // a block has all of a head's channels: norm and gate included
                __nv_bfloat16* out = static_cast<__nv_bfloat16*>(m.mix);
                if (s.rank > 0) {
                    L.launch(linear_chunk_tc_kernel<VP, true>, grid, block, Cf::CHUNK_SMEM, proj, m.lin_ws, s, plan, &c.state->error, sums, ld_sums);
                    chain(linear_chain_rows_kernel<kLinearChunkTc, true>);
                    L.launch(whole ? linear_attend_ch_tc_kernel<VP, true> : linear_attend_ch_tc_kernel<VP, false>, grid, dim3(lt::kAttendThreads), Cf::ATTEND_CH_SMEM, proj, ws, sums, ld_sums,
                             m.o, ld_o, out, l.mix_wp, s, plan, &c.state->error);
                } else {
                    L.launch(linear_chunk_tc_kernel<VP>, grid, block, Cf::CHUNK_SMEM, proj, m.lin_ws, s, plan, &c.state->error, sums, 0);
                    chain(linear_chain_rows_kernel<kLinearChunkTc>);
                    L.launch(whole ? linear_attend_tc_kernel<VP, true> : linear_attend_tc_kernel<VP>, grid, dim3(lt::kAttendThreads), Cf::ATTEND_SMEM, proj, ws, m.o, ld_o, s, plan,
                             &c.state->error, out, l.mix_wp);
                }
                if (!whole) output();
            };
            if (s.Dv <= 64) products(std::integral_constant<int, 64>{});
            else products(std::integral_constant<int, 128>{});
            return;
        }
    }
    if (s.rank > 0) {                                                  // token by token
        auto scan = [&](auto nc) {
            constexpr int NC = decltype(nc)::value;
            L.launch(linear_scan_rows_kernel<TA, NC>, dim3(s.heads * ((s.Dv + lc::kCols - 1) / lc::kCols), plan.n_entries), dim3(lc::kThreads), lc::smem_bytes(NC * 32), proj,
                     (const float*)m.decay, ld_sums, m.o, ld_o, m.state_pool, m.state_stride, run.state_off, s, plan);
        };
        if (s.D <= 32) scan(std::integral_constant<int, 1>{});
        else if (s.D <= 64) scan(std::integral_constant<int, 2>{});
        else if (s.D <= 128) scan(std::integral_constant<int, 4>{});
        else scan(std::integral_constant<int, 8>{});
        output();
        return;
    }
    auto chunk = [&](auto rm, auto rn) {
        constexpr int RM = decltype(rm)::value, RN = decltype(rn)::value;
        L.launch(linear_chunk_rows_kernel<TA, RM, RN>, dim3(chunks, s.heads, ((s.D + 16 * RM - 1) / (16 * RM)) * ((s.Vp + 16 * RN - 1) / (16 * RN))), dim3(ln::kThreads),
                 ln::chunk_smem_bytes(RM, RN), proj, m.lin_ws, s, plan);
    };
    auto attend = [&](auto rn) {
        constexpr int RN = decltype(rn)::value;
        L.launch(linear_attend_rows_kernel<TA, RN>, dim3(chunks, s.heads, (s.Dv + 16 * RN - 1) / (16 * RN)), dim3(ln::kThreads), ln::attend_smem_bytes(s.D, RN), proj,
                 (const float*)m.lin_ws, m.o, ld_o, s, plan);
    };
    const std::integral_constant<int, 4> k4{};
    const std::integral_constant<int, 8> k8{};
    if (s.D <= 64) { if (s.Dv <= 64) chunk(k4, k4); else chunk(k4, k8); }
    else if (s.Dv <= 64) chunk(k8, k4);
    else chunk(k8, k8);
    chain(linear_chain_rows_kernel<kLinearChunk, false>);
    if (s.Dv <= 64) attend(k4); else attend(k8);
    output();
}

// A layer of linear attention alone.
template <typename TA>
void linear_mixer_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const void* x, const RowPlan& plan) {
    DecoderModel& m = *c.decoder;
    const LinearShape s = linear_shape(m, l);
    if (s.rot.kind == kRotNone) {
        linear_act(c, L, l.in, x, m.proj_a, plan.rows);
    } else if (l.rot_table >= 0) {                                     // turned in the product's epilogue
        GemmParams g{static_cast<const __nv_bfloat16*>(x), l.in.w, l.in.bias, static_cast<__nv_bfloat16*>(m.proj_a), nullptr, plan.rows, l.in.Np, l.in.Kp};
        g.rot = m.rot_tables[l.rot_table].cs;
        g.rot_cols = s.off_v;
        g.rot_head = s.D;
        g.rot_dims = s.rot.dims;
        launch_gemm_epi(L, GemmEpi::Bf16Rotate, g, &c.state->error);
    } else {                                                           // turned in fp32, rounded once
        float* proj = std::is_same<TA, float>::value ? static_cast<float*>(m.proj_a) : m.proj_f;
        linear_f32(c, L, l.in, x, proj, plan.rows);
        L.launch(linear_rotate_rows_kernel<TA>, dim3(plan.rows), dim3(256), 0, (const float*)proj, static_cast<TA*>(m.proj_a), s, plan);
    }
    linear_rows<TA>(c, L, l, run, plan);
}

// TA: activation and cache type of the pass
template <typename TA>
void attention_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const void* x, const RowPlan& plan, const RowTiles& tiles) {
    DecoderModel& m = *c.decoder;
    WindowAttnShape s = attn_shape(m, l);
    if (l.d.out_gate) { s.gate = static_cast<const TA*>(m.proj_a) + gate_column(l); s.gate_ld = l.in.Np; s.gate_heads = 1; }
    if (l.parallel()) {
        const LinearShape z = linear_shape(m, l);
        if constexpr (std::is_same<TA, float>::value) {
            linear_f32(c, L, l.in, x, static_cast<float*>(m.proj_a), plan.rows);
            L.launch(silu_columns_kernel, dim3((z.off_g - z.off_q + 1023) / 1024, plan.rows), dim3(256), 0, static_cast<float*>(m.proj_a), l.in.Np, z.off_q, z.off_g);
        } else {
            GemmParams g{static_cast<const __nv_bfloat16*>(x), l.in.w, l.in.bias, static_cast<__nv_bfloat16*>(m.proj_a), nullptr, plan.rows, l.in.Np, l.in.Kp};
            g.silu0 = z.off_q;
            g.silu1 = z.off_g;
            launch_gemm_epi(L, GemmEpi::Bf16Silu, g, &c.state->error);
        }
        linear_rows<TA>(c, L, l, run, plan);
    } else {
        linear_act(c, L, l.in, x, m.proj_a, plan.rows);
    }
    TA* kp = static_cast<TA*>(run.k_pool);
    TA* vp = static_cast<TA*>(run.v_pool);
    int lanes = 8;                                                  // 8 channels each: at most 256 (padded) channels a head
    while (lanes * 8 < std::max(s.Dp, s.Vp)) lanes *= 2;
    L.launch(s.rot.kind != kRotNone ? qk_scatter_rows_kernel<TA, TA, TA, true> : qk_scatter_rows_kernel<TA, TA, TA, false>, dim3(plan.rows), dim3(256), 0,
             static_cast<const TA*>(m.proj_a), l.in.Np, static_cast<TA*>(m.q), kp, vp, s, plan, lanes);
    auto cuda_cores = [&](const RowTile* list, int n) {
        if (n > 0)
            L.launch(window_attention_rows_kernel<TA, TA, TA>, dim3(n, s.H), dim3(256), wa::rows_smem_bytes(s.Dp, s.Vp), static_cast<const TA*>(m.q),
                     (const TA*)kp, (const TA*)vp, static_cast<TA*>(m.mix), l.mix_wp, s, plan, list);
    };
    if constexpr (std::is_same<TA, __nv_bfloat16>::value) {
        if (decoder_layer_tc(m, l)) {
            if (tiles.listed) {
                launch_attention_tc(c, L, l, run, s, plan, tiles.tc, tiles.n_tc);
                cuda_cores(tiles.simt, tiles.n_simt);
                return;
            }
            if (plan.rows >= kTcMinRows) {
                launch_attention_tc(c, L, l, run, s, plan, nullptr, (plan.rows + wt::BM - 1) / wt::BM);
                return;
            }
        }
    }
    cuda_cores(tiles.all, tiles.listed ? tiles.n_all : (plan.rows + wa::QT - 1) / wa::QT);
}

template <typename TA>
void latent_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const void* x, const RowPlan& plan, const RowTiles& tiles) {
    DecoderModel& m = *c.decoder;
    const LatentShape s = latent_shape(m, l);
    const int T = plan.rows;
    linear_act(c, L, l.in, x, m.proj_a, T);
    TA* ws = nullptr;
    if constexpr (std::is_same<TA, __nv_bfloat16>::value) {
        if (decoder_layer_tc(m, l)) ws = m.ws_c;
    }
    L.launch(latent_rows_kernel<TA>, dim3((T + kLatentRowsPerBlock - 1) / kLatentRowsPerBlock), dim3(32 * kLatentRowsPerBlock), 0, static_cast<const TA*>(m.proj_a),
             l.in.Np, static_cast<TA*>(m.cq), static_cast<TA*>(run.k_pool), ws, kTcMinRows, s, plan);
    linear_act(c, L, l.uq, m.cq, m.q, T);
    L.launch(latent_rotate_rows_kernel<TA>, dim3(T), dim3(256), 0, static_cast<TA*>(m.q), s, plan);
    if constexpr (std::is_same<TA, __nv_bfloat16>::value) {
        if (decoder_layer_tc(m, l)) {
            if (tiles.listed) {
                if (tiles.n_tc > 0) launch_latent_tc(c, L, l, run, plan, tiles, tiles.tc, tiles.n_tc);
                if (tiles.n_short > 0) launch_latent_rows<TA>(c, L, l, run, plan, tiles.short_rows, tiles.n_short);
                return;
            }
            if (T >= kTcMinRows) {
                launch_latent_tc(c, L, l, run, plan, tiles, nullptr, (T + wt::BM - 1) / wt::BM);
                return;
            }
        }
    }
    launch_latent_rows<TA>(c, L, l, run, plan, nullptr, T);
}

GemmEpi expert_epi(const DecoderLayer& l) {
    return !l.gated_experts() ? GemmEpi::Bf16Relu2 : l.d.expert_glu == EFM_GLU_CLAMPED ? GemmEpi::ClampGlu : GemmEpi::SwiGlu;
}
// Routed experts of all rows: choice, rows sorted by expert, two grouped products.  The outputs stay sorted (m.ex_y); the norm
// that follows sums them (SumOf).
template <typename TA>
SumOf<TA> expert_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const void* h, int T) {
    DecoderModel& m = *c.decoder;
    const RouteShape r = route_shape(l);
    // the shared expert on a stream of its own, products unsplit: the split-K workspace belongs to the other stream
    Launcher S = L;
    S.stream = m.side;
    S.gemm_ws = nullptr;
    auto order = [&](cudaError_t e) { if (L.err == cudaSuccess) L.err = e; };
    if (l.d.shared_ff > 0) order(cudaEventRecord(m.side_start, L.stream));
    linear_f32(c, L, l.router, h, m.route_logits, T);
    if (l.d.shared_ff > 0) {
        order(cudaStreamWaitEvent(m.side, m.side_start, 0));
        if constexpr (std::is_same<TA, float>::value) {
            linear_f32(c, S, l.shared_in, h, m.sh_gu, T);
            S.launch(glu_rows_kernel, dim3((T + kExpertTile - 1) / kExpertTile), dim3(256), 0, (const float*)m.sh_gu, static_cast<float*>(m.sh_act), T, l.sfp,
                     (const int32_t*)nullptr, glu_kind(l), l.d.shared_limit);
            linear_f32(c, S, l.shared_out, m.sh_act, static_cast<float*>(m.sh_y), T);
        } else {
            GemmParams g{static_cast<const __nv_bfloat16*>(h), l.shared_in.w, nullptr, static_cast<__nv_bfloat16*>(m.sh_act), nullptr, T, l.shared_in.Np, l.shared_in.Kp};
            g.limit = l.d.shared_limit;
            launch_gemm_epi(S, expert_epi(l), g, &c.state->error);
            linear_act(c, S, l.shared_out, m.sh_act, m.sh_y, T);
        }
        order(S.err);
        order(cudaEventRecord(m.side_end, m.side));
    }
    L.launch(expert_route_rows_kernel, dim3((T + 7) / 8), dim3(256), 0, (const float*)m.route_logits, l.router.Np, T, r, m.ex);
    L.launch(l.d.expert_weight_input ? expert_gather_rows_kernel<TA, true> : expert_gather_rows_kernel<TA, false>, dim3(T), dim3(128), 0, static_cast<const TA*>(h), static_cast<TA*>(m.ex_in), m.Wp, r, m.ex);
    // tiles in use at most: every row tile but the last of an expert is full
    const int64_t picks = (int64_t)T * r.top;
    const int max_rows = (int)std::min<int64_t>(m.ex_rows, (picks / kExpertTile + std::min<int64_t>(picks, r.experts)) * kExpertTile);
    if constexpr (std::is_same<TA, float>::value) {
        auto product = [&](const DecLinear& w, int n, const float* a, float* out) {
            L.launch(gemm_f32_kernel, dim3((n + 63) / 64, (max_rows + 63) / 64), dim3(256), 0, a, w.Kp, (const __nv_bfloat16*)w.w, w.Kp, out, n, max_rows, n, w.Kp,
                     (const __nv_bfloat16*)nullptr, RowGroups{m.ex.tile, m.ex.n_tiles, n});
        };
        product(l.expert_in, l.up_rows(l.ffp), static_cast<const float*>(m.ex_in), m.ex_gu);
        L.launch(glu_rows_kernel, dim3(max_rows / kExpertTile), dim3(256), 0, (const float*)m.ex_gu, static_cast<float*>(m.ex_act), max_rows, l.ffp,
                 (const int32_t*)m.ex.n_tiles, glu_kind(l), l.d.expert_limit);
        product(l.expert_out, m.Wp, static_cast<const float*>(m.ex_act), static_cast<float*>(m.ex_y));
    } else {
        auto product = [&](const DecLinear& w, int n, GemmEpi epi, const void* a, void* out) {
            GemmParams g{static_cast<const __nv_bfloat16*>(a), w.w, nullptr, static_cast<__nv_bfloat16*>(out), nullptr, max_rows, n, w.Kp};
            g.group_tile = reinterpret_cast<const GroupTile*>(m.ex.tile);
            g.group_tiles = m.ex.n_tiles;
            g.group_rows = n;
            g.group_all = r.experts * n;
            g.limit = l.d.expert_limit;
            launch_gemm_epi(L, epi, g, &c.state->error);
        };
        product(l.expert_in, l.up_rows(l.ffp), expert_epi(l), m.ex_in, m.ex_act);
        product(l.expert_out, m.Wp, GemmEpi::Bf16Bias, m.ex_act, m.ex_y);
    }
    if (l.d.shared_ff > 0) order(cudaStreamWaitEvent(L.stream, m.side_end, 0));
    return SumOf<TA>{static_cast<const TA*>(m.ex_y), m.ex.place, m.ex.weight, r.top, m.ex.count, r.experts, l.d.expert_weight_input,
                     l.d.shared_ff > 0 ? static_cast<const TA*>(m.sh_y) : nullptr, m.ex.shared};
}

template <typename TA>
void delta_rows(efm_b200_ctx& c, Launcher& L, const DecoderLayer& l, const DecoderRun& run, const void* x, const RowPlan& plan) {
    DecoderModel& m = *c.decoder;
    const DeltaShape s = delta_shape(m, l);
    linear_f32(c, L, l.in, x, m.proj_f, plan.rows);
    L.launch(delta_tanh_rows_kernel, dim3(plan.rows), dim3(128), 0, (const float*)m.proj_f, m.tanh_w, l.w2.Kp, s);
    L.launch(gemm_f32_kernel, dim3((l.w2.Np + 63) / 64, (plan.rows + 63) / 64), dim3(256), 0, (const float*)m.tanh_w, l.w2.Kp, (const __nv_bfloat16*)l.w2.w,
             l.w2.Kp, m.decay, l.w2.Np, plan.rows, l.w2.Np, l.w2.Kp, (const __nv_bfloat16*)nullptr, RowGroups{});
    const bool chunked = plan.rows >= dc::C && s.Dp <= 128;         // short passes and larger heads: token by token
    if (chunked) {
        switch (s.Dp / 32) {
            case 1: launch_delta_chunks<32>(c, L, l, run, plan); break;
            case 2: launch_delta_chunks<64>(c, L, l, run, plan); break;
            case 3: launch_delta_chunks<96>(c, L, l, run, plan); break;
            default: launch_delta_chunks<128>(c, L, l, run, plan); break;
        }
    } else {
        L.launch(delta_inputs_rows_kernel, dim3(plan.rows), dim3(256), 0, (const float*)m.proj_f, (const float*)m.decay, l.w2.Np, m.pack, s);
        switch (s.Dp / 32) {
            case 1: launch_delta_scan<1>(c, L, l, run, plan); break;
            case 2: launch_delta_scan<2>(c, L, l, run, plan); break;
            case 3: launch_delta_scan<3>(c, L, l, run, plan); break;
            case 4: launch_delta_scan<4>(c, L, l, run, plan); break;
            case 5: launch_delta_scan<5>(c, L, l, run, plan); break;
            case 6: launch_delta_scan<6>(c, L, l, run, plan); break;
            case 7: launch_delta_scan<7>(c, L, l, run, plan); break;
            default: launch_delta_scan<8>(c, L, l, run, plan); break;
        }
    }
    int lanes = 1;
    while (lanes * 4 < s.D && lanes < 32) lanes *= 2;
    L.launch(delta_output_rows_kernel<TA>, dim3(plan.rows), dim3(256), 0, (const float*)m.o, l.mix_wp, (const float*)m.proj_f, static_cast<TA*>(m.mix), l.mix_wp,
             s, lanes);
}

template <typename TA>
void rows_pass(efm_b200_ctx& c, const RowPlan& plan, const int32_t* ids, const RowTiles& tiles, Launcher& L) {
    DecoderModel& m = *c.decoder;
    const int T = plan.rows;
    TA* xa = static_cast<TA*>(m.xa);                            // null: 32-bit mode without input norms reads the stream itself
    const void* xin = xa != nullptr ? (const void*)xa : c.resid;
    // the stream takes a sublayer's normed output; xa becomes the next sublayer's input
    // with an average over depth the embedding stays in its row of the history, behind a layer's last sublayer (avg) its result goes there
    const float* stream = c.resid;
    const size_t hist_rows = (size_t)m.d.max_step_tokens * m.Wp;
    auto add_norm = [&](const float* y, const __nv_bfloat16* w, const DecNorm& norm, const SumOf<TA>& sum = SumOf<TA>{}, const DepthAverage* avg = nullptr) {
        const bool experts = sum.place != nullptr;
        const __nv_bfloat16* pre = norm.w;
        if (m.tanh_norms()) {
            L.launch(experts ? add_tanh_rows_kernel<TA, true> : add_tanh_rows_kernel<TA, false>, dim3((m.Wp + 1023) / 1024, T), dim3(256), 0, c.resid, y,
                     m.d.residual_mult, xa, norm.w, norm.b, norm.alpha, m.Wp, sum);
            return;
        }
        if (avg != nullptr) {
            L.launch(experts ? add_norm_rows_kernel<TA, false, true, true> : add_norm_rows_kernel<TA, false, false, true>, dim3(T), dim3(256), 0, c.resid, stream, y, w,
                     (TA*)nullptr, (const __nv_bfloat16*)nullptr, m.W, m.Wp, m.d.norm_eps, sum, *avg);
            stream = c.resid;
            return;
        }
        L.launch(pre != nullptr ? (experts ? add_norm_rows_kernel<TA, true, true> : add_norm_rows_kernel<TA, true, false>)
                                : (experts ? add_norm_rows_kernel<TA, false, true> : add_norm_rows_kernel<TA, false, false>),
                 dim3(T), dim3(256), 0, c.resid, stream, y, w, m.d.conv_taps > 0 ? (TA*)nullptr : xa, pre, m.W, m.Wp, m.d.norm_eps, sum, DepthAverage{});
        stream = c.resid;
    };
    auto convolve = [&](const __nv_bfloat16* w, size_t off) {
        if (w == nullptr) return;
        auto run = [&](auto kernel) {
            const int rows = m.d.conv_taps >= 2 && m.d.conv_taps <= 4 ? kConvShortRows : kConvRows;
            L.launch(kernel, dim3((m.Wp / 4 + 127) / 128, max_chunks(plan, rows)), dim3(128), 0, stream, w, xa, m.Wp, m.state_pool, m.state_stride, off, m.d.conv_taps, plan);
        };
        switch (m.d.conv_taps) {
            case 2: run(input_conv_rows_kernel<TA, 2, kConvShortRows>); break;
            case 3: run(input_conv_rows_kernel<TA, 3, kConvShortRows>); break;
            case 4: run(input_conv_rows_kernel<TA, 4, kConvShortRows>); break;
            default: run(input_conv_rows_kernel<TA, 0, kConvRows>); break;
        }
    };
    // a sublayer's last product and what follows it; elementwise norms are part of the product
    auto sublayer_out = [&](const DecLinear& w, const void* a, const __nv_bfloat16* post, const DecNorm& norm, const DepthAverage* avg = nullptr) {
        if (m.tanh_norms() && !m.f32) {
            GemmParams g{static_cast<const __nv_bfloat16*>(a), w.w, nullptr, norm.w != nullptr ? static_cast<__nv_bfloat16*>(m.xa) : nullptr, c.resid, T, w.Np, w.Kp};
            g.mult = m.d.residual_mult;
            g.norm_w = norm.w; g.norm_b = norm.b; g.norm_alpha = norm.alpha;
            launch_gemm_epi(L, GemmEpi::ResidualTanh, g, &c.state->error);
            return;
        }
        linear_f32(c, L, w, a, m.y, T);
        add_norm(m.y, post, norm, SumOf<TA>{}, avg);
    };
    for (const DecoderModel::RotTable& t : m.rot_tables)
        L.launch(rot_rows_kernel, dim3((t.dims / 2 + 127) / 128, T), dim3(128), 0, t.cs, rot_shape(m.layers[t.layer]), plan);
    float* first = m.d.depth_average ? m.hist : c.resid;
    launch_embed_rows(L, ids, c.embed, nullptr, first, T, c.d.vocab, m.Wp, -1, 0, m.d.embed_scale);
    stream = first;
    if (xa != nullptr && m.d.conv_taps == 0) add_norm(nullptr, nullptr, m.layers[m.runs[0].layer].pre1);
    for (size_t i = 0; i < m.runs.size(); ++i) {
        const DecoderRun& run = m.runs[i];
        const DecoderLayer& l = m.layers[run.layer];
        const DecNorm next = i + 1 < m.runs.size() ? m.layers[m.runs[i + 1].layer].pre1 : DecNorm{};
        const DepthAverage depth{m.hist, hist_rows, l.dwa, (int)i + 1}, *avg = m.d.depth_average ? &depth : nullptr;
        convolve(l.canon1, run.conv1_off);
        if (l.attention()) attention_rows<TA>(c, L, l, run, xin, plan, tiles);
        else if (l.d.mixer == EFM_MIXER_LATENT_ATTENTION) latent_rows<TA>(c, L, l, run, xin, plan, tiles);
        else if (l.alone()) linear_mixer_rows<TA>(c, L, l, run, xin, plan);
        else delta_rows<TA>(c, L, l, run, xin, plan);
        sublayer_out(l.out, m.mix, l.post1, l.mlp() ? l.pre2 : next, l.mlp() ? nullptr : avg);
        if (l.mlp()) convolve(l.canon2, run.conv2_off);
        if (l.moe()) {
            add_norm(nullptr, l.post2, next, expert_rows<TA>(c, L, l, xin, T), avg);
        } else if (l.d.ff > 0) {
            const bool poly = l.d.ff_act == EFM_ACT_POLYNORM;
            if (poly) {
                linear_act(c, L, l.up, xin, m.ff, T);
                L.launch(poly_norm_rows_kernel<TA>, dim3(T), dim3(256), 0, static_cast<const TA*>(m.ff), static_cast<TA*>(m.ff2), (const __nv_bfloat16*)l.act, l.d.ff,
                         l.down.Kp, m.d.norm_eps);
            } else if (m.f32) {
                linear_f32(c, L, l.up, xin, static_cast<float*>(m.ff), T);
                const size_t n = (size_t)T * l.up.Np;
                L.launch(relu2_kernel, dim3((unsigned)((n + 1023) / 1024)), dim3(256), 0, static_cast<float*>(m.ff), n);
            } else {
                GemmParams g{static_cast<const __nv_bfloat16*>(xin), l.up.w, nullptr, static_cast<__nv_bfloat16*>(m.ff), nullptr, T, l.up.Np, l.up.Kp};
                launch_gemm_epi(L, GemmEpi::Bf16Relu2, g, &c.state->error);
            }
            sublayer_out(l.down, poly ? m.ff2 : m.ff, l.post2, next, avg);
        }
        if (m.d.side_dim > 0) {
            linear_f32(c, L, l.gate, xin, m.side_f, T);
            L.launch(token_gate_rows_kernel<TA>, dim3(T), dim3(128), 0, (const float*)m.side_f, ids, (const __nv_bfloat16*)m.side_embed,
                     m.d.side_dim * m.d.num_layers, run.layer * m.d.side_dim, c.d.vocab, static_cast<TA*>(m.side_a), m.d.side_dim, m.side_p);
            linear_f32(c, L, l.proj, m.side_a, m.y, T);
            add_norm(m.y, l.side_norm, DecNorm{});
        }
        if (m.tap != nullptr && m.tap_row0 + T <= m.tap_rows && L.err == cudaSuccess)
            L.err = cudaMemcpyAsync(m.tap + ((size_t)i * m.tap_rows + m.tap_row0) * m.Wp, stream, (size_t)T * m.Wp * 4, cudaMemcpyDeviceToDevice, L.stream);
    }
}

}  // namespace

void decoder_rows_pass(efm_b200_ctx& c, const RowPlan& plan, const int32_t* ids, const RowTiles& tiles, Launcher& L) {
    const bool pdl = L.pdl;
    L.pdl = false;
    if (c.decoder->f32) rows_pass<float>(c, plan, ids, tiles, L);
    else rows_pass<__nv_bfloat16>(c, plan, ids, tiles, L);
    L.pdl = pdl;
}

void decoder_rows_logits(efm_b200_ctx& c, const int32_t* rows, int n, Launcher& L) {
    DecoderModel& m = *c.decoder;
    const bool pdl = L.pdl;
    L.pdl = false;
    auto gather = [&](auto* out) {
        using TA = std::remove_pointer_t<decltype(out)>;
        const DecNorm& f = m.final_norm;
        if (m.tanh_norms())
            L.launch(gather_tanh_rows_kernel<TA>, dim3(n), dim3(256), 0, (const float*)c.resid, rows, (const __nv_bfloat16*)f.w, (const __nv_bfloat16*)f.b,
                     (const __nv_bfloat16*)f.alpha, out, m.Wp);
        else
            L.launch(gather_norm_rows_kernel<TA>, dim3(n), dim3(256), 0, (const float*)c.resid, rows, (const __nv_bfloat16*)f.w, out, m.W, m.Wp, m.d.norm_eps);
    };
    if (m.f32) gather(static_cast<float*>(m.head_a));
    else gather(static_cast<__nv_bfloat16*>(m.head_a));
    linear_f32(c, L, m.head, m.head_a, m.logits_rows, n);
    if (m.d.logit_softcap > 0.f || m.d.logit_scale != 1.0f)
        L.launch(cap_logits_rows_kernel, dim3((m.d.vocab + 255) / 256, n), dim3(256), 0, m.logits_rows, m.d.vocab, m.head.Np, m.d.logit_scale, m.d.logit_softcap);
    L.pdl = pdl;
}

// ---- set-up ------------------------------------------------------------------------------------------------------
namespace {
template <typename K>
cudaError_t smem_attr(K kernel, size_t bytes) { return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes); }

// widest cluster the decode attention kernel can be placed with
template <typename TC, int VM, bool ROT, bool LIN>
cudaError_t fit_cluster_v(int& width) {
    const auto kernel = window_attention_decode_kernel<TC, VM, ROT, LIN>;
    cudaError_t e = smem_attr(kernel, sizeof(wd::Smem<VM>));
    if (e != cudaSuccess) return e;
    const bool wide = cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess;
    int cs = wide ? 16 : 8;
    for (; cs > 1; cs >>= 1) {
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(cs, 1, 1);
        cfg.blockDim = dim3(wd::kThreads);
        cfg.dynamicSmemBytes = sizeof(wd::Smem<VM>);
        cudaLaunchAttribute at;
        at.id = cudaLaunchAttributeClusterDimension;
        at.val.clusterDim.x = (unsigned)cs;
        at.val.clusterDim.y = at.val.clusterDim.z = 1;
        cfg.attrs = &at;
        cfg.numAttrs = 1;
        int n = 0;
        if (cudaOccupancyMaxActiveClusters(&n, kernel, &cfg) == cudaSuccess && n >= 1) break;
    }
    (void)cudaGetLastError();
    width = std::min(width, cs);
    return cudaSuccess;
}
template <typename TC, int VM, bool ROT>
cudaError_t fit_cluster(int& width) {
    const cudaError_t e = fit_cluster_v<TC, VM, ROT, false>(width);
    return e == cudaSuccess ? fit_cluster_v<TC, VM, ROT, true>(width) : e;
}
}  // namespace

// token-by-token form: 6 vectors a row; chunked form: one packed block a chunk, the last chunk of every entry short
size_t decoder_delta_pack_floats(int heads, int dim, int rows, int entries) {
    const int Dp = round_up(dim, 32);
    size_t n = (size_t)rows * heads * kDeltaParts * Dp;
    if (Dp <= 128) n = std::max(n, (size_t)(rows / dc::C + 1 + entries) * heads * dc::pack_floats(Dp));
    return n;
}

size_t decoder_linear_ws_floats(const DecoderLayer& l, int rows, int entries) {
    return (size_t)(rows / kLinearChunk + 1 + entries) * l.d.linear_heads * l.d.linear_dim * l.lin_vp;
}

// Widest cluster the one-launch token input fits; 1: two products instead.
static cudaError_t fit_side_cluster(DecoderModel& m, int optin) {
    m.side_cluster = 1;
    if (m.d.side_dim <= 0) return cudaSuccess;
    const bool wide = cudaFuncSetAttribute(token_side_kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess;
    for (int cs = wide ? 16 : 8; cs > 1; cs >>= 1) {
        const size_t bytes = ts::layout(m.Wp, m.side_p, m.Wp, cs).bytes;
        if (bytes + 2048 > (size_t)optin) break;                   // narrower clusters need more per block
        if (smem_attr(token_side_kernel, bytes) != cudaSuccess) continue;
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(cs, 1, 1);
        cfg.blockDim = dim3(kGemvThreads);
        cfg.dynamicSmemBytes = bytes;
        cudaLaunchAttribute at;
        at.id = cudaLaunchAttributeClusterDimension;
        at.val.clusterDim.x = (unsigned)cs;
        at.val.clusterDim.y = at.val.clusterDim.z = 1;
        cfg.attrs = &at;
        cfg.numAttrs = 1;
        int n = 0;
        if (cudaOccupancyMaxActiveClusters(&n, token_side_kernel, &cfg) == cudaSuccess && n >= 1) { m.side_cluster = cs; break; }
    }
    (void)cudaGetLastError();
    return m.side_cluster > 1 ? smem_attr(token_side_kernel, (size_t)optin - 2048) : cudaSuccess;
}

// Heads per block and cluster width of the absorbed form.  A block reads its keys from shared memory once and the queries of
// its heads along with them; every further block of a cluster costs exchange; clusters that are not resident wait.
template <typename TC, int NH>
static cudaError_t fit_latent_heads(const DecoderModel& m, DecoderLayer& l, int optin, double& best) {
    cudaError_t e = smem_attr(latent_attention_kernel<TC, true, NH>, (size_t)optin - 8192);
    if (e == cudaSuccess) e = smem_attr(latent_attention_kernel<TC, false, NH>, (size_t)optin - 8192);
    if (e != cudaSuccess) return e;
    const bool wide = cudaFuncSetAttribute(latent_attention_kernel<TC, true, NH>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess &&
                      cudaFuncSetAttribute(latent_attention_kernel<TC, false, NH>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess;
    const LatentShape s = latent_shape(m, l);
    const int groups = (l.d.heads + NH - 1) / NH, most = latent_splits(l, m.d.cache_pages, wide ? 16 : 8);
    const int keys = std::min(m.d.cache_pages * kPageTokens, l.d.window > 0 ? l.d.window : 1 << 30);
    for (int tile = la::kMaxTile; tile >= 32; tile /= 2)             // shorter tiles: two blocks may share an SM
        for (int cs = most; cs >= 1; cs >>= 1) {
            const size_t bytes = la::layout(s, NH, cs, sizeof(TC), latent_tile(s, NH, cs, sizeof(TC), tile)).bytes;
            if (bytes > (size_t)optin - 8192) continue;
            cudaLaunchConfig_t cfg = {};
            cfg.gridDim = dim3(cs, 1, 1);
            cfg.blockDim = dim3(la::kThreads);
            cfg.dynamicSmemBytes = bytes;
            cudaLaunchAttribute at;
            at.id = cudaLaunchAttributeClusterDimension;
            at.val.clusterDim.x = (unsigned)cs;
            at.val.clusterDim.y = at.val.clusterDim.z = 1;
            cfg.attrs = &at;
            cfg.numAttrs = 1;
            int n = 0;
            if (cudaOccupancyMaxActiveClusters(&n, latent_attention_kernel<TC, true, NH>, &cfg) != cudaSuccess || n < 1) continue;
            const double cost = ((double)keys / cs * (4 + 2 * NH) + 40.0 * cs + 400.0 + 100.0 * ((keys + cs * tile - 1) / (cs * tile))) * ((groups + n - 1) / n);
            if (best < 0.0 || cost < best) {
                best = cost;
                l.la_heads = NH;
                l.la_cluster = cs;
                l.la_tile = tile;
            }
        }
    (void)cudaGetLastError();
    return best < 0.0 && NH == 4 ? cudaErrorInvalidConfiguration : cudaSuccess;
}
template <typename TC>
static cudaError_t fit_latent(const DecoderModel& m, DecoderLayer& l, int optin) {
    double best = -1.0;
    cudaError_t e = fit_latent_heads<TC, 1>(m, l, optin, best);
    if (e == cudaSuccess) e = fit_latent_heads<TC, 2>(m, l, optin, best);
    if (e == cudaSuccess) e = fit_latent_heads<TC, 4>(m, l, optin, best);
    return e;
}

cudaError_t configure_decoder(DecoderModel& m) {
    int dev = 0, optin = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e == cudaSuccess) e = cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
    const size_t gv = (size_t)optin - 2048;
    auto gemv_attr = [&](auto... kernels) { ((e = e == cudaSuccess ? smem_attr(kernels, gv) : e), ...); };
    gemv_attr(gemv_kernel<Epi::Store32, 1>, gemv_kernel<Epi::TokenGate, 1>, gemv_kernel<Epi::Logits, 1>, gemv_kernel<Epi::Store32, 2>, gemv_kernel<Epi::Logits, 2>,
              gemv_kernel<Epi::Store32Bias, 2>, gemv_kernel<Epi::Router, 2>, gemv_kernel<Epi::ExpertUp, 2>, gemv_kernel<Epi::ExpertDown, 2>);
    gemv_attr(gemv_kernel<Epi::Store32, 3>, gemv_kernel<Epi::Logits, 3>, gemv_kernel<Epi::Relu2, 3>, gemv_kernel<Epi::Router, 3>, gemv_kernel<Epi::ExpertUp, 3>,
              gemv_kernel<Epi::ExpertDown, 3>);
    gemv_attr(gemv_kernel<Epi::Store32, 4>, gemv_kernel<Epi::Store32Bias, 4>, gemv_kernel<Epi::Logits, 4>, gemv_kernel<Epi::Router, 4>, gemv_kernel<Epi::ExpertUp, 4>,
              gemv_kernel<Epi::ExpertDown, 4>);
    auto linear_attr = [&](auto type) {
        using T = decltype(type);
        auto chunk = [&](auto kernel, int rm, int rn) { if (e == cudaSuccess) e = smem_attr(kernel, ln::chunk_smem_bytes(rm, rn)); };
        chunk(linear_chunk_rows_kernel<T, 4, 4>, 4, 4); chunk(linear_chunk_rows_kernel<T, 4, 8>, 4, 8);
        chunk(linear_chunk_rows_kernel<T, 8, 4>, 8, 4); chunk(linear_chunk_rows_kernel<T, 8, 8>, 8, 8);
        if (e == cudaSuccess) e = smem_attr(linear_attend_rows_kernel<T, 4>, ln::attend_smem_bytes(256, 4));
        if (e == cudaSuccess) e = smem_attr(linear_attend_rows_kernel<T, 8>, ln::attend_smem_bytes(256, 8));
    };
    linear_attr(float());
    linear_attr(__nv_bfloat16());
    auto linear_tc_attr = [&](auto vp) {
        constexpr int VP = decltype(vp)::value;
        auto set = [&](auto kernel, size_t bytes) { if (e == cudaSuccess) e = smem_attr(kernel, bytes); };
        set(linear_chunk_tc_kernel<VP>, lt::Cfg<VP>::CHUNK_SMEM);
        set(linear_chunk_tc_kernel<VP, true>, lt::Cfg<VP>::CHUNK_SMEM);
        set(linear_attend_tc_kernel<VP>, lt::Cfg<VP>::ATTEND_SMEM);
        set(linear_attend_tc_kernel<VP, true>, lt::Cfg<VP>::ATTEND_SMEM);
        set(linear_attend_ch_tc_kernel<VP, false>, lt::Cfg<VP>::ATTEND_CH_SMEM);
        set(linear_attend_ch_tc_kernel<VP, true>, lt::Cfg<VP>::ATTEND_CH_SMEM);
    };
    linear_tc_attr(std::integral_constant<int, 64>{});
    linear_tc_attr(std::integral_constant<int, 128>{});
    const size_t rows = wa::rows_smem_bytes(256, 256);
    if (e == cudaSuccess) e = smem_attr(window_attention_rows_kernel<float, float, float>, rows);
    if (e == cudaSuccess) e = smem_attr(window_attention_rows_kernel<__nv_bfloat16, __nv_bfloat16, __nv_bfloat16>, rows);
    if (e == cudaSuccess) e = smem_attr(delta_scan_kernel<5>, ds::smem_bytes(160));
    if (e == cudaSuccess) e = smem_attr(delta_scan_kernel<6>, ds::smem_bytes(192));
    if (e == cudaSuccess) e = smem_attr(delta_scan_kernel<7>, ds::smem_bytes(224));
    if (e == cudaSuccess) e = smem_attr(delta_scan_kernel<8>, ds::smem_bytes(256));
    auto tc_attr = [&](auto dp, auto vp) {
        constexpr int DP = decltype(dp)::value, VP = decltype(vp)::value;
        if (e == cudaSuccess) e = smem_attr(window_attention_tc_kernel<DP, VP, 0, false>, wt::Cfg<DP, VP, 0>::SMEM);
        if (e == cudaSuccess) e = smem_attr(window_attention_tc_kernel<DP, VP, 0, true>, wt::Cfg<DP, VP, 0>::SMEM);
        if (e == cudaSuccess) e = smem_attr(window_attention_tc_kernel<DP, VP, 0, false, true>, wt::Cfg<DP, VP, 0>::SMEM);
        if (e == cudaSuccess) e = smem_attr(window_attention_tc_kernel<DP, VP, 64, false>, wt::Cfg<DP, VP, 64>::SMEM);
    };
    const std::integral_constant<int, 64> k64{};
    const std::integral_constant<int, 128> k128{};
    tc_attr(k64, k64); tc_attr(k64, k128); tc_attr(k128, k64); tc_attr(k128, k128);
    if (e == cudaSuccess) e = smem_attr(delta_prepare_kernel<96>, sizeof(dc::PrepSmem<96>));
    if (e == cudaSuccess) e = smem_attr(delta_prepare_kernel<128>, sizeof(dc::PrepSmem<128>));
    if (e == cudaSuccess) e = smem_attr(delta_chunk_scan_kernel<64>, sizeof(dc::ScanSmem<64>));
    if (e == cudaSuccess) e = smem_attr(delta_chunk_scan_kernel<96>, sizeof(dc::ScanSmem<96>));
    if (e == cudaSuccess) e = smem_attr(delta_chunk_scan_kernel<128>, sizeof(dc::ScanSmem<128>));
    if (e == cudaSuccess) e = fit_side_cluster(m, optin);
    for (DecoderLayer& l : m.layers)
        if (l.d.mixer == EFM_MIXER_LATENT_ATTENTION && e == cudaSuccess) e = m.f32 ? fit_latent<float>(m, l, optin) : fit_latent<__nv_bfloat16>(m, l, optin);
    m.attn_cluster = 16;
    auto fit = [&](auto type) {
        using TC = decltype(type);
        if (e == cudaSuccess) e = fit_cluster<TC, 64, false>(m.attn_cluster);
        if (e == cudaSuccess) e = fit_cluster<TC, 128, false>(m.attn_cluster);
        if (e == cudaSuccess) e = fit_cluster<TC, 256, false>(m.attn_cluster);
        if (e == cudaSuccess) e = fit_cluster<TC, 64, true>(m.attn_cluster);
        if (e == cudaSuccess) e = fit_cluster<TC, 128, true>(m.attn_cluster);
        if (e == cudaSuccess) e = fit_cluster<TC, 256, true>(m.attn_cluster);
    };
    if (m.f32) fit(float());
    else fit(__nv_bfloat16());
    return e;
}

}  // namespace efm
