// Layered decoder: a list of layers, each with its own mixer (attention | latent attention | generalised delta rule | linear attention |
// attention and linear attention side by side) and an optional feed-forward (dense | routed experts), sublayer outputs (and, sandwich
// layout, inputs; or the inputs alone, elementwise) normalised, optional per-layer token input, short convolutions of the sublayers'
// inputs, average over depth; a span of layers may run several times.  Weights, buffers and launch sequences (definitions in decoder.cu);
// the C ABI side is backends/b200/decoder_b200.cu.
#pragma once
#include <algorithm>
#include <set>
#include <string>
#include <vector>

#include "../backends/b200/ctx.h"
#include "../operators/expert_rows.h"
#include "../operators/row_plan.cuh"

namespace efm {
struct Launcher;

inline int round_up(int n, int m) { return (n + m - 1) / m * m; }

// bf16 weight [Np][Kp]: K padded to 8 (TMA rows, 128-bit loads), N to 2 (row pairs of the decode GEMV), pads zero.
struct DecLinear {
    __nv_bfloat16* w = nullptr;
    int N = 0, K = 0, Np = 0, Kp = 0;
    __nv_bfloat16* bias = nullptr;        // [Np] or null
};

// Weight of an RMS norm; with b and alpha tanh(alpha x) w + b.
struct DecNorm { __nv_bfloat16 *w = nullptr, *b = nullptr, *alpha = nullptr; };

struct DecoderLayer {
    efm_decoder_layer d{};
    int Dp = 0, Vp = 0;                   // attention: padded channels of a cache row; latent: padded head channels
    int mix_w = 0, mix_wp = 0;            // mixer output width (heads * value channels; parallel: both halves), padded
    DecLinear in;                         // attention: q | k | v; latent: dq | c | r | g, each padded to 8; delta: r | k | v | g | a | w1;
                                          // parallel: attention's, then q | k | v | g of linear attention, each padded to 8;
                                          // linear: q | k | v | g (| a1), each padded to 8; attention with a gate: q | k | v | g
    DecLinear out;                        // W_o (parallel: the two side by side)
    DecLinear w2;                         // delta, linear with projected decays: second factor of the decay projection
    DecLinear up, down, gate, proj;       // dense feed-forward; token side
    DecNorm pre1, pre2;
    __nv_bfloat16 *post1 = nullptr, *post2 = nullptr, *side_norm = nullptr, *act = nullptr;
    __nv_bfloat16 *q_norm = nullptr, *k_norm = nullptr, *temp = nullptr;
    __nv_bfloat16 *w0 = nullptr, *a_bias = nullptr, *mix_norm = nullptr;
    float* inv_freq = nullptr;            // rotation: [rot_dims / 2]
    // latent attention
    int Qp = 0, Lc = 0, Rc = 0;           // query latent, cached latent, rotated part: padded to 8
    DecLinear uq, ukv;                    // [heads][Dp + Rc] rows; [heads][Dp] key rows, then [heads][Vp] value rows
    __nv_bfloat16 *sink = nullptr, *shift = nullptr;      // shift: attention with sigmoid weights
    int la_heads = 1, la_cluster = 1, la_tile = 64;       // absorbed form: heads per block, widest cluster, keys per tile
    __nv_bfloat16 *canon1 = nullptr, *canon2 = nullptr;   // input convolutions of mixer and feed-forward, [taps][Wp]
    __nv_bfloat16* dwa = nullptr;         // average over depth, [layer + 2]
    // linear attention, alone or beside attention
    int lin_in = 0, lin_mix = 0;          // its first column in the projections and in the mixer output
    int rot_table = -1;                   // alone: its table among those of a pass (bf16), or none
    int lin_vp = 0;                       // value channels padded to 4 (state rows)
    float* lin_powers = nullptr;          // [linear_heads][kLinearPowers + 1]
    bool parallel() const { return d.mixer == EFM_MIXER_PARALLEL; }
    bool alone() const { return d.mixer == EFM_MIXER_LINEAR; }
    bool linear() const { return parallel() || alone(); }
    bool channel_decay() const { return alone() && d.linear_tau > 0.f; }
    int linear_qk() const { return round_up(d.linear_heads * d.linear_dim, 8); }      // columns of q (and k), of v (and g)
    int linear_v() const { return round_up(d.linear_heads * d.linear_vdim, 8); }
    bool attention() const { return d.mixer == EFM_MIXER_ATTENTION || d.mixer == EFM_MIXER_PARALLEL; }
    // routed experts
    DecLinear router, expert_in, expert_out;   // [experts], a shared expert's gate behind; [experts][up_rows()]; [experts][width][ffp]
    DecLinear shared_in, shared_out;      // the same of a shared expert
    int ffp = 0, sfp = 0;
    bool gated_experts() const { return d.expert_glu != EFM_GLU_NONE_RELU2; }
    int up_rows(int ffp_) const { return gated_experts() ? 2 * ffp_ : ffp_; }
    bool moe() const { return d.experts > 0; }
    bool mlp() const { return d.experts > 0 || d.ff > 0; }
};

// One run of a layer: a looped layer runs several times, every time with its own cache or state.
struct DecoderRun {
    int layer = 0;
    void *k_pool = nullptr, *v_pool = nullptr;       // attention: [pages * 64][kv_heads][Dp / Vp]; latent: [pages * 64][Lc + Rc] (k_pool); bf16 or fp32
    size_t state_off = 0;                 // recurrent mixers: first float of this run inside a state slot
    size_t conv1_off = 0, conv2_off = 0;  // input convolutions: the last inputs, [taps][Wp] by position modulo taps
};

struct DecoderModel {
    efm_decoder_desc d{};
    bool f32 = false;
    int W = 0, Wp = 0;                    // width, padded to 8
    int side_p = 0;                       // token-side width padded to 8
    bool tanh_norms() const { return d.norm_layout == EFM_NORM_INPUT; }
    // something that only level 4 of the decode GEMV (gemv.cuh) has
    bool extended = false;
    int gemv_level() const { return extended ? 4 : tanh_norms() ? 3 : d.norm_layout == EFM_NORM_SANDWICH || d.embed_scale != 1.0f ? 2 : 1; }
    std::vector<DecoderLayer> layers;
    std::vector<DecoderRun> runs;         // in order
    __nv_bfloat16* side_embed = nullptr;
    DecNorm final_norm;
    DecLinear head;
    std::set<std::string> seen;
    // caches
    int32_t* page_table = nullptr;        // [max_slots][cache_pages]
    float* state_pool = nullptr;          // [state_slots][state_stride]
    size_t state_stride = 0;
    std::vector<int> free_tables;
    // many-row buffers; "act" ones are bf16 or (32-bit mode) fp32
    void *xa = nullptr, *proj_a = nullptr, *q = nullptr, *mix = nullptr, *ff = nullptr, *ff2 = nullptr, *side_a = nullptr, *head_a = nullptr, *cq = nullptr;
    float *y = nullptr, *proj_f = nullptr, *pack = nullptr, *tanh_w = nullptr, *decay = nullptr, *o = nullptr, *side_f = nullptr, *logits_rows = nullptr;
    int tanh_ld = 0;
    // latent attention, long entries: visible cache rows and what they expand to
    __nv_bfloat16 *ws_c = nullptr, *ws_kv = nullptr;
    int ws_pages = 0, ws_window = 0;      // capacity (0: no layer uses it); largest window of the layers that use it (0: no window)
    // (cos, sin) of a pass's rows, one table for all layers that turn alike
    struct RotTable { int dims = 0, layer = 0; float2* cs = nullptr; };
    std::vector<RotTable> rot_tables;
    float* lin_ws = nullptr;              // linear attention: states of a pass's chunks
    float* hist = nullptr;                // average over depth: the embedding and every layer's result, [layers + 1][rows][Wp]
    float *d_hist = nullptr, *d_avg = nullptr;            // the same of one row; the sum behind the current layer without its own result
    // routed experts: rows sorted by expert
    void *ex_in = nullptr, *ex_act = nullptr, *ex_y = nullptr;
    void *sh_act = nullptr, *sh_y = nullptr;              // shared expert
    float *ex_gu = nullptr, *sh_gu = nullptr, *route_logits = nullptr;
    ExpertRows ex{};
    int ex_rows = 0;
    // a pass's shared expert runs beside the choice and the sorting of the rows
    cudaStream_t side = nullptr;
    cudaEvent_t side_start = nullptr, side_end = nullptr;
    int32_t* step_buf = nullptr;          // packed per-step indices
    size_t step_words = 0;
    int max_want = 0;
    float* tap = nullptr;                 // debugging / tests: residual stream after every layer run [runs][rows][Wp]
    int tap_rows = 0, tap_row0 = 0;
    // one-row buffers
    float *d_in = nullptr, *d_mix = nullptr, *d_y = nullptr, *d_y2 = nullptr, *d_ff = nullptr, *d_gate = nullptr;
    float *d_q = nullptr, *d_h = nullptr, *d_route = nullptr, *d_act = nullptr, *d_route_w = nullptr;
    int32_t* d_route_id = nullptr;
    unsigned int* d_route_ticket = nullptr;
    int attn_cluster = 8, side_cluster = 1;
};

// One decode step of the bound slot (reads the device state); sample: run the sampler and advance the state.
void decoder_decode_step(efm_b200_ctx& c, KvSlot& slot, Launcher& L, bool sample, bool want_logits);
// One pass over rows [0, plan.rows) with ids on the device; the residual stream is left in c.resid.
// Attention work lists of a batched pass (listed): tensor-core tiles of the long entries, CUDA-core tiles of the short
// ones, and every row in CUDA-core tiles (layers the tensor-core form does not take).  Not listed: the single entry.
struct RowTiles {
    const RowTile *tc = nullptr, *simt = nullptr, *all = nullptr;
    int n_tc = 0, n_simt = 0, n_all = 0;
    // latent attention: rows of the short entries (absorbed form); workspace pages of the long entries and those of them that
    // hold earlier tokens (listed, or from ws_page0 on)
    const int32_t* short_rows = nullptr;
    const RowTile* ws_pages = nullptr;
    int n_short = 0, n_ws = 0, n_gather = 0, ws_page0 = 0;
    bool listed = false;
};
void decoder_rows_pass(efm_b200_ctx& c, const RowPlan& plan, const int32_t* ids, const RowTiles& tiles, Launcher& L);
// logits_rows[i] = head . norm(resid[rows[i]]), i < n <= max_want; rows on the device
void decoder_rows_logits(efm_b200_ctx& c, const int32_t* rows, int n, Launcher& L);
// Rows of one entry that share an attention block; entries shorter than kTcMinRows run on the CUDA-core form.
constexpr int kTcMinRows = 16;
int decoder_tc_tile_rows();
int decoder_simt_tile_rows();
bool decoder_layer_tc(const DecoderModel& m, const DecoderLayer& l);
// scratch of one recurrent layer for `rows` rows of at most `entries` sequences
size_t decoder_delta_pack_floats(int heads, int dim, int rows, int entries);
// the same of a layer with linear attention: chunk states
size_t decoder_linear_ws_floats(const DecoderLayer& l, int rows, int entries);
// first cache page (of its sequence) that a long entry at position pos0 needs in the workspace
inline int decoder_ws_page0(const DecoderModel& m, int pos0) { return m.ws_window > 0 ? std::max(0, pos0 - m.ws_window + 1) / kPageTokens : 0; }
cudaError_t configure_decoder(DecoderModel& m);      // after the layers are set up

}  // namespace efm
