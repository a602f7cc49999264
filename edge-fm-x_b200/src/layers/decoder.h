// Layered decoder: a list of layers, each with its own mixer (attention | generalised delta rule) and an optional dense
// feed-forward, sublayer outputs normalised before the residual add, optional per-layer token input.  Weights, buffers
// and launch sequences (definitions in decoder.cu); the C ABI side is backends/b200/decoder_b200.cu.
#pragma once
#include <set>
#include <string>
#include <vector>

#include "../backends/b200/ctx.h"
#include "../operators/row_plan.cuh"

namespace efm {
struct Launcher;

inline int round_up(int n, int m) { return (n + m - 1) / m * m; }

// bf16 weight [Np][Kp]: K padded to 8 (TMA rows, 128-bit loads), N to 2 (row pairs of the decode GEMV), pads zero.
struct DecLinear {
    __nv_bfloat16* w = nullptr;
    int N = 0, K = 0, Np = 0, Kp = 0;
};

struct DecoderLayer {
    efm_decoder_layer d{};
    int Dp = 0, Vp = 0;                   // attention: padded channels of a cache row
    int mix_w = 0, mix_wp = 0;            // mixer output width (heads * value channels), padded
    DecLinear in;                         // attention: q | k | v; delta: r | k | v | g | a | w1
    DecLinear out;                        // W_o
    DecLinear w2;                         // delta: decay projection
    DecLinear up, down, gate, proj;       // feed-forward; token side
    __nv_bfloat16 *norm1 = nullptr, *norm2 = nullptr, *side_norm = nullptr, *act = nullptr;
    __nv_bfloat16 *q_norm = nullptr, *k_norm = nullptr, *temp = nullptr;
    __nv_bfloat16 *w0 = nullptr, *a_bias = nullptr, *mix_norm = nullptr;
    void *k_pool = nullptr, *v_pool = nullptr;       // [pages * 64][kv_heads][Dp / Vp], bf16 or fp32
    size_t state_off = 0;                 // delta: first float of this layer inside a state slot
};

struct DecoderModel {
    efm_decoder_desc d{};
    bool f32 = false;
    int W = 0, Wp = 0;                    // width, padded to 8
    int side_p = 0;                       // token-side width padded to 8
    std::vector<DecoderLayer> layers;
    __nv_bfloat16 *side_embed = nullptr, *final_norm = nullptr;
    DecLinear head;
    std::set<std::string> seen;
    // caches
    int32_t* page_table = nullptr;        // [max_slots][cache_pages]
    float* state_pool = nullptr;          // [state_slots][state_stride]
    size_t state_stride = 0;
    std::vector<int> free_tables;
    // many-row buffers; "act" ones are bf16 or (32-bit mode) fp32
    void *xa = nullptr, *proj_a = nullptr, *q = nullptr, *mix = nullptr, *ff = nullptr, *ff2 = nullptr, *side_a = nullptr, *head_a = nullptr;
    float *y = nullptr, *proj_f = nullptr, *pack = nullptr, *tanh_w = nullptr, *decay = nullptr, *o = nullptr, *side_f = nullptr, *logits_rows = nullptr;
    int tanh_ld = 0;
    int32_t* step_buf = nullptr;          // packed per-step indices
    size_t step_words = 0;
    int max_want = 0;
    float* tap = nullptr;                 // debugging / tests: residual stream after every layer [layers][rows][Wp]
    int tap_rows = 0, tap_row0 = 0;
    // one-row buffers
    float *d_in = nullptr, *d_mix = nullptr, *d_y = nullptr, *d_y2 = nullptr, *d_ff = nullptr, *d_gate = nullptr;
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
cudaError_t configure_decoder(DecoderModel& m);

}  // namespace efm
