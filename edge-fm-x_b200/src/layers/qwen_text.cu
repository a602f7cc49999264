// Launch sequences of the Qwen2.5 / Qwen2.5-VL text tower: one decode step and one prefill
// chunk.  Layer order and residual dataflow follow the reference's forward
// (src/models/qwen2_5/qwen2_5.cpp:534-930); what the reference runs as 9-10 kernels per layer
// at decode is five launches here:
//   [embed +] RMSNorm + QKV GEMV + bias + RoPE + KV append | attention | o_proj + residual |
//   RMSNorm + gate/up GEMV + SiLU*mul | down_proj + residual
// and norm + lm_head + block argmax | sampler + state advance at the end of the step.
#include "qwen_text.h"

#include "../operators/attention_mma.cuh"
#include "../operators/attention_tc.cuh"
#include "../operators/sage_attention.cuh"
#include "../operators/gemm_tc.cuh"
#include "../operators/prefill.cuh"
#define EFM_DECLARATIONS_ONLY
#include "../operators/sample.cuh"
#undef EFM_DECLARATIONS_ONLY
#include "../backends/b200/nccl_glue.h"
#include "launch.cuh"
#include "tensor_map.h"

namespace efm {

static GemvParams base_gemv(const __nv_bfloat16* W, int N, int K) {
    GemvParams p{};
    p.W = W;
    p.N = N;
    p.K = K;
    p.n_items = N / 2;
    p.prologue = kProPlain;
    return p;
}

// One decode GEMV: the INT4 copy of the linear when the context decodes from INT4 weights, else bf16.
template <Epi EPI>
static void launch_decode_gemv(efm_b200_ctx& c, Launcher& L, const GemvParams& p, const W4Linear* w4, int swiglu_half = 0) {
    if (c.decode_w4 && w4 != nullptr && w4->ready) {
        GemvW4Params q{};
        q.g = p;
        q.g.W = nullptr;
        q.Wq = w4->q;
        q.scales = static_cast<const __half2*>(w4->s);
        q.swiglu_half = swiglu_half;
        launch_gemv_w4<EPI>(L, q, c.num_sms);
        return;
    }
    launch_gemv<EPI>(L, p, c.num_sms);
}

static void tp_all_reduce(efm_b200_ctx& c, Launcher& L, const float* send, float* recv, size_t count);
static void tp_all_gather(efm_b200_ctx& c, Launcher& L, const float* send, float* recv, size_t count);
static void launch_sample_only(efm_b200_ctx& c, Launcher& L, int n_part, int advance);
bool tp_greedy_exchange(const efm_b200_ctx& c);

void launch_lm_head_and_sample(efm_b200_ctx& c, Launcher& L, const float* resid_row, int advance, bool decode_pass) {
    const efm_model_desc& d = c.d;
    GemvParams p = base_gemv(c.lm_head, c.vocab_l, d.hidden);      // this rank's rows (all of them without TP)
    p.prologue = kProRmsNorm;
    p.xr = resid_row;
    p.norm_w = c.final_norm;
    p.eps = d.rms_eps;
    p.logits = c.tp_size > 1 ? c.logits_l : c.logits;
    p.part_val = c.part_val;
    p.part_idx = c.part_idx;
    if (decode_pass) launch_decode_gemv<Epi::Logits>(c, L, p, &c.w4_lm_head);
    else launch_gemv<Epi::Logits>(L, p, c.num_sms);
    if (c.tp_size > 1) {
        const bool pdl = L.pdl;
        if (tp_greedy_exchange(c)) {
            // greedy: the ranks exchange their (maximum, id) as one word each inside the sampler; no collective, no
            // gathered logits (efm_b200_read_logits gathers on demand)
            launch_sample_only(c, L, /*n_part=*/c.num_sms, advance);
        } else {
            tp_all_gather(c, L, c.logits_l, c.logits, (size_t)c.vocab_l);
            launch_sample_only(c, L, /*n_part=*/0, advance);
        }
        L.pdl = pdl;
        return;
    }

    SampleParams s{};
    s.logits = c.logits;
    s.vocab = d.vocab;
    s.part_val = c.part_val;
    s.part_idx = c.part_idx;
    s.n_part = c.num_sms;
    s.temperature = c.sampling.temperature;
    s.top_p = c.sampling.top_p;
    s.seed = c.sampling.seed;
    s.state = c.state;
    s.tokens_out = c.tokens_out;
    s.max_response = d.max_response_tokens;
    s.advance = advance;
    s.wbuf = c.wbuf;
    s.xchg = sample_xchg(c.wbuf, d.vocab);
    launch_sample(L, s);
}

// Tensor parallel with imported peer buffers and greedy sampling: the sampler exchanges the ranks' maxima itself.
bool tp_greedy_exchange(const efm_b200_ctx& c) {
    return c.tp_size > 1 && c.peers_ready && c.sampling.temperature < 1e-6f;
}

static void launch_sample_only(efm_b200_ctx& c, Launcher& L, int n_part, int advance) {
    const efm_model_desc& d = c.d;
    SampleParams s{};
    s.logits = c.logits;
    s.vocab = d.vocab;
    s.part_val = c.part_val;
    s.part_idx = c.part_idx;
    s.n_part = n_part;
    if (n_part > 0 && tp_greedy_exchange(c)) {
        s.tp_n = c.tp_size;
        s.tp_rank = c.tp_rank;
        s.tp_vocab_offset = c.vocab_off;
        s.tp_count = reinterpret_cast<unsigned int*>(c.tp_xchg + 104);
        for (int r = 0; r < c.tp_size; ++r) s.tp_peer_slot[r] = reinterpret_cast<unsigned long long*>(c.peer_base[r] + c.tp_sample_off);
        s.tp_error = &c.state->error;
        s.tp_error_host = c.error_host;
        s.tp_wait_ns = c.peer_wait_ns;
    }
    s.temperature = c.sampling.temperature;
    s.top_p = c.sampling.top_p;
    s.seed = c.sampling.seed;
    s.state = c.state;
    s.tokens_out = c.tokens_out;
    s.max_response = d.max_response_tokens;
    s.advance = advance;
    s.wbuf = c.wbuf;
    s.xchg = sample_xchg(c.wbuf, d.vocab);
    launch_sample(L, s);
}

// Collectives on the context stream (graph-capturable).  A failure is recorded like a launch failure.
static void tp_all_reduce(efm_b200_ctx& c, Launcher& L, const float* send, float* recv, size_t count) {
    if (L.err != cudaSuccess) return;
    const NcclApi& api = nccl_api();
    if (!api.ok || c.nccl_comm == nullptr || api.all_reduce_f32_sum(send, recv, count, c.nccl_comm, L.stream) != 0)
        L.err = cudaErrorUnknown;
    else if (L.counter != nullptr) ++*L.counter;
}
static void tp_all_gather(efm_b200_ctx& c, Launcher& L, const float* send, float* recv, size_t count) {
    if (L.err != cudaSuccess) return;
    const NcclApi& api = nccl_api();
    if (!api.ok || c.nccl_comm == nullptr || api.all_gather_f32(send, recv, count, c.nccl_comm, L.stream) != 0)
        L.err = cudaErrorUnknown;
    else if (L.counter != nullptr) ++*L.counter;
}

void tp_gather_logits(efm_b200_ctx& c, Launcher& L) { tp_all_gather(c, L, c.logits_l, c.logits, (size_t)c.vocab_l); }

// Exchange buffer layout (ctx.h): count at byte 64, ticket at 68, receive buffer [2][tp][H] of {fp32, count} at 256.
static void peers_producer(const efm_b200_ctx& c, GemvParams& p, int parity) {
    const size_t H = (size_t)c.d.hidden;
    p.n_peers = c.tp_size;
    for (int r = 0; r < c.tp_size; ++r)
        p.peer_out[r] = reinterpret_cast<uint2*>(c.peer_base[r] + 256) + ((size_t)parity * c.tp_size + c.tp_rank) * H;
    p.epoch = reinterpret_cast<unsigned int*>(c.tp_xchg + 64);
    p.ticket = reinterpret_cast<unsigned int*>(c.tp_xchg + 68);
}
static void peers_consumer(const efm_b200_ctx& c, GemvParams& p, int parity) {
    p.addend_parts = reinterpret_cast<const uint2*>(c.tp_xchg + 256) + (size_t)parity * c.tp_size * c.d.hidden;
    p.n_parts = c.tp_size;
    p.epoch = reinterpret_cast<unsigned int*>(c.tp_xchg + 64);
    p.error = &c.state->error;
    p.error_host = c.error_host;
    p.wait_ns = c.peer_wait_ns;
}

// Tensor-parallel prefill: sum of the row-parallel partial c.ybuf [S, H] over the ranks, added to the residual.
// With imported peer buffers: reduce-scatter + all-gather over peer stores (operators/prefill.cuh); otherwise
// ncclAllReduce + add.  Header words of the exchange allocation (ctx.h): prefill exchange count at byte 96, ticket at
// 100, scatter flags [2][8] at 128, gather flags [2][8] at 192.
static void tp_prefill_sum(efm_b200_ctx& c, Launcher& L, int S, int parity) {
    const size_t H = (size_t)c.d.hidden, n = (size_t)S * H;
    if (!c.peers_ready) {
        tp_all_reduce(c, L, c.ybuf, c.ysum, n);
        L.launch(add_rows_kernel, dim3(std::min<size_t>((n / 2 + 255) / 256, (size_t)c.num_sms * 8)), dim3(256), 0, c.resid,
                 (const float*)c.ysum, n / 2);
        return;
    }
    const int tp = c.tp_size;
    const size_t slot = c.tp_slot_floats;                                    // floats per (parity, rank) receive slot
    PeerXchgParams pp{};
    pp.src = c.ybuf;
    pp.n_peers = tp;
    pp.rank = c.tp_rank;
    pp.S = S;
    pp.H = (int)H;
    pp.rows_per = (S + tp - 1) / tp;
    pp.slot_floats = slot;
    pp.epoch = reinterpret_cast<unsigned int*>(c.tp_xchg + 96);
    pp.ticket = reinterpret_cast<unsigned int*>(c.tp_xchg + 100);
    pp.error = &c.state->error;
    pp.error_host = c.error_host;
    pp.wait_ns = c.peer_wait_ns;
    pp.recv_local = reinterpret_cast<const float*>(c.tp_xchg + c.tp_prefill_off) + (size_t)parity * tp * slot;
    pp.gather_local = reinterpret_cast<const float*>(c.tp_xchg + c.tp_gather_off) + (size_t)parity * c.max_s * H;
    pp.resid = c.resid;
    for (int r = 0; r < tp; ++r) {
        pp.recv[r] = reinterpret_cast<float*>(c.peer_base[r] + c.tp_prefill_off) + ((size_t)parity * tp + c.tp_rank) * slot;
        pp.gather[r] = reinterpret_cast<float*>(c.peer_base[r] + c.tp_gather_off) + (size_t)parity * c.max_s * H;
    }
    const int grid_all = (int)std::min<size_t>((n / 4 + 255) / 256, (size_t)c.num_sms * 8);
    const int grid_own = (int)std::min<size_t>(((size_t)pp.rows_per * H / 4 + 255) / 256, (size_t)c.num_sms * 8);
    // 1. scatter (publishes this rank's scatter flag on every rank)
    for (int r = 0; r < tp; ++r) pp.flag[r] = reinterpret_cast<unsigned int*>(c.peer_base[r] + 128) + parity * 8 + c.tp_rank;
    L.launch(peer_scatter_rows_kernel, dim3(grid_all), dim3(256), 0, pp);
    // 2. reduce own rows, store them into every rank's gather buffer (waits for the scatter flags, publishes gather flags)
    pp.flags_local = reinterpret_cast<const unsigned int*>(c.tp_xchg + 128) + parity * 8;
    for (int r = 0; r < tp; ++r) pp.flag[r] = reinterpret_cast<unsigned int*>(c.peer_base[r] + 192) + parity * 8 + c.tp_rank;
    L.launch(peer_reduce_gather_kernel, dim3(std::max(1, grid_own)), dim3(256), 0, pp);
    // 3. resid += gathered sum (waits for the gather flags)
    pp.flags_local = reinterpret_cast<const unsigned int*>(c.tp_xchg + 192) + parity * 8;
    L.launch(peer_add_gathered_kernel, dim3(grid_all), dim3(256), 0, pp);
}

// Tensor-parallel decode step: column-parallel QKV / gate-up, row-parallel o_proj / down with an
// all-reduce of the fp32 partial [H]; the residual add moves into the next kernel's norm prologue
// (x = bf16(x + bf16(sum)), ping-ponging between two residual buffers so no block re-reads a row that
// block 0 already updated); lm_head rows are split and the logits all-gathered before sampling.
static void qwen_decode_step_tp(efm_b200_ctx& c, KvSlot& slot, Launcher& L) {
    const efm_model_desc& d = c.d;
    const int H = d.hidden, D = d.head_dim, QD = d.q_heads * D, KVD = d.kv_heads * D, I = d.intermediate;
    float* RA = c.resid_d;
    float* RB = c.resid_d2;
    const bool fused = c.peers_ready;        // exchange inside the GEMVs over peer memory instead of ncclAllReduce
    for (int l = 0; l < d.num_layers; ++l) {
        const LayerWeights& w = c.layers[l];
        {
            GemvParams p = base_gemv(w.qkv, QD + 2 * KVD, H);
            p.prologue = l == 0 ? kProEmbedRmsNorm : kProRmsNorm;
            p.xr = RB;                       // l > 0: residual after the previous layer's attention add
            if (l > 0) { if (fused) peers_consumer(c, p, 1); else p.addend = c.ysum; }
            p.resid_out = RA;
            p.norm_w = w.in_norm; p.eps = d.rms_eps; p.embed_table = c.embed; p.vocab = d.vocab; p.state = c.state;
            p.bias = w.qkv_bias; p.q_out_f = c.q_d; p.k_cache = slot.k[l]; p.v_cache = slot.v[l]; p.inv_freq = c.inv_freq;
            p.q_heads = d.q_heads; p.kv_heads = d.kv_heads; p.head_dim = D; p.use_mrope = d.use_mrope;
            p.sec0 = d.mrope_section[0]; p.sec1 = d.mrope_section[0] + d.mrope_section[1]; p.max_tokens = slot.max_tokens;
            launch_gemv<Epi::QkvRope>(L, p, c.num_sms);
        }
        {
            DecodeAttnParams a{};
            a.qf = c.q_d; a.k_cache = slot.k[l]; a.v_cache = slot.v[l]; a.outf = c.attn_d; a.state = c.state;
            a.q_heads = d.q_heads; a.kv_heads = d.kv_heads; a.group = d.q_heads / d.kv_heads;
            a.n_splits = slot.n_splits; a.chunk_cap = slot.chunk_cap; a.max_tokens = slot.max_tokens; a.cluster = slot.attn_cluster; a.early = l > 0 ? 1 : 0;
            a.scale = 1.0f / sqrtf((float)D);
            a.part_o = c.attn_part_o; a.part_ml = c.attn_part_ml; a.counters = c.attn_counters;
            launch_decode_attention(L, a, D);
        }
        {
            GemvParams p = base_gemv(w.o, H, c.o_k);
            p.xf = c.attn_d + (size_t)c.att_rep_idx * c.o_k;
            if (fused) {
                peers_producer(c, p, 0);
                launch_gemv<Epi::Peers>(L, p, c.num_sms);              // fp32 partial straight into every rank's buffer
            } else {
                p.logits = c.ybuf; p.part_val = c.part_val; p.part_idx = c.part_idx;
                launch_gemv<Epi::Logits>(L, p, c.num_sms);             // fp32 partial output
            }
        }
        if (!fused) tp_all_reduce(c, L, c.ybuf, c.ysum, (size_t)H);
        {
            GemvParams p = base_gemv(w.gate_up, 2 * I, H);
            p.prologue = kProRmsNorm;
            p.xr = RA; p.resid_out = RB;
            if (fused) peers_consumer(c, p, 0); else p.addend = c.ysum;
            p.norm_w = w.post_norm; p.eps = d.rms_eps; p.yf = c.act_d;
            launch_gemv<Epi::SwiGlu>(L, p, c.num_sms);
        }
        {
            GemvParams p = base_gemv(w.down, H, I);
            p.xf = c.act_d;
            if (fused) {
                peers_producer(c, p, 1);
                launch_gemv<Epi::Peers>(L, p, c.num_sms);
            } else {
                p.logits = c.ybuf; p.part_val = c.part_val; p.part_idx = c.part_idx;
                launch_gemv<Epi::Logits>(L, p, c.num_sms);
            }
        }
        if (!fused) tp_all_reduce(c, L, c.ybuf, c.ysum, (size_t)H);
    }
    {
        GemvParams p = base_gemv(c.lm_head, c.vocab_l, H);
        p.prologue = kProRmsNorm;
        p.xr = RB; p.resid_out = RA;
        if (fused) peers_consumer(c, p, 1); else p.addend = c.ysum;
        p.norm_w = c.final_norm; p.eps = d.rms_eps;
        p.logits = c.logits_l; p.part_val = c.part_val; p.part_idx = c.part_idx;
        launch_gemv<Epi::Logits>(L, p, c.num_sms);
    }
    tp_all_gather(c, L, c.logits_l, c.logits, (size_t)c.vocab_l);
    launch_sample_only(c, L, /*n_part=*/0, /*advance=*/1);
}

void launch_w4_repack(Launcher& L, const W4RepackParams& p) {
    const bool pdl = L.pdl;
    L.pdl = false;
    L.launch(w4_repack_kernel<0>, dim3(((p.n_items + 7) / 8) * 8), dim3(256), 0, p);
    L.pdl = pdl;
}

void qwen_decode_step(efm_b200_ctx& c, KvSlot& slot, Launcher& L) {
    if (c.tp_size > 1) {
        qwen_decode_step_tp(c, slot, L);
        return;
    }
    const efm_model_desc& d = c.d;
    const int H = d.hidden, D = d.head_dim, QD = d.q_heads * D, KVD = d.kv_heads * D, I = d.intermediate;
    for (int l = 0; l < d.num_layers; ++l) {
        const LayerWeights& w = c.layers[l];
        {
            GemvParams p = base_gemv(w.qkv, QD + 2 * KVD, H);
            p.prologue = l == 0 ? kProEmbedRmsNorm : kProRmsNorm;
            p.xr = c.resid_d;
            p.norm_w = w.in_norm;
            p.eps = d.rms_eps;
            p.embed_table = c.embed;
            p.vocab = d.vocab;
            p.resid_out = c.resid_d;
            p.state = c.state;
            p.bias = w.qkv_bias;
            p.q_out_f = c.q_d;
            p.k_cache = slot.k[l];
            p.v_cache = slot.v[l];
            p.inv_freq = c.inv_freq;
            p.q_heads = d.q_heads;
            p.kv_heads = d.kv_heads;
            p.head_dim = D;
            p.use_mrope = d.use_mrope;
            p.sec0 = d.mrope_section[0];
            p.sec1 = d.mrope_section[0] + d.mrope_section[1];
            p.max_tokens = slot.max_tokens;
            launch_decode_gemv<Epi::QkvRope>(c, L, p, &w.w4_qkv);
        }
        {
            DecodeAttnParams a{};
            a.qf = c.q_d;
            a.k_cache = slot.k[l];
            a.v_cache = slot.v[l];
            a.outf = c.attn_d;
            a.state = c.state;
            a.q_heads = d.q_heads;
            a.kv_heads = d.kv_heads;
            a.group = d.q_heads / d.kv_heads;
            a.n_splits = slot.n_splits;
            a.chunk_cap = slot.chunk_cap;
            a.cluster = slot.attn_cluster;
            a.early = l > 0 ? 1 : 0;       // layer 0 follows the sampler's state update: wait first
            a.max_tokens = slot.max_tokens;
            a.scale = 1.0f / sqrtf((float)D);
            a.part_o = c.attn_part_o;
            a.part_ml = c.attn_part_ml;
            a.counters = c.attn_counters;
            launch_decode_attention(L, a, D);
        }
        {
            GemvParams p = base_gemv(w.o, H, c.o_k);
            p.xf = c.attn_d;
            p.residual = c.resid_d;
            launch_decode_gemv<Epi::Residual>(c, L, p, &w.w4_o);
        }
        {
            GemvParams p = base_gemv(w.gate_up, 2 * I, H);
            p.prologue = kProRmsNorm;
            p.xr = c.resid_d;
            p.norm_w = w.post_norm;
            p.eps = d.rms_eps;
            p.yf = c.act_d;
            launch_decode_gemv<Epi::SwiGlu>(c, L, p, &w.w4_gate_up, I);
        }
        {
            GemvParams p = base_gemv(w.down, H, I);
            p.xf = c.act_d;
            p.residual = c.resid_d;
            launch_decode_gemv<Epi::Residual>(c, L, p, &w.w4_down);
        }
    }
    launch_lm_head_and_sample(c, L, c.resid_d, /*advance=*/1, /*decode_pass=*/true);
}

template <int D>
static void launch_sage_d(Launcher& L, const SageAttnParams& p) {
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(sage_attention_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sg::smem_bytes<D>());
        attr_set = true;
    }
    L.launch(sage_attention_kernel<D>, dim3((p.S + sg::BQ - 1) / sg::BQ, p.q_heads), dim3(sg::kThreads), sg::smem_bytes<D>(), p);
}

void launch_sage_prefill_attention(Launcher& L, const SageScratch& sc, const __nv_bfloat16* q, const __nv_bfloat16* k,
                                   const __nv_bfloat16* v, __nv_bfloat16* out, int S, int kv_offset, int q_heads,
                                   int kv_heads, int D, int* error) {
    const int T = kv_offset + S;
    if (S <= 0) return;
    if ((D != 128 && D != 64) || S > sc.q_rows || T > sc.kv_rows) {
        if (L.err == cudaSuccess) L.err = cudaErrorInvalidValue;
        return;
    }
    const bool pdl = L.pdl;
    L.pdl = false;
    const int kvw = kv_heads * D, qw = q_heads * D;
    const int nkb = (T + kSageBlock - 1) / kSageBlock;
    L.launch(sage_ksum_kernel, dim3(nkb, kv_heads), dim3(512), 0, k, kvw, T, kv_heads, D, sc.kmean);
    const dim3 gk(nkb, kv_heads), gq((S + kSageBlock - 1) / kSageBlock, q_heads);
    if (D == 128) {
        L.launch(sage_quant_kernel<128>, gk, dim3(512), 0, k, kvw, T, kv_heads, (const float*)sc.kmean, nkb, sc.k8, sc.sk);
        L.launch(sage_quant_kernel<128>, gq, dim3(512), 0, q, qw, S, q_heads, (const float*)nullptr, 0, sc.q8, sc.sq);
    } else {
        L.launch(sage_quant_kernel<64>, gk, dim3(512), 0, k, kvw, T, kv_heads, (const float*)sc.kmean, nkb, sc.k8, sc.sk);
        L.launch(sage_quant_kernel<64>, gq, dim3(512), 0, q, qw, S, q_heads, (const float*)nullptr, 0, sc.q8, sc.sq);
    }
    L.launch(sage_to_half_kernel, dim3(std::min(((size_t)T * kvw / 2 + 255) / 256, (size_t)L.num_sms * 8)), dim3(256), 0, v, kvw, T,
             kvw, static_cast<__half*>(sc.vh));
    if (D == 128 && attention_tc_enabled()) {
        // tcgen05 form: Qi8 . Ki8^T as kind::i8 into TMEM, P . V in fp16 (attention_tc.cuh, I8 variant)
        using C = at::Cfg<128, true>;
        static bool attr_set = false;
        if (!attr_set) {
            cudaFuncSetAttribute(seg_attention_tc_kernel<128, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM);
            attr_set = true;
        }
        CUtensorMap mq, mk, mv;
        const uint64_t qd[3] = {128, (uint64_t)q_heads, (uint64_t)S}, qs[2] = {128, (uint64_t)q_heads * 128};
        const uint64_t kd[3] = {128, (uint64_t)kv_heads, (uint64_t)T}, ks[2] = {128, (uint64_t)kv_heads * 128};
        const uint64_t vd[3] = {128, (uint64_t)kv_heads, (uint64_t)T}, vs[2] = {256, (uint64_t)kv_heads * 256};
        const uint32_t qb[3] = {128, 1, (uint32_t)at::BM}, kb[3] = {128, 1, (uint32_t)at::BN}, vb[3] = {64, 1, (uint32_t)at::BN};
        if (make_map_nd(&mq, sc.q8, 3, qd, qs, qb, CU_TENSOR_MAP_DATA_TYPE_UINT8) && make_map_nd(&mk, sc.k8, 3, kd, ks, kb, CU_TENSOR_MAP_DATA_TYPE_UINT8) &&
            make_map_nd(&mv, sc.vh, 3, vd, vs, vb, CU_TENSOR_MAP_DATA_TYPE_FLOAT16)) {
            SegAttnParams a{};
            a.out = out; a.out_stride = q_heads * D;
            a.S = S; a.kv_offset = kv_offset; a.q_heads = q_heads; a.kv_heads = kv_heads; a.kv_rows = T;
            a.scale = 1.0f / sqrtf((float)D);
            a.sq = sc.sq; a.sk = sc.sk; a.error = error;
            L.launch(seg_attention_tc_kernel<128, true>, dim3((S + at::BM - 1) / at::BM, q_heads), dim3(at::kThreads), C::SMEM, mq, mk, mv, a, error);
            L.pdl = pdl;
            return;
        }
    }
    SageAttnParams p{};
    p.q = sc.q8; p.k = sc.k8; p.v = static_cast<const __half*>(sc.vh); p.sq = sc.sq; p.sk = sc.sk; p.out = out;
    p.S = S; p.kv_offset = kv_offset; p.q_heads = q_heads; p.kv_heads = kv_heads;
    p.scale = 1.0f / sqrtf((float)D);
    if (D == 128) launch_sage_d<128>(L, p); else launch_sage_d<64>(L, p);
    L.pdl = pdl;
}

void qwen_prefill_chunk(efm_b200_ctx& c, KvSlot& slot, int S, int kv_offset, int n_custom, int embed_token_id,
                        bool sample_last, Launcher& L) {
    const efm_model_desc& d = c.d;
    const int H = d.hidden, D = d.head_dim, QD = d.q_heads * D, KVD = d.kv_heads * D, I = d.intermediate;
    const bool pdl = L.pdl;
    L.pdl = false;
    launch_embed_rows(L, c.ids, c.embed, n_custom > 0 ? c.custom_embeds : nullptr, c.resid, S, d.vocab, H, embed_token_id, n_custom);
    for (int l = 0; l < d.num_layers; ++l) {
        const LayerWeights& w = c.layers[l];
        launch_rmsnorm_rows(L, c.resid, w.in_norm, c.norm, S, H, d.rms_eps);
        {
            GemmParams g{c.norm, w.qkv, w.qkv_bias, c.qkv, nullptr, S, QD + 2 * KVD, H};
            launch_gemm_epi(L, GemmEpi::Bf16Bias, g, &c.state->error);
        }
        L.launch(rope_scatter_kernel, dim3(S), dim3(256), 0,
                 (const __nv_bfloat16*)c.qkv, c.qbuf, slot.k[l], slot.v[l], (const float*)c.inv_freq,
                 (const int32_t*)c.pos3, S, d.q_heads, d.kv_heads, D, kv_offset, d.use_mrope, d.mrope_section[0],
                 d.mrope_section[0] + d.mrope_section[1]);
        if (c.prefill_attention_kind == 1)
            launch_sage_prefill_attention(L, c.sage, c.qbuf, slot.k[l], slot.v[l], c.attn, S, kv_offset, d.q_heads, d.kv_heads, D, &c.state->error);
        else
            launch_prefill_attention(L, c.qbuf, slot.k[l], slot.v[l], c.attn, S, kv_offset, d.q_heads, d.kv_heads, D, &c.state->error);
        if (c.tp_size == 1) {
            GemmParams g{c.attn, w.o, nullptr, nullptr, c.resid, S, H, QD};
            launch_gemm_epi(L, GemmEpi::Residual, g, &c.state->error);
        } else {      // row-parallel: this rank's input columns, fp32 partial, all-reduce, then the residual add
            GemmParams g{c.attn + (size_t)c.att_rep_idx * c.o_k, w.o, nullptr, nullptr, c.ybuf, S, H, c.o_k, QD};
            launch_gemm_epi(L, GemmEpi::F32, g, &c.state->error);
            tp_prefill_sum(c, L, S, 0);
        }
        launch_rmsnorm_rows(L, c.resid, w.post_norm, c.norm, S, H, d.rms_eps);
        {     // gate|up with silu(gate) * up in the epilogue
            GemmParams g{c.norm, w.gate_up, nullptr, c.act, nullptr, S, 2 * I, H};
            launch_gemm_epi(L, GemmEpi::SwiGlu, g, &c.state->error);
        }
        if (c.tp_size == 1) {
            GemmParams g{c.act, w.down, nullptr, nullptr, c.resid, S, H, I};
            launch_gemm_epi(L, GemmEpi::Residual, g, &c.state->error);
        } else {
            GemmParams g{c.act, w.down, nullptr, nullptr, c.ybuf, S, H, I};
            launch_gemm_epi(L, GemmEpi::F32, g, &c.state->error);
            tp_prefill_sum(c, L, S, 1);
        }
    }
    if (sample_last) launch_lm_head_and_sample(c, L, c.resid + (size_t)(S - 1) * H, /*advance=*/0, /*decode_pass=*/false);
    L.pdl = pdl;
}

}  // namespace efm

