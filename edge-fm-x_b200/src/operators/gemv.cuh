// Batch-1 weight-streaming GEMV for the decode step, with the neighbouring element-wise work
// fused in so that one launch replaces a chain of the reference's kernels:
//
//   prologue  Plain            x is read as is                      (o_proj, down_proj)
//             RmsNorm          x = rmsnorm(residual) * w, residual stream and x in fp32
//                                                                   (K2/K3 + K4 of the reference:
//                                                                    src/operators/norm_op.cu:20-106)
//             EmbedRmsNorm     residual = embed_table[token] first  (src/layers/embed_head.cu:22-61)
//   epilogue  Plain            y = bf16(W x)
//             Residual         r += W x, r kept in fp32             (fused add of norm_op.cu:64-106; the
//                              reference stores r in bf16, which costs ~2x in logit error on deep stacks)
//             QkvRope          + bias, rotate-half RoPE / M-RoPE on q and k, append k, v to the
//                              cache row kv_len-1                    (linear_impl.cu:90-106,
//                              decode_runtime_kernels.cu:67-225)
//             SwiGlu           act = bf16(silu(gate) * up)          (fused_gate_up_activation_op.cu:198-277)
//             Logits           fp32 logits + per-block (max, argmax) (src/layers/linear.cu:187-270)
//
// Bound: HBM.  One block of 16 warps per SM.  Each weight byte is read once, as 128-bit streaming
// loads.  A warp (or `ks` warps sharing one row pair) walks its rows in units of 8 x 2 loads: 16
// loads of 16 bytes in flight per lane, ~19 MB chip-wide, which is what it takes to cover the
// ~2 us loaded DRAM latency at full bandwidth (halving it to 8 measurably costs 20 %).  Activations
// live in shared memory as fp32 (a decode step rounds nothing to bf16 but the K / V rows it appends: with bf16
// activations the rounding noise of 28-36 layers alone exceeds a 2e-2 logit tolerance on the 3B / 7B shapes);
// dot products reduce with warp shuffles (and a named-barrier exchange
// when ks > 1).  The first unit and the norm weight are fetched BEFORE the dependency wait
// (griddepcontrol.wait, or the grid barrier of the persistent decode kernel), because weights
// do not depend on the previous phase.
#pragma once
#include "common.cuh"
#include "expert_route.cuh"

namespace efm {

enum class Epi : int { Plain = 0, Residual = 1, QkvRope = 2, SwiGlu = 3, Logits = 4, Peers = 5, Store32 = 6, TokenGate = 7, ExpertUp = 8, ExpertDown = 9, Router = 10, Store32Bias = 11, Relu2 = 12 };
constexpr int kMaxPeers = 8;
// Embed and what follows it (and the epilogues from Store32 on) exist in the EXT instantiations only (layered decoders; level 2 adds
// input norms: Norm, and the second norm and the scale of Embed; level 3 elementwise input norms, AddTanh and Merge, the clamped
// and the shared expert and the cap of the logits; level 4 input convolutions, the average over depth and experts without a gate):
//   Embed    x = embed_table[token] * embed_scale; with norm2_w the product reads rmsnorm(x) * norm2_w
//   Norm     x = rmsnorm(xf) * norm_w
//   AddNorm  x = xr + rmsnorm(addend) * norm_w: a sublayer whose OUTPUT is normalised, folded into the next product;
//            with norm2_w the product reads rmsnorm(x) * norm2_w instead of x
//   PolyNorm x = c0 rms(z) + c1 rms(z^2) + c2 rms(z^3) + c3 with z = xf and the four numbers of `poly`
//   AddTanh  x = xr + add_mult * addend; the product reads tanh(alpha x) * norm_w + norm_b (Embed does the same when norm_b is given)
//            level 4, Embed and AddNorm: with avg the stream is avg + avg_w x instead of x, with conv_w the product reads the stream plus
//            its convolution over the last conv_taps tokens
//   Merge    channels [0, merge0) of xf as they are, the others rmsnorm(xf) * norm_w * sigmoid(merge_gate) * merge_scale
enum : int { kProPlain = 0, kProRmsNorm = 1, kProEmbedRmsNorm = 2, kProEmbed = 3, kProAddNorm = 4, kProPolyNorm = 5, kProNorm = 6, kProAddTanh = 7, kProMerge = 8 };

struct GemvParams {
    const __nv_bfloat16* W;   // [N, K] row-major
    int N, K, n_items;        // n_items = N / 2 (every epilogue consumes rows in pairs)
    // prologue
    int prologue;
    const __nv_bfloat16* x;   // Plain: activations [K] bf16 ...
    const float* xf;          // ... or, when non-null, fp32 (the decode step's own activations)
    const float* xr;          // norm prologues: residual stream [K] fp32
    const __nv_bfloat16* norm_w;
    float eps;
    const __nv_bfloat16* embed_table;
    int vocab;
    float* resid_out;         // EmbedRmsNorm / addend: block 0 stores the (updated) residual row here
    const float* addend;      // norm prologues, tensor parallel: x = x + addend first (summed partial output of
                              // the previous row-parallel linear); resid_out must differ from xr
    DecodeState* state;
    // epilogue
    __nv_bfloat16* y;         // Plain: [N]; SwiGlu: [N/2] ...
    float* yf;                // ... or, when non-null, SwiGlu output in fp32
    float* residual;          // Residual: [N] fp32 in/out
    const __nv_bfloat16* bias;
    __nv_bfloat16* q_out;     // QkvRope: rotated q in bf16 (q, k, v rounded to bf16 before the rotation as the prefill does) ...
    float* q_out_f;           // ... or, when non-null, in fp32: then nothing is rounded but the K / V rows written to the cache
    __nv_bfloat16* k_cache;
    __nv_bfloat16* v_cache;
    const float* inv_freq;
    int q_heads, kv_heads, head_dim, use_mrope, sec0, sec1, max_tokens;
    float* logits;            // Logits
    float* part_val;
    int* part_idx;
    // Peers (tensor parallel, row-parallel linear fused with its exchange): every output value travels as one
    // 8-byte word {fp32 value, exchange count} stored into this rank's row of EVERY rank's receive buffer (peer
    // memory over NVLink, own buffer included).  Value and count arrive together, so there is no fence and no
    // separate flag; the last block to finish bumps the local count (local atomics only).
    uint2* peer_out[kMaxPeers];
    int n_peers;
    unsigned int* epoch;      // local: number of exchanges completed by this rank
    unsigned int* ticket;     // local: block ticket, zero between launches
    // consumer side (norm prologues): x = x + sum over ranks, in rank order, of parts[r][:], every word being
    // re-read (bounded) until it carries the local count
    const uint2* addend_parts;            // local receive buffer [n_parts][K] of {value, count}
    int n_parts;
    int* error;               // raised (3) when a wait gives up
    volatile int* error_host; // optional mirror of `error` in mapped host memory (the host stops queueing steps)
    unsigned long long wait_ns;   // total wait budget of one kernel; 0 = kPeerWaitDefaultNs
    unsigned int want_override;   // != 0: wait for this count instead of *epoch (single-GPU test of the wait)
    // EXT instantiations.  Rows are padded to K (a multiple of 8) with zeros; means divide by k_true.
    int k_true;
    const __nv_bfloat16* norm2_w;
    const __nv_bfloat16* poly;
    float* out_f;             // Store32, TokenGate: [2 * n_items]
    // TokenGate: out[n] = gelu_tanh(W x)[n] * gate_table[token][gate_off + n] for n < N, 0 beyond
    const __nv_bfloat16* gate_table;
    int gate_ld, gate_off;
    float embed_scale;
    float* x_out;             // not null: block 0 stores the input of the product here (what the norms left)
    // Router: out_f = logits; the block that finishes last chooses this token's experts and publishes ids and weights.
    // ExpertUp: item = (choice, channel), out_f[choice * ffp + channel] = silu(gate) * up.  ExpertDown: x = the choices'
    // activations times their weights, K = choices * ffp, the row of W jumps from expert to expert.
    RouteShape route;
    unsigned int* route_ticket;           // zero between launches
    int32_t* route_id;        // [top]
    float* route_w;           // [top]
    int ff, ffp, expert_rows; // channels, padded channels, rows of one expert's matrix
    // level 3
    const __nv_bfloat16* norm_b;
    const __nv_bfloat16* norm_alpha;      // one number
    float add_mult;
    int merge0;
    const float* merge_gate;
    float merge_scale;
    float logit_scale, logit_softcap;     // Logits: softcap * tanh(logit_scale * z / softcap); softcap 0: logit_scale * z
    // ExpertUp / ExpertDown: the gated unit's form; a shared expert behind the chosen ones (rows of W2, activations behind theirs,
    // weight at route_w[top])
    int glu, weight_input;
    float limit, shared_limit;
    const __nv_bfloat16* W2;
    int shared_ff, shared_ffp;
    // level 4.  Relu2 experts: item = (choice, pair of channels), ff and shared_ff count pairs.
    // conv_ring: [conv_taps][K], the stream's earlier values by position modulo conv_taps; block 0 adds this token's.  conv_early: what
    // earlier steps left (and the device state) may be read before the dependency wait
    const __nv_bfloat16* conv_w;          // [conv_taps][K], null: none
    float* conv_ring;
    int conv_taps, conv_early;
    const float* avg;                     // [K], null: none
    const __nv_bfloat16* avg_w;           // one number
    float* hist_out;                      // not null: block 0 stores the layer's result (Embed: the embedding) here
    // a product that runs meanwhile prepares avg for the next one: sum_out = sum_{j < sum_n} sum_w[j] sum_in[j], rows of sum_k numbers
    const float* sum_in;
    const __nv_bfloat16* sum_w;
    float* sum_out;
    int sum_n, sum_k;
};

// gated units: silu(g) u, or (clamped) g sigmoid(1.702 g) (u + 1) with g at most and u within +- limit
enum : int { kGluSilu = 0, kGluClamped = 1, kGluRelu2 = 2 };       // Relu2: no gate, the square of relu
__device__ __forceinline__ float relu2(float z) {
    z = fmaxf(z, 0.f);
    return z * z;
}
__device__ __forceinline__ float glu(int kind, float g, float u, float limit) {
    if (kind == kGluSilu) return g / (1.0f + expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}
__device__ __forceinline__ float cap_logit(float z, float scale, float softcap) {
    z *= scale;
    return softcap > 0.f ? softcap * tanhf(z / softcap) : z;
}

__device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// One {value, count} word is ONE 64-bit element (value in the low half), so that value and count are read and
// written together by the memory model's own rule (a 64-bit access is single-copy atomic), not by the accident
// of how a 16-byte store travels.  Two words per access; relaxed, system scope: the consumer needs no ordering
// between words, only each word whole.
__device__ __forceinline__ void ld_peer_words(const uint2* p, unsigned long long& w0, unsigned long long& w1) {
    asm volatile("ld.relaxed.sys.global.v2.b64 {%0,%1}, [%2];" : "=l"(w0), "=l"(w1) : "l"(p) : "memory");
}
__device__ __forceinline__ void st_peer_words(uint2* p, unsigned long long w0, unsigned long long w1) {
    asm volatile("st.relaxed.sys.global.v2.b64 [%0], {%1,%2};" ::"l"(p), "l"(w0), "l"(w1) : "memory");
}
__device__ __forceinline__ unsigned long long peer_word(float v, unsigned int count) {
    return (unsigned long long)__float_as_uint(v) | ((unsigned long long)count << 32);
}
__device__ __forceinline__ void group_barrier(int id, int nthreads) {
    asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(nthreads) : "memory");
}

template <Epi EPI, int EXT = 0>
__device__ __forceinline__ void item_rows(const GemvParams& p, int item, int& r0, int& r1, const int* chosen = nullptr) {
    (void)chosen;
    if constexpr (EPI == Epi::QkvRope) {
        const int half = p.head_dim >> 1;
        const int head = item / half, d = item - head * half;
        r0 = head * p.head_dim + d;
        r1 = r0 + half;
    } else if constexpr (EPI == Epi::SwiGlu) {
        // fused weight: blocks of 64 gate rows followed by the 64 matching up rows
        r0 = ((item >> 6) << 7) + (item & 63);
        r1 = r0 + 64;
    } else if constexpr (EPI == Epi::ExpertUp) {
        const int k = item / p.ff, j = item - (EXT > 2 && k >= p.route.top ? p.route.top : k) * p.ff;
        if constexpr (EXT > 3) {
            if (p.glu == kGluRelu2) {
                r0 = (k >= p.route.top ? 0 : chosen[k] * p.expert_rows) + 2 * j;
                r1 = r0 + 1;
                return;
            }
        }
        r0 = (EXT > 2 && k >= p.route.top ? 0 : chosen[k] * p.expert_rows) + ((j >> 6) << 7) + (j & 63);
        r1 = r0 + 64;
    } else {
        r0 = item * 2;
        r1 = r0 + 1;
    }
}

template <Epi EPI, int EXT = 0>
__device__ __forceinline__ void item_epilogue(const GemvParams& p, int item, float a0, float a1,
                                              float& best_v, int& best_i, const int* chosen = nullptr) {
    (void)chosen;
    if constexpr (EPI == Epi::Plain) {
        p.y[item * 2] = __float2bfloat16_rn(a0);
        p.y[item * 2 + 1] = __float2bfloat16_rn(a1);
    } else if constexpr (EPI == Epi::Residual) {
        // L2 load: inside the persistent decode kernel another block wrote this value
        const float2 old = __ldcg(reinterpret_cast<const float2*>(p.residual + item * 2));
        *reinterpret_cast<float2*>(p.residual + item * 2) = make_float2(old.x + a0, old.y + a1);
    } else if constexpr (EPI == Epi::SwiGlu) {
        const float s = a0 / (1.0f + expf(-a0));
        if (p.yf != nullptr) p.yf[item] = s * a1;
        else p.y[item] = __float2bfloat16_rn(s * a1);
    } else if constexpr (EPI == Epi::Peers) {
        const unsigned int e = (unsigned int)best_i;           // exchange count of this launch (see gemv_kernel)
        const unsigned long long w0 = peer_word(a0, e), w1 = peer_word(a1, e);
#pragma unroll
        for (int r = 0; r < kMaxPeers; ++r)
            if (r < p.n_peers) st_peer_words(p.peer_out[r] + item * 2, w0, w1);
    } else if constexpr (EPI == Epi::Logits) {
        if constexpr (EXT > 2) {
            a0 = cap_logit(a0, p.logit_scale, p.logit_softcap);
            a1 = cap_logit(a1, p.logit_scale, p.logit_softcap);
        }
        *reinterpret_cast<float2*>(p.logits + item * 2) = make_float2(a0, a1);
        if (item * 2 >= p.N) a0 = -INFINITY;                          // padding rows
        if (item * 2 + 1 >= p.N) a1 = -INFINITY;
        if (a0 > best_v) { best_v = a0; best_i = item * 2; }          // ascending ids: strict > keeps
        if (a1 > best_v) { best_v = a1; best_i = item * 2 + 1; }      // the lowest id on ties
    } else if constexpr (EPI == Epi::ExpertUp) {
        const int k = item / p.ff;
        if constexpr (EXT > 3) {
            if (p.glu == kGluRelu2) {
                const int k2 = min(k, p.route.top);
                *reinterpret_cast<float2*>(p.out_f + k2 * p.ffp + 2 * (item - k2 * p.ff)) = make_float2(relu2(a0), relu2(a1));
                return;
            }
        }
        if constexpr (EXT > 2) {
            const bool shared = k >= p.route.top;
            const float w = !shared && p.weight_input ? __int_as_float(chosen[kMaxExpertTop + k]) : 1.0f;      // a product is linear in its input
            p.out_f[shared ? p.route.top * p.ffp + item - p.route.top * p.ff : k * p.ffp + item - k * p.ff] =
                glu(p.glu, a0 * w, a1 * w, shared ? p.shared_limit : p.limit);
        } else {
            p.out_f[k * p.ffp + item - k * p.ff] = a0 / (1.0f + expf(-a0)) * a1;
        }
    } else if constexpr (EPI == Epi::ExpertDown) {
        *reinterpret_cast<float2*>(p.out_f + item * 2) = make_float2(a0, a1);
    } else if constexpr (EPI == Epi::Router) {
        __stcg(reinterpret_cast<float2*>(p.out_f + item * 2), make_float2(a0, a1));
    } else if constexpr (EPI == Epi::Store32Bias) {
        *reinterpret_cast<float2*>(p.out_f + item * 2) = make_float2(a0 + __bfloat162float(p.bias[item * 2]), a1 + __bfloat162float(p.bias[item * 2 + 1]));
    } else if constexpr (EPI == Epi::Relu2) {
        *reinterpret_cast<float2*>(p.out_f + item * 2) = make_float2(relu2(a0), relu2(a1));
    } else if constexpr (EPI == Epi::Store32) {
        *reinterpret_cast<float2*>(p.out_f + item * 2) = make_float2(a0, a1);
    } else if constexpr (EPI == Epi::TokenGate) {
        const int n = item * 2, tok = p.state->token;
        const bool ok = tok >= 0 && tok < p.vocab;
        const __nv_bfloat16* e = p.gate_table + (size_t)(ok ? tok : 0) * p.gate_ld + p.gate_off + n;
        p.out_f[n] = ok && n < p.N ? gelu_tanh(a0) * __bfloat162float(e[0]) : 0.f;
        p.out_f[n + 1] = ok && n + 1 < p.N ? gelu_tanh(a1) * __bfloat162float(e[1]) : 0.f;
    } else {  // QkvRope
        const int D = p.head_dim, half = D >> 1;
        const int head = item / half, d = item - head * half;
        int r0 = head * D + d, r1 = r0 + half;
        float y0 = a0, y1 = a1;
        if (p.bias != nullptr) {
            y0 += __bfloat162float(p.bias[r0]);
            y1 += __bfloat162float(p.bias[r1]);
        }
        const bool full = p.q_out_f != nullptr;
        if (!full) {
            y0 = round_bf16(y0);
            y1 = round_bf16(y1);
        }
        const uint32_t kv_len = p.state->kv_len;
        if (kv_len == 0 || kv_len > (uint32_t)p.max_tokens) {
            p.state->error = 1;   // refuse the out-of-range cache row instead of faulting
            return;
        }
        const size_t row = (size_t)(kv_len - 1) * p.kv_heads * D;
        if (head < p.q_heads + p.kv_heads) {
            int pos;
            if (p.use_mrope) pos = p.state->pos[d < p.sec0 ? 0 : (d < p.sec1 ? 1 : 2)];
            else pos = (int)kv_len - 1;
            float sn, cs;
            sincosf((float)pos * p.inv_freq[d], &sn, &cs);
            const float o0 = y0 * cs - y1 * sn, o1 = y1 * cs + y0 * sn;
            if (head < p.q_heads) {
                if (full) {
                    p.q_out_f[r0] = o0;
                    p.q_out_f[r1] = o1;
                } else {
                    p.q_out[r0] = __float2bfloat16_rn(o0);
                    p.q_out[r1] = __float2bfloat16_rn(o1);
                }
            } else {
                const int kh = head - p.q_heads;
                p.k_cache[row + kh * D + d] = __float2bfloat16_rn(o0);
                p.k_cache[row + kh * D + d + half] = __float2bfloat16_rn(o1);
            }
        } else {
            const int vh = head - p.q_heads - p.kv_heads;
            p.v_cache[row + vh * D + d] = __float2bfloat16_rn(y0);
            p.v_cache[row + vh * D + d + half] = __float2bfloat16_rn(y1);
        }
    }
}

constexpr int kGemvThreads = 512, kGemvWarps = 16, kGemvU = 8;

struct GemvRegs { uint4 a[kGemvU][2]; };

// Per-thread view of the static schedule: which row pairs (items) this warp group walks and in
// how many units.
struct GemvSched {
    int ks, gi, wk, gl, stride, nch, upi, ig0, ig_stride, total;
};

__device__ __forceinline__ GemvSched gemv_sched(const GemvParams& p, const int ks, const int block, const int n_blocks) {
    GemvSched sc;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int gp = kGemvWarps / ks;
    sc.ks = ks;
    sc.gi = warp / ks;
    sc.wk = warp % ks;
    sc.gl = sc.wk * 32 + lane;
    sc.stride = ks * 32;
    sc.nch = p.K >> 3;
    const int cpl = (sc.nch + sc.stride - 1) / sc.stride;        // chunks per lane and row
    sc.upi = (cpl + kGemvU - 1) / kGemvU;                         // units per item
    sc.ig0 = block * gp + sc.gi;
    sc.ig_stride = n_blocks * gp;
    const int n_my = sc.ig0 < p.n_items ? (p.n_items - sc.ig0 + sc.ig_stride - 1) / sc.ig_stride : 0;
    sc.total = n_my * sc.upi;
    return sc;
}

template <Epi EPI, int EXT = 0>
__device__ __forceinline__ void gemv_load_unit(const GemvParams& p, const GemvSched& sc, const int u, uint4 (&buf)[kGemvU][2], const int* chosen = nullptr) {
    if (u >= sc.total) return;
    const int j = u / sc.upi, part = u - j * sc.upi;
    int r0, r1;
    item_rows<EPI, EXT>(p, sc.ig0 + j * sc.ig_stride, r0, r1, chosen);
    if constexpr (EPI == Epi::ExpertDown) {
        const int per = p.ffp >> 3;                                   // chunks of one expert's row
        const float inv = 1.0f / (float)per;                           // c / per exactly: half a chunk is far above the rounding
        const __nv_bfloat16* w[kGemvU];                                // all addresses first: the loads then leave back to back
        int ld[kGemvU];
#pragma unroll
        for (int uu = 0; uu < kGemvU; ++uu) {
            const int c = min((part * kGemvU + uu) * sc.stride + sc.gl, sc.nch - 1), k = (int)(((float)c + 0.5f) * inv);
            ld[uu] = p.ffp;
            if (EXT > 2 && c >= p.route.top * per) {
                ld[uu] = p.shared_ffp;
                w[uu] = p.W2 + (size_t)r0 * p.shared_ffp + (size_t)(c - p.route.top * per) * 8;
            } else {
                w[uu] = p.W + ((size_t)chosen[k] * p.expert_rows + r0) * p.ffp + (size_t)(c - k * per) * 8;
            }
        }
#pragma unroll
        for (int uu = 0; uu < kGemvU; ++uu)
            if ((part * kGemvU + uu) * sc.stride + sc.gl < sc.nch) {
                buf[uu][0] = ld_stream(w[uu]);
                buf[uu][1] = ld_stream(w[uu] + ld[uu]);
            }
        return;
    }
    const __nv_bfloat16* W = p.W;
    if constexpr (EPI == Epi::ExpertUp && EXT > 2) {
        if (sc.ig0 + j * sc.ig_stride >= p.route.top * p.ff) W = p.W2;
    }
    const __nv_bfloat16* a = W + (size_t)r0 * p.K;
    const __nv_bfloat16* b = W + (size_t)r1 * p.K;
#pragma unroll
    for (int uu = 0; uu < kGemvU; ++uu) {
        const int c = (part * kGemvU + uu) * sc.stride + sc.gl;
        if (c < sc.nch) {
            buf[uu][0] = ld_stream(a + (size_t)c * 8);
            buf[uu][1] = ld_stream(b + (size_t)c * 8);
        }
    }
}

// Shared memory of one GEMV phase: [xs: fp32 K][norm weight: bf16 K][red: 2 x 16 x 2 floats][misc: 16 floats].
__host__ __device__ inline unsigned int gemv_xbytes(int K) { return ((unsigned int)K * 4u + 15u) & ~15u; }
__host__ __device__ inline unsigned int gemv_wbytes(int K) { return ((unsigned int)K * 2u + 15u) & ~15u; }

// Offset of the second staged vector of the EXT prologues (behind red + misc).
__host__ __device__ inline unsigned int gemv_ext_off(int K) { return gemv_xbytes(K) + gemv_wbytes(K) + (2 * 16 * 2 + 16) * 4u; }

// Behind that, with an input convolution: what the earlier tokens contribute (fp32 K), the weight of the token itself (bf16 K).
__host__ __device__ inline unsigned int gemv_conv_off(int K) { return gemv_ext_off(K) + gemv_xbytes(K); }

template <int EXT>
__device__ __forceinline__ void gemv_stage_conv(const GemvParams& p, const int nch, unsigned char* smem) {
    float* past = reinterpret_cast<float*>(smem + gemv_conv_off(p.K));
    uint4* own = reinterpret_cast<uint4*>(smem + gemv_conv_off(p.K) + gemv_xbytes(p.K));
    const int taps = p.conv_taps, pos = (int)p.state->kv_len - 1;
    for (int c = threadIdx.x; c < nch; c += kGemvThreads) {
        float a[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        own[c] = ld_cached(p.conv_w + (size_t)(taps - 1) * p.K + 8 * c);
        for (int back = 1; back < taps && back <= pos; ++back) {
            float w[8];
            unpack8(ld_cached(p.conv_w + (size_t)(taps - 1 - back) * p.K + 8 * c), w);
            const float4* h = reinterpret_cast<const float4*>(p.conv_ring + (size_t)((pos - back) % taps) * p.K + 8 * c);
            const float4 x = __ldcg(h), y = __ldcg(h + 1);
            a[0] = fmaf(w[0], x.x, a[0]); a[1] = fmaf(w[1], x.y, a[1]); a[2] = fmaf(w[2], x.z, a[2]); a[3] = fmaf(w[3], x.w, a[3]);
            a[4] = fmaf(w[4], y.x, a[4]); a[5] = fmaf(w[5], y.y, a[5]); a[6] = fmaf(w[6], y.z, a[6]); a[7] = fmaf(w[7], y.w, a[7]);
        }
        *reinterpret_cast<float4*>(past + 8 * c) = make_float4(a[0], a[1], a[2], a[3]);
        *reinterpret_cast<float4*>(past + 8 * c + 4) = make_float4(a[4], a[5], a[6], a[7]);
    }
}

// Weights only: the first two units into registers, the norm weight into shared memory.
template <Epi EPI, int EXT>
__device__ __forceinline__ void gemv_prefetch(const GemvParams& p, const GemvSched& sc, GemvRegs& r, unsigned char* smem,
                                              const unsigned int xbytes) {
    if constexpr (EPI != Epi::ExpertUp && EPI != Epi::ExpertDown) gemv_load_unit<EPI, EXT>(p, sc, 0, r.a);
    if (EXT ? (p.prologue == kProAddNorm || (EXT > 1 && p.prologue == kProNorm) || (EXT > 2 && p.prologue == kProAddTanh)) : p.prologue != kProPlain) {
        uint4* gs = reinterpret_cast<uint4*>(smem + xbytes);        // xbytes = gemv_xbytes(K)
        for (int c = threadIdx.x; c < sc.nch; c += kGemvThreads) gs[c] = ld_cached(p.norm_w + (size_t)c * 8);
        if constexpr (EXT > 2) {
            uint4* bs = reinterpret_cast<uint4*>(smem + gemv_ext_off(p.K));
            if (p.prologue == kProAddTanh)
                for (int c = threadIdx.x; c < sc.nch; c += kGemvThreads) bs[c] = ld_cached(p.norm_b + (size_t)c * 8);
        }
    }
    if constexpr (EXT > 2) {
        if (p.prologue == kProMerge) {
            uint4* gs = reinterpret_cast<uint4*>(smem + xbytes);
            for (int c = threadIdx.x; c < sc.nch - p.merge0 / 8; c += kGemvThreads) gs[c] = ld_cached(p.norm_w + (size_t)c * 8);
        }
    }
    if constexpr (EXT > 3) {
        if (p.conv_w != nullptr && p.conv_early) gemv_stage_conv<EXT>(p, sc.nch, smem);
        // the rows of the sum are complete: their writers ran before the product this launch may overlap with
        if (p.sum_n > 0) {
            const int n4 = p.sum_k / 4, per = (n4 + (int)gridDim.x - 1) / (int)gridDim.x;
            for (int i = threadIdx.x; i < per; i += kGemvThreads) {
                const int c = (int)blockIdx.x * per + i;
                if (c >= n4) break;
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
                for (int j = 0; j < p.sum_n; ++j) {
                    const float4 v = __ldcg(reinterpret_cast<const float4*>(p.sum_in + (size_t)j * p.sum_k) + c);
                    const float w = __bfloat162float(p.sum_w[j]);
                    a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
                }
                reinterpret_cast<float4*>(p.sum_out)[c] = a;
            }
        }
    }
}

// Sums of N per-thread values over the block (all threads get them); red: N x kGemvWarps floats, free on return only after
// the next block barrier.
template <int N>
__device__ __forceinline__ void gemv_block_sums(float (&v)[N], float* red) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        v[i] = warp_sum(v[i]);
        if (lane == 0) red[i * kGemvWarps + warp] = v[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) {
        v[i] = 0.f;
#pragma unroll
        for (int w = 0; w < kGemvWarps; ++w) v[i] += red[i * kGemvWarps + w];
    }
}
__device__ __forceinline__ void ld8f(const float* p, float (&f)[8]) {
    const float4 lo = __ldcg(reinterpret_cast<const float4*>(p)), hi = __ldcg(reinterpret_cast<const float4*>(p) + 1);
    f[0] = lo.x; f[1] = lo.y; f[2] = lo.z; f[3] = lo.w; f[4] = hi.x; f[5] = hi.y; f[6] = hi.z; f[7] = hi.w;
}
__device__ __forceinline__ void st8f(float* p, const float (&f)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

// EXT prologues; false: not one of them.  Ends with a block barrier.
template <int EXT>
__device__ __forceinline__ bool gemv_stage_ext(const GemvParams& p, const int nch, unsigned char* smem, const unsigned int xbytes) {
    __shared__ float red3[3 * kGemvWarps];
    float* xs = reinterpret_cast<float*>(smem);
    const int tid = threadIdx.x;
    float sq[1] = {0.f};
    // the second norm: the product reads rmsnorm(x) * norm2_w
    auto norm2 = [&](float (&s2)[1]) {
        gemv_block_sums<1>(s2, red3 + kGemvWarps);
        const float inv2 = 1.0f / sqrtf(s2[0] / (float)p.k_true + p.eps);
        for (int c = tid; c < nch; c += kGemvThreads) {
            float w[8], x[8];
            unpack8(ld_cached(p.norm2_w + (size_t)c * 8), w);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = xs[8 * c + j] * inv2 * w[j];
            st8f(xs + 8 * c, x);
            if (EXT > 1 && p.x_out != nullptr && blockIdx.x == 0) st8f(p.x_out + 8 * c, x);
        }
    };
    const float alpha = EXT > 2 && p.norm_alpha != nullptr ? __bfloat162float(*p.norm_alpha) : 0.f;
    auto tanh8 = [&](int c, float (&f)[8], const uint4& wv, const uint4& bv) {
        float w[8], b[8];
        unpack8(wv, w);
        unpack8(bv, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = tanh_norm(f[j], alpha, w[j], b[j]);
        if (p.x_out != nullptr && blockIdx.x == 0) st8f(p.x_out + 8 * c, f);
    };
    (void)tanh8;
    // level 4: x, the stream of chunk c, becomes what the product reads (same thread and chunk as in gemv_stage_conv)
    auto conv8 = [&](int c, float (&x)[8]) {
        const float* past = reinterpret_cast<const float*>(smem + gemv_conv_off(p.K)) + 8 * c;
        const uint4 wv = reinterpret_cast<const uint4*>(smem + gemv_conv_off(p.K) + gemv_xbytes(p.K))[c];
        float w[8];
        unpack8(wv, w);
        const int pos = (int)p.state->kv_len - 1;
        if (blockIdx.x == 0 && pos >= 0) st8f(p.conv_ring + (size_t)(pos % p.conv_taps) * p.K + 8 * c, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = x[j] + fmaf(w[j], x[j], past[j]);
        if (p.x_out != nullptr && blockIdx.x == 0) st8f(p.x_out + 8 * c, x);
    };
    (void)conv8;
    if constexpr (EXT > 3) {
        if (p.conv_w != nullptr && !p.conv_early) gemv_stage_conv<EXT>(p, nch, smem);
    }
    const float avg_w = EXT > 3 && p.avg != nullptr ? __bfloat162float(*p.avg_w) : 0.f;
    (void)avg_w;
    if (p.prologue == kProEmbed) {
        const int tok = p.state->token;
        const bool zero = tok < 0 || tok >= p.vocab;
        const __nv_bfloat16* row = p.embed_table + (size_t)(zero ? 0 : tok) * p.K;
        for (int c = tid; c < nch; c += kGemvThreads) {
            float f[8];
            unpack8(zero ? make_uint4(0, 0, 0, 0) : ld_cached(row + (size_t)c * 8), f);
            if constexpr (EXT > 1) {
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    f[j] *= p.embed_scale;
                    sq[0] = fmaf(f[j], f[j], sq[0]);
                }
            }
            if (blockIdx.x == 0) st8f(p.resid_out + 8 * c, f);
            if constexpr (EXT > 3) {
                if (p.hist_out != nullptr && blockIdx.x == 0) st8f(p.hist_out + 8 * c, f);
                if (p.conv_w != nullptr) conv8(c, f);
            }
            if constexpr (EXT > 2) {
                if (p.norm_b != nullptr) tanh8(c, f, ld_cached(p.norm_w + (size_t)c * 8), ld_cached(p.norm_b + (size_t)c * 8));
            }
            st8f(xs + 8 * c, f);
        }
        if constexpr (EXT > 1) {
            if (p.norm2_w != nullptr) norm2(sq);
        }
    } else if (EXT > 1 && p.prologue == kProNorm) {
        const uint4* gs = reinterpret_cast<const uint4*>(smem + xbytes);
        for (int c = tid; c < nch; c += kGemvThreads) {
            float f[8];
            ld8f(p.xf + 8 * c, f);
#pragma unroll
            for (int j = 0; j < 8; ++j) sq[0] = fmaf(f[j], f[j], sq[0]);
            st8f(xs + 8 * c, f);
        }
        gemv_block_sums<1>(sq, red3);
        const float inv = 1.0f / sqrtf(sq[0] / (float)p.k_true + p.eps);
        for (int c = tid; c < nch; c += kGemvThreads) {
            float w[8], x[8];
            unpack8(gs[c], w);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = xs[8 * c + j] * inv * w[j];
            st8f(xs + 8 * c, x);
        }
    } else if (EXT > 2 && p.prologue == kProAddTanh) {
        const uint4 *gs = reinterpret_cast<const uint4*>(smem + xbytes), *bs = reinterpret_cast<const uint4*>(smem + gemv_ext_off(p.K));
        for (int c = tid; c < nch; c += kGemvThreads) {       // same thread, same chunks as in the prefetch
            float y[8], x[8];
            ld8f(p.addend + 8 * c, y);
            ld8f(p.xr + 8 * c, x);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = fmaf(p.add_mult, y[j], x[j]);
            if (blockIdx.x == 0) st8f(p.resid_out + 8 * c, x);
            tanh8(c, x, gs[c], bs[c]);
            st8f(xs + 8 * c, x);
        }
    } else if (EXT > 2 && p.prologue == kProMerge) {
        const uint4* gs = reinterpret_cast<const uint4*>(smem + xbytes);
        float* xs2 = reinterpret_cast<float*>(smem + gemv_ext_off(p.K));
        const int c0 = p.merge0 / 8;
        for (int c = tid; c < c0; c += kGemvThreads) {
            float x[8];
            ld8f(p.xf + 8 * c, x);
            st8f(xs + 8 * c, x);
        }
        for (int c = tid; c < nch - c0; c += kGemvThreads) {
            float x[8], g[8], w[8];
            ld8f(p.xf + 8 * (c0 + c), x);
            ld8f(p.merge_gate + 8 * c, g);
            unpack8(gs[c], w);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                if (8 * c + j >= p.k_true) x[j] = 0.f;                // pads
                sq[0] = fmaf(x[j], x[j], sq[0]);
                g[j] = w[j] / (1.0f + expf(-g[j]));
            }
            st8f(xs + 8 * (c0 + c), x);
            st8f(xs2 + 8 * c, g);
        }
        gemv_block_sums<1>(sq, red3);
        const float inv = p.merge_scale / sqrtf(sq[0] / (float)p.k_true + p.eps);
        for (int c = tid; c < nch - c0; c += kGemvThreads) {
            float* x = xs + 8 * (c0 + c);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] *= inv * xs2[8 * c + j];
        }
    } else if (p.prologue == kProAddNorm) {
        const uint4* gs = reinterpret_cast<const uint4*>(smem + xbytes);
        float* xs2 = reinterpret_cast<float*>(smem + gemv_ext_off(p.K));
        float ss[1] = {0.f};
        for (int c = tid; c < nch; c += kGemvThreads) {
            float y[8], x[8];
            ld8f(p.addend + 8 * c, y);
            ld8f(p.xr + 8 * c, x);
#pragma unroll
            for (int j = 0; j < 8; ++j) ss[0] = fmaf(y[j], y[j], ss[0]);
            st8f(xs + 8 * c, y);
            st8f(xs2 + 8 * c, x);
        }
        gemv_block_sums<1>(ss, red3);
        const float inv = 1.0f / sqrtf(ss[0] / (float)p.k_true + p.eps);
        float s2[1] = {0.f};
        for (int c = tid; c < nch; c += kGemvThreads) {       // same thread, same chunks as above
            float w[8], x[8];
            unpack8(gs[c], w);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = xs2[8 * c + j] + xs[8 * c + j] * inv * w[j];
            if constexpr (EXT > 3) {
                if (p.hist_out != nullptr && blockIdx.x == 0) st8f(p.hist_out + 8 * c, x);
                if (p.avg != nullptr) {
                    float a[8];
                    ld8f(p.avg + 8 * c, a);
#pragma unroll
                    for (int j = 0; j < 8; ++j) x[j] = fmaf(avg_w, x[j], a[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) s2[0] = fmaf(x[j], x[j], s2[0]);
            if (blockIdx.x == 0) st8f(p.resid_out + 8 * c, x);
            if constexpr (EXT > 3) {
                if (p.conv_w != nullptr) conv8(c, x);
            }
            st8f(xs + 8 * c, x);
        }
        if (p.norm2_w != nullptr) norm2(s2);
    } else if (p.prologue == kProPolyNorm) {
        float s[3] = {0.f, 0.f, 0.f};
        for (int c = tid; c < nch; c += kGemvThreads) {
            float z[8];
            ld8f(p.xf + 8 * c, z);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float z2 = z[j] * z[j], z4 = z2 * z2;
                s[0] += z2;
                s[1] += z4;
                s[2] = fmaf(z4, z2, s[2]);
            }
            st8f(xs + 8 * c, z);
        }
        gemv_block_sums<3>(s, red3);
        const float n = (float)p.k_true;
        const float c0 = __bfloat162float(p.poly[0]) / sqrtf(s[0] / n + p.eps), c1 = __bfloat162float(p.poly[1]) / sqrtf(s[1] / n + p.eps),
                    c2 = __bfloat162float(p.poly[2]) / sqrtf(s[2] / n + p.eps), c3 = __bfloat162float(p.poly[3]);
        for (int c = tid; c < nch; c += kGemvThreads) {
            float z[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                z[j] = xs[8 * c + j];
                z[j] = fmaf(z[j], fmaf(z[j], fmaf(z[j], c2, c1), c0), c3);
            }
            st8f(xs + 8 * c, z);
        }
    } else {
        return false;
    }
    __syncthreads();
    return true;
}

// Activations of one GEMV phase into shared memory as fp32 [K], with the fused prologue (embedding row / residual
// stream + tensor-parallel partials -> RMSNorm).  Ends with a block barrier.  xbytes = gemv_xbytes(K).
__device__ __forceinline__ void gemv_stage(const GemvParams& p, const int nch, unsigned char* smem, const unsigned int xbytes) {
    float* xs = reinterpret_cast<float*>(smem);
    const uint4* gs = reinterpret_cast<const uint4*>(smem + xbytes);
    float* red = reinterpret_cast<float*>(smem + xbytes + gemv_wbytes(p.K));
    float* misc = red + 2 * kGemvWarps * 2;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    // ---- activations (L2 loads: another block may have produced them) ------------------------
    if (p.prologue == kProPlain) {
        if (p.xf != nullptr) {
            for (int c = tid; c < 2 * nch; c += kGemvThreads)
                reinterpret_cast<float4*>(xs)[c] = __ldcg(reinterpret_cast<const float4*>(p.xf) + c);
        } else {
            for (int c = tid; c < nch; c += kGemvThreads) {
                float f[8];
                unpack8(ld_cg(p.x + (size_t)c * 8), f);
                reinterpret_cast<float4*>(xs)[2 * c] = make_float4(f[0], f[1], f[2], f[3]);
                reinterpret_cast<float4*>(xs)[2 * c + 1] = make_float4(f[4], f[5], f[6], f[7]);
            }
        }
    } else {
        // residual stream in fp32 (or the embedding row); staged unscaled until the norm is known
        const __nv_bfloat16* table_row = nullptr;
        bool zero = false, from_table = false;
        if (p.prologue == kProEmbedRmsNorm) {
            const int tok = p.state->token;
            zero = tok < 0 || tok >= p.vocab;
            table_row = p.embed_table + (size_t)(zero ? 0 : tok) * p.K;
            from_table = true;
        }
        float* xf32 = xs;                                          // normalised in place below
        // count to wait for: bumped by this GPU's producing kernel
        const unsigned int want = p.addend_parts == nullptr ? 0u : (p.want_override != 0u ? p.want_override : __ldcg(p.epoch));
        PeerWait pw = peer_wait_begin(p.addend_parts != nullptr ? p.error : nullptr);
        float ss = 0.f;
        for (int c = tid; c < nch; c += kGemvThreads) {
            float f[8];
            if (from_table) {
                unpack8(zero ? make_uint4(0, 0, 0, 0) : ld_cached(table_row + (size_t)c * 8), f);
            } else {
                const float4 lo = __ldcg(reinterpret_cast<const float4*>(p.xr + (size_t)c * 8));
                const float4 hi = __ldcg(reinterpret_cast<const float4*>(p.xr + (size_t)c * 8 + 4));
                f[0] = lo.x; f[1] = lo.y; f[2] = lo.z; f[3] = lo.w; f[4] = hi.x; f[5] = hi.y; f[6] = hi.z; f[7] = hi.w;
            }
            if (p.addend != nullptr) {
                const float4 a0 = __ldcg(reinterpret_cast<const float4*>(p.addend + (size_t)c * 8));
                const float4 a1 = __ldcg(reinterpret_cast<const float4*>(p.addend + (size_t)c * 8 + 4));
                f[0] += a0.x; f[1] += a0.y; f[2] += a0.z; f[3] += a0.w; f[4] += a1.x; f[5] += a1.y; f[6] += a1.z; f[7] += a1.w;
            }
            if (p.addend_parts != nullptr) {       // (p0 + p1 + ...) + x: the partials first, in rank order, as an all-reduce would
                float a[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                for (int r = 0; r < p.n_parts; ++r) {
                    const uint2* part = p.addend_parts + (size_t)r * p.K + (size_t)c * 8;
                    unsigned long long w[8];
                    int spins = 0;
                    for (;;) {                     // until all eight words carry this exchange's count
#pragma unroll
                        for (int j = 0; j < 4; ++j) ld_peer_words(part + 2 * j, w[2 * j], w[2 * j + 1]);
                        bool ok = true;
#pragma unroll
                        for (int j = 0; j < 8; ++j) ok = ok && (unsigned int)(w[j] >> 32) == want;
                        if (ok || pw.dead) break;
                        if ((++spins & 15) == 0) {
                            if (peer_wait_expired(pw, p.error, p.error_host, p.wait_ns)) break;
                            __nanosleep(32);
                        }
                    }
#pragma unroll
                    for (int j = 0; j < 8; ++j) a[j] += __uint_as_float((unsigned int)w[j]);
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) f[j] += a[j];
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
            reinterpret_cast<float4*>(xf32)[2 * c] = make_float4(f[0], f[1], f[2], f[3]);
            reinterpret_cast<float4*>(xf32)[2 * c + 1] = make_float4(f[4], f[5], f[6], f[7]);
            if ((from_table || p.addend != nullptr || p.addend_parts != nullptr) && blockIdx.x == 0) {
                reinterpret_cast<float4*>(p.resid_out)[2 * c] = make_float4(f[0], f[1], f[2], f[3]);
                reinterpret_cast<float4*>(p.resid_out)[2 * c + 1] = make_float4(f[4], f[5], f[6], f[7]);
            }
        }
        ss = warp_sum(ss);
        if (lane == 0) misc[warp] = ss;
        __syncthreads();
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < kGemvWarps; ++w) tot += misc[w];
        const float inv = 1.0f / sqrtf(tot / (float)p.K + p.eps);
        for (int c = tid; c < nch; c += kGemvThreads) {       // same thread, same chunks as above
            const float4 lo = reinterpret_cast<const float4*>(xf32)[2 * c], hi = reinterpret_cast<const float4*>(xf32)[2 * c + 1];
            float w[8];
            unpack8(gs[c], w);
            reinterpret_cast<float4*>(xs)[2 * c] = make_float4(lo.x * inv * w[0], lo.y * inv * w[1], lo.z * inv * w[2], lo.w * inv * w[3]);
            reinterpret_cast<float4*>(xs)[2 * c + 1] = make_float4(hi.x * inv * w[4], hi.y * inv * w[5], hi.z * inv * w[6], hi.w * inv * w[7]);
        }
    }
    __syncthreads();
}

// Stage activations (with the fused norm), stream the rows, reduce, epilogue.
template <Epi EPI, int EXT>
__device__ __forceinline__ void gemv_run(const GemvParams& p, const GemvSched& sc, GemvRegs& r, unsigned char* smem,
                                         const unsigned int xbytes, float& best_v, int& best_i, const int* early_chosen = nullptr) {
    const float* xs = reinterpret_cast<const float*>(smem);
    float* red = reinterpret_cast<float*>(smem + xbytes + gemv_wbytes(p.K));
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nch = sc.nch;

    // residual pair of the first item, fetched under the weight stream
    float2 old_first = make_float2(0.f, 0.f);
    if constexpr (EPI == Epi::Residual) {
        if (sc.wk == 0 && lane == 0 && sc.total > 0)
            old_first = __ldcg(reinterpret_cast<const float2*>(p.residual + sc.ig0 * 2));
    }
    __shared__ int chosen_s[EPI == Epi::ExpertUp ? 2 * kMaxExpertTop : 1];
    const int* chosen = nullptr;
    if constexpr (EPI == Epi::ExpertUp) {
        if (tid < p.route.top) {
            chosen_s[tid] = __ldcg(p.route_id + tid);
            if constexpr (EXT > 2) chosen_s[kMaxExpertTop + tid] = __float_as_int(__ldcg(p.route_w + tid));
        }
        chosen = chosen_s;
        __syncthreads();
        gemv_load_unit<EPI, EXT>(p, sc, 0, r.a, chosen);
        gemv_stage(p, nch, smem, xbytes);
    } else if constexpr (EPI == Epi::ExpertDown) {
        chosen = early_chosen;
        float* xw = reinterpret_cast<float*>(smem);
        const float* weight = reinterpret_cast<const float*>(early_chosen + kMaxExpertTop);
        const float inv = 4.0f / (float)p.ffp;
        for (int c = tid; c < 2 * nch; c += kGemvThreads) {            // padded channels are zero
            const float w = weight[EXT > 2 ? min((int)(((float)c + 0.5f) * inv), p.route.top) : (int)(((float)c + 0.5f) * inv)];
            const float4 v = __ldcg(reinterpret_cast<const float4*>(p.xf) + c);
            reinterpret_cast<float4*>(xw)[c] = make_float4(v.x * w, v.y * w, v.z * w, v.w * w);
        }
        __syncthreads();
    } else if constexpr (EXT) {
        if (!gemv_stage_ext<EXT>(p, nch, smem, xbytes)) gemv_stage(p, nch, smem, xbytes);
    } else {
        gemv_stage(p, nch, smem, xbytes);
    }
    (void)tid;
    (void)early_chosen;

    // ---- rows ------------------------------------------------------------------------------------
    float acc0 = 0.f, acc1 = 0.f;
    int parity = 0;
    auto compute_unit = [&](const int u, const uint4 (&buf)[kGemvU][2]) {
        const int j = u / sc.upi, part = u - j * sc.upi;
#pragma unroll
        for (int uu = 0; uu < kGemvU; ++uu) {
            const int c = (part * kGemvU + uu) * sc.stride + sc.gl;
            if (c < nch) {
                const float4 xlo = reinterpret_cast<const float4*>(xs)[2 * c], xhi = reinterpret_cast<const float4*>(xs)[2 * c + 1];
                const float xf[8] = {xlo.x, xlo.y, xlo.z, xlo.w, xhi.x, xhi.y, xhi.z, xhi.w};
                acc0 = dot8(buf[uu][0], xf, acc0);
                acc1 = dot8(buf[uu][1], xf, acc1);
            }
        }
        if (part != sc.upi - 1) return;
        // item complete
        const int ig = sc.ig0 + j * sc.ig_stride;
        float t0 = warp_sum(acc0), t1 = warp_sum(acc1);
        acc0 = 0.f;
        acc1 = 0.f;
        if (sc.ks > 1) {
            float* buf2 = red + parity * kGemvWarps * 2;
            if (lane == 0) { buf2[warp * 2] = t0; buf2[warp * 2 + 1] = t1; }
            group_barrier(1 + sc.gi, sc.ks * 32);
            if (sc.wk == 0) {
                t0 = 0.f;
                t1 = 0.f;
                for (int w = 0; w < sc.ks; ++w) { t0 += buf2[(sc.gi * sc.ks + w) * 2]; t1 += buf2[(sc.gi * sc.ks + w) * 2 + 1]; }
            }
            parity ^= 1;
        }
        if (sc.wk == 0 && lane == 0) {
            if constexpr (EPI == Epi::Residual) {
                const float2 old = j == 0 ? old_first : __ldcg(reinterpret_cast<const float2*>(p.residual + ig * 2));
                *reinterpret_cast<float2*>(p.residual + ig * 2) = make_float2(old.x + t0, old.y + t1);
            } else {
                item_epilogue<EPI, EXT>(p, ig, t0, t1, best_v, best_i, chosen);
            }
        }
    };
    for (int u = 0; u < sc.total; ++u) {
        if (u > 0) gemv_load_unit<EPI, EXT>(p, sc, u, r.a, chosen);       // unit 0 was fetched before the dependency wait
        compute_unit(u, r.a);
    }
}

// Per-block (max, argmax) of the Logits epilogue -> part_val / part_idx[block].
__device__ __forceinline__ void gemv_publish_best(const GemvParams& p, float best_v, int best_i, float* bv, int* bi) {
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best_v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
        if (ov > best_v || (ov == best_v && oi < best_i)) { best_v = ov; best_i = oi; }
    }
    if (lane == 0) { bv[warp] = best_v; bi[warp] = best_i; }
    __syncthreads();
    if (tid == 0) {
        float v = bv[0];
        int i = bi[0];
        for (int w = 1; w < kGemvWarps; ++w)
            if (bv[w] > v || (bv[w] == v && bi[w] < i)) { v = bv[w]; i = bi[w]; }
        p.part_val[blockIdx.x] = v;
        p.part_idx[blockIdx.x] = i;
    }
}

// One GEMV phase as its own launch (phase-per-launch decode form, prefill lm_head, operator API).
template <Epi EPI, int EXT = 0>
__global__ void __launch_bounds__(kGemvThreads, 1) gemv_kernel(const GemvParams p, const int ks) {
    extern __shared__ __align__(16) unsigned char gemv_smem[];
    __shared__ float bv[kGemvWarps];
    __shared__ int bi[kGemvWarps];
    const unsigned int xbytes = gemv_xbytes(p.K);
    GemvRegs regs;
    float best_v = -INFINITY;
    int best_i = 0x7fffffff;
    // Let the next kernel of the step start its own weight prefetch as soon as every block of this
    // one is resident, then prefetch (independent of every earlier kernel), then wait.
    // ExpertUp holds its dependents back until its own wait is over: the choice it waits for is then there for ExpertDown,
    // which fetches its first weights before its wait.  So does the router of level 4, whose dependents would only fill the SMs.
    constexpr bool kHold = EPI == Epi::ExpertUp || (EPI == Epi::Router && EXT > 3);
    if constexpr (!kHold) pdl_launch_dependents();
    const GemvSched sc = gemv_sched(p, ks, blockIdx.x, gridDim.x);
    __shared__ int early_s[EPI == Epi::ExpertDown ? 2 * kMaxExpertTop + 1 : 1];  // ids | weights (and that of the shared expert)
    if constexpr (EPI == Epi::ExpertDown) {
        if ((int)threadIdx.x < p.route.top) {
            early_s[threadIdx.x] = __ldcg(p.route_id + threadIdx.x);
            early_s[kMaxExpertTop + threadIdx.x] = EXT > 2 && p.weight_input ? __float_as_int(1.0f) : __float_as_int(__ldcg(p.route_w + threadIdx.x));
        }
        if (EXT > 2 && threadIdx.x == 0 && p.shared_ff > 0) early_s[kMaxExpertTop + p.route.top] = __float_as_int(__ldcg(p.route_w + p.route.top));
        __syncthreads();
        gemv_load_unit<EPI, EXT>(p, sc, 0, regs.a, early_s);
    }
    gemv_prefetch<EPI, EXT>(p, sc, regs, gemv_smem, xbytes);
    pdl_wait();
    if constexpr (kHold) pdl_launch_dependents();
    if constexpr (EPI == Epi::Peers) best_i = (int)(__ldcg(p.epoch) + 1u);      // this launch's exchange count rides in best_i
    gemv_run<EPI, EXT>(p, sc, regs, gemv_smem, xbytes, best_v, best_i, EPI == Epi::ExpertDown ? early_s : nullptr);
    if constexpr (EPI == Epi::Router) {
        __shared__ unsigned int last;
        __syncthreads();
        if (threadIdx.x == 0) {
            __threadfence();
            last = atomicAdd(p.route_ticket, 1u) == gridDim.x - 1 ? 1u : 0u;
            __threadfence();
        }
        __syncthreads();
        if (last != 0u && threadIdx.x < 32) {
            route_token(p.out_f, p.route, [&](int k, int e, float w) { p.route_id[k] = e; p.route_w[k] = w; });
            if (threadIdx.x == 0) {
                if (p.route.shared == kSharedGated) p.route_w[p.route.top] = 1.0f / (1.0f + expf(-__ldcg(p.out_f + p.route.experts)));
                else if (p.route.shared == kSharedPlain) p.route_w[p.route.top] = 1.0f;
                *p.route_ticket = 0u;
            }
        }
    }
    if constexpr (EPI == Epi::Logits) gemv_publish_best(p, best_v, best_i, bv, bi);
    if constexpr (EPI == Epi::Peers) {
        // every block has read the count by now; the one that draws the last ticket advances it for the consumer
        __syncthreads();
        if (threadIdx.x == 0) {
            const unsigned int t = atomicAdd(p.ticket, 1u);
            if (t == gridDim.x - 1) {
                *p.ticket = 0u;
                *p.epoch = (unsigned int)best_i;
            }
        }
    }
}

__host__ __device__ inline size_t gemv_smem_bytes(int K) {      // xs (fp32) | norm weight | red + misc
    return (size_t)gemv_xbytes(K) + gemv_wbytes(K) + (size_t)(2 * kGemvWarps * 2 + 16) * sizeof(float);
}

__host__ __device__ inline size_t gemv_conv_smem_bytes(int K) { return (size_t)gemv_conv_off(K) + gemv_xbytes(K) + gemv_wbytes(K); }

// EXT instantiations: room for the second vector of a prologue.
__host__ __device__ inline size_t gemv_ext_smem_bytes(int K) { return (size_t)gemv_ext_off(K) + (size_t)K * 4; }

}  // namespace efm
