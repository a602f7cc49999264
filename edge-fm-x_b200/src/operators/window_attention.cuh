// Causal softmax attention over a paged cache with a sliding window, kept first tokens and per-head score modification:
//   score(i, j) = (q_i . k_j) * scale * temp[h] - slope_h * (i - j),   0 <= i - j < window (window 0: no lower bound) or j < keep
// with slope_h = 2^(-8 (h + 1) / H), q and k RMS-normalised per head (with or without a weight, or not at all) or over all heads
// at once (with a weight), and then rotated before they are used / cached, value width free.  Instead of the softmax a key's weight may be
// sigmoid(score + shift[h]), not normalised; a head's output may be multiplied by sigmoid(gate_h).  A weightless norm commutes with the rotation, which keeps a head's length.
// Cache: per layer a K pool [pages * 64][kv_heads][Dp] and a V pool [pages * 64][kv_heads][Vp], channels zero-padded to
// Dp / Vp (multiples of 64); a sequence's pages are listed in a page table.  TC = bf16 or fp32 (the all-32-bit mode).
//
//   qk_scatter_rows      many rows: per-head norms and rotation, q -> [T][H][Dp], k and v -> cache rows
//   window_attention_rows many rows on the CUDA cores, fp32 throughout (32-bit mode, short portions, head sizes the
//                        tensor-core form does not take)
//   window_attention_decode one row: norms of q and k, cache append and split-key attention in one launch; the splits of
//                        a kv head are the blocks of one cluster and merge through distributed shared memory
#pragma once
#include <cooperative_groups.h>

#include <utility>

#include "common.cuh"
#include "linear_attention.cuh"
#include "rotary.cuh"
#include "row_plan.cuh"

namespace efm {

struct WindowAttnShape {
    int H, G, D, Dv, Dp, Vp;          // query heads, kv heads, channels and padded channels
    int window;                       // 0: full causal
    int keep;                         // first tokens that stay visible (with a window)
    int bias;                         // 1: distance bias
    int qk_norm;                      // 0: q and k as they are; 1: per head; 2: over all heads, weights [H * D] and [G * D]
    const __nv_bfloat16* shift;       // not null: sigmoid weights, [H]
    float scale, eps;
    float out_scale;                  // of the result
    const __nv_bfloat16* q_norm;      // [D], null: norm without a weight
    const __nv_bfloat16* k_norm;      // [D]
    const __nv_bfloat16* temp;        // [H], null: 1
    RotShape rot;
    // tensor-core form with a shared key part only: extra term exp(sink[h]) of the softmax denominator, and channels multiplied by
    // sigmoid(gate)
    const __nv_bfloat16* sink;        // [H], null: none
    const void* gate;                 // [T][H * Dv], or (gate_heads) [T][H], of the pass's activation type with row stride gate_ld, null: none
    int gate_ld, gate_heads;
};
__device__ __forceinline__ float sigmoid_weight(float score) { return 1.0f / (1.0f + expf(-score)); }

__device__ __forceinline__ float head_multiplier(const WindowAttnShape& s, int h) {
    return s.temp != nullptr ? s.scale * __bfloat162float(s.temp[h]) : s.scale;
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void store_f32(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_f32(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float distance_slope(int h, int H) { return exp2f(-8.0f * (float)(h + 1) / (float)H); }
template <typename T> __device__ __forceinline__ float round_as(float v);
template <> __device__ __forceinline__ float round_as<float>(float v) { return v; }
template <> __device__ __forceinline__ float round_as<__nv_bfloat16>(float v) { return round_bf16(v); }

__device__ __forceinline__ void load8_as_f32(const float* p, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8_as_f32(const __nv_bfloat16* p, float (&f)[8]) { unpack8(ld_cached(p), f); }
__device__ __forceinline__ float4 load4_as_f32(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4_as_f32(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf16lo(v.x), bf16hi(v.x), bf16lo(v.y), bf16hi(v.y));
}

// ---- many rows: norms and scatter --------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void load_head8(const T* x, int d, int D, bool vec, float (&f)[8]) {
    if (vec && d + 8 <= D) {
        if constexpr (sizeof(T) == 2) {
            unpack8(ld_cached(x + d), f);
        } else {
            const float4 a = *reinterpret_cast<const float4*>(x + d), b = *reinterpret_cast<const float4*>(x + d + 4);
            f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
        }
    } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = d + j < D ? to_f32(x[d + j]) : 0.f;
    }
}
template <typename T>
__device__ __forceinline__ void store_head8(T* p, const float (&f)[8]) {          // 16-byte aligned
    if constexpr (sizeof(T) == 2) {
        *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
    } else {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
    }
}

// One block per row; `lanes` (8, 16 or 32) threads share a head, 8 channels each.  TI: projections, TQ: q operand, TC: cache.
template <typename TI, typename TQ, typename TC, bool ROT>
__global__ void __launch_bounds__(256, 4) qk_scatter_rows_kernel(const TI* __restrict__ qkv, int ld, TQ* __restrict__ q_out, TC* __restrict__ k_pool,
                                                              TC* __restrict__ v_pool, const WindowAttnShape s, const RowPlan plan, int lanes) {
    __shared__ __align__(16) float cs[kRotMaxPairs];
    __shared__ __align__(16) float sn[kRotMaxPairs];
    __shared__ float stage[ROT ? 256 * 8 : 1];
    __shared__ float row_ss[2][8];
    const int row = blockIdx.x, l = threadIdx.x & (lanes - 1), per = 256 / lanes;
    const RowEntry e = plan.of_row(row);
    const int half = s.rot.dims / 2;
    const bool by_lanes = s.rot.kind == kRotHalf && (half & 7) == 0;   // a channel's partner sits in the same place of another lane
    if constexpr (ROT) {
        rot_table(s.rot, e.pos0 + row - e.row0, cs, sn);
        __syncthreads();
    }
    const size_t cr = plan.cache_row(e, e.pos0 + row - e.row0);
    const TI* src = qkv + (size_t)row * ld;                            // ld % 8 == 0
    const bool vec = (s.D & 7) == 0, vecv = vec && (s.Dv & 7) == 0;
    const int units = s.H + 2 * s.G, d = 8 * l;
    float inv_q = 1.f, inv_k = 1.f;
    if (s.qk_norm == 2) {
        float sq = 0.f, sk = 0.f;
        auto squares = [&](int c0, int n) {
            const bool v8 = (c0 & 7) == 0;
            float t = 0.f, f[8];
            for (int c = 8 * threadIdx.x; c < n; c += 2048) {
                load_head8(src + c0, c, n, v8, f);
#pragma unroll
                for (int j = 0; j < 8; ++j) t = fmaf(f[j], f[j], t);
            }
            return t;
        };
        sq = squares(0, s.H * s.D);
        sk = squares(s.H * s.D, s.G * s.D);
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if ((threadIdx.x & 31) == 0) { row_ss[0][threadIdx.x >> 5] = sq; row_ss[1][threadIdx.x >> 5] = sk; }
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) { sq += row_ss[0][i]; sk += row_ss[1][i]; }
        inv_q = 1.0f / sqrtf(sq / (float)(s.H * s.D) + s.eps);
        inv_k = 1.0f / sqrtf(sk / (float)(s.G * s.D) + s.eps);
    }
    for (int u0 = 0; u0 < units; u0 += per) {                          // every thread takes part in the shuffles
        const int u = u0 + threadIdx.x / lanes;
        const bool qk = u < s.H + s.G;
        float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (qk) load_head8(src + (size_t)u * s.D, d, s.D, vec, f);     // q heads, then k heads
        else if (u < units) load_head8(src + (size_t)(s.H + s.G) * s.D + (size_t)(u - s.H - s.G) * s.Dv, d, s.Dv, vecv, f);
        const __nv_bfloat16* w = u < s.H ? s.q_norm : s.k_norm;
        if (s.qk_norm == 2 && qk) w += (size_t)(u < s.H ? u : u - s.H) * s.D;
        float ss = 0.f, g[8];
        if (qk && w != nullptr) load_head8(w, d, s.D, vec, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
        for (int x = lanes / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
        if (qk) {
            const float inv = s.qk_norm == 2 ? (u < s.H ? inv_q : inv_k) : s.qk_norm ? 1.0f / sqrtf(ss / (float)s.D + s.eps) : 1.0f;
#pragma unroll
            for (int j = 0; j < 8; ++j) f[j] *= inv;                   // channels past D are zero
            if (w != nullptr) {
#pragma unroll
                for (int j = 0; j < 8; ++j) f[j] *= g[j];
            }
        }
        if constexpr (ROT) {
            if (by_lanes) {
                const bool low = d < half, in = qk && d < s.rot.dims;
                const int src = in ? (low ? l + half / 8 : l - half / 8) : l, i0 = in ? (low ? d : d - half) : 0;
                float c[8], n[8];
                load8_as_f32(cs + i0, c);
                load8_as_f32(sn + i0, n);
                const float sign = low ? -1.f : 1.f;
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const float o = __shfl_sync(0xffffffffu, f[j], src, lanes);
                    if (in) f[j] = fmaf(f[j], c[j], sign * o * n[j]);
                }
            } else {
                float* st = stage + (threadIdx.x & ~(lanes - 1)) * 8;  // this head's channels
#pragma unroll
                for (int j = 0; j < 8; ++j) st[d + j] = f[j];
                __syncwarp();
                if (qk && d < s.rot.dims) {
#pragma unroll
                    for (int j = 0; j < 8; ++j) f[j] = rot_channel(s.rot, st, d + j, cs, sn);
                }
                __syncwarp();
            }
        }
        if (qk) {
            if (d < s.Dp) {
                if (u < s.H) store_head8(q_out + ((size_t)row * s.H + u) * s.Dp + d, f);
                else store_head8(k_pool + (cr * s.G + (u - s.H)) * s.Dp + d, f);
            }
        } else if (u < units && d < s.Vp) {
            store_head8(v_pool + (cr * s.G + (u - s.H - s.G)) * s.Vp + d, f);
        }
    }
}

// ---- many rows on the CUDA cores ---------------------------------------------------------------------------------
namespace wa {
constexpr int QT = 16, KT = 32;
inline size_t rows_smem_bytes(int Dp, int Vp) { return (size_t)(QT * (Dp + 4) + KT * (Dp + 4) + KT * (Vp + 4) + QT * (KT + 1)) * sizeof(float); }
}  // namespace wa

// Block = 16 rows of one entry x one head; keys in tiles of 32 staged as fp32.  tiles: [gridDim.x] (null: the single
// entry's rows in order).  out: [T][H * Dv].
template <typename TQ, typename TC, typename TO>
__global__ void __launch_bounds__(256) window_attention_rows_kernel(const TQ* __restrict__ q, const TC* __restrict__ k_pool, const TC* __restrict__ v_pool,
                                                                    TO* __restrict__ out, int ld_out, const WindowAttnShape s, const RowPlan plan,
                                                                    const RowTile* __restrict__ tiles) {
    using namespace wa;
    extern __shared__ __align__(16) float wa_smem[];
    const int tid = threadIdx.x, h = blockIdx.y, g = h / (s.H / s.G);
    const int DS = s.Dp + 4, VS = s.Vp + 4;
    float* qs = wa_smem;
    float* ks = qs + QT * DS;
    float* vs = ks + KT * DS;
    float* ps = vs + KT * VS;
    RowEntry e;
    int r0;                                                            // first row inside the entry
    if (tiles != nullptr) { const RowTile t = tiles[blockIdx.x]; e = plan.entry(t.entry); r0 = t.row; }
    else { e = plan.one; r0 = blockIdx.x * QT; }
    const int nq = min(QT, e.n - r0);
    for (int i = tid; i < QT * s.Dp; i += 256) {
        const int r = i / s.Dp, d = i - r * s.Dp;
        qs[r * DS + d] = r < nq ? to_f32(q[((size_t)(e.row0 + r0 + r) * s.H + h) * s.Dp + d]) : 0.f;
    }
    const int r = tid >> 4, c = tid & 15;
    const int i_pos = e.pos0 + r0 + r;                                 // this row's position
    const int lo = s.window > 0 ? max(0, i_pos - s.window + 1) : 0;
    const int first = s.window > 0 ? max(0, e.pos0 + r0 - s.window + 1) : 0;
    const int end = e.pos0 + r0 + nq;                                  // one past the last visible key of the block
    const int first_tile = first & ~(KT - 1), kept = s.window > 0 ? min(s.keep, first) : 0;    // kept keys ahead of the window
    const float mul = head_multiplier(s, h);
    const float slope = s.bias ? distance_slope(h, s.H) : 0.f;
    float acc[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[n][j] = 0.f;
    const bool sig = s.shift != nullptr;
    const float shift = sig ? __bfloat162float(s.shift[h]) : 0.f;
    float m = -INFINITY, l = 0.f;
    for (int k0 = kept > 0 ? 0 : first_tile; k0 < end; k0 = k0 + KT >= kept ? max(k0 + KT, first_tile) : k0 + KT) {
        __syncthreads();
        for (int i = tid; i < KT * s.Dp; i += 256) {
            const int kr = i / s.Dp, d = i - kr * s.Dp;
            ks[kr * DS + d] = k0 + kr < end ? to_f32(k_pool[(plan.cache_row(e, k0 + kr) * s.G + g) * s.Dp + d]) : 0.f;
        }
        for (int i = tid; i < KT * s.Vp; i += 256) {
            const int kr = i / s.Vp, d = i - kr * s.Vp;
            vs[kr * VS + d] = k0 + kr < end ? to_f32(v_pool[(plan.cache_row(e, k0 + kr) * s.G + g) * s.Vp + d]) : 0.f;
        }
        __syncthreads();
        float sc[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int j = k0 + c + 16 * u;
            float d0 = 0.f, d1 = 0.f;
            const float4* a = reinterpret_cast<const float4*>(qs + r * DS);
            const float4* b = reinterpret_cast<const float4*>(ks + (c + 16 * u) * DS);
            for (int t = 0; t < s.Dp / 4; ++t) {
                const float4 x = a[t], y = b[t];
                d0 = fmaf(x.x, y.x, d0); d1 = fmaf(x.y, y.y, d1); d0 = fmaf(x.z, y.z, d0); d1 = fmaf(x.w, y.w, d1);
            }
            sc[u] = ((j >= lo || j < s.keep) && j <= i_pos) ? (d0 + d1) * mul - slope * (float)(i_pos - j) : -INFINITY;
        }
        if (sig) {
#pragma unroll
            for (int u = 0; u < 2; ++u) ps[r * (KT + 1) + c + 16 * u] = sc[u] == -INFINITY ? 0.f : sigmoid_weight(sc[u] + shift);
        } else {
            float mx = fmaxf(sc[0], sc[1]);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m, mx), mb = mn == -INFINITY ? 0.f : mn;
            const float alpha = m == -INFINITY ? 0.f : expf(m - mb);
            m = mn;
            float rs = 0.f;
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float p = sc[u] == -INFINITY ? 0.f : expf(sc[u] - mb);
                rs += p;
                ps[r * (KT + 1) + c + 16 * u] = p;
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) rs += __shfl_xor_sync(0xffffffffu, rs, o);
            l = l * alpha + rs;
#pragma unroll
            for (int n = 0; n < 4; ++n)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[n][j] *= alpha;
        }
        __syncwarp();                                                  // the 16 lanes of a row share a warp
        for (int kr = 0; kr < KT; ++kr) {
            const float p = ps[r * (KT + 1) + kr];
#pragma unroll
            for (int n = 0; n < 4; ++n)
                if (n * 64 < s.Vp) {
                    const float4 v = *reinterpret_cast<const float4*>(vs + kr * VS + n * 64 + c * 4);
                    acc[n][0] = fmaf(p, v.x, acc[n][0]); acc[n][1] = fmaf(p, v.y, acc[n][1]);
                    acc[n][2] = fmaf(p, v.z, acc[n][2]); acc[n][3] = fmaf(p, v.w, acc[n][3]);
                }
        }
    }
    if (r >= nq) return;
    float inv = sig ? s.out_scale : l > 0.f ? s.out_scale / l : 0.f;
    if (s.gate != nullptr) inv *= sigmoid_weight(to_f32(static_cast<const TQ*>(s.gate)[(size_t)(e.row0 + r0 + r) * s.gate_ld + h]));
    TO* dst = out + (size_t)(e.row0 + r0 + r) * ld_out + (size_t)h * s.Dv;
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = n * 64 + c * 4 + j;
            if (d < s.Dv) store_f32(dst + d, acc[n][j] * inv);
        }
}

// ---- one row -----------------------------------------------------------------------------------------------------
namespace wd {
constexpr int kThreads = 256, kHeads = 8;      // query heads per block (of one kv head)
template <int VM>
struct Smem {
    static constexpr int MAXP = VM;            // padded channels at most
    float q[kHeads][MAXP + 8];
    float knew[MAXP], vnew[MAXP];
    float p[kHeads][kPageTokens];
    float alpha[kHeads], m[kHeads], l[kHeads];
    float cs[kRotMaxPairs], sn[kRotMaxPairs];
    // what the blocks of the cluster hand to this one: its share of their un-normalised outputs, and everybody's (m, l)
    float rm[16][kHeads], rl[16][kHeads];
    float rout[kHeads * MAXP + 16 * 16];       // [split][share of the outputs]
    float red[8192];                           // [key groups][kHeads][Vp]: at most 256 / (Vp / 4) * 8 * Vp = 8192
};
}  // namespace wd

template <typename TC>
struct WindowDecodeParams {
    WindowAttnShape s;
    const float* qkv;                 // [H * D | G * D | G * Dv]
    TC* k_pool;
    TC* v_pool;
    const int32_t* pages;             // page table row of the sequence
    int max_pages;
    DecodeState* state;
    float* out;                       // [H * Dv]
    const float* gate;                // [H], null: none
    int early;                        // 1: state and the older cache rows may be read before the dependency wait
    LinearDecodeParams lin;           // linear attention beside this one: its blocks follow in grid.y
};

// 8 channels of a cache row as fp32
template <typename TC> struct Row8;
template <> struct Row8<__nv_bfloat16> {
    uint4 v;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = ld_cg(p); }
    __device__ __forceinline__ void get(float (&f)[8]) const { unpack8(v, f); }
};
template <> struct Row8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = __ldcg(reinterpret_cast<const float4*>(p)); b = __ldcg(reinterpret_cast<const float4*>(p) + 1); }
    __device__ __forceinline__ void get(float (&f)[8]) const { f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w; }
};
template <typename TC> struct Row4;
template <> struct Row4<__nv_bfloat16> {
    uint2 v;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = __ldcg(reinterpret_cast<const uint2*>(p)); }
    __device__ __forceinline__ void get(float (&f)[4]) const { f[0] = bf16lo(v.x); f[1] = bf16hi(v.x); f[2] = bf16lo(v.y); f[3] = bf16hi(v.y); }
};
template <> struct Row4<float> {
    float4 v;
    __device__ __forceinline__ void load(const float* p) { v = __ldcg(reinterpret_cast<const float4*>(p)); }
    __device__ __forceinline__ void get(float (&f)[4]) const { f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w; }
};

// grid (splits = cluster size, kv_heads * head blocks); the visible keys (kept first tokens, then the window) are numbered in
// order and dealt out evenly, block `split` walks its share in tiles of 64.  VM: upper bound of Dp and Vp.  Further rows of
// clusters (LIN) compute the linear attention that reads the same projections.
template <typename TC, int VM, bool ROT, bool LIN>
__global__ void __launch_bounds__(wd::kThreads) window_attention_decode_kernel(const WindowDecodeParams<TC> p) {
    using namespace wd;
    constexpr int KC = VM / 32;                                        // 8-channel chunks per thread and key (4 threads per key)
    constexpr int VK = VM <= 64 ? 4 : (VM <= 128 ? 8 : 16);            // keys per thread in the P.V phase
    extern __shared__ __align__(16) unsigned char wd_smem[];
    Smem<VM>& sm = *reinterpret_cast<Smem<VM>*>(wd_smem);
    const WindowAttnShape& s = p.s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, n_splits = gridDim.x;
    const int group = s.H / s.G, hb = (group + kHeads - 1) / kHeads;
    if constexpr (LIN) {
        if ((int)blockIdx.y >= s.G * hb) {                             // a whole cluster
            const int unit = ((int)blockIdx.y - s.G * hb) * n_splits + split;
            if (unit < p.lin.units)
                linear_decode_block(p.lin, unit, p.qkv, p.state, p.max_pages * kPageTokens, p.early, *reinterpret_cast<ln::DecodeSmem*>(wd_smem));
            else { pdl_wait(); pdl_launch_dependents(); }
            return;
        }
    }
    const int g = blockIdx.y / hb, h0 = g * group + (blockIdx.y % hb) * kHeads, nh = min(kHeads, (g + 1) * group - h0);
    const int key = tid >> 2, part = tid & 3;                          // score phase
    const int tpr = s.Vp / 4, kg = kThreads / tpr, dpart = tid % tpr, tg = tid / tpr;     // P.V phase: 4 channels per thread
    const bool pv = tg < kg;

    namespace cg = cooperative_groups;
    cg::cluster_group cl = cg::this_cluster();
    auto started = cl.barrier_arrive();                                // waited for before the first store into another block
    if (!p.early) { pdl_wait(); pdl_launch_dependents(); }
    const int kv_len = (int)p.state->kv_len, pos = kv_len - 1;
    const bool ok = kv_len > 0 && kv_len <= p.max_pages * kPageTokens;
    const int lo = s.window > 0 ? max(0, kv_len - s.window) : 0;
    const int kept = s.window > 0 ? min(s.keep, lo) : 0;               // visible key n stands at position n or, behind the kept ones, n + skip
    const int skip = lo - kept, n_vis = kv_len - skip, newest = n_vis - 1;
    const int chunk = ok ? (n_vis + n_splits - 1) / n_splits : 0;
    const int begin = split * chunk, end = ok ? min(n_vis, begin + chunk) : begin;

    Row8<TC> kr[KC];
    Row4<TC> vr[VK];
    auto position = [&](int n) { return n < kept ? n : n + skip; };
    auto pool_row = [&](int j) { return (size_t)p.pages[j / kPageTokens] * kPageTokens + j % kPageTokens; };
    // 64 keys from number j0, except the one this launch appends
    auto load_tile = [&](int j0) {
        const int j = j0 + key;
        if (j < end && j != newest) {
            const TC* src = p.k_pool + (pool_row(position(j)) * s.G + g) * s.Dp;
#pragma unroll
            for (int c = 0; c < KC; ++c)
                if ((c * 4 + part) * 8 < s.Dp) kr[c].load(src + (c * 4 + part) * 8);
        }
        if (pv) {
#pragma unroll
            for (int i = 0; i < VK; ++i) {
                const int kk = tg + i * kg, jj = j0 + kk;
                if (kk < kPageTokens && jj < end && jj != newest) vr[i].load(p.v_pool + (pool_row(position(jj)) * s.G + g) * s.Vp + dpart * 4);
            }
        }
    };
    if (begin < end) load_tile(begin);
    if constexpr (ROT) {
        if (ok) rot_table(s.rot, pos, sm.cs, sm.sn);
        __syncthreads();
    }
    if (p.early) { pdl_wait(); pdl_launch_dependents(); }

    // ---- norms and rotation of this token's q heads and k, v ------------------------------------------------------------------
    float inv_q = 1.f, inv_k = 1.f;
    if (s.qk_norm == 2) {                                              // over all heads: every block sums for itself
        float sq = 0.f, sk = 0.f;
        for (int c = tid; c < s.H * s.D; c += kThreads) { const float v = __ldcg(p.qkv + c); sq = fmaf(v, v, sq); }
        for (int c = tid; c < s.G * s.D; c += kThreads) { const float v = __ldcg(p.qkv + s.H * s.D + c); sk = fmaf(v, v, sk); }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) { sm.red[warp] = sq; sm.red[8 + warp] = sk; }
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) { sq += sm.red[i]; sk += sm.red[8 + i]; }
        inv_q = 1.0f / sqrtf(sq / (float)(s.H * s.D) + s.eps);
        inv_k = 1.0f / sqrtf(sk / (float)(s.G * s.D) + s.eps);
    }
    for (int u = warp; u < nh + 1; u += 8) {
        const bool is_q = u < nh;
        const float* x = is_q ? p.qkv + (size_t)(h0 + u) * s.D : p.qkv + (size_t)(s.H + g) * s.D;
        const __nv_bfloat16* w = is_q ? s.q_norm : s.k_norm;
        if (s.qk_norm == 2) w += is_q ? (size_t)(h0 + u) * s.D : (size_t)g * s.D;
        float f[VM / 32], ss = 0.f;
#pragma unroll
        for (int i = 0; i < VM / 32; ++i) {
            const int d = lane + 32 * i;
            f[i] = d < s.D ? __ldcg(x + d) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < VM / 32; ++i) ss = fmaf(f[i], f[i], ss);
        const float inv = s.qk_norm == 2 ? (is_q ? inv_q : inv_k) : s.qk_norm ? 1.0f / sqrtf(warp_sum(ss) / (float)s.D + s.eps) : 1.0f;
#pragma unroll
        for (int i = 0; i < VM / 32; ++i) {
            const int d = lane + 32 * i;
            if (d >= s.Dp) continue;
            const float v = d < s.D ? f[i] * inv * (w != nullptr ? __bfloat162float(w[d]) : 1.f) : 0.f;
            if (is_q) sm.q[u][d] = v; else sm.knew[d] = ROT ? v : round_as<TC>(v);
        }
        if constexpr (ROT) {
            float* y = is_q ? sm.q[u] : sm.knew;
            __syncwarp();
#pragma unroll
            for (int i = 0; i < VM / 32; ++i) {
                const int d = lane + 32 * i;
                if (d < s.Dp) {
                    f[i] = rot_channel(s.rot, y, d, sm.cs, sm.sn);
                    if (!is_q) f[i] = round_as<TC>(f[i]);
                }
            }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < VM / 32; ++i)
                if (lane + 32 * i < s.Dp) y[lane + 32 * i] = f[i];
        }
    }
    for (int d = tid; d < s.Vp; d += kThreads)
        sm.vnew[d] = d < s.Dv ? round_as<TC>(__ldcg(p.qkv + (size_t)(s.H + s.G) * s.D + (size_t)g * s.Dv + d)) : 0.f;
    if (tid < kHeads) { sm.m[tid] = -INFINITY; sm.l[tid] = 0.f; }
    __syncthreads();
    if (begin <= newest && newest < end && blockIdx.y % hb == 0) {     // the block that walks the newest key appends it
        const size_t cr = pool_row(pos);
        for (int d = tid; d < s.Dp; d += kThreads) store_f32(p.k_pool + (cr * s.G + g) * s.Dp + d, sm.knew[d]);
        for (int d = tid; d < s.Vp; d += kThreads) store_f32(p.v_pool + (cr * s.G + g) * s.Vp + d, sm.vnew[d]);
    }
    if (!ok && tid == 0) p.state->error = 2;

    float acc[kHeads][4];
#pragma unroll
    for (int h = 0; h < kHeads; ++h)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[h][j] = 0.f;

    for (int j0 = begin; j0 < end; j0 += kPageTokens) {
        const int j = j0 + key;
        const bool vis = j < end;
        // ---- scores: 4 threads per key ----------------------------------------------------------------------------
        float kf[KC][8];
#pragma unroll
        for (int c = 0; c < KC; ++c) {
            const int d0 = (c * 4 + part) * 8;
            if (d0 < s.Dp && j == newest) {
#pragma unroll
                for (int i = 0; i < 8; ++i) kf[c][i] = sm.knew[d0 + i];
            } else {
                kr[c].get(kf[c]);
            }
        }
        for (int h = 0; h < nh; ++h) {
            float d = 0.f;
            if (vis) {
#pragma unroll
                for (int c = 0; c < KC; ++c) {
                    const int d0 = (c * 4 + part) * 8;
                    if (d0 < s.Dp) {
                        const float4 a = *reinterpret_cast<const float4*>(&sm.q[h][d0]), b = *reinterpret_cast<const float4*>(&sm.q[h][d0 + 4]);
                        d = fmaf(a.x, kf[c][0], d); d = fmaf(a.y, kf[c][1], d); d = fmaf(a.z, kf[c][2], d); d = fmaf(a.w, kf[c][3], d);
                        d = fmaf(b.x, kf[c][4], d); d = fmaf(b.y, kf[c][5], d); d = fmaf(b.z, kf[c][6], d); d = fmaf(b.w, kf[c][7], d);
                    }
                }
            }
            d += __shfl_xor_sync(0xffffffffu, d, 1);
            d += __shfl_xor_sync(0xffffffffu, d, 2);
            if (part == 0) {
                const float slope = s.bias ? distance_slope(h0 + h, s.H) : 0.f;
                sm.p[h][key] = vis ? d * head_multiplier(s, h0 + h) - slope * (float)(pos - position(j)) : -INFINITY;
            }
        }
        __syncthreads();
        // ---- online softmax: one warp per head --------------------------------------------------------------------
        if (warp < nh && s.shift != nullptr) {                         // weights that need no other key's
            const float b = __bfloat162float(s.shift[h0 + warp]), s0 = sm.p[warp][lane], s1 = sm.p[warp][lane + 32];
            sm.p[warp][lane] = s0 == -INFINITY ? 0.f : sigmoid_weight(s0 + b);
            sm.p[warp][lane + 32] = s1 == -INFINITY ? 0.f : sigmoid_weight(s1 + b);
            if (lane == 0) sm.alpha[warp] = 1.0f;
        } else if (warp < nh) {
            const float s0 = sm.p[warp][lane], s1 = sm.p[warp][lane + 32];
            const float m_old = sm.m[warp], mn = fmaxf(m_old, warp_max(fmaxf(s0, s1)));       // the tile holds a visible key
            const float p0 = expf(s0 - mn), p1 = expf(s1 - mn);
            sm.p[warp][lane] = p0;
            sm.p[warp][lane + 32] = p1;
            const float sum = warp_sum(p0 + p1);
            if (lane == 0) {
                const float al = expf(m_old - mn);
                sm.alpha[warp] = al;
                sm.m[warp] = mn;
                sm.l[warp] = sm.l[warp] * al + sum;
            }
        }
        __syncthreads();
        if (pv) {
#pragma unroll
            for (int h = 0; h < kHeads; ++h)
                if (h < nh) {
                    const float al = sm.alpha[h];
#pragma unroll
                    for (int c = 0; c < 4; ++c) acc[h][c] *= al;
                }
#pragma unroll
            for (int i = 0; i < VK; ++i) {
                const int kk = tg + i * kg, jj = j0 + kk;
                if (kk < kPageTokens && jj < end) {
                    float v[4];
                    if (jj == newest) {
#pragma unroll
                        for (int c = 0; c < 4; ++c) v[c] = sm.vnew[dpart * 4 + c];
                    } else {
                        vr[i].get(v);
                    }
#pragma unroll
                    for (int h = 0; h < kHeads; ++h)
                        if (h < nh) {
                            const float w = sm.p[h][kk];
#pragma unroll
                            for (int c = 0; c < 4; ++c) acc[h][c] = fmaf(w, v[c], acc[h][c]);
                        }
                }
            }
        }
        if (j0 + kPageTokens < end) load_tile(j0 + kPageTokens);
        __syncthreads();
    }
    // ---- sum over the key groups, then over the splits -------------------------------------------------------------
    if (pv) {
#pragma unroll
        for (int h = 0; h < kHeads; ++h)
            if (h < nh) *reinterpret_cast<float4*>(sm.red + ((size_t)tg * kHeads + h) * s.Vp + dpart * 4) = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
    }
    __syncthreads();
    // every output belongs to one block of the cluster: hand it over, then merge the shares locally
    cl.barrier_wait(std::move(started));
    const int n_out = nh * s.Dv, share = (n_out + n_splits - 1) / n_splits;
    for (int i = tid; i < n_out; i += kThreads) {
        const int h = i / s.Dv, d = i - h * s.Dv;
        float v = 0.f;
        for (int t = 0; t < kg; ++t) v += sm.red[((size_t)t * kHeads + h) * s.Vp + d];
        const int owner = i / share;
        *cl.map_shared_rank(&sm.rout[split * share + i - owner * share], owner) = v;
    }
    for (int i = tid; i < n_splits * kHeads; i += kThreads) {
        const int r = i / kHeads, h = i - r * kHeads;
        *cl.map_shared_rank(&sm.rm[split][h], r) = sm.m[h];
        *cl.map_shared_rank(&sm.rl[split][h], r) = sm.l[h];
    }
    cl.sync();
    for (int i = tid; i < share && split * share + i < n_out; i += kThreads) {
        const int o = split * share + i, h = o / s.Dv, d = o - h * s.Dv;
        const float gate = p.gate != nullptr ? sigmoid_weight(__ldcg(p.gate + h0 + h)) : 1.0f;
        if (s.shift != nullptr) {
            float sum = 0.f;
            for (int r = 0; r < n_splits; ++r) sum += sm.rout[r * share + i];
            p.out[(size_t)(h0 + h) * s.Dv + d] = s.out_scale * gate * sum;
            continue;
        }
        float m = -INFINITY;
        for (int r = 0; r < n_splits; ++r) m = fmaxf(m, sm.rm[r][h]);
        float num = 0.f, den = 0.f;
        for (int r = 0; r < n_splits; ++r) {
            const float mr = sm.rm[r][h], w = mr == -INFINITY ? 0.f : expf(mr - m);
            num = fmaf(w, sm.rout[r * share + i], num);
            den = fmaf(w, sm.rl[r][h], den);
        }
        p.out[(size_t)(h0 + h) * s.Dv + d] = den > 0.f ? s.out_scale * gate * (num / den) : 0.f;
    }
}

}  // namespace efm
