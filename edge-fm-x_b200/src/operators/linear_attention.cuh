// Linear attention with a constant decay per head: a state S [D key channels x Dv value channels], fp32,
//   S_t = a S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t,   q, k, v = silu(projections),
// then one RMS norm over the channels of all heads, a plain weight, a sigmoid gate and a multiplier.  The projections are four
// column ranges of a row, each starting at a multiple of 8; in the many-row forms the product that makes them has applied silu (the
// 32-bit mode: silu_columns), so that q, k and v are rounded once.
//
// Many rows, in chunks of up to 64 tokens of one entry (128 on the tensor cores, linear_attention_tc.cuh).  A chunk's own contribution does not depend on the state it starts from, so
// all chunks run at once and only their sums are chained:
//   linear_chunk_rows    U_c = sum_t a^(n-1-t) k_t v_t^T of every chunk (n tokens)
//   linear_chain_rows    the states the chunks start from, S_{c+1} = a^n S_c + U_c, in place of the U_c; the last one to the pool
//   linear_attend_rows   o_t = a^(t+1) S_c^T q_t + sum_{s<=t} a^(t-s) (q_t . k_s) v_s
//   linear_output_rows   norm, weight, gate, multiplier
// One row: linear_decode_block, part of the launch of the attention beside it (window_attention.cuh).
//
// The same sum alone (`alone`): q, k and v enter without silu, q and k turned by their position first; o is scaled, RMS-normed per head
// (with a weight shared by the heads, or none) and multiplied by silu of the gate.  Its decay is the constant of the head or, from the
// projections, one number per token and key channel (`rank` > 0):
//   S_t = diag(alpha_t) S_{t-1} + k_t v_t^T,   alpha_t = sigmoid(W_a2 W_a1 x + b)^(1 / tau)
//   linear_rotate_rows       q and k of every row turned, everything rounded once (32-bit mode, and head sizes that the epilogue of the
//                            projections' product, gemm_tc.cuh, does not take); the pairs are neighbours, the weights' rows are laid out so
//   linear_decay_rows        alpha of every row, or (chunks on the tensor cores) sums of log alpha from the chunk's first token on
//   linear_scan_rows         channel decays token by token: 32-bit mode, short passes and heads the tensor-core form does not take
//   linear_head_output_rows  scale, norm per head, weight, gate
//   linear_decode            one row: all of it in one launch, a cluster per head
// State pool: [slots][slot_stride] floats, this layer at `offset`, head h at + h * D * Vp, row = key channel (Vp: Dv padded to 4,
// pads zero).  The powers of the decays come from the host, rounded once.
#pragma once
#include <cooperative_groups.h>

#include "common.cuh"
#include "rotary.cuh"
#include "row_plan.cuh"

namespace efm {

struct LinearShape {
    int heads, D, Dv, Vp;
    int off_q, off_k, off_v, off_g;   // columns of the projections
    int ld;                           // row length of the projections
    const float* powers;              // [heads][kLinearPowers + 1]: decay^i
    const __nv_bfloat16* norm;        // [heads * Dv]; alone: [Dv] or null
    float eps, scale;                 // scale: of the result; alone: of o, before the norm
    RotShape rot;                     // alone
    int rank, off_a;                  // decays from the projections: width and first column of W_a1 x (rank 0: constant decays)
    float inv_tau;
    const __nv_bfloat16 *a2, *a2_bias;    // [heads * D][ld_a2], [heads * D]
    int ld_a2;
    __host__ __device__ int width() const { return heads * Dv; }
    __host__ __device__ size_t head_floats() const { return (size_t)D * Vp; }
};

__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float lin_f32(float v) { return v; }
__device__ __forceinline__ float lin_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

namespace ln {
constexpr int C = kLinearChunk, kThreads = 256;

// dst[r][0 .. cols) (row stride ld_dst, cols % 4 == 0) = mul(r) times channels [c0, c0 + cols) of a head, zero past `width` and past row n
template <typename T, typename F>
__device__ __forceinline__ void stage_rows(float* dst, int ld_dst, const T* src, int ld_src, int c0, int cols, int width, int n, F mul) {
    const int per = cols / 4;
    const bool vec = ((reinterpret_cast<uintptr_t>(src) | (uintptr_t)(ld_src * sizeof(T))) & (4 * sizeof(T) - 1)) == 0;
    for (int i = threadIdx.x; i < C * per; i += kThreads) {
        const int r = i / per, c = (i - r * per) * 4;
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (r < n) {
            const T* p = src + (size_t)r * ld_src + c0 + c;
            if (vec && c0 + c + 4 <= width) {
                if constexpr (sizeof(T) == 2) {
                    const uint2 v = *reinterpret_cast<const uint2*>(p);
                    f[0] = bf16lo(v.x); f[1] = bf16hi(v.x); f[2] = bf16lo(v.y); f[3] = bf16hi(v.y);
                } else {
                    const float4 v = *reinterpret_cast<const float4*>(p);
                    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
                }
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (c0 + c + j < width) f[j] = lin_f32(p[j]);
            }
            const float m = mul(r);
#pragma unroll
            for (int j = 0; j < 4; ++j) f[j] *= m;
        }
        *reinterpret_cast<float4*>(dst + (size_t)r * ld_dst + c) = make_float4(f[0], f[1], f[2], f[3]);
    }
}
__host__ __device__ constexpr size_t chunk_smem_bytes(int RM, int RN) { return (size_t)C * (16 * RM + 16 * RN) * sizeof(float); }
// queries | keys, afterwards values | products | a slice of the state
__host__ __device__ inline int attend_key_floats(int D4, int RN) { const int k = C * (D4 + 4), v = C * 16 * RN; return k > v ? k : v; }
__host__ __device__ inline size_t attend_smem_bytes(int D, int RN) {
    const int D4 = (D + 3) / 4 * 4;
    return (size_t)(C * (D4 + 4) + attend_key_floats(D4, RN) + C * (C + 4) + 32 * 16 * RN) * sizeof(float);
}
}  // namespace ln

// columns [c0, c1) of every row (multiples of 4).  Grid (parts of a row, rows)
__global__ void __launch_bounds__(256) silu_columns_kernel(float* __restrict__ x, int ld, int c0, int c1) {
    const int c = c0 + 4 * (blockIdx.x * 256 + threadIdx.x);
    if (c >= c1) return;
    float4* p = reinterpret_cast<float4*>(x + (size_t)blockIdx.y * ld + c);
    const float4 v = *p;
    *p = make_float4(silu_f(v.x), silu_f(v.y), silu_f(v.z), silu_f(v.w));
}

// grid (chunks, heads, tiles of the state); a tile is 16 RM key channels x 16 RN value channels.  ws: [chunks][heads][D][Vp]
template <typename T, int RM, int RN>
__global__ void __launch_bounds__(ln::kThreads) linear_chunk_rows_kernel(const T* __restrict__ proj, float* __restrict__ ws, const LinearShape s, const RowPlan plan) {
    using namespace ln;
    constexpr int TM = 16 * RM, TN = 16 * RN;
    extern __shared__ __align__(16) float ln_smem[];
    float *ks = ln_smem, *vs = ln_smem + C * TM;
    RowEntry e;
    int t0;
    if (!locate_chunk<C>(plan, blockIdx.x, e, t0)) return;
    const int h = blockIdx.y, n = min(C, e.n - t0), tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int tiles_n = (s.Vp + TN - 1) / TN, d0 = blockIdx.z / tiles_n * TM, v0 = blockIdx.z % tiles_n * TN;
    const float* pw = s.powers + (size_t)h * (kLinearPowers + 1);
    const T* row = proj + (size_t)(e.row0 + t0) * s.ld;
    stage_rows(ks, TM, row + s.off_k + h * s.D, s.ld, d0, TM, s.D, n, [&](int r) { return pw[n - 1 - r]; });
    stage_rows(vs, TN, row + s.off_v + h * s.Dv, s.ld, v0, TN, s.Dv, n, [](int) { return 1.0f; });
    __syncthreads();
    float acc[RM][RN];
#pragma unroll
    for (int i = 0; i < RM; ++i)
#pragma unroll
        for (int j = 0; j < RN; ++j) acc[i][j] = 0.f;
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
        float a[RM], b[RN];
#pragma unroll
        for (int i = 0; i < RM; i += 4) *reinterpret_cast<float4*>(a + i) = *reinterpret_cast<const float4*>(ks + t * TM + i * 16 + ty * 4);
#pragma unroll
        for (int j = 0; j < RN; j += 4) *reinterpret_cast<float4*>(b + j) = *reinterpret_cast<const float4*>(vs + t * TN + j * 16 + tx * 4);
#pragma unroll
        for (int i = 0; i < RM; ++i)
#pragma unroll
            for (int j = 0; j < RN; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    float* out = ws + ((size_t)blockIdx.x * s.heads + h) * s.head_floats();
#pragma unroll
    for (int i = 0; i < RM; ++i) {
        const int d = d0 + (i & ~3) * 16 + ty * 4 + (i & 3);
        if (d >= s.D) continue;
#pragma unroll
        for (int j = 0; j < RN; j += 4) {
            const int v = v0 + j * 16 + tx * 4;
            if (v < s.Vp) *reinterpret_cast<float4*>(out + (size_t)d * s.Vp + v) = make_float4(acc[i][j], acc[i][j + 1], acc[i][j + 2], acc[i][j + 3]);
        }
    }
}

// grid (groups of 256 x 4 state numbers, entries); chunks of C tokens.  CH: decays per key channel, sums [rows][ld_sums] as
// linear_decay_sums leaves them
template <int C, bool CH = false>
__global__ void __launch_bounds__(256) linear_chain_rows_kernel(float* __restrict__ ws, float* __restrict__ pool, size_t slot_stride, size_t offset,
                                                                const LinearShape s, const RowPlan plan, const float* __restrict__ sums, int ld_sums) {
    constexpr int U = 8;
    const size_t all = s.heads * s.head_floats(), i = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= all) return;
    const RowEntry e = plan.entry(blockIdx.y);
    const float* pw = CH ? nullptr : s.powers + i / s.head_floats() * (kLinearPowers + 1);
    const float* sum = CH ? sums + (size_t)e.row0 * ld_sums + i / s.Vp : nullptr;      // head h's key channel d is column h D + d
    int chunk0 = 0;
    for (int k = 0; k < (int)blockIdx.y; ++k) chunk0 += (plan.entry(k).n + C - 1) / C;
    const int n_chunks = (e.n + C - 1) / C;
    float* st = pool + (size_t)e.state * slot_stride + offset + i;
    float* w = ws + (size_t)chunk0 * all + i;
    float4 S = e.pos0 > 0 ? *reinterpret_cast<const float4*>(st) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float full = CH ? 0.f : pw[C], last = CH ? 0.f : pw[e.n - (n_chunks - 1) * C];
    for (int c0 = 0; c0 < n_chunks; c0 += U) {
        float4 u[U];
        float f[U];
#pragma unroll
        for (int k = 0; k < U; ++k)
            if (c0 + k < n_chunks) {
                u[k] = *reinterpret_cast<const float4*>(w + (size_t)(c0 + k) * all);
                if constexpr (CH) f[k] = sum[(size_t)(min((c0 + k + 1) * C, e.n) - 1) * ld_sums];
            }
#pragma unroll
        for (int k = 0; k < U; ++k)
            if (c0 + k < n_chunks) {
                *reinterpret_cast<float4*>(w + (size_t)(c0 + k) * all) = S;
                const float a = CH ? expf(f[k]) : c0 + k == n_chunks - 1 ? last : full;
                S.x = fmaf(a, S.x, u[k].x); S.y = fmaf(a, S.y, u[k].y); S.z = fmaf(a, S.z, u[k].z); S.w = fmaf(a, S.w, u[k].w);
            }
    }
    *reinterpret_cast<float4*>(st) = S;
}

// grid (chunks, heads, tiles of 16 RN value channels)
template <typename T, int RN>
__global__ void __launch_bounds__(ln::kThreads) linear_attend_rows_kernel(const T* __restrict__ proj, const float* __restrict__ ws, float* __restrict__ o, int ld_o,
                                                                          const LinearShape s, const RowPlan plan) {
    using namespace ln;
    constexpr int TN = 16 * RN, LP = C + 4;
    extern __shared__ __align__(16) float ln_smem[];
    RowEntry e;
    int t0;
    if (!locate_chunk<C>(plan, blockIdx.x, e, t0)) return;
    const int h = blockIdx.y, v0 = blockIdx.z * TN, n = min(C, e.n - t0), tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int D4 = (s.D + 3) / 4 * 4, LD = D4 + 4;
    float *qs = ln_smem, *ks = qs + C * LD, *vs = ks, *ps = ks + attend_key_floats(D4, RN), *ss = ps + C * LP;
    __shared__ float pw[C + 1];
    if (tid <= C) pw[tid] = s.powers[(size_t)h * (kLinearPowers + 1) + tid];
    const T* row = proj + (size_t)(e.row0 + t0) * s.ld;
    auto one = [](int) { return 1.0f; };
    stage_rows(qs, LD, row + s.off_q + h * s.D, s.ld, 0, D4, s.D, n, one);
    stage_rows(ks, LD, row + s.off_k + h * s.D, s.ld, 0, D4, s.D, n, one);
    __syncthreads();
    {   // products of queries and keys, decayed; row ty + 16 i, column tx + 16 j
        float p[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) p[i][j] = 0.f;
        for (int d = 0; d < D4; d += 4) {
            float4 a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(qs + (ty + 16 * i) * LD + d);
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = *reinterpret_cast<const float4*>(ks + (tx + 16 * j) * LD + d);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    p[i][j] = fmaf(a[i].x, b[j].x, p[i][j]); p[i][j] = fmaf(a[i].y, b[j].y, p[i][j]);
                    p[i][j] = fmaf(a[i].z, b[j].z, p[i][j]); p[i][j] = fmaf(a[i].w, b[j].w, p[i][j]);
                }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = ty + 16 * i, u = tx + 16 * j;
                ps[t * LP + u] = u <= t ? p[i][j] * pw[t - u] : 0.f;
            }
    }
    __syncthreads();
    stage_rows(vs, TN, row + s.off_v + h * s.Dv, s.ld, v0, TN, s.Dv, n, one);      // in place of the keys
    float acc[4][RN];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < RN; ++j) acc[i][j] = 0.f;
    // four rows of b (row stride TN) times four columns of a (row stride lda)
    auto step = [&](const float* a, int lda, const float* b) {
        float x[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(x[i]) = *reinterpret_cast<const float4*>(a + (ty + 16 * i) * lda);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            float y[RN];
#pragma unroll
            for (int j = 0; j < RN; j += 4) *reinterpret_cast<float4*>(y + j) = *reinterpret_cast<const float4*>(b + k * TN + j * 16 + tx * 4);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < RN; ++j) acc[i][j] = fmaf(x[i][k], y[j], acc[i][j]);
        }
    };
    const float* S = ws + ((size_t)blockIdx.x * s.heads + h) * s.head_floats();
    if (e.pos0 + t0 > 0)                                               // the first chunk of a sequence starts from zero
        for (int d0 = 0; d0 < D4; d0 += 32) {
            for (int i = tid; i < 32 * TN / 4; i += kThreads) {
                const int r = i / (TN / 4), c = (i - r * (TN / 4)) * 4;
                *reinterpret_cast<float4*>(ss + r * TN + c) = d0 + r < s.D && v0 + c < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)(d0 + r) * s.Vp + v0 + c)
                                                                                            : make_float4(0.f, 0.f, 0.f, 0.f);
            }
            __syncthreads();
            for (int d = 0; d < min(32, D4 - d0); d += 4) step(qs + d0 + d, LD, ss + d * TN);
            __syncthreads();
        }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < RN; ++j) acc[i][j] *= pw[ty + 16 * i + 1];
    __syncthreads();
    for (int u = 0; u < n; u += 4) step(ps + u, LP, vs + u * TN);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty + 16 * i;
        if (t >= n) continue;
        float* dst = o + (size_t)(e.row0 + t0 + t) * ld_o + h * s.Dv;
#pragma unroll
        for (int j = 0; j < RN; j += 4) {
            const int v = v0 + j * 16 + tx * 4;
            if ((s.Dv & 3) == 0) {
                if (v < s.Dv) *reinterpret_cast<float4*>(dst + v) = make_float4(acc[i][j], acc[i][j + 1], acc[i][j + 2], acc[i][j + 3]);
            } else {
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (v + k < s.Dv) dst[v + k] = acc[i][j + k];
            }
        }
    }
}

// out[row][0 .. width) = rms(o) * norm * sigmoid(gate) * scale, columns up to `cols` zero.  One block per row; ld_o, cols multiples
// of 4.  The first 1024 * KEEP channels stay in registers.
template <typename T>
__global__ void __launch_bounds__(256, 5) linear_output_rows_kernel(const float* __restrict__ o, int ld_o, const T* __restrict__ proj, T* __restrict__ out, int ld_out,
                                                                 int cols, const LinearShape s) {
    constexpr int KEEP = 2;
    __shared__ float part[8];
    const int row = blockIdx.x, tid = threadIdx.x, n = s.width();
    const float* src = o + (size_t)row * ld_o;
    const T* gate = proj + (size_t)row * s.ld + s.off_g;
    T* dst = out + (size_t)row * ld_out;
    auto load = [&](int c) {
        float4 v = *reinterpret_cast<const float4*>(src + c);           // ld_o covers the pads
        if (c + 4 > n) { if (c >= n) v.x = 0.f; if (c + 1 >= n) v.y = 0.f; if (c + 2 >= n) v.z = 0.f; v.w = 0.f; }
        return v;
    };
    struct Factors { float g[4], w[4]; };
    auto factors = [&](int c) {
        Factors f;
        const uint2 w = *reinterpret_cast<const uint2*>(s.norm + c);       // padded with zeros
        f.w[0] = bf16lo(w.x); f.w[1] = bf16hi(w.x); f.w[2] = bf16lo(w.y); f.w[3] = bf16hi(w.y);
        if constexpr (sizeof(T) == 2) {
            const uint2 x = *reinterpret_cast<const uint2*>(gate + c);
            f.g[0] = bf16lo(x.x); f.g[1] = bf16hi(x.x); f.g[2] = bf16lo(x.y); f.g[3] = bf16hi(x.y);
        } else {
            const float4 x = *reinterpret_cast<const float4*>(gate + c);
            f.g[0] = x.x; f.g[1] = x.y; f.g[2] = x.z; f.g[3] = x.w;
        }
        return f;
    };
    float4 keep[KEEP];
    Factors fac[KEEP];                                                  // requested ahead of the sum
    float ss = 0.f;
    auto square = [&](const float4& v) { ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss)))); };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (4 * (tid + 256 * i) < cols) { keep[i] = load(4 * (tid + 256 * i)); fac[i] = factors(4 * (tid + 256 * i)); }
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (4 * (tid + 256 * i) < cols) square(keep[i]);
    for (int c = 4 * (tid + 256 * KEEP); c < cols; c += 1024) square(load(c));
    ss = warp_sum(ss);
    if ((tid & 31) == 0) part[tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += part[i];
    const float inv = s.scale / sqrtf(ss / (float)n + s.eps);
    auto emit = [&](int c, const float4& v, const Factors& k) {
        const float f[4] = {v.x, v.y, v.z, v.w};
        float r[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) r[j] = f[j] * inv * k.w[j] / (1.0f + expf(-k.g[j]));
        if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16(r[0], r[1]), pack_bf16(r[2], r[3]));
        else *reinterpret_cast<float4*>(dst + c) = make_float4(r[0], r[1], r[2], r[3]);
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (4 * (tid + 256 * i) < cols) emit(4 * (tid + 256 * i), keep[i], fac[i]);
    for (int c = 4 * (tid + 256 * KEEP); c < cols; c += 1024) emit(c, load(c), factors(c));
}

// ---- the sum alone -----------------------------------------------------------------------------------------------------
// log of alpha; the product z / tau is what matters when z is far below zero
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau; }

// (cos, sin) of every pair of every row of a pass.  Grid (parts of a row, rows)
__global__ void __launch_bounds__(128) rot_rows_kernel(float2* __restrict__ out, const RotShape r, const RowPlan plan) {
    const int i = blockIdx.x * 128 + threadIdx.x, row = blockIdx.y;
    if (i >= r.dims / 2) return;
    const RowEntry e = plan.of_row(row);
    float2 v;
    rot_sincos(r, e.pos0 + row - e.row0, i, &v.y, &v.x);
    out[(size_t)row * (r.dims / 2) + i] = v;
}

// proj -> out with q and k turned; in 32-bit mode both may be the same rows.  One block per row; ld % 8 == 0, dims % 2 == 0.
template <typename T>
__global__ void __launch_bounds__(256) linear_rotate_rows_kernel(const float* proj, T* out, const LinearShape s, const RowPlan plan) {
    __shared__ float cs[kRotMaxPairs], sn[kRotMaxPairs];
    const int row = blockIdx.x, half = s.rot.dims / 2;
    const RowEntry e = plan.of_row(row);
    rot_table(s.rot, e.pos0 + row - e.row0, cs, sn);
    __syncthreads();
    const float* src = proj + (size_t)row * s.ld;
    T* dst = out + (size_t)row * s.ld;
    auto put = [](T* p, float v) { if constexpr (sizeof(T) == 2) *p = __float2bfloat16_rn(v); else *p = v; };
    for (int i = threadIdx.x; i < 2 * s.heads * half; i += 256) {
        const int u = i / half, pair = i - u * half;                    // a head of q, then of k
        const int c = (u < s.heads ? s.off_q + u * s.D : s.off_k + (u - s.heads) * s.D) + 2 * pair;
        const float a = src[c], b = src[c + 1];
        put(dst + c, a * cs[pair] - b * sn[pair]);
        put(dst + c + 1, b * cs[pair] + a * sn[pair]);
    }
    if constexpr (sizeof(T) == 2) {                                     // everything else
        const int rest = s.D - s.rot.dims;
        if (rest > 0)
            for (int i = threadIdx.x; i < 2 * s.heads * rest; i += 256) {
                const int u = i / rest, c = (u < s.heads ? s.off_q + u * s.D : s.off_k + (u - s.heads) * s.D) + s.rot.dims + i - u * rest;
                put(dst + c, src[c]);
            }
        for (int c = s.off_v + 4 * threadIdx.x; c < s.ld; c += 1024) {
            const float4 v = *reinterpret_cast<const float4*>(src + c);
            *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
        }
    }
}

// z [rows][ld] (W_a2 W_a1 x + b) in place: alpha.  Grid (parts of a row, rows)
__global__ void __launch_bounds__(256) linear_decay_rows_kernel(float* __restrict__ z, int ld, float inv_tau) {
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c < ld) z[(size_t)blockIdx.y * ld + c] = expf(log_decay(z[(size_t)blockIdx.y * ld + c], inv_tau));
}
// the same: sums of log alpha from the first token of the chunk to this one.  Grid (parts of a row, chunks of C tokens)
template <int C>
__global__ void __launch_bounds__(128) linear_decay_sums_kernel(float* __restrict__ z, int ld, float inv_tau, const RowPlan plan) {
    constexpr int U = 16;
    RowEntry e;
    int t0;
    const int c = blockIdx.x * 128 + threadIdx.x;
    if (!locate_chunk<C>(plan, blockIdx.y, e, t0) || c >= ld) return;
    const int n = min(C, e.n - t0);
    float* p = z + (size_t)(e.row0 + t0) * ld + c;
    float sum = 0.f, v[U];
    for (int r0 = 0; r0 < n; r0 += U) {
#pragma unroll
        for (int i = 0; i < U; ++i)
            if (r0 + i < n) v[i] = p[(size_t)(r0 + i) * ld];
#pragma unroll
        for (int i = 0; i < U; ++i)
            if (r0 + i < n) {
                sum += log_decay(v[i], inv_tau);
                p[(size_t)(r0 + i) * ld] = sum;
            }
    }
}

// the same without branches; the logarithm of 1 + e as a series in e / (2 + e), at most 1/3
__device__ __forceinline__ float log_decay_fast(float z, float inv_tau) {
    const float e = __expf(-fabsf(z)), q = __fdividef(e, 2.0f + e), q2 = q * q;
    const float l = 2.0f * q * fmaf(q2, fmaf(q2, fmaf(q2, fmaf(q2, fmaf(q2, 1.0f / 11.0f, 1.0f / 9.0f), 1.0f / 7.0f), 0.2f), 1.0f / 3.0f), 1.0f);
    return (fminf(z, 0.f) - l) * inv_tau;
}
// linear_decay_sums with the product W_a2 (W_a1 x) + b in front of it, W_a1 x of at most RANK bf16 numbers a row.  Grid (64 channels, chunks
// of C tokens): eight threads a channel, an eighth of the chunk each.
template <int C, int RANK>
__global__ void __launch_bounds__(512, 2) linear_decay_product_sums_kernel(const __nv_bfloat16* __restrict__ proj, float* __restrict__ sums, int ld_sums, const LinearShape s,
                                                                        const RowPlan plan) {
    constexpr int PART = C / 8;
    __shared__ __align__(16) float a1[C][RANK];
    __shared__ float part[8][64];
    RowEntry e;
    int t0;
    if (!locate_chunk<C>(plan, blockIdx.y, e, t0)) return;
    const int n = min(C, e.n - t0), tid = threadIdx.x, c = blockIdx.x * 64 + (tid & 63), eighth = tid >> 6, all = s.heads * s.D;
    const __nv_bfloat16* src = proj + (size_t)(e.row0 + t0) * s.ld + s.off_a;
    auto row8 = [](const __nv_bfloat16* p, bool in, float (&f)[8]) { unpack8(in ? ld_cached(p) : make_uint4(0u, 0u, 0u, 0u), f); };
    for (int i = tid; i < C * RANK / 8; i += 512) {                     // columns past the rank are zero in W_a1, so here
        const int r = i / (RANK / 8), k = 8 * (i - r * (RANK / 8));
        float f[8];
        row8(src + (size_t)r * s.ld + k, r < n && k < s.ld_a2, f);
        *reinterpret_cast<float4*>(&a1[r][k]) = make_float4(f[0], f[1], f[2], f[3]);
        *reinterpret_cast<float4*>(&a1[r][k + 4]) = make_float4(f[4], f[5], f[6], f[7]);
    }
    float w[RANK], b = 0.f;
#pragma unroll
    for (int k = 0; k < RANK; k += 8) {
        float f[8];
        row8(s.a2 + (size_t)c * s.ld_a2 + k, c < all && k < s.ld_a2, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) w[k + j] = f[j];
    }
    if (c < all) b = __bfloat162float(s.a2_bias[c]);
    __syncthreads();
    float v[PART], sum = 0.f;
#pragma unroll
    for (int r = 0; r < PART; ++r) {
        const float4* x = reinterpret_cast<const float4*>(a1[eighth * PART + r]);
        float z = b;
#pragma unroll
        for (int k = 0; k < RANK / 4; ++k) {
            const float4 y = x[k];
            z = fmaf(w[4 * k], y.x, z); z = fmaf(w[4 * k + 1], y.y, z); z = fmaf(w[4 * k + 2], y.z, z); z = fmaf(w[4 * k + 3], y.w, z);
        }
        sum += log_decay_fast(z, s.inv_tau);
        v[r] = sum;
    }
    part[eighth][tid & 63] = sum;
    __syncthreads();
    float before = 0.f;
    for (int k = 0; k < eighth; ++k) before += part[k][tid & 63];
    float* out = sums + (size_t)(e.row0 + t0 + eighth * PART) * ld_sums + c;
#pragma unroll
    for (int r = 0; r < PART; ++r)
        if (eighth * PART + r < n && c < ld_sums) out[(size_t)r * ld_sums] = before + v[r];
}

namespace lc {
constexpr int kThreads = 128, kCols = 16, kBatch = 8;                  // value channels per block, tokens per staged batch
inline size_t smem_bytes(int D) { return (size_t)kBatch * (3 * ((D + 31) / 32 * 32) + kCols) * sizeof(float); }
}  // namespace lc
// grid (heads * slices of 16 value channels, entries); eight lanes share a state column.  NC: float4 chunks of a column per lane.
template <typename T, int NC>
__global__ void __launch_bounds__(lc::kThreads) linear_scan_rows_kernel(const T* __restrict__ proj, const float* __restrict__ alpha, int ld_alpha,
                                                                        float* __restrict__ o, int ld_o, float* __restrict__ pool, size_t slot_stride,
                                                                        size_t offset, const LinearShape s, const RowPlan plan) {
    using namespace lc;
    extern __shared__ __align__(16) float lc_smem[];
    constexpr int Dp = NC * 32, step = 3 * Dp + kCols;
    const int slices = (s.Dv + kCols - 1) / kCols, h = blockIdx.x / slices, c0 = blockIdx.x % slices * kCols;
    const RowEntry e = plan.entry(blockIdx.y);
    const int tid = threadIdx.x, col = tid >> 3, l8 = tid & 7;
    const bool in = c0 + col < s.Dv;
    float* st = pool + (size_t)e.state * slot_stride + offset + h * s.head_floats() + c0 + col;
    float S[NC][4];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = (c * 8 + l8) * 4 + j;
            S[c][j] = e.pos0 > 0 && in && d < s.D ? st[(size_t)d * s.Vp] : 0.f;
        }
    for (int t0 = 0; t0 < e.n; t0 += kBatch) {
        const int n = min(kBatch, e.n - t0);
        __syncthreads();
        for (int i = tid; i < n * Dp; i += kThreads) {
            const int t = i / Dp, d = i - t * Dp;
            const size_t row = (size_t)(e.row0 + t0 + t);
            const T* x = proj + row * s.ld + h * s.D + d;
            float* to = lc_smem + t * step + d;
            to[0] = d < s.D ? alpha[row * ld_alpha + h * s.D + d] : 0.f;
            to[Dp] = d < s.D ? lin_f32(x[s.off_k]) : 0.f;
            to[2 * Dp] = d < s.D ? lin_f32(x[s.off_q]) : 0.f;
        }
        for (int i = tid; i < n * kCols; i += kThreads) {
            const int t = i / kCols, v = c0 + i - t * kCols;
            lc_smem[t * step + 3 * Dp + i - t * kCols] = v < s.Dv ? lin_f32(proj[(size_t)(e.row0 + t0 + t) * s.ld + s.off_v + h * s.Dv + v]) : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float4 *a4 = reinterpret_cast<const float4*>(lc_smem + t * step) + l8, *k4 = a4 + Dp / 4, *q4 = k4 + Dp / 4;
            const float v = lc_smem[t * step + 3 * Dp + col];
            float x = 0.f, y = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float4 a = a4[c * 8], k = k4[c * 8], q = q4[c * 8];
                S[c][0] = fmaf(a.x, S[c][0], k.x * v); S[c][1] = fmaf(a.y, S[c][1], k.y * v);
                S[c][2] = fmaf(a.z, S[c][2], k.z * v); S[c][3] = fmaf(a.w, S[c][3], k.w * v);
                x = fmaf(q.x, S[c][0], x); y = fmaf(q.y, S[c][1], y); x = fmaf(q.z, S[c][2], x); y = fmaf(q.w, S[c][3], y);
            }
            x += y;
#pragma unroll
            for (int m = 4; m > 0; m >>= 1) x += __shfl_xor_sync(0xffffffffu, x, m);
            if (l8 == 0 && in) o[(size_t)(e.row0 + t0 + t) * ld_o + h * s.Dv + c0 + col] = x;
        }
    }
    const bool pad = c0 + col < s.Vp;                                   // pads of the state stay zero
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = (c * 8 + l8) * 4 + j;
            if (pad && d < s.D) st[(size_t)d * s.Vp] = in ? S[c][j] : 0.f;
        }
}

// out[row][0 .. width) = rms of every head of scale * o, times norm, times silu(gate).  A warp per (row, head); Dv <= 256.
template <typename T>
__global__ void __launch_bounds__(256) linear_head_output_rows_kernel(const float* __restrict__ o, int ld_o, const T* __restrict__ proj, T* __restrict__ out,
                                                                      int ld_out, int rows, const LinearShape s) {
    const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, row = unit / s.heads, h = unit - row * s.heads;
    if (row >= rows) return;
    const float* src = o + (size_t)row * ld_o + h * s.Dv;
    const T* gate = proj + (size_t)row * s.ld + s.off_g + h * s.Dv;
    T* dst = out + (size_t)row * ld_out + h * s.Dv;
    float v[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        v[i] = c < s.Dv ? src[c] * s.scale : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)s.Dv + s.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c >= s.Dv) continue;
        const float r = v[i] * inv * (s.norm != nullptr ? __bfloat162float(s.norm[c]) : 1.0f) * silu_f(lin_f32(gate[c]));
        if constexpr (sizeof(T) == 2) dst[c] = __float2bfloat16_rn(r);
        else dst[c] = r;
    }
}

// ---- one row -----------------------------------------------------------------------------------------------------------
namespace ln {
constexpr int kCols = 64;             // value channels per decode block
struct DecodeSmem { float q[256], k[256], red[16][kCols]; };
struct AloneSmem {
    float a1[512], alpha[256], cs[kRotMaxPairs], sn[kRotMaxPairs];
    float sums[4], part[2];           // sums of squares: the head's slices, this block's two warps
};
inline int decode_units(const LinearShape& s) { return s.heads * ((s.Dv + kCols - 1) / kCols); }
}  // namespace ln

struct LinearDecodeParams {
    LinearShape s;
    float* pool;                      // this layer's state of the sequence
    float* out;                       // [heads * Dv], before the norm
    int units;                        // blocks: (head, 64 value channels); 0: no linear attention in this launch
};

// One block of 256 threads: 16 threads per state row (4 channels each), 16 rows at a time.  The state is read before the
// dependency wait when `early`.  Returns channel `tid` of the block's 64 (the first 64 threads).
template <bool ALONE = false>
__device__ __forceinline__ float linear_decode_block(const LinearDecodeParams& p, int unit, const float* proj, const DecodeState* state, int max_tokens, int early,
                                                     ln::DecodeSmem& sm, ln::AloneSmem* alone = nullptr) {
    using namespace ln;
    constexpr int NR = 16, PRE = 4;
    const LinearShape& s = p.s;
    const int slices = (s.Dv + kCols - 1) / kCols, h = unit / slices, tid = threadIdx.x, rg = tid >> 4, c = unit % slices * kCols + (tid & 15) * 4;
    const bool act = c < s.Vp;
    float* S = p.pool + h * s.head_floats() + c;
    if (!early) { pdl_wait(); pdl_launch_dependents(); }
    const int kv_len = (int)state->kv_len;
    const bool ok = kv_len > 0 && kv_len <= max_tokens, fresh = kv_len <= 1;
    float4 r[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rg + 16 * i;
        r[i] = act && d < s.D && !fresh ? __ldcg(reinterpret_cast<const float4*>(S + (size_t)d * s.Vp)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float a = 0.f, a2b = 0.f;
    uint4 a2[PRE];                                                      // this channel's row of W_a2, its first 8 PRE columns
    const __nv_bfloat16* a2_row = nullptr;
    if (!ALONE || s.rank == 0) {
        a = s.powers[(size_t)h * (kLinearPowers + 1) + 1];
    } else if (tid < s.D) {
        a2_row = s.a2 + (size_t)(h * s.D + tid) * s.ld_a2;
        a2b = __bfloat162float(s.a2_bias[h * s.D + tid]);
#pragma unroll
        for (int i = 0; i < PRE; ++i)
            if (8 * i < s.ld_a2) a2[i] = ld_cached(a2_row + 8 * i);
    }
    if (ALONE && ok) rot_table(s.rot, kv_len - 1, alone->cs, alone->sn);
    if (early) { pdl_wait(); pdl_launch_dependents(); }
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float x = c + j < s.Dv ? __ldcg(proj + s.off_v + h * s.Dv + c + j) : 0.f;
        v[j] = ALONE ? x : silu_f(x);
    }
    for (int d = tid; d < s.D; d += 256) {
        const float q = __ldcg(proj + s.off_q + h * s.D + d), k = __ldcg(proj + s.off_k + h * s.D + d);
        sm.q[d] = ALONE ? q : silu_f(q);
        sm.k[d] = ALONE ? k : silu_f(k);
    }
    if constexpr (ALONE) {
        for (int i = tid; i < s.ld_a2 && s.rank > 0; i += 256) alone->a1[i] = i < s.rank ? __ldcg(proj + s.off_a + i) : 0.f;
    }
    __syncthreads();
    if constexpr (ALONE) {
        if (s.rot.kind != kRotNone) {
            const float q = tid < s.D ? rot_channel(s.rot, sm.q, tid, alone->cs, alone->sn) : 0.f;
            const float k = tid < s.D ? rot_channel(s.rot, sm.k, tid, alone->cs, alone->sn) : 0.f;
            __syncthreads();
            if (tid < s.D) { sm.q[tid] = q; sm.k[tid] = k; }
        }
        if (tid < s.D) {
            if (s.rank > 0) {
                float z = 0.f;
                auto add = [&](const uint4& w, int i) {
                    const float4 x = *reinterpret_cast<const float4*>(alone->a1 + 8 * i), y = *reinterpret_cast<const float4*>(alone->a1 + 8 * i + 4);
                    const float f[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w};
                    z = dot8(w, f, z);
                };
#pragma unroll
                for (int i = 0; i < PRE; ++i)
                    if (8 * i < s.ld_a2) add(a2[i], i);
                for (int i = PRE; 8 * i < s.ld_a2; ++i) add(ld_cached(a2_row + 8 * i), i);
                alone->alpha[tid] = expf(log_decay(z + a2b, s.inv_tau));
            } else {
                alone->alpha[tid] = a;
            }
        }
        __syncthreads();
    }
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rg + 16 * i;
        if (d < s.D) {
            const float k = sm.k[d], q = sm.q[d];
            if constexpr (ALONE) a = alone->alpha[d];
            r[i].x = fmaf(a, r[i].x, k * v[0]); r[i].y = fmaf(a, r[i].y, k * v[1]);
            r[i].z = fmaf(a, r[i].z, k * v[2]); r[i].w = fmaf(a, r[i].w, k * v[3]);
            if (act && ok) *reinterpret_cast<float4*>(S + (size_t)d * s.Vp) = r[i];
            o.x = fmaf(q, r[i].x, o.x); o.y = fmaf(q, r[i].y, o.y); o.z = fmaf(q, r[i].z, o.z); o.w = fmaf(q, r[i].w, o.w);
        }
    }
    *reinterpret_cast<float4*>(&sm.red[rg][(tid & 15) * 4]) = o;
    __syncthreads();
    float t = 0.f;
    if (tid < kCols) {
#pragma unroll
        for (int g = 0; g < 16; ++g) t += sm.red[g][tid];
    }
    const int ch = unit % slices * kCols + tid;
    if (!ALONE && tid < kCols && ch < s.Dv) p.out[h * s.Dv + ch] = t;
    return t;
}

// grid (slices of 64 value channels = cluster size, heads): the sum alone, normed and gated
__global__ void __launch_bounds__(256) linear_decode_kernel(const LinearDecodeParams p, const float* __restrict__ proj, DecodeState* state, int max_tokens, int early) {
    using namespace ln;
    namespace cg = cooperative_groups;
    __shared__ __align__(16) DecodeSmem sm;
    __shared__ __align__(16) AloneSmem alone;
    const LinearShape& s = p.s;
    const int slices = gridDim.x, h = blockIdx.y, tid = threadIdx.x, ch = blockIdx.x * kCols + tid;
    float o = linear_decode_block<true>(p, h * slices + blockIdx.x, proj, state, max_tokens, early, sm, &alone) * s.scale;
    const bool in = tid < kCols && ch < s.Dv;
    if (!in) o = 0.f;
    float gate = 0.f, w = 1.f;
    if (in) {
        gate = __ldcg(proj + s.off_g + h * s.Dv + ch);
        if (s.norm != nullptr) w = __bfloat162float(s.norm[ch]);
    }
    const float ss = warp_sum(o * o);
    if (tid < kCols && (tid & 31) == 0) alone.part[tid >> 5] = ss;
    __syncthreads();
    float sum = alone.part[0] + alone.part[1];
    if (slices > 1) {
        cg::cluster_group cl = cg::this_cluster();
        cl.sync();                                                      // the other blocks have started
        if (tid < slices) *cl.map_shared_rank(&alone.sums[blockIdx.x], tid) = sum;
        cl.sync();
        sum = 0.f;
        for (int i = 0; i < slices; ++i) sum += alone.sums[i];
    }
    if (in) p.out[h * s.Dv + ch] = o * (1.0f / sqrtf(sum / (float)s.Dv + s.eps)) * w * silu_f(gate);
    if (tid == 0 && blockIdx.x == 0 && h == 0 && ((int)state->kv_len <= 0 || (int)state->kv_len > max_tokens)) state->error = 2;
}

}  // namespace efm
