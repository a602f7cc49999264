// Row kernels of the layered decoders' many-row pass: norms with the residual add, PolyNorm, the per-layer token input,
// gathered final norms, the cap of the logits, and the all-32-bit matrix product.  T = bf16 (tensor-core operands) or fp32.
#pragma once
#include "common.cuh"
#include "conv_limits.h"
#include "gemv.cuh"
#include "window_attention.cuh"

namespace efm {

__device__ __forceinline__ float block_sum_256(float v, float* part) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    v = warp_sum(v);
    if (lane == 0) part[warp] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) t += part[i];
    return t;
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf16lo(v.x), bf16hi(v.x), bf16lo(v.y), bf16hi(v.y));
}

// Where a row's sublayer output comes from: row i of y, or (SUM) the weighted sum of the rows place[i][..] of ye.
template <typename T>
struct SumOf {
    const T* ye;
    const int32_t* place;             // [rows][top], null: the row itself
    const float* weight;              // [rows][top]
    int top;
    int32_t* count;                   // rows per expert, zeroed for the next pass by block 0
    int experts;
    int plain;                        // 1: the weights are in the experts' inputs already
    const T* shared;                  // output of a shared expert (null: none) ...
    const float* shared_weight;       // ... and its weight, [rows]
};

// Average over depth behind a layer: its result x goes to hist[n], the stream becomes sum_{j < n} w[j] hist[j] + w[n] x.
struct DepthAverage {
    float* hist;                      // [n + 1][stride], this pass's rows
    size_t stride;
    const __nv_bfloat16* w;
    int n;
};

// x = x_in + y / sqrt(mean(y^2) + eps) * w (w null: x unchanged); out (null: none) = x as T, or (PRE) x / sqrt(mean(x^2) + eps) * pre,
// the next sublayer's input.  AVG: the average over depth behind it (out: none).  One block per row; the first 1024 * KEEP channels
// stay in registers.
template <typename T, bool PRE, bool SUM, bool AVG = false>
__global__ void __launch_bounds__(256) add_norm_rows_kernel(float* x, const float* x_in, const float* __restrict__ y, const __nv_bfloat16* __restrict__ w,
                                                            T* __restrict__ out, const __nv_bfloat16* __restrict__ pre, int n, int ld, float eps,
                                                            const SumOf<T> sum, const DepthAverage avg) {
    constexpr int KEEP = 4;
    __shared__ float part[2][8];
    const size_t base = (size_t)blockIdx.x * ld;
    const int nv = ld / 4, tid = threadIdx.x;
    if (SUM && blockIdx.x == 0)
        for (int e = tid; e < sum.experts; e += 256) sum.count[e] = 0;
    auto load_y = [&](int c) {
        if constexpr (!SUM) return load4(y + base + 4 * c);
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k = 0; k < sum.top; ++k) {
            const size_t i = (size_t)blockIdx.x * sum.top + k;
            const float g = sum.weight[i];
            const float4 v = load4(sum.ye + (size_t)sum.place[i] * ld + 4 * c);
            a.x = fmaf(g, v.x, a.x); a.y = fmaf(g, v.y, a.y); a.z = fmaf(g, v.z, a.z); a.w = fmaf(g, v.w, a.w);
        }
        if (sum.shared != nullptr) {
            const float g = sum.shared_weight[blockIdx.x];
            const float4 v = load4(sum.shared + base + 4 * c);
            a.x = fmaf(g, v.x, a.x); a.y = fmaf(g, v.y, a.y); a.z = fmaf(g, v.z, a.z); a.w = fmaf(g, v.w, a.w);
        }
        return a;
    };
    auto square = [](float s, const float4& v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s)))); };
    float4 keep[KEEP], old[KEEP];
    float s2 = 0.f;
    if (w != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < KEEP; ++i)
            if (tid + 256 * i < nv) { old[i] = load4(x_in + base + 4 * (tid + 256 * i)); keep[i] = load_y(tid + 256 * i); }
#pragma unroll
        for (int i = 0; i < KEEP; ++i)
            if (tid + 256 * i < nv) ss = square(ss, keep[i]);
        for (int c = tid + 256 * KEEP; c < nv; c += 256) ss = square(ss, load_y(c));
        const float inv = 1.0f / sqrtf(block_sum_256(ss, part[0]) / (float)n + eps);
        auto add = [&](int c, const float4& v, float4 r) {
            const float4 g = load4(w + 4 * c);
            r.x += v.x * inv * g.x; r.y += v.y * inv * g.y; r.z += v.z * inv * g.z; r.w += v.w * inv * g.w;
            if constexpr (AVG) {
                store4(avg.hist + avg.n * avg.stride + base + 4 * c, r);
                const float own = __bfloat162float(avg.w[avg.n]);
                r.x *= own; r.y *= own; r.z *= own; r.w *= own;
#pragma unroll 4
                for (int j = 0; j < avg.n; ++j) {
                    const float k = __bfloat162float(avg.w[j]);
                    const float4 h = load4(avg.hist + j * avg.stride + base + 4 * c);
                    r.x = fmaf(k, h.x, r.x); r.y = fmaf(k, h.y, r.y); r.z = fmaf(k, h.z, r.z); r.w = fmaf(k, h.w, r.w);
                }
            }
            store4(x + base + 4 * c, r);
            if constexpr (PRE) s2 = square(s2, r);
            if (!PRE && out != nullptr) store4(out + base + 4 * c, r);
            return r;
        };
#pragma unroll
        for (int i = 0; i < KEEP; ++i)
            if (tid + 256 * i < nv) keep[i] = add(tid + 256 * i, keep[i], old[i]);
        for (int c = tid + 256 * KEEP; c < nv; c += 256) (void)add(c, load_y(c), load4(x_in + base + 4 * c));
    } else {
#pragma unroll
        for (int i = 0; i < KEEP; ++i)
            if (tid + 256 * i < nv) { keep[i] = load4(x + base + 4 * (tid + 256 * i)); s2 = square(s2, keep[i]); }
        for (int c = tid + 256 * KEEP; c < nv; c += 256) s2 = square(s2, load4(x + base + 4 * c));
        if (!PRE && out != nullptr)
            for (int c = tid; c < nv; c += 256) store4(out + base + 4 * c, load4(x + base + 4 * c));
    }
    if constexpr (!PRE) return;
    const float inv = 1.0f / sqrtf(block_sum_256(s2, part[1]) / (float)n + eps);
    auto emit = [&](int c, const float4& v) {
        const float4 g = load4(pre + 4 * c);
        store4(out + base + 4 * c, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (tid + 256 * i < nv) emit(tid + 256 * i, keep[i]);
    for (int c = tid + 256 * KEEP; c < nv; c += 256) emit(c, load4(x + base + 4 * c));
}

// Input convolution: out = x + sum_back w[taps - 1 - back] x_{t - back}, w [taps][ld]; rows before the pass come from the sequence's
// ring [taps][ld] (position modulo taps), which the thread with an entry's first rows brings up to date.  Grid (parts of a row, chunks of
// ROWS rows); a thread has four channels.  taps - 1 <= ROWS.
template <typename T, int TAPS, int ROWS>
__global__ void __launch_bounds__(128) input_conv_rows_kernel(const float* __restrict__ x, const __nv_bfloat16* __restrict__ w, T* __restrict__ out, int ld,
                                                              float* __restrict__ pool, size_t slot_stride, size_t offset, int taps_any, const RowPlan plan) {
    constexpr int MAXT = TAPS > 0 ? TAPS : kMaxConvTaps;
    const int taps = TAPS > 0 ? TAPS : taps_any, c = 4 * (blockIdx.x * 128 + threadIdx.x);
    RowEntry e;
    int t0;
    if (!locate_chunk<ROWS>(plan, blockIdx.y, e, t0) || c >= ld) return;
    const int n = min(ROWS, e.n - t0);
    float* ring = pool + (size_t)e.state * slot_stride + offset + c;
    const float* src = x + (size_t)(e.row0 + t0) * ld + c;
    T* dst = out + (size_t)(e.row0 + t0) * ld + c;
    float4 past[MAXT], k[MAXT], now[TAPS > 0 ? ROWS : 1];              // past[b]: the value b + 1 tokens back
    if constexpr (TAPS > 0) {
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            if (r < n) now[r] = load4(src + (size_t)r * ld);
    }
#pragma unroll
    for (int b = 0; b < MAXT; ++b) {
        past[b] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (b < taps) k[b] = load4(w + (size_t)(taps - 1 - b) * ld + c);
        const int t = t0 - 1 - b;
        if (b + 1 < taps && e.pos0 + t >= 0) past[b] = t >= 0 ? load4(src - (size_t)(b + 1) * ld) : load4(ring + (size_t)((e.pos0 + t) % taps) * ld);
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (r >= n) break;
        const float4 v = TAPS > 0 ? now[TAPS > 0 ? r : 0] : load4(src + (size_t)r * ld);
        float4 a = make_float4(fmaf(k[0].x, v.x, v.x), fmaf(k[0].y, v.y, v.y), fmaf(k[0].z, v.z, v.z), fmaf(k[0].w, v.w, v.w));
#pragma unroll
        for (int b = 0; b + 1 < MAXT; ++b)
            if (b + 1 < taps) {
                a.x = fmaf(k[b + 1].x, past[b].x, a.x); a.y = fmaf(k[b + 1].y, past[b].y, a.y);
                a.z = fmaf(k[b + 1].z, past[b].z, a.z); a.w = fmaf(k[b + 1].w, past[b].w, a.w);
            }
        store4(dst + (size_t)r * ld, a);
#pragma unroll
        for (int b = MAXT - 1; b > 0; --b) past[b] = past[b - 1];
        past[0] = v;
    }
    if (t0 == 0)
        for (int t = max(0, e.n - taps + 1); t < e.n; ++t) store4(ring + (size_t)((e.pos0 + t) % taps) * ld, load4(src + (size_t)t * ld));
}

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
    const float4 a = load4(p), b = load4(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) { unpack8(ld_cached(p), f); }
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
    store4(p, make_float4(f[0], f[1], f[2], f[3]));
    store4(p + 4, make_float4(f[4], f[5], f[6], f[7]));
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}

// out = c0 rms(z) + c1 rms(z^2) + c2 rms(z^3) + c3 over n channels; pads [n, ld) become zero.  One block per row; the first
// 8 * 256 * KEEP channels of the row stay in registers between the sums and the polynomial.
template <typename T>
__global__ void __launch_bounds__(256) poly_norm_rows_kernel(const T* __restrict__ z, T* __restrict__ out, const __nv_bfloat16* __restrict__ coef, int n,
                                                             int ld, float eps) {
    constexpr int KEEP = 4;
    __shared__ float part[3][8];
    const size_t base = (size_t)blockIdx.x * ld;
    const int nv = ld / 8;                                              // ld % 8 == 0, pads of z are zero
    float keep[KEEP][8];
    float s0 = 0.f, s1 = 0.f, s2 = 0.f;
    auto add = [&](const float (&f)[8]) {
#pragma unroll
        for (int j = 0; j < 8; ++j) { const float v2 = f[j] * f[j], v4 = v2 * v2; s0 += v2; s1 += v4; s2 = fmaf(v4, v2, s2); }
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if ((int)threadIdx.x + 256 * i < nv) load8(z + base + 8 * (threadIdx.x + 256 * i), keep[i]);
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if ((int)threadIdx.x + 256 * i < nv) add(keep[i]);
    for (int c = threadIdx.x + 256 * KEEP; c < nv; c += 256) { float f[8]; load8(z + base + 8 * c, f); add(f); }
    s0 = block_sum_256(s0, part[0]);
    s1 = block_sum_256(s1, part[1]);
    s2 = block_sum_256(s2, part[2]);
    const float c0 = __bfloat162float(coef[0]) / sqrtf(s0 / (float)n + eps), c1 = __bfloat162float(coef[1]) / sqrtf(s1 / (float)n + eps),
                c2 = __bfloat162float(coef[2]) / sqrtf(s2 / (float)n + eps), c3 = __bfloat162float(coef[3]);
    auto emit = [&](int c, const float (&f)[8]) {
        float r[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) r[j] = 8 * c + j < n ? fmaf(f[j], fmaf(f[j], fmaf(f[j], c2, c1), c0), c3) : 0.f;
        store8(out + base + 8 * c, r);
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if ((int)threadIdx.x + 256 * i < nv) emit(threadIdx.x + 256 * i, keep[i]);
    for (int c = threadIdx.x + 256 * KEEP; c < nv; c += 256) { float f[8]; load8(z + base + 8 * c, f); emit(c, f); }
}

// out[row][c] = gelu_tanh(s[row][c]) * table[id(row)][off + c] for c < n, zero in the pads.
template <typename T>
__global__ void __launch_bounds__(128) token_gate_rows_kernel(const float* __restrict__ s, const int32_t* __restrict__ ids,
                                                              const __nv_bfloat16* __restrict__ table, int table_ld, int off, int vocab,
                                                              T* __restrict__ out, int n, int ld) {
    const int row = blockIdx.x, id = ids[row];
    const bool ok = id >= 0 && id < vocab;
    const __nv_bfloat16* e = table + (size_t)(ok ? id : 0) * table_ld + off;
    for (int c = threadIdx.x; c < ld; c += 128)
        store_f32(out + (size_t)row * ld + c, ok && c < n ? gelu_tanh(s[(size_t)row * ld + c]) * __bfloat162float(e[c]) : 0.f);
}

// Elementwise input norm: x += mult * y, out = tanh(alpha x) w + b.  y: null (SUM: the experts' outputs of the row instead); w null: no
// output.  Grid (parts of a row, rows): a thread has four channels.
template <typename T, bool SUM>
__global__ void __launch_bounds__(256) add_tanh_rows_kernel(float* __restrict__ x, const float* __restrict__ y, float mult, T* __restrict__ out,
                                                            const __nv_bfloat16* __restrict__ w, const __nv_bfloat16* __restrict__ b,
                                                            const __nv_bfloat16* __restrict__ alpha, int ld, const SumOf<T> sum) {
    const int c = 4 * (blockIdx.x * 256 + threadIdx.x);
    const size_t row = blockIdx.y, base = row * ld;
    if (SUM && row == 0)
        for (int e = blockIdx.x * 256 + threadIdx.x; e < sum.experts; e += 256 * gridDim.x) sum.count[e] = 0;
    if (c >= ld) return;
    float4 r = load4(x + base + c);
    if (SUM || y != nullptr) {
        float4 a;
        if constexpr (SUM) {
            a = make_float4(0.f, 0.f, 0.f, 0.f);
            auto add = [&](float g, const float4& v) { a.x = fmaf(g, v.x, a.x); a.y = fmaf(g, v.y, a.y); a.z = fmaf(g, v.z, a.z); a.w = fmaf(g, v.w, a.w); };
            for (int k = 0; k < sum.top; ++k) {
                const size_t i = row * sum.top + k;
                add(sum.plain ? 1.0f : sum.weight[i], load4(sum.ye + (size_t)sum.place[i] * ld + c));
            }
            if (sum.shared != nullptr) add(sum.shared_weight[row], load4(sum.shared + base + c));
        } else {
            a = load4(y + base + c);
        }
        r.x = fmaf(mult, a.x, r.x); r.y = fmaf(mult, a.y, r.y); r.z = fmaf(mult, a.z, r.z); r.w = fmaf(mult, a.w, r.w);
        store4(x + base + c, r);
    }
    if (w == nullptr) return;
    const float al = __bfloat162float(*alpha);
    const float4 g = load4(w + c), h = load4(b + c);
    store4(out + base + c, make_float4(tanh_norm(r.x, al, g.x, h.x), tanh_norm(r.y, al, g.y, h.y), tanh_norm(r.z, al, g.z, h.z), tanh_norm(r.w, al, g.w, h.w)));
}

// out[i] = tanh(alpha x[rows[i]]) w + b
template <typename T>
__global__ void __launch_bounds__(256) gather_tanh_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, const __nv_bfloat16* __restrict__ w,
                                                               const __nv_bfloat16* __restrict__ b, const __nv_bfloat16* __restrict__ alpha, T* __restrict__ out, int ld) {
    const float al = __bfloat162float(*alpha);
    const float* src = x + (size_t)rows[blockIdx.x] * ld;
    for (int c = threadIdx.x; c < ld / 4; c += 256) {
        const float4 v = load4(src + 4 * c), g = load4(w + 4 * c), h = load4(b + 4 * c);
        store4(out + (size_t)blockIdx.x * ld + 4 * c,
               make_float4(tanh_norm(v.x, al, g.x, h.x), tanh_norm(v.y, al, g.y, h.y), tanh_norm(v.z, al, g.z, h.z), tanh_norm(v.w, al, g.w, h.w)));
    }
}

// logits in place; grid (parts of a row, rows)
__global__ void __launch_bounds__(256) cap_logits_rows_kernel(float* __restrict__ z, int n, int ld, float scale, float softcap) {
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c < n) z[(size_t)blockIdx.y * ld + c] = cap_logit(z[(size_t)blockIdx.y * ld + c], scale, softcap);
}

// z = relu(z)^2, n numbers, a multiple of 4
__global__ void __launch_bounds__(256) relu2_kernel(float* __restrict__ z, size_t n) {
    const size_t i = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= n) return;
    float4 v = load4(z + i);
    v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
    store4(z + i, make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w));
}

// out[i] = rms(x[rows[i]]) * w
template <typename T>
__global__ void __launch_bounds__(256) gather_norm_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows,
                                                               const __nv_bfloat16* __restrict__ w, T* __restrict__ out, int n, int ld, float eps) {
    __shared__ float part[8];
    const float* src = x + (size_t)rows[blockIdx.x] * ld;
    float ss = 0.f;
    for (int c = threadIdx.x; c < ld / 4; c += 256) {
        const float4 v = load4(src + 4 * c);
        ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum_256(ss, part) / (float)n + eps);
    for (int c = threadIdx.x; c < ld / 4; c += 256) {
        const float4 v = load4(src + 4 * c), g = load4(w + 4 * c);
        store4(out + (size_t)blockIdx.x * ld + 4 * c, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
    }
}

// C[M, N] = A[M, K] . W[N, K]^T in fp32 FMAs (fp32 activations, bf16 weights): the products of the all-32-bit mode and
// the small ones that feed a recurrence.  64 x 64 tiles, 256 threads, 4 x 4 outputs per thread.  bias may be null.  Grouped
// (group.tile not null): rows sorted by group as in gemm_tc.cuh, rows [group of the tile * group.rows, + N) of W.
struct RowGroups { const int4* tile; const int32_t* n_tiles; int rows; };
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, int lda, const __nv_bfloat16* __restrict__ W, int ldw,
                                                       float* __restrict__ C, int ldc, int M, int N, int K, const __nv_bfloat16* __restrict__ bias,
                                                       const RowGroups group) {
    __shared__ float as[16][64 + 4], ws[16][64 + 4];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    if (group.tile != nullptr) {
        const int t = m0 / kExpertTile;
        if (t >= *group.n_tiles) return;
        W += (size_t)group.tile[t].x * group.rows * ldw;
    }
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    const int lr = tid >> 2, lk = (tid & 3) * 4;
    for (int k0 = 0; k0 < K; k0 += 16) {                                // K % 4 == 0
        const bool kin = k0 + lk < K;
        const float4 a = kin && m0 + lr < M ? load4(A + (size_t)(m0 + lr) * lda + k0 + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 w = kin && n0 + lr < N ? load4(W + (size_t)(n0 + lr) * ldw + k0 + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
        __syncthreads();
        as[lk][lr] = a.x; as[lk + 1][lr] = a.y; as[lk + 2][lr] = a.z; as[lk + 3][lr] = a.w;
        ws[lk][lr] = w.x; ws[lk + 1][lr] = w.y; ws[lk + 2][lr] = w.z; ws[lk + 3][lr] = w.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float4 x = *reinterpret_cast<const float4*>(&as[k][ty * 4]), y = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
            const float xa[4] = {x.x, x.y, x.z, x.w}, ya[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xa[i], ya[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n < N) C[(size_t)m * ldc + n] = acc[i][j] + (bias != nullptr ? __bfloat162float(bias[n]) : 0.f);
        }
    }
}

}  // namespace efm
