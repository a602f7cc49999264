// Generalised delta rule with per-channel decay: per head a state S [D key channels x D value channels], fp32,
//   S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,   o_t = S_t^T r_t,   u_t = k_t / sqrt(|k_t|^2 + 1e-6)
//   w_t = exp(-e^{-1/2} sigmoid(W2 tanh(W1 x) + w0)),   a_t = sigmoid(A x + b)
// followed by a per-head RMS norm of o, a plain weight and a sigmoid gate.  Everything here is fp32; the projections
// arrive as one fp32 row [r | k | v | g | a | W1 x] (segments of heads * D, the last of `rank`).
//
//   delta_tanh_rows, delta_inputs_rows   many rows: step inputs (w, a u, u, k, r, v) packed per (row, head)
//   delta_scan                           many rows: the recurrence, token by token, one block per (entry, head, 16 value
//                                        channels); 8 lanes share a state column, inputs stream through shared memory
//   delta_output_rows                    many rows: head norm, weight, gate
//   delta_decode                         one row: all of it in one launch, one block per head
// State pool: [slots][slot_stride] floats, this layer at `offset`, head h at + h * D * D, row = key channel.
#pragma once
#include "common.cuh"
#include "row_plan.cuh"
#include "window_attention.cuh"

namespace efm {

struct DeltaShape {
    int heads, D, Dp;                 // Dp: D rounded up to 32 (packed inputs)
    int rank;                         // of the decay projection
    int ld;                           // row length of the projections
    float eps;
    const __nv_bfloat16* w0;          // [heads * D]
    const __nv_bfloat16* a_bias;      // [heads * D]
    const __nv_bfloat16* norm;        // [heads * D]
};

__device__ __forceinline__ void store_vec4(float* p, const float (&r)[4]) { *reinterpret_cast<float4*>(p) = make_float4(r[0], r[1], r[2], r[3]); }
__device__ __forceinline__ void store_vec4(__nv_bfloat16* p, const float (&r)[4]) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r[0], r[1]), pack_bf16(r[2], r[3])); }
constexpr float kDecayRate = 0.6065306597126334f;      // e^{-1/2}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

// out[row][0 .. ld_out) = tanh of the last projection segment, zero-padded
__global__ void __launch_bounds__(128) delta_tanh_rows_kernel(const float* __restrict__ proj, float* __restrict__ out, int ld_out, const DeltaShape s) {
    const float* src = proj + (size_t)blockIdx.x * s.ld + 5 * s.heads * s.D;
    for (int i = threadIdx.x; i < ld_out; i += 128) out[(size_t)blockIdx.x * ld_out + i] = i < s.rank ? tanhf(src[i]) : 0.f;
}

enum : int { kDeltaW = 0, kDeltaAU = 1, kDeltaU = 2, kDeltaK = 3, kDeltaR = 4, kDeltaV = 5, kDeltaParts = 6 };

// pack[(row * heads + h) * 6 + part][Dp]; decay_in [rows][ld_decay] = W2 tanh(W1 x)
__global__ void __launch_bounds__(256) delta_inputs_rows_kernel(const float* __restrict__ proj, const float* __restrict__ decay_in, int ld_decay,
                                                                float* __restrict__ pack, const DeltaShape s) {
    const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int HD = s.heads * s.D;
    const float* x = proj + (size_t)row * s.ld;
    for (int h = warp; h < s.heads; h += 8) {
        const int c0 = h * s.D;
        float ss = 0.f;
        for (int d = lane; d < s.D; d += 32) { const float k = x[HD + c0 + d]; ss = fmaf(k, k, ss); }
        const float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
        float* dst = pack + ((size_t)row * s.heads + h) * kDeltaParts * s.Dp;
        for (int d = lane; d < s.Dp; d += 32) {
            float w = 0.f, au = 0.f, u = 0.f, k = 0.f, r = 0.f, v = 0.f;
            if (d < s.D) {
                r = x[c0 + d];
                k = x[HD + c0 + d];
                v = x[2 * HD + c0 + d];
                u = k * inv;
                au = sigmoid_f(x[4 * HD + c0 + d] + __bfloat162float(s.a_bias[c0 + d])) * u;
                w = expf(-kDecayRate * sigmoid_f(decay_in[(size_t)row * ld_decay + c0 + d] + __bfloat162float(s.w0[c0 + d])));
            }
            dst[kDeltaW * s.Dp + d] = w;
            dst[kDeltaAU * s.Dp + d] = au;
            dst[kDeltaU * s.Dp + d] = u;
            dst[kDeltaK * s.Dp + d] = k;
            dst[kDeltaR * s.Dp + d] = r;
            dst[kDeltaV * s.Dp + d] = v;
        }
    }
}

namespace ds {
constexpr int kThreads = 128, kCols = kThreads / 8, kBatch = 8;        // value channels per block, tokens per staged batch
inline size_t smem_bytes(int Dp) { return (size_t)2 * kBatch * (5 * Dp + kCols) * sizeof(float); }
__device__ __forceinline__ void cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
}  // namespace ds

// grid (heads * ceil(Dp / 16), entries).  NC = Dp / 32: float4 chunks of a state column per lane.
template <int NC>
__global__ void __launch_bounds__(ds::kThreads) delta_scan_kernel(const float* __restrict__ pack, float* __restrict__ o, int ld_o,
                                                                  float* __restrict__ pool, size_t slot_stride, size_t offset, const DeltaShape s,
                                                                  const RowPlan plan) {
    using namespace ds;
    extern __shared__ __align__(16) float ds_smem[];
    const int Dp = NC * 32, step_f = 5 * Dp + kCols;
    const int groups = (s.Dp + kCols - 1) / kCols;
    const int h = blockIdx.x / groups, c0 = (blockIdx.x % groups) * kCols;
    if (c0 >= s.D) return;
    const RowEntry e = plan.entry(blockIdx.y);
    const int tid = threadIdx.x, col = tid >> 3, l8 = tid & 7;
    const bool col_ok = c0 + col < s.D;
    float* st = pool + (size_t)e.state * slot_stride + offset + (size_t)h * s.D * s.D + c0 + col;
    float S[NC][4];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = (c * 8 + l8) * 4 + j;
            S[c][j] = (e.pos0 > 0 && col_ok && i < s.D) ? st[(size_t)i * s.D] : 0.f;
        }
    auto stage = [&](int t0, int buf) {                                // tokens t0 .. t0 + kBatch of the entry
        const int n = min(kBatch, e.n - t0);
        const int per = 5 * Dp / 4 + kCols / 4;
        for (int i = tid; i < n * per; i += kThreads) {
            const int t = i / per, c = i - t * per;
            const float* src = pack + ((size_t)(e.row0 + t0 + t) * s.heads + h) * kDeltaParts * Dp;
            float* dst = ds_smem + ((size_t)buf * kBatch + t) * step_f;
            if (c < 5 * Dp / 4) cp16(dst + c * 4, src + c * 4);
            else cp16(dst + c * 4, src + kDeltaV * Dp + c0 + (c - 5 * Dp / 4) * 4);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    for (int t0 = 0, b = 0; t0 < e.n; t0 += kBatch, b ^= 1) {
        if (t0 + kBatch < e.n) {
            stage(t0 + kBatch, b ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int n = min(kBatch, e.n - t0);
        for (int t = 0; t < n; ++t) {
            const float* in = ds_smem + ((size_t)b * kBatch + t) * step_f;
            const float4* w4 = reinterpret_cast<const float4*>(in + kDeltaW * Dp) + l8;
            const float4* a4 = reinterpret_cast<const float4*>(in + kDeltaAU * Dp) + l8;
            const float4* u4 = reinterpret_cast<const float4*>(in + kDeltaU * Dp) + l8;
            const float4* k4 = reinterpret_cast<const float4*>(in + kDeltaK * Dp) + l8;
            const float4* r4 = reinterpret_cast<const float4*>(in + kDeltaR * Dp) + l8;
            const float v = in[5 * Dp + col];
            float d0 = 0.f, d1 = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float4 u = u4[c * 8];
                d0 = fmaf(u.x, S[c][0], d0); d1 = fmaf(u.y, S[c][1], d1);
                d0 = fmaf(u.z, S[c][2], d0); d1 = fmaf(u.w, S[c][3], d1);
            }
            float d = d0 + d1;
#pragma unroll
            for (int x = 4; x > 0; x >>= 1) d += __shfl_xor_sync(0xffffffffu, d, x);
            float q0 = 0.f, q1 = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float4 w = w4[c * 8], a = a4[c * 8], k = k4[c * 8], r = r4[c * 8];
                S[c][0] = fmaf(w.x, S[c][0], fmaf(k.x, v, -a.x * d));
                S[c][1] = fmaf(w.y, S[c][1], fmaf(k.y, v, -a.y * d));
                S[c][2] = fmaf(w.z, S[c][2], fmaf(k.z, v, -a.z * d));
                S[c][3] = fmaf(w.w, S[c][3], fmaf(k.w, v, -a.w * d));
                q0 = fmaf(r.x, S[c][0], q0); q1 = fmaf(r.y, S[c][1], q1);
                q0 = fmaf(r.z, S[c][2], q0); q1 = fmaf(r.w, S[c][3], q1);
            }
            float q = q0 + q1;
#pragma unroll
            for (int x = 4; x > 0; x >>= 1) q += __shfl_xor_sync(0xffffffffu, q, x);
            if (l8 == 0 && col_ok) o[(size_t)(e.row0 + t0 + t) * ld_o + h * s.D + c0 + col] = q;
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = (c * 8 + l8) * 4 + j;
            if (col_ok && i < s.D) st[(size_t)i * s.D] = S[c][j];
        }
}

// out[row] = rms(o per head) * norm * sigmoid(g), row length ld_out (pads untouched).  One block per row; `lanes` (a power
// of two, at least D / 4 where possible) threads share a head, four channels at a time.
template <typename TO>
__global__ void __launch_bounds__(256) delta_output_rows_kernel(const float* __restrict__ o, int ld_o, const float* __restrict__ proj, TO* __restrict__ out,
                                                                int ld_out, const DeltaShape s, int lanes) {
    const int row = blockIdx.x, HD = s.heads * s.D, l = threadIdx.x & (lanes - 1), per = 256 / lanes;
    const float* orow = o + (size_t)row * ld_o;
    const float* grow = proj + (size_t)row * s.ld + 3 * HD;
    TO* dst = out + (size_t)row * ld_out;
    const bool vec = (s.D & 3) == 0;
    for (int h0 = 0; h0 < s.heads; h0 += per) {                    // every thread takes part in the shuffles
        const int h = h0 + threadIdx.x / lanes, c0 = h * s.D;
        const bool in = h < s.heads;
        float ss = 0.f;
        if (in)
            for (int d = 4 * l; d < s.D; d += 4 * lanes) {
                if (vec) {
                    const float4 v = *reinterpret_cast<const float4*>(orow + c0 + d);
                    ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
                } else {
                    for (int j = d; j < min(d + 4, s.D); ++j) ss = fmaf(orow[c0 + j], orow[c0 + j], ss);
                }
            }
        for (int x = lanes / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
        if (!in) continue;
        const float inv = 1.0f / sqrtf(ss / (float)s.D + s.eps);
        for (int d = 4 * l; d < s.D; d += 4 * lanes) {
            if (vec) {
                const float4 v = *reinterpret_cast<const float4*>(orow + c0 + d), g = *reinterpret_cast<const float4*>(grow + c0 + d);
                const uint2 w = *reinterpret_cast<const uint2*>(s.norm + c0 + d);
                const float r[4] = {v.x * inv * bf16lo(w.x) * sigmoid_f(g.x), v.y * inv * bf16hi(w.x) * sigmoid_f(g.y),
                                    v.z * inv * bf16lo(w.y) * sigmoid_f(g.z), v.w * inv * bf16hi(w.y) * sigmoid_f(g.w)};
                store_vec4(dst + c0 + d, r);
            } else {
                for (int j = d; j < min(d + 4, s.D); ++j)
                    store_f32(dst + c0 + j, orow[c0 + j] * inv * __bfloat162float(s.norm[c0 + j]) * sigmoid_f(grow[c0 + j]));
            }
        }
    }
}

struct DeltaDecodeParams {
    DeltaShape s;
    const float* proj;                // one row
    const __nv_bfloat16* w2;          // [heads * D][ld_w2]
    int ld_w2;
    float* pool;                      // this layer's state of the sequence
    DecodeState* state;
    float* out;                       // [heads * D]
    int early;                        // 1: the state may be read before the dependency wait
};

// One block per head.  Threads = D columns x RG row groups; RPT = state rows per thread held in registers (0: D > 128,
// the state is read twice).
template <int RPT>
__global__ void __launch_bounds__(512) delta_decode_kernel(const DeltaDecodeParams p) {
    constexpr int NT = 512;
    __shared__ float sa[256], sw[256], sau[256], su[256], sk[256], sr[256], sv[256], tw[512], red[NT], dot[256], part[16];
    const DeltaShape& s = p.s;
    const int D = s.D, HD = s.heads * D, h = blockIdx.x, c0 = h * D;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int RG = NT / D, rg = tid / D, col = tid - rg * D;
    const bool act = rg < RG;
    float* S = p.pool + (size_t)h * D * D + col;
    constexpr int R = RPT > 0 ? RPT : 1;
    float reg[R];
    uint4 w2_first = make_uint4(0u, 0u, 0u, 0u);                       // weights: independent of earlier launches
    if ((tid >> 3) < D && (tid & 7) * 8 < p.ld_w2) w2_first = ld_cached(p.w2 + (size_t)(c0 + (tid >> 3)) * p.ld_w2 + (tid & 7) * 8);
    if (!p.early) { pdl_wait(); pdl_launch_dependents(); }
    const bool fresh = p.state->kv_len <= 1u;                          // first token: the state is zero
    if (RPT > 0 && act) {
#pragma unroll
        for (int n = 0; n < R; ++n) {
            const int i = rg + RG * n;
            reg[n] = (i < D && !fresh) ? __ldcg(S + (size_t)i * D) : 0.f;
        }
    }
    if (p.early) { pdl_wait(); pdl_launch_dependents(); }
    for (int i = tid; i < p.ld_w2; i += NT) tw[i] = i < s.rank ? tanhf(__ldcg(p.proj + 5 * HD + i)) : 0.f;
    float ss = 0.f;
    for (int d = tid; d < D; d += NT) {
        const float k = __ldcg(p.proj + HD + c0 + d);
        sk[d] = k;
        sr[d] = __ldcg(p.proj + c0 + d);
        sv[d] = __ldcg(p.proj + 2 * HD + c0 + d);
        sa[d] = __ldcg(p.proj + 4 * HD + c0 + d);
        ss = fmaf(k, k, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 16; ++w) tot += part[w];
    const float inv = 1.0f / sqrtf(tot + 1e-6f);
    for (int d = tid >> 3; d < D; d += NT / 8) {                       // decay: eight lanes per channel
        float a = 0.f;
        for (int i = (tid & 7) * 8; i < p.ld_w2; i += 64) {
            float f[8];
            unpack8(d == (tid >> 3) && i == (tid & 7) * 8 ? w2_first : ld_cached(p.w2 + (size_t)(c0 + d) * p.ld_w2 + i), f);
#pragma unroll
            for (int j = 0; j < 8; ++j) a = fmaf(f[j], tw[i + j], a);
        }
#pragma unroll
        for (int x = 4; x > 0; x >>= 1) a += __shfl_xor_sync(0xffffffffu, a, x);
        if ((tid & 7) == 0) {
            sw[d] = expf(-kDecayRate * sigmoid_f(a + __bfloat162float(s.w0[c0 + d])));
            const float u = sk[d] * inv;
            su[d] = u;
            sau[d] = sigmoid_f(sa[d] + __bfloat162float(s.a_bias[c0 + d])) * u;
        }
    }
    __syncthreads();
    float a = 0.f;
    if (act) {
        if constexpr (RPT > 0) {
#pragma unroll
            for (int n = 0; n < R; ++n) {
                const int i = rg + RG * n;
                if (i < D) a = fmaf(su[i], reg[n], a);
            }
        } else if (!fresh) {
            for (int i = rg; i < D; i += RG) a = fmaf(su[i], __ldcg(S + (size_t)i * D), a);
        }
    }
    red[tid] = a;
    __syncthreads();
    for (int d = tid; d < D; d += NT) {
        float t = 0.f;
        for (int g = 0; g < RG; ++g) t += red[g * D + d];
        dot[d] = t;
    }
    __syncthreads();
    float q = 0.f;
    if (act) {
        const float dc = dot[col], v = sv[col];
        if constexpr (RPT > 0) {
#pragma unroll
            for (int n = 0; n < R; ++n) {
                const int i = rg + RG * n;
                if (i < D) {
                    const float x = fmaf(sw[i], reg[n], fmaf(sk[i], v, -sau[i] * dc));
                    S[(size_t)i * D] = x;
                    q = fmaf(sr[i], x, q);
                }
            }
        } else {
            for (int i = rg; i < D; i += RG) {
                const float x = fmaf(sw[i], fresh ? 0.f : __ldcg(S + (size_t)i * D), fmaf(sk[i], v, -sau[i] * dc));
                S[(size_t)i * D] = x;
                q = fmaf(sr[i], x, q);
            }
        }
    }
    red[tid] = q;
    __syncthreads();
    float o = 0.f;
    if (tid < D) {
        for (int g = 0; g < RG; ++g) o += red[g * D + tid];
    }
    ss = warp_sum(tid < D ? o * o : 0.f);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    if (tid < D) {
        tot = 0.f;
#pragma unroll
        for (int w = 0; w < 16; ++w) tot += part[w];
        p.out[c0 + tid] = o / sqrtf(tot / (float)D + s.eps) * __bfloat162float(s.norm[c0 + tid]) * sigmoid_f(__ldcg(p.proj + 3 * HD + c0 + tid));
    }
}

}  // namespace efm
