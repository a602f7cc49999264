// Chunked form of the generalised delta rule (delta_rule.cuh) for many rows, fp32 throughout.  Inside a chunk of 16 tokens,
// with P_t the product of the chunk's decays up to t (per key channel, P_0 = 1) and S~_t = P_t^{-1} S_t,
//   S~_t = S~_{t-1} - b_t d_t^T + c_t v_t^T,   d_t = S~_{t-1}^T x_t,   o_t = S~_t^T q_t,
//   x_t = P_{t-1} u_t,   b_t = P_t^{-1} a_t u_t,   c_t = P_t^{-1} k_t,   q_t = P_t r_t.
// All d of a chunk solve one unit lower-triangular 16 x 16 system, so everything but the state can be prepared for every
// chunk at once (delta_prepare): with A = [x_t . b_s]_{s<t}, M = [x_t . c_s]_{s<t}, A' = [q_t . b_s]_{s<=t}, M' likewise,
//   X' = (I + A)^{-1} X,  V1 = (I + A)^{-1} M V,  Q' = Q - A' X',  O1 = M' V - A' V1.
// What is left in sequence (delta_chunk_scan, per head and 16 value channels) is a few small matrix products per chunk:
//   Y = X' S + V1,   O = Q' S + O1,   S <- P_16 (S + C^T V - B^T Y).
// Decays are at least e^{-0.61}, so P_16^{-1} stays below 2e4 and every factor of the dot products is of moderate size.
// A chunk that is cut short is filled with tokens that change nothing (w = 1, the rest 0).
// Packed chunk (floats, D padded to DP): XQ [DP][32] = X'^T | Q'^T, CB [32][DP] = C | -B, V, V1, O1 [16][DP], P [DP].
#pragma once
#include "delta_rule.cuh"

namespace efm {

namespace dc {
constexpr int C = 16, kThreads = 128, kCols = 16;
__host__ __device__ constexpr int pack_floats(int DP) { return 113 * DP; }

// Chunk `idx` of the pass -> entry, first token; false past the last chunk.  first: index of the entry's first chunk.
__device__ __forceinline__ bool locate(const RowPlan& plan, int idx, RowEntry& e, int& t0) {
    int at = 0;
    for (int i = 0; i < plan.n_entries; ++i) {
        e = plan.entry(i);
        const int n = (e.n + C - 1) / C;
        if (idx < at + n) { t0 = (idx - at) * C; return true; }
        at += n;
    }
    return false;
}

template <int DP>
struct PrepSmem {
    float xq[32][DP + 4];             // X rows, then Q rows
    float bc[32][DP + 4];             // B rows, then C rows
    float w[C][DP];
    float v[C][DP];
    float g[32][36];                  // masked products: rows x / q, columns b | c
};
template <int DP>
struct ScanSmem {
    float xq[2][DP][40];
    float cb[2][32][DP];
    float vin[2][3][C][kCols];        // V | V1 | O1
    float p[2][DP];
    float s[DP][kCols];
    float y[C][kCols];
};
}  // namespace dc

// grid (chunks, heads)
template <int DP>
__global__ void __launch_bounds__(dc::kThreads) delta_prepare_kernel(const float* __restrict__ proj, const float* __restrict__ decay_in, int ld_decay,
                                                                     float* __restrict__ pack, const DeltaShape s, const RowPlan plan) {
    using namespace dc;
    extern __shared__ __align__(16) unsigned char dc_smem[];
    PrepSmem<DP>& sm = *reinterpret_cast<PrepSmem<DP>*>(dc_smem);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, HD = s.heads * s.D, c0 = h * s.D;
    RowEntry e;
    int t0;
    if (!locate(plan, blockIdx.x, e, t0)) return;
    const int nv = min(C, e.n - t0);
    // ---- step inputs: a warp per token ----------------------------------------------------------------------------
    for (int t = warp; t < C; t += 4) {
        const size_t row = (size_t)(e.row0 + t0 + t);
        const float* x = proj + row * s.ld + c0;
        const float* dec = decay_in + row * ld_decay + c0;
        float k[DP / 32], ss = 0.f;
#pragma unroll
        for (int i = 0; i < DP / 32; ++i) {
            const int d = lane + 32 * i;
            k[i] = t < nv && d < s.D ? x[HD + d] : 0.f;
            ss = fmaf(k[i], k[i], ss);
        }
        const float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
#pragma unroll
        for (int i = 0; i < DP / 32; ++i) {
            const int d = lane + 32 * i;
            const bool in = t < nv && d < s.D;
            const float u = k[i] * inv;
            sm.xq[t][d] = u;
            sm.xq[C + t][d] = in ? x[d] : 0.f;
            sm.bc[t][d] = in ? sigmoid_f(x[4 * HD + d] + __bfloat162float(s.a_bias[c0 + d])) * u : 0.f;
            sm.bc[C + t][d] = k[i];
            sm.w[t][d] = in ? expf(-kDecayRate * sigmoid_f(dec[d] + __bfloat162float(s.w0[c0 + d]))) : 1.f;
            sm.v[t][d] = in ? x[2 * HD + d] : 0.f;
        }
    }
    __syncthreads();
    float* out = pack + ((size_t)blockIdx.x * s.heads + h) * pack_floats(DP);
    float* o_cb = out + 32 * DP;
    float* o_v = out + 64 * DP;
    // ---- decay products, a thread per channel ----------------------------------------------------------------------
    if (tid < DP) {
        float P = 1.f;
#pragma unroll
        for (int t = 0; t < C; ++t) {
            sm.xq[t][tid] *= P;
            P *= sm.w[t][tid];
            const float inv = 1.0f / P;
            sm.xq[C + t][tid] *= P;
            const float b = sm.bc[t][tid] * inv, c = sm.bc[C + t][tid] * inv;
            sm.bc[t][tid] = b;
            sm.bc[C + t][tid] = c;
            o_cb[t * DP + tid] = c;
            o_cb[(C + t) * DP + tid] = -b;
        }
        out[112 * DP + tid] = P;
    }
    __syncthreads();
    // ---- 32 x 32 products, 2 x 4 per thread ------------------------------------------------------------------------
    {
        const int ct = tid & 7, rt = tid >> 3;
        float acc[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 4
        for (int d = 0; d < DP; d += 4) {
            float4 a[2], b[4];
#pragma unroll
            for (int i = 0; i < 2; ++i) a[i] = *reinterpret_cast<const float4*>(&sm.xq[i * 16 + rt][d]);
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = *reinterpret_cast<const float4*>(&sm.bc[j * 8 + ct][d]);
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(a[i].x, b[j].x, acc[i][j]); acc[i][j] = fmaf(a[i].y, b[j].y, acc[i][j]);
                    acc[i][j] = fmaf(a[i].z, b[j].z, acc[i][j]); acc[i][j] = fmaf(a[i].w, b[j].w, acc[i][j]);
                }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int col = j * 8 + ct, src = col & 15;
                sm.g[i * 16 + rt][col] = (i == 0 ? src < rt : src <= rt) ? acc[i][j] : 0.f;
            }
    }
    __syncthreads();
    // ---- triangular solves: a thread per channel of X' / Q' or of V1 / O1 ------------------------------------------
    for (int role = tid; role < 2 * DP; role += kThreads) {
        if (role < DP) {
            float x[C], y[C];
#pragma unroll
            for (int t = 0; t < C; ++t) {
                float a = sm.xq[t][role];
#pragma unroll
                for (int q = 0; q < t; ++q) a = fmaf(-sm.g[t][q], x[q], a);
                x[t] = a;
            }
            float4* dst = reinterpret_cast<float4*>(out + role * 32);
#pragma unroll
            for (int t = 0; t < C; t += 4) dst[t / 4] = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
#pragma unroll
            for (int t = 0; t < C; ++t) {
                float a = sm.xq[C + t][role];
#pragma unroll
                for (int q = 0; q <= t; ++q) a = fmaf(-sm.g[C + t][q], x[q], a);
                y[t] = a;
            }
#pragma unroll
            for (int t = 0; t < C; t += 4) dst[4 + t / 4] = make_float4(y[t], y[t + 1], y[t + 2], y[t + 3]);
        } else {
            const int ch = role - DP;
            float v[C], v1[C];
#pragma unroll
            for (int t = 0; t < C; ++t) { v[t] = sm.v[t][ch]; o_v[t * DP + ch] = v[t]; }
#pragma unroll
            for (int t = 0; t < C; ++t) {
                float a = 0.f;
#pragma unroll
                for (int q = 0; q < t; ++q) a = fmaf(sm.g[t][C + q], v[q], fmaf(-sm.g[t][q], v1[q], a));
                v1[t] = a;
                o_v[(C + t) * DP + ch] = a;
            }
#pragma unroll
            for (int t = 0; t < C; ++t) {
                float a = 0.f;
#pragma unroll
                for (int q = 0; q <= t; ++q) a = fmaf(sm.g[C + t][C + q], v[q], fmaf(-sm.g[C + t][q], v1[q], a));
                o_v[(2 * C + t) * DP + ch] = a;
            }
        }
    }
}

// grid (heads * ceil(DP / 16), entries): the sequential part for 16 value channels of one head.
template <int DP>
__global__ void __launch_bounds__(dc::kThreads) delta_chunk_scan_kernel(const float* __restrict__ pack, float* __restrict__ o, int ld_o,
                                                                        float* __restrict__ pool, size_t slot_stride, size_t offset, const DeltaShape s,
                                                                        const RowPlan plan) {
    using namespace dc;
    using ds::cp16;
    constexpr int CT = DP == 32 ? 1 : (DP == 64 ? 2 : 4);          // state columns per thread (4 rows each)
    constexpr int RT = DP / 4;                                     // row tiles of the state
    constexpr int GROUPS = DP / kCols;
    extern __shared__ __align__(16) unsigned char dc_smem[];
    ScanSmem<DP>& sm = *reinterpret_cast<ScanSmem<DP>*>(dc_smem);
    const int h = blockIdx.x / GROUPS, c0 = (blockIdx.x % GROUPS) * kCols;
    if (c0 >= s.D) return;
    const RowEntry e = plan.entry(blockIdx.y);
    int chunk0 = 0;
    for (int i = 0; i < (int)blockIdx.y; ++i) chunk0 += (plan.entry(i).n + C - 1) / C;
    const int n_chunks = (e.n + C - 1) / C;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    auto stage = [&](int c, int b) {
        const float* src = pack + ((size_t)(chunk0 + c) * s.heads + h) * pack_floats(DP);
        for (int i = tid; i < DP * 8; i += kThreads) cp16(&sm.xq[b][i >> 3][(i & 7) * 4], src + i * 4);
        for (int i = tid; i < DP * 8; i += kThreads) cp16(&sm.cb[b][0][0] + i * 4, src + 32 * DP + i * 4);
        for (int i = tid; i < 3 * C * 4; i += kThreads) cp16(&sm.vin[b][0][i >> 2][(i & 3) * 4], src + 64 * DP + (i >> 2) * DP + c0 + (i & 3) * 4);
        if (tid < DP / 4) cp16(&sm.p[b][tid * 4], src + 112 * DP + tid * 4);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    // this thread's tile of the state: rows 4 it .. 4 it + 3, columns CT jt ..
    const int it = tid % RT, jt = tid / RT;
    const bool own = jt < kCols / CT;
    float* st = pool + (size_t)e.state * slot_stride + offset + (size_t)h * s.D * s.D + c0 + CT * jt;
    float S[4][CT];
    if (own) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < CT; ++j) {
                const int r = 4 * it + i;
                S[i][j] = e.pos0 > 0 && r < s.D && c0 + CT * jt + j < s.D ? st[(size_t)r * s.D + j] : 0.f;
                sm.s[r][CT * jt + j] = S[i][j];
            }
    }
    // first product: 4 x 4 outputs per thread, k split over the four lanes of a quad
    const int ks = lane & 3, ct = (lane >> 2) & 3, rt = (lane >> 4) | (warp << 1);
    for (int c = 0; c < n_chunks; ++c) {
        const int b = c & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                           // chunk c has landed, the state is written, the other buffer is free
        if (c + 1 < n_chunks) stage(c + 1, b ^ 1);
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 8
        for (int k = 0; k < DP / 4; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&sm.xq[b][4 * k + ks][rt * 4]);
            const float4 y = *reinterpret_cast<const float4*>(&sm.s[4 * k + ks][ct * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], yv[j], acc[i][j]);
        }
        // sum over the quad; lane ks keeps row ks of the tile
        float half[2][4], rowv[4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float mine = ks & 1 ? acc[2 * i + 1][j] : acc[2 * i][j], other = ks & 1 ? acc[2 * i][j] : acc[2 * i + 1][j];
                half[i][j] = mine + __shfl_xor_sync(0xffffffffu, other, 1);
            }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float mine = ks & 2 ? half[1][j] : half[0][j], other = ks & 2 ? half[0][j] : half[1][j];
            rowv[j] = mine + __shfl_xor_sync(0xffffffffu, other, 2);
        }
        const int row = rt * 4 + ks;
        if (row < C) {
            const float4 v1 = *reinterpret_cast<const float4*>(&sm.vin[b][1][row][ct * 4]);
            *reinterpret_cast<float4*>(&sm.y[row][ct * 4]) = make_float4(rowv[0] + v1.x, rowv[1] + v1.y, rowv[2] + v1.z, rowv[3] + v1.w);
        } else if (c * C + row - C < e.n) {
            const float4 o1 = *reinterpret_cast<const float4*>(&sm.vin[b][2][row - C][ct * 4]);
            float* dst = o + (size_t)(e.row0 + c * C + row - C) * ld_o + h * s.D + c0 + ct * 4;
            const float r[4] = {rowv[0] + o1.x, rowv[1] + o1.y, rowv[2] + o1.z, rowv[3] + o1.w};
            if ((s.D & 3) == 0) {
                if (c0 + ct * 4 < s.D) *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (c0 + ct * 4 + j < s.D) dst[j] = r[j];
            }
        }
        __syncthreads();
        if (own) {
            float u[4][CT];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < CT; ++j) u[i][j] = S[i][j];
#pragma unroll 8
            for (int k = 0; k < 32; ++k) {
                const float4 a = *reinterpret_cast<const float4*>(&sm.cb[b][k][4 * it]);
                const float* vy = k < C ? &sm.vin[b][0][k][CT * jt] : &sm.y[k - C][CT * jt];
                const float av[4] = {a.x, a.y, a.z, a.w};
                float yv[CT];
#pragma unroll
                for (int j = 0; j < CT; ++j) yv[j] = vy[j];
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < CT; ++j) u[i][j] = fmaf(av[i], yv[j], u[i][j]);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < CT; ++j) {
                    S[i][j] = u[i][j] * sm.p[b][4 * it + i];
                    sm.s[4 * it + i][CT * jt + j] = S[i][j];
                }
        }
    }
    if (own) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < CT; ++j) {
                const int r = 4 * it + i;
                if (r < s.D && c0 + CT * jt + j < s.D) st[(size_t)r * s.D + j] = S[i][j];
            }
    }
}

}  // namespace efm
