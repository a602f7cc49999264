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
// Packed chunk (floats, D padded to DP): XQ [32][DP] = X' | Q', CB [32][DP] = C | -B, V, V1, O1 [16][DP], P [DP].
#pragma once
#include "delta_rule.cuh"

namespace efm {

namespace dc {
constexpr int C = 16, kThreads = 128, kScanThreads = 256, kCols = 16;
__host__ __device__ constexpr int pack_floats(int DP) { return 113 * DP; }

template <int DP>
struct PrepSmem {
    float xq[32][DP + 4];             // X rows, then Q rows
    float bc[32][DP + 4];             // B rows, then C rows
    float w[C][DP];
    float v[C][DP];
    float g[32][36];                  // masked products, transposed: [b | c of token s][x | q of token t]
};
template <int DP>
struct ScanSmem {
    float xq[2][32][DP + 4];
    float cb[2][32][DP];
    float vin[2][3][C][kCols];        // V | V1 | O1
    float p[2][DP];
    float st[kCols][DP + 4];          // the state, transposed
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
    if (!locate_chunk<C>(plan, blockIdx.x, e, t0)) return;
    const int nv = min(C, e.n - t0);
    // ---- step inputs: a warp per token ----------------------------------------------------------------------------
    constexpr int NT = C / 4, NI = DP / 32;
    float k[NT][NI], r[NT][NI], v[NT][NI], a[NT][NI], dec[NT][NI];
#pragma unroll
    for (int q = 0; q < NT; ++q) {
        const int t = warp + 4 * q;
        const size_t row = (size_t)(e.row0 + t0 + t);
        const float* x = proj + row * s.ld + c0;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = lane + 32 * i;
            const bool in = t < nv && d < s.D;
            r[q][i] = in ? x[d] : 0.f;
            k[q][i] = in ? x[HD + d] : 0.f;
            v[q][i] = in ? x[2 * HD + d] : 0.f;
            a[q][i] = in ? x[4 * HD + d] : 0.f;
            dec[q][i] = in ? decay_in[row * ld_decay + c0 + d] : 0.f;
        }
    }
#pragma unroll
    for (int q = 0; q < NT; ++q) {
        const int t = warp + 4 * q;
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) ss = fmaf(k[q][i], k[q][i], ss);
        const float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = lane + 32 * i;
            const bool in = t < nv && d < s.D;
            const float u = k[q][i] * inv;
            sm.xq[t][d] = u;
            sm.xq[C + t][d] = r[q][i];
            sm.bc[t][d] = in ? sigmoid_f(a[q][i] + __bfloat162float(s.a_bias[c0 + d])) * u : 0.f;
            sm.bc[C + t][d] = k[q][i];
            sm.w[t][d] = in ? expf(-kDecayRate * sigmoid_f(dec[q][i] + __bfloat162float(s.w0[c0 + d]))) : 1.f;
            sm.v[t][d] = v[q][i];
        }
    }
    __syncthreads();
    float* out = pack + ((size_t)blockIdx.x * s.heads + h) * pack_floats(DP);
    float* o_cb = out + 32 * DP;
    float* o_v = out + 64 * DP;
    // ---- decay products: two threads per channel, half of the tokens each -------------------------------------------
    for (int r = tid; r < 2 * DP; r += kThreads) {
        const int ch = r % DP, half = (r / DP) * (C / 2);
        float w[C], P = 1.f;
#pragma unroll
        for (int t = 0; t < C; ++t) w[t] = sm.w[t][ch];
        float before[C / 2], after[C / 2];
#pragma unroll
        for (int t = 0; t < C; ++t) {
            const float prev = P;
            P *= w[t];
            if (t < C / 2 ? half == 0 : half != 0) { before[t % (C / 2)] = prev; after[t % (C / 2)] = P; }
        }
#pragma unroll
        for (int q = 0; q < C / 2; ++q) {
            const int t = half + q;
            const float inv = 1.0f / after[q];
            sm.xq[t][ch] *= before[q];
            sm.xq[C + t][ch] *= after[q];
            const float b = sm.bc[t][ch] * inv, c = sm.bc[C + t][ch] * inv;
            sm.bc[t][ch] = b;
            sm.bc[C + t][ch] = c;
            o_cb[t * DP + ch] = c;
            o_cb[(C + t) * DP + ch] = -b;
        }
        if (half != 0) out[112 * DP + ch] = P;
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
sm.g[col][i * 16 + rt] = (i == 0 ? src < rt : src <= rt) ? acc[i][j] : 0.f;
            }
    }
    __syncthreads();
    // ---- triangular solves, a thread per channel of X' / Q' or of V1 / O1: once token q is solved, its share leaves every
    // later row (independent multiply-adds, coefficients of one q are consecutive)
    for (int role = tid; role < 2 * DP; role += kThreads) {
        const bool is_x = role < DP;
        const int ch = is_x ? role : role - DP;
        float x[C], y[C];
        auto subtract = [&](int q, float v, int col, float sign) {
#pragma unroll
            for (int t4 = 0; t4 < C; t4 += 4) {
                const float4 gx = *reinterpret_cast<const float4*>(&sm.g[col][t4]), gq = *reinterpret_cast<const float4*>(&sm.g[col][C + t4]);
                const float ax[4] = {gx.x, gx.y, gx.z, gx.w}, aq[4] = {gq.x, gq.y, gq.z, gq.w};
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    if (t4 + t > q) x[t4 + t] = fmaf(sign * ax[t], v, x[t4 + t]);
                    if (t4 + t >= q) y[t4 + t] = fmaf(sign * aq[t], v, y[t4 + t]);
                }
            }
        };
        float* o_x = is_x ? out + ch : o_v + C * DP + ch;              // X' and Q' rows, or V1 and O1 rows
        if (is_x) {
#pragma unroll
            for (int t = 0; t < C; ++t) { x[t] = sm.xq[t][ch]; y[t] = sm.xq[C + t][ch]; }
        } else {
#pragma unroll
            for (int t = 0; t < C; ++t) { x[t] = 0.f; y[t] = 0.f; }
#pragma unroll
            for (int t = 0; t < C; ++t) {
                const float v = sm.v[t][ch];
                o_v[t * DP + ch] = v;
                subtract(t, v, C + t, 1.f);
            }
        }
#pragma unroll
        for (int t = 0; t < C; ++t) subtract(t, x[t], t, -1.f);
#pragma unroll
        for (int t = 0; t < C; ++t) { o_x[t * DP] = x[t]; o_x[(C + t) * DP] = y[t]; }
    }
}

// grid (heads * ceil(DP / 16), entries): the sequential part for 16 value channels of one head.
template <int DP>
__global__ void __launch_bounds__(dc::kScanThreads) delta_chunk_scan_kernel(const float* __restrict__ pack, float* __restrict__ o, int ld_o,
                                                                        float* __restrict__ pool, size_t slot_stride, size_t offset, const DeltaShape s,
                                                                        const RowPlan plan) {
    using namespace dc;
    using ds::cp16;
    constexpr int RT = DP / 4;                                     // row tiles of the state (4 x 4 each)
    constexpr int TI = (RT * 4 + 63) / 64;                         // tiles per group of four lanes
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
        for (int i = tid; i < DP * 8; i += kScanThreads) cp16(&sm.xq[b][i / RT][(i % RT) * 4], src + i * 4);
        for (int i = tid; i < DP * 8; i += kScanThreads) cp16(&sm.cb[b][0][0] + i * 4, src + 32 * DP + i * 4);
        for (int i = tid; i < 3 * C * 4; i += kScanThreads) cp16(&sm.vin[b][0][i >> 2][(i & 3) * 4], src + 64 * DP + (i >> 2) * DP + c0 + (i & 3) * 4);
        if (tid < DP / 4) cp16(&sm.p[b][tid * 4], src + 112 * DP + tid * 4);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    // Second product: a 4 x 4 tile of the state per four lanes (8 apart), each with a quarter of k; a lane then keeps one
    // column of its tiles: rows 4 it .., column 4 jt + lane / 8.
    const int kq = lane >> 3;
    int it[TI], jc[TI];
    bool own[TI];
    float S[TI][4];
    float* st = pool + (size_t)e.state * slot_stride + offset + (size_t)h * s.D * s.D + c0;
#pragma unroll
    for (int n = 0; n < TI; ++n) {
        const int tile = warp * 8 + (lane & 7) + 64 * n;
        own[n] = tile < RT * 4;
        it[n] = tile % RT;
        jc[n] = tile / RT * 4;
        if (!own[n]) continue;                                     // whole groups of eight tiles: a warp's lanes agree
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = 4 * it[n] + i, j = jc[n] + kq;
            S[n][i] = e.pos0 > 0 && r < s.D && c0 + j < s.D ? st[(size_t)r * s.D + j] : 0.f;
            sm.st[j][r] = S[n][i];
        }
    }
    // first product: 4 x 4 outputs per thread, k split over eight lanes
    const int ks = lane & 7, ct = lane >> 3, rt = warp;
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
#pragma unroll
        for (int k4 = 0; k4 < DP / 32; ++k4) {
            const int k = (k4 * 8 + ks) * 4;
            float4 a[4], y[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(&sm.xq[b][rt * 4 + i][k]);
#pragma unroll
            for (int j = 0; j < 4; ++j) y[j] = *reinterpret_cast<const float4*>(&sm.st[ct * 4 + j][k]);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(a[i].x, y[j].x, acc[i][j]); acc[i][j] = fmaf(a[i].y, y[j].y, acc[i][j]);
                    acc[i][j] = fmaf(a[i].z, y[j].z, acc[i][j]); acc[i][j] = fmaf(a[i].w, y[j].w, acc[i][j]);
                }
        }
        // sum over the eight lanes; lane ks keeps row ks & 3 and one pair of columns
        float half[2][4], rowv[4], v2[2];
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
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const float mine = ks & 4 ? rowv[2 + j] : rowv[j], other = ks & 4 ? rowv[j] : rowv[2 + j];
            v2[j] = mine + __shfl_xor_sync(0xffffffffu, other, 4);
        }
        const int row = rt * 4 + (ks & 3), col = ct * 4 + (ks >> 2) * 2;
        if (row < C) {
            const float2 v1 = *reinterpret_cast<const float2*>(&sm.vin[b][1][row][col]);
            *reinterpret_cast<float2*>(&sm.y[row][col]) = make_float2(v2[0] + v1.x, v2[1] + v1.y);
        } else if (c * C + row - C < e.n) {
            const float2 o1 = *reinterpret_cast<const float2*>(&sm.vin[b][2][row - C][col]);
            float* dst = o + (size_t)(e.row0 + c * C + row - C) * ld_o + h * s.D + c0 + col;
            if ((s.D & 1) == 0) {
                if (c0 + col < s.D) *reinterpret_cast<float2*>(dst) = make_float2(v2[0] + o1.x, v2[1] + o1.y);
            } else {
                if (c0 + col < s.D) dst[0] = v2[0] + o1.x;
                if (c0 + col + 1 < s.D) dst[1] = v2[1] + o1.y;
            }
        }
        __syncthreads();
#pragma unroll
        for (int n = 0; n < TI; ++n) {
            if (!own[n]) continue;
            float u[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) u[i][j] = 0.f;
#pragma unroll
            for (int kk = 0; kk < 8; ++kk) {
                const int k = kk * 4 + kq;
                const float4 a = *reinterpret_cast<const float4*>(&sm.cb[b][k][4 * it[n]]);
                const float4 y = *reinterpret_cast<const float4*>(kk < 4 ? &sm.vin[b][0][k][jc[n]] : &sm.y[k - C][jc[n]]);
                const float av[4] = {a.x, a.y, a.z, a.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) u[i][j] = fmaf(av[i], yv[j], u[i][j]);
            }
            float r[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                float p2[2];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const float mine = kq & 2 ? u[i][2 + j] : u[i][j], other = kq & 2 ? u[i][j] : u[i][2 + j];
                    p2[j] = mine + __shfl_xor_sync(0xffffffffu, other, 16);
                }
                const float mine = kq & 1 ? p2[1] : p2[0], other = kq & 1 ? p2[0] : p2[1];
                r[i] = mine + __shfl_xor_sync(0xffffffffu, other, 8);
            }
            const float4 pd = *reinterpret_cast<const float4*>(&sm.p[b][4 * it[n]]);
            S[n][0] = (S[n][0] + r[0]) * pd.x; S[n][1] = (S[n][1] + r[1]) * pd.y;
            S[n][2] = (S[n][2] + r[2]) * pd.z; S[n][3] = (S[n][3] + r[3]) * pd.w;
            *reinterpret_cast<float4*>(&sm.st[jc[n] + kq][4 * it[n]]) = make_float4(S[n][0], S[n][1], S[n][2], S[n][3]);
        }
    }
#pragma unroll
    for (int n = 0; n < TI; ++n) {
        if (!own[n]) continue;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = 4 * it[n] + i, j = jc[n] + kq;
            if (r < s.D && c0 + j < s.D) st[(size_t)r * s.D + j] = S[n][i];
        }
    }
}

}  // namespace efm
