// Per-layer token input of one decode step in a single launch:
//   x = xr + rms(addend) * norm_w      (the pending sublayer output, as in the AddNorm prologue of gemv.cuh)
//   g = gelu_tanh(Gate x) * table[token][gate_off ..],   y = Proj g
// One cluster: every block stages x, computes its share of Gate's rows, hands its values of g to the other blocks through
// distributed shared memory and computes its share of Proj's rows.  Both weight slices are requested into shared memory
// before the dependency wait.  Bound: latency (the two matrices are a few hundred KB).
#pragma once
#include <cooperative_groups.h>

#include <utility>

#include "gemv.cuh"

namespace efm {

namespace ts {
struct Layout {
    int gate_rows, proj_rows;          // per block
    unsigned int off_gate, off_proj, off_g, off_red, bytes;
};
// K = Kp of Gate (= padded width), side_p = Kp of Proj, n_out = rows of Proj
__host__ __device__ inline Layout layout(int K, int side_p, int n_out, int cluster) {
    Layout l;
    l.gate_rows = (side_p + cluster - 1) / cluster;
    l.proj_rows = (n_out + cluster - 1) / cluster;
    unsigned int at = (unsigned int)((gemv_ext_off(K) + (unsigned int)K * 4u + 15u) & ~15u);
    l.off_gate = at; at += (unsigned int)l.gate_rows * K * 2u;
    l.off_proj = at; at += (unsigned int)l.proj_rows * side_p * 2u;
    at = (at + 15u) & ~15u;
    l.off_g = at; at += (unsigned int)side_p * 4u;
    l.off_red = at; at += kGemvWarps * 4u;
    l.bytes = at;
    return l;
}
}  // namespace ts

struct TokenSideParams {
    GemvParams p;                      // AddNorm prologue (xr, addend, norm_w, resid_out, eps, k_true, K), token gate, state; W = Gate
    const __nv_bfloat16* proj;         // [n_out][side_p]
    int side_p, n_out;
    float* y;                          // [n_out]
};

__global__ void __launch_bounds__(kGemvThreads, 1) token_side_kernel(const TokenSideParams q) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) unsigned char ts_smem[];
    cg::cluster_group cl = cg::this_cluster();
    const GemvParams& p = q.p;
    const int n_blocks = gridDim.x, rank = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const ts::Layout l = ts::layout(p.K, q.side_p, q.n_out, n_blocks);
    __nv_bfloat16* gate = reinterpret_cast<__nv_bfloat16*>(ts_smem + l.off_gate);
    __nv_bfloat16* proj = reinterpret_cast<__nv_bfloat16*>(ts_smem + l.off_proj);
    float* g = reinterpret_cast<float*>(ts_smem + l.off_g);
    float* red = reinterpret_cast<float*>(ts_smem + l.off_red);
    const int g0 = rank * l.gate_rows, ng = max(0, min(l.gate_rows, q.side_p - g0)), o0 = rank * l.proj_rows, no = max(0, min(l.proj_rows, q.n_out - o0));
    auto started = cl.barrier_arrive();                              // waited for before the first store into another block
    pdl_launch_dependents();
    auto cp16 = [](void* dst, const void* src) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
    };
    for (int i = tid; i < ng * p.K / 8; i += kGemvThreads) cp16(gate + i * 8, p.W + (size_t)g0 * p.K + i * 8);
    for (int i = tid; i < no * q.side_p / 8; i += kGemvThreads) cp16(proj + i * 8, q.proj + (size_t)o0 * q.side_p + i * 8);
    {
        uint4* gs = reinterpret_cast<uint4*>(ts_smem + gemv_xbytes(p.K));        // norm weight, where the prologue reads it
        for (int c = tid; c < p.K / 8; c += kGemvThreads) gs[c] = ld_cached(p.norm_w + (size_t)c * 8);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    pdl_wait();
    gemv_stage_ext<1>(p, p.K >> 3, ts_smem, gemv_xbytes(p.K));
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    cl.barrier_wait(std::move(started));
    const float* xs = reinterpret_cast<const float*>(ts_smem);
    // ---- gate rows: `parts` warps share a row ----------------------------------------------------------------------
    int parts = 1;
    while (parts * 2 * max(ng, 1) <= kGemvWarps) parts *= 2;
    const int per = kGemvWarps / parts;                              // rows at a time
    for (int r0 = 0; r0 < ng; r0 += per) {
        const int r = r0 + warp / parts, part = warp % parts;
        float a = 0.f;
        if (r < ng)
            for (int c = part * 32 + lane; c < p.K / 8; c += parts * 32) {
                const float4 lo = reinterpret_cast<const float4*>(xs)[2 * c], hi = reinterpret_cast<const float4*>(xs)[2 * c + 1];
                const float f[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
                a = dot8(*reinterpret_cast<const uint4*>(gate + (size_t)r * p.K + c * 8), f, a);
            }
        a = warp_sum(a);
        if (lane == 0) red[warp] = a;
        __syncthreads();
        if (tid < per && r0 + tid < ng) {
            float t = 0.f;
            for (int w = 0; w < parts; ++w) t += red[tid * parts + w];
            const int n = g0 + r0 + tid, tok = p.state->token;
            const bool ok = tok >= 0 && tok < p.vocab && n < p.N;
            const float v = ok ? gelu_tanh(t) * __bfloat162float(p.gate_table[(size_t)tok * p.gate_ld + p.gate_off + n]) : 0.f;
            for (int b = 0; b < n_blocks; ++b) *cl.map_shared_rank(g + n, b) = v;
        }
        __syncthreads();
    }
    cl.sync();
    // ---- projection rows: eight lanes per row ------------------------------------------------------------------------
    for (int r = tid >> 3; r < (no + 3) / 4 * 4; r += kGemvThreads / 8) {        // the four rows of a warp stay together
        float a = 0.f;
        if (r < no)
            for (int c = tid & 7; c < q.side_p / 8; c += 8) {
                const float4 lo = *reinterpret_cast<const float4*>(g + c * 8), hi = *reinterpret_cast<const float4*>(g + c * 8 + 4);
                const float f[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
                a = dot8(*reinterpret_cast<const uint4*>(proj + (size_t)r * q.side_p + c * 8), f, a);
            }
        const unsigned int mask = __activemask();
#pragma unroll
        for (int x = 4; x > 0; x >>= 1) a += __shfl_xor_sync(mask, a, x);
        if ((tid & 7) == 0 && r < no) q.y[o0 + r] = a;
    }
}

}  // namespace efm
