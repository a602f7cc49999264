// Routed feed-forward: every token uses `top` of `experts` small gated feed-forwards,
//   y = sum_k s_k W_down[e_k] (silu(W_gate[e_k] h) * W_up[e_k] h),   s = softmax(W_router h) or sigmoid(W_router h),
// where e_k are the best experts of the best groups (a group's score is its largest expert score) and s_k their scores as they
// are; they may scale the experts' inputs instead of their outputs.  A shared expert runs for every token beside them.
// Experts without a gate are W_down[e_k] relu(W_up[e_k] h)^2.
// Weights: [experts][2 * ffp rows][K] with blocks of 64 gate rows followed by the 64 matching up rows ([experts][ffp rows][K] without
// a gate), and [experts][n_out][ffp]; ffp is the expert width padded to 64 with zero rows / columns.
//
//   route_token          one token's choice, by one warp (expert_route.cuh; the decode GEMV of gemv.cuh chooses the same way)
//   expert_route_rows    many rows: choices, weights, and each choice's place among its expert's rows
//   expert_gather_rows   the rows sorted by expert, every expert's share starting at a multiple of kExpertTile rows, and the
//                        expert of each such tile: the A operand of the grouped products (gemm_tc.cuh, gemm_f32)
//   glu_rows             32-bit mode: the gated unit (gemv.cuh)
// The weighted sum of the expert outputs is part of the output norm (add_norm_rows, decoder_rows.cuh).
#pragma once
#include "common.cuh"
#include "expert_route.cuh"
#include "gemv.cuh"

namespace efm {

// one warp per row
__global__ void __launch_bounds__(256) expert_route_rows_kernel(const float* __restrict__ logits, int ld, int rows, const RouteShape r, const ExpertRows o) {
    const int row = blockIdx.x * 8 + (int)(threadIdx.x >> 5);
    if (row >= rows) return;
    route_token(logits + (size_t)row * ld, r, [&](int k, int e, float w) {
        o.id[(size_t)row * r.top + k] = e;
        o.weight[(size_t)row * r.top + k] = w;
        o.place[(size_t)row * r.top + k] = atomicAdd(o.count + e, 1);
    });
    if (r.shared != kSharedNone && (threadIdx.x & 31) == 0)
        o.shared[row] = r.shared == kSharedGated ? 1.0f / (1.0f + expf(-logits[(size_t)row * ld + r.experts])) : 1.0f;
}

// First row of every expert in the sorted order, by the first warp; block 0 describes the tiles.
__device__ __forceinline__ void expert_offsets(const int32_t* count, int experts, int32_t* off, const ExpertRows* publish) {
    const int lane = threadIdx.x & 31;
    int base = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
        const int e = e0 + lane, n = e < experts ? (__ldcg(count + e) + kExpertTile - 1) / kExpertTile : 0;
        int x = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= o) x += y;
        }
        const int first = base + x - n;
        if (e < experts) off[e] = first * kExpertTile;
        if (publish != nullptr)
            for (int t = 0; t < n; ++t) publish->tile[first + t] = make_int4(e, first, n, 0);
        base += __shfl_sync(0xffffffffu, x, 31);
    }
    if (publish != nullptr && lane == 0) *publish->n_tiles = base;
}

// Row `row` of h, or (SCALE) each choice's weight times it, to its places in the sorted order.  One block per row; ld % 8 == 0.
template <typename T, bool SCALE>
__global__ void __launch_bounds__(128) expert_gather_rows_kernel(const T* __restrict__ h, T* __restrict__ out, int ld, const RouteShape r, const ExpertRows o) {
    __shared__ int32_t off[kMaxExperts];
    __shared__ int32_t dst[kMaxExpertTop];
    __shared__ float weight[SCALE ? kMaxExpertTop : 1];
    const int row = blockIdx.x;
    if (threadIdx.x < 32) {
        expert_offsets(o.count, r.experts, off, row == 0 ? &o : nullptr);
        __syncwarp();
        if ((int)threadIdx.x < r.top) {
            const size_t i = (size_t)row * r.top + threadIdx.x;
            const int d = off[o.id[i]] + o.place[i];
            dst[threadIdx.x] = d;
            o.place[i] = d;
            if constexpr (SCALE) weight[threadIdx.x] = o.weight[i];
        }
    }
    __syncthreads();
    constexpr int V = 16 / sizeof(T);
    for (int c = threadIdx.x; c < ld / V; c += 128) {
        const uint4 v = ld_cached(h + (size_t)row * ld + c * V);
        for (int k = 0; k < r.top; ++k) {
            uint4 x = v;
            if constexpr (SCALE) {
                const float w = weight[k];
                if constexpr (sizeof(T) == 2)
                    x = make_uint4(pack_bf16(w * bf16lo(v.x), w * bf16hi(v.x)), pack_bf16(w * bf16lo(v.y), w * bf16hi(v.y)),
                                   pack_bf16(w * bf16lo(v.z), w * bf16hi(v.z)), pack_bf16(w * bf16lo(v.w), w * bf16hi(v.w)));
                else
                    x = make_uint4(__float_as_uint(w * __uint_as_float(v.x)), __float_as_uint(w * __uint_as_float(v.y)),
                                   __float_as_uint(w * __uint_as_float(v.z)), __float_as_uint(w * __uint_as_float(v.w)));
            }
            *reinterpret_cast<uint4*>(out + (size_t)dst[k] * ld + c * V) = x;
        }
    }
}

// gu: rows of 64 gate values followed by the 64 matching up values -> gated unit, ffp columns (Relu2: ffp values -> their unit).  Grid: tiles of kExpertTile rows, of
// which *n_tiles (null: all) are in use.
__global__ void __launch_bounds__(256) glu_rows_kernel(const float* __restrict__ gu, float* __restrict__ out, int rows, int ffp, const int32_t* __restrict__ n_tiles,
                                                       int kind, float limit) {
    const int tile = blockIdx.x;
    if (n_tiles != nullptr && tile >= *n_tiles) return;
    for (int i = threadIdx.x; i < kExpertTile * ffp; i += 256) {
        const int r = i / ffp, c = i - r * ffp;
        if (tile * kExpertTile + r >= rows) return;
        if (kind == kGluRelu2) {
            out[(size_t)(tile * kExpertTile + r) * ffp + c] = relu2(gu[(size_t)(tile * kExpertTile + r) * ffp + c]);
            continue;
        }
        const float* src = gu + (size_t)(tile * kExpertTile + r) * 2 * ffp + (c >> 6) * 128 + (c & 63);
        out[(size_t)(tile * kExpertTile + r) * ffp + c] = glu(kind, src[0], src[64], limit);
    }
}

}  // namespace efm
