// Choice of experts for one token, by one warp.
#pragma once
#include "common.cuh"
#include "expert_rows.h"

namespace efm {

// z: router logits of all experts.  Scores softmax(z) or sigmoid(z); the groups whose best scores are the largest stay open; the best `top`
// experts of those are handed to store(k, expert, score * scale) in lane 0.  Ties go to the lower number.
template <int N, typename Store>
__device__ __forceinline__ void route_token_n(const float* z, const RouteShape& r, Store store) {      // at most 32 N experts
    const int lane = threadIdx.x & 31, per = r.experts / r.groups;
    float v[N], mx = -INFINITY, sum = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int e = lane + 32 * i;
        v[i] = e < r.experts ? __ldcg(z + e) : -INFINITY;
        mx = fmaxf(mx, v[i]);
    }
    if (r.sigmoid) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = lane + 32 * i < r.experts ? 1.0f / (1.0f + expf(-v[i])) : -1.f;
    } else {
        mx = warp_max(mx);
#pragma unroll
        for (int i = 0; i < N; ++i) {
            v[i] = lane + 32 * i < r.experts ? expf(v[i] - mx) : 0.f;
            sum += v[i];
        }
        const float inv = 1.0f / warp_sum(sum);
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = lane + 32 * i < r.experts ? v[i] * inv : -1.f;
    }
    if (r.keep < r.groups) {                                            // close all but the best groups
        float best[2] = {-1.f, -1.f};                                   // lane l: groups l and l + 32
        for (int g = 0; g < r.groups; ++g) {
            float m = -1.f;
#pragma unroll
            for (int i = 0; i < N; ++i)
                if ((lane + 32 * i) / per == g) m = fmaxf(m, v[i]);
            m = warp_max(m);
            if ((g & 31) == lane) best[g >> 5] = m;
        }
        unsigned long long open = 0ull;
        for (int k = 0; k < r.keep; ++k) {
            float m = fmaxf(best[0], best[1]);
            const float top = warp_max(m);
            const unsigned a = __ballot_sync(0xffffffffu, best[0] == top), b = __ballot_sync(0xffffffffu, best[1] == top);
            const int g = a != 0u ? __ffs(a) - 1 : 31 + __ffs(b);
            open |= 1ull << g;
            if ((g & 31) == lane) best[g >> 5] = -2.f;
        }
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const int e = lane + 32 * i;
            if (e < r.experts && ((open >> (e / per)) & 1ull) == 0ull) v[i] = -1.f;
        }
    }
    for (int k = 0; k < r.top; ++k) {
        float m = -2.f;
        int at = 0x7fffffff;
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (v[i] > m) { m = v[i]; at = lane + 32 * i; }
        const float best = warp_max(m);
        int e = m == best ? at : 0x7fffffff;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) e = min(e, __shfl_xor_sync(0xffffffffu, e, o));
        e = min(e, r.experts - 1);                                      // logits that are no numbers choose something
        if (lane == 0) store(k, e, best * r.scale);
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (e == lane + 32 * i) v[i] = -2.f;
    }
}
template <typename Store>
__device__ __forceinline__ void route_token(const float* z, const RouteShape& r, Store store) {
    static_assert(kMaxExperts == 32 * 16, "widest instantiation");
    if (r.experts <= 32) route_token_n<1>(z, r, store);
    else if (r.experts <= 64) route_token_n<2>(z, r, store);
    else if (r.experts <= 128) route_token_n<4>(z, r, store);
    else route_token_n<16>(z, r, store);
}

}  // namespace efm
