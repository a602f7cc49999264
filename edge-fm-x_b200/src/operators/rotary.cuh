// Rotary positions of the layered decoders: pair i of a head at position p turns by the angle p * inv_freq[i],
//   (u, v) -> (u cos - v sin, v cos + u sin),
// with channels i and i + dims / 2 as the pair (half) or the neighbours 2 i and 2 i + 1 (pairs).  Angles are fp32; cos and sin
// are multiplied by mag (scaled rotations); channels from dims on pass unchanged.
#pragma once
#include "common.cuh"

namespace efm {

enum : int { kRotNone = 0, kRotHalf = 1, kRotPairs = 2 };
constexpr int kRotMaxPairs = 128;

struct RotShape {
    int kind, dims;
    const float* inv_freq;            // [dims / 2]
    float mag;
};

__device__ __forceinline__ void rot_sincos(const RotShape& r, int pos, int i, float* sn, float* cs) {
    float s, c;
    sincosf((float)pos * r.inv_freq[i], &s, &c);
    *sn = s * r.mag;
    *cs = c * r.mag;
}
// cos / sin of one position into shared memory (readers synchronise)
__device__ __forceinline__ void rot_table(const RotShape& r, int pos, float* cs, float* sn) {
    if (r.kind == kRotNone) return;
    for (int i = threadIdx.x; i < r.dims / 2; i += blockDim.x) rot_sincos(r, pos, i, sn + i, cs + i);
}
// channel c of the rotated vector, x: the vector before the rotation
__device__ __forceinline__ float rot_channel(const RotShape& r, const float* x, int c, const float* cs, const float* sn) {
    if (c >= r.dims) return x[c];
    if (r.kind == kRotHalf) {
        const int half = r.dims / 2, i = c < half ? c : c - half;
        const float u = x[i], v = x[i + half];
        return c < half ? u * cs[i] - v * sn[i] : v * cs[i] + u * sn[i];
    }
    const int i = c >> 1;
    const float u = x[c & ~1], v = x[c | 1];
    return (c & 1) == 0 ? u * cs[i] - v * sn[i] : v * cs[i] + u * sn[i];
}

}  // namespace efm
