// Row kernels every model's many-row pass shares: embedding gather, RMSNorm rows.
#pragma once
#include "common.cuh"

namespace efm {

// Embedding gather with custom-embedding injection.  One block per token.
// Same contract as the reference's embedding_lookup_with_embedding_insertion_kernel
// (src/layers/embed_head.cu:63-132): ids in [embed_token_id, embed_token_id + n_custom) take
// row id - embed_token_id of `custom`; other ids inside the vocabulary take the table row; any
// other id yields zeros.
__global__ void __launch_bounds__(128) embed_rows_kernel(const int32_t* __restrict__ ids,
                                                         const __nv_bfloat16* __restrict__ table,
                                                         const __nv_bfloat16* __restrict__ custom,
                                                         float* __restrict__ out, int vocab, int hidden,
                                                         int embed_token_id, int n_custom, float scale) {
    const int t = blockIdx.x;
    const int id = ids[t];
    const __nv_bfloat16* src = nullptr;
    if (custom != nullptr && embed_token_id >= 0 && id >= embed_token_id && id < embed_token_id + n_custom)
        src = custom + (size_t)(id - embed_token_id) * hidden;
    else if (id >= 0 && id < vocab)
        src = table + (size_t)id * hidden;
    float4* dst = reinterpret_cast<float4*>(out + (size_t)t * hidden);      // residual stream: fp32
    for (int c = threadIdx.x; c < hidden / 8; c += blockDim.x) {
        float f[8];
        unpack8(src != nullptr ? ld_cached(src + (size_t)c * 8) : make_uint4(0, 0, 0, 0), f);
        dst[2 * c] = make_float4(f[0] * scale, f[1] * scale, f[2] * scale, f[3] * scale);
        dst[2 * c + 1] = make_float4(f[4] * scale, f[5] * scale, f[6] * scale, f[7] * scale);
    }
}

// y[s,:] = bf16(x[s,:] * rsqrt(mean(x^2) + eps) * w), x = fp32 residual stream, fp32 inside (reference: FlashInfer RMSNorm
// through src/operators/norm_op.cu:20-62; formula pinned by tests/operators/test_norm_sampler.py:62-64).
__global__ void __launch_bounds__(256) rmsnorm_rows_kernel(const float* __restrict__ x,
                                                           const __nv_bfloat16* __restrict__ w,
                                                           __nv_bfloat16* __restrict__ y, int hidden, float eps) {
    __shared__ float part[8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_launch_dependents();
    pdl_wait();            // no-ops unless launched with programmatic stream serialization
    const float* xr = x + (size_t)blockIdx.x * hidden;
    const int nch = hidden >> 3;
    float ss = 0.f;
    for (int c = tid; c < nch; c += 256) {
        const float4 lo = reinterpret_cast<const float4*>(xr)[2 * c], hi = reinterpret_cast<const float4*>(xr)[2 * c + 1];
        const float f[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
        for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) tot += part[i];
    const float inv = 1.0f / sqrtf(tot / (float)hidden + eps);
    uint4* yr = reinterpret_cast<uint4*>(y + (size_t)blockIdx.x * hidden);
    for (int c = tid; c < nch; c += 256) {
        const float4 lo = reinterpret_cast<const float4*>(xr)[2 * c], hi = reinterpret_cast<const float4*>(xr)[2 * c + 1];
        const float f[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
        float g[8];
        unpack8(ld_cached(w + (size_t)c * 8), g);
        uint4 o;
        o.x = pack_bf16(f[0] * inv * g[0], f[1] * inv * g[1]);
        o.y = pack_bf16(f[2] * inv * g[2], f[3] * inv * g[3]);
        o.z = pack_bf16(f[4] * inv * g[4], f[5] * inv * g[5]);
        o.w = pack_bf16(f[6] * inv * g[6], f[7] * inv * g[7]);
        yr[c] = o;
    }
}

// The same for rows of at most 2048 channels (hidden % 4 == 0): one warp per row, the row stays in registers between the
// sum of squares and the scaling (one read of x, no block barrier); 8 rows per block.
__global__ void __launch_bounds__(256) rmsnorm_rows_warp_kernel(const float* __restrict__ x, const __nv_bfloat16* __restrict__ w,
                                                                __nv_bfloat16* __restrict__ y, int rows, int hidden, float eps) {
    constexpr int MAXV = 16;                                   // float4 per lane: 16 x 32 x 4 = 2048 channels
    const int row = blockIdx.x * 8 + (int)(threadIdx.x >> 5), lane = threadIdx.x & 31;
    pdl_launch_dependents();
    pdl_wait();            // no-ops unless launched with programmatic stream serialization
    if (row >= rows) return;
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)row * hidden);
    const int nv = hidden >> 2;
    float4 v[MAXV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int c = lane + 32 * i;
        if (c < nv) {
            v[i] = xr[c];
            ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss); ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
        }
    }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)hidden + eps);
    uint2* yr = reinterpret_cast<uint2*>(y + (size_t)row * hidden);
    const uint2* wr = reinterpret_cast<const uint2*>(w);
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int c = lane + 32 * i;
        if (c < nv) {
            const uint2 g = __ldg(wr + c);
            yr[c] = make_uint2(pack_bf16(v[i].x * inv * bf16lo(g.x), v[i].y * inv * bf16hi(g.x)),
                               pack_bf16(v[i].z * inv * bf16lo(g.y), v[i].w * inv * bf16hi(g.y)));
        }
    }
}

}  // namespace efm
