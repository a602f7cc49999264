// Device set-up of the text-tower kernels (cluster widths, opt-in shared memory), shared by the contexts and the
// single-operator entry points.  Never called inside a stream capture.
#pragma once
#include "../../layers/launch.cuh"
#include "../../layers/qwen_text.h"
#include "ctx_util.h"

namespace efm {

inline efm_status require_b200(efm_b200_ctx* c, int device_id) {
    const efm_status st = require_device(c, device_id);
    if (st != EFM_OK) return st;
    EFM_CK(c, configure_decode_attention());
    EFM_CK(c, configure_sampler());
    int optin = 0;
    EFM_CK(c, cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, device_id));
    EFM_CK(c, configure_gemv(optin - 2048));        // leave room for the kernels' static shared memory
    return EFM_OK;
}

// INT8 attention scratch for up to q_rows queries and kv_rows keys (one scale per 128-token block and head);
// plain cudaMalloc, caller frees with free_sage.
inline cudaError_t alloc_sage(SageScratch& sc, int q_rows, int kv_rows, int q_heads, int kv_heads, int D) {
    cudaError_t e = cudaMalloc(&sc.q8, (size_t)q_rows * q_heads * D);
    if (e == cudaSuccess) e = cudaMalloc(&sc.k8, (size_t)kv_rows * kv_heads * D);
    if (e == cudaSuccess) e = cudaMalloc(&sc.vh, (size_t)kv_rows * kv_heads * D * 2);
    if (e == cudaSuccess) e = cudaMalloc(&sc.sq, (size_t)(q_rows / 128 + 1) * q_heads * sizeof(float));
    if (e == cudaSuccess) e = cudaMalloc(&sc.sk, (size_t)(kv_rows / 128 + 1) * kv_heads * sizeof(float));
    if (e == cudaSuccess) e = cudaMalloc(&sc.kmean, (size_t)(kv_rows / 128 + 1) * kv_heads * D * sizeof(float));
    sc.q_rows = q_rows;
    sc.kv_rows = kv_rows;
    return e;
}
inline void free_sage(SageScratch& sc) {
    cudaFree(sc.q8); cudaFree(sc.k8); cudaFree(sc.vh); cudaFree(sc.sq); cudaFree(sc.sk); cudaFree(sc.kmean);
    sc = SageScratch{};
}

}  // namespace efm
