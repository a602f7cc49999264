// Helpers shared by the translation units of the backend: error reporting, device allocation owned by a context,
// launcher set-up, stream synchronisation.
#pragma once
#include <cstdlib>
#include <cstring>
#include <new>
#include <string>

#include "../../layers/launcher.h"
#include "ctx.h"
#include "nccl_glue.h"

namespace efm {

std::string& create_error();        // message of the last failure without a context (per thread)

inline efm_status fail(efm_b200_ctx* c, efm_status st, const std::string& msg) {
    if (c != nullptr) c->error = msg; else create_error() = msg;
    return st;
}
inline efm_status cuda_fail(efm_b200_ctx* c, cudaError_t e, const char* what) {
    const efm_status st = e == cudaErrorMemoryAllocation ? EFM_ERR_OUT_OF_MEMORY : EFM_ERR_CUDA;
    return fail(c, st, std::string(what) + ": " + cudaGetErrorString(e));
}
#define EFM_CK(ctx, call)                                              \
    do {                                                               \
        cudaError_t e_ = (call);                                       \
        if (e_ != cudaSuccess) return cuda_fail(ctx, e_, #call);       \
    } while (0)

template <typename T>
inline cudaError_t dev_alloc(efm_b200_ctx* c, T** p, size_t count, bool zero = true) {
    void* raw = nullptr;
    const size_t bytes = std::max<size_t>(count * sizeof(T), 16);
    cudaError_t e = cudaMalloc(&raw, bytes);
    if (e != cudaSuccess) return e;
    c->allocations.push_back(raw);
    if (zero) e = cudaMemsetAsync(raw, 0, bytes, c->stream);
    *p = static_cast<T*>(raw);
    return e;
}

// a usable sm_100 device, made current, or an error: there is no CPU path behind this library
efm_status require_device(efm_b200_ctx* c, int device_id);
Launcher make_launcher(efm_b200_ctx* c);
efm_status ctx_sync(efm_b200_ctx* c);
void drop_decode_graphs(efm_b200_ctx* c);
void drop_prefill_graphs(efm_b200_ctx* c);

inline efm_status copy_rows(efm_b200_ctx* c, void* dst, const void* src, size_t bytes, int mem_kind) {
    EFM_CK(c, cudaMemcpyAsync(dst, src, bytes, mem_kind == EFM_MEM_DEVICE ? cudaMemcpyDeviceToDevice : cudaMemcpyHostToDevice, c->stream));
    return EFM_OK;
}
inline bool shape_is(const int64_t* shape, int ndim, int64_t a, int64_t b = -1) {
    if (b < 0) return ndim == 1 && shape[0] == a;
    return ndim == 2 && shape[0] == a && shape[1] == b;
}

}  // namespace efm
