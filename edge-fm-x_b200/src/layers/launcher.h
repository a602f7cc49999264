// Host-side launch plumbing shared by all layer sequences: attaches the programmatic-dependent-launch attribute and
// thread-block clusters, counts launches, keeps the first failure.
#pragma once
#include <cuda_runtime.h>

#include <algorithm>
#include <cstdint>
#include <cstdlib>
#include <vector>

namespace efm {

struct Launcher {
    cudaStream_t stream = nullptr;
    bool pdl = true;                 // programmatic stream serialization between consecutive kernels
    bool pdl_rows = false;           // keep `pdl` for the row / attention kernels of the prefill family too (they open with the wait)
    int cluster_x = 0;               // next launch only: thread-block cluster of this many blocks along x
    float* gemm_ws = nullptr;        // split-K workspace of the owning context (nullptr: GEMMs never split)
    size_t gemm_ws_floats = 0;
    int num_sms = 148;
    int64_t* counter = nullptr;
    cudaError_t err = cudaSuccess;   // first failure sticks
    std::vector<cudaEvent_t>* trace = nullptr;   // when set: one event recorded after every launch

    template <typename... KArgs, typename... Args>
    void launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args&&... args) {
        if (err != cudaSuccess) return;
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = grid;
        cfg.blockDim = block;
        cfg.dynamicSmemBytes = smem;
        cfg.stream = stream;
        cudaLaunchAttribute attr[2];
        int na = 0;
        if (pdl) {
            attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
            attr[na++].val.programmaticStreamSerializationAllowed = 1;
        }
        if (cluster_x > 1) {
            attr[na].id = cudaLaunchAttributeClusterDimension;
            attr[na].val.clusterDim.x = (unsigned)cluster_x;
            attr[na].val.clusterDim.y = 1;
            attr[na++].val.clusterDim.z = 1;
        }
        cfg.attrs = na > 0 ? attr : nullptr;
        cfg.numAttrs = na;
        cluster_x = 0;
        err = cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
        if (counter != nullptr) ++*counter;
        if (trace != nullptr && err == cudaSuccess) {
            cudaEvent_t ev = nullptr;
            if (cudaEventCreate(&ev) == cudaSuccess) { cudaEventRecord(ev, stream); trace->push_back(ev); }
        }
    }
};

}  // namespace efm
