// Host-side launch helpers shared by the dense-decoder libraries.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#include <algorithm>
#include <map>
#include <mutex>
#include <utility>

#include "decoder_ops.h"

namespace tsp {


inline int sm_count() {
    static int sms[64] = {0};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) dev = 0;
    if (!sms[dev]) {
        int v = 0;
        if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || v <= 0) v = 148;
        sms[dev] = v;
    }
    return sms[dev];
}

inline int bad(int code, const char* what) {
    fprintf(stderr, "decoder_ops: %s\n", what);
    return code;
}
inline bool misaligned(const void* p, unsigned n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) != 0; }

// Attributes of a kernel that depend on its shared memory, set when they change.
//  * Requests above 48 KB in all (what a kernel has beside it in fixed arrays counts) have to be announced.
//  * Kernels of a decode step ask for a moderate share of the SM's memory as shared memory.  Without a wish of their own
//    they would run in whatever split the last kernel with a large request left behind, and with most of the SM's
//    memory taken away from L1 far fewer weight loads are in flight.
inline bool set_attributes(const void* kernel, size_t smem, int pdl) {
    static std::mutex lock;
    static std::map<std::pair<int, const void*>, std::pair<size_t, int>> done;
    int dev = 0;
    cudaGetDevice(&dev);
    const int share = pdl && smem <= 100 * 1024 ? (int)std::max<size_t>(30, 200 * (smem + 12 * 1024) / (228 * 1024)) : 0;   // two CTAs
    const std::lock_guard<std::mutex> guard(lock);
    auto& d = done[{dev, kernel}];
    if (smem > std::max<size_t>(d.first, 16 * 1024)) {
        if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return false;
        d.first = smem;
    }
    if (share > d.second) {
        if (cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, std::min(share, 100)) != cudaSuccess) return false;
        d.second = share;
    }
    return true;
}

template <typename... P, typename... Q>
inline int launch(void (*kernel)(P...), dim3 grid, int threads, size_t smem, int pdl, void* stream, int cluster, Q... args) {
    if (!set_attributes(reinterpret_cast<const void*>(kernel), smem, pdl)) return bad(DECODER_LAUNCH, "shared memory request refused");
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(threads, 1, 1);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = static_cast<cudaStream_t>(stream);
    cudaLaunchAttribute at[2];
    int n = 0;
    if (pdl) {
        at[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        at[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 1) {
        at[n].id = cudaLaunchAttributeClusterDimension;
        at[n].val.clusterDim.x = cluster, at[n].val.clusterDim.y = 1, at[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = at, cfg.numAttrs = n;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, args...);
    if (e != cudaSuccess) {
        fprintf(stderr, "decoder_ops: launch failed: %s\n", cudaGetErrorString(e));
        return DECODER_LAUNCH;
    }
    return DECODER_OK;
}

// bf16 matrix [rows][cols] with rows ld elements apart, read in tiles of 64 columns (128-byte swizzle) by box_rows
inline bool encode_rows(CUtensorMap* map, const void* base, long long rows, long long cols, long long ld, int box_rows) {
    typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                 const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                 CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static EncodeFn fn = nullptr;
    if (!fn) {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || !ptr) return false;
        fn = reinterpret_cast<EncodeFn>(ptr);
    }
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64, (cuuint32_t)box_rows}, step[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}


}  // namespace tsp
