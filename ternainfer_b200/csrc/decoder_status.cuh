// Device-side status of a dense-decoder library: one word that a kernel sets when a bounded wait has run out.
#pragma once
#include <cuda_runtime.h>

#include "decoder_ops.h"

namespace tsp {

__device__ int g_decoder_status = 0;

// the status since the last call (synchronises)
static int read_decoder_status() {
    int v = 0;
    if (cudaMemcpyFromSymbol(&v, g_decoder_status, sizeof(v)) != cudaSuccess) return DECODER_LAUNCH;
    if (v) {
        const int zero = 0;
        cudaMemcpyToSymbol(g_decoder_status, &zero, sizeof(zero));
    }
    return v;
}

}  // namespace tsp
