// Elementwise pieces of the dense decoders.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"

namespace tsp {

// in place: the square of relu
template <typename A>
__global__ void __launch_bounds__(256) relu2_kernel(A* x, long long n) {
    griddep_launch_dependents();
    griddep_wait();
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n / 4; i += stride) {
        float4 v = ld_cg4(x + 4 * i);
        v.x = fmaxf(v.x, 0.f), v.y = fmaxf(v.y, 0.f), v.z = fmaxf(v.z, 0.f), v.w = fmaxf(v.w, 0.f);
        st4(x + 4 * i, make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w));
    }
    if (blockIdx.x == 0 && threadIdx.x < (n & 3)) {
        const long long i = (n & ~3ll) + threadIdx.x;
        const float v = fmaxf(ld_cg(x + i), 0.f);
        x[i] = from_f<A>(v * v);
    }
}

// t1[row][j] = tanh of the low-rank decay projection, contiguous (input of the second projection of a prompt)
template <typename A>
__global__ void __launch_bounds__(256) tanh_cols_kernel(const A* proj, long long ld, int off, int rank, long long rows, A* out) {
    griddep_launch_dependents();
    griddep_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < rows * rank; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / rank;
        out[i] = from_f<A>(tanhf(ld_cg(proj + r * ld + off + (i - r * rank))));
    }
}

}  // namespace tsp
