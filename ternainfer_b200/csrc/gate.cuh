// Activations of gated feed-forwards from a gate and an up projection.
//   kind 1: silu(g) * u
//   kind 2: g * sigmoid(alpha * g) * (u + 1) with g at most limit and u within +-limit
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"

namespace tsp {

// FAST: the logistic function with the approximate reciprocal
template <bool FAST = false>
__device__ __forceinline__ float gated(float g, float u, const decoder_gate& s) {
    const auto sigma = [](float z) { return FAST ? sigmoid_fast(z) : sigmoid_f(z); };
    if (s.kind == 1) return g * sigma(g) * u;
    g = fminf(g, s.limit), u = fminf(fmaxf(u, -s.limit), s.limit);
    return g * sigma(s.alpha * g) * (u + 1.f);
}

// z [rows][2 * n] in blocks of 8 gate and 8 up columns, bias alike -> out [rows][n]
template <typename A>
__global__ void __launch_bounds__(256) gated_kernel(const A* z, const float* bias, A* out, long long rows, int n, const decoder_gate s) {
    griddep_launch_dependents();
    griddep_wait();
    const long long total = rows * n, stride = (long long)gridDim.x * blockDim.x;
    if (n % 4 == 0) {
        for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total / 4; i += stride) {
            const long long r = 4 * i / n;
            const int c = (int)(4 * i - r * n), at = c / 8 * 16 + c % 8;
            float4 g = ld_cg4(z + r * 2 * n + at), u = ld_cg4(z + r * 2 * n + at + 8);
            if (bias) {
                const float4 bg = *reinterpret_cast<const float4*>(bias + at), bu = *reinterpret_cast<const float4*>(bias + at + 8);
                g = make_float4(g.x + bg.x, g.y + bg.y, g.z + bg.z, g.w + bg.w);
                u = make_float4(u.x + bu.x, u.y + bu.y, u.z + bu.z, u.w + bu.w);
            }
            st4(out + r * n + c, make_float4(gated(g.x, u.x, s), gated(g.y, u.y, s), gated(g.z, u.z, s), gated(g.w, u.w, s)));
        }
    }
}

}  // namespace tsp
