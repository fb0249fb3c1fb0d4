// Dense bf16 linear for decode-sized batches (up to 8 rows) on sm_100a: out[m][n] = act(sum_k W[n][k] x[m][k] + bias[n]).
//
// HBM-bound: W is read exactly once.  A CTA owns 16 rows of W; its eight warps split K, each streaming its
// slice with one 128-bit load per lane and row (lane (g, q) of the MMA holds rows g and g+8, 8 consecutive k
// starting at 8q; k is only a summation index, so the fragments of mma.sync m16n8k16 are filled straight from
// those registers, as in lm_head.cuh).  The first kRowsPre k-steps of W are requested before the wait for the
// previous kernel of the stream, so the weights' latency runs underneath its tail.  The rows of x are the
// MMA's N = 8 and come from L2.  Warp partials meet in shared memory in a fixed order.
// W may consist of segments of rows with an input each (projections of one token's differently mixed inputs in one
// launch).  A second product of the same row length (a router's logits) may ride along in CTAs of its own, with fp32
// results.  Gated feed-forwards: W holds blocks of 8 gate and 8 up rows, so a CTA makes 8 activations.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "gate.cuh"
#include "lm_head.cuh"

namespace tsp {

constexpr int kRowsWarps = 8;
constexpr int kRowsPre = 6;   // k-steps of 32 whose weights are in flight per warp: what two CTAs per SM have registers for

typedef decoder_linear_args RowsLinearParams;

template <typename O>
__global__ void __launch_bounds__(kRowsWarps * 32, 2) rows_linear_kernel(const RowsLinearParams p) {
    __shared__ float part[kRowsWarps][16][9];
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, q = lane & 3;
    const int K = p.K, steps = (K + 31) >> 5;
    const int blocks = (p.N + 15) >> 4;
    const bool side = (int)blockIdx.x >= blocks;
    const int n0 = ((int)blockIdx.x - (side ? blocks : 0)) * 16, N = side ? p.N2 : p.N;
    const int s0 = steps * warp / kRowsWarps, s1 = steps * (warp + 1) / kRowsWarps;
    const bool ok0 = n0 + g < N, ok1 = n0 + g + 8 < N;
    const bf16* w = reinterpret_cast<const bf16*>(side ? p.w2 : p.w);
    const bf16* w0 = w + (size_t)(ok0 ? n0 + g : 0) * K + q * 8;
    const bf16* w1 = w + (size_t)(ok1 ? n0 + g + 8 : 0) * K + q * 8;
    const int seg = !side && p.seg_rows > 0 ? min(n0 / p.seg_rows, p.n_seg - 1) : 0;
    const bf16* x = reinterpret_cast<const bf16*>(side ? p.x2 : p.x) + (size_t)seg * p.M * K + (size_t)(g < p.M ? g : 0) * K + q * 8;
    const bool xok = g < p.M;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    uint4 a[kRowsPre], b[kRowsPre];
    auto fetch = [&](int u, int s) {
        const bool in = s < s1 && 32 * s + q * 8 < K;
        a[u] = in ? ldg_stream_128(w0 + 32 * s) : zero;
        b[u] = in ? ldg_stream_128(w1 + 32 * s) : zero;
    };
#pragma unroll
    for (int u = 0; u < kRowsPre; ++u) fetch(u, s0 + u);
    griddep_wait();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = s0; s < s1; s += kRowsPre) {
        uint4 xv[kRowsPre];
#pragma unroll
        for (int u = 0; u < kRowsPre; ++u)
            xv[u] = (xok && s + u < s1 && 32 * (s + u) + q * 8 < K) ? ld_cg_128(x + 32 * (s + u)) : zero;
#pragma unroll
        for (int u = 0; u < kRowsPre; ++u) {
            mma_bf16_16x8x16(acc, a[u].x, b[u].x, a[u].y, b[u].y, xv[u].x, xv[u].y);
            mma_bf16_16x8x16(acc, a[u].z, b[u].z, a[u].w, b[u].w, xv[u].z, xv[u].w);
            fetch(u, s + kRowsPre + u);
        }
    }
    part[warp][g][2 * q] = acc[0], part[warp][g][2 * q + 1] = acc[1];
    part[warp][g + 8][2 * q] = acc[2], part[warp][g + 8][2 * q + 1] = acc[3];
    __syncthreads();
    if (tid < 128) {
        const int r = tid & 15, t = tid >> 4;
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < kRowsWarps; ++i) v += part[i][r][t];
        const bool live = t < p.M && n0 + r < N;
        if (side) {
            if (live) p.out2[(size_t)t * N + n0 + r] = v;
            if (p.zero && n0 == 0 && tid == 0) *p.zero = 0;
            return;
        }
        if (p.bias && n0 + r < p.N) v += p.bias[n0 + r];
        if (p.gate.kind) {
            const float up = __shfl_down_sync(0xffffffffu, v, 8);
            if (live && r < 8) reinterpret_cast<O*>(p.out)[(size_t)t * (p.N / 2) + n0 / 2 + r] = from_f<O>(gated(v, up, p.gate));
        } else if (live) {
            if (p.relu2) v = fmaxf(v, 0.f), v *= v;
            reinterpret_cast<O*>(p.out)[(size_t)t * p.N + n0 + r] = from_f<O>(v);
        }
    }
}

}  // namespace tsp
