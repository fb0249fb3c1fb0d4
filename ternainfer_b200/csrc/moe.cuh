// Mixture of gated experts: routing, and the feed-forward of a token's chosen experts.
//
//   z = W_router h + b;  the `top` largest logits choose, weight = softmax over the chosen logits alone
//   y = sum over the chosen of weight * W_down (act(W_gate h) (W_up h))
//
// Weights: gate and up rows in blocks of eight in one matrix [E][2 * ff][K] (gate.cuh), down [E][D][ff]; ff padded to a
// multiple of 8.  Prompts (bf16): rows are sorted by expert and go through the grouped GEMM (group_gemm_tc.cuh); the
// residual kernel adds the weighted results (hyper.cuh).  Up to eight tokens: one launch routes and makes the
// activations, expert by expert, so that an expert's weights are read once for all its tokens; a second one sums the
// down projections of all experts, and the mixer's output projection with them, without leaving the registers.
// Other types and sizes: one warp per output.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "gate.cuh"
#include "rows_linear.cuh"

namespace tsp {

typedef decoder_moe_args MoeParams;

// One warp: the next choice after (v, e) in the order of falling logits, lower experts first among equals.
__device__ __forceinline__ void next_choice(const float* z, int E, int lane, float& v, int& e) {
    float bv = -INFINITY;
    int be = 0x7fffffff;
    for (int i = lane; i < E; i += 32) {
        const float x = z[i];
        if ((x < v || (x == v && i > e)) && (x > bv || (x == bv && i < be))) bv = x, be = i;
    }
#pragma unroll
    for (int d = 16; d; d >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, d);
        const int oe = __shfl_xor_sync(0xffffffffu, be, d);
        if (ov > bv || (ov == bv && oe < be)) bv = ov, be = oe;
    }
    v = bv, e = be < E ? be : E - 1;                         // (NaN logits: stay inside the table)
}

// One warp: the chosen experts of one token and their weights, top <= 32: lane j holds choice j.  z: [E] in shared memory.
__device__ __forceinline__ void route_token(const MoeParams& p, int token, float* z, int lane, int& expert, float& weight) {
    const float* logits = p.logits + (size_t)token * p.E;
    for (int i = lane; i < p.E; i += 32) z[i] = __ldcg(logits + i) + p.router_bias[i];
    __syncwarp();
    float v = INFINITY, best = 0.f, mine = 0.f;
    int e = -1;
    expert = 0;
    for (int j = 0; j < p.top; ++j) {
        next_choice(z, p.E, lane, v, e);
        if (j == 0) best = v;
        if (lane == j) expert = e, mine = expf(v - best);
    }
    weight = mine / warp_sum(mine);
}

// chosen, weights; with counts also every choice's place among its expert's
static __global__ void __launch_bounds__(256) route_kernel(const MoeParams p) {
    extern __shared__ __align__(16) float route_smem[];      // [8][E]
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, token = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (token >= p.M) return;
    int e;
    float w;
    route_token(p, token, route_smem + (threadIdx.x >> 5) * p.E, lane, e, w);
    if (lane < p.top) {
        const int i = token * p.top + lane;
        p.chosen[i] = e, p.weight[i] = w;
        if (p.counts) p.rank[i] = atomicAdd(p.counts + e, 1);
    }
}

// Rows sorted by expert: one warp per choice finds its slot and copies the token's row there.
static __global__ void __launch_bounds__(256) sort_rows_kernel(const MoeParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, i = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= p.M * p.top) return;
    const int e = __ldcg(p.chosen + i);
    int before = 0;
    for (int c = lane; c < e; c += 32) before += __ldcg(p.counts + c);
#pragma unroll
    for (int d = 16; d; d >>= 1) before += __shfl_xor_sync(0xffffffffu, before, d);
    const int slot = before + __ldcg(p.rank + i);
    if (lane == 0) p.slots[i] = slot;
    const bf16* src = reinterpret_cast<const bf16*>(p.x) + (size_t)(i / p.top) * p.K;
    bf16* dst = reinterpret_cast<bf16*>(p.sorted) + (size_t)slot * p.K;
    for (int c = lane; c < p.K / 8; c += 32) stg_128(dst + c * 8, ld_cg_128(src + c * 8));
}

// ------------------------------------------------------------------------------------------ any type, any size
// act[choice][f]: CTA x = choice, y = 64 activations, one warp each in turn
template <typename A>
__global__ void __launch_bounds__(256) moe_up_plain_kernel(const MoeParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, i = blockIdx.x;
    const A* x = reinterpret_cast<const A*>(p.x) + (size_t)(i / p.top) * p.K;
    const A* w = reinterpret_cast<const A*>(p.w_up) + (size_t)__ldcg(p.chosen + i) * 2 * p.ff * p.K;
    for (int f = blockIdx.y * 64 + warp; f < min(p.ff, blockIdx.y * 64 + 64); f += 8) {
        const A *wg = w + (size_t)(f / 8 * 16 + f % 8) * p.K, *wu = wg + (size_t)8 * p.K;
        float g = 0.f, u = 0.f;
        for (int c = lane; c < p.K; c += 32) {
            const float v = ld_cg(x + c);
            g = fmaf(to_f(wg[c]), v, g), u = fmaf(to_f(wu[c]), v, u);
        }
        g = warp_sum(g), u = warp_sum(u);
        if (lane == 0) reinterpret_cast<A*>(p.act)[(size_t)i * p.ff + f] = from_f<A>(gated(g, u, p.gate));
    }
}
// out[choice][d], not weighted
template <typename A>
__global__ void __launch_bounds__(256) moe_down_plain_kernel(const MoeParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, i = blockIdx.x;
    const A* x = reinterpret_cast<const A*>(p.act) + (size_t)i * p.ff;
    const A* w = reinterpret_cast<const A*>(p.w_down) + (size_t)__ldcg(p.chosen + i) * p.D * p.ff;
    for (int d = blockIdx.y * 64 + warp; d < min(p.D, blockIdx.y * 64 + 64); d += 8) {
        const A* wd = w + (size_t)d * p.ff;
        float v = 0.f;
        for (int c = lane; c < p.ff; c += 32) v = fmaf(to_f(wd[c]), ld_cg(x + c), v);
        v = warp_sum(v);
        if (lane == 0) reinterpret_cast<A*>(p.out)[(size_t)i * p.D + d] = from_f<A>(v);
    }
}

// ------------------------------------------------------------------------------------------ up to eight bf16 tokens
constexpr int kMoeMaxTop = 32;

constexpr int kMoeMaxExperts = 1024;

// The experts in chosen[0 .. n), each once and in rising order -> list, their number; all threads of the CTA take part.
__device__ __forceinline__ int distinct_experts(const int* chosen, int n, int E, int* list) {
    __shared__ unsigned mask[kMoeMaxExperts / 32];
    const int words = (E + 31) / 32;
    for (int i = threadIdx.x; i < words; i += blockDim.x) mask[i] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) atomicOr(&mask[chosen[i] >> 5], 1u << (chosen[i] & 31));
    __syncthreads();
    int count = 0;
    for (int i = 0; i < words; ++i) count += __popc(mask[i]);
    for (int e = threadIdx.x; e < E; e += blockDim.x)
        if (mask[e >> 5] >> (e & 31) & 1) {
            int before = __popc(mask[e >> 5] & ((1u << (e & 31)) - 1));
            for (int i = 0; i < e >> 5; ++i) before += __popc(mask[i]);
            list[before] = e;
        }
    __syncthreads();
    return count;
}

// act[token * top + j][f]: CTAs x = 16 rows of gate and up (8 activations), y = one of the chosen experts
static __global__ void __launch_bounds__(kRowsWarps * 32, 2) moe_up_step_kernel(const MoeParams p) {
    extern __shared__ __align__(16) float moe_step_smem[];   // logits [8][E]
    __shared__ float part[kRowsWarps][16][9];
    __shared__ int chosen[8 * kMoeMaxTop], list[8 * kMoeMaxTop], pair_of[8];
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, q = lane & 3;
    const int K = p.K, steps = (K + 31) >> 5, top = p.top, n0 = blockIdx.x * 16;
    const int s0 = steps * warp / kRowsWarps, s1 = steps * (warp + 1) / kRowsWarps;
    if (tid < 8) pair_of[tid] = -1;
    griddep_wait();
    if (warp < p.M) {
        int e;
        float w;
        route_token(p, warp, moe_step_smem + warp * p.E, lane, e, w);
        if (lane < top) {
            chosen[warp * top + lane] = e;
            if (blockIdx.x == 0 && blockIdx.y == 0) p.chosen[warp * top + lane] = e, p.weight[warp * top + lane] = w;
        }
    }
    __syncthreads();
    const int n = distinct_experts(chosen, p.M * top, p.E, list);
    if ((int)blockIdx.y >= n) return;
    const int e = list[blockIdx.y];
    for (int i = tid; i < p.M * top; i += blockDim.x)
        if (chosen[i] == e) pair_of[i / top] = i;
    __syncthreads();
    const bf16* w = reinterpret_cast<const bf16*>(p.w_up) + ((size_t)e * 2 * p.ff + n0) * K + q * 8;
    const bf16 *w0 = w + (size_t)g * K, *w1 = w + (size_t)(g + 8) * K;
    const bf16* x = reinterpret_cast<const bf16*>(p.x) + (size_t)(g < p.M ? g : 0) * K + q * 8;
    const bool xok = g < p.M && pair_of[g] >= 0;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = s0; s < s1; s += kRowsPre) {
        uint4 a[kRowsPre], b[kRowsPre], xv[kRowsPre];
#pragma unroll
        for (int u = 0; u < kRowsPre; ++u) {
            const bool in = s + u < s1 && 32 * (s + u) + q * 8 < K;
            a[u] = in ? ldg_stream_128(w0 + 32 * (s + u)) : zero;
            b[u] = in ? ldg_stream_128(w1 + 32 * (s + u)) : zero;
            xv[u] = in && xok ? ld_cg_128(x + 32 * (s + u)) : zero;
        }
#pragma unroll
        for (int u = 0; u < kRowsPre; ++u) {
            mma_bf16_16x8x16(acc, a[u].x, b[u].x, a[u].y, b[u].y, xv[u].x, xv[u].y);
            mma_bf16_16x8x16(acc, a[u].z, b[u].z, a[u].w, b[u].w, xv[u].z, xv[u].w);
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
        const float up = __shfl_down_sync(0xffffffffu, v, 8);
        if (r < 8 && pair_of[t] >= 0) reinterpret_cast<bf16*>(p.act)[(size_t)pair_of[t] * p.ff + n0 / 2 + r] = from_f<bf16>(gated(v, up, p.gate));
    }
}

// y[token][d] = sum over the chosen experts of weight * (W_down act)[d], plus W_rest rest and a bias (dense feed-forward:
// E = top = 1, weight NULL, act [M][ff]).  CTAs of 16 rows; the warps split the summation index over all products.
static __global__ void __launch_bounds__(kRowsWarps * 32, 2) moe_down_step_kernel(const MoeParams p) {
    __shared__ float part[kRowsWarps][16][9];
    __shared__ int chosen[8 * kMoeMaxTop], list[8 * kMoeMaxTop];
    __shared__ float weight[8 * kMoeMaxTop];
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, q = lane & 3;
    const int top = p.top, n0 = blockIdx.x * 16;
    const bool routed = p.weight != nullptr;
    const bool ok0 = n0 + g < p.D, ok1 = n0 + g + 8 < p.D;
    const int d0 = ok0 ? n0 + g : 0, d1 = ok1 ? n0 + g + 8 : 0;
    griddep_wait();
    int n = p.w_down ? 1 : 0;
    if (routed) {
        for (int i = tid; i < p.M * top; i += blockDim.x) chosen[i] = __ldcg(p.chosen + i), weight[i] = __ldcg(p.weight + i);
        __syncthreads();
        n = distinct_experts(chosen, p.M * top, p.E, list);
    }
    const int rest_steps = p.w_rest ? (p.K_rest + 31) >> 5 : 0, steps = (p.ff + 31) >> 5;
    const int total = rest_steps + n * steps;
    const int s0 = (int)((long long)total * warp / kRowsWarps), s1 = (int)((long long)total * (warp + 1) / kRowsWarps);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float sum[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = s0; s < s1;) {                              // one product at a time: rest, then expert by expert
        const bool rest = s < rest_steps;
        const int i = rest ? 0 : (s - rest_steps) / steps;
        const int first = rest ? 0 : rest_steps + i * steps, last = rest ? min(s1, rest_steps) : min(s1, first + steps);
        const int K = rest ? p.K_rest : p.ff, e = rest || !routed ? 0 : list[i];
        const bf16* w = rest ? reinterpret_cast<const bf16*>(p.w_rest) : reinterpret_cast<const bf16*>(p.w_down) + (size_t)e * p.D * K;
        const bf16 *w0 = w + (size_t)d0 * K + q * 8, *w1 = w + (size_t)d1 * K + q * 8;
        int row = g < p.M ? g : -1;
        float wt[2] = {1.f, 1.f};                            // of tokens 2q and 2q + 1
        if (!rest && routed) {
            row = -1, wt[0] = wt[1] = 0.f;
            for (int j = 0; j < top; ++j) {
                if (g < p.M && chosen[g * top + j] == e) row = g * top + j;
#pragma unroll
                for (int c = 0; c < 2; ++c)
                    if (2 * q + c < p.M && chosen[(2 * q + c) * top + j] == e) wt[c] = weight[(2 * q + c) * top + j];
            }
        }
        const bf16* x = reinterpret_cast<const bf16*>(rest ? p.rest : p.act) + (size_t)max(row, 0) * K + q * 8;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (; s < last; s += kRowsPre) {
            uint4 a[kRowsPre], b[kRowsPre], xv[kRowsPre];
#pragma unroll
            for (int u = 0; u < kRowsPre; ++u) {
                const int at = 32 * (s + u - first);
                const bool in = s + u < last && at + q * 8 < K;
                a[u] = in ? ldg_stream_128(w0 + at) : zero;
                b[u] = in ? ldg_stream_128(w1 + at) : zero;
                xv[u] = in && row >= 0 ? ld_cg_128(x + at) : zero;
            }
#pragma unroll
            for (int u = 0; u < kRowsPre; ++u) {
                mma_bf16_16x8x16(acc, a[u].x, b[u].x, a[u].y, b[u].y, xv[u].x, xv[u].y);
                mma_bf16_16x8x16(acc, a[u].z, b[u].z, a[u].w, b[u].w, xv[u].z, xv[u].w);
            }
        }
        s = last;
#pragma unroll
        for (int c = 0; c < 4; ++c) sum[c] = fmaf(wt[c & 1], acc[c], sum[c]);
    }
    part[warp][g][2 * q] = sum[0], part[warp][g][2 * q + 1] = sum[1];
    part[warp][g + 8][2 * q] = sum[2], part[warp][g + 8][2 * q + 1] = sum[3];
    __syncthreads();
    if (tid < 128) {
        const int r = tid & 15, t = tid >> 4;
        if (t < p.M && n0 + r < p.D) {
            float v = p.bias ? p.bias[n0 + r] : 0.f;
#pragma unroll
            for (int i = 0; i < kRowsWarps; ++i) v += part[i][r][t];
            reinterpret_cast<bf16*>(p.out)[(size_t)t * p.D + n0 + r] = from_f<bf16>(v);
        }
    }
}

}  // namespace tsp
