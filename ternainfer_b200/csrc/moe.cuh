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
__device__ __forceinline__ void choose(const float* z, int E, int top, int lane, int& expert, float& weight) {
    float v = INFINITY, best = 0.f, mine = 0.f;
    int e = -1;
    expert = 0;
    for (int j = 0; j < top; ++j) {
        next_choice(z, E, lane, v, e);
        if (j == 0) best = v;
        if (lane == j) expert = e, mine = expf(v - best);
    }
    weight = mine / warp_sum(mine);
}

// chosen, weights; with counts also every choice's place among its expert's: places inside the CTA's 32 tokens first, then
// one addition per CTA and expert
static __global__ void __launch_bounds__(1024) route_kernel(const MoeParams p) {
    extern __shared__ __align__(16) float route_smem[];      // logits [32][E], choices per expert [E]
    griddep_launch_dependents();
    griddep_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, token = blockIdx.x * 32 + warp, E = p.E;
    int* count = reinterpret_cast<int*>(route_smem + 32 * E);
    for (int i = tid; i < E; i += 1024) count[i] = 0;
    int e = 0, rank = 0;
    float w = 0.f;
    if (token < p.M) {
        float* z = route_smem + warp * E;
        for (int i = lane; i < E; i += 32) z[i] = __ldcg(p.logits + (size_t)token * E + i) + p.router_bias[i];
        __syncwarp();
        choose(z, E, p.top, lane, e, w);
    }
    const bool mine = token < p.M && lane < p.top;
    const int i = token * p.top + lane;
    if (mine) p.chosen[i] = e, p.weight[i] = w;
    if (!p.counts) return;
    __syncthreads();
    if (mine) rank = atomicAdd(count + e, 1);
    __syncthreads();
    for (int j = tid; j < E; j += 1024)
        if (count[j]) count[j] = atomicAdd(p.counts + j, count[j]);
    __syncthreads();
    if (mine) p.rank[i] = count[e] + rank;
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
    for (int c0 = lane; c0 < p.K / 8; c0 += 32 * 8) {        // eight loads in flight
        uint4 v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + 32 * j < p.K / 8) v[j] = __ldcg(reinterpret_cast<const uint4*>(src) + c0 + 32 * j);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + 32 * j < p.K / 8) stg_128(dst + (c0 + 32 * j) * 8, v[j]);
    }
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

// Routing, then act[token * top + j][f].  Every CTA makes the choices for itself.  Work items of 16 rows of gate and up of one chosen expert (8 activations), handed out as
// the CTAs come for them (kernels before and after share the SMs unevenly); the weights' stream runs on across items, P k-steps per warp ahead.  The inputs lie in shared memory.
template <int P>
__global__ void __launch_bounds__(kRowsWarps * 32, 2) moe_up_step_kernel(const MoeParams p) {
    extern __shared__ __align__(16) uint8_t moe_up_smem[];   // inputs [M][K] bf16, rows 64 bytes longer; logits [M][E]
    __shared__ float part[2][kRowsWarps][16][9];
    __shared__ int chosen[8 * kMoeMaxTop], list[8 * kMoeMaxTop], drawn[2];
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, q = lane & 3;
    const int K = p.K, steps = (K + 31) >> 5, top = p.top, blocks = p.ff / 8, xs = K * 2 + 64;
    const int s0 = steps * warp / kRowsWarps, s1 = steps * (warp + 1) / kRowsWarps;
    griddep_wait();
    const auto draw = [&]() { return (int)gridDim.x + atomicAdd(p.ticket, 1); };
    if (tid == 0) drawn[0] = draw();
    if (warp < p.M) {
        float* z = reinterpret_cast<float*>(moe_up_smem + p.M * xs) + warp * p.E;
        for (int i = lane; i < p.E; i += 32) z[i] = __ldcg(p.logits + (size_t)warp * p.E + i) + p.router_bias[i];
        __syncwarp();
        int e;
        float w;
        choose(z, p.E, top, lane, e, w);
        if (lane < top) {
            chosen[warp * top + lane] = e;
            if (blockIdx.x == 0) p.chosen[warp * top + lane] = e, p.weight[warp * top + lane] = w;
        }
    }
    for (int i = tid; i < p.M * (K / 8); i += blockDim.x) {
        const int t = i / (K / 8), c = i - t * (K / 8);
        *reinterpret_cast<uint4*>(moe_up_smem + t * xs + c * 16) = __ldcg(reinterpret_cast<const uint4*>(p.x) + i);
    }
    __syncthreads();
    const int n = distinct_experts(chosen, p.M * top, p.E, list);
    const int items = n * blocks;
    const bf16* w_up = reinterpret_cast<const bf16*>(p.w_up);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const int batches = max(1, (s1 - s0 + P - 1) / P);       // per item
    uint4 a[P], b[P];
    auto fetch = [&](int u, int item, int batch) {
        const int s = s0 + batch * P + u;
        const bool in = item < items && s < s1 && 32 * s + q * 8 < K;
        const bf16* w = w_up;
        if (in) w += ((size_t)list[item / blocks] * 2 * p.ff + item % blocks * 16 + g) * K + 32 * s + q * 8;
        a[u] = in ? ldg_stream_128(w) : zero;
        b[u] = in ? ldg_stream_128(w + (size_t)8 * K) : zero;
    };
    const uint8_t* xrow = moe_up_smem + g * xs + q * 16;
    int item = (int)blockIdx.x, next = drawn[0];
#pragma unroll
    for (int u = 0; u < P; ++u) fetch(u, item, 0);
    for (int turn = 0; item < items; ++turn) {
        int after = 0;
        if (tid == 0) after = draw();
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int batch = 0; batch < batches; ++batch) {
            const bool last = batch + 1 == batches;
#pragma unroll
            for (int u = 0; u < P; ++u) {
                const int s = s0 + batch * P + u;
                const uint4 xv = g < p.M && s < s1 && 32 * s + q * 8 < K ? *reinterpret_cast<const uint4*>(xrow + 64 * s) : zero;
                mma_bf16_16x8x16(acc, a[u].x, b[u].x, a[u].y, b[u].y, xv.x, xv.y);
                mma_bf16_16x8x16(acc, a[u].z, b[u].z, a[u].w, b[u].w, xv.z, xv.w);
                fetch(u, last ? next : item, last ? 0 : batch + 1);
            }
        }
        if (tid == 0) drawn[(turn + 1) & 1] = after;
        float (*pt)[16][9] = part[turn & 1];          // written again two items later, behind a barrier
        pt[warp][g][2 * q] = acc[0], pt[warp][g][2 * q + 1] = acc[1];
        pt[warp][g + 8][2 * q] = acc[2], pt[warp][g + 8][2 * q + 1] = acc[3];
        __syncthreads();
        if (tid < 128) {
            const int r = tid & 15, t = tid >> 4, e = list[item / blocks];
            float v = 0.f;
#pragma unroll
            for (int i = 0; i < kRowsWarps; ++i) v += pt[i][r][t];
            const float up = __shfl_down_sync(0xffffffffu, v, 8);
            int pair = -1;
            for (int j = 0; t < p.M && j < top; ++j)
                if (chosen[t * top + j] == e) pair = t * top + j;
            if (r < 8 && pair >= 0) reinterpret_cast<bf16*>(p.act)[(size_t)pair * p.ff + item % blocks * 8 + r] = from_f<bf16>(gated(v, up, p.gate));
        }
        item = next, next = drawn[(turn + 1) & 1];
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
