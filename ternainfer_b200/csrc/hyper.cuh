// Embedding and the residual stream of decoders with hyper-connections (several parallel residual
// streams per token, mixed anew around every sublayer), with the sublayer's RMS norm fused in.
//
// The streams live in fp32, x [rows][S][D].  One launch does what stands between two sublayers:
//   x_t <- sum_s mix[s][t] x_s + m * out[t] * y        (write the previous sublayer's output y back)
//   u = sum_s in[s] x_s                                (read for the next one)
//   h = u / sqrt(mean(u^2) + eps) * (w_offset + w)     (its norm, rounded to the activation type)
// Without y it only reads (first sublayer); with in = null the read is the plain sum of the streams
// (final norm); with a row list it reads and normalises those rows only and leaves x alone.
// One CTA per row; HBM traffic: the streams once in, once out, y in, h out.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"

namespace tsp {

typedef decoder_embed_args EmbedParams;

// x = embed[token] + bigram[(prev * mul_prev + token * mul_cur) mod buckets], all S streams alike.  A
// sequence's first token (position 0) takes the extra last bigram row.  prev is read and renewed by the
// CTA of a sequence's first token only.
template <typename E>
__global__ void __launch_bounds__(256) embed_kernel(const EmbedParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int row = blockIdx.x, b = row / p.T, t = row - b * p.T;
    const long long* tok = p.tokens + (size_t)b * p.T;
    const long long cur = tok[t];
    long long before = 0;
    bool first = false;
    if (t > 0) before = tok[t - 1];
    else if (p.pos[0] == 0) first = true;
    else before = p.prev ? p.prev[b] : 0;
    __syncthreads();
    if (t == 0 && threadIdx.x == 0 && p.prev) p.prev[b] = tok[p.T - 1];
    const bool tok_ok = cur >= 0 && cur < p.V;
    long long r = first ? p.buckets : (before * p.mul_prev + cur * p.mul_cur) % p.buckets;
    if (r < 0) r += p.buckets;
    const E* e = reinterpret_cast<const E*>(p.embed) + (tok_ok ? cur : 0) * (size_t)p.D;
    const E* g = reinterpret_cast<const E*>(p.bigram) + r * (size_t)p.D;
    float* x = p.x + (size_t)row * p.S * p.D;
    for (int d = threadIdx.x; d < p.D; d += blockDim.x) {
        float v = tok_ok ? to_f(e[d]) : 0.f;
        if (p.bigram) v += to_f(g[d]);
        for (int s = 0; s < p.S; ++s) x[(size_t)s * p.D + d] = v;
    }
}

typedef decoder_hyper_args HyperParams;

template <typename A, int S, int V>
__global__ void __launch_bounds__(1024) hyper_kernel(const HyperParams p) {
    extern __shared__ __align__(16) float u_s[];
    __shared__ float red[32];
    __shared__ float coef[S * S + 2 * S];
    griddep_launch_dependents();
    const int tid = threadIdx.x, D = p.D;
    for (int i = tid; i < S * S + 2 * S; i += blockDim.x) {
        if (i < S * S) coef[i] = p.y ? p.mix[i] : 0.f;
        else if (i < S * S + S) coef[i] = p.y ? p.m * p.out[i - S * S] : 0.f;
        else coef[i] = p.in ? p.in[i - S * S - S] : 1.f;
    }
    __syncthreads();
    float mix[S][S], out[S], in[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s][t] = coef[s * S + t];
        out[s] = coef[S * S + s];
        in[s] = coef[S * S + S + s];
    }
    griddep_wait();
    const size_t row = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
    float* xr = p.x + row * S * D;
    const A* yr = reinterpret_cast<const A*>(p.y) + row * D;
    const bool store = p.y && !p.rows;
    float ss = 0.f;
    for (int d = tid * V; d < D; d += blockDim.x * V) {
        float x[S][V];
#pragma unroll
        for (int s = 0; s < S; ++s) {
            if constexpr (V == 4) {
                const float4 v = ld_cg4(xr + (size_t)s * D + d);
                x[s][0] = v.x, x[s][1] = v.y, x[s][2] = v.z, x[s][3] = v.w;
            } else {
                x[s][0] = ld_cg(xr + (size_t)s * D + d);
            }
        }
        if (p.y) {
            float y[V], n[S][V];
            if constexpr (V == 4) {
                const float4 v = ld_cg4(yr + d);
                y[0] = v.x, y[1] = v.y, y[2] = v.z, y[3] = v.w;
            } else {
                y[0] = ld_cg(yr + d);
            }
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    float a = out[t] * y[i];
#pragma unroll
                    for (int s = 0; s < S; ++s) a = fmaf(mix[s][t], x[s][i], a);
                    n[t][i] = a;
                }
#pragma unroll
            for (int s = 0; s < S; ++s) {
#pragma unroll
                for (int i = 0; i < V; ++i) x[s][i] = n[s][i];
                if (store) {
                    if constexpr (V == 4) st4(xr + (size_t)s * D + d, make_float4(x[s][0], x[s][1], x[s][2], x[s][3]));
                    else xr[(size_t)s * D + d] = x[s][0];
                }
            }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) {
            float u = 0.f;
#pragma unroll
            for (int s = 0; s < S; ++s) u = fmaf(in[s], x[s][i], u);
            u_s[d + i] = u;
            ss = fmaf(u, u, ss);
        }
    }
    if (!p.h) return;
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)D + p.eps);
    A* h = reinterpret_cast<A*>(p.h) + (size_t)blockIdx.x * D;
    for (int d = tid * V; d < D; d += blockDim.x * V) {   // each thread reads back what it wrote itself
        if constexpr (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(p.w + d);
            const float4 u = *reinterpret_cast<const float4*>(u_s + d);
            st4(h + d, make_float4(u.x * inv * (p.w_offset + w.x), u.y * inv * (p.w_offset + w.y),
                                   u.z * inv * (p.w_offset + w.z), u.w * inv * (p.w_offset + w.w)));
        } else {
            h[d] = from_f<A>(u_s[d] * inv * (p.w_offset + p.w[d]));
        }
    }
}

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

}  // namespace tsp
