// Embedding and the residual stream of decoders with hyper-connections (several parallel residual
// streams per token, mixed anew around every sublayer), with the sublayer's RMS norm fused in.
//
// The streams live in fp32, x [rows][S][D].  One launch does what stands between two sublayers:
//   x_t <- sum_s mix[s][t] x_s + m * out[t] * y        (write the previous sublayer's output y back)
// where, for a single stream, y may be the sum of two sublayers' outputs, the second optionally a weighted sum of gathered rows (the
// chosen experts of a token); without mix and out the streams stay apart and y goes to all of them.
//   u = sum_s in[s] x_s                                (read for the next one)
//   h = u / sqrt(mean(u^2) + eps) * (w_offset + w)     (its norm, rounded to the activation type)
// Without y it only reads (first sublayer); with in = null the read is the plain sum of the streams
// (final norm); with a row list it reads and normalises those rows only and leaves x alone.
// In a decode step of a single stream the same launch makes the inputs of projections that look one token back:
//   mixed_j = h + (h_before - h) * mu_j                 (h_before: the sequence's previous h, kept in prev)
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

__device__ __forceinline__ float shifted(float h, float before, float mu) { return fmaf(before - h, mu, h); }
template <typename A>
__device__ __forceinline__ float4 round_to(float4 v) {
    return make_float4(to_f(from_f<A>(v.x)), to_f(from_f<A>(v.y)), to_f(from_f<A>(v.z)), to_f(from_f<A>(v.w)));
}

template <typename A, int S, int V>
__global__ void __launch_bounds__(1024) hyper_kernel(const HyperParams p) {
    extern __shared__ __align__(16) float u_s[];
    __shared__ float red[32];
    __shared__ float coef[S * S + 2 * S];
    griddep_launch_dependents();
    const int tid = threadIdx.x, D = p.D;
    for (int i = tid; i < S * S + 2 * S; i += blockDim.x) {
        if (i < S * S) coef[i] = p.mix ? p.mix[i] : i % (S + 1) == 0 ? 1.f : 0.f;
        else if (i < S * S + S) coef[i] = p.out ? p.m * p.out[i - S * S] : p.m;
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
    const A* y2 = reinterpret_cast<const A*>(p.y2);
    const int n2 = S == 1 && p.y2 ? (p.top > 0 ? p.top : 1) : 0;
    const int n_mu = S == 1 ? p.n_mu : 0;
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
            for (int j = 0; j < n2; ++j) {
                const size_t r2 = p.top > 0 ? (size_t)__ldcg(p.slots + row * p.top + j) : row;
                const float w2 = p.top > 0 ? __ldcg(p.slot_w + row * p.top + j) : 1.f;
                if constexpr (V == 4) {
                    const float4 v = ld_cg4(y2 + r2 * D + d);
                    y[0] = fmaf(w2, v.x, y[0]), y[1] = fmaf(w2, v.y, y[1]), y[2] = fmaf(w2, v.z, y[2]), y[3] = fmaf(w2, v.w, y[3]);
                } else {
                    y[0] = fmaf(w2, ld_cg(y2 + r2 * D + d), y[0]);
                }
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
    const bool first = n_mu > 0 && p.pos[0] == 0;
    A* prev = reinterpret_cast<A*>(p.prev) + row * D;
    A* mixed = reinterpret_cast<A*>(p.mixed) + (size_t)blockIdx.x * D;
    for (int d = tid * V; d < D; d += blockDim.x * V) {   // each thread reads back what it wrote itself
        if constexpr (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(p.w + d);
            const float4 u = *reinterpret_cast<const float4*>(u_s + d);
            float4 n = make_float4(u.x * inv * (p.w_offset + w.x), u.y * inv * (p.w_offset + w.y), u.z * inv * (p.w_offset + w.z),
                                   u.w * inv * (p.w_offset + w.w));
            st4(h + d, n);
            if (n_mu > 0) {
                const float4 b = first ? make_float4(0.f, 0.f, 0.f, 0.f) : ld_cg4(prev + d);
                n = round_to<A>(n);                      // what later tokens and the prompt kernel see
                st4(prev + d, n);
                for (int j = 0; j < n_mu; ++j) {
                    const float4 m = *reinterpret_cast<const float4*>(p.mu + (size_t)j * D + d);
                    st4(mixed + (size_t)j * p.n_rows * D + d, make_float4(shifted(n.x, b.x, m.x), shifted(n.y, b.y, m.y),
                                                                          shifted(n.z, b.z, m.z), shifted(n.w, b.w, m.w)));
                }
            }
        } else {
            const A n = from_f<A>(u_s[d] * inv * (p.w_offset + p.w[d]));
            h[d] = n;
            if (n_mu > 0) {
                const float b = first ? 0.f : ld_cg(prev + d);
                prev[d] = n;
                for (int j = 0; j < n_mu; ++j)
                    mixed[(size_t)j * p.n_rows * D + d] = from_f<A>(shifted(to_f(n), b, p.mu[(size_t)j * D + d]));
            }
        }
    }
}

// Inputs of projections that look one token back, for a prompt portion: mixed[j][row] = h + (h_before - h) * mu_j.
// h_before of a sequence's first row is what earlier calls left in prev (zeros at position 0); the CTA of that row
// also renews prev, with the last row's h.
typedef decoder_shift_args ShiftParams;

template <typename A, int V>
__global__ void __launch_bounds__(256) token_shift_kernel(const ShiftParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int row = blockIdx.x, b = row / p.T, t = row - b * p.T, D = p.D;
    const size_t n = (size_t)p.B * p.T * D;
    const A* h = reinterpret_cast<const A*>(p.h) + (size_t)row * D;
    const A* last = reinterpret_cast<const A*>(p.h) + ((size_t)b * p.T + p.T - 1) * D;
    A* prev = reinterpret_cast<A*>(p.prev) + (size_t)b * D;
    A* mixed = reinterpret_cast<A*>(p.mixed) + (size_t)row * D;
    const bool first = t == 0 && p.pos[0] == 0;
    const A* before = t == 0 ? prev : h - D;
    for (int d = threadIdx.x * V; d < D; d += blockDim.x * V) {
        if constexpr (V == 4) {
            const float4 c = ld_cg4(h + d), o = first ? make_float4(0.f, 0.f, 0.f, 0.f) : ld_cg4(before + d);
            if (t == 0) st4(prev + d, ld_cg4(last + d));
            for (int j = 0; j < p.n_mu; ++j) {
                const float4 m = *reinterpret_cast<const float4*>(p.mu + (size_t)j * D + d);
                st4(mixed + j * n + d, make_float4(shifted(c.x, o.x, m.x), shifted(c.y, o.y, m.y), shifted(c.z, o.z, m.z),
                                                   shifted(c.w, o.w, m.w)));
            }
        } else {
            const float c = ld_cg(h + d), o = first ? 0.f : ld_cg(before + d);
            if (t == 0) prev[d] = from_f<A>(ld_cg(last + d));
            for (int j = 0; j < p.n_mu; ++j) mixed[j * n + d] = from_f<A>(shifted(c, o, p.mu[(size_t)j * D + d]));
        }
    }
}

}  // namespace tsp
