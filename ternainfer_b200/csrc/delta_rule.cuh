// Generalised delta rule: a matrix-valued recurrent state per head with per-channel decay and a removal term.
//
//   u_t = k_t / sqrt(sum(k_t^2) + 1e-6)                               unit key
//   S_t = diag(w_t) S_{t-1} - (a_t * u_t) (u_t^T S_{t-1}) + k_t v_t^T  state [dk][dv], fp32
//   o_t = S_t^T r_t
//   y_t = o_t / sqrt(mean(o_t^2) + eps) * norm * sigmoid(g_t)          per head
// with w = exp(-exp(-1/2) sigmoid(zw + w0)) and a = sigmoid(za + a_b); everything but the projections in fp32.
//
// Columns of S are independent of one another given the per-token vectors, so the prompt kernel gives each
// CTA 16 columns of one head: four warps hold them in registers (lane = 8 row groups x 4 columns, packed
// fp32 pairs) and walk the tokens, four more warps turn the projections of the NEXT 16 tokens into the fp32
// vectors (u, w, a*u, k, r) in shared memory meanwhile.  A second kernel normalises and gates (the root mean
// square runs over all columns of a head).  The decode kernel does one token of one head in one CTA, from the
// projections to the gated output, the state read and written once.
// A sequence starts with a zero state: position 0 ignores what the state buffer holds.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "lm_head.cuh"

namespace tsp {

constexpr float kDecayScale = 0.60653065971263342f;   // exp(-1/2)

typedef decoder_delta_args DeltaParams;

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)),
          "l"(reinterpret_cast<const unsigned long long&>(c)));
    return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.rn.f32x2 %0, %1, %2;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)));
    return d;
}

// ------------------------------------------------------------------------------------------ prompts
constexpr int kScanCols = 16;
template <int RPT>
struct ScanShape {
    static constexpr int DK = 8 * RPT;                      // padded key channels
    static constexpr int CH = RPT > 16 ? 8 : 16;            // tokens staged at a time
    static constexpr int TPW = CH / 4;                      // tokens per producer warp
    static constexpr int CPL = DK / 32;                     // channels per producer lane
    static constexpr int smem = (2 * CH * 5 * DK + 2 * CH * kScanCols) * 4;
};

template <typename A, int RPT>
__global__ void __launch_bounds__(256) delta_scan_kernel(const DeltaParams p) {
    using L = ScanShape<RPT>;
    constexpr int DK = L::DK, CH = L::CH;
    extern __shared__ __align__(16) float scan_smem[];
    float* vec = scan_smem;                                 // [2][CH][5][DK]: u, w, a*u, k, r
    float* val = scan_smem + 2 * CH * 5 * DK;               // [2][CH][16]
    griddep_launch_dependents();
    griddep_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c0 = blockIdx.x * kScanCols, head = blockIdx.y, b = blockIdx.z;
    const int T = p.T, dk = p.dk, dv = p.dv;
    const int chunks = (T + CH - 1) / CH;
    const size_t row0 = (size_t)b * T;

    if (warp >= 4) {
        // ------------------------------------------------ producers: projections -> fp32 vectors
        const int pw = warp - 4;
        const A* proj = reinterpret_cast<const A*>(p.proj);
        float zk[L::TPW][L::CPL], zr[L::TPW][L::CPL], za[L::TPW][L::CPL], zw[L::TPW][L::CPL], zv[L::TPW];
        float w0[L::CPL], ab[L::CPL];
#pragma unroll
        for (int j = 0; j < L::CPL; ++j) {
            const int c = lane + 32 * j;
            w0[j] = c < dk ? p.w0[head * dk + c] : 0.f;
            ab[j] = c < dk ? p.a_bias[head * dk + c] : 0.f;
        }
        auto load = [&](int chunk) {
#pragma unroll
            for (int i = 0; i < L::TPW; ++i) {
                const int t = chunk * CH + pw + 4 * i;
                const bool live = t < T;
                const A* row = proj + (row0 + (live ? t : 0)) * p.ld;
#pragma unroll
                for (int j = 0; j < L::CPL; ++j) {
                    const int c = lane + 32 * j;
                    const bool ok = live && c < dk;
                    zk[i][j] = ok ? ld_cg(row + p.off_k + head * dk + c) : 0.f;
                    zr[i][j] = ok ? ld_cg(row + p.off_r + head * dk + c) : 0.f;
                    za[i][j] = ok ? ld_cg(row + p.off_a + head * dk + c) : 0.f;
                    zw[i][j] = ok ? ld_cg(p.zw + (row0 + t) * ((size_t)p.H * dk) + head * dk + c) : 0.f;
                }
                zv[i] = (live && lane < kScanCols && c0 + lane < dv) ? ld_cg(row + p.off_v + head * dv + c0 + lane) : 0.f;
            }
        };
        auto emit = [&](int chunk) {
            float* vb = vec + (size_t)(chunk & 1) * CH * 5 * DK;
            float* wb = val + (chunk & 1) * CH * kScanCols;
#pragma unroll
            for (int i = 0; i < L::TPW; ++i) {
                const int tt = pw + 4 * i;
                float ss = 0.f;
#pragma unroll
                for (int j = 0; j < L::CPL; ++j) ss = fmaf(zk[i][j], zk[i][j], ss);
                const float inv = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
#pragma unroll
                for (int j = 0; j < L::CPL; ++j) {
                    const int c = lane + 32 * j;
                    const float u = zk[i][j] * inv;
                    float* dst = vb + tt * 5 * DK + c;
                    dst[0] = u;
                    dst[DK] = __expf(-kDecayScale * sigmoid_f(zw[i][j] + w0[j]));
                    dst[2 * DK] = sigmoid_f(za[i][j] + ab[j]) * u;
                    dst[3 * DK] = zk[i][j];
                    dst[4 * DK] = zr[i][j];
                }
                if (lane < kScanCols) wb[tt * kScanCols + lane] = zv[i];
            }
        };
        load(0);
        emit(0);
        if (chunks > 1) load(1);
        __syncthreads();
        for (int c = 0; c < chunks; ++c) {
            if (c + 1 < chunks) {
                emit(c + 1);
                if (c + 2 < chunks) load(c + 2);
            }
            __syncthreads();
        }
        return;
    }

    // -------------------------------------------------- consumers: the recurrence
    const int ks = lane & 7, cl = warp * 4 + (lane >> 3), col = c0 + cl;
    const bool live_col = col < dv;
    float2 s[RPT / 2];                                      // rows 32*i + 4*ks + 0..3, i = 0 .. RPT/4 - 1
    float* st = p.state + ((size_t)b * p.H + head) * dk * dv;
    const bool fresh = p.pos[0] == 0;
#pragma unroll
    for (int i = 0; i < RPT / 4; ++i) {
        float f[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int k = 32 * i + 4 * ks + e;
            f[e] = (!fresh && live_col && k < dk) ? ld_cg(st + (size_t)k * dv + col) : 0.f;
        }
        s[2 * i] = make_float2(f[0], f[1]), s[2 * i + 1] = make_float2(f[2], f[3]);
    }
    __syncthreads();
    for (int c = 0; c < chunks; ++c) {
        const float* vb = vec + (size_t)(c & 1) * CH * 5 * DK + 4 * ks;
        const float* wb = val + (c & 1) * CH * kScanCols + cl;
        const int n = min(CH, T - c * CH);
        for (int t8 = 0; t8 < n; t8 += 8) {
            float part[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                part[j] = 0.f;
                if (t8 + j < n) {
                    const float* q = vb + (t8 + j) * 5 * DK;
                    float2 d0 = make_float2(0.f, 0.f), d1 = d0;
#pragma unroll
                    for (int i = 0; i < RPT / 4; ++i) {
                        const float4 u = *reinterpret_cast<const float4*>(q + 32 * i);
                        d0 = fma2(make_float2(u.x, u.y), s[2 * i], d0);
                        d1 = fma2(make_float2(u.z, u.w), s[2 * i + 1], d1);
                    }
                    float seen = (d0.x + d0.y) + (d1.x + d1.y);
                    seen += __shfl_xor_sync(0xffffffffu, seen, 1);
                    seen += __shfl_xor_sync(0xffffffffu, seen, 2);
                    seen += __shfl_xor_sync(0xffffffffu, seen, 4);
                    const float2 neg = make_float2(-seen, -seen);
                    const float v = wb[(t8 + j) * kScanCols];
                    const float2 vv = make_float2(v, v);
                    float2 o0 = make_float2(0.f, 0.f), o1 = o0;
#pragma unroll
                    for (int i = 0; i < RPT / 4; ++i) {
                        const float4 w = *reinterpret_cast<const float4*>(q + DK + 32 * i);
                        const float4 au = *reinterpret_cast<const float4*>(q + 2 * DK + 32 * i);
                        const float4 k = *reinterpret_cast<const float4*>(q + 3 * DK + 32 * i);
                        const float4 r = *reinterpret_cast<const float4*>(q + 4 * DK + 32 * i);
                        // decayed state plus the new pair does not wait for the removal term
                        const float2 m0 = fma2(make_float2(w.x, w.y), s[2 * i], mul2(make_float2(k.x, k.y), vv));
                        const float2 m1 = fma2(make_float2(w.z, w.w), s[2 * i + 1], mul2(make_float2(k.z, k.w), vv));
                        s[2 * i] = fma2(make_float2(au.x, au.y), neg, m0);
                        s[2 * i + 1] = fma2(make_float2(au.z, au.w), neg, m1);
                        o0 = fma2(make_float2(r.x, r.y), s[2 * i], o0);
                        o1 = fma2(make_float2(r.z, r.w), s[2 * i + 1], o1);
                    }
                    part[j] = (o0.x + o0.y) + (o1.x + o1.y);
                }
            }
            // eight partial outputs over eight row groups: a transposing butterfly leaves token t8 + ks in lane ks
            float h4[4], h2[2];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float keep = (ks & 4) ? part[j + 4] : part[j], give = (ks & 4) ? part[j] : part[j + 4];
                h4[j] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
            }
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const float keep = (ks & 2) ? h4[j + 2] : h4[j], give = (ks & 2) ? h4[j] : h4[j + 2];
                h2[j] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
            }
            const float keep = (ks & 1) ? h2[1] : h2[0], give = (ks & 1) ? h2[0] : h2[1];
            const float o = keep + __shfl_xor_sync(0xffffffffu, give, 1);
            const int t = c * CH + t8 + ks;
            if (t8 + ks < n && live_col) p.o[(row0 + t) * ((size_t)p.H * dv) + (size_t)head * dv + col] = o;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < RPT / 4; ++i) {
        const float f[4] = {s[2 * i].x, s[2 * i].y, s[2 * i + 1].x, s[2 * i + 1].y};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int k = 32 * i + 4 * ks + e;
            if (live_col && k < dk) st[(size_t)k * dv + col] = f[e];
        }
    }
}

// y = o / rms(o) * norm * sigmoid(gate), one warp per row and head
template <typename A>
__global__ void __launch_bounds__(256) delta_finish_kernel(const DeltaParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long unit = (long long)blockIdx.x * 8 + warp;
    if (unit >= (long long)p.B * p.T * p.H) return;
    const long long row = unit / p.H;
    const int head = (int)(unit - row * p.H), dv = p.dv;
    const float* o = p.o + row * ((long long)p.H * dv) + head * dv;
    const A* g = reinterpret_cast<const A*>(p.proj) + row * p.ld + p.off_g + head * dv;
    A* y = reinterpret_cast<A*>(p.y) + row * ((long long)p.H * dv) + head * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) {
        const float v = ld_cg(o + c);
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
    for (int c = lane; c < dv; c += 32)
        y[c] = from_f<A>(ld_cg(o + c) * inv * p.norm[head * dv + c] * sigmoid_f(ld_cg(g + c)));
}

// The same with four neighbouring columns per lane: dv a power of two from 4 to 128, so that dv / 4 lanes share a head;
// two units of 128 columns per warp in flight.
template <typename A>
__global__ void __launch_bounds__(256) delta_finish4_kernel(const DeltaParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long n = (long long)p.H * p.dv, total = (long long)p.B * p.T * n;
    float4 o[2], g[2];
    long long at[2];
    int col[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        at[i] = (((long long)blockIdx.x * 8 + warp) * 2 + i) * 128 + lane * 4;
        const long long e = min(at[i], total - 4), row = e / n;
        col[i] = (int)(e - row * n);
        o[i] = ld_cg4(p.o + e);
        g[i] = ld_cg4(reinterpret_cast<const A*>(p.proj) + row * p.ld + p.off_g + col[i]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        float ss = o[i].x * o[i].x + o[i].y * o[i].y + o[i].z * o[i].z + o[i].w * o[i].w;
        for (int d = p.dv / 8; d; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
        const float inv = 1.f / sqrtf(ss / (float)p.dv + p.eps);
        const float4 w = *reinterpret_cast<const float4*>(p.norm + col[i]);
        if (at[i] < total)
            st4(reinterpret_cast<A*>(p.y) + at[i], make_float4(o[i].x * inv * w.x * sigmoid_fast(g[i].x), o[i].y * inv * w.y * sigmoid_fast(g[i].y),
                                                               o[i].z * inv * w.z * sigmoid_fast(g[i].z), o[i].w * inv * w.w * sigmoid_fast(g[i].w)));
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

// ------------------------------------------------------------------------------------------ one token
constexpr int kStepThreads = 512;

// NR: state rows a thread keeps in registers (dk <= NR * row groups); 0: the state is read twice instead.
// WIDE: rank a multiple of 8 and dk * rank / 8 words of 16 bytes of w2 (bf16) are at most WIDE per thread: they are
// requested before the wait for the projections.
template <typename A, int NR, int WIDE>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const DeltaParams p, const int dvp) {
    extern __shared__ __align__(16) float step_smem[];
    __shared__ float red[32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = kStepThreads / 32;
    const int dk = p.dk, dv = p.dv, rank = p.rank;
    const int head = blockIdx.x, b = blockIdx.y;
    const int RG = kStepThreads / dvp;                      // row groups; dvp a power of two >= dv
    float* u_s = step_smem;
    float *w_s = u_s + dk, *au_s = w_s + dk, *k_s = au_s + dk, *r_s = k_s + dk, *t1_s = r_s + dk;
    float* part = t1_s + (rank + 3) / 4 * 4;                // [RG][dvp], and the decay's partial sums [dk][rank / 8]
    griddep_launch_dependents();
    const A* w2 = reinterpret_cast<const A*>(p.w2) + (size_t)head * dk * rank;
    const int per = rank / 8, words = dk * per;             // (WIDE) a word = 8 ranks of one channel
    uint4 wv[WIDE > 0 ? WIDE : 1];
    if constexpr (WIDE > 0) {
#pragma unroll
        for (int i = 0; i < WIDE; ++i) {
            const int e = tid + i * kStepThreads;
            wv[i] = e < words ? ldg_stream_128(w2 + (size_t)e * 8) : make_uint4(0, 0, 0, 0);
        }
    }
    griddep_wait();
    const A* row = reinterpret_cast<const A*>(p.proj) + (size_t)b * p.ld;
    float* st = p.state + ((size_t)b * p.H + head) * dk * dv;
    const int col = tid & (dvp - 1), rg = tid / dvp;
    const bool live = col < dv;
    float s[NR > 0 ? NR : 1];
    if constexpr (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int k = rg + i * RG;
            s[i] = (live && k < dk) ? ld_cg(st + (size_t)k * dv + col) : 0.f;
        }
    }
    const bool fresh = p.pos[0] == 0;
    const float v = live ? ld_cg(row + p.off_v + head * dv + col) : 0.f;
    const float gate = live ? ld_cg(row + p.off_g + head * dv + col) : 0.f;
    float ss = 0.f;
    for (int c = tid; c < dk; c += kStepThreads) {
        const float k = ld_cg(row + p.off_k + head * dk + c);
        k_s[c] = k, r_s[c] = ld_cg(row + p.off_r + head * dk + c);
        au_s[c] = sigmoid_f(ld_cg(row + p.off_a + head * dk + c) + p.a_bias[head * dk + c]);
        ss = fmaf(k, k, ss);
    }
    for (int c = tid; c < rank; c += kStepThreads) t1_s[c] = tanhf(ld_cg(row + p.off_w1 + c));
    const float inv = 1.f / sqrtf(block_sum(ss, red) + 1e-6f);
    if constexpr (WIDE > 0) {
#pragma unroll
        for (int i = 0; i < WIDE; ++i) {
            const int e = tid + i * kStepThreads;
            if (e < words) {
                float f[8], z = 0.f;
                unpack8(wv[i], f);
                const float* t = t1_s + (e % per) * 8;
#pragma unroll
                for (int j = 0; j < 8; ++j) z = fmaf(f[j], t[j], z);
                part[e] = z;
            }
        }
        __syncthreads();
    }
    for (int c = WIDE > 0 ? tid : warp; c < dk; c += WIDE > 0 ? kStepThreads : nw) {
        float z = 0.f;
        if constexpr (WIDE > 0) {
            for (int j = 0; j < per; ++j) z += part[c * per + j];
        } else {                                            // one warp per channel, lanes over the rank
            for (int j = lane; j < rank; j += 32) z = fmaf(to_f(w2[(size_t)c * rank + j]), t1_s[j], z);
            z = warp_sum(z);
        }
        if (WIDE > 0 || lane == 0) {
            const float u = k_s[c] * inv;
            u_s[c] = u, au_s[c] *= u;
            w_s[c] = __expf(-kDecayScale * sigmoid_f(z + p.w0[head * dk + c]));
        }
    }
    if (fresh) {
#pragma unroll
        for (int i = 0; i < (NR > 0 ? NR : 1); ++i) s[i] = 0.f;
    }
    __syncthreads();
    float seen = 0.f;
    if constexpr (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int k = rg + i * RG;
            if (k < dk) seen = fmaf(u_s[k], s[i], seen);
        }
    } else {
        for (int k = rg; k < dk; k += RG)
            seen = fmaf(u_s[k], (!fresh && live) ? ld_cg(st + (size_t)k * dv + col) : 0.f, seen);
    }
    part[rg * dvp + col] = seen;
    __syncthreads();
    seen = 0.f;
    for (int i = 0; i < RG; ++i) seen += part[i * dvp + col];
    float o = 0.f;
    auto update = [&](int k, float old) {
        const float n = fmaf(w_s[k], old, fmaf(k_s[k], v, -au_s[k] * seen));
        o = fmaf(r_s[k], n, o);
        if (live) st[(size_t)k * dv + col] = n;
    };
    if constexpr (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int k = rg + i * RG;
            if (k < dk) update(k, s[i]);
        }
    } else {
        for (int k = rg; k < dk; k += RG) update(k, (!fresh && live) ? ld_cg(st + (size_t)k * dv + col) : 0.f);
    }
    __syncthreads();
    part[rg * dvp + col] = o;
    __syncthreads();
    o = 0.f;
    if (rg == 0)
        for (int i = 0; i < RG; ++i) o += part[i * dvp + col];
    __syncthreads();                                        // red is reused
    const float on = 1.f / sqrtf(block_sum(rg == 0 && live ? o * o : 0.f, red) / (float)dv + p.eps);
    if (rg == 0 && live) {
        reinterpret_cast<A*>(p.y)[(size_t)b * p.H * dv + head * dv + col] = from_f<A>(o * on * p.norm[head * dv + col] * sigmoid_f(gate));
    }
}

}  // namespace tsp
