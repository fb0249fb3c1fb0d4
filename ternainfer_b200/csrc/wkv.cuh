// wkv recurrence: a matrix-valued state per head with a per-channel decay; a token reads the state as the tokens
// before it left it, and itself through a bonus u.
//
//   o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t
//   S_t = diag(w_t) S_{t-1} + k_t v_t^T                 state [dk][dv], fp32
//   y_t = o_t / sqrt(mean(o_t^2) + eps) * norm * silu(g_t)   per head
// with w = exp(-exp(zw + w0)); everything but the projections in fp32.
//
// Prompts.  The state has no reduction in its recurrence, so a sequence can be cut in time: one launch makes every
// segment's own contribution and total decay from a zero state, a small one turns these into the state at every
// segment's start, a third walks all segments at once and writes the outputs.  Inside a segment four tokens go in
// one step,
//   o_j = q_j S0 + sum_{i<j} C_ij v_i + C_jj v_j       q_j = r_j W_{<j}   C_ij = r_j W_{i<.<j} k_i   C_jj = r_j u k_j
//   S4  = G S0 + sum_i e_i v_i                          e_i = W_{>i} k_i   G = W_{0..3}
// (W: products of decays inside the block; no division, so a decay of zero is as good as any other).  All warps of a
// CTA first prepare a chunk of 16 tokens in shared memory (a block of four per warp), then hold the state's rows and
// columns in registers and walk the chunk while the next one's projections are under way.
// One token: one launch from the projections to the gated output, the state read and written once.
// A sequence starts with a zero state: position 0 ignores what the state buffer holds.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "lm_head.cuh"

namespace tsp {

typedef decoder_wkv_args WkvParams;

__device__ __forceinline__ float wkv_decay(float z) { return expf(-expf(z)); }

constexpr int kWkvChunk = 16;
// RL lanes over the key channels, RPL state rows and CPT columns per lane
template <int RL, int RPL, int CPT_>
struct WkvShape {
    static constexpr int DK = RL * RPL, CPT = CPT_, CPL = DK / 32;
    static constexpr int warp_cols = 32 / RL * CPT, cols = 4 * warp_cols;
    static constexpr int val = 9 * DK, sc = val + 4 * cols, block = sc + 16;   // q, e, G, then v, then C [j][i]
    static constexpr int smem = 2 * 4 * block * 4;
};

// OUT: walk from the segment's initial state and write outputs; otherwise only the segment's own contribution
template <typename A, int RL, int RPL, int CPT, bool OUT>
__global__ void __launch_bounds__(128) wkv_scan_kernel(const WkvParams p) {
    using L = WkvShape<RL, RPL, CPT>;
    constexpr int DK = L::DK, CPL = L::CPL, PAIRS = RPL / 2, CH = kWkvChunk;
    extern __shared__ __align__(16) float wkv_smem[];       // [2][4 blocks][block]
    griddep_launch_dependents();
    griddep_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slice = blockIdx.x, head = blockIdx.y, seg = blockIdx.z % p.n_seg, b = blockIdx.z / p.n_seg;
    if (!OUT && seg == p.n_seg - 1) return;                  // nothing follows the last segment
    const int c0 = slice * L::cols, dk = p.dk, dv = p.dv;
    const int t_lo = seg * p.seg_len, t_hi = min(p.T, t_lo + p.seg_len);
    const int chunks = (t_hi - t_lo + CH - 1) / CH;
    const size_t row0 = (size_t)b * p.T;
    const A *pr = reinterpret_cast<const A*>(p.r), *pk = reinterpret_cast<const A*>(p.k), *pv = reinterpret_cast<const A*>(p.v);

    // ---- preparation: this warp's block of four tokens, CPL channels per lane
    Raw<A> rr[4][CPL], rk[4][CPL], rv[4][(L::cols + 31) / 32];
    float rw[4][CPL], w0[CPL], u[CPL];
#pragma unroll
    for (int j = 0; j < CPL; ++j) {
        const int c = lane + 32 * j;
        w0[j] = c < dk ? p.w0[head * dk + c] : 0.f;
        u[j] = c < dk ? p.u[head * dk + c] : 0.f;
    }
    auto load = [&](int chunk) {                             // unconditional, clamped: masked when used
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const size_t r = row0 + min(t_lo + chunk * CH + warp * 4 + i, t_hi - 1);
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int c = head * dk + min(lane + 32 * j, dk - 1);
                if (OUT) rr[i][j].load(pr + r * p.ld + c);
                rk[i][j].load(pk + r * p.ld + c);
                rw[i][j] = __ldcg(p.zw + r * ((size_t)p.H * dk) + c);
            }
#pragma unroll
            for (int j = 0; j < (L::cols + 31) / 32; ++j) rv[i][j].load(pv + r * p.ld + head * dv + min(c0 + lane + 32 * j, dv - 1));
        }
    };
    auto emit = [&](int chunk) {
        float* blk = wkv_smem + (size_t)((chunk & 1) * 4 + warp) * L::block;
        bool live[4];
        float acc[16];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            live[i] = t_lo + chunk * CH + warp * 4 + i < t_hi;
#pragma unroll
            for (int j = 0; j < (L::cols + 31) / 32; ++j) {
                const int c = lane + 32 * j;
                if (c < L::cols) blk[L::val + i * L::cols + c] = live[i] && c0 + c < dv ? rv[i][j].get() : 0.f;
            }
        }
#pragma unroll
        for (int n = 0; n < 16; ++n) acc[n] = 0.f;
#pragma unroll
        for (int j = 0; j < CPL; ++j) {
            const int c = lane + 32 * j;
            float w[4], k[4], r[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const bool in = live[i] && c < dk;
                w[i] = in ? wkv_decay(rw[i][j] + w0[j]) : 1.f;
                k[i] = in ? rk[i][j].get() : 0.f;
                r[i] = OUT && in ? rr[i][j].get() : 0.f;
            }
            const float w23 = w[2] * w[3], w123 = w[1] * w23, w01 = w[0] * w[1], w12 = w[1] * w[2];
            float* d = blk + c;
            if (OUT) {
                d[0 * DK] = r[0], d[1 * DK] = r[1] * w[0], d[2 * DK] = r[2] * w01, d[3 * DK] = r[3] * (w01 * w[2]);
                acc[0] = fmaf(r[0] * u[j], k[0], acc[0]);                         // slots [j][i] of C
                acc[4] = fmaf(r[1], k[0], acc[4]), acc[5] = fmaf(r[1] * u[j], k[1], acc[5]);
                acc[8] = fmaf(r[2] * w[1], k[0], acc[8]), acc[9] = fmaf(r[2], k[1], acc[9]), acc[10] = fmaf(r[2] * u[j], k[2], acc[10]);
                acc[12] = fmaf(r[3] * w12, k[0], acc[12]), acc[13] = fmaf(r[3] * w[2], k[1], acc[13]);
                acc[14] = fmaf(r[3], k[2], acc[14]), acc[15] = fmaf(r[3] * u[j], k[3], acc[15]);
            }
            d[4 * DK] = w123 * k[0], d[5 * DK] = w23 * k[1], d[6 * DK] = w[3] * k[2], d[7 * DK] = k[3];
            d[8 * DK] = w[0] * w123;
        }
        if (chunk + 1 < chunks) load(chunk + 1);
        if (OUT) {                                           // 16 sums over 32 lanes: sum l / 2 ends in lane l
#pragma unroll
            for (int d = 16; d > 1; d >>= 1)
#pragma unroll
                for (int i = 0; i < d / 2; ++i) {
                    const float keep = (lane & d) ? acc[i + d / 2] : acc[i], give = (lane & d) ? acc[i] : acc[i + d / 2];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, d);
                }
            acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1);
            if (!(lane & 1)) blk[L::sc + (lane >> 1)] = acc[0];
        }
    };

    // ---- state: lane = RL row groups x 32 / RL groups of CPT columns
    constexpr int REM = 4 * CPT >= RL ? 4 * CPT / RL : 1;    // sums left per lane of the 4 * CPT products
    constexpr int DUP = 4 * CPT >= RL ? 1 : RL / (4 * CPT);  // lanes that share a sum
    const int ks = lane & (RL - 1), cl = warp * L::warp_cols + lane / RL * CPT, col = c0 + cl;
    auto row_of = [&](int pair, int e) { return (pair >> 1) * (4 * RL) + 4 * ks + 2 * (pair & 1) + e; };
    const size_t unit = (size_t)b * p.H + head, words = (size_t)dk * dv + dk;
    float* mine = p.part + (unit * p.n_seg + seg) * words;   // n_seg > 1: a segment's contribution, then its initial state
    const float* init = p.n_seg > 1 ? mine : p.state + unit * dk * dv;
    const bool zero = !OUT || (p.n_seg == 1 && p.pos[0] == 0);
    float2 s[CPT][PAIRS], decay[PAIRS];
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            float f[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int k = row_of(i, e);
                f[e] = (!zero && col + x < dv && k < dk) ? ld_cg(init + (size_t)k * dv + col + x) : 0.f;
            }
            s[x][i] = make_float2(f[0], f[1]);
        }
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) decay[i] = make_float2(1.f, 1.f);
    auto vec = [&](const float* src, float2 (&v)[PAIRS]) {
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
            const float4 q = *reinterpret_cast<const float4*>(src + 4 * RL * i + 4 * ks);
            v[2 * i] = make_float2(q.x, q.y), v[2 * i + 1] = make_float2(q.z, q.w);
        }
    };
    const int n0 = ks / DUP * REM, jo = n0 / CPT, x0 = n0 % CPT;   // this lane's sums: token jo, columns x0 ..
    load(0);
    emit(0);
    for (int c = 0; c < chunks; ++c) {
        __syncthreads();
        if (c + 1 < chunks) emit(c + 1);
        const int t0 = t_lo + c * CH, blocks = min(4, (t_hi - t0 + 3) >> 2);
#pragma unroll 1
        for (int q = 0; q < blocks; ++q) {
            const float* blk = wkv_smem + (size_t)((c & 1) * 4 + q) * L::block;
            float2 v[PAIRS];
            float val[4][CPT];
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int x = 0; x < CPT; x += 2) {
                    const float2 t = *reinterpret_cast<const float2*>(blk + L::val + j * L::cols + cl + x);
                    val[j][x] = t.x, val[j][x + 1] = t.y;
                }
            float d[4 * CPT];
            if (OUT) {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    vec(blk + j * DK, v);
#pragma unroll
                    for (int x = 0; x < CPT; ++x) {
                        float2 t = mul2(v[0], s[x][0]);
#pragma unroll
                        for (int i = 1; i < PAIRS; ++i) t = fma2(v[i], s[x][i], t);
                        d[j * CPT + x] = t.x + t.y;
                    }
                }
            }
            vec(blk + 8 * DK, v);
#pragma unroll
            for (int x = 0; x < CPT; ++x)
#pragma unroll
                for (int i = 0; i < PAIRS; ++i) s[x][i] = mul2(v[i], s[x][i]);
            if (!OUT)
#pragma unroll
                for (int i = 0; i < PAIRS; ++i) decay[i] = mul2(v[i], decay[i]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                vec(blk + (4 + j) * DK, v);
#pragma unroll
                for (int x = 0; x < CPT; ++x)
#pragma unroll
                    for (int i = 0; i < PAIRS; ++i) s[x][i] = fma2(v[i], make_float2(val[j][x], val[j][x]), s[x][i]);
            }
            if (OUT) {
#pragma unroll
                for (int h = RL / 2, n = 2 * CPT; h; h >>= 1, n >>= 1) {
                    if (n >= 1) {
#pragma unroll
                        for (int i = 0; i < n; ++i) {
                            const float keep = (ks & h) ? d[i + n] : d[i], give = (ks & h) ? d[i] : d[i + n];
                            d[i] = keep + __shfl_xor_sync(0xffffffffu, give, h);
                        }
                    } else {
                        d[0] += __shfl_xor_sync(0xffffffffu, d[0], h);
                    }
                }
                const float4 cc = *reinterpret_cast<const float4*>(blk + L::sc + 4 * jo);   // zeros beyond i = jo
                const int t = t0 + 4 * q + jo;
                float* out = p.o + (row0 + t) * ((size_t)p.H * dv) + (size_t)head * dv + col + x0;
                const float* vs = blk + L::val + cl + x0;
#pragma unroll
                for (int i = 0; i < REM; ++i) {
                    const float o = fmaf(cc.x, vs[i], fmaf(cc.y, vs[L::cols + i], fmaf(cc.z, vs[2 * L::cols + i], fmaf(cc.w, vs[3 * L::cols + i], d[i]))));
                    if (ks % DUP == 0 && t < t_hi && col + x0 + i < dv) out[i] = o;
                }
            }
        }
    }
    if (OUT && seg != p.n_seg - 1) return;
    float* dst = OUT ? p.state + unit * dk * dv : mine;
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int k = row_of(i, e);
                if (col + x < dv && k < dk) dst[(size_t)k * dv + col + x] = e ? s[x][i].y : s[x][i].x;
            }
    if (!OUT && slice == 0 && warp == 0 && lane < RL)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int k = row_of(i, e);
                if (k < dk) mine[(size_t)dk * dv + k] = e ? decay[i].y : decay[i].x;
            }
}

// The state at every segment's start, from the segments' contributions and total decays; element by element.
static __global__ void __launch_bounds__(256) wkv_carry_kernel(const WkvParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int n = p.dk * p.dv, e = blockIdx.x * 256 + threadIdx.x;
    if (e >= n) return;
    const size_t unit = blockIdx.y, words = (size_t)n + p.dk;
    float* part = p.part + unit * p.n_seg * words;
    float s = p.pos[0] == 0 ? 0.f : ld_cg(p.state + unit * n + e);
    constexpr int U = 8;                                     // segments in flight
    for (int i = 0; i < p.n_seg; i += U) {
        float own[U], w[U];
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const bool in = i + j < p.n_seg - 1;             // nothing follows the last segment
            const float* at = part + (size_t)(in ? i + j : 0) * words;
            own[j] = in ? ld_cg(at + e) : 0.f, w[j] = in ? ld_cg(at + n + e / p.dv) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < U; ++j)
            if (i + j < p.n_seg) {
                part[(size_t)(i + j) * words + e] = s;
                s = fmaf(w[j], s, own[j]);
            }
    }
}

// y = o / rms(o) * norm * silu(gate), one warp per row and head
template <typename A>
__global__ void __launch_bounds__(256) wkv_finish_kernel(const WkvParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long unit = (long long)blockIdx.x * 8 + warp;
    if (unit >= (long long)p.B * p.T * p.H) return;
    const long long row = unit / p.H;
    const int head = (int)(unit - row * p.H), dv = p.dv;
    const float* o = p.o + row * ((long long)p.H * dv) + head * dv;
    const A* g = reinterpret_cast<const A*>(p.g) + row * p.ld + head * dv;
    A* y = reinterpret_cast<A*>(p.y) + row * ((long long)p.H * dv) + head * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) {
        const float v = ld_cg(o + c);
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
    for (int c = lane; c < dv; c += 32) {
        const float z = ld_cg(g + c);
        y[c] = from_f<A>(ld_cg(o + c) * inv * p.norm[head * dv + c] * (z * sigmoid_f(z)));
    }
}

// The same with four neighbouring columns per lane: dv a power of two from 4 to 128, so that dv / 4 lanes share a head;
// two units of 128 columns per warp in flight.
template <typename A>
__global__ void __launch_bounds__(256) wkv_finish4_kernel(const WkvParams p) {
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
        g[i] = ld_cg4(reinterpret_cast<const A*>(p.g) + row * p.ld + col[i]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        float ss = o[i].x * o[i].x + o[i].y * o[i].y + o[i].z * o[i].z + o[i].w * o[i].w;
        for (int d = p.dv / 8; d; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
        const float inv = 1.f / sqrtf(ss / (float)p.dv + p.eps);
        const float4 w = *reinterpret_cast<const float4*>(p.norm + col[i]);
        if (at[i] < total)
            st4(reinterpret_cast<A*>(p.y) + at[i],
                make_float4(o[i].x * inv * w.x * (g[i].x * sigmoid_f(g[i].x)), o[i].y * inv * w.y * (g[i].y * sigmoid_f(g[i].y)),
                            o[i].z * inv * w.z * (g[i].z * sigmoid_f(g[i].z)), o[i].w * inv * w.w * (g[i].w * sigmoid_f(g[i].w))));
    }
}

// ------------------------------------------------------------------------------------------ one token
constexpr int kWkvThreads = 512;

// NR: state rows a thread keeps in registers (dk <= NR * row groups); 0: it walks them in memory.
// WIDE: rank a multiple of 8 and dk * rank / 8 words of 16 bytes of w2 (bf16) are at most WIDE per thread: they are
// requested before the wait for the projections.
template <typename A, int NR, int WIDE>
__global__ void __launch_bounds__(kWkvThreads) wkv_step_kernel(const WkvParams p, const int dvp) {
    extern __shared__ __align__(16) float wkv_step_smem[];
    __shared__ float red[32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = kWkvThreads / 32;
    const int dk = p.dk, dv = p.dv, rank = p.rank;
    const int head = blockIdx.x, b = blockIdx.y;
    const int RG = kWkvThreads / dvp;                        // row groups; dvp a power of two >= dv
    float* w_s = wkv_step_smem;
    float *k_s = w_s + dk, *r_s = k_s + dk, *uk_s = r_s + dk, *t1_s = uk_s + dk;
    float* part = t1_s + (rank + 3) / 4 * 4;                 // [RG][dvp], and the decay's partial sums [dk][rank / 8]
    griddep_launch_dependents();
    const A* w2 = reinterpret_cast<const A*>(p.w2) + (size_t)head * dk * rank;
    const int per = rank / 8, words = dk * per;              // (WIDE) a word = 8 ranks of one channel
    uint4 wv[WIDE > 0 ? WIDE : 1];
    if constexpr (WIDE > 0) {
#pragma unroll
        for (int i = 0; i < WIDE; ++i) {
            const int e = tid + i * kWkvThreads;
            wv[i] = e < words ? ldg_stream_128(w2 + (size_t)e * 8) : make_uint4(0, 0, 0, 0);
        }
    }
    griddep_wait();
    const size_t at = (size_t)b * p.ld + (size_t)head * dk, at_v = (size_t)b * p.ld + (size_t)head * dv;
    const A *pr = reinterpret_cast<const A*>(p.r) + at, *pk = reinterpret_cast<const A*>(p.k) + at;
    const A *pv = reinterpret_cast<const A*>(p.v) + at_v, *pg = reinterpret_cast<const A*>(p.g) + at_v;
    const A* t1 = reinterpret_cast<const A*>(p.t1) + (size_t)b * p.ld_t;
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
    const float v = live ? ld_cg(pv + col) : 0.f, gate = live ? ld_cg(pg + col) : 0.f;
    for (int c = tid; c < dk; c += kWkvThreads) {
        const float k = ld_cg(pk + c);
        k_s[c] = k, r_s[c] = ld_cg(pr + c);
        uk_s[c] = p.u[head * dk + c] * k;
    }
    for (int c = tid; c < rank; c += kWkvThreads) t1_s[c] = tanhf(ld_cg(t1 + c));
    __syncthreads();
    if constexpr (WIDE > 0) {
#pragma unroll
        for (int i = 0; i < WIDE; ++i) {
            const int e = tid + i * kWkvThreads;
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
    for (int c = WIDE > 0 ? tid : warp; c < dk; c += WIDE > 0 ? kWkvThreads : nw) {
        float z = 0.f;
        if constexpr (WIDE > 0) {
            for (int j = 0; j < per; ++j) z += part[c * per + j];
        } else {                                             // one warp per channel, lanes over the rank
            for (int j = lane; j < rank; j += 32) z = fmaf(to_f(w2[(size_t)c * rank + j]), t1_s[j], z);
            z = warp_sum(z);
        }
        if (WIDE > 0 || lane == 0) w_s[c] = wkv_decay(z + p.w0[head * dk + c]);
    }
    if (fresh) {
#pragma unroll
        for (int i = 0; i < (NR > 0 ? NR : 1); ++i) s[i] = 0.f;
    }
    __syncthreads();
    float o = 0.f;
    auto update = [&](int k, float old) {
        o = fmaf(r_s[k], fmaf(uk_s[k], v, old), o);
        if (live) st[(size_t)k * dv + col] = fmaf(w_s[k], old, k_s[k] * v);
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
    part[rg * dvp + col] = o;                                // (the decay's partial sums have been read)
    __syncthreads();
    o = 0.f;
    if (rg == 0)
        for (int i = 0; i < RG; ++i) o += part[i * dvp + col];
    const float on = 1.f / sqrtf(block_sum(rg == 0 && live ? o * o : 0.f, red) / (float)dv + p.eps);
    if (rg == 0 && live)
        reinterpret_cast<A*>(p.y)[(size_t)b * p.H * dv + head * dv + col] = from_f<A>(o * on * p.norm[head * dv + col] * (gate * sigmoid_f(gate)));
}

}  // namespace tsp
