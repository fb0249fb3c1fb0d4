// Generalised delta rule: a matrix-valued recurrent state per head with per-channel decay and a removal term.
//
//   u_t = k_t / sqrt(sum(k_t^2) + 1e-6)                               unit key
//   S_t = diag(w_t) S_{t-1} - (a_t * u_t) (u_t^T S_{t-1}) + k_t v_t^T  state [dk][dv], fp32
//   o_t = S_t^T r_t
//   y_t = o_t / sqrt(mean(o_t^2) + eps) * norm * sigmoid(g_t)          per head
// with w = exp(-exp(-1/2) sigmoid(zw + w0)) and a = sigmoid(za + a_b); everything but the projections in fp32.
//
// Columns of S are independent of one another given the per-token vectors, so the prompt kernel gives each
// CTA 32 columns of one head (16 beyond 128 key channels): a few warps hold them in registers and walk the tokens
// four at a time, more warps turn the projections of the tokens ahead into the fp32 vectors they need, in shared
// memory, meanwhile.  A second kernel normalises and gates (the root mean square runs over all columns of a head).
// The decode kernel does one token of one head in one CTA, from the projections to the gated output, the state
// read and written once.
// A sequence starts with a zero state: position 0 ignores what the state buffer holds.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "lm_head.cuh"

namespace tsp {

constexpr float kDecayScale = 0.60653065971263342f;   // exp(-1/2)

typedef decoder_delta_args DeltaParams;

// ------------------------------------------------------------------------------------------ prompts
// Four tokens per step of the recurrence.  With S0 the state before them, p_j = u_j^T S_{j-1} (what the state
// holds under key j), v'_j = |k_j| v_j and W_{i..j} the product of the decays of tokens i..j,
//   p_j = c_j S0 + sum_{i<j} (A_ij v'_i - B_ij p_i)      c_j = W_{1..j-1} u_j    A_ij = u_j W_{i+1..j-1} u_i
//   o_j = q_j S0 + sum_{i<=j} (C_ij v'_i - D_ij p_i)     q_j = W_{1..j} r_j      C_ij = r_j W_{i+1..j} u_i
//   S4  = G S0 + sum_j (e_j v'_j - f_j p_j)              e_j = W_{j+1..4} u_j    f_j = a_j e_j    G = W_{1..4}
// with B and D as A and C but a_i u_i in place of u_i.  Exact, no division, decay products of four factors at
// most; one reduction over the key channels per four tokens on the critical path instead of four.  Places beyond
// the prompt's end are filled with w = 1 and zeros, which leave the state as it is.
//
// Two costs pull against each other.  A 16-byte shared load takes four cycles of its pipe however many lanes read
// the same address, so handing the vectors to the lanes costs DK / (32 * CPT) cycles per vector and state column:
// few columns per lane fill that pipe.  Many columns per lane make a warp's chain of dependent instructions per
// four tokens longer, and that chain is what the recurrence waits for.  The shapes chosen by the host were measured.
constexpr int kScanTokens = 16;                             // tokens staged at a time: one block of four per producer warp
// RL consumer lanes over the key channels, RPL state rows and CPT columns per lane, CW consumer warps, GR producer groups
template <int RL, int RPL, int CPT_, int CW, int GR>
struct ScanShape {
    static constexpr int DK = RL * RPL, CPT = CPT_;         // DK: padded key channels
    static constexpr int CPL = DK / 32;                     // channels per producer lane
    static constexpr int consumers = CW;                    // 32 / RL * CPT state columns each
    static constexpr int cols = 32 / RL * CPT * consumers;  // state columns per CTA
    static constexpr int groups = GR;                       // of four producer warps
    static constexpr int threads = 32 * (consumers + 4 * groups);
    static constexpr int sync = 32 * (consumers + 4);       // threads at a hand-over: the consumers and one group
    static constexpr int val = 17 * DK;                     // a block: c, q, e, f of four tokens and G; then v' [4][cols];
    static constexpr int sc = val + 4 * cols;               // then A, B [4][4] as [j][i], then C, D [4][4] as [j][i]
    static constexpr int block = sc + 64;
    static constexpr int buffers = CPL <= 2 ? 4 : CPL <= 4 ? 3 : 2;
    static constexpr int smem = buffers * 4 * block * 4;
};

// hardware barriers 1 .. 15 between one side that waits and one that only arrives
__device__ __forceinline__ void named_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void named_arrive(int id, int threads) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

template <typename A, int RL, int RPL, int CPT, int CW, int GR>
__global__ void __launch_bounds__(ScanShape<RL, RPL, CPT, CW, GR>::threads) delta_scan_kernel(const DeltaParams p) {
    using L = ScanShape<RL, RPL, CPT, CW, GR>;
    constexpr int DK = L::DK, CH = kScanTokens, CPL = L::CPL;
    extern __shared__ __align__(16) float scan_smem[];      // [buffers][4 blocks][block]
    griddep_launch_dependents();
    griddep_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c0 = blockIdx.x * L::cols, head = blockIdx.y, b = blockIdx.z;
    const int T = p.T, dk = p.dk, dv = p.dv;
    const int chunks = (T + CH - 1) / CH;
    const size_t row0 = (size_t)b * T;
    for (int i = tid; i < 4 * L::buffers * 64; i += L::threads) scan_smem[(i >> 6) * L::block + L::sc + (i & 63)] = 0.f;   // i > j stays zero
    __syncthreads();

    // chunk c lies in buffer c mod buffers; producer group g makes the chunks c with c mod groups = g
    const auto full = [](int c) { return 1 + c % L::buffers; };
    const auto empty = [](int c) { return 1 + L::buffers + c % L::buffers; };
    if (warp >= CW) {
        // ------------------------------------------------ producers: projections -> vectors and scalars of a block
        const int pw = (warp - CW) & 3, group = (warp - CW) >> 2;
        const A* proj = reinterpret_cast<const A*>(p.proj);
        // raw values of the next block: every address is clamped into the prompt and the loads are unconditional and
        // unconverted, so that all of them are in flight at once; what lies outside is masked when they are used
        Raw<A> rk[4][CPL], rr[4][CPL], ra[4][CPL], rv[4];
        float rw[4][CPL];
        float w0[CPL], ab[CPL];
#pragma unroll
        for (int j = 0; j < CPL; ++j) {
            const int c = lane + 32 * j;
            w0[j] = c < dk ? p.w0[head * dk + c] : 0.f;
            ab[j] = c < dk ? p.a_bias[head * dk + c] : 0.f;
        }
        // where lane l's scalar goes: A and B (j > i) first, then C and D (j >= i)
        int slot = 0;
        {
            int n = 0;
            for (int m = 0; m < 2; ++m)
                for (int j = 1; j < 4; ++j)
                    for (int i = 0; i < j; ++i, ++n)
                        if (n == lane) slot = m * 16 + j * 4 + i;
            for (int m = 2; m < 4; ++m)
                for (int j = 0; j < 4; ++j)
                    for (int i = 0; i <= j; ++i, ++n)
                        if (n == lane) slot = m * 16 + j * 4 + i;
        }
        auto load = [&](int chunk) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const size_t r = row0 + min(chunk * CH + pw * 4 + i, T - 1);
                const A* row = proj + r * p.ld;
#pragma unroll
                for (int j = 0; j < CPL; ++j) {
                    const int c = head * dk + min(lane + 32 * j, dk - 1);
                    rk[i][j].load(row + p.off_k + c);
                    rr[i][j].load(row + p.off_r + c);
                    ra[i][j].load(row + p.off_a + c);
                    rw[i][j] = __ldcg(p.zw + r * ((size_t)p.H * dk) + c);
                }
                rv[i].load(row + p.off_v + head * dv + min(c0 + min(lane, L::cols - 1), dv - 1));
            }
        };
        auto emit = [&](int chunk) {
            float* blk = scan_smem + (size_t)(chunk % L::buffers * 4 + pw) * L::block;
            float len[4], acc[32];
            bool live[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                live[i] = chunk * CH + pw * 4 + i < T;
                len[i] = 0.f;
#pragma unroll
                for (int j = 0; j < CPL; ++j) {
                    const float k = live[i] && lane + 32 * j < dk ? rk[i][j].get() : 0.f;
                    len[i] = fmaf(k, k, len[i]);
                }
            }
#pragma unroll
            for (int d = 16; d; d >>= 1)
#pragma unroll
                for (int i = 0; i < 4; ++i) len[i] += __shfl_xor_sync(0xffffffffu, len[i], d);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                len[i] = sqrtf(len[i] + 1e-6f);
                static_assert(L::cols <= 32, "one producer lane per column");
                if (lane < L::cols) blk[L::val + i * L::cols + lane] = live[i] && c0 + lane < dv ? rv[i].get() * len[i] : 0.f;
                len[i] = 1.f / len[i];
            }
#pragma unroll
            for (int n = 0; n < 32; ++n) acc[n] = 0.f;
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int c = lane + 32 * j;
                float w[4], u[4], a[4], r[4], au[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const bool in = live[i] && c < dk;
                    u[i] = in ? rk[i][j].get() * len[i] : 0.f;
                    w[i] = in ? __expf(-kDecayScale * sigmoid_fast(rw[i][j] + w0[j])) : 1.f;
                    a[i] = sigmoid_fast(ra[i][j].get() + ab[j]);
                    r[i] = in ? rr[i][j].get() : 0.f;
                    au[i] = a[i] * u[i];
                }
                const float w01 = w[0] * w[1], w23 = w[2] * w[3], w12 = w[1] * w[2];
                const float w012 = w01 * w[2], w123 = w[1] * w23, w0123 = w01 * w23;
                float* d = blk + c;
                d[0 * DK] = u[0], d[1 * DK] = w[0] * u[1], d[2 * DK] = w01 * u[2], d[3 * DK] = w012 * u[3];               // c
                d[4 * DK] = w[0] * r[0], d[5 * DK] = w01 * r[1], d[6 * DK] = w012 * r[2], d[7 * DK] = w0123 * r[3];      // q
                const float e0 = w123 * u[0], e1 = w23 * u[1], e2 = w[3] * u[2], e3 = u[3];
                d[8 * DK] = e0, d[9 * DK] = e1, d[10 * DK] = e2, d[11 * DK] = e3;
                d[12 * DK] = a[0] * e0, d[13 * DK] = a[1] * e1, d[14 * DK] = a[2] * e2, d[15 * DK] = a[3] * e3;          // f
                d[16 * DK] = w0123;
                const float x[6] = {u[1], u[2] * w[1], u[2], u[3] * w12, u[3] * w[2], u[3]};                             // (1,0) (2,0) (2,1) (3,0) (3,1) (3,2)
                const float y[10] = {r[0], r[1] * w[1], r[1], r[2] * w12, r[2] * w[2], r[2], r[3] * w123, r[3] * w23, r[3] * w[3], r[3]};
                int n = 0;
#pragma unroll
                for (int t = 1; t < 4; ++t)
#pragma unroll
                    for (int i = 0; i < t; ++i, ++n) acc[n] = fmaf(x[n], u[i], acc[n]), acc[6 + n] = fmaf(x[n], au[i], acc[6 + n]);
                n = 0;
#pragma unroll
                for (int t = 0; t < 4; ++t)
#pragma unroll
                    for (int i = 0; i <= t; ++i, ++n) acc[12 + n] = fmaf(y[n], u[i], acc[12 + n]), acc[22 + n] = fmaf(y[n], au[i], acc[22 + n]);
            }
            if (chunk + L::groups < chunks) load(chunk + L::groups);   // underneath the sums
            // 32 sums over 32 lanes: a transposing butterfly leaves sum l in lane l
#pragma unroll
            for (int d = 16; d; d >>= 1)
#pragma unroll
                for (int i = 0; i < d; ++i) {
                    const float keep = (lane & d) ? acc[i + d] : acc[i], give = (lane & d) ? acc[i] : acc[i + d];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, d);
                }
            blk[L::sc + slot] = acc[0];
        };
        if (group < chunks) load(group);
        for (int c = group; c < chunks; c += L::groups) {
            if (c >= L::buffers) named_sync(empty(c), L::sync);
            emit(c);
            named_arrive(full(c), L::sync);
        }
        return;
    }

    // -------------------------------------------------- consumers: lane = RL row groups x 32 / RL groups of CPT columns
    constexpr int PAIRS = RPL / 2, REM = 8 * CPT / RL;      // REM: sums left per lane of the 8 * CPT products
    const int ks = lane & (RL - 1), cl = warp * (32 / RL * CPT) + lane / RL * CPT, col = c0 + cl;
    float2 s[CPT][PAIRS];                                   // rows 4*RL*i + 4*ks + 0 .. 3
    float* st = p.state + ((size_t)b * p.H + head) * dk * dv;
    const bool fresh = p.pos[0] == 0;
    auto row_of = [&](int pair, int e) { return (pair >> 1) * (4 * RL) + 4 * ks + 2 * (pair & 1) + e; };
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            float f[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int k = row_of(i, e);
                f[e] = (!fresh && col + x < dv && k < dk) ? ld_cg(st + (size_t)k * dv + col + x) : 0.f;
            }
            s[x][i] = make_float2(f[0], f[1]);
        }
    auto vec = [&](const float* src, float2 (&v)[PAIRS]) {
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
            const float4 q = *reinterpret_cast<const float4*>(src + 4 * RL * i + 4 * ks);
            v[2 * i] = make_float2(q.x, q.y), v[2 * i + 1] = make_float2(q.z, q.w);
        }
    };
    const int n0 = ks * REM, jo = (n0 / CPT) & 3, x0 = n0 % CPT;   // the sums of this lane: product n0 / CPT, columns x0 ..
    for (int c = 0; c < chunks; ++c) {
        const int blocks = min(4, (T - c * CH + 3) >> 2);
        named_sync(full(c), L::sync);
#pragma unroll 1
        for (int q = 0; q < blocks; ++q) {
            const float* blk = scan_smem + (size_t)(c % L::buffers * 4 + q) * L::block;
            // products with the state before the block: c_j, then q_j, column x in place (4 * kind + j) * CPT + x
            float d[8 * CPT];
            float2 v[PAIRS];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                vec(blk + j * DK, v);
#pragma unroll
                for (int x = 0; x < CPT; ++x) {
                    float2 t = mul2(v[0], s[x][0]);
#pragma unroll
                    for (int i = 1; i < PAIRS; ++i) t = fma2(v[i], s[x][i], t);
                    d[j * CPT + x] = t.x + t.y;
                }
            }
#pragma unroll
            for (int h = RL / 2; h; h >>= 1)
#pragma unroll
                for (int i = 0; i < h * REM; ++i) {
                    const float keep = (ks & h) ? d[i + h * REM] : d[i], give = (ks & h) ? d[i] : d[i + h * REM];
                    d[i] = keep + __shfl_xor_sync(0xffffffffu, give, h);
                }
            float val[4][CPT], pj[4][CPT];
            vec(blk + 16 * DK, v);
#pragma unroll
            for (int x = 0; x < CPT; ++x)
#pragma unroll
                for (int i = 0; i < PAIRS; ++i) s[x][i] = mul2(v[i], s[x][i]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float* src = blk + L::val + j * L::cols + cl;
                if constexpr (CPT == 4) {
                    const float4 t = *reinterpret_cast<const float4*>(src);
                    val[j][0] = t.x, val[j][1] = t.y, val[j][2] = t.z, val[j][3] = t.w;
                } else {
                    const float2 t = *reinterpret_cast<const float2*>(src);
                    val[j][0] = t.x, val[j][1] = t.y;
                }
                vec(blk + (8 + j) * DK, v);
#pragma unroll
                for (int x = 0; x < CPT; ++x)
#pragma unroll
                    for (int i = 0; i < PAIRS; ++i) s[x][i] = fma2(v[i], make_float2(val[j][x], val[j][x]), s[x][i]);
            }
            const float* sc = blk + L::sc;
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int x = 0; x < CPT; ++x) {
                    const int n = j * CPT + x;
                    pj[j][x] = __shfl_sync(0xffffffffu, d[n % REM], (lane & ~(RL - 1)) | (n / REM));
                }
            // what does not depend on p first, then the triangular solve
            float bj[4][3];
#pragma unroll
            for (int j = 1; j < 4; ++j) {
                const float4 a = *reinterpret_cast<const float4*>(sc + 4 * j), bb = *reinterpret_cast<const float4*>(sc + 16 + 4 * j);
                const float aj[3] = {a.x, a.y, a.z};
                bj[j][0] = bb.x, bj[j][1] = bb.y, bj[j][2] = bb.z;
#pragma unroll
                for (int x = 0; x < CPT; ++x)
#pragma unroll
                    for (int i = 0; i < j; ++i) pj[j][x] = fmaf(aj[i], val[i][x], pj[j][x]);
            }
#pragma unroll
            for (int i = 0; i < 3; ++i)
#pragma unroll
                for (int j = i + 1; j < 4; ++j)
#pragma unroll
                    for (int x = 0; x < CPT; ++x) pj[j][x] = fmaf(-bj[j][i], pj[i][x], pj[j][x]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                vec(blk + (12 + j) * DK, v);
#pragma unroll
                for (int x = 0; x < CPT; ++x)
#pragma unroll
                    for (int i = 0; i < PAIRS; ++i) s[x][i] = fma2(v[i], make_float2(-pj[j][x], -pj[j][x]), s[x][i]);
            }
            // the upper half of the lanes holds q_j S0: the outputs of token jo
            const int t = c * CH + 4 * q + jo;
            const float4 cc = *reinterpret_cast<const float4*>(sc + 32 + 4 * jo), dd = *reinterpret_cast<const float4*>(sc + 48 + 4 * jo);
            float* out = p.o + (row0 + t) * ((size_t)p.H * dv) + (size_t)head * dv + col + x0;
#pragma unroll
            for (int i = 0; i < REM; ++i) {
                float vx[4], px[4];                          // column x0 + i
#pragma unroll
                for (int m = 0; m < 4; ++m) {
                    vx[m] = val[m][i], px[m] = pj[m][i];
#pragma unroll
                    for (int x = REM; x < CPT; x += REM)
                        if (x0 == x) vx[m] = val[m][x + i], px[m] = pj[m][x + i];
                }
                const float o = fmaf(cc.x, vx[0], fmaf(cc.y, vx[1], fmaf(cc.z, vx[2], fmaf(cc.w, vx[3], d[i]))));
                const float o2 = fmaf(dd.x, px[0], fmaf(dd.y, px[1], fmaf(dd.z, px[2], dd.w * px[3])));
                if (ks >= RL / 2 && t < T && col + x0 + i < dv) out[i] = o - o2;
            }
        }
        if (c + L::buffers < chunks) named_arrive(empty(c), L::sync);
    }
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int k = row_of(i, e);
                if (col + x < dv && k < dk) st[(size_t)k * dv + col + x] = e ? s[x][i].y : s[x][i].x;
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
