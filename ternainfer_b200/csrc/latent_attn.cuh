// Attention over a shared latent: what a token leaves in the cache is one normalised latent c [R] and one rotated key
// part [rot] for all heads; a head's key is (W_uk c, rotated part), its value W_uv c.
//
//   score = (q_u . W_uk c + q_r . k_r) * scale = ((W_uk^T q_u) . c + q_r . k_r) * scale
//   weight = exp(score) / (sum over the visible keys of exp(score) + exp(sink_h))
//
// Cache: [B][slots][ld] per layer, position p in slot p; the latent in the first R columns, zeros up to r_at (a
// multiple of 8), the rotated part from there, zeros up to ld.  Layers that share a latent read the same tensor.
//
// Two forms.  Prompts expand keys and values per head (latent_attn_tc.cuh).  Few tokens absorb W_uk into the query
// and W_uv into the output and read the cache as it is: all heads of a token share one stream of keys, which are
// their values too.  The kernels here: norms, rotation and cache append; the absorbed form for any type and size;
// the absorbed form for few bf16 tokens on mma.sync, the keys split over the chip; the join of the parts with the
// product with W_uv.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "decoder_status.cuh"
#include "lm_head.cuh"
#include "tcgen05_sm100.cuh"

namespace tsp {

constexpr float kLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------ norms, rotation, append
typedef decoder_latent_prep_args LatentPrepParams;

// One CTA per row: the query latent normalised to cq, the key latent normalised and the shared key part rotated into
// the cache.  trig [positions][dims] holds cosine and sine of every pair.
template <typename A>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepParams p) {
    extern __shared__ __align__(16) float latent_prep_smem[];    // the row's query latent, key latent, key part
    __shared__ float2 red[8];
    griddep_launch_dependents();
    griddep_wait();
    const int row = blockIdx.x, b = row / p.T, t = row - b * p.T, tid = threadIdx.x;
    const A* z = reinterpret_cast<const A*>(p.z) + (size_t)row * p.ld_z;
    float *q_s = latent_prep_smem, *k_s = q_s + p.q_rank;
    const long long pos = p.pos[0] + t;
    const bool append = p.cache && pos < p.slots;
    float2 ss = make_float2(0.f, 0.f);
    for (int c = tid; c < p.q_rank; c += 256) {
        const float v = ld_cg(z + p.off_q + c);
        q_s[c] = v;
        ss.x = fmaf(v, v, ss.x);
    }
    if (append)
        for (int c = tid; c < p.R + p.rot; c += 256) {
            const float v = ld_cg(z + p.off_kv + c);
            k_s[c] = v;
            if (c < p.R) ss.y = fmaf(v, v, ss.y);
        }
    ss = make_float2(warp_sum(ss.x), warp_sum(ss.y));
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    ss = red[0];
#pragma unroll
    for (int i = 1; i < 8; ++i) ss.x += red[i].x, ss.y += red[i].y;
    const float iq = 1.f / sqrtf(ss.x / (float)p.q_rank + p.eps);
    A* cq = reinterpret_cast<A*>(p.cq) + (size_t)row * p.q_rank;
    for (int c = tid; c < p.q_rank; c += 256) cq[c] = from_f<A>(q_s[c] * iq * p.q_norm[c]);
    if (!append) return;
    const float ik = 1.f / sqrtf(ss.y / (float)p.R + p.eps);
    A* k = reinterpret_cast<A*>(p.cache) + ((size_t)b * p.slots + pos) * p.ld;
    for (int c = tid; c < p.R; c += 256) k[c] = from_f<A>(k_s[c] * ik * p.kv_norm[c]);
    const float* trig = p.trig + (size_t)pos * p.dims;
    for (int c = tid; c < p.rot; c += 256) {
        float v = k_s[p.R + c];
        if (c < p.dims) {
            const float o = k_s[p.R + (c ^ 1)], cs = trig[c & ~1], sn = trig[c | 1];
            v = (c & 1) ? v * cs + o * sn : v * cs - o * sn;
        }
        k[p.r_at + c] = from_f<A>(v);
    }
}

// The rotated part of every head's query, from one layout to another (or in place).
typedef decoder_rotate_args RotateParams;
template <typename A>
__global__ void __launch_bounds__(256) rotate_kernel(const RotateParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int pairs = (p.rot + 1) / 2;
    const long long total = (long long)p.B * p.T * p.H * pairs, stride = (long long)gridDim.x * blockDim.x;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
        const int c = (int)(i % pairs) * 2, h = (int)(i / pairs % p.H);
        const long long row = i / pairs / p.H, pos = p.pos[0] + row % p.T;
        const A* s = reinterpret_cast<const A*>(p.src) + row * p.ld_src + (long long)h * p.head_src + p.off_src + c;
        A* d = reinterpret_cast<A*>(p.dst) + row * p.ld_dst + (long long)h * p.head_dst + p.off_dst + c;
        const float u = ld_cg(s), v = c + 1 < p.rot ? ld_cg(s + 1) : 0.f;
        float x = u, y = v;
        if (c < p.dims) {
            const float cs = p.trig[(size_t)pos * p.dims + c], sn = p.trig[(size_t)pos * p.dims + c + 1];
            x = u * cs - v * sn, y = v * cs + u * sn;
        }
        d[0] = from_f<A>(x);
        if (c + 1 < p.rot) d[1] = from_f<A>(y);
    }
}

// ------------------------------------------------------------------------------------------ any type, any size
typedef decoder_latent_attn_args LatentAttnParams;

// One CTA per row and head, 128 keys at a time, running maximum.  qa [rows][H][ld]: absorbed queries in the cache's
// layout; out: weighted latents [rows][H][R].
template <typename A>
__global__ void __launch_bounds__(128) latent_attn_plain_kernel(const LatentAttnParams p) {
    extern __shared__ __align__(16) float latent_plain_smem[];   // q [ld], o [R]
    __shared__ float w_s[128], red[4];
    griddep_launch_dependents();
    griddep_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.x, h = blockIdx.y;
    const int b = row / p.T, t = row - b * p.T, ld = p.ld, R = p.R;
    const long long n = min(p.pos[0] + t + 1, (long long)p.slots);
    const A* q = reinterpret_cast<const A*>(p.qa) + ((size_t)row * p.H + h) * ld;
    const A* cache = reinterpret_cast<const A*>(p.cache) + (size_t)b * p.slots * ld;
    float *q_s = latent_plain_smem, *o_s = q_s + ld;
    for (int c = tid; c < ld; c += 128) q_s[c] = ld_cg(q + c) * p.scale * kLog2e;
    for (int c = tid; c < R; c += 128) o_s[c] = 0.f;
    float m = p.sink[h] * kLog2e, l = 1.f;
    __syncthreads();
    for (long long j0 = 0; j0 < n; j0 += 128) {
        const long long j = j0 + tid;
        float s = -INFINITY;
        if (j < n) {
            const A* k = cache + (size_t)j * ld;
            s = 0.f;
            for (int c = 0; c < ld; c += 4) {                // ld is a multiple of 8
                const float4 x = ld_cg4(k + c), y = *reinterpret_cast<const float4*>(q_s + c);
                s = fmaf(x.x, y.x, s), s = fmaf(x.y, y.y, s), s = fmaf(x.z, y.z, s), s = fmaf(x.w, y.w, s);
            }
        }
        float mx = s;
#pragma unroll
        for (int d = 16; d; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
        if (lane == 0) red[warp] = mx;
        __syncthreads();
        const float mn = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), m);
        const float f = exp2f(m - mn), w = exp2f(s - mn);
        w_s[tid] = w;
        __syncthreads();
        float sum = 0.f;
        for (int e = lane; e < 128; e += 32) sum += w_s[e];
        l = fmaf(l, f, warp_sum(sum)), m = mn;
        const int cnt = (int)min((long long)128, n - j0);
        for (int c = tid; c < R; c += 128) {
            float o = o_s[c] * f;
            for (int e = 0; e < cnt; ++e) o = fmaf(w_s[e], ld_cg(cache + (size_t)(j0 + e) * ld + c), o);
            o_s[c] = o;
        }
        __syncthreads();
    }
    A* out = reinterpret_cast<A*>(p.out) + ((size_t)row * p.H + h) * R;
    for (int c = tid; c < R; c += 128) out[c] = from_f<A>(o_s[c] / l);
}

// ------------------------------------------------------------------------------------------ few bf16 tokens
// qa[row][h][r] = sum_d q[row][h][d] W_uk^T[h][r][d] for up to eight rows, and the rotated part behind it: CTAs
// x = 128 latents of one head (y), 16 per warp as rows of an MMA whose columns are the rows of q; the last x rotates.
// The weights are requested before the wait.
typedef decoder_absorb_args AbsorbParams;

static __global__ void __launch_bounds__(256) absorb_kernel(const AbsorbParams p) {
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, dim = p.dim, M = p.B * p.T;
    const int dq = dim + p.rot, g = lane >> 2, qd = lane & 3;
    const bf16* q = reinterpret_cast<const bf16*>(p.q);
    bf16* qa = reinterpret_cast<bf16*>(p.qa);
    if (blockIdx.x == gridDim.x - 1) {                       // rotation, and zeros where the layout has gaps
        griddep_wait();
        for (int i = tid; i < M * (p.ld - p.R); i += 256) {
            const int row = i / (p.ld - p.R), c = p.R + i % (p.ld - p.R), e = c - p.r_at;
            float v = 0.f;
            if (e >= 0 && e < p.rot) {
                const bf16* s = q + (size_t)row * p.H * dq + h * dq + dim;
                v = ld_cg(s + e);
                if (e < p.dims) {
                    const float* trig = p.trig + (size_t)(p.pos[0] + row % p.T) * p.dims;
                    const float o = ld_cg(s + (e ^ 1)), cs = trig[e & ~1], sn = trig[e | 1];
                    v = (e & 1) ? v * cs + o * sn : v * cs - o * sn;
                }
            }
            qa[((size_t)row * p.H + h) * p.ld + c] = from_f<bf16>(v);
        }
        return;
    }
    constexpr int PRE = 4;                                   // k-steps of 32 in flight
    const int r0 = blockIdx.x * 128 + warp * 16;
    const bool ok0 = r0 + g < p.R, ok1 = r0 + g + 8 < p.R;
    const bf16* w = reinterpret_cast<const bf16*>(p.w_uk_t) + (size_t)h * p.R * dim + qd * 8;
    const bf16 *w0 = w + (size_t)(ok0 ? r0 + g : 0) * dim, *w1 = w + (size_t)(ok1 ? r0 + g + 8 : 0) * dim;
    const bf16* x = q + (size_t)(g < M ? g : 0) * p.H * dq + h * dq + qd * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    uint4 a[PRE], b[PRE], xv[PRE];
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int d = 0; d < dim; d += 32 * PRE) {
#pragma unroll
        for (int u = 0; u < PRE; ++u) {
            const bool in = d + 32 * u + qd * 8 < dim;
            a[u] = in && ok0 ? ldg_stream_128(w0 + d + 32 * u) : zero;
            b[u] = in && ok1 ? ldg_stream_128(w1 + d + 32 * u) : zero;
        }
        if (d == 0) griddep_wait();
#pragma unroll
        for (int u = 0; u < PRE; ++u) xv[u] = g < M && d + 32 * u + qd * 8 < dim ? ld_cg_128(x + d + 32 * u) : zero;
#pragma unroll
        for (int u = 0; u < PRE; ++u) {
            mma_bf16_16x8x16(acc, a[u].x, b[u].x, a[u].y, b[u].y, xv[u].x, xv[u].y);
            mma_bf16_16x8x16(acc, a[u].z, b[u].z, a[u].w, b[u].w, xv[u].z, xv[u].w);
        }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        const int row = 2 * qd + (c & 1), r = r0 + g + (c >> 1) * 8;
        if (row < M && r < p.R) qa[((size_t)row * p.H + h) * p.ld + r] = from_f<bf16>(acc[c]);
    }
}

__device__ __forceinline__ void ldmatrix4(uint32_t addr, uint32_t (&v)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t addr, uint32_t (&v)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(addr));
}
__device__ __forceinline__ float ld_cluster(uint32_t addr, int rank) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(map_to_rank(addr, rank)));
    return v;
}
__device__ __forceinline__ float4 ld_cluster4(uint32_t addr, int rank) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(map_to_rank(addr, rank)));
    return v;
}

// Up to 32 heads of one row against the keys, which are cut into one range per CTA of the grid's x.  Queries and keys, 64
// at a time, arrive by TMA in boxes of 64 columns with 128-byte swizzle, the next tile under the work on this one.  Scores: a
// warp takes 16 keys and half of the columns.  Weighted sum: a warp takes an eighth of the latents.  The CTAs of a
// cluster add their sums up in distributed shared memory, a share of the columns each, and leave unnormalised sums,
// maximum (base 2) and sum of weights of the cluster's ranges.
struct LatentStepSmem {
    static constexpr int bar = 0, abort_flag = 16, st = 128, data = 1024;    // st: maxima, sums, factors [32] each
    int boxes, tile, stages, q, s, p, total;                 // bytes, from a 1024-byte boundary
    __host__ __device__ LatentStepSmem(int ld, int mt, int limit) {
        boxes = (ld + 63) / 64, tile = boxes * 64 * 128;
        const int rest = mt * 16 * (boxes * 128 + 2 * 68 * 4 + 72 * 2);
        stages = 1024 + data + 2 * tile + rest <= limit ? 2 : 1;
        q = data + stages * tile, s = q + mt * 16 * boxes * 128, p = s + 2 * mt * 16 * 68 * 4;
        total = 1024 + data + stages * tile + rest;
    }
};

template <int NT, int MT>   // 16-latent tiles per warp: R <= 128 * NT; 16-head tiles
__global__ void __launch_bounds__(256)
    latent_step_kernel(const LatentAttnParams p, const int smem_limit, const __grid_constant__ CUtensorMap map_q,
                       const __grid_constant__ CUtensorMap map_cache) {
    extern __shared__ __align__(128) uint8_t latent_step_smem[];
    const LatentStepSmem L(p.ld, MT, smem_limit);
    const uint32_t dyn = smem_u32(latent_step_smem), base = (dyn + 1023u) & ~1023u;
    uint8_t* mem = latent_step_smem + (base - dyn);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(mem + L.abort_flag);
    float *s_s = reinterpret_cast<float*>(mem + L.s), *o_s = reinterpret_cast<float*>(mem + L.data);
    bf16* p_s = reinterpret_cast<bf16*>(mem + L.p);
    float *m_s = reinterpret_cast<float*>(mem + L.st), *l_s = m_s + 32, *f_s = m_s + 64;
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int split = blockIdx.x, splits = gridDim.x, C = p.cluster, rank = split % C;
    const int h0 = blockIdx.y * 16 * MT, row = blockIdx.z, b = row / p.T, t = row - b * p.T;
    const int ld = p.ld, ksteps = (ld + 15) / 16, hn = min(16 * MT, p.H - h0);
    if (tid == 0) {
        mbar_init(base + L.bar, 1), mbar_init(base + L.bar + 8, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (tid < 32) m_s[tid] = -INFINITY, l_s[tid] = 0.f;
    __syncthreads();
    griddep_wait();
    const int n = (int)min(p.pos[0] + t + 1, (long long)p.slots);
    const int lo = (int)((long long)n * split / splits), hi = (int)((long long)n * (split + 1) / splits);
    const int tiles = (hi - lo + 63) / 64;
    auto fetch = [&](int it) {                               // one thread; whole 32-row groups, rows beyond hi are masked
        const int buf = it % L.stages, groups = min(2, (hi - lo - 64 * it + 31) / 32);
        const uint32_t bar = base + L.bar + 8 * buf;
        mbar_arrive_expect_tx(bar, groups * L.boxes * 4096 + (it == 0 ? MT * 16 * 128 * L.boxes : 0));
        if (it == 0)
            for (int i = 0; i < L.boxes; ++i) tma_load_2d(base + L.q + i * MT * 2048, &map_q, 64 * i, row * p.H + h0, bar);
        for (int i = 0; i < L.boxes; ++i)
            for (int r = 0; r < groups; ++r)
                tma_load_2d(base + L.data + buf * L.tile + i * 8192 + r * 4096, &map_cache, 64 * i, b * p.slots + lo + 64 * it + 32 * r, bar);
    };
    if (tid == 0)
        for (int it = 0; it < min(tiles, L.stages); ++it) fetch(it);
    float acc[NT][MT][2][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int c = 0; c < 4; ++c) acc[i][m][j][c] = 0.f;
    const int g = lane >> 2, qd = lane & 3;
    const int key0 = (warp & 3) * 16, half = warp >> 2, k0 = half * ((ksteps + 1) / 2), k1 = half ? ksteps : (ksteps + 1) / 2;
    bool ok = true;
    for (int it = 0; it < tiles; ++it) {
        const int j0 = lo + it * 64, buf = it % L.stages;
        const uint32_t kv = base + L.data + buf * L.tile;
        ok = wait_or_abort(base + L.bar + 8 * buf, (it / L.stages) & 1, abort_flag);
        ok = __syncthreads_and(ok);
        if (!ok) break;
        {   // scores of 16 keys over half of the columns
            float d[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int c = 0; c < 4; ++c) d[m][j][c] = 0.f;
            const int kr = key0 + (lane >> 4) * 8 + (lane & 7);
            const uint32_t qa = base + L.q + (lane & 15) * 128, ka = kv + kr * 128;
#pragma unroll 4
            for (int k = k0; k < k1; ++k) {
                uint32_t kb[4], a[4];
                const int piece = 2 * k + ((lane >> 3) & 1), qp = 2 * k + (lane >> 4);   // eight columns
                ldmatrix4(ka + (piece >> 3) * 8192 + (((piece & 7) ^ (kr & 7)) << 4), kb);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    ldmatrix4(qa + (qp >> 3) * MT * 2048 + m * 2048 + (((qp & 7) ^ (lane & 7)) << 4), a);
                    mma_bf16_16x8x16(d[m][0], a[0], a[1], a[2], a[3], kb[0], kb[1]);
                    mma_bf16_16x8x16(d[m][1], a[0], a[1], a[2], a[3], kb[2], kb[3]);
                }
            }
            const float f = p.scale * kLog2e;
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int c = 0; c < 4; c += 2) {
                        const int key = key0 + j * 8 + 2 * qd, head = m * 16 + g + (c >> 1) * 8;
                        *reinterpret_cast<float2*>(s_s + (half * 16 * MT + head) * 68 + key) = make_float2(d[m][j][c] * f, d[m][j][c + 1] * f);
                    }
        }
        __syncthreads();
        {                                                    // softmax: 16 / MT threads per head, pairs of keys
            constexpr int TPH = 16 / MT, N = 32 / TPH;
            const int head = tid / TPH, sub = tid % TPH;
            const float *sa = s_s + head * 68 + 2 * sub, *sb = sa + 16 * MT * 68;
            float2 w[N];
            const float mo = m_s[head];
            float mn = mo, sum = 0.f;
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const float2 x = *reinterpret_cast<const float2*>(sa + 2 * TPH * i), y = *reinterpret_cast<const float2*>(sb + 2 * TPH * i);
                const int key = j0 + 2 * (sub + TPH * i);
                w[i] = make_float2(key < hi ? x.x + y.x : -INFINITY, key + 1 < hi ? x.y + y.y : -INFINITY);
                mn = fmaxf(mn, fmaxf(w[i].x, w[i].y));       // finite in the end: the first key of a tile always counts
            }
#pragma unroll
            for (int d = TPH / 2; d; d >>= 1) mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, d));
#pragma unroll
            for (int i = 0; i < N; ++i) {
                w[i] = make_float2(exp2f(w[i].x - mn), exp2f(w[i].y - mn));
                sum += w[i].x + w[i].y;
                *reinterpret_cast<uint32_t*>(p_s + head * 72 + 2 * (sub + TPH * i)) = pack_bf16(w[i].x, w[i].y);
            }
#pragma unroll
            for (int d = TPH / 2; d; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
            if (sub == 0) {
                const float f = exp2f(mo - mn);
                f_s[head] = f, m_s[head] = mn, l_s[head] = fmaf(l_s[head], f, sum);
            }
        }
        __syncthreads();
        if (it > 0)
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const float fa = f_s[m * 16 + g], fb = f_s[m * 16 + g + 8];
#pragma unroll
                for (int i = 0; i < NT; ++i)
#pragma unroll
                    for (int j = 0; j < 2; ++j)
                        acc[i][m][j][0] *= fa, acc[i][m][j][1] *= fa, acc[i][m][j][2] *= fb, acc[i][m][j][3] *= fb;
            }
        const int live = min(4, (hi - j0 + 15) / 16);        // 16-key groups with weights other than zero
#pragma unroll 1
        for (int kk = 0; kk < live; ++kk) {
            uint32_t a[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) ldmatrix4(base + L.p + (m * 16 + (lane & 15)) * 144 + kk * 32 + (lane >> 4) * 16, a[m]);
            const int kr = kk * 16 + (lane & 15);
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c = (warp * NT + i) * 16;
                if (c < p.R) {                               // uniform over the warp
                    uint32_t v[4];
                    const int piece = c / 8 + (lane >> 4);
                    ldmatrix4_trans(kv + (piece >> 3) * 8192 + kr * 128 + (((piece & 7) ^ (kr & 7)) << 4), v);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_bf16_16x8x16(acc[i][m][0], a[m][0], a[m][1], a[m][2], a[m][3], v[0], v[1]);
                        mma_bf16_16x8x16(acc[i][m][1], a[m][0], a[m][1], a[m][2], a[m][3], v[2], v[3]);
                    }
                }
            }
        }
        __syncthreads();                                     // the buffer, the scores and the weights are used again
        if (tid == 0 && it + L.stages < tiles) fetch(it + L.stages);
    }
    const int ro = p.R + 8;                                  // row of o_s: eight rows apart in different banks
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int r = (warp * NT + i) * 16 + j * 8 + 2 * qd;   // R is a multiple of 8
                if (r < p.R) {
                    float* o = o_s + (m * 16 + g) * ro + r;
                    *reinterpret_cast<float2*>(o) = make_float2(acc[i][m][j][0], acc[i][m][j][1]);
                    *reinterpret_cast<float2*>(o + 8 * ro) = make_float2(acc[i][m][j][2], acc[i][m][j][3]);
                }
            }
    cluster_arrive();
    cluster_wait();
    const int part_at = split / C, parts = splits / C;
    for (int i = rank * 256 + tid; i < hn * (p.R / 4); i += C * 256) {
        const int head = i / (p.R / 4), c = (i - head * (p.R / 4)) * 4;
        const uint32_t at = base + L.data + 4 * (head * ro + c), m_at = base + L.st + 4 * head;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f), v[8];
        float m[8], l[8], top = -INFINITY, sum = 0.f;
#pragma unroll
        for (int r = 0; r < 8; ++r)
            if (r < C) m[r] = ld_cluster(m_at, r), l[r] = ld_cluster(m_at + 128, r), v[r] = ld_cluster4(at, r);
#pragma unroll
        for (int r = 0; r < 8; ++r)
            if (r < C) top = fmaxf(top, m[r]);
#pragma unroll
        for (int r = 0; r < 8; ++r)
            if (r < C) {
                const float w = m[r] == -INFINITY ? 0.f : exp2f(m[r] - top);
                o.x = fmaf(w, v[r].x, o.x), o.y = fmaf(w, v[r].y, o.y), o.z = fmaf(w, v[r].z, o.z), o.w = fmaf(w, v[r].w, o.w);
                sum = fmaf(w, l[r], sum);
            }
        const size_t dst = ((size_t)row * p.H + h0 + head) * parts + part_at;
        st4(p.part + dst * p.R + c, o);
        if (c == 0) p.ml[2 * dst] = top, p.ml[2 * dst + 1] = sum;
    }
    cluster_arrive();                                        // nobody leaves while another CTA still reads
    cluster_wait();
    if (*abort_flag && tid == 0) atomicExch(&g_decoder_status, DECODER_WAIT_TIMEOUT);
}

// Joins the ranges' parts, adds the sink to the denominator and multiplies with W_uv: y[row][h][v].  CTAs x = 32 values
// of one head (y) for RB rows (z); the weights are requested before the wait.
template <int RW, int RB>   // words of 16 bytes per lane and row of W_uv: R <= 256 * RW, a multiple of 8
__global__ void __launch_bounds__(256) latent_join_kernel(const LatentAttnParams p) {
    extern __shared__ __align__(16) float c_s[];             // the latents [RB][R]
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, row0 = blockIdx.z * RB, R = p.R, splits = p.splits, M = p.B * p.T;
    const bf16* w = reinterpret_cast<const bf16*>(p.w_uv) + (size_t)h * p.vdim * R;
    uint4 wv[4][RW];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < RW; ++j) {
            const int v = blockIdx.x * 32 + warp * 4 + i, c = (lane + 32 * j) * 8;
            wv[i][j] = v < p.vdim && c < R ? ldg_stream_128(w + (size_t)v * R + c) : make_uint4(0, 0, 0, 0);
        }
    griddep_wait();
    constexpr int PRE = RB == 1 ? 8 : 4;                     // parts in flight, with their maxima and sums
    const float sink = p.sink[h] * kLog2e;
    float o[RB][RW], top[RB], l[RB];
#pragma unroll
    for (int b = 0; b < RB; ++b) {
        top[b] = sink, l[b] = 1.f;
#pragma unroll
        for (int j = 0; j < RW; ++j) o[b][j] = 0.f;
    }
    for (int s0 = 0; s0 < splits; s0 += PRE) {
        float2 st[RB][PRE];
        float v[RB][RW][PRE];
#pragma unroll
        for (int b = 0; b < RB; ++b) {
            const size_t at = ((size_t)min(row0 + b, M - 1) * p.H + h) * splits;
#pragma unroll
            for (int s = 0; s < PRE; ++s) {
                const bool in = s0 + s < splits;
                st[b][s] = in ? __ldcg(reinterpret_cast<const float2*>(p.ml) + at + s0 + s) : make_float2(-INFINITY, 0.f);
#pragma unroll
                for (int j = 0; j < RW; ++j) v[b][j][s] = in && tid + 256 * j < R ? __ldcg(p.part + (at + s0 + s) * R + tid + 256 * j) : 0.f;
            }
        }
#pragma unroll
        for (int b = 0; b < RB; ++b) {
            float m = top[b];
#pragma unroll
            for (int s = 0; s < PRE; ++s) m = fmaxf(m, st[b][s].x);
            const float f = exp2f(top[b] - m);
            top[b] = m, l[b] *= f;
#pragma unroll
            for (int j = 0; j < RW; ++j) o[b][j] *= f;
#pragma unroll
            for (int s = 0; s < PRE; ++s) {
                const float w = exp2f(st[b][s].x - m);       // 0 for a range without keys
                l[b] = fmaf(w, st[b][s].y, l[b]);
#pragma unroll
                for (int j = 0; j < RW; ++j) o[b][j] = fmaf(w, v[b][j][s], o[b][j]);
            }
        }
    }
#pragma unroll
    for (int b = 0; b < RB; ++b)
#pragma unroll
        for (int j = 0; j < RW; ++j)
            if (tid + 256 * j < R) c_s[b * R + tid + 256 * j] = o[b][j] / l[b];
    __syncthreads();
#pragma unroll
    for (int b = 0; b < RB; ++b) {
        if (row0 + b >= M) break;
        float d[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < RW; ++j) {
            const int c = (lane + 32 * j) * 8;
            if (c < R) {
                const float4 x = *reinterpret_cast<const float4*>(c_s + b * R + c), y = *reinterpret_cast<const float4*>(c_s + b * R + c + 4);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    float f[8];
                    unpack8(wv[i][j], f);
                    d[i] = fmaf(f[0], x.x, fmaf(f[1], x.y, fmaf(f[2], x.z, fmaf(f[3], x.w, d[i]))));
                    d[i] = fmaf(f[4], y.x, fmaf(f[5], y.y, fmaf(f[6], y.z, fmaf(f[7], y.w, d[i]))));
                }
            }
        }
        // four sums over 32 lanes: sum i ends in the lanes of group i of eight
#pragma unroll
        for (int n = 2, s = 16; n; n >>= 1, s >>= 1)
#pragma unroll
            for (int i = 0; i < n; ++i) {
                const float keep = (lane & s) ? d[i + n] : d[i], give = (lane & s) ? d[i] : d[i + n];
                d[i] = keep + __shfl_xor_sync(0xffffffffu, give, s);
            }
#pragma unroll
        for (int s = 4; s; s >>= 1) d[0] += __shfl_xor_sync(0xffffffffu, d[0], s);
        const int v = blockIdx.x * 32 + warp * 4 + lane / 8;
        if (lane % 8 == 0 && v < p.vdim) reinterpret_cast<bf16*>(p.y)[((size_t)(row0 + b) * p.H + h) * p.vdim + v] = from_f<bf16>(d[0]);
    }
}

}  // namespace tsp
