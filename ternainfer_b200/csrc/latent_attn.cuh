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
// the absorbed form for up to eight bf16 tokens on mma.sync, the keys split over the chip; the join of the parts
// with the product with W_uv.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "lm_head.cuh"

namespace tsp {

constexpr float kLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------ norms, rotation, append
typedef decoder_latent_prep_args LatentPrepParams;

// One CTA per row: the query latent normalised to cq, the key latent normalised and the shared key part rotated into
// the cache.  trig [positions][dims] holds cosine and sine of every pair.
template <typename A>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepParams p) {
    __shared__ float red[32], red2[32];
    griddep_launch_dependents();
    griddep_wait();
    const int row = blockIdx.x, b = row / p.T, t = row - b * p.T, tid = threadIdx.x;
    const A* z = reinterpret_cast<const A*>(p.z) + (size_t)row * p.ld_z;
    const A *zq = z + p.off_q, *zk = z + p.off_kv;
    const long long pos = p.pos[0] + t;
    float sq = 0.f, sk = 0.f;
    for (int c = tid; c < p.q_rank; c += 256) {
        const float v = ld_cg(zq + c);
        sq = fmaf(v, v, sq);
    }
    if (p.cache)
        for (int c = tid; c < p.R; c += 256) {
            const float v = ld_cg(zk + c);
            sk = fmaf(v, v, sk);
        }
    const float iq = 1.f / sqrtf(block_sum(sq, red) / (float)p.q_rank + p.eps);
    A* cq = reinterpret_cast<A*>(p.cq) + (size_t)row * p.q_rank;
    for (int c = tid; c < p.q_rank; c += 256) cq[c] = from_f<A>(ld_cg(zq + c) * iq * p.q_norm[c]);
    if (!p.cache || pos >= p.slots) return;
    const float ik = 1.f / sqrtf(block_sum(sk, red2) / (float)p.R + p.eps);
    A* k = reinterpret_cast<A*>(p.cache) + ((size_t)b * p.slots + pos) * p.ld;
    for (int c = tid; c < p.R; c += 256) k[c] = from_f<A>(ld_cg(zk + c) * ik * p.kv_norm[c]);
    const float* trig = p.trig + (size_t)pos * p.dims;
    for (int c = tid; c < p.rot; c += 256) {
        float v = ld_cg(zk + p.R + c);
        if (c < p.dims) {
            const float o = ld_cg(zk + p.R + (c ^ 1)), cs = trig[c & ~1], sn = trig[c | 1];
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
// qa[row][h][r] = sum_d q[row][h][d] W_uk[h][d][r] for up to eight rows, and the rotated part behind it: CTAs
// x = 128 latents of one head (y), the last x rotates.  Eight warps split d; partial sums meet in shared memory.
typedef decoder_absorb_args AbsorbParams;

static __global__ void __launch_bounds__(256) absorb_kernel(const AbsorbParams p) {
    extern __shared__ __align__(16) float absorb_smem[];     // q [8][dim], partial sums [8 warps][M][128]
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, dim = p.dim, M = p.B * p.T;
    const int dq = dim + p.rot;
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
    float* q_s = absorb_smem;
    float* part = q_s + (8 * dim + 3) / 4 * 4;
    const int r0 = blockIdx.x * 128 + lane * 4;              // R is a multiple of 4: a lane's latents are in or out together
    const int d0 = dim * warp / 8, d1 = dim * (warp + 1) / 8;
    const bf16* w = reinterpret_cast<const bf16*>(p.w_uk) + (size_t)h * dim * p.R + r0;
    const bool in = r0 < p.R;
    constexpr int PRE = 16;
    uint2 wv[PRE];
    auto fetch = [&](int u, int d) { wv[u] = in && d < d1 ? __ldg(reinterpret_cast<const uint2*>(w + (size_t)d * p.R)) : make_uint2(0, 0); };
#pragma unroll
    for (int u = 0; u < PRE; ++u) fetch(u, d0 + u);
    griddep_wait();
    for (int i = tid; i < M * dim; i += 256) q_s[i] = ld_cg(q + (size_t)(i / dim) * p.H * dq + h * dq + i % dim);
    __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int m = 0; m < 8; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[m][j] = 0.f;
    for (int d = d0; d < d1; d += PRE) {
#pragma unroll
        for (int u = 0; u < PRE; ++u) {
            const float f[4] = {__uint_as_float(wv[u].x << 16), __uint_as_float(wv[u].x & 0xffff0000u), __uint_as_float(wv[u].y << 16),
                                __uint_as_float(wv[u].y & 0xffff0000u)};
            if (d + u < d1) {
#pragma unroll
                for (int m = 0; m < 8; ++m)
                    if (m < M) {
                        const float x = q_s[m * dim + d + u];
#pragma unroll
                        for (int j = 0; j < 4; ++j) acc[m][j] = fmaf(f[j], x, acc[m][j]);
                    }
            }
            fetch(u, d + PRE + u);
        }
    }
#pragma unroll
    for (int m = 0; m < 8; ++m)
        if (m < M) *reinterpret_cast<float4*>(part + ((size_t)warp * M + m) * 128 + lane * 4) = make_float4(acc[m][0], acc[m][1], acc[m][2], acc[m][3]);
    __syncthreads();
    for (int i = tid; i < M * 128; i += 256) {
        const int r = blockIdx.x * 128 + (i & 127);
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) v += part[k * M * 128 + i];
        if (r < p.R) qa[((size_t)(i >> 7) * p.H + h) * p.ld + r] = from_f<bf16>(v);
    }
}

__device__ __forceinline__ void ldmatrix4(uint32_t addr, uint32_t (&v)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t addr, uint32_t (&v)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(addr));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool in) {   // 16 bytes, zeros when out of range
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(__cvta_generic_to_global(src)), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// One CTA: 16 heads of one row against one of gridDim.x ranges of the keys, 64 at a time.  Scores: a warp takes eight
// keys, k = the latent and rotated columns.  Weighted sum: a warp takes an eighth of the latents.  Output: unnormalised
// sums, running maximum (base 2) and sum of weights per range.
struct LatentStepSmem {
    int stride, q, s, p, st, kv, total;                      // bytes
    __host__ __device__ explicit LatentStepSmem(int ld) {
        stride = ((ld + 15) / 16 * 16 + 8) * 2;              // an odd number of 16-byte units: ldmatrix without conflicts
        q = 0, s = q + 16 * stride, p = s + 16 * 68 * 4, st = p + 16 * 72 * 2, kv = st + 3 * 16 * 4;
        kv = (kv + 15) / 16 * 16;
        total = kv + 2 * 64 * stride;
    }
};

template <int NT>   // 16-latent tiles per warp: R <= 128 * NT
__global__ void __launch_bounds__(256) latent_step_kernel(const LatentAttnParams p) {
    extern __shared__ __align__(16) uint8_t latent_step_smem[];
    const LatentStepSmem L(p.ld);
    const uint32_t base = smem_u32(latent_step_smem);
    float* s_s = reinterpret_cast<float*>(latent_step_smem + L.s);
    bf16* p_s = reinterpret_cast<bf16*>(latent_step_smem + L.p);
    float *m_s = reinterpret_cast<float*>(latent_step_smem + L.st), *l_s = m_s + 16, *f_s = m_s + 32;
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * 16, row = blockIdx.z, b = row / p.T, t = row - b * p.T;
    const int ld = p.ld, words = ld / 8, ksteps = (ld + 15) / 16, hn = min(16, p.H - h0);
    griddep_wait();
    const int n = (int)min(p.pos[0] + t + 1, (long long)p.slots);
    const int lo = (int)((long long)n * split / splits), hi = (int)((long long)n * (split + 1) / splits);
    const bf16* cache = reinterpret_cast<const bf16*>(p.cache) + (size_t)b * p.slots * ld;
    const bf16* q = reinterpret_cast<const bf16*>(p.qa) + ((size_t)row * p.H + h0) * ld;
    auto fetch = [&](int buf, int j0) {                      // every row up to the padded width, zeros outside
        const int w16 = 2 * ksteps;
        for (int i = tid; i < 64 * w16; i += 256) {
            const int r = i / w16, c = i - r * w16;
            const bool in = j0 + r < hi && c < words;
            cp_async16(base + L.kv + (buf * 64 + r) * L.stride + c * 16, cache + (in ? (size_t)(j0 + r) * ld + c * 8 : 0), in);
        }
        cp_async_commit();
    };
    for (int i = tid; i < 16 * 2 * ksteps; i += 256) {
        const int r = i / (2 * ksteps), c = i - r * 2 * ksteps;
        const bool in = r < hn && c < words;
        cp_async16(base + L.q + r * L.stride + c * 16, q + (in ? (size_t)r * ld + c * 8 : 0), in);
    }
    fetch(0, lo);
    if (tid < 16) m_s[tid] = -INFINITY, l_s[tid] = 0.f;
    float acc[NT][2][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[i][j][c] = 0.f;
    const int g = lane >> 2, qd = lane & 3;
    const int tiles = (hi - lo + 63) / 64;
    for (int it = 0; it < tiles; ++it) {
        const int j0 = lo + it * 64, buf = it & 1;
        if (it + 1 < tiles) fetch(buf ^ 1, j0 + 64), cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();
        {   // scores of keys j0 + 8 warp .. + 7
            float d0[4] = {0.f, 0.f, 0.f, 0.f}, d1[4] = {0.f, 0.f, 0.f, 0.f};
            const uint32_t qa = base + L.q + (lane & 15) * L.stride + (lane >> 4) * 16;
            const uint32_t ka = base + L.kv + (buf * 64 + warp * 8 + (lane & 7)) * L.stride + (lane >> 3) * 16;
            for (int k = 0; k < ksteps; k += 2) {
                uint32_t a[4], a2[4], kb[4];
                ldmatrix4(qa + k * 32, a);
                // four 8-column pieces of the keys: two k-steps (the second may lie in the row's padding, read but unused)
                if (k + 1 < ksteps) {
                    ldmatrix4(ka + k * 32, kb);
                    ldmatrix4(qa + k * 32 + 32, a2);
                    mma_bf16_16x8x16(d1, a2[0], a2[1], a2[2], a2[3], kb[2], kb[3]);
                } else {
                    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(kb[0]), "=r"(kb[1]) : "r"(ka - (lane >> 4) * 32 + k * 32));
                }
                mma_bf16_16x8x16(d0, a[0], a[1], a[2], a[3], kb[0], kb[1]);
            }
            const float f = p.scale * kLog2e;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int key = warp * 8 + 2 * qd + (c & 1), head = g + (c >> 1) * 8;
                s_s[head * 68 + key] = j0 + key < hi ? (d0[c] + d1[c]) * f : -INFINITY;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {                        // two heads per warp
            const int head = warp * 2 + i;
            const float s0 = s_s[head * 68 + lane], s1 = s_s[head * 68 + 32 + lane], mo = m_s[head];
            float mx = fmaxf(s0, s1);
#pragma unroll
            for (int d = 16; d; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float mn = fmaxf(mo, mx);                  // finite: the first key of a tile always counts
            const float w0 = exp2f(s0 - mn), w1 = exp2f(s1 - mn), sum = warp_sum(w0 + w1);
            p_s[head * 72 + lane] = from_f<bf16>(w0), p_s[head * 72 + 32 + lane] = from_f<bf16>(w1);
            __syncwarp();
            if (lane == 0) {
                const float f = exp2f(mo - mn);
                f_s[head] = f, m_s[head] = mn, l_s[head] = fmaf(l_s[head], f, sum);
            }
        }
        __syncthreads();
        const float fa = f_s[g], fb = f_s[g + 8];
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) acc[i][j][0] *= fa, acc[i][j][1] *= fa, acc[i][j][2] *= fb, acc[i][j][3] *= fb;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t a[4];
            ldmatrix4(base + L.p + (lane & 15) * 144 + kk * 32 + (lane >> 4) * 16, a);
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c = (warp * NT + i) * 16;
                if (c < p.R) {                               // uniform over the warp; a tile is inside the padded row
                    uint32_t v[4];
                    ldmatrix4_trans(base + L.kv + (buf * 64 + kk * 16 + (lane & 15)) * L.stride + (c + (lane >> 4) * 8) * 2, v);
                    mma_bf16_16x8x16(acc[i][0], a[0], a[1], a[2], a[3], v[0], v[1]);
                    mma_bf16_16x8x16(acc[i][1], a[0], a[1], a[2], a[3], v[2], v[3]);
                }
            }
        }
        __syncthreads();                                     // the buffer, the scores and the weights are used again
    }
    __syncthreads();
    float* part = p.part + (((size_t)row * p.H + h0) * splits + split) * p.R;
    if (tiles > 0)
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const int r = (warp * NT + i) * 16 + j * 8 + 2 * qd + (c & 1), head = g + (c >> 1) * 8;
                    if (r < p.R && head < hn) part[(size_t)head * splits * p.R + r] = acc[i][j][c];
                }
    if (tid < hn) {
        float* ml = p.ml + (((size_t)row * p.H + h0 + tid) * splits + split) * 2;
        ml[0] = m_s[tid], ml[1] = l_s[tid];
    }
}

// Joins the ranges' parts, adds the sink to the denominator and multiplies with W_uv: y[row][h][v].  CTAs x = 32 values
// of one head (y) and row (z); the weights are requested before the wait.
template <int RW>   // words of 16 bytes per lane and row of W_uv: R <= 256 * RW, a multiple of 8
__global__ void __launch_bounds__(256) latent_join_kernel(const LatentAttnParams p) {
    extern __shared__ __align__(16) float latent_join_smem[];   // weights of the ranges [splits], latent [R]
    __shared__ float inv_s;
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, row = blockIdx.z, R = p.R, splits = p.splits;
    float *w_s = latent_join_smem, *c_s = w_s + (splits + 3) / 4 * 4;
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
    const float* ml = p.ml + ((size_t)row * p.H + h) * splits * 2;
    if (warp == 0) {
        const float sink = p.sink[h] * kLog2e;
        float m = sink;
        for (int s = lane; s < splits; s += 32) m = fmaxf(m, __ldcg(ml + 2 * s));
#pragma unroll
        for (int d = 16; d; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
        float l = 0.f;
        for (int s = lane; s < splits; s += 32) {
            const float e = exp2f(__ldcg(ml + 2 * s) - m);   // 0 for a range without keys (m = -inf)
            w_s[s] = e;
            l = fmaf(e, __ldcg(ml + 2 * s + 1), l);
        }
        l = warp_sum(l) + exp2f(sink - m);
        if (lane == 0) inv_s = 1.f / l;
    }
    __syncthreads();
    const float* part = p.part + ((size_t)row * p.H + h) * splits * R;
    for (int c = tid; c < R; c += 256) {
        float o = 0.f;
#pragma unroll 8
        for (int s = 0; s < splits; ++s) {
            const float e = w_s[s];
            o = fmaf(e, e > 0.f ? __ldcg(part + (size_t)s * R + c) : 0.f, o);
        }
        c_s[c] = o * inv_s;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        float d = 0.f;
#pragma unroll
        for (int j = 0; j < RW; ++j) {
            const int c = (lane + 32 * j) * 8;
            if (c < R) {
                float f[8];
                unpack8(wv[i][j], f);
#pragma unroll
                for (int e = 0; e < 8; ++e) d = fmaf(f[e], c_s[c + e], d);
            }
        }
        d = warp_sum(d);
        const int v = blockIdx.x * 32 + warp * 4 + i;
        if (lane == 0 && v < p.vdim) reinterpret_cast<bf16*>(p.y)[((size_t)row * p.H + h) * p.vdim + v] = from_f<bf16>(d);
    }
}

}  // namespace tsp
