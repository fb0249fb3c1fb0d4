// Attention without softmax: the weight of a visible key is sigmoid(q.k * scale - slope_h * distance + bias_h),
// not normalised over the keys; optional chunked visibility (a query sees its own chunk of `chunk` positions, up
// to itself; chunks are counted from position 0 of the sequence); output gate sigmoid(g) per element.
//
// Cache.  A query never looks past the start of its chunk, so a sequence holds one chunk of keys and values per
// layer: position p lives in slot p mod chunk, [B][G][slots][dim] (keys normalised) and [B][G][slots][vdim].
// chunk = slots = the longest sequence gives plain causal attention.  A prompt portion reads what earlier calls
// left of its first chunk from the cache and its own keys from the projection buffer, and stores its last
// chunk's keys afterwards, because later chunks use the slots that its first queries still read.
#pragma once
#include "decoder_common.cuh"
#include "decoder_ops.h"
#include "lm_head.cuh"

namespace tsp {

typedef decoder_attn_args AttnParams;

// RMS norm of every query and key head in place; one warp per row and head
template <typename A>
__global__ void __launch_bounds__(256) head_norm_kernel(const AttnParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int heads = p.H + p.G, dim = p.dim;
    const long long unit = (long long)blockIdx.x * 8 + warp;
    if (unit >= (long long)p.B * p.T * heads) return;
    const long long row = unit / heads;
    const int h = (int)(unit - row * heads);
    A* x = reinterpret_cast<A*>(p.proj) + row * p.ld + (h < p.H ? p.off_q + h * dim : p.off_k + (h - p.H) * dim);
    const float* w = h < p.H ? p.q_norm : p.k_norm;
    float ss = 0.f;
    for (int c = lane; c < dim; c += 32) {
        const float v = ld_cg(x + c);
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dim + p.eps);
    for (int c = lane; c < dim; c += 32) x[c] = from_f<A>(ld_cg(x + c) * inv * w[c]);
}

// The same with four neighbouring channels per lane: dim a power of two from 4 to 128 (dim / 4 lanes share a head), q
// and k side by side; two units of 128 channels per warp in flight.
template <typename A>
__global__ void __launch_bounds__(256) head_norm4_kernel(const AttnParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long n = (long long)(p.H + p.G) * p.dim, total = (long long)p.B * p.T * n;
    float4 x[2];
    long long at[2];
    A* dst[2];
    const float* w[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        at[i] = (((long long)blockIdx.x * 8 + warp) * 2 + i) * 128 + lane * 4;
        const long long e = min(at[i], total - 4), row = e / n;
        const int c = (int)(e - row * n);
        dst[i] = reinterpret_cast<A*>(p.proj) + row * p.ld + p.off_q + c;
        w[i] = (c < p.H * p.dim ? p.q_norm : p.k_norm) + (c & (p.dim - 1));
        x[i] = ld_cg4(dst[i]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        float ss = x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
        for (int d = p.dim / 8; d; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
        const float inv = 1.f / sqrtf(ss / (float)p.dim + p.eps);
        const float4 g = *reinterpret_cast<const float4*>(w[i]);
        if (at[i] < total) st4(dst[i], make_float4(x[i].x * inv * g.x, x[i].y * inv * g.y, x[i].z * inv * g.z, x[i].w * inv * g.w));
    }
}

// Any type, any sizes: one CTA per query and head, 128 keys at a time.  Queries and keys already normalised.
template <typename A>
__global__ void __launch_bounds__(128) sigmoid_attn_plain_kernel(const AttnParams p) {
    extern __shared__ __align__(16) float plain_smem[];
    __shared__ float w_s[128];
    griddep_launch_dependents();
    griddep_wait();
    const int tid = threadIdx.x, t = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
    const int g = h / (p.H / p.G), dim = p.dim, vdim = p.vdim;
    const long long t0 = p.pos[0], i = t0 + t, lo = i / p.chunk * p.chunk;
    const A* proj = reinterpret_cast<const A*>(p.proj) + (size_t)b * p.T * p.ld;
    const A* ck = reinterpret_cast<const A*>(p.ck) + ((size_t)b * p.G + g) * p.slots * dim;
    const A* cv = reinterpret_cast<const A*>(p.cv) + ((size_t)b * p.G + g) * p.slots * vdim;
    float* q_s = plain_smem;                    // [dim]
    float* o_s = plain_smem + dim;              // [vdim]
    for (int c = tid; c < dim; c += 128) q_s[c] = ld_cg(proj + t * p.ld + p.off_q + h * dim + c);
    for (int c = tid; c < vdim; c += 128) o_s[c] = 0.f;
    __syncthreads();
    const float slope = p.slope[h], bias = p.bias[h];
    for (long long j0 = lo; j0 <= i; j0 += 128) {
        const long long j = j0 + tid;
        float w = 0.f;
        if (j <= i) {
            const A* k = j >= t0 ? proj + (j - t0) * p.ld + p.off_k + g * dim : ck + (size_t)(j % p.chunk) * dim;
            float s = 0.f;
            for (int c = 0; c < dim; ++c) s = fmaf(q_s[c], ld_cg(k + c), s);
            w = sigmoid_f(s * p.scale - slope * (float)(i - j) + bias);
        }
        w_s[tid] = w;
        __syncthreads();
        const int n = (int)min((long long)128, i - j0 + 1);
        for (int c = tid; c < vdim; c += 128) {
            float o = o_s[c];
            for (int e = 0; e < n; ++e) {
                const long long jj = j0 + e;
                const A* v = jj >= t0 ? proj + (jj - t0) * p.ld + p.off_v + g * vdim : cv + (size_t)(jj % p.chunk) * vdim;
                o = fmaf(w_s[e], ld_cg(v + c), o);
            }
            o_s[c] = o;
        }
        __syncthreads();
    }
    A* y = reinterpret_cast<A*>(p.y) + ((size_t)b * p.T + t) * p.H * vdim + h * vdim;
    for (int c = tid; c < vdim; c += 128)
        y[c] = from_f<A>(o_s[c] * sigmoid_f(ld_cg(proj + t * p.ld + p.off_g + h * vdim + c)));
}

// After a prompt portion: the keys (normalised) and values of its last chunk go to their slots.
template <typename A>
__global__ void __launch_bounds__(128) attn_cache_store_kernel(const AttnParams p) {
    griddep_launch_dependents();
    griddep_wait();
    const int b = blockIdx.y, t = p.T - 1 - (int)blockIdx.x;
    if (t < 0) return;
    const long long t0 = p.pos[0], i = t0 + t, last = t0 + p.T - 1;
    if (i < last / p.chunk * p.chunk) return;                // an earlier chunk: never read again
    const size_t slot = (size_t)(i % p.chunk);
    if (slot >= (size_t)p.slots) return;
    const A* row = reinterpret_cast<const A*>(p.proj) + ((size_t)b * p.T + t) * p.ld;
    const int g = blockIdx.z;
    A* k = reinterpret_cast<A*>(p.ck) + (((size_t)b * p.G + g) * p.slots + slot) * p.dim;
    A* v = reinterpret_cast<A*>(p.cv) + (((size_t)b * p.G + g) * p.slots + slot) * p.vdim;
    for (int c = threadIdx.x; c < p.dim; c += blockDim.x) k[c] = from_f<A>(ld_cg(row + p.off_k + g * p.dim + c));
    for (int c = threadIdx.x; c < p.vdim; c += blockDim.x) v[c] = from_f<A>(ld_cg(row + p.off_v + g * p.vdim + c));
}

// ------------------------------------------------------------------------------------------ one token
// bf16, dim and vdim multiples of 8 and at most 8 * LPK.  Norms of the new query and key, cache append,
// attention over the visible slots and the gate in one launch.  A cluster of CTAs shares one key/value head
// and RT of its query heads: each CTA takes a slice of the slots, a key being handled by LPK lanes with eight
// channels each; partial outputs (plain sums, as the weights are not normalised) meet in distributed shared
// memory in a fixed order.
//
// A warp has U keys per lane group in flight.  Their RT * U scores are summed over the LPK lanes by a transposing
// butterfly that leaves each score in one lane (or a few), where its weight is computed once; the weights are then
// handed back to all lanes for the values' sum.
template <int RT, int LPK>
__global__ void __launch_bounds__(256, RT <= 4 ? 2 : 1) sigmoid_attn_step_kernel(const AttnParams p) {
    constexpr int KPW = 32 / LPK, VD = 8 * LPK;              // keys per warp at a time, padded width
    constexpr int U = RT <= 2 ? 8 : RT <= 4 ? 4 : 2, NV = RT * U;
    constexpr int LL = LPK == 4 ? 2 : LPK == 8 ? 3 : LPK == 16 ? 4 : 5, LN = NV == 8 ? 3 : 4;
    constexpr int EX = LL < LN ? LL : LN, REM = NV >> EX;    // exchange levels of the butterfly, scores left per lane
    __shared__ __align__(16) float q_s[RT][VD];
    __shared__ __align__(16) float k_s[VD];
    __shared__ __align__(16) float v_s[VD];
    __shared__ __align__(16) float part[8][RT][VD];
    __shared__ __align__(16) float sum_s[RT][VD];
    griddep_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int rep = p.H / p.G, hgroups = (rep + RT - 1) / RT;
    const int g = blockIdx.y / hgroups, h0 = g * rep + (blockIdx.y % hgroups) * RT;
    const int hn = min(RT, (g + 1) * rep - h0);
    const int b = blockIdx.z, rank = blockIdx.x, nr = gridDim.x;
    const int dim = p.dim, vdim = p.vdim;
    bf16* ck = reinterpret_cast<bf16*>(p.ck) + ((size_t)b * p.G + g) * p.slots * dim;
    bf16* cv = reinterpret_cast<bf16*>(p.cv) + ((size_t)b * p.G + g) * p.slots * vdim;
    griddep_wait();
    const bf16* row = reinterpret_cast<const bf16*>(p.proj) + (size_t)b * p.ld;
    const int cur = (int)((unsigned)p.pos[0] % (unsigned)p.chunk);   // slot of this token = number of earlier visible keys
    const bool writer = rank == 0 && blockIdx.y % hgroups == 0 && cur < p.slots;

    for (int e = warp; e < RT + 2; e += 8) {
        if (e < RT + 1) {                                    // norms: RT query heads, then the key
            const bool is_k = e == RT;
            const bool on = is_k || e < hn;
            const bf16* x = row + (is_k ? p.off_k + g * dim : p.off_q + (h0 + (on ? e : 0)) * dim);
            float v[VD / 32 > 0 ? VD / 32 : 1], ss = 0.f;
#pragma unroll
            for (int j = 0; j < VD / 32; ++j) {
                const int c = lane + 32 * j;
                v[j] = (on && c < dim) ? ld_cg(x + c) : 0.f;
                ss = fmaf(v[j], v[j], ss);
            }
            const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dim + p.eps);
#pragma unroll
            for (int j = 0; j < VD / 32; ++j) {
                const int c = lane + 32 * j;
                const float n = c < dim ? v[j] * inv * (is_k ? p.k_norm[c] : p.q_norm[c]) : 0.f;
                if (is_k) {
                    const bf16 kb = from_f<bf16>(n);         // the value every later token will read
                    k_s[c] = to_f(kb);
                    if (writer && c < dim) ck[(size_t)cur * dim + c] = kb;
                } else {
                    q_s[e][c] = n * p.scale;
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < VD / 32; ++j) {
                const int c = lane + 32 * j;
                const float v = c < vdim ? ld_cg(row + p.off_v + g * vdim + c) : 0.f;
                v_s[c] = v;
                if (writer && c < vdim) cv[(size_t)cur * vdim + c] = from_f<bf16>(v);
            }
        }
    }
    __syncthreads();

    const int sub = lane / LPK, c8 = (lane % LPK) * 8;
    const int v0 = ((lane % LPK) >> (LL - EX)) * REM;        // first of the scores whose weights this lane computes
    float q[RT][8], acc[RT][8], slope[REM], bias[REM];
#pragma unroll
    for (int i = 0; i < REM; ++i) {
        const int r = (v0 + i) / U;
        slope[i] = r < hn ? p.slope[h0 + r] : 0.f;
        bias[i] = r < hn ? p.bias[h0 + r] : 0.f;
    }
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
        for (int c = 0; c < 8; ++c) q[r][c] = q_s[r][c8 + c], acc[r][c] = 0.f;
    // scores of keys j0 + u * KPW + sub for u < U (those below hi count), weights, weighted values
    auto use = [&](const uint4 (&kv)[U], const uint4 (&vv)[U], int j0, int hi) {
        float s[NV];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            float k[8];
            unpack8(kv[u], k);
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                float d = q[r][0] * k[0];
#pragma unroll
                for (int c = 1; c < 8; ++c) d = fmaf(q[r][c], k[c], d);
                s[r * U + u] = d;
            }
        }
#pragma unroll
        for (int l = 0; l < LL; ++l) {
            const int d = LPK >> (l + 1), n = NV >> (l + 1);
            if (l < EX) {
#pragma unroll
                for (int i = 0; i < n; ++i) {
                    const bool up = lane & d;
                    const float keep = up ? s[i + n] : s[i], give = up ? s[i] : s[i + n];
                    s[i] = keep + __shfl_xor_sync(0xffffffffu, give, d);
                }
            } else {
                s[0] += __shfl_xor_sync(0xffffffffu, s[0], d);
            }
        }
#pragma unroll
        for (int i = 0; i < REM; ++i) {
            const int j = j0 + (v0 + i) % U * KPW + sub;
            s[i] = j < hi ? sigmoid_fast(s[i] - slope[i] * (float)(cur - j) + bias[i]) : 0.f;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            float v[8];
            unpack8(vv[u], v);
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                const int n = r * U + u;
                const float w = __shfl_sync(0xffffffffu, s[n % REM], sub * LPK + ((n / REM) << (LL - EX)));
#pragma unroll
                for (int c = 0; c < 8; ++c) acc[r][c] = fmaf(w, v[c], acc[r][c]);
            }
        }
    };
    const int lo = (int)((long long)cur * rank / nr), hi = (int)((long long)cur * (rank + 1) / nr);
    const bool kin = c8 < dim, vin = c8 < vdim;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    for (int j0 = lo + warp * KPW * U; j0 < hi; j0 += 8 * KPW * U) {
        uint4 kv[U], vv[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int j = j0 + u * KPW + sub;
            kv[u] = (j < hi && kin) ? ld_cg_128(ck + (size_t)j * dim + c8) : zero;
            vv[u] = (j < hi && vin) ? ld_cg_128(cv + (size_t)j * vdim + c8) : zero;
        }
        use(kv, vv, j0, hi);
    }
    if (rank == nr - 1 && warp == 7) {                       // the token itself: bf16 values, so packing loses nothing
        uint4 kv[U], vv[U];
#pragma unroll
        for (int u = 0; u < U; ++u) kv[u] = vv[u] = zero;
        if (sub == 0) {
            const float *k = k_s + c8, *v = v_s + c8;
            kv[0] = make_uint4(pack_bf16(k[0], k[1]), pack_bf16(k[2], k[3]), pack_bf16(k[4], k[5]), pack_bf16(k[6], k[7]));
            vv[0] = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
        }
        use(kv, vv, cur, cur + 1);
    }
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
        for (int c = 0; c < 8; ++c) {
#pragma unroll
            for (int d = LPK; d < 32; d <<= 1) acc[r][c] += __shfl_xor_sync(0xffffffffu, acc[r][c], d);
            if (sub == 0) part[warp][r][c8 + c] = acc[r][c];
        }
    __syncthreads();
    for (int e = tid; e < RT * VD; e += 256) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) s += (&part[w][0][0])[e];
        (&sum_s[0][0])[e] = s;
    }
    cluster_arrive();
    cluster_wait();
    if (rank == 0) {
        const uint32_t base = smem_u32(&sum_s[0][0]);
        bf16* y = reinterpret_cast<bf16*>(p.y) + (size_t)b * p.H * vdim;
        for (int e = tid; e < RT * VD; e += 256) {
            const int r = e / VD, c = e - r * VD;
            float s = 0.f;
            for (int k = 0; k < nr; ++k) {
                float v;
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(map_to_rank(base + 4 * e, k)));
                s += v;
            }
            if (r < hn && c < vdim) {
                const int h = h0 + r;
                y[h * vdim + c] = from_f<bf16>(s * sigmoid_f(ld_cg(row + p.off_g + h * vdim + c)));
            }
        }
    }
    cluster_arrive();                                        // nobody leaves while rank 0 still reads
    cluster_wait();
}

}  // namespace tsp
