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
    for (int g = 0; g < p.G; ++g) {
        A* k = reinterpret_cast<A*>(p.ck) + (((size_t)b * p.G + g) * p.slots + slot) * p.dim;
        A* v = reinterpret_cast<A*>(p.cv) + (((size_t)b * p.G + g) * p.slots + slot) * p.vdim;
        for (int c = threadIdx.x; c < p.dim; c += blockDim.x) k[c] = from_f<A>(ld_cg(row + p.off_k + g * p.dim + c));
        for (int c = threadIdx.x; c < p.vdim; c += blockDim.x) v[c] = from_f<A>(ld_cg(row + p.off_v + g * p.vdim + c));
    }
}

// ------------------------------------------------------------------------------------------ one token
// bf16, dim and vdim multiples of 8 and at most 8 * LPK.  Norms of the new query and key, cache append,
// attention over the visible slots and the gate in one launch.  A cluster of CTAs shares one key/value head
// and RT of its query heads: each CTA takes a slice of the slots, a key being handled by LPK lanes with eight
// channels each; partial outputs (plain sums, as the weights are not normalised) meet in distributed shared
// memory in a fixed order.
template <int RT, int LPK>
__global__ void __launch_bounds__(256) sigmoid_attn_step_kernel(const AttnParams p) {
    constexpr int KPW = 32 / LPK, VD = 8 * LPK, U = 4;       // keys per warp at a time, padded width, unroll
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
    const int cur = (int)(p.pos[0] % p.chunk);               // slot of this token = number of earlier visible keys
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
    float q[RT][8], acc[RT][8], slope[RT], bias[RT];
#pragma unroll
    for (int r = 0; r < RT; ++r) {
        slope[r] = r < hn ? p.slope[h0 + r] : 0.f;
        bias[r] = r < hn ? p.bias[h0 + r] : 0.f;
#pragma unroll
        for (int c = 0; c < 8; ++c) q[r][c] = q_s[r][c8 + c], acc[r][c] = 0.f;
    }
    auto use = [&](const float (&k)[8], const float (&v)[8], int j, bool on) {
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            float s = 0.f;
#pragma unroll
            for (int c = 0; c < 8; ++c) s = fmaf(q[r][c], k[c], s);
#pragma unroll
            for (int d = LPK / 2; d; d >>= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
            const float w = on ? sigmoid_f(s - slope[r] * (float)(cur - j) + bias[r]) : 0.f;
#pragma unroll
            for (int c = 0; c < 8; ++c) acc[r][c] = fmaf(w, v[c], acc[r][c]);
        }
    };
    const int lo = (int)((long long)cur * rank / nr), hi = (int)((long long)cur * (rank + 1) / nr);
    const bool kin = c8 < dim, vin = c8 < vdim;
    for (int j0 = lo + warp * KPW * U; j0 < hi; j0 += 8 * KPW * U) {
        uint4 kv[U], vv[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int j = j0 + u * KPW + sub;
            kv[u] = (j < hi && kin) ? ld_cg_128(ck + (size_t)j * dim + c8) : make_uint4(0, 0, 0, 0);
            vv[u] = (j < hi && vin) ? ld_cg_128(cv + (size_t)j * vdim + c8) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int j = j0 + u * KPW + sub;
            float k[8], v[8];
            unpack8(kv[u], k), unpack8(vv[u], v);
            use(k, v, j, j < hi);
        }
    }
    if (rank == nr - 1 && warp == 7) {                       // the token itself
        float k[8], v[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) k[c] = k_s[c8 + c], v[c] = v_s[c8 + c];
        use(k, v, cur, sub == 0);
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
