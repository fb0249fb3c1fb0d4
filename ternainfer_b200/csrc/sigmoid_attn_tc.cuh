// Prompt kernel of the sigmoid attention (sigmoid_attn.cuh) on the tensor cores of sm_100a.
//
// One CTA per 128 queries of one head.  Scores S = Q K^T (tcgen05.mma, Q and K by TMA in 128-byte-swizzled
// K-major tiles) go to tensor memory; eight warps turn them into weights and write those back to tensor memory
// as bf16 over the scores they have read; O += P V takes P from there and V by TMA as an N-contiguous operand.
// The weights are not normalised over the keys, so O is a plain accumulation: no running maximum, no rescaling.
// Keys of earlier calls (the part of the first query's chunk before this call) come from the cache's tensor maps,
// the call's own keys from the projection buffer's; a tile of keys has one source.
//
// The weight 1 / (1 + 2^x) costs an exponential and a reciprocal in the special-function unit, which would
// take twice the tensor cores' time at 128 channels; four weights share one reciprocal of the product of their
// denominators (x is clamped to 30, where a weight is 1e-9, so the product stays finite).
//
// Half of the tensor memory and less than half of the shared memory per CTA: two CTAs share an SM, one's MMAs
// under the other's sigmoids.  Roles: warp 0 TMA, warp 1 MMA issue and tensor memory, warps 2-9 weights (one
// 32-lane quarter of tensor memory and one half of the keys each) and the gated output.  Every wait is bounded.
#pragma once
#include "decoder_status.cuh"
#include "sigmoid_attn.cuh"
#include "tcgen05_sm100.cuh"

namespace tsp {

struct AttnTcSmem {
    static constexpr int threads = 320;
    static constexpr int block = 128 * 128;              // bytes: 128 rows of 64 bf16
    static constexpr int bar_q = 0, bar_k = 8, bar_k_free = 16, bar_v = 24, bar_v_free = 32, bar_s = 40, bar_p = 48, bar_o = 56;
    static constexpr int tmem_slot = 64, abort_flag = 68;
    static constexpr int data = 1024;
    static int total(int qk_blocks, int v_blocks) { return 1024 + data + (2 * qk_blocks + v_blocks) * block; }
};

// 1 / (1 + 2^x) of four values with one reciprocal
__device__ __forceinline__ void sigmoid4(float2 x01, float2 x23, float (&w)[4]) {
    const float2 one = make_float2(1.f, 1.f);
    const float2 a01 = add2(make_float2(ex2_approx(fminf(x01.x, 30.f)), ex2_approx(fminf(x01.y, 30.f))), one);
    const float2 a23 = add2(make_float2(ex2_approx(fminf(x23.x, 30.f)), ex2_approx(fminf(x23.y, 30.f))), one);
    const float p01 = a01.x * a01.y, p23 = a23.x * a23.y;
    const float r = rcp_approx(p01 * p23);
    const float r01 = r * p23, r23 = r * p01;
    w[0] = r01 * a01.y, w[1] = r01 * a01.x, w[2] = r23 * a23.y, w[3] = r23 * a23.x;
}

__global__ void __launch_bounds__(AttnTcSmem::threads, 2)
    sigmoid_attn_tc_kernel(const AttnParams p, const __grid_constant__ CUtensorMap map_proj, const __grid_constant__ CUtensorMap map_ck,
                           const __grid_constant__ CUtensorMap map_cv) {
    using L = AttnTcSmem;
    extern __shared__ __align__(128) uint8_t attn_smem[];
    const uint32_t dyn = smem_u32(attn_smem), sbase = (dyn + 1023u) & ~1023u;
    uint8_t* base = attn_smem + (sbase - dyn);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(base + L::abort_flag);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int tile = (int)(gridDim.x - 1 - blockIdx.x);      // the tiles with the most keys start first
    const int h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G);
    const int dim = p.dim, vdim = p.vdim, qb = (dim + 63) >> 6, vb = (vdim + 63) >> 6;
    const uint32_t q_s = sbase + L::data, k_s = q_s + qb * L::block, v_s = k_s + qb * L::block;
    const int r0 = tile * 128, rows = min(128, p.T - r0);

    if (tid == 0) {
        mbar_init(sbase + L::bar_q, 1);
        mbar_init(sbase + L::bar_k, 1);
        mbar_init(sbase + L::bar_k_free, 1);
        mbar_init(sbase + L::bar_v, 1);
        mbar_init(sbase + L::bar_v_free, 1);
        mbar_init(sbase + L::bar_s, 1);
        mbar_init(sbase + L::bar_p, 8);
        mbar_init(sbase + L::bar_o, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc(sbase + L::tmem_slot, 256);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(base + L::tmem_slot);   // S and P: columns 0-127, O: 128-255

    // keys: first the chunk's part before this call (cache), then the call's own rows
    const long long t0 = p.pos[0], q0 = t0 + r0, q1 = q0 + rows - 1;
    const long long lo = q0 / p.chunk * p.chunk;
    const long long own0 = lo > t0 ? lo : t0;
    const int n_cache = lo < t0 ? (int)((t0 - lo + 127) >> 7) : 0;
    const int n_tiles = n_cache + (int)((q1 - own0 + 128) >> 7);
    bool ok = true;

    if (warp == 0) {
        if (lane == 0) {
            mbar_arrive_expect_tx(sbase + L::bar_q, qb * L::block);
            for (int i = 0; i < qb; ++i)
                tma_load_2d(q_s + i * L::block, &map_proj, p.off_q + h * dim + 64 * i, b * p.T + r0, sbase + L::bar_q);
            for (int j = 0; j < n_tiles && ok; ++j) {
                const bool cached = j < n_cache;
                const int row = cached ? (b * p.G + g) * p.slots + 128 * j : b * p.T + (int)(own0 - t0) + 128 * (j - n_cache);
                if (j > 0) ok = wait_or_abort(sbase + L::bar_k_free, (j - 1) & 1, abort_flag);
                if (!ok) break;
                mbar_arrive_expect_tx(sbase + L::bar_k, qb * L::block);
                for (int i = 0; i < qb; ++i)
                    tma_load_2d(k_s + i * L::block, cached ? &map_ck : &map_proj, (cached ? 0 : p.off_k + g * dim) + 64 * i, row,
                                sbase + L::bar_k);
                if (j > 0) ok = wait_or_abort(sbase + L::bar_v_free, (j - 1) & 1, abort_flag);
                if (!ok) break;
                mbar_arrive_expect_tx(sbase + L::bar_v, vb * L::block);
                for (int i = 0; i < vb; ++i)
                    tma_load_2d(v_s + i * L::block, cached ? &map_cv : &map_proj, (cached ? 0 : p.off_v + g * vdim) + 64 * i, row,
                                sbase + L::bar_v);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t id_s = umma_idesc_bf16(128, 128, false), id_o = umma_idesc_bf16(128, vdim, true);
            ok = wait_or_abort(sbase + L::bar_q, 0, abort_flag);
            for (int j = 0; j < n_tiles && ok; ++j) {
                ok = wait_or_abort(sbase + L::bar_k, j & 1, abort_flag);
                if (!ok) break;
                tc_fence_after();
                for (int kk = 0; kk < dim / 16; ++kk) {
                    const uint32_t at = (kk >> 2) * L::block + (kk & 3) * 32;
                    umma_bf16_ss(tmem, umma_desc_sw128(q_s + at), umma_desc_sw128(k_s + at), id_s, kk != 0);
                }
                umma_commit(sbase + L::bar_k_free);
                umma_commit(sbase + L::bar_s);
                ok = wait_or_abort(sbase + L::bar_v, j & 1, abort_flag) && wait_or_abort(sbase + L::bar_p, j & 1, abort_flag);
                if (!ok) break;
                tc_fence_after();
                for (int kk = 0; kk < 8; ++kk)   // weights of keys 16 kk: 8 columns, each half of the keys in its own half of S
                    umma_bf16_ts(tmem + 128, tmem + (kk & 3) * 8 + (kk >> 2) * 64, umma_desc_mn_sw128(v_s + kk * 2048, L::block), id_o,
                                 (j | kk) != 0);
                umma_commit(sbase + L::bar_v_free);
            }
            if (ok) umma_commit(sbase + L::bar_o);
        }
    } else {
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        const uint32_t lanes = (uint32_t)(32 * quarter) << 16;
        const long long q = q0 + 32 * quarter + lane;        // this lane's query
        const long long q_lo = q / p.chunk * p.chunk;
        constexpr float kLog2e = 1.4426950408889634f;
        const float mul = -p.scale * kLog2e, sl = p.slope[h] * kLog2e, bias = p.bias[h] * kLog2e;
        const float2 mul_2 = make_float2(mul, mul), two_sl = make_float2(-2.f * sl, -2.f * sl);
        for (int j = 0; j < n_tiles; ++j) {
            const bool cached = j < n_cache;
            const long long k0 = cached ? lo + 128 * j : own0 + 128 * (j - n_cache);
            const int vis_lo = (int)max(0ll, q_lo - k0);
            const int vis_hi = (int)min(min(128ll, q + 1 - k0), (cached ? t0 : q1 + 1) - k0);   // may be <= 0
            if (ok) ok = wait_or_abort(sbase + L::bar_s, j & 1, abort_flag);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
#pragma unroll 1
            for (int c = 0; c < 2; ++c) {
                const int col = 64 * half + 32 * c;
                uint32_t s[32], w[16];
                tmem_ld32(tmem + lanes + col, s);
                // x = (slope * (q - key) - bias - score) * log2 e, two keys at a time
                const float x0 = sl * (float)(int)(q - k0 - col) - bias;
                float2 off = make_float2(x0, x0 - sl);
                const bool whole = __all_sync(0xffffffffu, vis_lo <= col && vis_hi >= col + 32);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    float wt[4];
                    const float2 xa = fma2(make_float2(__uint_as_float(s[4 * i]), __uint_as_float(s[4 * i + 1])), mul_2, off);
                    off = add2(off, two_sl);
                    const float2 xb = fma2(make_float2(__uint_as_float(s[4 * i + 2]), __uint_as_float(s[4 * i + 3])), mul_2, off);
                    off = add2(off, two_sl);
                    sigmoid4(xa, xb, wt);
                    if (!whole) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const int key = col + 4 * i + e;
                            if (key < vis_lo || key >= vis_hi) wt[e] = 0.f;
                        }
                    }
                    w[2 * i] = pack_bf16(wt[0], wt[1]), w[2 * i + 1] = pack_bf16(wt[2], wt[3]);
                }
                tmem_st16(tmem + lanes + 64 * half + 16 * c, w);
            }
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(sbase + L::bar_p);
        }
        if (ok) ok = wait_or_abort(sbase + L::bar_o, 0, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            tc_fence_after();
            const int r = 32 * quarter + lane;
            const bool live = r < rows;
            const size_t row = (size_t)b * p.T + r0 + (live ? r : 0);
            const bf16* gate = reinterpret_cast<const bf16*>(p.proj) + row * p.ld + p.off_g + h * vdim;
            bf16* y = reinterpret_cast<bf16*>(p.y) + row * ((size_t)p.H * vdim) + h * vdim;
            for (int c = 16 * half; c < vdim; c += 32) {
                int o[16];
                tmem_ld16(tmem + lanes + 128 + c, o);
                float gf[2][8];
                unpack8(ldg_128(gate + c), gf[0]), unpack8(ldg_128(gate + c + 8), gf[1]);
                uint32_t out[8];
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    out[i] = pack_bf16(__int_as_float(o[2 * i]) * sigmoid_f((&gf[0][0])[2 * i]),
                                       __int_as_float(o[2 * i + 1]) * sigmoid_f((&gf[0][0])[2 * i + 1]));
                if (live) {
                    stg_128(y + c, make_uint4(out[0], out[1], out[2], out[3]));
                    stg_128(y + c + 8, make_uint4(out[4], out[5], out[6], out[7]));
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag && tid == 0) atomicExch(&g_decoder_status, 4);
    if (warp == 1) tmem_dealloc(tmem, 256);
}

}  // namespace tsp
