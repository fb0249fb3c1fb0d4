// Prompt kernel of the attention over a latent (latent_attn.cuh) on the tensor cores of sm_100a: causal softmax with
// a sink over expanded keys and values.
//
// One CTA per 128 queries of one head, 64 keys at a time.  A score has two parts, q_u . k_u over the head's own key
// columns and q_r . k_r over the key part that all heads share, which is read straight from the cache; both accumulate
// into one tile of tensor memory.  Four warps hold a query per lane: maximum and exponentials of a tile in registers,
// weights back to tensor memory as bf16 over the scores, then O += P V with P as the tensor-memory operand.
//
// The reference point of the exponentials starts at the sink with a sum of one, which is all that the sink needs.  It
// moves only when a tile's maximum lies more than 2^8 above it; only then is O read, rescaled and written back.
//
// Scores are double-buffered: the MMAs of tile j + 1's scores run under the exponentials of tile j.  256 columns of
// tensor memory and at most 112 KB of shared memory per CTA, so that two CTAs share an SM.  Roles: warp 0 TMA,
// warp 1 MMA issue and tensor memory, warps 2-5 softmax and output.  Every wait is bounded.
#pragma once
#include "decoder_status.cuh"
#include "latent_attn.cuh"
#include "tcgen05_sm100.cuh"

namespace tsp {

typedef decoder_latent_prompt_args LatentPromptParams;

struct LatentTcSmem {
    static constexpr int threads = 192;
    static constexpr int qblock = 128 * 128, kblock = 64 * 128;   // bytes: 128 / 64 rows of 64 bf16
    static constexpr int bar_q = 0, bar_k = 8, bar_k_free = 16, bar_v = 24, bar_v_free = 32, bar_s = 40, bar_p = 56, bar_o = 72;
    static constexpr int tmem_slot = 80, abort_flag = 84, data = 1024;
    static int total(int qk, int rot, int v) { return 1024 + data + (qk + rot) * qblock + (qk + rot + v) * kblock; }
};

__global__ void __launch_bounds__(LatentTcSmem::threads, 2)
    latent_attn_tc_kernel(const LatentPromptParams p, const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                          const __grid_constant__ CUtensorMap map_cache) {
    using L = LatentTcSmem;
    extern __shared__ __align__(128) uint8_t latent_tc_smem[];
    const uint32_t dyn = smem_u32(latent_tc_smem), sbase = (dyn + 1023u) & ~1023u;
    uint8_t* base = latent_tc_smem + (sbase - dyn);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(base + L::abort_flag);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int tile = (int)(gridDim.x - 1 - blockIdx.x);      // the tiles with the most keys start first
    const int h = blockIdx.y, b = blockIdx.z;
    const int dim = p.dim, rot = p.rot, vdim = p.vdim, qb = (dim + 63) >> 6, rb = (rot + 63) >> 6, vb = (vdim + 63) >> 6;
    const uint32_t q_s = sbase + L::data, k_s = q_s + (qb + rb) * L::qblock, v_s = k_s + (qb + rb) * L::kblock;
    const int r0 = tile * 128, rows = min(128, p.T - r0);
    const int n_tiles = (p.start + r0 + rows + 63) >> 6;
    auto bar_s = [&](int j) { return sbase + L::bar_s + 8 * (j & 1); };
    auto bar_p = [&](int j) { return sbase + L::bar_p + 8 * (j & 1); };

    if (tid == 0) {
        mbar_init(sbase + L::bar_q, 1);
        mbar_init(sbase + L::bar_k, 1);
        mbar_init(sbase + L::bar_k_free, 1);
        mbar_init(sbase + L::bar_v, 1);
        mbar_init(sbase + L::bar_v_free, 1);
        for (int j = 0; j < 2; ++j) mbar_init(bar_s(j), 1), mbar_init(bar_p(j), 4);
        mbar_init(sbase + L::bar_o, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc(sbase + L::tmem_slot, 256);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(base + L::tmem_slot);   // S and P: columns 0-63 and 64-127, O: 128-255
    bool ok = true;

    if (warp == 0) {
        if (lane == 0) {
            mbar_arrive_expect_tx(sbase + L::bar_q, (qb + rb) * L::qblock);
            for (int i = 0; i < qb; ++i) tma_load_2d(q_s + i * L::qblock, &map_q, h * (dim + rot) + 64 * i, b * p.T + r0, sbase + L::bar_q);
            for (int i = 0; i < rb; ++i)
                tma_load_2d(q_s + (qb + i) * L::qblock, &map_q, h * (dim + rot) + dim + 64 * i, b * p.T + r0, sbase + L::bar_q);
            const int len = p.start + p.T;
            for (int j = 0; j < n_tiles && ok; ++j) {
                if (j > 0) ok = wait_or_abort(sbase + L::bar_k_free, (j - 1) & 1, abort_flag);
                if (!ok) break;
                mbar_arrive_expect_tx(sbase + L::bar_k, (qb + rb) * L::kblock);
                for (int i = 0; i < qb; ++i) tma_load_2d(k_s + i * L::kblock, &map_kv, h * dim + 64 * i, b * len + 64 * j, sbase + L::bar_k);
                for (int i = 0; i < rb; ++i)
                    tma_load_2d(k_s + (qb + i) * L::kblock, &map_cache, p.r_at + 64 * i, b * p.slots + 64 * j, sbase + L::bar_k);
                if (j > 0) ok = wait_or_abort(sbase + L::bar_v_free, (j - 1) & 1, abort_flag);
                if (!ok) break;
                mbar_arrive_expect_tx(sbase + L::bar_v, vb * L::kblock);
                for (int i = 0; i < vb; ++i) tma_load_2d(v_s + i * L::kblock, &map_kv, p.off_v + h * vdim + 64 * i, b * len + 64 * j, sbase + L::bar_v);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t id_s = umma_idesc_bf16(128, 64, false), id_o = umma_idesc_bf16(128, vdim, true);
            auto scores = [&](int j) {
                ok = wait_or_abort(sbase + L::bar_k, j & 1, abort_flag);
                if (!ok) return;
                tc_fence_after();
                for (int kk = 0; kk < dim / 16; ++kk)
                    umma_bf16_ss(tmem + 64 * (j & 1), umma_desc_sw128(q_s + (kk >> 2) * L::qblock + (kk & 3) * 32),
                                 umma_desc_sw128(k_s + (kk >> 2) * L::kblock + (kk & 3) * 32), id_s, kk != 0);
                for (int kk = 0; kk < rot / 16; ++kk)
                    umma_bf16_ss(tmem + 64 * (j & 1), umma_desc_sw128(q_s + (qb + (kk >> 2)) * L::qblock + (kk & 3) * 32),
                                 umma_desc_sw128(k_s + (qb + (kk >> 2)) * L::kblock + (kk & 3) * 32), id_s, 1);
                umma_commit(sbase + L::bar_k_free);
                umma_commit(bar_s(j));
            };
            ok = wait_or_abort(sbase + L::bar_q, 0, abort_flag);
            if (ok) scores(0);
            for (int j = 0; j < n_tiles && ok; ++j) {
                if (j + 1 < n_tiles) scores(j + 1);          // its buffer's last weights were read by MMAs issued before
                if (!ok) break;
                ok = wait_or_abort(sbase + L::bar_v, j & 1, abort_flag) && wait_or_abort(bar_p(j), (j >> 1) & 1, abort_flag);
                if (!ok) break;
                tc_fence_after();
                for (int kk = 0; kk < 4; ++kk)               // weights of keys 16 kk: 8 columns
                    umma_bf16_ts(tmem + 128, tmem + 64 * (j & 1) + 8 * kk, umma_desc_mn_sw128(v_s + kk * 2048, L::kblock), id_o, (j | kk) != 0);
                umma_commit(sbase + L::bar_v_free);
            }
            if (ok) umma_commit(sbase + L::bar_o);
        }
    } else {
        const int quarter = warp & 3;
        const uint32_t lanes = (uint32_t)(32 * quarter) << 16;
        const int q = p.start + r0 + 32 * quarter + lane;    // this lane's query position
        const float mul = p.scale * kLog2e;
        float m = p.sink[h] * kLog2e, l = 1.f;
        for (int j = 0; j < n_tiles; ++j) {
            if (ok) ok = wait_or_abort(bar_s(j), (j >> 1) & 1, abort_flag);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            uint32_t sr[2][32];
            tmem_ld32(tmem + lanes + 64 * (j & 1), sr[0]);
            tmem_ld32(tmem + lanes + 64 * (j & 1) + 32, sr[1]);
            const int vis = q + 1 - 64 * j;                  // keys of the tile that this query sees (may be <= 0 or >= 64)
            if (!__all_sync(0xffffffffu, vis >= 64)) {
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (32 * c + i >= vis) sr[c][i] = 0xff800000u;       // -inf
            }
            float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int i = 0; i < 32; ++i) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(sr[c][i]));
            // a negative scale turns the order round; the maximum is then taken of the products
            float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * mul;
            if (mul < 0.f) {
                top = -INFINITY;
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (32 * c + i < vis) top = fmaxf(top, __uint_as_float(sr[c][i]) * mul);
            }
            const bool move = top > m + 8.f;
            if (__any_sync(0xffffffffu, move)) {
                const float mn = move ? top : m, f = ex2_approx(m - mn);
                if (j > 0) {
                    ok = wait_or_abort(sbase + L::bar_v_free, (j - 1) & 1, abort_flag);
                    ok = __all_sync(0xffffffffu, ok);
                    if (!ok) break;
                    tc_fence_after();
                    for (int c = 0; c < vdim; c += 16) {
                        int o[16];
                        uint32_t w[16];
                        tmem_ld16(tmem + lanes + 128 + c, o);
#pragma unroll
                        for (int i = 0; i < 16; ++i) w[i] = __float_as_uint(__int_as_float(o[i]) * f);
                        tmem_st16(tmem + lanes + 128 + c, w);
                    }
                }
                l *= f, m = mn;
            }
            float2 sum = make_float2(0.f, 0.f);
            const float2 mul2v = make_float2(mul, mul), off = make_float2(-m, -m);
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                uint32_t w[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    float2 x = fma2(make_float2(__uint_as_float(sr[c][2 * i]), __uint_as_float(sr[c][2 * i + 1])), mul2v, off);
                    if (mul <= 0.f) {                        // a hidden score must stay hidden
                        if (32 * c + 2 * i >= vis) x.x = -INFINITY;
                        if (32 * c + 2 * i + 1 >= vis) x.y = -INFINITY;
                    }
                    x.x = ex2_approx(x.x), x.y = ex2_approx(x.y);
                    sum = add2(sum, x);
                    w[i] = pack_bf16(x.x, x.y);
                }
                tmem_st16(tmem + lanes + 64 * (j & 1) + 16 * c, w);
            }
            l += sum.x + sum.y;
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_p(j));
        }
        if (ok) ok = wait_or_abort(sbase + L::bar_o, 0, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            tc_fence_after();
            const int r = 32 * quarter + lane;
            const bool live = r < rows;
            const float inv = 1.f / l;
            bf16* y = reinterpret_cast<bf16*>(p.y) + ((size_t)b * p.T + r0 + (live ? r : 0)) * ((size_t)p.H * vdim) + h * vdim;
            for (int c = 0; c < vdim; c += 16) {
                int o[16];
                tmem_ld16(tmem + lanes + 128 + c, o);
                uint32_t out[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) out[i] = pack_bf16(__int_as_float(o[2 * i]) * inv, __int_as_float(o[2 * i + 1]) * inv);
                if (live) {
                    stg_128(y + c, make_uint4(out[0], out[1], out[2], out[3]));
                    stg_128(y + c + 8, make_uint4(out[4], out[5], out[6], out[7]));
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag && tid == 0) atomicExch(&g_decoder_status, DECODER_WAIT_TIMEOUT);
    if (warp == 1) tmem_dealloc(tmem, 256);
}

}  // namespace tsp
