// Grouped dense bf16 GEMM on the tensor cores of sm_100a: rows sorted by group, every group with its own weights,
//   out[row][n] = epilogue(sum_k A[row][k] W[group of row][n][k]),
// the plain product or the activation of a gated feed-forward (gate and up rows of W in blocks of eight, gate.cuh).
//
// Persistent: one CTA per SM walks the tiles of 128 rows x 256 weight rows.  A group's rows start anywhere: its tiles
// start at its first row, and what a tile reads beyond its last one is computed and dropped.  The rows per group are
// read on the device.  Operands by TMA (128-byte swizzle, no multicast), four stages of 64 k; tcgen05.mma kind::f16
// 128 x 256 x 16; two accumulators of 256 columns in tensor memory, so that a tile's epilogue runs under the next
// tile's MMAs.  Roles: warp 0 TMA, warp 1 MMA issue and tensor memory, warps 2-5 epilogue, one row per lane.
// Every wait is bounded.
#pragma once
#include "decoder_status.cuh"
#include "gate.cuh"
#include "tcgen05_sm100.cuh"

namespace tsp {

typedef decoder_group_gemm_args GroupGemmParams;
constexpr int kGroupMax = 1024;

struct GroupGemmSmem {
    static constexpr int threads = 192, stages = 4, a_bytes = 128 * 128, b_bytes = 256 * 128;
    static constexpr int bar_full = 0, bar_empty = 32, bar_acc_full = 64, bar_acc_empty = 80, tmem_slot = 96, abort_flag = 100;
    static constexpr int first = 128, tiles = first + (kGroupMax + 1) * 4;          // prefix sums of rows and of row tiles
    static constexpr int a = (tiles + (kGroupMax + 1) * 4 + 1023) / 1024 * 1024, b = a + stages * a_bytes;
    static constexpr int total = 1024 + b + stages * b_bytes;
};

__global__ void __launch_bounds__(GroupGemmSmem::threads, 1)
    group_gemm_kernel(const GroupGemmParams p, const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w) {
    using L = GroupGemmSmem;
    extern __shared__ __align__(128) uint8_t group_smem[];
    const uint32_t dyn = smem_u32(group_smem), sbase = (dyn + 1023u) & ~1023u;
    uint8_t* base = group_smem + (sbase - dyn);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(base + L::abort_flag);
    int *first = reinterpret_cast<int*>(base + L::first), *tile0 = reinterpret_cast<int*>(base + L::tiles);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    auto bar_full = [&](int s) { return sbase + L::bar_full + 8 * s; };
    auto bar_empty = [&](int s) { return sbase + L::bar_empty + 8 * s; };
    auto bar_acc_full = [&](int i) { return sbase + L::bar_acc_full + 8 * i; };
    auto bar_acc_empty = [&](int i) { return sbase + L::bar_acc_empty + 8 * i; };
    if (tid == 0) {
        for (int s = 0; s < L::stages; ++s) mbar_init(bar_full(s), 1), mbar_init(bar_empty(s), 1);
        for (int i = 0; i < 2; ++i) mbar_init(bar_acc_full(i), 1), mbar_init(bar_acc_empty(i), 4);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc(sbase + L::tmem_slot, 512);
    if (warp == 2) {                                         // prefix sums over the groups
        int rows = 0, tiles = 0;
        for (int g0 = 0; g0 < p.groups; g0 += 32) {
            const int g = g0 + lane, c = g < p.groups ? (p.counts ? __ldcg(p.counts + g) : p.rows) : 0;
            int r = c, t = (c + 127) >> 7;
#pragma unroll
            for (int d = 1; d < 32; d <<= 1) {
                const int ro = __shfl_up_sync(0xffffffffu, r, d), to = __shfl_up_sync(0xffffffffu, t, d);
                if (lane >= d) r += ro, t += to;
            }
            if (g < p.groups) first[g + 1] = rows + r, tile0[g + 1] = tiles + t;
            rows += __shfl_sync(0xffffffffu, r, 31), tiles += __shfl_sync(0xffffffffu, t, 31);
        }
        if (lane == 0) first[0] = 0, tile0[0] = 0;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(base + L::tmem_slot);
    const int KS = (p.K + 63) >> 6, n_tiles = (p.N + 255) >> 8, total = tile0[p.groups] * n_tiles;
    bool ok = true;
    // tile number -> group, first row, first weight row; row tiles of a group next to one another
    int grp = 0;
    auto locate = [&](int tile, int& row, int& n0, int& end) {
        while (tile >= tile0[grp + 1] * n_tiles) ++grp;
        const int mt = tile0[grp + 1] - tile0[grp], rest = tile - tile0[grp] * n_tiles;
        row = first[grp] + rest % mt * 128, n0 = rest / mt * 256, end = first[grp + 1];
    };

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
                int row, n0, end;
                locate(tile, row, n0, end);
                for (int ks = 0; ks < KS; ++ks, ++it) {
                    const int s = it % L::stages, use = it / L::stages;
                    if (use > 0) ok = wait_or_abort(bar_empty(s), (use - 1) & 1, abort_flag);
                    if (!ok) break;
                    mbar_arrive_expect_tx(bar_full(s), L::a_bytes + L::b_bytes);
                    tma_load_2d(sbase + L::a + s * L::a_bytes, &map_a, 64 * ks, row, bar_full(s));
                    tma_load_2d(sbase + L::b + s * L::b_bytes, &map_w, 64 * ks, grp * p.N + n0, bar_full(s));
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(128, 256, false);
            int it = 0, n = 0;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x, ++n) {
                if (n > 1) ok = wait_or_abort(bar_acc_empty(n & 1), ((n >> 1) - 1) & 1, abort_flag);
                if (!ok) break;
                tc_fence_after();
                for (int ks = 0; ks < KS; ++ks, ++it) {
                    const int s = it % L::stages, use = it / L::stages;
                    ok = wait_or_abort(bar_full(s), use & 1, abort_flag);
                    if (!ok) break;
                    tc_fence_after();
#pragma unroll
                    for (int j = 0; j < 4; ++j)
                        umma_bf16_ss(tmem + 256 * (n & 1), umma_desc_sw128(sbase + L::a + s * L::a_bytes + 32 * j),
                                     umma_desc_sw128(sbase + L::b + s * L::b_bytes + 32 * j), idesc, (ks | j) != 0);
                    umma_commit(bar_empty(s));
                }
                if (ok) umma_commit(bar_acc_full(n & 1));
            }
        }
    } else {
        const int quarter = warp & 3;
        const uint32_t lanes = (uint32_t)(32 * quarter) << 16;
        const bool act = p.gate.kind != 0;
        const int ldo = act ? p.N / 2 : p.N;
        int n = 0;
        for (int tile = blockIdx.x; tile < total; tile += gridDim.x, ++n) {
            int row, n0, end;
            locate(tile, row, n0, end);
            ok = wait_or_abort(bar_acc_full(n & 1), (n >> 1) & 1, abort_flag);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const int r = row + 32 * quarter + lane;
            const bool live = r < end;
            const int cols = min(256, p.N - n0);
            bf16* out = reinterpret_cast<bf16*>(p.out) + (size_t)(live ? r : 0) * ldo + (act ? n0 / 2 : n0);
            const float* bias = p.bias ? p.bias + (size_t)grp * p.N + n0 : nullptr;
#pragma unroll 1
            for (int c = 0; c < cols; c += 32) {             // N is a multiple of 16: the second half may be missing
                uint32_t v[32];
                tmem_ld32(tmem + lanes + 256 * (n & 1) + c, v);
                const bool both = c + 16 < cols;
                if (bias)
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (i < 16 || both) v[i] = __float_as_uint(__uint_as_float(v[i]) + bias[c + i]);
                if (act) {
                    uint32_t o[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const int at = i / 4 * 16 + i % 4 * 2;
                        o[i] = pack_bf16(gated(__uint_as_float(v[at]), __uint_as_float(v[at + 8]), p.gate),
                                         gated(__uint_as_float(v[at + 1]), __uint_as_float(v[at + 9]), p.gate));
                    }
                    if (live) {
                        stg_128(out + c / 2, make_uint4(o[0], o[1], o[2], o[3]));
                        if (both) stg_128(out + c / 2 + 8, make_uint4(o[4], o[5], o[6], o[7]));
                    }
                } else if (live) {
                    uint32_t o[16];
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = pack_bf16(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]));
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (i < 2 || both) stg_128(out + c + 8 * i, make_uint4(o[4 * i], o[4 * i + 1], o[4 * i + 2], o[4 * i + 3]));
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_acc_empty(n & 1));
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag && tid == 0) atomicExch(&g_decoder_status, DECODER_WAIT_TIMEOUT);
    if (warp == 1) tmem_dealloc(tmem, 512);
}

}  // namespace tsp
