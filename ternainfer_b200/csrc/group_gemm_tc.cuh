// Grouped dense bf16 GEMM on the tensor cores of sm_100a: rows sorted by group, every group with its own weights,
//   out[row][n] = epilogue(sum_k A[row][k] W[group of row][n][k]),
// the plain product or the activation of a gated feed-forward (gate and up rows of W in blocks of eight, gate.cuh).
//
// CTA pairs (tcgen05.mma.cta_group::2): a tile is 256 rows of W by up to 256 rows of A.  W's rows are the MMA's M - 128
// per CTA - and A's its N, a multiple of 64 that is chosen for every tile, so that a group of a few rows or of a few more
// than 256 wastes little; a CTA holds half of both operands in shared memory and the results of its 128 rows of W
// in tensor memory.  Persistent: pairs walk the tiles, row tiles of a group next to one another.  The rows per group
// are read on the device; a group's rows start anywhere, and what a tile reads beyond its group is dropped.
// Operands by TMA (128-byte swizzle, no multicast), six stages of 64 k; two accumulators, so that a tile's epilogue runs
// under the next tile's MMAs.  Roles per CTA: warp 0 TMA, warp 1 tensor memory and (leader) MMA issue, warps 2-9
// epilogue: gate and up meet by a shuffle, 16 rows of A at a time are transposed through shared memory and
// stored 16 bytes per lane.  Every wait is bounded.
#pragma once
#include "decoder_status.cuh"
#include "gate.cuh"
#include "tcgen05_sm100.cuh"

namespace tsp {

typedef decoder_group_gemm_args GroupGemmParams;
constexpr int kGroupMax = 1024;

struct GroupGemmSmem {
    static constexpr int epi_warps = 8, threads = 64 + 32 * epi_warps, stages = 6, half = 128 * 128;   // bytes: 128 rows of 64 bf16
    static constexpr int bar_full = 0, bar_empty = 48, bar_acc_full = 96, bar_acc_empty = 112, tmem_slot = 128, abort_flag = 132;
    static constexpr int first = 256, tiles = first + (kGroupMax + 1) * 4;          // prefix sums of rows and of row tiles
    static constexpr int stage_out = (tiles + (kGroupMax + 1) * 4 + 15) / 16 * 16;  // 1 KB per epilogue warp
    static constexpr int a = (stage_out + epi_warps * 1024 + 1023) / 1024 * 1024, b = a + stages * half;
    static constexpr int total = 1024 + b + stages * half;
};

__global__ void __launch_bounds__(GroupGemmSmem::threads, 1)
    group_gemm_kernel(const GroupGemmParams p, const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w) {
    using L = GroupGemmSmem;
    extern __shared__ __align__(128) uint8_t group_smem[];
    const uint32_t dyn = smem_u32(group_smem), sbase = (dyn + 1023u) & ~1023u;      // the same offset in both CTAs of the pair
    uint8_t* base = group_smem + (sbase - dyn);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(base + L::abort_flag);
    int *first = reinterpret_cast<int*>(base + L::first), *tile0 = reinterpret_cast<int*>(base + L::tiles);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t crank = cluster_ctarank();                // 0 = leader
    const int pair = (int)blockIdx.x >> 1, npairs = (int)gridDim.x >> 1;
    auto bar_full = [&](int s) { return sbase + L::bar_full + 8 * s; };
    auto bar_empty = [&](int s) { return sbase + L::bar_empty + 8 * s; };
    auto bar_acc_full = [&](int i) { return sbase + L::bar_acc_full + 8 * i; };
    auto bar_acc_empty = [&](int i) { return sbase + L::bar_acc_empty + 8 * i; };
    if (tid == 0) {
        for (int s = 0; s < L::stages; ++s) mbar_init(bar_full(s), 1), mbar_init(bar_empty(s), 1);
        for (int i = 0; i < 2; ++i) mbar_init(bar_acc_full(i), 1), mbar_init(bar_acc_empty(i), 2 * L::epi_warps);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc_pair(sbase + L::tmem_slot, 512);
    if (warp == 2) {                                         // prefix sums over the groups
        int rows = 0, tiles = 0;
        for (int g0 = 0; g0 < p.groups; g0 += 32) {
            const int g = g0 + lane, c = g < p.groups ? (p.counts ? __ldcg(p.counts + g) : p.rows) : 0;
            int r = c, t = (c + 255) >> 8;
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
    cluster_arrive();                                        // the peer's barriers exist before anything is sent to them
    cluster_wait();
    tc_fence_after();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(base + L::tmem_slot);
    const int KS = (p.K + 63) >> 6, n_tiles = (p.N + 255) >> 8, total = tile0[p.groups] * n_tiles;
    bool ok = true;
    // tile number -> group, first row and number of rows (a multiple of 64), first row of W
    int grp = 0;
    struct Tile {
        int row, nt, n0, end;
    };
    auto locate = [&](int tile) {
        while (tile >= tile0[grp + 1] * n_tiles) ++grp;
        const int rt = tile0[grp + 1] - tile0[grp], rest = tile - tile0[grp] * n_tiles, c = first[grp + 1] - first[grp];
        const int nt = ((c + rt - 1) / rt + 63) / 64 * 64;
        return Tile{first[grp] + rest % rt * nt, nt, rest / rt * 256, first[grp + 1]};
    };

    if (warp == 0) {
        // ------------------------------------------------ operand loader (both CTAs)
        if (lane == 0) {
            int it = 0;
            for (int tile = pair; tile < total && ok; tile += npairs) {
                const Tile t = locate(tile);
                const int w_row = grp * p.N + t.n0 + (int)crank * 128, a_row = t.row + (int)crank * (t.nt / 2);
                for (int ks = 0; ks < KS; ++ks, ++it) {
                    const int s = it % L::stages, use = it / L::stages;
                    if (use > 0) ok = wait_or_abort(bar_empty(s), (use - 1) & 1, abort_flag);
                    if (!ok) break;
                    const uint32_t full = map_to_rank(bar_full(s), 0);
                    if (crank == 0) mbar_arrive_expect_tx(bar_full(s), 2 * L::half + t.nt * 128);
                    tma_load_2d_pair(sbase + L::a + s * L::half, &map_w, 64 * ks, w_row, full);
                    for (int i = 0; i < t.nt / 64; ++i) tma_load_2d_pair(sbase + L::b + s * L::half + i * 4096, &map_a, 64 * ks, a_row + 32 * i, full);
                }
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------ MMA issuer (leader only)
        if (lane == 0 && crank == 0) {
            int it = 0, n = 0;
            for (int tile = pair; tile < total && ok; tile += npairs, ++n) {
                const Tile t = locate(tile);
                const uint32_t idesc = umma_idesc_bf16(256, t.nt, false);
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
                        umma_bf16_pair(tmem + 256 * (n & 1), umma_desc_sw128(sbase + L::a + s * L::half + 32 * j),
                                       umma_desc_sw128(sbase + L::b + s * L::half + 32 * j), idesc, (ks | j) != 0);
                    umma_commit_pair(bar_empty(s));          // frees the stage in both CTAs
                }
                if (ok) umma_commit_pair(bar_acc_full(n & 1));
            }
        }
    } else {
        // ---------------------------------------------------------- epilogue (both CTAs, own 128 rows of W)
        const int quarter = warp & 3, side = (warp - 2) >> 2;    // 32 rows of W, half of the rows of A
        const uint32_t lanes = (uint32_t)(32 * quarter) << 16, st = sbase + L::stage_out + (warp - 2) * 1024;
        const bool act = p.gate.kind != 0;
        const int ldo = act ? p.N / 2 : p.N;
        int n = 0;
        for (int tile = pair; tile < total; tile += npairs, ++n) {
            const Tile t = locate(tile);
            ok = wait_or_abort(bar_acc_full(n & 1), (n >> 1) & 1, abort_flag);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const int w0 = t.n0 + (int)crank * 128 + 32 * quarter;   // this warp's first row of W
            const float bias = p.bias && w0 + lane < p.N ? p.bias[(size_t)grp * p.N + w0 + lane] : 0.f;
            const int c0 = side * (t.nt / 2), cols = w0 < p.N ? max(0, min(t.nt / 2, t.end - t.row - c0)) : 0;
#pragma unroll 1
            for (int c32 = 0; c32 < cols; c32 += 32) {       // (the tile's half is a multiple of 32)
                uint32_t v[32];
                tmem_ld32(tmem + lanes + 256 * (n & 1) + c0 + c32, v);
#pragma unroll
                for (int h = 0; h < 32; h += 16) {
                    const int c = c32 + h;
                    __syncwarp();                            // the staging of the slice before has been read
                    if (act) {                               // of two rows of A, the lane with the gate takes one and the lane with up the other
                        const bool hi = lane & 8;
                        const uint32_t at = st + (hi ? 32 : 0) + (lane >> 4) * 16 + (lane & 7) * 2;
#pragma unroll
                        for (int i = 0; i < 16; i += 2) {
                            const float z0 = __uint_as_float(v[h + i]) + bias, z1 = __uint_as_float(v[h + i + 1]) + bias;
                            const float other = __shfl_xor_sync(0xffffffffu, hi ? z0 : z1, 8);
                            sts_b16(at + i * 32, __bfloat16_as_ushort(__float2bfloat16_rn(gated<true>(hi ? other : z0, hi ? z1 : other, p.gate))));
                        }
                        __syncwarp();
                        const int r = lane >> 1, f = w0 / 2 + (lane & 1) * 8;
                        if (c + r < cols && f < ldo)
                            stg_128(reinterpret_cast<bf16*>(p.out) + (size_t)(t.row + c0 + c + r) * ldo + f, lds128(st + r * 32 + (lane & 1) * 16));
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i) sts_b16(st + i * 64 + lane * 2, __bfloat16_as_ushort(__float2bfloat16_rn(__uint_as_float(v[h + i]) + bias)));
                        __syncwarp();
#pragma unroll
                        for (int j = 0; j < 2; ++j) {
                            const int r = (lane >> 2) + 8 * j, f = w0 + (lane & 3) * 8;
                            if (c + r < cols && f < ldo)
                                stg_128(reinterpret_cast<bf16*>(p.out) + (size_t)(t.row + c0 + c + r) * ldo + f, lds128(st + r * 64 + (lane & 3) * 16));
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive_cluster(map_to_rank(bar_acc_empty(n & 1), 0));   // the leader may overwrite this buffer
        }
    }
    if (*abort_flag && tid == 0) atomicExch(&g_decoder_status, DECODER_WAIT_TIMEOUT);
    tc_fence_before();
    __syncthreads();
    cluster_arrive();                                        // neither CTA frees tensor memory or leaves while the other may still signal it
    cluster_wait();
    if (warp == 1) tmem_dealloc_pair(tmem, 512);
}

}  // namespace tsp
