// liblatentops.so for NVIDIA B200 (sm_100a): the parts of include/decoder_ops.h for the wkv recurrence, attention over a
// shared latent and mixtures of experts.
#include "decoder_launch.cuh"
#include "group_gemm_tc.cuh"
#include "latent_attn.cuh"
#include "latent_attn_tc.cuh"
#include "moe.cuh"
#include "wkv.cuh"

namespace tsp {

template <typename A, int RL, int RPL, int CPT>
static int wkv_scan(const WkvParams& p, int pdl, void* stream) {
    using L = WkvShape<RL, RPL, CPT>;
    const dim3 grid((p.dv + L::cols - 1) / L::cols, p.H, p.B * p.n_seg);
    if (p.n_seg > 1) {
        int rc = launch(wkv_scan_kernel<A, RL, RPL, CPT, false>, grid, 128, L::smem, pdl, stream, 1, p);
        if (rc) return rc;
        rc = launch(wkv_carry_kernel, dim3((p.dk * p.dv + 255) / 256, p.B * p.H), 256, 0, pdl, stream, 1, p);
        if (rc) return rc;
    }
    return launch(wkv_scan_kernel<A, RL, RPL, CPT, true>, grid, 128, L::smem, pdl, stream, 1, p);
}

template <typename A>
static int wkv_prompt(const WkvParams& p, int pdl, void* stream) {
    int rc;
    if (p.dk <= 32) rc = wkv_scan<A, 8, 4, 2>(p, pdl, stream);
    else if (p.dk <= 64) rc = wkv_scan<A, 8, 8, 4>(p, pdl, stream);
    else if (p.dk <= 128) rc = wkv_scan<A, 16, 8, 4>(p, pdl, stream);
    else rc = wkv_scan<A, 32, 8, 4>(p, pdl, stream);
    if (rc) return rc;
    const long long units = (long long)p.B * p.T * p.H;
    const bool quads = p.dv >= 4 && p.dv <= 128 && (p.dv & (p.dv - 1)) == 0;
    if (quads && p.ld % 4 == 0 && !misaligned(p.g, 16) && !misaligned(p.y, 16) && !misaligned(p.norm, 16))
        return launch(wkv_finish4_kernel<A>, dim3((unsigned)((units * p.dv + 2047) / 2048)), 256, 0, pdl, stream, 1, p);
    return launch(wkv_finish_kernel<A>, dim3((unsigned)((units + 7) / 8)), 256, 0, pdl, stream, 1, p);
}

template <typename A, int NR>
static int wkv_one_n(const WkvParams& p, int dvp, int pdl, void* stream) {
    const int words = p.dk * (p.rank / 8);
    const bool wide = sizeof(A) == 2 && p.rank % 8 == 0 && words <= 4 * kWkvThreads && !misaligned(p.w2, 16);
    const size_t smem = ((size_t)4 * p.dk + (p.rank + 3) / 4 * 4 + std::max(kWkvThreads, wide ? words : 0)) * 4;
    const dim3 grid(p.H, p.B);
    if constexpr (sizeof(A) == 2) {
        if (wide && words <= kWkvThreads) return launch(wkv_step_kernel<A, NR, 1>, grid, kWkvThreads, smem, pdl, stream, 1, p, dvp);
        if (wide) return launch(wkv_step_kernel<A, NR, 4>, grid, kWkvThreads, smem, pdl, stream, 1, p, dvp);
    }
    return launch(wkv_step_kernel<A, NR, 0>, grid, kWkvThreads, smem, pdl, stream, 1, p, dvp);
}

template <typename A>
static int wkv_one(const WkvParams& p, int pdl, void* stream) {
    int dvp = 32;
    while (dvp < p.dv) dvp <<= 1;
    const int rows = (p.dk + kWkvThreads / dvp - 1) / (kWkvThreads / dvp);
    if (rows <= 8) return wkv_one_n<A, 8>(p, dvp, pdl, stream);
    if (rows <= 32) return wkv_one_n<A, 32>(p, dvp, pdl, stream);
    return wkv_one_n<A, 0>(p, dvp, pdl, stream);
}

constexpr int kLatentSmemLimit = 227 * 1024;

template <int NT, int MT>
static int latent_step_m(const LatentAttnParams& p, const CUtensorMap& map, int pdl, void* stream) {
    CUtensorMap map_q;
    if (!encode_rows(&map_q, p.qa, (long long)p.B * p.T * p.H, p.ld, p.ld, 16 * MT)) return bad(DECODER_LAUNCH, "latent_step: tensor map refused");
    const dim3 grid(p.splits * p.cluster, (p.H + 16 * MT - 1) / (16 * MT), p.B * p.T);
    return launch(latent_step_kernel<NT, MT>, grid, 256, (size_t)LatentStepSmem(p.ld, MT, kLatentSmemLimit).total, pdl, stream, p.cluster, p, kLatentSmemLimit, map_q, map);
}
template <int NT>
static int latent_step(const LatentAttnParams& p, const CUtensorMap& map, int pdl, void* stream) {
    if constexpr (NT <= 4)
        if (p.H > 16 && LatentStepSmem(p.ld, 2, kLatentSmemLimit).total <= kLatentSmemLimit) return latent_step_m<NT, 2>(p, map, pdl, stream);
    return latent_step_m<NT, 1>(p, map, pdl, stream);
}

template <int RW>
static int latent_join(const LatentAttnParams& p, int pdl, void* stream) {
    const int M = p.B * p.T;
    const dim3 grid((p.vdim + 31) / 32, p.H, M);
    if (M == 1) return launch(latent_join_kernel<RW, 1>, grid, 256, (size_t)p.R * 4, pdl, stream, 1, p);
    return launch(latent_join_kernel<RW, 4>, dim3(grid.x, grid.y, (M + 3) / 4), 256, (size_t)p.R * 16, pdl, stream, 1, p);
}

}  // namespace tsp

using namespace tsp;

extern "C" int decoder_latent_status(void) { return read_decoder_status(); }

extern "C" int decoder_wkv(const decoder_wkv_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->dk < 1 || a->dv < 1 || a->rank < 1 || a->dk > 256 || a->dv > 512)
        return bad(DECODER_BAD_SHAPE, "wkv: 1 <= dk <= 256, 1 <= dv <= 512");
    if (a->T > 1 && (a->n_seg < 1 || a->seg_len < 1 || (a->n_seg > 1 && a->seg_len % kWkvChunk) || (long long)a->n_seg * a->seg_len < a->T ||
                     (long long)(a->n_seg - 1) * a->seg_len >= a->T))
        return bad(DECODER_BAD_SHAPE, "wkv: the segments do not cover the portion");
    if (!a->r || !a->k || !a->v || !a->g || !a->w0 || !a->u || !a->norm || !a->pos || !a->state || !a->y ||
        (a->T > 1 ? !a->zw || !a->o || misaligned(a->o, 16) || (a->n_seg > 1 && !a->part) : !a->w2 || !a->t1))
        return bad(DECODER_BAD_POINTER, "wkv: null or misaligned pointer");
    if (a->T == 1) return dtype ? wkv_one<float>(*a, pdl, stream) : wkv_one<bf16>(*a, pdl, stream);
    return dtype ? wkv_prompt<float>(*a, pdl, stream) : wkv_prompt<bf16>(*a, pdl, stream);
}

extern "C" int decoder_latent_prep(const decoder_latent_prep_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->q_rank < 1 || a->off_q < 0 || a->off_q + a->q_rank > a->ld_z) return bad(DECODER_BAD_SHAPE, "latent_prep: columns outside the row");
    if (a->cache && (a->R < 1 || a->rot < 0 || a->dims < 0 || a->dims % 2 || a->dims > a->rot || a->r_at < a->R || a->r_at + a->rot > a->ld ||
                     a->off_kv < 0 || a->off_kv + a->R + a->rot > a->ld_z || a->slots < 1))
        return bad(DECODER_BAD_SHAPE, "latent_prep: cache layout");
    if (!a->z || !a->cq || !a->q_norm || !a->pos || (a->cache && (!a->kv_norm || (a->dims && !a->trig)))) return bad(DECODER_BAD_POINTER, "latent_prep: null pointer");
    const dim3 grid((unsigned)(a->B * a->T));
    const size_t smem = (size_t)(a->q_rank + (a->cache ? a->R + a->rot : 0)) * 4;
    if (smem > 200 * 1024) return bad(DECODER_BAD_SHAPE, "latent_prep: rows of at most 51200");
    return dtype ? launch(latent_prep_kernel<float>, grid, 256, smem, pdl, stream, 1, *a) : launch(latent_prep_kernel<bf16>, grid, 256, smem, pdl, stream, 1, *a);
}

extern "C" int decoder_rotate(const decoder_rotate_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->rot < 1 || a->dims < 0 || a->dims % 2 || a->dims > a->rot) return bad(DECODER_BAD_SHAPE, "rotate: dims even, at most rot");
    if (!a->src || !a->dst || !a->pos || (a->dims && !a->trig)) return bad(DECODER_BAD_POINTER, "rotate: null pointer");
    const long long n = (long long)a->B * a->T * a->H * ((a->rot + 1) / 2);
    const dim3 grid((unsigned)std::min<long long>((n + 255) / 256, 16ll * sm_count()));
    return dtype ? launch(rotate_kernel<float>, grid, 256, 0, pdl, stream, 1, *a) : launch(rotate_kernel<bf16>, grid, 256, 0, pdl, stream, 1, *a);
}

extern "C" int decoder_absorb(const decoder_absorb_args* a, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->B * a->T > 8 || a->H < 1 || a->dim < 8 || a->dim % 8 || a->R < 1 || a->rot < 0 || a->rot % 8 || a->dims % 2 || a->dims > a->rot ||
        a->r_at < a->R || a->r_at + a->rot > a->ld)
        return bad(DECODER_BAD_SHAPE, "absorb: up to 8 rows, dim and rot multiples of 8");
    if (!a->q || !a->w_uk_t || !a->qa || !a->pos || misaligned(a->q, 16) || misaligned(a->w_uk_t, 16) || (a->dims && !a->trig)) return bad(DECODER_BAD_POINTER, "absorb: null or misaligned pointer");
    return launch(absorb_kernel, dim3((a->R + 127) / 128 + 1, a->H), 256, 0, pdl, stream, 1, *a);
}

static int latent_attn_check(const decoder_latent_attn_args* a) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->R < 1 || a->ld < a->R || a->ld % 8 || a->slots < 1) return bad(DECODER_BAD_SHAPE, "latent_attn: cache layout");
    if (!a->qa || !a->cache || !a->sink || !a->pos || misaligned(a->cache, 16) || misaligned(a->qa, 16)) return bad(DECODER_BAD_POINTER, "latent_attn: null or misaligned pointer");
    return DECODER_OK;
}

extern "C" int decoder_latent_attn(const decoder_latent_attn_args* a, int dtype, int pdl, void* stream) {
    if (int rc = latent_attn_check(a)) return rc;
    if (a->ld > 8192) return bad(DECODER_BAD_SHAPE, "latent_attn: rows of at most 8192");
    if (!a->out) return bad(DECODER_BAD_POINTER, "latent_attn: null pointer");
    const dim3 grid((unsigned)(a->B * a->T), a->H);
    const size_t smem = (size_t)(a->ld + a->R) * 4;
    return dtype ? launch(latent_attn_plain_kernel<float>, grid, 128, smem, pdl, stream, 1, *a) : launch(latent_attn_plain_kernel<bf16>, grid, 128, smem, pdl, stream, 1, *a);
}

extern "C" int decoder_latent_step_width(void) {
    int ld = 8;
    while (LatentStepSmem(ld + 8, 1, kLatentSmemLimit).total <= kLatentSmemLimit) ld += 8;
    return ld;
}

extern "C" int decoder_latent_step(const decoder_latent_attn_args* a, int pdl, void* stream) {
    if (int rc = latent_attn_check(a)) return rc;
    if (a->R % 8 || a->R > 1024 || a->splits < 1 || a->splits > 1024 || a->cluster < 1 || a->cluster > 8 || a->vdim < 1 ||
        LatentStepSmem(a->ld, 1, kLatentSmemLimit).total > kLatentSmemLimit)
        return bad(DECODER_BAD_SHAPE, "latent_step: R a multiple of 8 up to 1024, rows that fit shared memory");
    if (!a->part || !a->ml || !a->w_uv || !a->y || misaligned(a->w_uv, 16)) return bad(DECODER_BAD_POINTER, "latent_step: null or misaligned pointer");
    CUtensorMap map;
    if (!encode_rows(&map, a->cache, (long long)a->B * a->slots, a->ld, a->ld, 32)) return bad(DECODER_LAUNCH, "latent_step: tensor map refused");
    const int rc = a->R <= 128   ? latent_step<1>(*a, map, pdl, stream)
                   : a->R <= 256 ? latent_step<2>(*a, map, pdl, stream)
                   : a->R <= 512 ? latent_step<4>(*a, map, pdl, stream)
                                 : latent_step<8>(*a, map, pdl, stream);
    if (rc) return rc;
    if (a->R <= 256) return latent_join<1>(*a, pdl, stream);
    if (a->R <= 512) return latent_join<2>(*a, pdl, stream);
    return latent_join<4>(*a, pdl, stream);
}

extern "C" int decoder_latent_prompt(const decoder_latent_prompt_args* a, void* stream) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->start < 0 || a->start + a->T > a->slots || a->dim < 16 || a->rot < 16 || a->vdim < 16 || a->dim % 16 ||
        a->rot % 16 || a->vdim % 16 || a->dim > 128 || a->vdim > 128 || a->rot > 64 || a->ld % 8 || a->r_at % 8 || a->ld_kv % 8 || a->off_v % 8 ||
        a->r_at + a->rot > a->ld)
        return bad(DECODER_BAD_SHAPE, "latent_prompt: dim and vdim multiples of 16 up to 128, rot up to 64");
    if (!a->q || !a->kv || !a->cache || !a->sink || !a->y || misaligned(a->q, 16) || misaligned(a->kv, 16) || misaligned(a->cache, 16) || misaligned(a->y, 16))
        return bad(DECODER_BAD_POINTER, "latent_prompt: null or misaligned pointer");
    CUtensorMap q, kv, cache;
    const long long ld_q = (long long)a->H * (a->dim + a->rot), len = a->start + a->T;
    if (!encode_rows(&q, a->q, (long long)a->B * a->T, ld_q, ld_q, 128) || !encode_rows(&kv, a->kv, a->B * len, a->ld_kv, a->ld_kv, 64) ||
        !encode_rows(&cache, a->cache, (long long)a->B * a->slots, a->ld, a->ld, 64))
        return bad(DECODER_LAUNCH, "latent_prompt: tensor map refused");
    const int smem = LatentTcSmem::total((a->dim + 63) / 64, (a->rot + 63) / 64, (a->vdim + 63) / 64);
    return launch(latent_attn_tc_kernel, dim3((a->T + 127) / 128, a->H, a->B), LatentTcSmem::threads, (size_t)smem, 0, stream, 1, *a, q, kv, cache);
}

static int moe_check(const decoder_moe_args* a) {
    if (a->M < 1 || a->E < 1 || a->E > kMoeMaxExperts || a->top < 1 || a->top > kMoeMaxTop || a->top > a->E || a->K < 1 || a->ff < 8 || a->ff % 8)
        return bad(DECODER_BAD_SHAPE, "moe: top <= min(32, E), E <= 1024, ff a multiple of 8");
    return DECODER_OK;
}

extern "C" int decoder_moe_route(const decoder_moe_args* a, int pdl, void* stream) {
    if (int rc = moe_check(a)) return rc;
    if (!a->logits || !a->router_bias || !a->chosen || !a->weight) return bad(DECODER_BAD_POINTER, "moe_route: null pointer");
    int rc = launch(route_kernel, dim3((a->M + 31) / 32), 1024, (size_t)33 * a->E * 4, pdl, stream, 1, *a);
    if (rc || !a->counts) return rc;
    if (a->K % 8) return bad(DECODER_BAD_SHAPE, "moe_route: K a multiple of 8");
    if (!a->rank || !a->slots || !a->x || !a->sorted || misaligned(a->x, 16) || misaligned(a->sorted, 16)) return bad(DECODER_BAD_POINTER, "moe_route: null or misaligned pointer");
    return launch(sort_rows_kernel, dim3((unsigned)(((long long)a->M * a->top + 7) / 8)), 256, 0, pdl, stream, 1, *a);
}

extern "C" int decoder_moe_plain(const decoder_moe_args* a, int dtype, int pdl, void* stream) {
    if (int rc = moe_check(a)) return rc;
    if (a->D < 1 || a->gate.kind < 1 || a->gate.kind > 2) return bad(DECODER_BAD_SHAPE, "moe_plain: empty shape");
    if (!a->chosen || !a->x || !a->w_up || !a->act || !a->w_down || !a->out) return bad(DECODER_BAD_POINTER, "moe_plain: null pointer");
    const unsigned n = (unsigned)(a->M * a->top);
    const dim3 up(n, (a->ff + 63) / 64), down(n, (a->D + 63) / 64);
    int rc = dtype ? launch(moe_up_plain_kernel<float>, up, 256, 0, pdl, stream, 1, *a) : launch(moe_up_plain_kernel<bf16>, up, 256, 0, pdl, stream, 1, *a);
    if (rc) return rc;
    return dtype ? launch(moe_down_plain_kernel<float>, down, 256, 0, pdl, stream, 1, *a) : launch(moe_down_plain_kernel<bf16>, down, 256, 0, pdl, stream, 1, *a);
}

template <int P>
static int moe_up_step(const MoeParams& p, int pdl, void* stream) {
    const int items = p.ff / 8 * std::min(p.E, p.M * p.top);
    return launch(moe_up_step_kernel<P>, dim3(std::min(items, 2 * sm_count())), kRowsWarps * 32, (size_t)p.M * (p.K * 2 + 64 + p.E * 4), pdl, stream, 1, p);
}

extern "C" int decoder_moe_up_step(const decoder_moe_args* a, int pdl, void* stream) {
    if (int rc = moe_check(a)) return rc;
    if (a->M > 8 || a->K % 8 || a->K > 12288 || a->gate.kind < 1 || a->gate.kind > 2) return bad(DECODER_BAD_SHAPE, "moe_up_step: M <= 8, K a multiple of 8 up to 12288");
    if (!a->logits || !a->router_bias || !a->chosen || !a->weight || !a->ticket || !a->x || !a->w_up || !a->act || misaligned(a->x, 16) ||
        misaligned(a->w_up, 16))
        return bad(DECODER_BAD_POINTER, "moe_up_step: null or misaligned pointer");
    // k-steps in flight: what leaves the last batch of a warp's share the fullest
    const int steps = ((a->K + 31) / 32 + kRowsWarps - 1) / kRowsWarps;
    const auto waste = [&](int n) { return (steps + n - 1) / n * n - steps; };
    if (waste(8) <= waste(6) && waste(8) <= waste(5)) return moe_up_step<8>(*a, pdl, stream);
    return waste(6) <= waste(5) ? moe_up_step<6>(*a, pdl, stream) : moe_up_step<5>(*a, pdl, stream);
}

extern "C" int decoder_moe_down_step(const decoder_moe_args* a, int pdl, void* stream) {
    if (a->M < 1 || a->M > 8 || a->D < 1 || (!a->w_down && !a->w_rest) || (a->w_down && (a->ff < 8 || a->ff % 8)) || (a->w_rest && (a->K_rest < 8 || a->K_rest % 8)) ||
        (a->weight && (a->E < 1 || a->E > kMoeMaxExperts || a->top < 1 || a->top > kMoeMaxTop)))
        return bad(DECODER_BAD_SHAPE, "moe_down_step: M <= 8, ff and K_rest multiples of 8");
    if (!a->out || (a->w_down && (!a->act || misaligned(a->w_down, 16) || misaligned(a->act, 16))) ||
        (a->w_rest && (!a->rest || misaligned(a->w_rest, 16) || misaligned(a->rest, 16))) || (a->weight && (!a->chosen || !a->w_down)))
        return bad(DECODER_BAD_POINTER, "moe_down_step: null or misaligned pointer");
    return launch(moe_down_step_kernel, dim3((a->D + 15) / 16), kRowsWarps * 32, 0, pdl, stream, 1, *a);
}

extern "C" int decoder_group_gemm(const decoder_group_gemm_args* a, void* stream) {
    if (a->rows < 1 || a->groups < 1 || a->groups > kGroupMax || a->N < 16 || a->N % 16 || a->K < 8 || a->K % 8 || a->gate.kind < 0 || a->gate.kind > 2 ||
        (!a->counts && a->groups != 1))
        return bad(DECODER_BAD_SHAPE, "group_gemm: N a multiple of 16, K of 8");
    if (!a->a || !a->w || !a->out || misaligned(a->a, 16) || misaligned(a->w, 16) || misaligned(a->out, 16)) return bad(DECODER_BAD_POINTER, "group_gemm: null or misaligned pointer");
    CUtensorMap ma, mw;
    if (!encode_rows(&ma, a->a, a->rows, a->K, a->K, 32) || !encode_rows(&mw, a->w, (long long)a->groups * a->N, a->K, a->K, 128))
        return bad(DECODER_LAUNCH, "group_gemm: tensor map refused");
    return launch(group_gemm_kernel, dim3(sm_count() & ~1), GroupGemmSmem::threads, (size_t)GroupGemmSmem::total, 0, stream, 2, *a, ma, mw);
}
