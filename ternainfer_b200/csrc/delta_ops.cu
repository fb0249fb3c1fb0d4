// libdeltaops.so for NVIDIA B200 (sm_100a): the parts of include/decoder_ops.h for the generalised delta rule and
// attention with sigmoid weights.
#include "decoder_launch.cuh"
#include "delta_rule.cuh"
#include "sigmoid_attn.cuh"
#include "sigmoid_attn_tc.cuh"

namespace tsp {

static bool quads(int n) { return n >= 4 && n <= 128 && (n & (n - 1)) == 0; }

template <typename A, int RL, int RPL, int CPT, int CW, int GR>
static int delta_scan(const DeltaParams& p, int pdl, void* stream) {
    using L = ScanShape<RL, RPL, CPT, CW, GR>;
    return launch(delta_scan_kernel<A, RL, RPL, CPT, CW, GR>, dim3((p.dv + L::cols - 1) / L::cols, p.H, p.B), L::threads, L::smem, pdl, stream, 1, p);
}

template <typename A>
static int delta_prompt(const DeltaParams& p, int pdl, void* stream) {
    int rc;
    if (p.dk <= 32) rc = delta_scan<A, 8, 4, 4, 2, 2>(p, pdl, stream);
    else if (p.dk <= 64) rc = delta_scan<A, 16, 4, 2, 8, 2>(p, pdl, stream);
    else if (p.dk <= 128) rc = delta_scan<A, 16, 8, 4, 4, 2>(p, pdl, stream);
    else rc = delta_scan<A, 16, 16, 2, 4, 2>(p, pdl, stream);
    if (rc) return rc;
    const long long units = (long long)p.B * p.T * p.H;
    if (quads(p.dv) && p.ld % 4 == 0 && p.off_g % 4 == 0 && !misaligned(p.proj, 16) && !misaligned(p.y, 16) && !misaligned(p.norm, 16))
        return launch(delta_finish4_kernel<A>, dim3((unsigned)((units * p.dv + 2047) / 2048)), 256, 0, pdl, stream, 1, p);
    return launch(delta_finish_kernel<A>, dim3((unsigned)((units + 7) / 8)), 256, 0, pdl, stream, 1, p);
}

template <typename A, int NR>
static int delta_one_n(const DeltaParams& p, int dvp, int pdl, void* stream) {
    const int words = p.dk * (p.rank / 8);
    const bool wide = sizeof(A) == 2 && p.rank % 8 == 0 && words <= 4 * kStepThreads && !misaligned(p.w2, 16);
    const size_t smem = ((size_t)5 * p.dk + (p.rank + 3) / 4 * 4 + std::max(kStepThreads, wide ? words : 0)) * 4;
    const dim3 grid(p.H, p.B);
    if constexpr (sizeof(A) == 2) {
        if (wide && words <= kStepThreads) return launch(delta_step_kernel<A, NR, 1>, grid, kStepThreads, smem, pdl, stream, 1, p, dvp);
        if (wide) return launch(delta_step_kernel<A, NR, 4>, grid, kStepThreads, smem, pdl, stream, 1, p, dvp);
    }
    return launch(delta_step_kernel<A, NR, 0>, grid, kStepThreads, smem, pdl, stream, 1, p, dvp);
}

template <typename A>
static int delta_one(const DeltaParams& p, int pdl, void* stream) {
    int dvp = 32;
    while (dvp < p.dv) dvp <<= 1;
    const int rows = (p.dk + kStepThreads / dvp - 1) / (kStepThreads / dvp);
    if (rows <= 8) return delta_one_n<A, 8>(p, dvp, pdl, stream);
    if (rows <= 32) return delta_one_n<A, 32>(p, dvp, pdl, stream);
    return delta_one_n<A, 0>(p, dvp, pdl, stream);
}

template <int RT, int LPK>
static int attn_one(const AttnParams& p, int pdl, void* stream) {
    const int rep = p.H / p.G, units = p.G * ((rep + RT - 1) / RT);
    // slices of the slots: as many CTAs as the chip holds at a time, at least 64 slots each
    const int nr = std::max(1, std::min(std::min(8, (RT <= 4 ? 2 : 1) * sm_count() / (units * p.B)), p.slots / 64));
    return launch(sigmoid_attn_step_kernel<RT, LPK>, dim3(nr, units, p.B), 256, 0, pdl, stream, nr, p);
}
template <int LPK>
static int attn_one_l(const AttnParams& p, int pdl, void* stream) {
    const int rep = p.H / p.G;
    if (rep == 1) return attn_one<1, LPK>(p, pdl, stream);
    if (rep == 2) return attn_one<2, LPK>(p, pdl, stream);
    if (rep <= 4 || LPK == 32) return attn_one<4, LPK>(p, pdl, stream);
    if constexpr (LPK <= 16) return attn_one<8, LPK>(p, pdl, stream);
    return DECODER_BAD_SHAPE;
}

// 16-byte starts for every tile, whole MMA steps: what the tensor-core kernel asks of a call
static bool attn_tc_fits(const AttnParams& p) {
    return p.dim % 16 == 0 && p.vdim % 16 == 0 && p.dim <= 128 && p.vdim <= 128 && p.ld % 8 == 0 && p.off_q % 8 == 0 && p.off_k % 8 == 0 &&
           p.off_v % 8 == 0 && p.off_g % 8 == 0 && !misaligned(p.proj, 16) && !misaligned(p.ck, 16) && !misaligned(p.cv, 16) &&
           !misaligned(p.y, 16);
}

static int attn_tc(const AttnParams& p, void* stream) {
    CUtensorMap proj, ck, cv;
    const long long cache_rows = (long long)p.B * p.G * p.slots;
    if (!encode_rows(&proj, p.proj, (long long)p.B * p.T, p.ld, p.ld, 128) || !encode_rows(&ck, p.ck, cache_rows, p.dim, p.dim, 128) ||
        !encode_rows(&cv, p.cv, cache_rows, p.vdim, p.vdim, 128))
        return bad(DECODER_LAUNCH, "attn: tensor map refused");
    const int smem = AttnTcSmem::total((p.dim + 63) / 64, (p.vdim + 63) / 64);
    return launch(sigmoid_attn_tc_kernel, dim3((p.T + 127) / 128, p.H, p.B), AttnTcSmem::threads, (size_t)smem, 0, stream, 1, p, proj, ck, cv);
}

template <typename A>
static int attn_prompt(const AttnParams& p, bool tensor_cores, int pdl, void* stream) {
    const long long units = (long long)p.B * p.T * (p.H + p.G);
    const bool vec = quads(p.dim) && p.ld % 4 == 0 && p.off_q % 4 == 0 && p.off_k == p.off_q + p.H * p.dim && !misaligned(p.proj, 16) &&
                     !misaligned(p.q_norm, 16) && !misaligned(p.k_norm, 16);
    int rc = vec ? launch(head_norm4_kernel<A>, dim3((unsigned)((units * p.dim + 2047) / 2048)), 256, 0, pdl, stream, 1, p)
                 : launch(head_norm_kernel<A>, dim3((unsigned)((units + 7) / 8)), 256, 0, pdl, stream, 1, p);
    if (rc) return rc;
    rc = tensor_cores ? attn_tc(p, stream)
                      : launch(sigmoid_attn_plain_kernel<A>, dim3(p.T, p.H, p.B), 128, (size_t)(p.dim + p.vdim) * 4, pdl, stream, 1, p);
    if (rc) return rc;
    return launch(attn_cache_store_kernel<A>, dim3(std::min(p.T, p.slots), p.B, p.G), 128, 0, pdl, stream, 1, p);
}

}  // namespace tsp

using namespace tsp;

extern "C" int decoder_delta(const decoder_delta_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->dk < 1 || a->dv < 1 || a->rank < 1 || a->dk > 256 || a->dv > 512)
        return bad(DECODER_BAD_SHAPE, "delta: 1 <= dk <= 256, 1 <= dv <= 512");
    if (!a->proj || !a->w0 || !a->a_bias || !a->norm || !a->pos || !a->state || !a->y || (a->T > 1 ? !a->zw || !a->o || misaligned(a->o, 16) : !a->w2))
        return bad(DECODER_BAD_POINTER, "delta: null or misaligned pointer");
    if (a->T == 1) return dtype ? delta_one<float>(*a, pdl, stream) : delta_one<bf16>(*a, pdl, stream);
    return dtype ? delta_prompt<float>(*a, pdl, stream) : delta_prompt<bf16>(*a, pdl, stream);
}

extern "C" int decoder_attn(const decoder_attn_args* a, int dtype, int path, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->G < 1 || a->H % a->G || a->dim < 1 || a->vdim < 1 || a->dim > 4096 || a->vdim > 4096 ||
        a->chunk < 1 || a->slots < 1 || a->slots > a->chunk)
        return bad(DECODER_BAD_SHAPE, "attn: heads a multiple of kv heads, 1 <= slots <= chunk");
    if (!a->proj || !a->ck || !a->cv || !a->q_norm || !a->k_norm || !a->bias || !a->slope || !a->pos || !a->y)
        return bad(DECODER_BAD_POINTER, "attn: null pointer");
    const int widest = std::max(a->dim, a->vdim);
    if (path == 0 && dtype == 0 && a->T == 1 && a->dim % 8 == 0 && a->vdim % 8 == 0 && widest <= 256 && !misaligned(a->ck, 16) &&
        !misaligned(a->cv, 16)) {
        if (widest <= 32) return attn_one_l<4>(*a, pdl, stream);
        if (widest <= 64) return attn_one_l<8>(*a, pdl, stream);
        if (widest <= 128) return attn_one_l<16>(*a, pdl, stream);
        return attn_one_l<32>(*a, pdl, stream);
    }
    return dtype ? attn_prompt<float>(*a, false, pdl, stream) : attn_prompt<bf16>(*a, path == 0 && attn_tc_fits(*a), pdl, stream);
}

extern "C" int decoder_status(void) { return read_decoder_status(); }
