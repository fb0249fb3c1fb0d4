// libdecoderops.so for NVIDIA B200 (sm_100a): the extern "C" surface declared in include/decoder_ops.h and
// the host-side launch logic behind it.
#include <stdio.h>

#include <algorithm>

#include "decoder_ops.h"

#include "delta_rule.cuh"
#include "hyper.cuh"
#include "rows_linear.cuh"
#include "sigmoid_attn.cuh"
#include "sigmoid_attn_tc.cuh"

namespace tsp {

static int sm_count() {
    static int sms[64] = {0};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) dev = 0;
    if (!sms[dev]) {
        int v = 0;
        if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || v <= 0) v = 148;
        sms[dev] = v;
    }
    return sms[dev];
}

static int bad(int code, const char* what) {
    fprintf(stderr, "decoder_ops: %s\n", what);
    return code;
}
static bool misaligned(const void* p, unsigned n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) != 0; }

template <typename... P, typename... Q>
static int launch(void (*kernel)(P...), dim3 grid, int threads, size_t smem, int pdl, void* stream, int cluster, Q... args) {
    if (smem > 48 * 1024 &&
        cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return bad(DECODER_LAUNCH, "shared memory request refused");
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(threads, 1, 1);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = static_cast<cudaStream_t>(stream);
    cudaLaunchAttribute at[2];
    int n = 0;
    if (pdl) {
        at[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        at[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 1) {
        at[n].id = cudaLaunchAttributeClusterDimension;
        at[n].val.clusterDim.x = cluster, at[n].val.clusterDim.y = 1, at[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = at, cfg.numAttrs = n;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, args...);
    if (e != cudaSuccess) {
        fprintf(stderr, "decoder_ops: launch failed: %s\n", cudaGetErrorString(e));
        return DECODER_LAUNCH;
    }
    return DECODER_OK;
}

template <typename A, int S>
static int hyper_s(const HyperParams& p, int pdl, void* stream) {
    const bool v4 = p.D % 4 == 0 && !misaligned(p.x, 16) && !misaligned(p.w, 16) && !misaligned(p.y, 16) && !misaligned(p.h, 16);
    const int per = v4 ? 4 : 1;
    // few rows: one row's latency counts, so the whole row is in flight at once; many rows: several CTAs per SM
    const int want = (p.D / per + 31) / 32 * 32;
    const int threads = std::min(p.n_rows <= 2 * sm_count() ? 1024 : 256, std::max(64, want));
    const size_t smem = (size_t)p.D * 4;
    return v4 ? launch(hyper_kernel<A, S, 4>, dim3(p.n_rows), threads, smem, pdl, stream, 1, p)
              : launch(hyper_kernel<A, S, 1>, dim3(p.n_rows), threads, smem, pdl, stream, 1, p);
}
template <typename A>
static int hyper(const HyperParams& p, int pdl, void* stream) {
    switch (p.S) {
        case 1: return hyper_s<A, 1>(p, pdl, stream);
        case 2: return hyper_s<A, 2>(p, pdl, stream);
        case 3: return hyper_s<A, 3>(p, pdl, stream);
        case 4: return hyper_s<A, 4>(p, pdl, stream);
        case 5: return hyper_s<A, 5>(p, pdl, stream);
        case 6: return hyper_s<A, 6>(p, pdl, stream);
        case 7: return hyper_s<A, 7>(p, pdl, stream);
        case 8: return hyper_s<A, 8>(p, pdl, stream);
    }
    return bad(DECODER_BAD_SHAPE, "hyper: 1 to 8 streams");
}

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

static bool encode_rows(CUtensorMap* map, const void* base, long long rows, long long cols, long long ld) {
    typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                 const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                 CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static EncodeFn fn = nullptr;
    if (!fn) {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || !ptr) return false;
        fn = reinterpret_cast<EncodeFn>(ptr);
    }
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64, 128}, step[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
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
    if (!encode_rows(&proj, p.proj, (long long)p.B * p.T, p.ld, p.ld) || !encode_rows(&ck, p.ck, cache_rows, p.dim, p.dim) ||
        !encode_rows(&cv, p.cv, cache_rows, p.vdim, p.vdim))
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

extern "C" int decoder_embed(const decoder_embed_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->S < 1 || a->D < 1 || a->V < 1 || (a->bigram && a->buckets < 1))
        return bad(DECODER_BAD_SHAPE, "embed: empty shape");
    if (!a->tokens || !a->pos || !a->embed || !a->x) return bad(DECODER_BAD_POINTER, "embed: null pointer");
    decoder_embed_args p = *a;
    if (!p.bigram) p.buckets = 1;
    const dim3 grid((unsigned)(p.B * p.T));
    return dtype ? launch(embed_kernel<float>, grid, 256, 0, pdl, stream, 1, p) : launch(embed_kernel<bf16>, grid, 256, 0, pdl, stream, 1, p);
}

extern "C" int decoder_hyper(const decoder_hyper_args* a, int dtype, int pdl, void* stream) {
    if (a->n_rows < 1 || a->D < 1 || a->D > 12288) return bad(DECODER_BAD_SHAPE, "hyper: rows >= 1, 1 <= width <= 12288");
    if (!a->x || (a->h && !a->w) || (a->y && (!a->mix || !a->out))) return bad(DECODER_BAD_POINTER, "hyper: null pointer");
    return dtype ? hyper<float>(*a, pdl, stream) : hyper<bf16>(*a, pdl, stream);
}

extern "C" int decoder_rows_linear(const void* x, const void* w, void* out, int M, int N, int K, int act, int out_fp32, int pdl,
                                   void* stream) {
    if (M < 1 || M > 8 || N < 1 || K < 8 || K % 8) return bad(DECODER_BAD_SHAPE, "rows_linear: 1 <= M <= 8, K a multiple of 8");
    if (!x || !w || !out || misaligned(x, 16) || misaligned(w, 16)) return bad(DECODER_BAD_POINTER, "rows_linear: null or misaligned pointer");
    RowsLinearParams p = {static_cast<const bf16*>(x), static_cast<const bf16*>(w), out, M, N, K, act};
    const dim3 grid((N + 15) / 16);
    return out_fp32 ? launch(rows_linear_kernel<float>, grid, kRowsWarps * 32, 0, pdl, stream, 1, p)
                    : launch(rows_linear_kernel<bf16>, grid, kRowsWarps * 32, 0, pdl, stream, 1, p);
}

extern "C" long long decoder_head_scratch_bytes(void) { return (long long)kHeadScratchBytes; }

extern "C" int decoder_head_argmax(const void* h, const void* w, int M, int V, int K, float* logits, long long* argmax,
                                   void* scratch, void* stream) {
    if (M < 1 || M > 8 || V < 1 || K < 32 || K % 32 || K > 12288)
        return bad(DECODER_BAD_SHAPE, "head_argmax: 1 <= M <= 8, K a multiple of 32 up to 12288");
    if (!h || !w || !argmax || !scratch || misaligned(h, 16) || misaligned(w, 16) || misaligned(scratch, 16))
        return bad(DECODER_BAD_POINTER, "head_argmax: null or misaligned pointer");
    HeadParams p;
    p.h = static_cast<const bf16*>(h), p.emb = static_cast<const bf16*>(w), p.logits = logits, p.argmax = argmax;
    p.counter = static_cast<unsigned int*>(scratch);
    p.cand = reinterpret_cast<HeadCandidate*>(static_cast<uint8_t*>(scratch) + 16);
    p.M = M, p.V = V, p.K = K, p.round_bf16 = 0;
    const int ctas = std::min(std::min(sm_count(), (V + 15) / 16), kHeadMaxCtas);
    return launch(lm_head_kernel, dim3(ctas), kHeadWarps * 32, (size_t)8 * (K * 2 + 64), 0, stream, 1, p);
}

extern "C" int decoder_relu2(void* x, long long n, int dtype, int pdl, void* stream) {
    if (n < 1) return bad(DECODER_BAD_SHAPE, "relu2: empty");
    if (!x || misaligned(x, 16)) return bad(DECODER_BAD_POINTER, "relu2: null or misaligned pointer");
    const dim3 grid((unsigned)std::min<long long>((n / 4 + 255) / 256 + 1, 8ll * sm_count()));
    return dtype ? launch(relu2_kernel<float>, grid, 256, 0, pdl, stream, 1, static_cast<float*>(x), n)
                 : launch(relu2_kernel<bf16>, grid, 256, 0, pdl, stream, 1, static_cast<bf16*>(x), n);
}

extern "C" int decoder_delta(const decoder_delta_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->H < 1 || a->dk < 1 || a->dv < 1 || a->rank < 1 || a->dk > 256 || a->dv > 512)
        return bad(DECODER_BAD_SHAPE, "delta: 1 <= dk <= 256, 1 <= dv <= 512");
    if (!a->proj || !a->w0 || !a->a_bias || !a->norm || !a->pos || !a->state || !a->y || (a->T > 1 ? !a->zw || !a->o || misaligned(a->o, 16) : !a->w2))
        return bad(DECODER_BAD_POINTER, "delta: null or misaligned pointer");
    if (a->T == 1) return dtype ? delta_one<float>(*a, pdl, stream) : delta_one<bf16>(*a, pdl, stream);
    return dtype ? delta_prompt<float>(*a, pdl, stream) : delta_prompt<bf16>(*a, pdl, stream);
}

extern "C" int decoder_tanh_cols(const void* proj, long long ld, int off, int rank, long long rows, void* out, int dtype, int pdl,
                                 void* stream) {
    if (rank < 1 || rows < 1 || off < 0 || off + rank > ld) return bad(DECODER_BAD_SHAPE, "tanh_cols: columns outside the row");
    if (!proj || !out) return bad(DECODER_BAD_POINTER, "tanh_cols: null pointer");
    const dim3 grid((unsigned)std::min<long long>((rows * rank + 255) / 256, 8ll * sm_count()));
    return dtype ? launch(tanh_cols_kernel<float>, grid, 256, 0, pdl, stream, 1, static_cast<const float*>(proj), ld, off, rank, rows,
                          static_cast<float*>(out))
                 : launch(tanh_cols_kernel<bf16>, grid, 256, 0, pdl, stream, 1, static_cast<const bf16*>(proj), ld, off, rank, rows,
                          static_cast<bf16*>(out));
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

extern "C" int decoder_status(void) {
    int v = 0;
    if (cudaMemcpyFromSymbol(&v, g_decoder_status, sizeof(v)) != cudaSuccess) return DECODER_LAUNCH;
    if (v) {
        const int zero = 0;
        cudaMemcpyToSymbol(g_decoder_status, &zero, sizeof(zero));
    }
    return v;
}
