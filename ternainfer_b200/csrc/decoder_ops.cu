// libdecoderops.so for NVIDIA B200 (sm_100a): the parts of include/decoder_ops.h that every dense decoder uses -
// embedding, residual streams and norms, decode linears, output head, elementwise pieces.
#include "decoder_launch.cuh"
#include "elementwise.cuh"
#include "hyper.cuh"
#include "rows_linear.cuh"

namespace tsp {

template <typename A, int S>
static int hyper_s(const HyperParams& p, int pdl, void* stream) {
    const bool v4 = p.D % 4 == 0 && !misaligned(p.x, 16) && !misaligned(p.w, 16) && !misaligned(p.y, 16) && !misaligned(p.h, 16) &&
                    !misaligned(p.y2, 16) && !misaligned(p.mu, 16) && !misaligned(p.prev, 16) && !misaligned(p.mixed, 16);
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
    if (a->S > 1 && (a->y2 || a->n_mu > 0)) return bad(DECODER_BAD_SHAPE, "hyper: a second output and shifted inputs need one stream");
    if (!a->x || (a->h && !a->w) || (a->y2 && (!a->y || (a->top > 0 && (!a->slots || !a->slot_w)))) ||
        (a->n_mu > 0 && (!a->h || !a->mu || !a->prev || !a->mixed || !a->pos || a->rows)))
        return bad(DECODER_BAD_POINTER, "hyper: null pointer");
    return dtype ? hyper<float>(*a, pdl, stream) : hyper<bf16>(*a, pdl, stream);
}

extern "C" int decoder_rows_linear(const decoder_linear_args* a, int out_fp32, int pdl, void* stream) {
    if (a->M < 1 || a->M > 8 || a->N < 1 || a->K < 8 || a->K % 8) return bad(DECODER_BAD_SHAPE, "rows_linear: 1 <= M <= 8, K a multiple of 8");
    if (a->seg_rows < 0 || a->seg_rows % 16 || (a->seg_rows && a->n_seg < 1)) return bad(DECODER_BAD_SHAPE, "rows_linear: segments of 16 rows");
    if (a->gate.kind < 0 || a->gate.kind > 2 || (a->gate.kind && a->N % 16)) return bad(DECODER_BAD_SHAPE, "rows_linear: gated rows come in blocks of 16");
    if (!a->x || !a->w || !a->out || misaligned(a->x, 16) || misaligned(a->w, 16)) return bad(DECODER_BAD_POINTER, "rows_linear: null or misaligned pointer");
    if (a->N2 < 0 || (a->N2 && (!a->w2 || !a->x2 || !a->out2 || misaligned(a->w2, 16) || misaligned(a->x2, 16)))) return bad(DECODER_BAD_POINTER, "rows_linear: second product");
    const dim3 grid((a->N + 15) / 16 + (a->N2 + 15) / 16);
    return out_fp32 ? launch(rows_linear_kernel<float>, grid, kRowsWarps * 32, 0, pdl, stream, 1, *a)
                    : launch(rows_linear_kernel<bf16>, grid, kRowsWarps * 32, 0, pdl, stream, 1, *a);
}

extern "C" int decoder_gated(const void* z, const float* bias, void* out, long long rows, int n, const decoder_gate* gate, int dtype, int pdl,
                             void* stream) {
    if (rows < 1 || n < 8 || n % 8 || gate->kind < 1 || gate->kind > 2) return bad(DECODER_BAD_SHAPE, "gated: columns in blocks of 8");
    if (!z || !out || misaligned(z, 16) || misaligned(out, 16) || misaligned(bias, 16)) return bad(DECODER_BAD_POINTER, "gated: null or misaligned pointer");
    const dim3 grid((unsigned)std::min<long long>((rows * n / 4 + 255) / 256, 16ll * sm_count()));
    return dtype ? launch(gated_kernel<float>, grid, 256, 0, pdl, stream, 1, static_cast<const float*>(z), bias, static_cast<float*>(out), rows, n, *gate)
                 : launch(gated_kernel<bf16>, grid, 256, 0, pdl, stream, 1, static_cast<const bf16*>(z), bias, static_cast<bf16*>(out), rows, n, *gate);
}

extern "C" int decoder_token_shift(const decoder_shift_args* a, int dtype, int pdl, void* stream) {
    if (a->B < 1 || a->T < 1 || a->D < 1 || a->n_mu < 1) return bad(DECODER_BAD_SHAPE, "token_shift: empty shape");
    if (!a->h || !a->prev || !a->mu || !a->mixed || !a->pos) return bad(DECODER_BAD_POINTER, "token_shift: null pointer");
    const bool v4 = a->D % 4 == 0 && !misaligned(a->h, 16) && !misaligned(a->prev, 16) && !misaligned(a->mu, 16) && !misaligned(a->mixed, 16);
    const dim3 grid((unsigned)(a->B * a->T));
    const int threads = std::min(256, std::max(32, (a->D / (v4 ? 4 : 1) + 31) / 32 * 32));
    if (v4) return dtype ? launch(token_shift_kernel<float, 4>, grid, threads, 0, pdl, stream, 1, *a) : launch(token_shift_kernel<bf16, 4>, grid, threads, 0, pdl, stream, 1, *a);
    return dtype ? launch(token_shift_kernel<float, 1>, grid, threads, 0, pdl, stream, 1, *a) : launch(token_shift_kernel<bf16, 1>, grid, threads, 0, pdl, stream, 1, *a);
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
