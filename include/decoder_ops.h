/* Kernels of dense decoders for NVIDIA B200 (sm_100a), in three libraries so that a model needs only its own:
 *   libdecoderops.so  what all of them use: embedding, residual streams with norms, decode linears, output head
 *   libdeltaops.so    the generalised delta rule and attention with sigmoid weights
 *   liblatentops.so   the wkv recurrence, attention over a shared latent, mixtures of experts
 *
 * Conventions.  All pointers are device pointers unless said otherwise.  dtype: the activation (and table)
 * type, 0 = bf16, 1 = fp32; parameters that enter 32-bit arithmetic (norm weights, biases, mixing weights)
 * are fp32.  Every call returns 0 or one of the codes below and launches nothing when it fails; nothing is
 * allocated and nothing but the status calls synchronises, so all of it can be captured in a CUDA graph.  pdl != 0: launch with
 * programmatic dependent launch (decode steps: the kernels' weight fetches start under their predecessor).
 * Positions are read from device memory (pos[0] = position of the call's first token in its sequence; all
 * sequences of a call are at the same position); position 0 starts a sequence: recurrent state and token
 * history are then taken as empty, whatever the buffers hold.
 */
#ifndef DECODER_OPS_H
#define DECODER_OPS_H
#ifdef __cplusplus
extern "C" {
#endif

#define DECODER_OK 0
#define DECODER_BAD_SHAPE 1
#define DECODER_BAD_POINTER 2
#define DECODER_LAUNCH 3
#define DECODER_WAIT_TIMEOUT 4

/* x[row][s][:] = embed[token] + bigram[(previous * mul_prev + token * mul_cur) mod buckets], the same for all
 * S streams; a sequence's first token takes bigram row number `buckets`.  prev [B]: token before this call's
 * first, replaced by the call's last. */
typedef struct {
    const long long* tokens;   /* [B][T] */
    const long long* pos;      /* [T] */
    long long* prev;           /* [B], or NULL */
    const void* embed;         /* [V][D] */
    const void* bigram;        /* [buckets + 1][D], or NULL */
    float* x;                  /* [B*T][S][D] */
    long long mul_prev, mul_cur, buckets;
    int B, T, S, D, V;
} decoder_embed_args;
int decoder_embed(const decoder_embed_args* a, int dtype, int pdl, void* stream);

/* Between two sublayers: x_t <- sum_s mix[s][t] x_s + m * out[t] * y (skipped when y is NULL; mix NULL: every stream
 * keeps to itself, out NULL: all ones), then h = rmsnorm(sum_s in[s] x_s) * (w_offset + w) (in NULL: all ones).
 * y2 (one stream only): a second output to be added to y - its row of the same number, or, with top > 0, the sum over j < top of
 * slot_w[row][j] times its row slots[row][j].  With a row list, n_rows rows of h are made from those rows of x and
 * y, and x is not written.  n_mu > 0 (one stream, one row per sequence, no row list): also mixed[j][row] = h + (prev - h) * mu[j],
 * prev taken as zeros at position 0, and prev becomes h. */
typedef struct {
    float* x;                  /* [rows][S][D] */
    const void* y;             /* [rows][D], or NULL */
    const float* mix;          /* [S][S], [from][to] */
    const float* out;          /* [S] */
    const float* in;           /* [S], or NULL */
    const float* w;            /* [D] */
    const long long* rows;     /* [n_rows], or NULL for all rows in order */
    void* h;                   /* [n_rows][D], or NULL */
    const void* y2;            /* [rows or slots][D], or NULL */
    const int* slots;          /* [rows][top] */
    const float* slot_w;       /* [rows][top] */
    const float* mu;           /* [n_mu][D] */
    void* prev;                /* [n_rows][D] */
    void* mixed;               /* [n_mu][n_rows][D] */
    const long long* pos;      /* n_mu > 0 */
    float m, w_offset, eps;
    int D, S, n_rows, top, n_mu;
} decoder_hyper_args;
int decoder_hyper(const decoder_hyper_args* a, int dtype, int pdl, void* stream);

/* mixed[j][row] = h + (h_before - h) * mu[j] for every row of B prompt portions of T rows: h_before is the row before,
 * prev (zeros at position 0) for a portion's first row; prev becomes the last row's h. */
typedef struct {
    const void* h;             /* [B*T][D] */
    void* prev;                /* [B][D] */
    const float* mu;           /* [n_mu][D] */
    void* mixed;               /* [n_mu][B*T][D] */
    const long long* pos;      /* [T] */
    int B, T, D, n_mu;
} decoder_shift_args;
int decoder_token_shift(const decoder_shift_args* a, int dtype, int pdl, void* stream);

/* Activation of a gated feed-forward: kind 1 = silu(g) * u; kind 2 = g * sigmoid(alpha * g) * (u + 1) with g at most
 * limit and u within +-limit. */
typedef struct {
    int kind;
    float alpha, limit;
} decoder_gate;

/* out[m][n] = act(sum_k w[n][k] x[m][k] + bias[n]), bf16 in, M <= 8, K a multiple of 8; out_fp32: fp32 instead of bf16
 * results.  seg_rows > 0: rows [s * seg_rows, (s + 1) * seg_rows) of w (the last of n_seg segments: all further rows)
 * read x + s * M * K.  gate.kind > 0: w and bias hold blocks of 8 gate and 8 up rows, out is [M][N / 2].  N2 > 0: in the
 * same launch out2 = w2 x2, fp32; zero: a word to be set to 0 with it (decoder_moe_up_step's ticket). */
typedef struct {
    const void* x;             /* [n_seg][M][K] */
    const void* w;             /* [N][K] */
    const float* bias;         /* [N], or NULL */
    void* out;                 /* [M][N] */
    const void* x2;            /* [M][K] */
    const void* w2;            /* [N2][K] */
    float* out2;               /* [M][N2] */
    int* zero;                 /* or NULL */
    int M, N, K, relu2, seg_rows, n_seg, N2;
    decoder_gate gate;
} decoder_linear_args;
int decoder_rows_linear(const decoder_linear_args* a, int out_fp32, int pdl, void* stream);
/* The gate alone: z [rows][2 * n] and bias (fp32, or NULL) in blocks of 8 gate and 8 up columns -> out [rows][n]. */
int decoder_gated(const void* z, const float* bias, void* out, long long rows, int n, const decoder_gate* gate, int dtype, int pdl,
                  void* stream);

/* Greedy token (and fp32 logits, unrounded, when logits != NULL) of up to 8 rows over a bf16 output matrix
 * [V][K], K a multiple of 32 up to 12288.  scratch: decoder_head_scratch_bytes() bytes, zero before the first call. */
long long decoder_head_scratch_bytes(void);
int decoder_head_argmax(const void* h, const void* w, int M, int V, int K, float* logits, long long* argmax, void* scratch,
                        void* stream);

/* x[i] = max(x[i], 0)^2 in place */
int decoder_relu2(void* x, long long n, int dtype, int pdl, void* stream);

/* out[row][j] = tanh(proj[row][off + j]), j < rank */
int decoder_tanh_cols(const void* proj, long long ld, int off, int rank, long long rows, void* out, int dtype, int pdl,
                      void* stream);

/* ---- libdeltaops.so ---- */

/* Device-side status of libdeltaops.so since the last call (synchronises): 0, or DECODER_WAIT_TIMEOUT when a bounded
 * wait inside a kernel ran out, in which case that kernel's output is incomplete. */
int decoder_status(void);

/* Generalised delta rule (see delta_rule.cuh).  T = 1: one launch from the projections to the gated output.
 * T > 1: the second decay projection zw [B*T][H*dk] (fp32, before w0) comes from the caller - out of
 * decoder_tanh_cols and a matrix product - and o [B*T][H*dv] is fp32 workspace. */
typedef struct {
    const void* proj;          /* [B*T][ld] */
    const float* zw;           /* T > 1 */
    const void* w2;            /* T = 1: [H*dk][rank] */
    const float* w0;           /* [H*dk] */
    const float* a_bias;       /* [H*dk] */
    const float* norm;         /* [H*dv] */
    const long long* pos;      /* [T] */
    float* state;              /* [B][H][dk][dv] */
    float* o;                  /* T > 1 */
    void* y;                   /* [B*T][H*dv] */
    int B, T, H, dk, dv, rank;
    long long ld;
    int off_r, off_k, off_v, off_a, off_g, off_w1;
    float eps;
} decoder_delta_args;
int decoder_delta(const decoder_delta_args* a, int dtype, int pdl, void* stream);

/* Sigmoid-weighted attention over a chunk (see sigmoid_attn.cuh): norms of queries and keys (in place in proj),
 * cache reads and writes, attention, output gate.  path: 0 = the library chooses, 1 = the kernel for any type
 * and size (also for one token). */
typedef struct {
    void* proj;                /* [B*T][ld] */
    void* ck;                  /* [B][G][slots][dim] */
    void* cv;                  /* [B][G][slots][vdim] */
    const float* q_norm;       /* [dim] */
    const float* k_norm;       /* [dim] */
    const float* bias;         /* [H] */
    const float* slope;        /* [H] */
    const long long* pos;      /* [T] */
    void* y;                   /* [B*T][H*vdim] */
    int B, T, H, G, dim, vdim;
    long long ld;
    int off_q, off_k, off_v, off_g;
    int chunk, slots;          /* slots = min(chunk, longest sequence) */
    float scale, eps;
} decoder_attn_args;
int decoder_attn(const decoder_attn_args* a, int dtype, int path, int pdl, void* stream);

/* ---- liblatentops.so ---- */

/* As decoder_status, of liblatentops.so. */
int decoder_latent_status(void);

/* wkv recurrence (see wkv.cuh).  r, k, v and g are rows of ld elements, t1 of ld_t.  T = 1: one launch from the projections to
 * the gated output; t1 is the low-rank decay projection before its tanh.  T > 1: the second decay projection zw
 * [B*T][H*dk] (fp32, before w0) comes from the caller; the portion is cut into n_seg segments of seg_len tokens (a
 * multiple of 16), for which part [B][H][n_seg][dk*dv + dk] is workspace when n_seg > 1; o is workspace too. */
typedef struct {
    const void* r;             /* [B*T][ld] */
    const void* k;
    const void* v;
    const void* g;
    const void* t1;            /* T = 1 */
    const float* zw;           /* T > 1 */
    const void* w2;            /* T = 1: [H*dk][rank] */
    const float* w0;           /* [H*dk] */
    const float* u;            /* [H*dk] */
    const float* norm;         /* [H*dv] */
    const long long* pos;      /* [T] */
    float* state;              /* [B][H][dk][dv] */
    float* part;               /* T > 1, n_seg > 1 */
    float* o;                  /* T > 1: [B*T][H*dv] */
    void* y;                   /* [B*T][H*dv] */
    int B, T, H, dk, dv, rank;
    long long ld, ld_t;
    int n_seg, seg_len;
    float eps;
} decoder_wkv_args;
int decoder_wkv(const decoder_wkv_args* a, int dtype, int pdl, void* stream);

/* Latent attention, what enters the cache (see latent_attn.cuh): z holds the query latent (q_rank columns from off_q)
 * and, unless cache is NULL, the key latent (R) and the shared key part (rot) from off_kv.  cq = rmsnorm(query latent)
 * * q_norm; cache row pos: rmsnorm(key latent) * kv_norm, and from column r_at the rotated key part.  trig [.][dims]:
 * cosine and sine per position and pair; channels from dims on are not turned. */
typedef struct {
    const void* z;             /* [B*T][ld_z] */
    void* cq;                  /* [B*T][q_rank] */
    void* cache;               /* [B][slots][ld], or NULL */
    const float* q_norm;       /* [q_rank] */
    const float* kv_norm;      /* [R] */
    const float* trig;         /* [slots][dims] */
    const long long* pos;      /* [T] */
    int B, T, slots, ld, r_at, R, rot, dims, q_rank;
    long long ld_z;
    int off_q, off_kv;
    float eps;
} decoder_latent_prep_args;
int decoder_latent_prep(const decoder_latent_prep_args* a, int dtype, int pdl, void* stream);

/* The rot channels of every head turned by the position: src row r, head h from off_src + h * head_src, to dst alike
 * (src = dst: in place). */
typedef struct {
    const void* src;           /* [B*T][ld_src] */
    void* dst;                 /* [B*T][ld_dst] */
    const float* trig;         /* [positions][dims] */
    const long long* pos;      /* [T] */
    int B, T, H, rot, dims;
    long long ld_src, ld_dst;
    int head_src, head_dst, off_src, off_dst;
} decoder_rotate_args;
int decoder_rotate(const decoder_rotate_args* a, int dtype, int pdl, void* stream);

/* Up to eight bf16 rows: queries q [rows][H][dim + rot] (not rotated) to absorbed queries qa [rows][H][ld] in the cache's
 * layout; dim and rot multiples of 8. */
typedef struct {
    const void* q;
    const void* w_uk_t;        /* [H][R][dim] */
    void* qa;
    const float* trig;         /* [positions][dims] */
    const long long* pos;      /* [T] */
    int B, T, H, dim, rot, dims, R, r_at, ld;
} decoder_absorb_args;
int decoder_absorb(const decoder_absorb_args* a, int pdl, void* stream);

/* Attention in the absorbed form: causal softmax over the cache with the sink in the denominator.
 * decoder_latent_attn: any type and size, out = weighted latents [rows][H][R].
 * decoder_latent_step: bf16, R a multiple of 8 up to 1024, ld up to decoder_latent_step_width(): the keys in splits *
 * cluster ranges, those of a cluster (up to 8) joined on the way, then the product with w_uv: y [rows][H*vdim]. */
typedef struct {
    const void* qa;            /* [rows][H][ld], rows = B*T */
    const void* cache;         /* [B][slots][ld], ld a multiple of 8 */
    const float* sink;         /* [H] */
    const long long* pos;      /* [T] */
    void* out;                 /* [rows][H][R] */
    const void* w_uv;          /* [H*vdim][R] */
    float* part;               /* [rows][H][splits][R] */
    float* ml;                 /* [rows][H][splits][2] */
    void* y;                   /* [rows][H*vdim] */
    int B, T, H, R, ld, vdim, slots, splits, cluster;
    float scale;
} decoder_latent_attn_args;
int decoder_latent_attn(const decoder_latent_attn_args* a, int dtype, int pdl, void* stream);
int decoder_latent_step(const decoder_latent_attn_args* a, int pdl, void* stream);
int decoder_latent_step_width(void);

/* Prompt attention over expanded keys and values (latent_attn_tc.cuh), bf16; dim, rot and vdim multiples of 16, dim and
 * vdim up to 128, rot up to 64.  Positions start .. start + T - 1; kv holds all start + T of every sequence. */
typedef struct {
    const void* q;             /* [B*T][H][dim + rot], rotated */
    const void* kv;            /* [B*(start + T)][ld_kv]: keys [H][dim], from column off_v values [H][vdim] */
    const void* cache;         /* [B][slots][ld]: the shared key part from column r_at */
    const float* sink;         /* [H] */
    void* y;                   /* [B*T][H*vdim] */
    int B, T, H, dim, rot, vdim, slots, ld, r_at, start, off_v;
    long long ld_kv;
    float scale;
} decoder_latent_prompt_args;
int decoder_latent_prompt(const decoder_latent_prompt_args* a, void* stream);

/* Mixture of gated experts (see moe.cuh).  top <= 32, E <= 1024; w_up holds blocks of 8 gate and 8 up rows.
 * decoder_moe_route: chosen experts and weights; with counts (zeroed by the caller) also every choice's rank among its
 *   expert's, then the rows of x sorted by expert, slots[token][j] saying where a choice's row went (bf16, K % 8 = 0).
 * decoder_moe_plain: any type and size, chosen and weight given: act, and out [M*top][D] not weighted.
 * decoder_moe_up_step: bf16, M <= 8, K a multiple of 8 up to 12288: routing and activations; ticket must be 0 before.
 * decoder_moe_down_step: bf16, M <= 8: out [M][D] = weighted sum + w_rest rest + bias.  Dense: weight NULL, E = top = 1. */
typedef struct {
    const float* logits;       /* [M][E], without bias */
    const float* router_bias;  /* [E] */
    int* chosen;               /* [M][top] */
    float* weight;             /* [M][top] */
    int* counts;               /* [E], or NULL */
    int* rank;                 /* [M][top] */
    int* slots;                /* [M][top] */
    int* ticket;               /* decoder_moe_up_step: one word of workspace */
    const void* x;             /* [M][K] */
    void* sorted;              /* [M*top][K] */
    const void* w_up;          /* [E][2*ff][K] */
    void* act;                 /* [M*top][ff] */
    const void* w_down;        /* [E][D][ff], or NULL */
    const void* w_rest;        /* [D][K_rest], or NULL */
    const void* rest;          /* [M][K_rest] */
    const float* bias;         /* [D], or NULL */
    void* out;
    int M, E, top, K, ff, D, K_rest;
    decoder_gate gate;
} decoder_moe_args;
int decoder_moe_route(const decoder_moe_args* a, int pdl, void* stream);
int decoder_moe_plain(const decoder_moe_args* a, int dtype, int pdl, void* stream);
int decoder_moe_up_step(const decoder_moe_args* a, int pdl, void* stream);
int decoder_moe_down_step(const decoder_moe_args* a, int pdl, void* stream);

/* Grouped GEMM (group_gemm_tc.cuh): rows of a sorted by group, counts[g] of each (NULL: one group of all rows), out
 * [rows][N], or with gate.kind > 0 (w and bias in blocks of 8 gate and 8 up rows) [rows][N / 2].  bf16; K a multiple of
 * 8, N of 16. */
typedef struct {
    const void* a;             /* [rows][K] */
    const void* w;             /* [groups][N][K] */
    const float* bias;         /* [groups][N], or NULL */
    const int* counts;         /* [groups], or NULL */
    void* out;
    int rows, groups, N, K;
    decoder_gate gate;
} decoder_group_gemm_args;
int decoder_group_gemm(const decoder_group_gemm_args* a, void* stream);

#ifdef __cplusplus
}
#endif
#endif
