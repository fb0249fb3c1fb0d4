/* libdecoderops.so for NVIDIA B200 (sm_100a): kernels of dense decoders that are more than attention plus
 * feed-forward - several residual streams (hyper-connections), the generalised delta rule, attention with
 * sigmoid weights - and the dense bf16 linear of their decode step.
 *
 * Conventions.  All pointers are device pointers unless said otherwise.  dtype: the activation (and table)
 * type, 0 = bf16, 1 = fp32; parameters that enter 32-bit arithmetic (norm weights, biases, mixing weights)
 * are fp32.  Every call returns 0 or one of the codes below and launches nothing when it fails; nothing is
 * allocated and nothing but decoder_status synchronises, so all of it can be captured in a CUDA graph.  pdl != 0: launch with
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

/* Device-side status since the last call (synchronises): 0, or DECODER_WAIT_TIMEOUT when a bounded wait inside a
 * kernel ran out, in which case that kernel's output is incomplete. */
int decoder_status(void);

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

/* Between two sublayers: x_t <- sum_s mix[s][t] x_s + m * out[t] * y (skipped when y is NULL), then
 * h = rmsnorm(sum_s in[s] x_s) * (w_offset + w) (in NULL: all ones).  With a row list, n_rows rows of h are made
 * from those rows of x and y, and x is not written. */
typedef struct {
    float* x;                  /* [rows][S][D] */
    const void* y;             /* [rows][D], or NULL */
    const float* mix;          /* [S][S], [from][to] */
    const float* out;          /* [S] */
    const float* in;           /* [S], or NULL */
    const float* w;            /* [D] */
    const long long* rows;     /* [n_rows], or NULL for all rows in order */
    void* h;                   /* [n_rows][D], or NULL */
    float m, w_offset, eps;
    int D, S, n_rows;
} decoder_hyper_args;
int decoder_hyper(const decoder_hyper_args* a, int dtype, int pdl, void* stream);

/* out[m][n] = act(sum_k w[n][k] x[m][k]), bf16 in, M <= 8, K a multiple of 8; act 1 = square of relu;
 * out_fp32: fp32 instead of bf16 results. */
int decoder_rows_linear(const void* x, const void* w, void* out, int M, int N, int K, int act, int out_fp32, int pdl,
                        void* stream);

/* Greedy token (and fp32 logits, unrounded, when logits != NULL) of up to 8 rows over a bf16 output matrix
 * [V][K], K a multiple of 32 up to 12288.  scratch: decoder_head_scratch_bytes() bytes, zero before the first call. */
long long decoder_head_scratch_bytes(void);
int decoder_head_argmax(const void* h, const void* w, int M, int V, int K, float* logits, long long* argmax, void* scratch,
                        void* stream);

/* x[i] = max(x[i], 0)^2 in place */
int decoder_relu2(void* x, long long n, int dtype, int pdl, void* stream);

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
/* out[row][j] = tanh(proj[row][off + j]), j < rank */
int decoder_tanh_cols(const void* proj, long long ld, int off, int rank, long long rows, void* out, int dtype, int pdl,
                      void* stream);

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

#ifdef __cplusplus
}
#endif
#endif
