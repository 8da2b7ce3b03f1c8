/* C ABI of libfloatops.so: the floating-point decoder kernels (sm_100a).
 *
 * Device pointers throughout.  dtype: 0 = float32, 1 = bfloat16.  Every call is asynchronous on `stream` and
 * returns a status (0 ok, 1 bad argument, 3 CUDA error, 6 unsupported shape).  Sizes called "padded" are
 * multiples of 8 and padding holds zeros; row pitches are counted in elements and are multiples of 8.
 *
 * Rows of a batched step: row r belongs to sequence r / seq and sits at position start[r / seq] + r % seq.
 */
#ifndef ZKDS_FLOAT_H
#define ZKDS_FLOAT_H

#ifdef __cplusplus
extern "C" {
#endif

#define ZKFP_F32 0
#define ZKFP_BF16 1

/* epilogues of zkfp_linear, applied to the 32-bit accumulators */
#define ZKFP_EPI_STORE 0   /* out[m][n] = acc */
#define ZKFP_EPI_ROTATE 1  /* columns come in groups of `period`; from `offset` on, `pairs` adjacent pairs turn */
#define ZKFP_EPI_GATE 2    /* out[m][n] = sigmoid(acc) * aux[m][n] */
#define ZKFP_EPI_GLU 3     /* out[m][n / 2] = silu(acc[n]) * acc[n + 1] for even n */

typedef struct {
    const void* A;         /* [M][lda] activations */
    const void* W;         /* [N][ldw] weights */
    void* out;             /* [M][ldo] */
    const void* aux;       /* gate: [M][ldaux], dtype */
    const float* table;    /* rotate: (cos, sin) pairs, [position][pairs] */
    const int* start;      /* rotate: first position of every sequence */
    long long lda, ldw, ldo, ldaux;
    long long M, N, K;     /* N, K padded (GLU: N a multiple of 16) */
    long long seq;         /* rotate: rows per sequence */
    long long positions;   /* rotate: rows of the table; a position outside them leaves its row unrotated */
    int dtype, out_dtype, epilogue;
    int pairs, period, offset;
} zkfp_linear_args;

int zkfp_linear(const zkfp_linear_args* a, void* stream);

/* x[r] = table[tokens[r]] in 32-bit; xb (may be null) the same in bfloat16.  Ids outside [0, vocab) give zeros. */
int zkfp_embed(const long long* tokens, const void* table, long long ld_table, long long vocab, float* x, void* xb,
               long long ldx, long long rows, int dtype, void* stream);

/* x[r] += w * y[r] / sqrt(mean(y[r]^2) + eps) over `width` values, in 32-bit; xb (may be null) = bfloat16(x) */
int zkfp_add_norm(float* x, const float* y, const float* w, void* xb, long long ldx, long long ldy, long long rows,
                  long long width, double eps, void* stream);

/* out[i] = w * x[index[i]] / sqrt(mean(x^2) + eps); index null: every row */
int zkfp_norm_rows(const float* x, long long ldx, const int* index, const float* w, void* out, long long ldo,
                   long long n, long long width, double eps, int dtype, void* stream);

typedef struct {
    const float* y;        /* [rows][ldy]: query latent, then (own_kv) key/value latent, then rotated key part */
    const float* wq;       /* norm weights, padded */
    const float* wc;
    void* cq;              /* [rows][ldq] normed query latent, dtype */
    void* cache;           /* [slot][capacity][pitch] of this layer, dtype: latent at 0, rotated part at c_pad */
    const float* table;
    const int* start;
    const int* slots;      /* cache slot of every sequence */
    long long ldy, ldq, rows, seq;
    long long slot_stride, pitch, capacity;
    int q_rank, q_pad, c, c_pad, pairs;
    int own_kv, dtype;
    double eps;
} zkfp_latent_args;

/* the norms of both latents, the rotation of the shared key part and the cache write.  Rows whose position is
 * not below the capacity are not written. */
int zkfp_latent_post(const zkfp_latent_args* a, void* stream);

/* per-head products of the absorbed (decode) form: weights [heads][rows_per_head][ldw].
 * absorb:  out[t][h][c] = sum_d q[t][h][d] * W[h][d][c]
 * expand:  out[t][h][v] = sum_c x[t][h][c] * W[h][v][c] */
typedef struct {
    const void* x;
    const void* W;
    void* out;
    long long x_tok, x_head, o_tok, o_head;   /* element strides */
    long long w_head, ldw;
    long long tokens, heads;
    int n_out, n_in, transposed, dtype;       /* transposed = 1: absorb */
    int copy_from, copy_to, copy_n;           /* absorb: also out[t][h][copy_to + i] = x[t][h][copy_from + i] */
} zkfp_perhead_args;
int zkfp_perhead(const zkfp_perhead_args* a, void* stream);

/* Windowed softmax attention, one query row per (token, head).
 *   score = (q[0:d1] . k1 + q[d1:d1+d2] . k2) * scale, visible keys: 0 <= i - j < window (window <= 0: all j <= i)
 * Keys and values are addressed by position minus base.  `shared` = 1: all heads read the same keys and values
 * (the absorbed form), rows are (token, head) pairs. */
typedef struct {
    const void* q;         /* [batch][seq][heads][q_head] */
    const void* k1;        /* position p, head h: k1 + (p - base) * k1_tok + h * k1_head */
    const void* k2;        /* shared by all heads: k2 + (p - base) * k2_tok */
    const void* v;
    void* out;             /* [batch][seq][heads][o_head] */
    const int* start;
    const int* slots;      /* null: sequence b is cache slot b */
    float* scratch;        /* decode form: partial results, zkfp_attention_scratch() floats; may be null */
    long long q_head, o_head;
    long long k1_tok, k1_head, k2_tok, v_tok, v_head;
    long long slot_stride;        /* elements between slots of k1, k2 and v (shared form) */
    long long base, keys;         /* expanded form: k1 / v hold positions base .. base + keys - 1 */
    long long batch, seq, heads;
    int d1, d2, dv, window, shared, dtype;
    float scale;
    int max_keys;          /* decode form: host bound on the visible keys of a step (sizes the grid) */
} zkfp_attention_args;
int zkfp_attention(const zkfp_attention_args* a, void* stream);
long long zkfp_attention_scratch(const zkfp_attention_args* a);

/* which kernel a call takes: 0 plain CUDA cores, 1 tensor cores, 2 weight streaming; for tests and reports */
int zkfp_linear_path(const zkfp_linear_args* a);
int zkfp_attention_path(const zkfp_attention_args* a);

/* 5 if a finished kernel gave up a bounded wait since the last call, else 0 */
int zkfp_device_status(void);
long long zkfp_launches(void);      /* kernels launched by this library so far */
int zkfp_cuda_error(void);          /* cudaError_t behind the last status 3 of this thread */

#ifdef __cplusplus
}
#endif
#endif
