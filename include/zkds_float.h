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

/* epilogues of zkfp_linear, applied to the 32-bit accumulators after the bias */
#define ZKFP_EPI_STORE 0   /* out[m][n] = acc */
#define ZKFP_EPI_ROTATE 1  /* columns rot_begin .. rot_end - 1 come in groups of `period`; from `offset` on, `pairs`
                              adjacent pairs turn */
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
    int rot_begin, rot_end;   /* rotate: rot_end 0 = all columns */
    const float* bias;     /* may be null: [N], added to the accumulators */
    float* out2;           /* may be null: columns from `split` (a multiple of 32) on go here, in 32-bit, unrotated */
    long long ldo2;
    long long split;
} zkfp_linear_args;

int zkfp_linear(const zkfp_linear_args* a, void* stream);

/* x[r] = scale * table[tokens[r]] in 32-bit; xb (may be null) the same in bfloat16.  Ids outside [0, vocab) give zeros. */
int zkfp_embed(const long long* tokens, const void* table, long long ld_table, long long vocab, float* x, void* xb,
               long long ldx, long long rows, float scale, int dtype, void* stream);

/* x[r] += w * y[r] / sqrt(mean(y[r]^2) + eps) over `width` values, in 32-bit.  h (may be null) receives the next
 * sublayer's input, in h_dtype: the new x, or with w2 its norm w2 * x / sqrt(mean(x^2) + eps). */
int zkfp_add_norm(float* x, const float* y, const float* w, const float* w2, void* h, long long ldx, long long ldy,
                  long long rows, long long width, double eps, int h_dtype, void* stream);

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
    /* expanded form only */
    int heads_per_kv;      /* query heads that share a key / value head; 0 = 1 */
    const void* gate;      /* may be null: out is multiplied by sigmoid(gate[row][head][d]) * out_scale */
    long long gate_tok, gate_head;
    long long o_tok;       /* out row pitch, 0 = heads * o_head */
    float out_scale;       /* with a gate */
} zkfp_attention_args;
int zkfp_attention(const zkfp_attention_args* a, void* stream);
long long zkfp_attention_scratch(const zkfp_attention_args* a);

/* Heads of a grouped attention layer after their projection: queries and keys are divided by their root mean square
 * over `dim` values, weighted, turned (`pairs` adjacent pairs from the first element on) and stored; the projected keys
 * themselves are stored as the values.  Cache rows hold [kv_heads][d] keys, then [kv_heads][d] values; rows whose
 * position is not below the capacity are not written. */
typedef struct {
    const void* y;         /* [rows][ldy]: queries [heads][d] at q_col, keys [kv_heads][d] at k_col, dtype */
    const float* wq;       /* [d], padding zero */
    const float* wk;
    void* q;               /* [rows][heads][d] */
    void* cache;           /* [slot][capacity][pitch] */
    const float* table;    /* (cos, sin), [position][pairs] */
    const int* start;
    const int* slots;
    long long ldy, q_col, k_col, rows, seq;
    long long slot_stride, pitch, capacity;
    int heads, kv_heads, d, dim, pairs, dtype;
    double eps;
} zkfp_heads_args;
int zkfp_heads_post(const zkfp_heads_args* a, void* stream);

/* Grouped attention of a few tokens per sequence over the cache: chunks of keys side by side, merged by a second kernel
 * that also applies the gate (as in zkfp_attention_args). */
typedef struct {
    const void* q;         /* [batch * seq][heads][d] */
    const void* cache;     /* [slot][capacity][pitch]: keys at 0, values at v_off, head stride d */
    void* out;             /* [batch * seq][o_tok], heads d apart */
    const void* gate;      /* may be null; [batch * seq][gate_tok], heads d apart */
    const int* start;
    const int* slots;
    float* scratch;        /* zkfp_grouped_scratch() floats */
    long long slot_stride, pitch, capacity, v_off, o_tok, gate_tok;
    long long batch, seq;
    int heads, kv_heads, d, window, max_keys, dtype;
    float scale, out_scale;
} zkfp_grouped_args;
int zkfp_grouped_attention(const zkfp_grouped_args* a, void* stream);
long long zkfp_grouped_scratch(const zkfp_grouped_args* a);

/* Causal convolution per channel and silu: out[t][c] = silu(b[c] + sum_j w[j][c] * x[t - taps + 1 + j][c]).  `state`
 * holds the taps - 1 inputs before the step and is left with the last ones after it; at position 0 it counts as zero. */
typedef struct {
    const void* x;         /* [rows][ldx] */
    const float* w;        /* [taps][channels] */
    const float* b;        /* [channels] */
    void* out;             /* [rows][ldo] */
    void* state;           /* [slot][taps - 1][channels], dtype */
    const int* start;
    const int* slots;
    long long ldx, ldo, batch, seq, n_slots;
    int channels, taps, dtype;
} zkfp_conv_args;
int zkfp_short_conv(const zkfp_conv_args* a, void* stream);

/* Linear attention with a decaying 32-bit state per (sequence, head):
 *   S_t = a_t S_{t-1} + w_t k_t v_t^T,  out_t = S_t^T q_t + skip v_t
 * step null:  a_t = decay[head], w_t = k_scale
 * otherwise   d_t = softplus(step[row][head] + step_bias[head]), a_t = exp(-decay[head] d_t), w_t = k_scale d_t
 * At position 0 the state counts as zero. */
typedef struct {
    const void* q;         /* [rows][tok], head h at (h / heads_per_qk) * qk_head, dtype; likewise k */
    const void* k;
    const void* v;         /* [rows][v_tok], head h at h * v_head */
    void* out;             /* [rows][o_tok], heads o_head apart */
    const float* decay;
    const float* step;
    const float* step_bias;
    const float* skip;     /* may be null: [heads] */
    float* state;          /* [slot][heads][n][p] */
    float* scratch;        /* zkfp_scan_scratch() floats, may be null */
    const int* start;
    const int* slots;
    long long q_tok, k_tok, v_tok, o_tok, qk_head, v_head, o_head, step_tok;
    long long batch, seq, heads, n_slots;
    int heads_per_qk, n, p, dtype;
    float k_scale;
} zkfp_scan_args;
int zkfp_scan(const zkfp_scan_args* a, void* stream);
long long zkfp_scan_scratch(const zkfp_scan_args* a);

/* Norm of equal parts of a row together with its silu gate:
 *   weight null:  out = scale * silu(g) * x / rms_part(x)
 *   otherwise     y = silu(g) * x, out = weight * y / rms_part(y)
 * Rows hold heads of `vdim` values, p apart; a part is `part` consecutive values, head boundaries not counted. */
typedef struct {
    const void* x;         /* [rows][ldx] */
    const void* g;         /* [rows][ldg] */
    const float* weight;   /* [heads * p] or null */
    void* out;             /* [rows][ldo] */
    long long ldx, ldg, ldo, rows;
    int heads, vdim, p, part, dtype;
    float scale;
    double eps;
} zkfp_gated_norm_args;
int zkfp_gated_norm(const zkfp_gated_norm_args* a, void* stream);

/* which kernel a call takes: 0 plain CUDA cores, 1 tensor cores, 2 weight streaming; for tests and reports */
int zkfp_linear_path(const zkfp_linear_args* a);
int zkfp_attention_path(const zkfp_attention_args* a);
int zkfp_scan_path(const zkfp_scan_args* a);

/* 5 if a finished kernel gave up a bounded wait since the last call, else 0 */
int zkfp_device_status(void);
long long zkfp_launches(void);      /* kernels launched by this library so far */
int zkfp_cuda_error(void);          /* cudaError_t behind the last status 3 of this thread */

#ifdef __cplusplus
}
#endif
#endif
