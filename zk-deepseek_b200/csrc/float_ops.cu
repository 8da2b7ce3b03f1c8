// Streaming kernels of the floating-point decoders: embedding, norms, latent post-processing, the per-head
// products of the absorbed form, and the plain attention kernel that takes any size in either number format.
// Norms, rotations and the residual are 32-bit whatever the activations are.
#include "float_common.cuh"

namespace zkds {

namespace {

template <typename T>
__global__ void __launch_bounds__(256)
embed_kernel(const long long* __restrict__ tokens, const T* __restrict__ table, long long ld_table, long long vocab,
             float* __restrict__ x, bf16* __restrict__ xb, long long ldx, float scale)
{
    const long long r = blockIdx.x, t = tokens[r];
    const bool ok = t >= 0 && t < vocab;
    for (long long c = threadIdx.x * 8; c < ldx; c += 256 * 8) {
        float v[8] = {};
        if (ok) load8(table + t * ld_table + c, v);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= scale;
        store8(x + r * ldx + c, v);
        if (xb) store8(xb + r * ldx + c, v);
    }
}

__device__ __forceinline__ float sum_squares8(const float (&v)[8])
{
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s = fmaf(v[i], v[i], s);
    return s;
}

// x += w * y / rms(y), then h = x or, with w2, h = w2 * x / rms(x): one block per row; what does not fit the registers
// is found again in L1 / L2
template <typename T>
__global__ void __launch_bounds__(256)
add_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w,
                const float* __restrict__ w2, T* __restrict__ h, long long ldx, long long ldy, int width, int padded,
                float eps)
{
    __shared__ float red[8];
    const long long r = blockIdx.x;
    float* xr = x + r * ldx;
    const float* yr = y + r * ldy;
    T* hr = h + r * ldx;
    constexpr int KEEP = 4;               // 8192 values stay in registers
    float keep[KEEP][8];
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 256 + threadIdx.x) * 8;
        if (c < padded) {
            load8(yr + c, keep[k]);
            s += sum_squares8(keep[k]);
        }
    }
    for (int c = (KEEP * 256 + threadIdx.x) * 8; c < padded; c += 256 * 8) {
        float v[8];
        load8(yr + c, v);
        s += sum_squares8(v);
    }
    s = block_sum(s, red);
    const float rs = 1.0f / sqrtf(s / (float)width + eps);
    s = 0.f;
    auto apply = [&](int c, float (&v)[8]) {          // leaves the new x in v
        float a[8], g[8];
        load8(xr + c, a);
        load8(w + c, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = a[i] + v[i] * rs * g[i];
        store8(xr + c, v);
        if (w2) s += sum_squares8(v);
        else if (h) store8(hr + c, v);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 256 + threadIdx.x) * 8;
        if (c < padded) apply(c, keep[k]);
    }
    for (int c = (KEEP * 256 + threadIdx.x) * 8; c < padded; c += 256 * 8) {
        float v[8];
        load8(yr + c, v);
        apply(c, v);
    }
    if (!w2) return;
    s = block_sum(s, red);
    const float rx = 1.0f / sqrtf(s / (float)width + eps);
    auto write = [&](int c, const float (&v)[8]) {
        float g[8];
        load8(w2 + c, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) g[i] *= v[i] * rx;
        store8(hr + c, g);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 256 + threadIdx.x) * 8;
        if (c < padded) write(c, keep[k]);
    }
    for (int c = (KEEP * 256 + threadIdx.x) * 8; c < padded; c += 256 * 8) {
        float v[8];
        load8(xr + c, v);                 // written by this thread above
        write(c, v);
    }
}

// out = w * x / rms(x) of one row by the whole block
template <typename T>
__device__ __forceinline__ void norm_row(const float* xr, const float* w, T* out, int width, int padded, float eps,
                                         float* red)
{
    float s = 0.f;
    for (int c = threadIdx.x * 8; c < padded; c += blockDim.x * 8) {
        float v[8];
        load8(xr + c, v);
        s += sum_squares8(v);
    }
    s = block_sum(s, red);
    const float rs = 1.0f / sqrtf(s / (float)width + eps);
    for (int c = threadIdx.x * 8; c < padded; c += blockDim.x * 8) {
        float v[8], g[8];
        load8(xr + c, v);
        load8(w + c, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = v[i] * rs * g[i];
        store8(out + c, v);
    }
}

template <typename T>
__global__ void __launch_bounds__(256)
norm_rows_kernel(const float* __restrict__ x, long long ldx, const int* __restrict__ index, const float* __restrict__ w,
                 T* __restrict__ out, long long ldo, int width, int padded, float eps)
{
    __shared__ float red[8];
    const long long r = index ? index[blockIdx.x] : (long long)blockIdx.x;
    norm_row(x + r * ldx, w, out + blockIdx.x * ldo, width, padded, eps, red);
}

// blockIdx.y 0: the query latent; 1: the key/value latent, the rotated key part, both into the cache
template <typename T>
__global__ void __launch_bounds__(256)
latent_post_kernel(const zkfp_latent_args a)
{
    __shared__ float red[8];
    const long long r = blockIdx.x;
    const float* yr = a.y + r * a.ldy;
    if (blockIdx.y == 0) {
        norm_row(yr, a.wq, (T*)a.cq + r * a.ldq, a.q_rank, a.q_pad, (float)a.eps, red);
        return;
    }
    const int b = (int)(r / a.seq);
    const int pos = a.start[b] + (int)(r - (long long)b * a.seq);
    if (pos < 0 || pos >= a.capacity) return;
    T* row = (T*)a.cache + a.slots[b] * a.slot_stride + (long long)pos * a.pitch;
    norm_row(yr + a.q_pad, a.wc, row, a.c, a.c_pad, (float)a.eps, red);
    const float* kr = yr + a.q_pad + a.c_pad;
    const float2* tab = (const float2*)a.table + (long long)pos * a.pairs;
    for (int i = threadIdx.x; i < (int)(a.pitch - a.c_pad) / 2; i += blockDim.x) {
        float u = 0.f, v = 0.f;
        if (i < a.pairs) {
            const float2 cs = tab[i];
            const float p = kr[2 * i], q = kr[2 * i + 1];
            u = p * cs.x - q * cs.y;
            v = q * cs.x + p * cs.y;
        }
        row[a.c_pad + 2 * i] = from_f32<T>(u);
        row[a.c_pad + 2 * i + 1] = from_f32<T>(v);
    }
}

// ---- per-head products of the absorbed form --------------------------------------------------------------
constexpr int kPerHeadTokens = 4;       // tokens that share one pass over the weights

// out[t][h][c] = sum_d x[t][h][d] * W[h][d][c].  A thread owns eight columns, the block's eight warps split d.
// grid (heads, columns / 256, token groups)
template <typename T>
__global__ void __launch_bounds__(256)
perhead_absorb_kernel(const zkfp_perhead_args a)
{
    __shared__ float part[8][256];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, c = (blockIdx.y * 32 + lane) * 8;
    const long long t0 = (long long)blockIdx.z * kPerHeadTokens;
    const int nt = (int)(a.tokens - t0 < kPerHeadTokens ? a.tokens - t0 : kPerHeadTokens);
    const T* W = (const T*)a.W + h * a.w_head;
    const T* x = (const T*)a.x + t0 * a.x_tok + h * a.x_head;
    T* out = (T*)a.out + t0 * a.o_tok + h * a.o_head;
    float acc[kPerHeadTokens][8] = {};
    if (c < a.n_out) {
#pragma unroll 4
        for (int d = warp; d < a.n_in; d += 8) {
            float w[8];
            load8(W + d * a.ldw + c, w);
#pragma unroll
            for (int t = 0; t < kPerHeadTokens; ++t) {
                if (t < nt) {
                    const float q = to_f32(x[t * a.x_tok + d]);
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[t][i] = fmaf(q, w[i], acc[t][i]);
                }
            }
        }
    }
#pragma unroll
    for (int t = 0; t < kPerHeadTokens; ++t) {
        if (t >= nt) break;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) part[warp][i * 32 + lane] = acc[t][i];     // column lane * 8 + i at i * 32 + lane
        __syncthreads();
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) s += part[k][threadIdx.x];
        const int col = blockIdx.y * 256 + (threadIdx.x & 31) * 8 + (threadIdx.x >> 5);
        if (col < a.n_out) out[t * a.o_tok + col] = from_f32<T>(s);
    }
    if (blockIdx.y == 0)
        for (int i = threadIdx.x; i < a.copy_n * nt; i += 256) {
            const int t = i / a.copy_n, k = i - t * a.copy_n;
            out[t * a.o_tok + a.copy_to + k] = x[t * a.x_tok + a.copy_from + k];
        }
}

// out[t][h][v] = sum_c x[t][h][c] * W[h][v][c]: one warp per output row.  grid (rows / 8, heads, token groups)
template <typename T>
__global__ void __launch_bounds__(256)
perhead_expand_kernel(const zkfp_perhead_args a)
{
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y, v = blockIdx.x * 8 + warp;
    if (v >= a.n_out) return;
    const long long t0 = (long long)blockIdx.z * kPerHeadTokens;
    const int nt = (int)(a.tokens - t0 < kPerHeadTokens ? a.tokens - t0 : kPerHeadTokens);
    const T* W = (const T*)a.W + h * a.w_head + v * a.ldw;
    const T* x = (const T*)a.x + t0 * a.x_tok + h * a.x_head;
    float acc[kPerHeadTokens] = {};
    for (int c = lane * 8; c < a.n_in; c += 256) {
        float w[8];
        load8(W + c, w);
#pragma unroll
        for (int t = 0; t < kPerHeadTokens; ++t) {
            if (t < nt) {
                float q[8];
                load8(x + t * a.x_tok + c, q);
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[t] = fmaf(q[i], w[i], acc[t]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < kPerHeadTokens; ++t) {
        if (t >= nt) break;
        const float s = warp_sum(acc[t]);
        if (lane == 0) ((T*)a.out)[(t0 + t) * a.o_tok + h * a.o_head + v] = from_f32<T>(s);
    }
}

// ---- plain attention ------------------------------------------------------------------------------------------
// A block handles ROWS query rows that read the same keys: consecutive tokens of one head (expanded form) or
// consecutive (token, head) pairs (shared form).  Keys come in tiles of 32; scores, weights and running sums are
// 32-bit in shared memory.
constexpr int kRows = 16, kKeys = 32, kDimChunk = 64;

template <typename T>
__global__ void __launch_bounds__(256)
attention_plain_kernel(const zkfp_attention_args a)
{
    extern __shared__ float sm[];
    const int dk = a.d1 + a.d2;
    float* Q = sm;                                   // [kRows][dk]
    float* O = Q + kRows * dk;                       // [kRows][dv]
    float* K = O + kRows * a.dv;                     // [kKeys][kDimChunk + 1]
    float* P = K + kKeys * (kDimChunk + 1);          // [kRows][kKeys]
    float* alpha = P + kRows * kKeys;                // [kRows]
    float* mrow = alpha + kRows;
    float* lrow = mrow + kRows;
    const int b = blockIdx.z, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kv_head = a.heads_per_kv > 1 ? head / a.heads_per_kv : head;
    const long long row0 = (long long)blockIdx.x * kRows;
    const long long rows = a.shared ? a.seq * a.heads : a.seq;
    const int per_tok = a.shared ? (int)a.heads : 1;
    const int start = a.start[b];
    if (start < 0 || start + a.seq > a.base + a.keys) return;      // not a step of these keys
    const long long slot = a.slots ? a.slots[b] : b;
    const T* q = (const T*)a.q + (long long)b * a.seq * a.heads * a.q_head;
    T* out = (T*)a.out + (long long)b * a.seq * a.heads * a.o_head;
    const T* k1 = (const T*)a.k1 + slot * a.slot_stride + (a.shared ? 0 : kv_head * a.k1_head);
    const T* k2 = (const T*)a.k2 + slot * a.slot_stride;
    const T* v = (const T*)a.v + slot * a.slot_stride + (a.shared ? 0 : kv_head * a.v_head);
    const int nrow = (int)(rows - row0 < kRows ? rows - row0 : kRows);
    auto flat = [&](int i) { return a.shared ? row0 + i : (row0 + i) * a.heads + head; };   // (token, head) pair
    for (int i = threadIdx.x; i < kRows * dk; i += 256) {
        const int rr = i / dk, d = i - rr * dk;
        Q[i] = rr < nrow ? to_f32(q[flat(rr) * a.q_head + d]) : 0.f;
    }
    for (int i = threadIdx.x; i < kRows * a.dv; i += 256) O[i] = 0.f;
    if (threadIdx.x < kRows) { mrow[threadIdx.x] = -INFINITY; lrow[threadIdx.x] = 0.f; }
    const int first = start + (int)(row0 / per_tok), last = start + (int)((row0 + nrow - 1) / per_tok);
    int lo = a.window > 0 ? first - a.window + 1 : 0;
    if (lo < (int)a.base) lo = (int)a.base;
    for (int j0 = lo; j0 <= last; j0 += kKeys) {
        const int nk = last - j0 + 1 < kKeys ? last - j0 + 1 : kKeys;
        float s0 = 0.f, s1 = 0.f;                     // rows warp and warp + 8, key lane
        for (int d0 = 0; d0 < dk; d0 += kDimChunk) {
            __syncthreads();
            for (int i = threadIdx.x; i < kKeys * kDimChunk; i += 256) {
                const int kk = i / kDimChunk, d = d0 + i % kDimChunk;
                float val = 0.f;
                if (kk < nk && d < dk) {
                    const long long p = j0 + kk - a.base;
                    val = d < a.d1 ? to_f32(k1[p * a.k1_tok + d]) : to_f32(k2[p * a.k2_tok + d - a.d1]);
                }
                K[kk * (kDimChunk + 1) + i % kDimChunk] = val;
            }
            __syncthreads();
            const int nd = dk - d0 < kDimChunk ? dk - d0 : kDimChunk;
            for (int d = 0; d < nd; ++d) {
                const float kv = K[lane * (kDimChunk + 1) + d];
                s0 = fmaf(Q[warp * dk + d0 + d], kv, s0);
                s1 = fmaf(Q[(warp + 8) * dk + d0 + d], kv, s1);
            }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int rr = warp + 8 * half;
            const int i = start + (int)((row0 + rr) / per_tok), j = j0 + lane;
            const bool seen = rr < nrow && lane < nk && j <= i && (a.window <= 0 || i - j < a.window);
            const float s = seen ? (half ? s1 : s0) * a.scale : -INFINITY;
            const float m_old = mrow[rr], m_new = fmaxf(m_old, warp_max(s));
            const float p = seen ? expf(s - m_new) : 0.f;
            const float l = warp_sum(p);
            const float al = m_old == -INFINITY ? 0.f : expf(m_old - m_new);
            P[rr * kKeys + lane] = p;
            __syncwarp();
            if (lane == 0) {
                alpha[rr] = al;
                mrow[rr] = m_new;
                lrow[rr] = lrow[rr] * al + l;
            }
        }
        __syncthreads();
        for (int d = threadIdx.x; d < a.dv; d += 256) {
            float acc[kRows];
#pragma unroll
            for (int rr = 0; rr < kRows; ++rr) acc[rr] = O[rr * a.dv + d] * alpha[rr];
            for (int kk = 0; kk < nk; ++kk) {
                const float vv = to_f32(v[(j0 + kk - a.base) * a.v_tok + d]);
#pragma unroll
                for (int rr = 0; rr < kRows; ++rr) acc[rr] = fmaf(P[rr * kKeys + kk], vv, acc[rr]);
            }
#pragma unroll
            for (int rr = 0; rr < kRows; ++rr) O[rr * a.dv + d] = acc[rr];
        }
        __syncthreads();
    }
    for (int i = threadIdx.x; i < nrow * a.dv; i += 256) {
        const int rr = i / a.dv, d = i - rr * a.dv;
        float o = O[i] / lrow[rr];
        if (a.gate) o *= sigmoid_f(to_f32(((const T*)a.gate)[(row0 + rr) * a.gate_tok + head * a.gate_head + d])) * a.out_scale;
        if (a.o_tok) out[(row0 + rr) * a.o_tok + head * a.o_head + d] = from_f32<T>(o);
        else out[flat(rr) * a.o_head + d] = from_f32<T>(o);
    }
}

}  // namespace

template <typename T>
static int attention_plain(const zkfp_attention_args& a, cudaStream_t st)
{
    const size_t smem = sizeof(float) * ((size_t)kRows * (a.d1 + a.d2 + a.dv) + kKeys * (kDimChunk + 1) + kRows * kKeys +
                                         3 * kRows);
    if (smem > (size_t)kSharedMax) return ZKDS_ERR_UNSUPPORTED;
    // always the same limit: a captured launch keeps its own size, but is run under the function's current attribute
    ZKDS_CUDA(cudaFuncSetAttribute(attention_plain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSharedMax));
    const long long rows = a.shared ? a.seq * a.heads : a.seq;
    const dim3 grid((unsigned)((rows + kRows - 1) / kRows), a.shared ? 1u : (unsigned)a.heads, (unsigned)a.batch);
    attention_plain_kernel<T><<<grid, 256, smem, st>>>(a);
    return fp_launched();
}

int launch_attention_plain(const zkfp_attention_args& a, cudaStream_t st)
{
    return a.dtype == ZKFP_BF16 ? attention_plain<bf16>(a, st) : attention_plain<float>(a, st);
}

}  // namespace zkds

using namespace zkds;

extern "C" {

int zkfp_embed(const long long* tokens, const void* table, long long ld_table, long long vocab, float* x, void* xb,
               long long ldx, long long rows, float scale, int dtype, void* stream)
{
    if (!tokens || !table || !x || rows < 0 || (ldx & 7) || ld_table < ldx) return ZKDS_ERR_ARG;
    if (rows == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == ZKFP_BF16)
        embed_kernel<bf16><<<(unsigned)rows, 256, 0, st>>>(tokens, (const bf16*)table, ld_table, vocab, x, (bf16*)xb, ldx, scale);
    else
        embed_kernel<float><<<(unsigned)rows, 256, 0, st>>>(tokens, (const float*)table, ld_table, vocab, x, (bf16*)xb, ldx, scale);
    return fp_launched();
}

int zkfp_add_norm(float* x, const float* y, const float* w, const float* w2, void* h, long long ldx, long long ldy,
                  long long rows, long long width, double eps, int h_dtype, void* stream)
{
    if (!x || !y || !w || (w2 && !h) || rows < 0 || width <= 0 || (ldx & 7) || (ldy & 7) || ldy < ldx || ldx < width) return ZKDS_ERR_ARG;
    if (rows == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    if (h_dtype == ZKFP_BF16)
        add_norm_kernel<bf16><<<(unsigned)rows, 256, 0, st>>>(x, y, w, w2, (bf16*)h, ldx, ldy, (int)width, (int)ldx, (float)eps);
    else
        add_norm_kernel<float><<<(unsigned)rows, 256, 0, st>>>(x, y, w, w2, (float*)h, ldx, ldy, (int)width, (int)ldx, (float)eps);
    return fp_launched();
}

int zkfp_norm_rows(const float* x, long long ldx, const int* index, const float* w, void* out, long long ldo,
                   long long n, long long width, double eps, int dtype, void* stream)
{
    if (!x || !w || !out || n < 0 || width <= 0 || (ldx & 7) || ldx < width || ldo < ldx) return ZKDS_ERR_ARG;
    if (n == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == ZKFP_BF16)
        norm_rows_kernel<bf16><<<(unsigned)n, 256, 0, st>>>(x, ldx, index, w, (bf16*)out, ldo, (int)width, (int)ldx, (float)eps);
    else
        norm_rows_kernel<float><<<(unsigned)n, 256, 0, st>>>(x, ldx, index, w, (float*)out, ldo, (int)width, (int)ldx, (float)eps);
    return fp_launched();
}

int zkfp_latent_post(const zkfp_latent_args* a, void* stream)
{
    if (!a || !a->y || !a->cq || !a->wq || a->rows < 0 || a->seq <= 0 || (a->q_pad & 7) || (a->c_pad & 7)) return ZKDS_ERR_ARG;
    if (a->own_kv && (!a->wc || !a->cache || !a->start || !a->slots || !a->table || (a->pitch & 7))) return ZKDS_ERR_ARG;
    if (a->rows == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 grid((unsigned)a->rows, a->own_kv ? 2u : 1u);
    if (a->dtype == ZKFP_BF16) latent_post_kernel<bf16><<<grid, 256, 0, st>>>(*a);
    else latent_post_kernel<float><<<grid, 256, 0, st>>>(*a);
    return fp_launched();
}

int zkfp_perhead(const zkfp_perhead_args* a, void* stream)
{
    if (!a || !a->x || !a->W || !a->out || a->tokens < 0 || a->heads <= 0 || (a->n_out & 7) || (a->n_in & 7) ||
        (a->ldw & 7) || ((a->x_tok | a->x_head | a->o_tok | a->o_head | a->w_head) & 7))
        return ZKDS_ERR_ARG;
    if (a->tokens == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const unsigned tz = (unsigned)((a->tokens + kPerHeadTokens - 1) / kPerHeadTokens);
    if (a->transposed) {
        const dim3 grid((unsigned)a->heads, (unsigned)((a->n_out + 255) / 256), tz);
        if (a->dtype == ZKFP_BF16) perhead_absorb_kernel<bf16><<<grid, 256, 0, st>>>(*a);
        else perhead_absorb_kernel<float><<<grid, 256, 0, st>>>(*a);
    } else {
        const dim3 grid((unsigned)((a->n_out + 7) / 8), (unsigned)a->heads, tz);
        if (a->dtype == ZKFP_BF16) perhead_expand_kernel<bf16><<<grid, 256, 0, st>>>(*a);
        else perhead_expand_kernel<float><<<grid, 256, 0, st>>>(*a);
    }
    return fp_launched();
}

}  // extern "C"
