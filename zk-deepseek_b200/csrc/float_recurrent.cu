// Layers with a recurrent state: short convolution, linear attention with a decaying state token by token, and the gated
// norm behind both.  States, decays, step sizes and norms are 32-bit in both number formats.
#include "float_common.cuh"

namespace zkds {

namespace {

// ---- short convolution -------------------------------------------------------------------------------------------
// A thread owns eight channels of a tile of tokens.  The threads of a sequence's first tile read the inputs before the
// step from the state, and are the ones that replace it.  TAPS 0: any number of taps, inputs read again for every tap.
constexpr int kConvTokens = 32, kConvBatch = 8;    // tokens of a tile, and those whose inputs are in flight together

template <typename T>
__device__ __forceinline__ void conv_input(const zkfp_conv_args& a, const T* x, const T* state, int t, int c, bool fresh,
                                           float (&v)[8])
{
    if (t >= 0) load8(x + t * a.ldx + c, v);
    else if (!fresh) load8(state + (long long)(a.taps - 1 + t) * a.channels + c, v);
    else {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = 0.f;
    }
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_kernel(const zkfp_conv_args a)
{
    const int c = (int)(blockIdx.x * 128 + threadIdx.x) * 8, b = blockIdx.z, t0 = blockIdx.y * kConvTokens;
    const int t1 = min(t0 + kConvTokens, (int)a.seq), taps = TAPS ? TAPS : a.taps;
    const long long slot = a.slots[b];
    if (c >= a.channels || slot < 0 || slot >= a.n_slots) return;
    const bool fresh = a.start[b] == 0;
    const T* x = (const T*)a.x + (long long)b * a.seq * a.ldx;
    T* out = (T*)a.out + (long long)b * a.seq * a.ldo + c;
    T* state = (T*)a.state + slot * (taps - 1) * a.channels;
    float bias[8];
    load8(a.b + c, bias);
    if constexpr (TAPS > 0) {
        float w[TAPS][8], ring[TAPS][8];                 // ring[j]: input of token t - TAPS + 1 + j
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load8(a.w + (long long)j * a.channels + c, w[j]);
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) conv_input(a, x, state, t0 - (TAPS - 1) + j, c, fresh, ring[j]);
        for (int tb = t0; tb < t1; tb += kConvBatch) {
            uint4 raw[kConvBatch][sizeof(T) / 2];
#pragma unroll
            for (int k = 0; k < kConvBatch; ++k)
                if (tb + k < t1)
#pragma unroll
                    for (int q = 0; q < (int)sizeof(T) / 2; ++q) raw[k][q] = reinterpret_cast<const uint4*>(x + (tb + k) * a.ldx + c)[q];
#pragma unroll
            for (int k = 0; k < kConvBatch; ++k) {
                if (tb + k >= t1) break;
                load8(reinterpret_cast<const T*>(raw[k]), ring[TAPS - 1]);
                float v[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    v[i] = bias[i];
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) v[i] = fmaf(w[j][i], ring[j][i], v[i]);
                    v[i] *= sigmoid_for<T>(v[i]);
                }
                store8(out + (tb + k) * a.ldo, v);
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
                    for (int i = 0; i < 8; ++i) ring[j][i] = ring[j + 1][i];
            }
        }
    } else {
        for (int t = t0; t < t1; ++t) {
            float v[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = bias[i];
            for (int j = 0; j < taps; ++j) {
                float w[8], in[8];
                load8(a.w + (long long)j * a.channels + c, w);
                conv_input(a, x, state, t - (taps - 1) + j, c, fresh, in);
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] = fmaf(w[i], in[i], v[i]);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= sigmoid_for<T>(v[i]);
            store8(out + t * a.ldo, v);
        }
    }
    if (blockIdx.y == 0)                                 // oldest first: an entry is read before it is replaced
        for (int j = 0; j < taps - 1; ++j) {
            float v[8];
            conv_input(a, x, state, (int)a.seq - (taps - 1) + j, c, fresh, v);
            store8(state + (long long)j * a.channels + c, v);
        }
}

template <typename T>
int short_conv(const zkfp_conv_args& a, cudaStream_t st)
{
    const dim3 grid((unsigned)((a.channels / 8 + 127) / 128), (unsigned)((a.seq + kConvTokens - 1) / kConvTokens), (unsigned)a.batch);
    if (grid.y > 65535u) return ZKDS_ERR_UNSUPPORTED;
    switch (a.taps) {
    case 2: short_conv_kernel<T, 2><<<grid, 128, 0, st>>>(a); break;
    case 3: short_conv_kernel<T, 3><<<grid, 128, 0, st>>>(a); break;
    case 4: short_conv_kernel<T, 4><<<grid, 128, 0, st>>>(a); break;
    default: short_conv_kernel<T, 0><<<grid, 128, 0, st>>>(a);
    }
    return fp_launched();
}

// ---- linear attention with a decaying state, token by token ---------------------------------------------------------
// A block holds 32 columns of one head's state in registers: a warp has NR rows of it, a lane one column.  Tokens come in
// tiles of kScanTokens; within a tile nothing waits, the row sums of the eight warps meet at its end.
constexpr int kScanTokens = 8;

template <typename T, int NR>
__global__ void __launch_bounds__(256)
scan_kernel(const zkfp_scan_args a)
{
    constexpr int N = 8 * NR;
    __shared__ float qs[kScanTokens][N], ks[kScanTokens][N], vs[kScanTokens][32], part[kScanTokens][8][32];
    __shared__ float as[kScanTokens], ws[kScanTokens];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, b = blockIdx.z, head = blockIdx.y;
    const int p0 = blockIdx.x * 32, col = p0 + lane;
    const long long slot = a.slots[b];
    if (slot < 0 || slot >= a.n_slots) return;
    const bool col_ok = col < a.p;
    float* state = a.state + ((slot * a.heads + head) * a.n + warp * NR) * a.p + col;
    const int nrows = max(0, min(NR, a.n - warp * NR));
    float S[NR];
    const bool fresh = a.start[b] == 0;
#pragma unroll
    for (int i = 0; i < NR; ++i) S[i] = !fresh && col_ok && i < nrows ? state[(long long)i * a.p] : 0.f;
    const long long row0 = (long long)b * a.seq;
    const long long qk_off = (long long)(head / a.heads_per_qk) * a.qk_head;
    const T* q = (const T*)a.q + row0 * a.q_tok + qk_off;
    const T* k = (const T*)a.k + row0 * a.k_tok + qk_off;
    const T* v = (const T*)a.v + row0 * a.v_tok + head * a.v_head;
    T* out = (T*)a.out + row0 * a.o_tok + head * a.o_head;
    const float decay = a.decay[head], skip = a.skip ? a.skip[head] : 0.f;
    for (int t0 = 0; t0 < a.seq; t0 += kScanTokens) {
        const int nt = min(kScanTokens, (int)a.seq - t0);
        __syncthreads();
        for (int i = tid; i < kScanTokens * (N / 8); i += 256) {
            const int t = i / (N / 8), c = (i - t * (N / 8)) * 8;
            float x[8] = {}, y[8] = {};
            if (t < nt && c < a.n) {
                load8(q + (t0 + t) * a.q_tok + c, x);
                load8(k + (t0 + t) * a.k_tok + c, y);
            }
            store8(&qs[t][c], x);
            store8(&ks[t][c], y);
        }
        {
            const int t = warp;                          // eight warps, eight tokens
            vs[t][lane] = t < nt && col_ok ? to_f32(v[(t0 + t) * a.v_tok + col]) : 0.f;
            if (lane == 0) {
                float at = decay, wt = a.k_scale;
                if (a.step && t < nt) {
                    const float dt = softplus_f(a.step[(row0 + t0 + t) * a.step_tok + head] + a.step_bias[head]);
                    at = expf(-decay * dt);
                    wt = a.k_scale * dt;
                }
                as[t] = at;
                ws[t] = wt;
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float at = as[t], wv = ws[t] * vs[t][lane];
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int i = 0; i < NR; i += 4) {
                const float4 kk = *reinterpret_cast<const float4*>(&ks[t][warp * NR + i]);
                const float4 qq = *reinterpret_cast<const float4*>(&qs[t][warp * NR + i]);
                S[i] = fmaf(at, S[i], kk.x * wv);
                S[i + 1] = fmaf(at, S[i + 1], kk.y * wv);
                S[i + 2] = fmaf(at, S[i + 2], kk.z * wv);
                S[i + 3] = fmaf(at, S[i + 3], kk.w * wv);
                y0 = fmaf(qq.x, S[i], y0);
                y1 = fmaf(qq.y, S[i + 1], y1);
                y0 = fmaf(qq.z, S[i + 2], y0);
                y1 = fmaf(qq.w, S[i + 3], y1);
            }
            part[t][warp][lane] = y0 + y1;
        }
        __syncthreads();
        if (warp < nt && col_ok) {
            float y = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) y += part[warp][w][lane];
            out[(t0 + warp) * a.o_tok + col] = from_f32<T>(fmaf(skip, vs[warp][lane], y));
        }
    }
    if (col_ok)
#pragma unroll
        for (int i = 0; i < NR; ++i)
            if (i < nrows) state[(long long)i * a.p] = S[i];
}

template <typename T>
int scan(const zkfp_scan_args& a, cudaStream_t st)
{
    const dim3 grid((unsigned)((a.p + 31) / 32), (unsigned)a.heads, (unsigned)a.batch);
    if (a.n <= 32) scan_kernel<T, 4><<<grid, 256, 0, st>>>(a);
    else if (a.n <= 64) scan_kernel<T, 8><<<grid, 256, 0, st>>>(a);
    else if (a.n <= 128) scan_kernel<T, 16><<<grid, 256, 0, st>>>(a);
    else if (a.n <= 256) scan_kernel<T, 32><<<grid, 256, 0, st>>>(a);
    else if (a.n <= 512) scan_kernel<T, 64><<<grid, 256, 0, st>>>(a);
    else return ZKDS_ERR_UNSUPPORTED;
    return fp_launched();
}

// ---- gated norm --------------------------------------------------------------------------------------------------
// Parts that are contiguous runs of whole 8-element vectors (a head with its zero padding, or several whole heads without
// any): THREADS threads take one part of one row and keep KEEP vectors each.  FIRST: the gate comes before the norm.
template <typename T, int THREADS, int KEEP, bool FIRST>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const zkfp_gated_norm_args a, int parts, int stride)
{
    __shared__ float red[8];
    const long long unit = (long long)blockIdx.x * (256 / THREADS) + threadIdx.x / THREADS;
    if (unit >= a.rows * parts) return;                  // whole warps, or the whole block
    const long long r = unit / parts;
    const int c0 = (int)(unit - r * parts) * stride, lane = threadIdx.x % THREADS;
    const T* x = (const T*)a.x + r * a.ldx + c0;
    const T* g = (const T*)a.g + r * a.ldg + c0;
    T* out = (T*)a.out + r * a.ldo + c0;
    float y[KEEP][8], z[FIRST ? 1 : KEEP][8];
    float s = 0.f;
    auto load = [&](int c, float (&v)[8], float (&u)[8]) {
        load8(x + c, v);
        load8(g + c, u);
#pragma unroll
        for (int i = 0; i < 8; ++i) u[i] *= sigmoid_for<T>(u[i]);
        if (FIRST) {
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= u[i];
        }
    };
    auto add = [&](const float (&v)[8]) {
#pragma unroll
        for (int i = 0; i < 8; ++i) s = fmaf(v[i], v[i], s);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * THREADS + lane) * 8;
        if (c < stride) {
            load(c, y[k], z[FIRST ? 0 : k]);
            add(y[k]);
        }
    }
    for (int c = (KEEP * THREADS + lane) * 8; c < stride; c += THREADS * 8) {
        float v[8], u[8];
        load(c, v, u);
        add(v);
    }
    s = THREADS == 32 ? warp_sum(s) : block_sum(s, red);
    const float rs = 1.0f / sqrtf(s / (float)a.part + (float)a.eps);
    auto write = [&](int c, float (&v)[8], const float (&u)[8]) {
        if (FIRST) {
            float w[8];
            load8(a.weight + c0 + c, w);
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= rs * w[i];
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= rs * u[i] * a.scale;
        }
        store8(out + c, v);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * THREADS + lane) * 8;
        if (c < stride) write(c, y[k], z[FIRST ? 0 : k]);
    }
    for (int c = (KEEP * THREADS + lane) * 8; c < stride; c += THREADS * 8) {
        float v[8], u[8];
        load(c, v, u);
        write(c, v, u);
    }
}

// any part: a block per part of a row, elements one by one
template <typename T>
__global__ void __launch_bounds__(256)
gated_norm_any_kernel(const zkfp_gated_norm_args a, int parts)
{
    __shared__ float red[8];
    const long long r = blockIdx.x / parts;
    const int part = (int)(blockIdx.x - r * parts);
    const T* x = (const T*)a.x + r * a.ldx;
    const T* g = (const T*)a.g + r * a.ldg;
    T* out = (T*)a.out + r * a.ldo;
    auto at = [&](int e) {
        const int h = e / a.vdim;
        return h * a.p + e - h * a.vdim;
    };
    auto gate = [&](int c) {
        const float u = to_f32(g[c]);
        return u * sigmoid_for<T>(u);
    };
    float s = 0.f;
    for (int e = part * a.part + threadIdx.x; e < (part + 1) * a.part; e += 256) {
        const int c = at(e);
        const float v = to_f32(x[c]) * (a.weight ? gate(c) : 1.f);
        s = fmaf(v, v, s);
    }
    s = block_sum(s, red);
    const float rs = 1.0f / sqrtf(s / (float)a.part + (float)a.eps);
    for (int e = part * a.part + threadIdx.x; e < (part + 1) * a.part; e += 256) {
        const int c = at(e);
        out[c] = from_f32<T>(to_f32(x[c]) * gate(c) * rs * (a.weight ? a.weight[c] : a.scale));
    }
    if (part == 0 && a.p > a.vdim)                       // padding of every head
        for (int e = threadIdx.x; e < a.heads * (a.p - a.vdim); e += 256) {
            const int h = e / (a.p - a.vdim);
            out[h * a.p + a.vdim + e - h * (a.p - a.vdim)] = from_f32<T>(0.f);
        }
}

template <typename T, bool FIRST>
int gated_norm_packed(const zkfp_gated_norm_args& a, int parts, int stride, cudaStream_t st)
{
    const long long units = a.rows * parts;
    if (units > 0x7fffffffll) return ZKDS_ERR_UNSUPPORTED;
    const unsigned warps = (unsigned)((units + 7) / 8);
    if (stride <= 256) gated_norm_kernel<T, 32, 1, FIRST><<<warps, 256, 0, st>>>(a, parts, stride);
    else if (stride <= 512) gated_norm_kernel<T, 32, 2, FIRST><<<warps, 256, 0, st>>>(a, parts, stride);
    else if (stride <= 1024) gated_norm_kernel<T, 32, 4, FIRST><<<warps, 256, 0, st>>>(a, parts, stride);
    else if (stride <= 2048) gated_norm_kernel<T, 32, 8, FIRST><<<warps, 256, 0, st>>>(a, parts, stride);
    else gated_norm_kernel<T, 256, 4, FIRST><<<(unsigned)units, 256, 0, st>>>(a, parts, stride);
    return fp_launched();
}

template <typename T>
int gated_norm(const zkfp_gated_norm_args& a, cudaStream_t st)
{
    const bool whole_head = a.part == a.vdim;
    const int parts = a.heads * a.vdim / a.part, stride = whole_head ? a.p : a.part;
    if (whole_head || (a.p == a.vdim && a.part % 8 == 0))
        return a.weight ? gated_norm_packed<T, true>(a, parts, stride, st) : gated_norm_packed<T, false>(a, parts, stride, st);
    if (a.rows * parts > 0x7fffffffll) return ZKDS_ERR_UNSUPPORTED;
    gated_norm_any_kernel<T><<<(unsigned)(a.rows * parts), 256, 0, st>>>(a, parts);
    return fp_launched();
}

}  // namespace

}  // namespace zkds

using namespace zkds;

extern "C" {

int zkfp_short_conv(const zkfp_conv_args* a, void* stream)
{
    if (!a || !a->x || !a->w || !a->b || !a->out || !a->start || !a->slots || a->batch <= 0 || a->batch > 65535 || a->seq < 0 ||
        a->channels <= 0 || (a->channels & 7) || a->taps < 1 || a->taps > kConvTokens || (a->taps > 1 && !a->state) || a->ldx < a->channels ||
        a->ldo < a->channels || ((a->ldx | a->ldo) & 7))
        return ZKDS_ERR_ARG;
    if (a->seq == 0) return ZKDS_OK;
    return a->dtype == ZKFP_BF16 ? short_conv<bf16>(*a, (cudaStream_t)stream) : short_conv<float>(*a, (cudaStream_t)stream);
}

static bool scan_ok(const zkfp_scan_args* a)
{
    return a && a->q && a->k && a->v && a->out && a->decay && a->state && a->start && a->slots && a->batch > 0 &&
           a->batch <= 65535 && a->seq >= 0 && a->heads > 0 && a->heads <= 65535 && a->heads_per_qk > 0 && a->n > 0 && a->p > 0 &&
           !(a->n & 7) && !(a->p & 7) && (!a->step || a->step_bias) &&
           !((a->q_tok | a->k_tok | a->v_tok | a->o_tok | a->qk_head | a->v_head | a->o_head) & 7) &&
           !(((uintptr_t)a->q | (uintptr_t)a->k | (uintptr_t)a->v | (uintptr_t)a->out) & 15);
}

int zkfp_scan_path(const zkfp_scan_args* a) { return a->dtype == ZKFP_BF16 && scan_tc_takes(*a) ? 1 : 0; }

long long zkfp_scan_scratch(const zkfp_scan_args* a) { return zkfp_scan_path(a) == 1 ? scan_tc_scratch(*a) : 0; }

int zkfp_scan(const zkfp_scan_args* a, void* stream)
{
    if (!scan_ok(a)) return ZKDS_ERR_ARG;
    if (a->seq == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    if (zkfp_scan_path(a) == 1) return launch_scan_tc(*a, st);
    return a->dtype == ZKFP_BF16 ? scan<bf16>(*a, st) : scan<float>(*a, st);
}

int zkfp_gated_norm(const zkfp_gated_norm_args* a, void* stream)
{
    if (!a || !a->x || !a->g || !a->out || a->rows < 0 || a->heads <= 0 || a->vdim <= 0 || a->p < a->vdim || (a->p & 7) ||
        a->part <= 0 || (a->heads * a->vdim) % a->part || ((a->ldx | a->ldg | a->ldo) & 7) ||
        (!a->weight && a->part != a->vdim))
        return ZKDS_ERR_ARG;
    if (a->rows == 0) return ZKDS_OK;
    return a->dtype == ZKFP_BF16 ? gated_norm<bf16>(*a, (cudaStream_t)stream) : gated_norm<float>(*a, (cudaStream_t)stream);
}

}  // extern "C"
