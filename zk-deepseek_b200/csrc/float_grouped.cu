// Grouped attention layers: heads after the projection (norm, rotation, cache write) and attention of a few tokens per
// sequence over the cache.  Norms, rotations, scores and weights are 32-bit in both number formats.
#include "float_common.cuh"

namespace zkds {

namespace {

// ---- norm, rotation, cache write -----------------------------------------------------------------------------
// LANES lanes of a warp take one head of one row, eight elements each and V such vectors.
template <typename T, int LANES, int V>
__global__ void __launch_bounds__(256)
heads_post_kernel(const zkfp_heads_args a)
{
    const int lane = threadIdx.x % LANES, units = a.heads + a.kv_heads;
    const long long unit = (long long)blockIdx.x * (256 / LANES) + threadIdx.x / LANES;
    if (unit >= a.rows * units) return;              // whole groups of lanes leave together
    const unsigned group = LANES == 32 ? 0xffffffffu : ((1u << (LANES & 31)) - 1u) << ((threadIdx.x & 31) / LANES * LANES);
    const long long r = unit / units;
    const int head = (int)(unit - r * units), b = (int)(r / a.seq);
    const int pos = a.start[b] + (int)(r - (long long)b * a.seq);
    if (pos < 0 || pos >= a.capacity) return;
    const bool is_q = head < a.heads;
    const int kv = head - a.heads;
    const T* src = (const T*)a.y + r * a.ldy + (is_q ? a.q_col + (long long)head * a.d : a.k_col + (long long)kv * a.d);
    T* row = (T*)a.cache + a.slots[b] * a.slot_stride + (long long)pos * a.pitch;
    T* dst = is_q ? (T*)a.q + (r * a.heads + head) * a.d : row + (long long)kv * a.d;
    const float* w = is_q ? a.wq : a.wk;
    float x[V][8];
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < V; ++k) {
        const int c = (k * LANES + lane) * 8;
        if (c < a.d) {
            load8(src + c, x[k]);
            if (!is_q) store8(row + (long long)(a.kv_heads + kv) * a.d + c, x[k]);
#pragma unroll
            for (int i = 0; i < 8; ++i) s = fmaf(x[k][i], x[k][i], s);
        }
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) s += __shfl_xor_sync(group, s, o);
    const float rs = 1.0f / sqrtf(s / (float)a.dim + (float)a.eps);
    const float2* tab = (const float2*)a.table + (long long)pos * a.pairs;
#pragma unroll
    for (int k = 0; k < V; ++k) {
        const int c = (k * LANES + lane) * 8;
        if (c >= a.d) continue;
        float g[8];
        load8(w + c, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) g[i] *= x[k][i] * rs;
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
            if (c + i < 2 * a.pairs) {
                const float2 cs = tab[(c + i) >> 1];
                const float u = g[i] * cs.x - g[i + 1] * cs.y;
                g[i + 1] = g[i + 1] * cs.x + g[i] * cs.y;
                g[i] = u;
            }
        }
        store8(dst + c, g);
    }
}

template <typename T, int LANES, int V>
int heads_post(const zkfp_heads_args& a, cudaStream_t st)
{
    const long long per = 256 / LANES, blocks = (a.rows * (a.heads + a.kv_heads) + per - 1) / per;
    if (blocks > 0x7fffffffll) return ZKDS_ERR_UNSUPPORTED;
    heads_post_kernel<T, LANES, V><<<(unsigned)blocks, 256, 0, st>>>(a);
    return fp_launched();
}

template <typename T>
int heads_post(const zkfp_heads_args& a, cudaStream_t st)
{
    if (a.d <= 64) return heads_post<T, 8, 1>(a, st);
    if (a.d <= 128) return heads_post<T, 16, 1>(a, st);
    if (a.d <= 256) return heads_post<T, 32, 1>(a, st);
    if (a.d <= 1024) return heads_post<T, 32, 4>(a, st);
    return ZKDS_ERR_UNSUPPORTED;
}

// ---- attention over the cache ----------------------------------------------------------------------------------
// A block takes one chunk of keys of one key head and all query rows (token, head of the group) that read it: keys and
// values come into shared memory once, rows are worked off in passes of kRowPass.  Partial sums and (maximum, sum) go
// to scratch; grouped_combine_kernel merges the chunks.
constexpr int kRowPass = 16, kGroupedThreads = 128;

struct GroupedShape {
    int chunk;                  // keys per block
    int kpitch;                 // row pitch of the staged keys (elements)
    size_t smem;
};

template <typename T>
GroupedShape grouped_shape(int d)
{
    GroupedShape g;
    g.kpitch = d + 16 / (int)sizeof(T);                    // rows shifted by one 16-byte piece: no bank conflicts
    for (g.chunk = 64; g.chunk >= 8; g.chunk >>= 1) {
        g.smem = (size_t)g.chunk * (g.kpitch + d) * sizeof(T) + sizeof(float) * ((size_t)kRowPass * d + kRowPass * g.chunk);
        if (g.smem <= 100 * 1024) break;
    }
    return g;
}

__device__ __forceinline__ int first_key(int start, int window) { return window > 0 && start + 1 > window ? start + 1 - window : 0; }

template <typename T>
__global__ void __launch_bounds__(kGroupedThreads)
grouped_partial_kernel(const zkfp_grouped_args a, int chunk, int kpitch, int chunks)
{
    extern __shared__ __align__(16) uint8_t sm[];
    const int b = blockIdx.z, kv = blockIdx.y, tid = threadIdx.x, d = a.d, vecs = d / 8;
    const int start = a.start[b];
    if (start < 0 || start + a.seq > a.capacity) return;   // not a step of this cache
    const int lo = first_key(start, a.window), last = start + (int)a.seq - 1;
    const int j0 = lo + (int)blockIdx.x * chunk;
    if (j0 > last) return;
    const int nk = min(chunk, last - j0 + 1);
    T* Ks = (T*)sm;
    T* Vs = Ks + chunk * kpitch;
    float* Q = (float*)(Vs + chunk * d);
    float* P = Q + kRowPass * d;
    const T* base = (const T*)a.cache + a.slots[b] * a.slot_stride + (long long)kv * d;
    for (int i = tid; i < nk * vecs; i += kGroupedThreads) {
        const int j = i / vecs, c = (i - j * vecs) * 8;
        const T* src = base + (long long)(j0 + j) * a.pitch + c;
#pragma unroll
        for (int q = 0; q < (int)sizeof(T) / 2; ++q) {
            *reinterpret_cast<uint4*>(Ks + j * kpitch + c + q * 4) = *reinterpret_cast<const uint4*>(src + q * 4);
            *reinterpret_cast<uint4*>(Vs + j * d + c + q * 4) = *reinterpret_cast<const uint4*>(src + a.v_off + q * 4);
        }
    }
    const int per_kv = a.heads / a.kv_heads, rows = (int)a.seq * per_kv;
    const long long all_rows = a.seq * a.heads;
    float* part = a.scratch;
    float* ml = part + (long long)a.batch * all_rows * chunks * d;
    for (int r0 = 0; r0 < rows; r0 += kRowPass) {
        const int nr = min(kRowPass, rows - r0);
        __syncthreads();                                   // the previous pass is done with Q and P
        for (int i = tid; i < kRowPass * vecs; i += kGroupedThreads) {
            const int r = i / vecs, c = (i - r * vecs) * 8;
            float v[8] = {};
            if (r < nr) {
                const int t = (r0 + r) / per_kv, h = kv * per_kv + (r0 + r) % per_kv;
                load8((const T*)a.q + (((long long)b * a.seq + t) * a.heads + h) * d + c, v);
            }
            store8(Q + r * d + c, v);
        }
        __syncthreads();
        // scores: a thread takes one key and four rows
        for (int i = tid; i < chunk * (kRowPass / 4); i += kGroupedThreads) {
            const int j = i % chunk, r = i / chunk * 4;
            if (j >= nk || r >= nr) continue;
            float acc[4] = {};
            for (int c = 0; c < d; c += 8) {
                float k8[8];
                load8(Ks + j * kpitch + c, k8);
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    float q8[8];
                    load8(Q + (r + q) * d + c, q8);
#pragma unroll
                    for (int e = 0; e < 8; ++e) acc[q] = fmaf(q8[e], k8[e], acc[q]);
                }
            }
#pragma unroll
            for (int q = 0; q < 4; ++q) P[(r + q) * chunk + j] = acc[q];
        }
        __syncthreads();
        // softmax of the chunk, a warp per row
        for (int r = tid >> 5; r < nr; r += kGroupedThreads / 32) {
            const int t = (r0 + r) / per_kv, h = kv * per_kv + (r0 + r) % per_kv, i = start + t;
            float m = -INFINITY;
            for (int j = tid & 31; j < chunk; j += 32) {
                const int p = j0 + j;
                const bool seen = j < nk && p <= i && (a.window <= 0 || i - p < a.window);
                const float s = seen ? P[r * chunk + j] * a.scale : -INFINITY;
                P[r * chunk + j] = s;
                m = fmaxf(m, s);
            }
            m = warp_max(m);
            float l = 0.f;
            for (int j = tid & 31; j < chunk; j += 32) {
                const float s = P[r * chunk + j];
                const float e = s == -INFINITY ? 0.f : expf(s - m);
                P[r * chunk + j] = e;
                l += e;
            }
            l = warp_sum(l);
            if ((tid & 31) == 0) {
                const long long o = (((long long)b * all_rows + (long long)t * a.heads + h) * chunks + blockIdx.x) * 2;
                ml[o] = m;
                ml[o + 1] = l;
            }
        }
        __syncthreads();
        for (int i = tid; i < nr * vecs; i += kGroupedThreads) {
            const int r = i / vecs, c = (i - r * vecs) * 8;
            float acc[8] = {};
#pragma unroll 4
            for (int j = 0; j < nk; ++j) {
                float v[8];
                load8(Vs + j * d + c, v);
                const float p = P[r * chunk + j];
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[e] = fmaf(p, v[e], acc[e]);
            }
            const int t = (r0 + r) / per_kv, h = kv * per_kv + (r0 + r) % per_kv;
            store8(part + (((long long)b * all_rows + (long long)t * a.heads + h) * chunks + blockIdx.x) * d + c, acc);
        }
    }
}

// one block per (token, head): warps share the chunks, lanes the columns
template <typename T>
__global__ void __launch_bounds__(256)
grouped_combine_kernel(const zkfp_grouped_args a, int chunk, int chunks)
{
    extern __shared__ float red[];                          // [8][d] sums, then [8] sums of weights
    const long long all_rows = a.seq * a.heads, rh = blockIdx.x;          // (sequence, token, head)
    const int b = (int)(rh / all_rows), rest = (int)(rh - (long long)b * all_rows), t = rest / a.heads, h = rest - t * a.heads;
    const int start = a.start[b], warp = threadIdx.x >> 5, lane = threadIdx.x & 31, d = a.d;
    if (start < 0 || start + a.seq > a.capacity) return;
    const int lo = first_key(start, a.window), n = (start + (int)a.seq - 1 - lo) / chunk + 1;
    const float* part = a.scratch + rh * chunks * d;
    const float* ml = a.scratch + (long long)a.batch * all_rows * chunks * d + rh * chunks * 2;
    float m = -INFINITY;
    for (int i = lane; i < n; i += 32) m = fmaxf(m, ml[2 * i]);
    m = warp_max(m);
    float l = 0.f;
    for (int i = warp; i < n; i += 8) {
        const float mi = ml[2 * i];
        l += mi == -INFINITY ? 0.f : expf(mi - m) * ml[2 * i + 1];
    }
    for (int c = lane * 4; c < d; c += 128) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int i = warp; i < n; i += 8) {
            const float mi = ml[2 * i], w = mi == -INFINITY ? 0.f : expf(mi - m);
            const float4 v = *reinterpret_cast<const float4*>(part + (long long)i * d + c);
            acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y);
            acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
        }
        *reinterpret_cast<float4*>(red + warp * d + c) = acc;
    }
    if (lane == 0) red[8 * d + warp] = l;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) total += red[8 * d + w];
    const long long row = (long long)b * a.seq + t;
    for (int c = threadIdx.x; c < d; c += 256) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v += red[w * d + c];
        v /= total;
        if (a.gate) v *= sigmoid_f(to_f32(((const T*)a.gate)[row * a.gate_tok + (long long)h * d + c])) * a.out_scale;
        ((T*)a.out)[row * a.o_tok + (long long)h * d + c] = from_f32<T>(v);
    }
}

template <typename T>
int grouped_chunks(const zkfp_grouped_args& a)
{
    const int chunk = grouped_shape<T>(a.d).chunk;
    return (a.max_keys + chunk - 1) / chunk;
}

template <typename T>
int grouped_attention(const zkfp_grouped_args& a, cudaStream_t st)
{
    const GroupedShape g = grouped_shape<T>(a.d);
    const int chunks = grouped_chunks<T>(a);
    if (g.smem > 100 * 1024 || a.batch * a.seq * a.heads > 0x7fffffffll || a.kv_heads > 65535) return ZKDS_ERR_UNSUPPORTED;
    ZKDS_CUDA(cudaFuncSetAttribute(grouped_partial_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
    grouped_partial_kernel<T><<<dim3((unsigned)chunks, (unsigned)a.kv_heads, (unsigned)a.batch), kGroupedThreads, g.smem, st>>>(
        a, g.chunk, g.kpitch, chunks);
    const int rc = fp_launched();
    if (rc != ZKDS_OK) return rc;
    const size_t smem = sizeof(float) * (8 * (size_t)a.d + 8);
    if (smem > 48 * 1024) return ZKDS_ERR_UNSUPPORTED;
    grouped_combine_kernel<T><<<(unsigned)(a.batch * a.seq * a.heads), 256, smem, st>>>(a, g.chunk, chunks);
    return fp_launched();
}

}  // namespace

}  // namespace zkds

using namespace zkds;

extern "C" {

int zkfp_heads_post(const zkfp_heads_args* a, void* stream)
{
    if (!a || !a->y || !a->wq || !a->wk || !a->q || !a->cache || !a->table || !a->start || !a->slots || a->rows < 0 ||
        a->seq <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->d <= 0 || (a->d & 7) || a->dim <= 0 || a->dim > a->d ||
        a->pairs < 0 || 2 * a->pairs > a->d || a->pitch < 2ll * a->kv_heads * a->d ||
        ((a->ldy | a->q_col | a->k_col | a->pitch | a->slot_stride) & 7))
        return ZKDS_ERR_ARG;
    if (a->rows == 0) return ZKDS_OK;
    return a->dtype == ZKFP_BF16 ? heads_post<bf16>(*a, (cudaStream_t)stream) : heads_post<float>(*a, (cudaStream_t)stream);
}

long long zkfp_grouped_scratch(const zkfp_grouped_args* a)
{
    const long long chunks = a->dtype == ZKFP_BF16 ? grouped_chunks<bf16>(*a) : grouped_chunks<float>(*a);
    return a->batch * a->seq * a->heads * chunks * (a->d + 2);
}

int zkfp_grouped_attention(const zkfp_grouped_args* a, void* stream)
{
    if (!a || !a->q || !a->cache || !a->out || !a->start || !a->slots || !a->scratch || a->batch <= 0 || a->batch > 65535 ||
        a->seq < 0 || a->seq > 65535 || a->kv_heads <= 0 || a->heads <= 0 || a->heads % a->kv_heads || a->d <= 0 || (a->d & 7) ||
        a->max_keys <= 0 || a->o_tok < (long long)a->heads * a->d || (a->gate && a->gate_tok < (long long)a->heads * a->d) ||
        a->pitch < a->v_off + (long long)a->kv_heads * a->d || ((a->pitch | a->slot_stride | a->v_off | a->o_tok | a->gate_tok) & 7))
        return ZKDS_ERR_ARG;
    if (a->seq == 0) return ZKDS_OK;
    return a->dtype == ZKFP_BF16 ? grouped_attention<bf16>(*a, (cudaStream_t)stream)
                                 : grouped_attention<float>(*a, (cudaStream_t)stream);
}

}  // extern "C"
