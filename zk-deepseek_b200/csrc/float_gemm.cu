// Linear layers of the floating-point decoders: out = epilogue(A W^T) with 32-bit accumulation.
//   few rows (decode)   linear_stream_kernel: every weight is read once, sixteen bytes a lane
//   many rows, bfloat16 linear_tc_kernel (float_gemm_tc.cu): tcgen05 tiles fed by TMA
//   many rows, float32  linear_plain_kernel: true 32-bit products on the CUDA cores
#include "float_common.cuh"

namespace zkds {

namespace {

// ---- CUDA-core tiles: 64 x 64 x 16, 4 x 8 outputs a thread ---------------------------------------------
constexpr int kPM = 64, kPN = 64, kPK = 16;

template <typename T>
__global__ void __launch_bounds__(128)
linear_plain_kernel(const T* __restrict__ A, long long lda, const T* __restrict__ W, long long ldw, int M, int N, int K,
                    const LinEpi e)
{
    __shared__ float As[kPK][kPM + 4], Ws[kPK][kPN + 4];
    const int m0 = blockIdx.y * kPM, n0 = blockIdx.x * kPN;
    const int tx = threadIdx.x & 7, ty = threadIdx.x >> 3;        // columns tx * 8 .. + 7, rows ty * 4 .. + 3
    const int lr = threadIdx.x >> 1, lk = (threadIdx.x & 1) * 8;  // loader: one row, eight k
    float acc[4][8] = {};
    for (int k0 = 0; k0 < K; k0 += kPK) {
        float va[8] = {}, vw[8] = {};
        if (k0 + lk < K) {
            if (m0 + lr < M) load8(A + (long long)(m0 + lr) * lda + k0 + lk, va);
            if (n0 + lr < N) load8(W + (long long)(n0 + lr) * ldw + k0 + lk, vw);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            As[lk + i][lr] = va[i];
            Ws[lk + i][lr] = vw[i];
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kPK; ++k) {
            float a[4], w[8];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 8; ++j) w[j] = Ws[k][tx * 8 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
    }
    const int n = n0 + tx * 8;
    if (n >= N) return;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m < M) epilogue8(e, e.kind == ZKFP_EPI_ROTATE ? epi_position(e, m) : 0, m, n, acc[i]);
    }
}

// ---- weight streaming ---------------------------------------------------------------------------------------
// A warp accumulates eight weight rows against MT activation rows over its share of K; `ksplit` warps of the
// block share the eight rows.  The butterfly leaves column (lane >> 2) of a token's eight sums in its lane.
__device__ __forceinline__ float reduce8(float (&v)[8], int lane)
{
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const bool up = lane & 16;
        const float send = up ? v[i] : v[i + 4], keep = up ? v[i + 4] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, 16);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const bool up = lane & 8;
        const float send = up ? v[i] : v[i + 2], keep = up ? v[i + 2] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, 8);
    }
    const bool up = lane & 4;
    const float send = up ? v[0] : v[1], keep = up ? v[1] : v[0];
    float s = keep + __shfl_xor_sync(0xffffffffu, send, 4);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    return s + __shfl_xor_sync(0xffffffffu, s, 1);
}

template <typename T, int MT>
__global__ void __launch_bounds__(256)
linear_stream_kernel(const T* __restrict__ A, long long lda, const T* __restrict__ W, long long ldw, int M, int N, int K,
                     int ksplit, const LinEpi e)
{
    __shared__ float part[8][MT][8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int groups = 8 / ksplit, ks = warp % ksplit;
    const int n = (blockIdx.x * groups + warp / ksplit) * 8;
    const int m0 = blockIdx.y * MT;
    float acc[MT][8] = {};
    if (n < N) {
        const T* w = W + (long long)n * ldw;
        const T* a = A + (long long)m0 * lda;
        const int step = 256 * ksplit;
#pragma unroll 2
        for (int k = ks * 256 + lane * 8; k < K; k += step) {
            float x[MT][8];
#pragma unroll
            for (int t = 0; t < MT; ++t) {
                if (m0 + t < M) load8(a + t * lda + k, x[t]);
                else {
#pragma unroll
                    for (int i = 0; i < 8; ++i) x[t][i] = 0.f;
                }
            }
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                float v[8];
                load8(w + r * ldw + k, v);
#pragma unroll
                for (int t = 0; t < MT; ++t)
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[t][r] = fmaf(v[i], x[t][i], acc[t][r]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < MT; ++t) {
        const float s = reduce8(acc[t], lane);
        if ((lane & 3) == 0) part[warp][t][lane >> 2] = s;
    }
    __syncthreads();
    if (threadIdx.x < groups * MT) {
        const int g = threadIdx.x / MT, t = threadIdx.x % MT;
        const int ng = (blockIdx.x * groups + g) * 8, m = m0 + t;
        if (ng < N && m < M) {
            float v[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                v[i] = 0.f;
                for (int s = 0; s < ksplit; ++s) v[i] += part[g * ksplit + s][t][i];
            }
            epilogue8(e, e.kind == ZKFP_EPI_ROTATE ? epi_position(e, m) : 0, m, ng, v);
        }
    }
}

template <typename T>
int linear_stream(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st)
{
    int ksplit = 1;
    while (ksplit < 8 && (long long)ksplit * 512 < a.K) ksplit *= 2;
    // narrow outputs: more warps on the same rows until every SM has work
    while (ksplit < 8 && a.N / 8 * ksplit < 8LL * fp_sm_count() && ksplit * 256 < a.K) ksplit *= 2;
    const int groups = 8 / ksplit;
    const unsigned gx = (unsigned)((a.N / 8 + groups - 1) / groups);
    const T *A = (const T*)a.A, *W = (const T*)a.W;
    const int M = (int)a.M, N = (int)a.N, K = (int)a.K;
    if (M == 1) linear_stream_kernel<T, 1><<<dim3(gx, 1), 256, 0, st>>>(A, a.lda, W, a.ldw, M, N, K, ksplit, e);
    else if (M == 2) linear_stream_kernel<T, 2><<<dim3(gx, 1), 256, 0, st>>>(A, a.lda, W, a.ldw, M, N, K, ksplit, e);
    else linear_stream_kernel<T, 4><<<dim3(gx, (M + 3) / 4), 256, 0, st>>>(A, a.lda, W, a.ldw, M, N, K, ksplit, e);
    return fp_launched();
}

template <typename T>
int linear_plain(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st)
{
    const dim3 grid((unsigned)((a.N + kPN - 1) / kPN), (unsigned)((a.M + kPM - 1) / kPM));
    if (grid.y > 65535u) return ZKDS_ERR_UNSUPPORTED;
    linear_plain_kernel<T><<<grid, 128, 0, st>>>((const T*)a.A, a.lda, (const T*)a.W, a.ldw, (int)a.M, (int)a.N, (int)a.K, e);
    return fp_launched();
}

}  // namespace

int launch_linear_plain(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st)
{
    return a.dtype == ZKFP_BF16 ? linear_plain<bf16>(a, e, st) : linear_plain<float>(a, e, st);
}

int launch_linear_stream(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st)
{
    return a.dtype == ZKFP_BF16 ? linear_stream<bf16>(a, e, st) : linear_stream<float>(a, e, st);
}

}  // namespace zkds
