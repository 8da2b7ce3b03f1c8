// Shared helpers of the floating-point kernels: bfloat16 / float32 access, reductions, launch accounting.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/zkds_float.h"
#include "common.cuh"

namespace zkds {

using bf16 = __nv_bfloat16;

constexpr int kSharedMax = 227 * 1024;  // dynamic shared memory a CTA may ask for

int fp_sm_count();
int fp_launched();                      // cudaGetLastError -> status, counts the launch
int* fp_error_flag();                   // device view of the host-mapped word that bounded waits set

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi)
{
    __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&p);
}
__device__ __forceinline__ float bf16_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t u) { return __uint_as_float(u & 0xFFFF0000u); }

// eight consecutive elements, 16-byte aligned
__device__ __forceinline__ void load8(const float* p, float (&v)[8])
{
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void unpack8(const uint4& u, float (&v)[8])
{
    v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
    v[4] = bf16_lo(u.z); v[5] = bf16_hi(u.z); v[6] = bf16_lo(u.w); v[7] = bf16_hi(u.w);
}
__device__ __forceinline__ void load8(const bf16* p, float (&v)[8])
{
    unpack8(*reinterpret_cast<const uint4*>(p), v);
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8])
{
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8])
{
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]),
                                              pack_bf16(v[6], v[7]));
}

__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// sum over the block, the same value in every thread; `red` holds one float per warp.  Ends with a barrier.
__device__ __forceinline__ float block_sum(float v, float* red)
{
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    const int warps = (blockDim.x + 31) >> 5;
    for (int i = 0; i < warps; ++i) t += red[i];
    return t;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
// for results that are rounded to T: a few ulps of 32-bit where T is bfloat16
template <typename T> __device__ __forceinline__ float sigmoid_for(float z);
template <> __device__ __forceinline__ float sigmoid_for<float>(float z) { return sigmoid_f(z); }
template <> __device__ __forceinline__ float sigmoid_for<bf16>(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// ---- epilogues of the linear layers ------------------------------------------------------------------
struct LinEpi {
    void* out;
    const void* aux;
    const float2* table;
    const int* start;
    long long ldo, ldaux, seq, positions;
    int kind, out_bf16, aux_bf16;
    int pairs, period, offset, rot_begin, rot_end;
    const float* bias;
    float* out2;
    long long ldo2, split;          // split: past the last column when there is no second output
};

__device__ __forceinline__ float aux_at(const LinEpi& e, long long m, long long n)
{
    return e.aux_bf16 ? __bfloat162float(((const bf16*)e.aux)[m * e.ldaux + n]) : ((const float*)e.aux)[m * e.ldaux + n];
}

__device__ __forceinline__ int epi_position(const LinEpi& e, long long m)
{
    const int b = (int)((unsigned)m / (unsigned)e.seq);
    return e.start[b] + (int)((unsigned)m - (unsigned)b * (unsigned)e.seq);
}

// the pair at columns (n, n + 1), n even, of the row at position pos
__device__ __forceinline__ void rotate_pair(const LinEpi& e, int pos, int n, float& u, float& v)
{
    if (n < e.rot_begin || n >= e.rot_end) return;
    const int w = (n - e.rot_begin) % e.period - e.offset;
    if (w < 0 || (w >> 1) >= e.pairs || (unsigned)pos >= (unsigned)e.positions) return;
    const float2 cs = e.table[(long long)pos * e.pairs + (w >> 1)];
    const float a = u * cs.x - v * cs.y;
    v = v * cs.x + u * cs.y;
    u = a;
}

// eight finished accumulators of row m at columns n .. n + 7 (n a multiple of 8)
__device__ __forceinline__ void epilogue8(const LinEpi& e, int pos, long long m, long long n, float (&v)[8])
{
    if (e.bias) {
        float b[8];
        load8(e.bias + n, b);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] += b[i];
    }
    if (n >= e.split) {
        store8(e.out2 + m * e.ldo2 + (n - e.split), v);
        return;
    }
    if (e.kind == ZKFP_EPI_ROTATE) {
#pragma unroll
        for (int i = 0; i < 8; i += 2) rotate_pair(e, pos, (int)n + i, v[i], v[i + 1]);
    } else if (e.kind == ZKFP_EPI_GATE) {
        float g[8];
        if (e.aux_bf16) load8((const bf16*)e.aux + m * e.ldaux + n, g);
        else load8((const float*)e.aux + m * e.ldaux + n, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = sigmoid_f(v[i]) * g[i];
    } else if (e.kind == ZKFP_EPI_GLU) {
        float h[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = v[2 * i] * sigmoid_f(v[2 * i]) * v[2 * i + 1];
        const long long o = m * e.ldo + (n >> 1);
        if (e.out_bf16) *reinterpret_cast<uint2*>((bf16*)e.out + o) = make_uint2(pack_bf16(h[0], h[1]), pack_bf16(h[2], h[3]));
        else *reinterpret_cast<float4*>((float*)e.out + o) = make_float4(h[0], h[1], h[2], h[3]);
        return;
    }
    if (e.out_bf16) store8((bf16*)e.out + m * e.ldo + n, v);
    else store8((float*)e.out + m * e.ldo + n, v);
}

// ---- launchers (float_ops.cu, float_gemm.cu, float_attention.cu) -------------------------------------------
int launch_linear_plain(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st);
int launch_linear_stream(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st);
int launch_linear_tc(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st);
int launch_attention_plain(const zkfp_attention_args& a, cudaStream_t st);
bool attention_prefill_tc_takes(const zkfp_attention_args& a);
int launch_attention_prefill_tc(const zkfp_attention_args& a, cudaStream_t st);
bool attention_decode_tc_takes(const zkfp_attention_args& a);
int launch_attention_decode_tc(const zkfp_attention_args& a, cudaStream_t st);
long long attention_decode_scratch(const zkfp_attention_args& a);
bool scan_tc_takes(const zkfp_scan_args& a);
int launch_scan_tc(const zkfp_scan_args& a, cudaStream_t st);
long long scan_tc_scratch(const zkfp_scan_args& a);

}  // namespace zkds
