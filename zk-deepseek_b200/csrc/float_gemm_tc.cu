// bfloat16 linear layers on the tensor cores: out = epilogue(A W^T), 32-bit accumulators in tensor memory.
//
// A pair of CTAs (cta_group::2) computes a 256 x NT tile: each CTA holds its 128 rows of A and half of the NT rows of
// W, so a K block of 64 costs every SM 16 KB + NT * 64 bytes of operand traffic for 128 x NT x 64 products.  The
// kernel is persistent; accumulators are double buffered, so the epilogue of a tile runs under the MMAs of the next.
//   warp 0  TMA loads of this CTA's operand halves; bytes are counted on the even CTA's barriers
//   warp 1  (even CTA) issues the MMAs of the pair; commits free the stages and publish the accumulators in both CTAs
//   warps 2-9  epilogue: a warp owns a quarter of the 128 rows and half of the columns
// Every wait is bounded; one that runs out sets a host-visible flag and the CTAs leave through the normal path.
#include <cuda.h>

#include "float_common.cuh"
#include "tcgen05.cuh"

namespace zkds {

namespace {

constexpr int kTM = 128;                 // rows per CTA
constexpr int kBK = 64;                  // K elements per stage (128 bytes)
constexpr int kEpiWarps = 8;
constexpr int kThreadsTc = 64 + 32 * kEpiWarps;
constexpr int kMaxStages = 12;
constexpr uint32_t kBytesA = kTM * kBK * 2;

struct TcParams {
    int M, N, NT, kblocks, stages;
    int m_tiles, n_tiles, panel;         // tiles of 256 x NT; panel: row tiles walked before the next column tile
    int* error_flag;
    LinEpi e;
};

struct TcShared {
    uint64_t full[kMaxStages], empty[kMaxStages], acc_full[2], acc_empty[2];
    uint32_t tmem;
    int abort;
};

__device__ __forceinline__ void tile_coords(const TcParams& p, int t, int& mt, int& nt)
{
    const int per_panel = p.panel * p.n_tiles;
    const int pn = t / per_panel, r = t - pn * per_panel;
    const int height = min(p.panel, p.m_tiles - pn * p.panel);
    nt = r / height;
    mt = pn * p.panel + r - nt * height;
}

__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(kThreadsTc, 1)
linear_tc_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmW, const TcParams p)
{
    extern __shared__ uint8_t raw[];
    uint8_t* base = (uint8_t*)(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    __shared__ TcShared s;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t rank = cluster_rank();
    const uint32_t bytes_w = (uint32_t)(p.NT / 2) * kBK * 2, stage_bytes = kBytesA + bytes_w;
    const uint32_t smem0 = smem_u32(base);
    const int total = p.m_tiles * p.n_tiles, pairs = gridDim.x >> 1, first = blockIdx.x >> 1;
    volatile int* abort_flag = &s.abort;

    if (threadIdx.x == 0) {
        s.abort = 0;
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(smem_u32(&s.full[i]), 1);
            mbar_init(smem_u32(&s.empty[i]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&s.acc_full[i]), 1);
            mbar_init(smem_u32(&s.acc_empty[i]), 2 * kEpiWarps);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    if (warp == 1) tmem_alloc_pair(smem_u32(&s.tmem), 512);
    tc_fence_before();
    __syncthreads();
    cluster_sync_all();
    tc_fence_after();
    const uint32_t tmem = s.tmem;

    if (warp == 0) {
        if (lane == 0) {
            int stage = 0;
            uint32_t phase = 0;
            bool ok = true;
            for (int t = first; t < total && ok; t += pairs) {
                int mt, nt;
                tile_coords(p, t, mt, nt);
                const int row_a = mt * 256 + (int)rank * kTM, row_w = nt * p.NT + (int)rank * (p.NT / 2);
                for (int kb = 0; kb < p.kblocks; ++kb) {
                    if (!mbar_wait(smem_u32(&s.empty[stage]), phase ^ 1u, abort_flag)) { ok = false; break; }
                    const uint32_t full = smem_u32(&s.full[stage]), dst = smem0 + (uint32_t)stage * stage_bytes;
                    if (rank == 0) mbar_expect_tx(full, 2 * stage_bytes);
                    tma_load_2d_pair(dst, &tmA, kb * kBK, row_a, full);
                    tma_load_2d_pair(dst + kBytesA, &tmW, kb * kBK, row_w, full);
                    if (++stage == p.stages) { stage = 0; phase ^= 1u; }
                }
            }
        }
    } else if (warp == 1) {
        if (rank == 0 && lane == 0) {
            const uint32_t idesc = idesc_bf16(256, p.NT);
            int stage = 0, buf = 0;
            uint32_t phase = 0, acc_phase = 0;
            bool ok = true;
            for (int t = first; t < total && ok; t += pairs) {
                if (!mbar_wait(smem_u32(&s.acc_empty[buf]), acc_phase ^ 1u, abort_flag)) break;
                tc_fence_after();
                const uint32_t acc = tmem + (uint32_t)buf * 256u;
                for (int kb = 0; kb < p.kblocks; ++kb) {
                    if (!mbar_wait(smem_u32(&s.full[stage]), phase, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t sa = smem0 + (uint32_t)stage * stage_bytes;
                    const uint64_t ad = smem_desc_sw128(sa), wd = smem_desc_sw128(sa + kBytesA);
#pragma unroll
                    for (int k = 0; k < kBK / 16; ++k)
                        umma_bf16_pair(acc, ad + (uint64_t)(k * 2), wd + (uint64_t)(k * 2), idesc, (kb | k) ? 1u : 0u);
                    umma_commit_pair(smem_u32(&s.empty[stage]));
                    if (++stage == p.stages) { stage = 0; phase ^= 1u; }
                }
                if (ok) umma_commit_pair(smem_u32(&s.acc_full[buf]));
                if (++buf == 2) { buf = 0; acc_phase ^= 1u; }
            }
        }
    } else {
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        const uint32_t tq = tmem + ((uint32_t)(quarter * 32) << 16);
        const int c_begin = half * (p.NT / 2), c_end = c_begin + p.NT / 2;
        int buf = 0;
        uint32_t acc_phase = 0;
        for (int t = first; t < total; t += pairs) {
            int mt, nt;
            tile_coords(p, t, mt, nt);
            if (!mbar_wait(smem_u32(&s.acc_full[buf]), acc_phase, abort_flag)) break;
            tc_fence_after();
            const int m = mt * 256 + (int)rank * kTM + quarter * 32 + lane, n0 = nt * p.NT;
            const bool row_ok = m < p.M;
            const int pos = (row_ok && p.e.kind == ZKFP_EPI_ROTATE) ? epi_position(p.e, m) : 0;
            for (int c = c_begin; c < c_end; c += 32) {
                float v[32];
                tmem_ld32(tq + (uint32_t)(buf * 256 + c), v);
                tmem_ld_wait();
                if (c + 32 >= c_end) {
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive_remote(smem_u32(&s.acc_empty[buf]), 0);
                }
                if (row_ok) {
#pragma unroll
                    for (int j = 0; j < 32; j += 8) {
                        if (n0 + c + j < p.N) {
                            float w[8];
#pragma unroll
                            for (int i = 0; i < 8; ++i) w[i] = v[j + i];
                            epilogue8(p.e, pos, m, n0 + c + j, w);
                        }
                    }
                }
            }
            if (++buf == 2) { buf = 0; acc_phase ^= 1u; }
        }
    }
    __syncthreads();
    tc_fence_before();
    cluster_sync_all();
    tc_fence_after();
    if (warp == 1) tmem_dealloc_pair(tmem, 512);
    if (threadIdx.x == 0 && s.abort && p.error_flag) *(volatile int*)p.error_flag = 1;
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiledFn encode_fn()
{
    static EncodeTiledFn fn = nullptr;
    if (!fn) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
            q == cudaDriverEntryPointSuccess)
            fn = (EncodeTiledFn)p;
    }
    return fn;
}

}  // namespace

bool fp_tensor_map(CUtensorMap* map, const void* base, int rank, const uint64_t* dims, const uint64_t* strides_bytes,
                   const uint32_t* box)
{
    EncodeTiledFn fn = encode_fn();
    if (!fn) return false;
    cuuint64_t gd[5], gs[4];
    cuuint32_t bx[5], es[5];
    for (int i = 0; i < rank; ++i) {
        gd[i] = dims[i];
        bx[i] = box[i];
        es[i] = 1;
        if (i) gs[i - 1] = strides_bytes[i - 1];
    }
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)rank, const_cast<void*>(base), gd, gs, bx, es,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

int launch_linear_tc(const zkfp_linear_args& a, const LinEpi& e, cudaStream_t st)
{
    TcParams p;
    p.M = (int)a.M;
    p.N = (int)a.N;
    p.kblocks = (int)((a.K + kBK - 1) / kBK);
    p.e = e;
    p.error_flag = fp_error_flag();
    if (!p.error_flag) return ZKDS_ERR_WORKSPACE;
    p.m_tiles = (p.M + 255) / 256;
    const int pairs = fp_sm_count() / 2;
    // the widest tile unless narrower ones spread the work over more pairs: cost = rounds x (tile width + what a
    // tile costs whatever its width)
    long long best = 0;
    for (int nt = 256; nt >= 64; nt >>= 1) {
        const long long tiles = (long long)p.m_tiles * ((p.N + nt - 1) / nt);
        const long long cost = (tiles + pairs - 1) / pairs * (nt + 48);
        if (nt == 256 || cost < best) { best = cost; p.NT = nt; }
    }
    p.n_tiles = (p.N + p.NT - 1) / p.NT;
    p.panel = p.m_tiles < 8 ? p.m_tiles : 8;
    if ((long long)p.m_tiles * p.n_tiles > 0x7fffffffll) return ZKDS_ERR_UNSUPPORTED;
    const uint32_t stage_bytes = kBytesA + (uint32_t)(p.NT / 2) * kBK * 2;
    p.stages = (int)((220u * 1024u) / stage_bytes);
    if (p.stages > kMaxStages) p.stages = kMaxStages;
    CUtensorMap tmA, tmW;
    const uint64_t da[2] = {(uint64_t)a.K, (uint64_t)a.M}, dw[2] = {(uint64_t)a.K, (uint64_t)a.N};
    const uint64_t sa[1] = {(uint64_t)a.lda * 2}, sw[1] = {(uint64_t)a.ldw * 2};
    const uint32_t ba[2] = {kBK, kTM}, bw[2] = {kBK, (uint32_t)p.NT / 2};
    if (!fp_tensor_map(&tmA, a.A, 2, da, sa, ba) || !fp_tensor_map(&tmW, a.W, 2, dw, sw, bw)) return ZKDS_ERR_UNSUPPORTED;
    const size_t smem = (size_t)stage_bytes * p.stages + 1024;
    ZKDS_CUDA(cudaFuncSetAttribute(linear_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const int tiles = p.m_tiles * p.n_tiles;
    const unsigned grid = 2u * (unsigned)(tiles < pairs ? tiles : pairs);
    linear_tc_kernel<<<grid, kThreadsTc, smem, st>>>(tmA, tmW, p);
    return fp_launched();
}

}  // namespace zkds
