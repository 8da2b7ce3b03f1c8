// bfloat16 linear layers on the tensor cores: out = epilogue(A W^T), 32-bit accumulators in tensor memory.
//
// A pair of CTAs (cta_group::2) computes a 256 x NT tile: each CTA holds its 128 rows of A and half of the NT rows of
// W, so a K block of 64 costs every SM 16 KB + NT * 64 bytes of operand traffic for 128 x NT x 64 products.  The
// kernel is persistent; accumulators are double buffered, so the epilogue of a tile runs under the MMAs of the next.
//   warp 0  TMA loads of this CTA's operand halves; bytes are counted on the even CTA's barriers
//   warp 1  (even CTA) issues the MMAs of the pair; commits free the stages and publish the accumulators in both CTAs
//   warps 2-9  epilogue: a warp owns a quarter of the 128 rows and half of the columns; 32 x 32 blocks pass through
//              shared memory so that global accesses are whole row segments
// Shapes with few tiles and a deep K split K over several pairs: each leaves its 32-bit sums in a workspace, and the
// epilogue warp that arrives last at its part of a tile adds them up in a fixed order.
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
constexpr uint32_t kStageBlock = 32 * 32 * 4;      // staging per epilogue warp
constexpr int kLinearSmemMax = 226 * 1024;         // leaves room for the static part

struct TcParams {
    int M, N, NT, kblocks, stages;
    int m_tiles, n_tiles, panel;         // tiles of 256 x NT; panel: row tiles walked before the next column tile
    int ksplit, kb_per_split;
    float* partial;                      // [item][rank][column of the tile][128 rows]
    unsigned* counter;                   // [tile][rank][epilogue warp]
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

// 16-byte piece `piece` of row `row` in a 32-row block of `P` pieces per row, spread over the banks
template <int P>
__device__ __forceinline__ uint32_t piece_at(int row, int piece)
{
    return (uint32_t)((row * P + (piece ^ ((row / (8 / P)) & (P - 1)))) * 16);
}

// global rows of P pieces <-> staging block; `pitch` in bytes, cols_ok pieces are inside the matrix
template <int P, bool LOAD>
__device__ __forceinline__ void move_block(uint8_t* stage, uint8_t* g, long long pitch, int rows_ok, int pieces_ok, int lane)
{
#pragma unroll
    for (int i = 0; i < P; ++i) {
        const int idx = i * 32 + lane, row = idx / P, piece = idx % P;
        if (row < rows_ok && piece < pieces_ok) {
            uint4* s = reinterpret_cast<uint4*>(stage + piece_at<P>(row, piece));
            uint4* d = reinterpret_cast<uint4*>(g + row * pitch + piece * 16);
            if (LOAD) *s = *d;
            else *d = *s;
        }
    }
}

// 32 finished accumulators of this lane's row at columns n .. n + 31; the warp's rows start at m0
__device__ __forceinline__ void epilogue_block(const TcParams& p, float (&v)[32], int m0, int n, int pos, uint8_t* stage,
                                               int lane)
{
    const LinEpi& e = p.e;
    const int rows_ok = min(p.M - m0, 32), cols_ok = min(p.N - n, 32);
    if (rows_ok <= 0 || cols_ok <= 0) return;
    if (e.bias) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            if (q * 8 < cols_ok) {
                float b[8];
                load8(e.bias + n + q * 8, b);
#pragma unroll
                for (int i = 0; i < 8; ++i) v[q * 8 + i] += b[i];
            }
        }
    }
    if (n >= e.split) {                      // the split is a multiple of 32: whole blocks
#pragma unroll
        for (int q = 0; q < 8; ++q)
            *reinterpret_cast<float4*>(stage + piece_at<8>(lane, q)) = make_float4(v[q * 4], v[q * 4 + 1], v[q * 4 + 2], v[q * 4 + 3]);
        __syncwarp();
        move_block<8, false>(stage, (uint8_t*)(e.out2 + (long long)m0 * e.ldo2 + (n - e.split)), e.ldo2 * 4, rows_ok, cols_ok / 4,
                             lane);
        __syncwarp();
        return;
    }
    if (e.kind == ZKFP_EPI_ROTATE) {
        if (lane < rows_ok && n < e.rot_end && n + 32 > e.rot_begin) {
#pragma unroll
            for (int i = 0; i < 32; i += 2) rotate_pair(e, pos, n + i, v[i], v[i + 1]);
        }
    } else if (e.kind == ZKFP_EPI_GATE) {
        move_block<4, true>(stage, (uint8_t*)e.aux + ((long long)m0 * e.ldaux + n) * 2, e.ldaux * 2, rows_ok, cols_ok / 8, lane);
        __syncwarp();
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            float g[8];
            unpack8(*reinterpret_cast<const uint4*>(stage + piece_at<4>(lane, q)), g);
#pragma unroll
            for (int i = 0; i < 8; ++i) v[q * 8 + i] = sigmoid_f(v[q * 8 + i]) * g[i];
        }
        __syncwarp();
    } else if (e.kind == ZKFP_EPI_GLU) {
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] = v[2 * i] * sigmoid_f(v[2 * i]) * v[2 * i + 1];
        const long long o = (long long)m0 * e.ldo + (n >> 1);
        if (e.out_bf16) {
#pragma unroll
            for (int q = 0; q < 2; ++q)
                *reinterpret_cast<uint4*>(stage + piece_at<2>(lane, q)) =
                    make_uint4(pack_bf16(v[q * 8], v[q * 8 + 1]), pack_bf16(v[q * 8 + 2], v[q * 8 + 3]),
                               pack_bf16(v[q * 8 + 4], v[q * 8 + 5]), pack_bf16(v[q * 8 + 6], v[q * 8 + 7]));
            __syncwarp();
            move_block<2, false>(stage, (uint8_t*)((bf16*)e.out + o), e.ldo * 2, rows_ok, cols_ok / 16, lane);
        } else {
#pragma unroll
            for (int q = 0; q < 4; ++q)
                *reinterpret_cast<float4*>(stage + piece_at<4>(lane, q)) = make_float4(v[q * 4], v[q * 4 + 1], v[q * 4 + 2], v[q * 4 + 3]);
            __syncwarp();
            move_block<4, false>(stage, (uint8_t*)((float*)e.out + o), e.ldo * 4, rows_ok, cols_ok / 8, lane);
        }
        __syncwarp();
        return;
    }
    const long long o = (long long)m0 * e.ldo + n;
    if (e.out_bf16) {
#pragma unroll
        for (int q = 0; q < 4; ++q)
            *reinterpret_cast<uint4*>(stage + piece_at<4>(lane, q)) =
                make_uint4(pack_bf16(v[q * 8], v[q * 8 + 1]), pack_bf16(v[q * 8 + 2], v[q * 8 + 3]),
                           pack_bf16(v[q * 8 + 4], v[q * 8 + 5]), pack_bf16(v[q * 8 + 6], v[q * 8 + 7]));
        __syncwarp();
        move_block<4, false>(stage, (uint8_t*)((bf16*)e.out + o), e.ldo * 2, rows_ok, cols_ok / 8, lane);
    } else {
#pragma unroll
        for (int q = 0; q < 8; ++q)
            *reinterpret_cast<float4*>(stage + piece_at<8>(lane, q)) = make_float4(v[q * 4], v[q * 4 + 1], v[q * 4 + 2], v[q * 4 + 3]);
        __syncwarp();
        move_block<8, false>(stage, (uint8_t*)((float*)e.out + o), e.ldo * 4, rows_ok, cols_ok / 4, lane);
    }
    __syncwarp();
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
    // work items: (tile, share of K); all shares of a tile run at the same time
    const int total = p.m_tiles * p.n_tiles * p.ksplit, pairs = gridDim.x >> 1, first = blockIdx.x >> 1;
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
                tile_coords(p, t / p.ksplit, mt, nt);
                const int kb0 = (t % p.ksplit) * p.kb_per_split, kb1 = min(kb0 + p.kb_per_split, p.kblocks);
                const int row_a = mt * 256 + (int)rank * kTM, row_w = nt * p.NT + (int)rank * (p.NT / 2);
                for (int kb = kb0; kb < kb1; ++kb) {
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
                const int kb0 = (t % p.ksplit) * p.kb_per_split, kb1 = min(kb0 + p.kb_per_split, p.kblocks);
                for (int kb = kb0; kb < kb1; ++kb) {
                    if (!mbar_wait(smem_u32(&s.full[stage]), phase, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t sa = smem0 + (uint32_t)stage * stage_bytes;
                    const uint64_t ad = smem_desc_sw128(sa), wd = smem_desc_sw128(sa + kBytesA);
#pragma unroll
                    for (int k = 0; k < kBK / 16; ++k)
                        umma_bf16_pair(acc, ad + (uint64_t)(k * 2), wd + (uint64_t)(k * 2), idesc, (kb > kb0 || k) ? 1u : 0u);
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
        uint8_t* stage = base + (uint32_t)p.stages * stage_bytes + (uint32_t)(warp - 2) * kStageBlock;
        int buf = 0;
        uint32_t acc_phase = 0;
        for (int t = first; t < total; t += pairs) {
            int mt, nt;
            const int tile = t / p.ksplit;
            tile_coords(p, tile, mt, nt);
            if (!mbar_wait(smem_u32(&s.acc_full[buf]), acc_phase, abort_flag)) break;
            tc_fence_after();
            const int m0 = mt * 256 + (int)rank * kTM + quarter * 32, n0 = nt * p.NT;
            const int pos = (p.e.kind == ZKFP_EPI_ROTATE && m0 + lane < p.M) ? epi_position(p.e, m0 + lane) : 0;
            float* part = p.partial + (((long long)t * 2 + rank) * p.NT) * kTM + quarter * 32 + lane;
            for (int c = c_begin; c < c_end; c += 32) {
                float v[32];
                tmem_ld32(tq + (uint32_t)(buf * 256 + c), v);
                tmem_ld_wait();
                if (c + 32 >= c_end) {
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive_remote(smem_u32(&s.acc_empty[buf]), 0);
                }
                if (p.ksplit == 1) {
                    epilogue_block(p, v, m0, n0 + c, pos, stage, lane);
                } else if (m0 < p.M && n0 + c < p.N) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) __stcg(part + (long long)(c + i) * kTM, v[i]);
                }
            }
            if (p.ksplit > 1) {
                __threadfence();
                __syncwarp();
                unsigned* cnt = p.counter + (tile * 2 + (int)rank) * kEpiWarps + (warp - 2);
                unsigned seen = 0;
                if (lane == 0) seen = atomicAdd(cnt, 1u);
                seen = __shfl_sync(0xffffffffu, seen, 0);
                if (seen == (unsigned)p.ksplit - 1u) {
                    __threadfence();
                    const long long step = (long long)2 * p.NT * kTM;
                    const float* src = p.partial + (((long long)tile * p.ksplit * 2 + rank) * p.NT) * kTM + quarter * 32 + lane;
                    for (int c = c_begin; c < c_end; c += 32) {
                        if (m0 >= p.M || n0 + c >= p.N) break;
                        float v[32] = {};
                        int k = 0;
                        for (; k + 4 <= p.ksplit; k += 4) {      // four shares in flight, added in order
                            float a[4][32];
#pragma unroll
                            for (int q = 0; q < 4; ++q)
#pragma unroll
                                for (int i = 0; i < 32; ++i) a[q][i] = __ldcg(src + (k + q) * step + (long long)(c + i) * kTM);
#pragma unroll
                            for (int q = 0; q < 4; ++q)
#pragma unroll
                                for (int i = 0; i < 32; ++i) v[i] += a[q][i];
                        }
                        for (; k < p.ksplit; ++k) {
#pragma unroll
                            for (int i = 0; i < 32; ++i) v[i] += __ldcg(src + k * step + (long long)(c + i) * kTM);
                        }
                        epilogue_block(p, v, m0, n0 + c, pos, stage, lane);
                    }
                    if (lane == 0) *cnt = 0;
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

// partial sums and arrival counters of split launches: one block per device, allocated at first use (calls on
// several streams of one device must not overlap, like every call that uses library-owned scratch)
static bool split_workspace(int pairs, float** partial, unsigned** counter, cudaStream_t st)
{
    static struct { float* p; unsigned* c; } ws[64];
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return false;
    if (!ws[dev].p) {
        void *a = nullptr, *b = nullptr;
        const size_t bytes_c = (size_t)pairs * 2 * kEpiWarps * sizeof(unsigned);
        if (cudaMalloc(&a, (size_t)pairs * 2 * 256 * kTM * sizeof(float)) != cudaSuccess) return false;
        if (cudaMalloc(&b, bytes_c) != cudaSuccess || cudaMemsetAsync(b, 0, bytes_c, st) != cudaSuccess) return false;
        ws[dev].p = (float*)a;
        ws[dev].c = (unsigned*)b;
    }
    *partial = ws[dev].p;
    *counter = ws[dev].c;
    return true;
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
    // few tiles, deep K: several pairs per tile, each with at least four K blocks
    auto split = [&](long long tiles) {
        if (tiles * 2 > pairs || p.kblocks < 8) return 1ll;
        const long long want = pairs / tiles < p.kblocks / 4 ? pairs / tiles : p.kblocks / 4;
        const long long per = (p.kblocks + want - 1) / want;
        return (p.kblocks + per - 1) / per;
    };
    // the widest tile unless narrower ones spread the work over more pairs: cost = rounds x K blocks x time of one
    // block's MMAs, which depends only weakly on the width
    long long best = 0;
    for (int nt = 256; nt >= 64; nt >>= 1) {
        const long long tiles = (long long)p.m_tiles * ((p.N + nt - 1) / nt), ks = split(tiles);
        const long long cost = (tiles * ks + pairs - 1) / pairs * ((p.kblocks + ks - 1) / ks) * (nt + 256);
        if (nt == 256 || cost < best) { best = cost; p.NT = nt; }
    }
    p.n_tiles = (p.N + p.NT - 1) / p.NT;
    p.panel = p.m_tiles < 8 ? p.m_tiles : 8;
    if ((long long)p.m_tiles * p.n_tiles > 0x7fffffffll) return ZKDS_ERR_UNSUPPORTED;
    const uint32_t stage_bytes = kBytesA + (uint32_t)(p.NT / 2) * kBK * 2;
    const int few = p.m_tiles * p.n_tiles;
    p.ksplit = (int)split(few);
    p.kb_per_split = (p.kblocks + p.ksplit - 1) / p.ksplit;
    p.partial = nullptr;
    p.counter = nullptr;
    if (p.ksplit > 1 && !split_workspace(pairs, &p.partial, &p.counter, st)) return ZKDS_ERR_WORKSPACE;
    p.stages = (int)((192u * 1024u) / stage_bytes);
    if (p.stages > kMaxStages) p.stages = kMaxStages;
    CUtensorMap tmA, tmW;
    const uint64_t da[2] = {(uint64_t)a.K, (uint64_t)a.M}, dw[2] = {(uint64_t)a.K, (uint64_t)a.N};
    const uint64_t sa[1] = {(uint64_t)a.lda * 2}, sw[1] = {(uint64_t)a.ldw * 2};
    const uint32_t ba[2] = {kBK, kTM}, bw[2] = {kBK, (uint32_t)p.NT / 2};
    if (!fp_tensor_map(&tmA, a.A, 2, da, sa, ba) || !fp_tensor_map(&tmW, a.W, 2, dw, sw, bw)) return ZKDS_ERR_UNSUPPORTED;
    const size_t smem = (size_t)stage_bytes * p.stages + kEpiWarps * kStageBlock + 1024;
    // always the same limit, not this launch's size: earlier launches may sit in a captured graph
    ZKDS_CUDA(cudaFuncSetAttribute(linear_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kLinearSmemMax));
    const int tiles = few * p.ksplit;
    const unsigned grid = 2u * (unsigned)(tiles < pairs ? tiles : pairs);
    linear_tc_kernel<<<grid, kThreadsTc, smem, st>>>(tmA, tmW, p);
    return fp_launched();
}

}  // namespace zkds
