// Linear attention with a decaying state on the tensor cores (bfloat16 operands, 32-bit state), in chunks of 128 tokens.
//
// With l_t = log2 a_1 + .. + log2 a_t inside a chunk and S the state before it,
//   out_t  = 2^(l_t) S^T q_t + sum_{j <= t} 2^(l_t - l_j) w_j (q_t . k_j) v_j
//   S_next = 2^(l_end) S + sum_j k_j (2^(l_end - l_j) w_j v_j)^T
// A CTA owns 64 value columns of one head and walks over the chunks; its state stays in registers, 32 values a thread.
// Scores, both output terms and the state's increment are MMAs.  What feeds the state or is read from it enters the MMAs as
// two bfloat16 numbers (value and remainder), so the state keeps 32-bit accuracy; decayed scores are rounded once, like
// softmax weights.  Decays over whole blocks of 32 columns are split at the block's end into a column and a row factor,
// neither above 1; only the blocks on the diagonal take an exponential per score.
//   warps 0-7  element-wise work: two threads share a row (token or state row), half of the columns each
//   warp 8     MMA issue        warp 9  TMA loads, running decays
// Sequences with few heads are cut into segments that run side by side: a first launch leaves the state that each segment
// builds from zero, scan_segments_kernel chains them, and the output launch starts every segment from its own state.
#include <cuda.h>

#include "float_common.cuh"
#include "tcgen05.cuh"

namespace zkds {

bool fp_tensor_map(CUtensorMap* map, const void* base, int rank, const uint64_t* dims, const uint64_t* strides_bytes,
                   const uint32_t* box);

namespace {

constexpr int kL = 128;                        // tokens per chunk
constexpr int kPT = 64;                        // value columns per CTA
constexpr uint32_t kSegB = kL * 128;           // bytes of 128 rows x 64 bfloat16
constexpr int kScanThreads = 320;
constexpr int kScanMinTokens = 17;             // shorter steps go token by token
constexpr size_t kScanSmemAll = 227 * 1024;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float exp2_fast(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct ScanTcParams {
    bf16* out;
    const float* decay;
    const float* step;
    const float* step_bias;
    const float* skip;
    float* state;
    float* seg_state;                          // [batch][head][segment][n][p]
    float* seg_decay;                          // [batch][head][segment]: log2 of the segment's whole decay
    const int* start;
    const int* slots;
    long long o_tok, o_head, step_tok, n_slots;
    int seq, heads, heads_per_qk, n, p, segq, chunks, chunks_per_segment, segments;
    float k_scale;
    uint32_t smem_bytes;
    int* error_flag;
};

struct ScanTcShared {
    float l[2][kL], w[2][kL];                  // running log2 decay, weight
    float col[kL];                             // decay from a token to the end of its block of 32, times its weight
    uint64_t full[2], empty[2], s_full[2], vp_full, p_full, ds_full, st_full, o_full;
    uint32_t tmem;
    int abort;
};

// columns of tensor memory
constexpr uint32_t kColS = 0, kColO = 256, kColQS = 320, kColD = 448;

// 32 values of row `row` as bfloat16 pieces 4 * half .. + 3 of its 128 bytes, and what the rounding left in a second tile
__device__ __forceinline__ void store_split(uint8_t* hi, uint8_t* lo, int row, int half, const float (&v)[32])
{
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        uint32_t h[4], r[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float a = v[q * 8 + 2 * i], b = v[q * 8 + 2 * i + 1];
            h[i] = pack_bf16(a, b);
            r[i] = pack_bf16(a - bf16_lo(h[i]), b - bf16_hi(h[i]));
        }
        const uint32_t at = (uint32_t)row * 128u + (uint32_t)(((half * 4 + q) ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(hi + at) = make_uint4(h[0], h[1], h[2], h[3]);
        *reinterpret_cast<uint4*>(lo + at) = make_uint4(r[0], r[1], r[2], r[3]);
    }
}

__device__ __forceinline__ void load_row(const uint8_t* tile, int row, int half, float (&v)[32])
{
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        float x[8];
        unpack8(*reinterpret_cast<const uint4*>(tile + row * 128 + (((half * 4 + q) ^ (row & 7)) << 4)), x);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[q * 8 + i] = x[i];
    }
}

// OUT false: only the state that a segment builds from zero
template <bool OUT>
__global__ void __launch_bounds__(kScanThreads, 1)
scan_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                  const __grid_constant__ CUtensorMap tmV, const ScanTcParams p)
{
    extern __shared__ __align__(1024) uint8_t raw[];
    uint8_t* base = (uint8_t*)(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    const int rows_s = p.segq * 64;                                       // rows of the state tiles
    const uint32_t bytes_q = OUT ? (uint32_t)p.segq * kSegB : 0u, stage_bytes = bytes_q + 3 * kSegB;
    const uint32_t bytes_s = (uint32_t)rows_s * 128u, tile_bytes = 2 * stage_bytes + 2 * kSegB + 2 * bytes_s;
    if (base + tile_bytes + sizeof(ScanTcShared) > raw + p.smem_bytes) {  // not the alignment the host counted on
        if (threadIdx.x == 0) *(volatile int*)p.error_flag = 1;
        return;
    }
    ScanTcShared& s = *reinterpret_cast<ScanTcShared*>(base + tile_bytes);
    uint8_t* vp = base + 2 * stage_bytes;                                 // scaled values: rounded, remainder
    uint8_t* st = vp + 2 * kSegB;                                         // state: rounded, remainder
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slice = blockIdx.x, head = blockIdx.y, b = blockIdx.z / p.segments, seg = blockIdx.z % p.segments;
    const int c_begin = seg * p.chunks_per_segment, nc = min(p.chunks_per_segment, p.chunks - c_begin);
    const long long slot = p.slots[b];
    if (slot < 0 || slot >= p.n_slots || nc <= 0) return;
    const uint32_t smem0 = smem_u32(base);
    volatile int* abort_flag = &s.abort;

    if (threadIdx.x == 0) {
        s.abort = 0;
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&s.full[i]), 2);
            mbar_init(smem_u32(&s.empty[i]), 9);
            mbar_init(smem_u32(&s.s_full[i]), 1);
        }
        mbar_init(smem_u32(&s.vp_full), 8);
        mbar_init(smem_u32(&s.p_full), 8);
        mbar_init(smem_u32(&s.ds_full), 1);
        mbar_init(smem_u32(&s.st_full), 8);
        mbar_init(smem_u32(&s.o_full), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    if (warp == 8) tmem_alloc(smem_u32(&s.tmem), 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s.tmem;

    if (warp == 9) {
        const float decay = p.decay[head], bias = p.step ? p.step_bias[head] : 0.f;
        const float fixed = fmaxf(log2f(decay), -150.f);
        for (int c = 0; c < nc; ++c) {
            const int stage = c & 1, t0 = (c_begin + c) * kL, y = b * p.seq + t0;
            if (!mbar_wait(smem_u32(&s.empty[stage]), (uint32_t)((c >> 1) & 1) ^ 1u, abort_flag)) break;
            if (lane == 0) {
                const uint32_t bar = smem_u32(&s.full[stage]), dst = smem0 + (uint32_t)stage * stage_bytes;
                mbar_expect_tx(bar, stage_bytes);
                const int hq = head / p.heads_per_qk;
                if (OUT)
                    for (int k = 0; k < p.segq; ++k) tma_load_3d(dst + (uint32_t)k * kSegB, &tmQ, k * 64, hq, y, bar);
                for (int k = 0; k < 2; ++k) tma_load_3d(dst + bytes_q + (uint32_t)k * kSegB, &tmK, k * 64, hq, y, bar);
                tma_load_3d(dst + bytes_q + 2 * kSegB, &tmV, slice * kPT, head, y, bar);
            }
            float l[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int t = lane * 4 + i;
                l[i] = 0.f;                     // tokens behind the end: no decay, no weight
                w[i] = 0.f;
                if (t0 + t < p.seq) {
                    l[i] = fixed;
                    w[i] = p.k_scale;
                    if (p.step) {
                        const float dt = softplus_f(p.step[(long long)(y + t) * p.step_tok + head] + bias);
                        l[i] = -decay * dt * kLog2e;
                        w[i] = p.k_scale * dt;
                    }
                }
                if (i) l[i] += l[i - 1];
            }
            float before = l[3];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, before, o);
                if (lane >= o) before += x;
            }
            before = __shfl_up_sync(0xffffffffu, before, 1);
            if (lane == 0) before = 0.f;
            *reinterpret_cast<float4*>(&s.l[stage][lane * 4]) = make_float4(before + l[0], before + l[1], before + l[2], before + l[3]);
            *reinterpret_cast<float4*>(&s.w[stage][lane * 4]) = make_float4(w[0], w[1], w[2], w[3]);
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s.full[stage]));
        }
    } else if (warp == 8) {
        if (lane == 0) {
            const uint32_t idesc_qk = idesc_bf16(kL, kL), idesc_v = idesc_bf16(kL, kPT, true);
            const uint32_t idesc_d = idesc_v | (1u << 15);              // both operands with their tokens as rows
            const uint32_t vhi = smem_u32(vp), vlo = vhi + kSegB, shi = smem_u32(st), slo = shi + bytes_s;
            auto scores = [&](int c) {
                const uint32_t q = smem0 + (uint32_t)(c & 1) * stage_bytes, k = q + bytes_q;
                const uint32_t d = tmem + kColS + (uint32_t)(c & 1) * 128u;
                for (int sg = 0; sg < p.segq; ++sg) {
                    const uint64_t ad = smem_desc_sw128(q + (uint32_t)sg * kSegB), bd = smem_desc_sw128(k + (uint32_t)sg * kSegB);
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (sg * 64 + i * 16 < p.n)
                            umma_bf16(d, ad + (uint64_t)(i * 2), bd + (uint64_t)(i * 2), idesc_qk, (sg | i) ? 1u : 0u);
                }
                umma_commit(smem_u32(&s.s_full[c & 1]));
            };
            auto from_state = [&](int c) {
                const uint32_t q = smem0 + (uint32_t)(c & 1) * stage_bytes, d = tmem + kColQS + (uint32_t)(c & 1) * 64u;
                for (int sg = 0; sg < p.segq; ++sg) {
                    const uint64_t ad = smem_desc_sw128(q + (uint32_t)sg * kSegB);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int k = sg * 4 + i;
                        if (k * 16 >= p.n) continue;
                        umma_bf16(d, ad + (uint64_t)(i * 2), smem_desc_mn_sw128(shi, kSegB) + (uint64_t)(k * 128), idesc_v, k ? 1u : 0u);
                        umma_bf16(d, ad + (uint64_t)(i * 2), smem_desc_mn_sw128(slo, kSegB) + (uint64_t)(k * 128), idesc_v, 1u);
                    }
                }
            };
            bool ok = true;
            if (OUT) {
                ok = mbar_wait(smem_u32(&s.full[0]), 0, abort_flag);
                tc_fence_after();
                if (ok) scores(0);
                if (ok) ok = mbar_wait(smem_u32(&s.st_full), 0, abort_flag);
                tc_fence_after();
                if (ok) from_state(0);
            }
            for (int c = 0; c < nc && ok; ++c) {
                const uint32_t ph = (uint32_t)(c & 1), tile = smem0 + (uint32_t)(c & 1) * stage_bytes + bytes_q;
                if (!(ok = mbar_wait(smem_u32(&s.full[c & 1]), (uint32_t)((c >> 1) & 1), abort_flag) &&
                           mbar_wait(smem_u32(&s.vp_full), ph, abort_flag)))
                    break;
                tc_fence_after();
                const uint64_t kd = smem_desc_mn_sw128(tile, kSegB);
#pragma unroll
                for (int k = 0; k < kL / 16; ++k) {
                    umma_bf16(tmem + kColD, kd + (uint64_t)(k * 128), smem_desc_mn_sw128(vhi, kSegB) + (uint64_t)(k * 128), idesc_d, k ? 1u : 0u);
                    umma_bf16(tmem + kColD, kd + (uint64_t)(k * 128), smem_desc_mn_sw128(vlo, kSegB) + (uint64_t)(k * 128), idesc_d, 1u);
                }
                umma_commit(smem_u32(&s.ds_full));
                if (OUT) {
                    if (c + 1 < nc) {
                        if (!(ok = mbar_wait(smem_u32(&s.full[(c + 1) & 1]), (uint32_t)(((c + 1) >> 1) & 1), abort_flag))) break;
                        tc_fence_after();
                        scores(c + 1);
                    }
                    if (!(ok = mbar_wait(smem_u32(&s.p_full), ph, abort_flag))) break;
                    tc_fence_after();
                    const uint32_t a = tmem + kColS + ph * 128u;
                    const uint64_t vd = smem_desc_mn_sw128(tile + 2 * kSegB, kSegB);
#pragma unroll
                    for (int k = 0; k < kL / 16; ++k)                   // weights of columns 64.. start 64 columns further on
                        umma_bf16_ts(tmem + kColO, a + (uint32_t)((k >> 2) * 64 + (k & 3) * 8), vd + (uint64_t)(k * 128), idesc_v, k ? 1u : 0u);
                    umma_commit(smem_u32(&s.o_full));
                }
                umma_commit(smem_u32(&s.empty[c & 1]));
                if (OUT && c + 1 < nc) {
                    if (!(ok = mbar_wait(smem_u32(&s.st_full), (uint32_t)((c + 1) & 1), abort_flag))) break;
                    tc_fence_after();
                    from_state(c + 1);
                }
            }
        }
    } else {
        const int half = warp >> 2, quarter = warp & 3, row = quarter * 32 + lane;
        const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
        const int col0 = slice * kPT + half * 32;
        const bool fresh = p.start[b] == 0;
        const long long sh = ((long long)b * p.heads + head) * p.segments + seg;
        float* state = p.state + ((slot * p.heads + head) * p.n + row) * p.p + col0;
        float* seg_state = p.seg_state + (sh * p.n + row) * p.p + col0;
        const float* from = !OUT ? nullptr : p.segments > 1 ? seg_state : fresh ? nullptr : state;
        float S[32];
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
            float v[8] = {};
            if (from && row < p.n && col0 + i < p.p) load8(from + i, v);
#pragma unroll
            for (int k = 0; k < 8; ++k) S[i + k] = v[k];
        }
        auto publish = [&](uint64_t* bar) {                              // shared-memory tiles for the tensor core
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(bar));
        };
        if (OUT) {
            if (row < rows_s) store_split(st, st + bytes_s, row, half, S);
            publish(&s.st_full);
        }
        const float skip = p.skip ? p.skip[head] : 0.f;
        float total = 0.f;
        for (int c = 0; c < nc; ++c) {
            const int stage = c & 1;
            const uint32_t ph = (uint32_t)(c & 1);
            const uint8_t* tile_v = base + (uint32_t)stage * stage_bytes + bytes_q + 2 * kSegB;
            if (!mbar_wait(smem_u32(&s.full[stage]), (uint32_t)((c >> 1) & 1), abort_flag)) break;
            const float* l = s.l[stage];
            const float l_row = l[row], l_end = l[kL - 1];
            // values scaled by what is left of them at the chunk's end
            const float col = exp2_fast(l[row | 31] - l_row) * s.w[stage][row];
            {
                if (OUT && half == 0) s.col[row] = col;
                const float f = exp2_fast(l_end - l[row | 31]) * col;
                float v[32];
                load_row(tile_v, row, half, v);
#pragma unroll
                for (int i = 0; i < 32; ++i) v[i] *= f;
                store_split(vp, vp + kSegB, row, half, v);
                publish(&s.vp_full);
            }
            if (OUT) {
                asm volatile("bar.sync 1, 256;" ::: "memory");          // every column factor is there
                if (!mbar_wait(smem_u32(&s.s_full[c & 1]), (uint32_t)((c >> 1) & 1), abort_flag)) break;
                tc_fence_after();
                const uint32_t tS = tmem + kColS + ph * 128u + lanes + (uint32_t)half * 64u;
                float v[2][32];
                if (half * 2 <= quarter) tmem_ld32(tS, v[0]);
                if (half * 2 + 1 <= quarter) tmem_ld32(tS + 32u, v[1]);
                tmem_ld_wait();
#pragma unroll
                for (int q = 0; q < 2; ++q) {
                    const int cb = half * 2 + q;                        // block of 32 columns
                    uint32_t w[16];
                    if (cb > quarter) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) w[i] = 0u;
                    } else {
                        if (cb < quarter) {
                            const float f = exp2_fast(l_row - l[cb * 32 + 31]);
#pragma unroll
                            for (int i = 0; i < 32; i += 4) {
                                const float4 g = *reinterpret_cast<const float4*>(&s.col[cb * 32 + i]);
                                v[q][i] *= f * g.x;
                                v[q][i + 1] *= f * g.y;
                                v[q][i + 2] *= f * g.z;
                                v[q][i + 3] *= f * g.w;
                            }
                        } else {
#pragma unroll
                            for (int i = 0; i < 32; ++i) {
                                const float g = exp2_fast(l_row - l[cb * 32 + i]) * s.w[stage][cb * 32 + i];
                                v[q][i] = i <= lane ? v[q][i] * g : 0.f;
                            }
                        }
#pragma unroll
                        for (int i = 0; i < 16; ++i) w[i] = pack_bf16(v[q][2 * i], v[q][2 * i + 1]);
                    }
                    tmem_st16(tS + (uint32_t)(q * 16), w);
                }
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&s.p_full));
            }
            // the state behind the chunk
            if (!mbar_wait(smem_u32(&s.ds_full), ph, abort_flag)) break;
            tc_fence_after();
            {
                float d[32];
                tmem_ld32(tmem + kColD + lanes + (uint32_t)half * 32u, d);
                tmem_ld_wait();
                const float f = exp2_fast(l_end);
#pragma unroll
                for (int i = 0; i < 32; ++i) S[i] = fmaf(f, S[i], d[i]);
                total += l_end;
                if (OUT && c + 1 < nc) {
                    if (row < rows_s) store_split(st, st + bytes_s, row, half, S);
                    publish(&s.st_full);
                }
            }
            if (OUT) {
                if (!mbar_wait(smem_u32(&s.o_full), ph, abort_flag)) break;
                tc_fence_after();
                float o[32], x[32];
                tmem_ld32(tmem + kColO + lanes + (uint32_t)half * 32u, o);
                tmem_ld32(tmem + kColQS + ph * 64u + lanes + (uint32_t)half * 32u, x);
                tmem_ld_wait();
                const float f = exp2_fast(l_row);
#pragma unroll
                for (int i = 0; i < 32; ++i) o[i] = fmaf(f, x[i], o[i]);
                if (p.skip) {
                    load_row(tile_v, row, half, x);
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = fmaf(skip, x[i], o[i]);
                }
                const int t = (c_begin + c) * kL + row;
                if (t < p.seq) {
                    bf16* dst = p.out + ((long long)b * p.seq + t) * p.o_tok + head * p.o_head + col0;
#pragma unroll
                    for (int i = 0; i < 32; i += 8)
                        if (col0 + i < p.p) {
                            float y[8];
#pragma unroll
                            for (int k = 0; k < 8; ++k) y[k] = o[i + k];
                            store8(dst + i, y);
                        }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s.empty[stage]));
        }
        float* to = OUT ? (seg == p.segments - 1 ? state : nullptr) : seg_state;
        if (to && row < p.n) {
#pragma unroll
            for (int i = 0; i < 32; i += 8)
                if (col0 + i < p.p) {
                    float y[8];
#pragma unroll
                    for (int k = 0; k < 8; ++k) y[k] = S[i + k];
                    store8(to + i, y);
                }
        }
        if (!OUT && slice == 0 && threadIdx.x == 0) p.seg_decay[sh] = total;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 8) tmem_dealloc(tmem, 512);
    if (threadIdx.x == 0 && s.abort) *(volatile int*)p.error_flag = 1;
}

// the state before every segment, in the place of the state that the segment builds from zero.  grid (n * p / 1024, heads,
// batch), four values a thread
__global__ void __launch_bounds__(256)
scan_segments_kernel(const ScanTcParams p)
{
    const int b = blockIdx.z, head = blockIdx.y, size = p.n * p.p, i = (int)(blockIdx.x * 256 + threadIdx.x) * 4;
    const long long slot = p.slots[b];
    if (i >= size || slot < 0 || slot >= p.n_slots) return;
    float4 run = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.start[b] != 0) run = *reinterpret_cast<const float4*>(p.state + (slot * p.heads + head) * size + i);
    const long long sh = ((long long)b * p.heads + head) * p.segments;
    for (int s = 0; s < p.segments; ++s) {
        float4* at = reinterpret_cast<float4*>(p.seg_state + (sh + s) * size + i);
        const float4 mine = *at;
        const float f = exp2_fast(p.seg_decay[sh + s]);
        *at = run;
        run.x = fmaf(f, run.x, mine.x); run.y = fmaf(f, run.y, mine.y);
        run.z = fmaf(f, run.z, mine.z); run.w = fmaf(f, run.w, mine.w);
    }
}

size_t scan_smem(int n)
{
    const size_t segq = (size_t)(n + 63) / 64;
    const size_t bytes = 2 * (segq + 3) * kSegB + 2 * kSegB + 2 * segq * 64 * 128 + sizeof(ScanTcShared) + 256;
    return bytes + 1024 < kScanSmemAll ? bytes + 1024 : kScanSmemAll;
}

// segments that run side by side: enough CTAs for every SM, no segment shorter than four chunks
int scan_segments(const zkfp_scan_args& a)
{
    const long long chunks = (a.seq + kL - 1) / kL, ctas = (a.p + kPT - 1) / kPT * a.heads * a.batch;
    long long s = fp_sm_count() / ctas;
    if (s > chunks / 4) s = chunks / 4;
    if (s < 2) return 1;
    const long long per = (chunks + s - 1) / s;
    return (int)((chunks + per - 1) / per);
}

}  // namespace

bool scan_tc_takes(const zkfp_scan_args& a)
{
    return a.dtype == ZKFP_BF16 && a.seq >= kScanMinTokens && a.n <= 128 && a.heads % a.heads_per_qk == 0 &&
           a.batch * a.seq < 0x40000000;
}

long long scan_tc_scratch(const zkfp_scan_args& a)
{
    const long long s = scan_segments(a);
    return s > 1 ? a.batch * a.heads * s * ((long long)a.n * a.p + 1) : 0;
}

int launch_scan_tc(const zkfp_scan_args& a, cudaStream_t st)
{
    ScanTcParams p;
    p.out = (bf16*)a.out; p.decay = a.decay; p.step = a.step; p.step_bias = a.step_bias; p.skip = a.skip; p.state = a.state;
    p.start = a.start; p.slots = a.slots; p.o_tok = a.o_tok; p.o_head = a.o_head; p.step_tok = a.step_tok;
    p.n_slots = a.n_slots; p.seq = (int)a.seq; p.heads = (int)a.heads; p.heads_per_qk = a.heads_per_qk; p.n = a.n; p.p = a.p;
    p.segq = (a.n + 63) / 64;
    p.chunks = (p.seq + kL - 1) / kL;
    p.segments = scan_segments(a);
    p.chunks_per_segment = (p.chunks + p.segments - 1) / p.segments;
    p.seg_state = a.scratch;
    p.seg_decay = a.scratch ? a.scratch + a.batch * a.heads * p.segments * (long long)a.n * a.p : nullptr;
    if (p.segments > 1 && !a.scratch) return ZKDS_ERR_ARG;
    p.k_scale = a.k_scale;
    p.error_flag = fp_error_flag();
    if (!p.error_flag) return ZKDS_ERR_WORKSPACE;
    const uint64_t rows = (uint64_t)(a.batch * a.seq), hqk = (uint64_t)(a.heads / a.heads_per_qk);
    const uint64_t dqk[3] = {(uint64_t)a.n, hqk, rows}, dv[3] = {(uint64_t)a.p, (uint64_t)a.heads, rows};
    const uint64_t sq[2] = {(uint64_t)a.qk_head * 2, (uint64_t)a.q_tok * 2}, sk[2] = {(uint64_t)a.qk_head * 2, (uint64_t)a.k_tok * 2};
    const uint64_t sv[2] = {(uint64_t)a.v_head * 2, (uint64_t)a.v_tok * 2};
    const uint32_t box[3] = {64, 1, kL};
    CUtensorMap q, k, v;
    if (!fp_tensor_map(&q, a.q, 3, dqk, sq, box) || !fp_tensor_map(&k, a.k, 3, dqk, sk, box) || !fp_tensor_map(&v, a.v, 3, dv, sv, box))
        return ZKDS_ERR_UNSUPPORTED;
    p.smem_bytes = (uint32_t)scan_smem(a.n);
    const dim3 grid((unsigned)((a.p + kPT - 1) / kPT), (unsigned)a.heads, (unsigned)(a.batch * p.segments));
    if (grid.z > 65535u) return ZKDS_ERR_UNSUPPORTED;
    if (p.segments > 1) {
        ZKDS_CUDA(cudaFuncSetAttribute(scan_chunk_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kScanSmemAll));
        scan_chunk_kernel<false><<<grid, kScanThreads, p.smem_bytes, st>>>(q, k, v, p);
        int rc = fp_launched();
        if (rc != ZKDS_OK) return rc;
        scan_segments_kernel<<<dim3((unsigned)((a.n * a.p + 1023) / 1024), (unsigned)a.heads, (unsigned)a.batch), 256, 0, st>>>(p);
        rc = fp_launched();
        if (rc != ZKDS_OK) return rc;
    }
    ZKDS_CUDA(cudaFuncSetAttribute(scan_chunk_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kScanSmemAll));
    scan_chunk_kernel<true><<<grid, kScanThreads, p.smem_bytes, st>>>(q, k, v, p);
    return fp_launched();
}

}  // namespace zkds
