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
//   warps 0-15  element-wise work: four threads share a row (token or state row), a quarter of the columns each
//   warp 16     issues the MMAs of scores and their product with the values      warp 17  TMA loads
//   warp 19     issues the MMAs of the state's increment and of its output        warp 18  TMA stores
// The running decays of every chunk are made beforehand (scan_decay_kernel) and come with the values.  While the tensor core
// works on a chunk's last product the element-wise warps already scale the next chunk's values.  The output tile takes the
// place of the chunk's queries in shared memory.
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
constexpr int kElemWarps = 16;
constexpr int kScanThreads = 32 * (kElemWarps + 4);
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
    const float* decay;
    const float* step;
    const float* step_bias;
    const float* skip;
    float* state;
    float* seg_state;                          // [batch][head][segment][n][p]
    float* seg_decay;                          // [batch][head][segment]: log2 of the segment's whole decay
    float* decays;                             // [batch][head][chunk]: ChunkDecays
    const int* start;
    const int* slots;
    long long step_tok, n_slots;
    int seq, heads, heads_per_qk, n, p, segq, chunks, chunks_per_segment, segments;
    float k_scale;
    uint32_t smem_bytes[2];                    // without and with outputs
    int* error_flag;
};

struct ChunkDecays {
    float l[kL];                               // running log2 decay
    float lw[kL];                              // the same less log2 of the token's weight
    float col[kL - 32];                        // decay from a token to the end of its block of 32, times its weight
};

template <int STAGES>
struct ScanTcShared {
    ChunkDecays d[STAGES];
    uint64_t qk_full[STAGES], qk_empty[STAGES], v_full[STAGES], v_empty[STAGES], out_full[2], vp_full[2], ds_full[2], s_full, p_full, st_full, o_full;
    uint32_t tmem;
    int abort;
};
static_assert(sizeof(ChunkDecays) % 16 == 0, "copied in 16-byte units");

// columns of tensor memory: scores, weights, both output terms (of the state's two numbers side by side), increment (same)
constexpr uint32_t kColS = 0, kColP = 128, kColO = 192, kColQS = 256, kColD = 384;

// byte offset of 16-byte piece `piece` of row `row`
__device__ __forceinline__ uint32_t at_piece(int row, int piece) { return (uint32_t)row * 128u + (uint32_t)((piece ^ (row & 7)) << 4); }

// 16 values of row `row` as pieces 2 * part, 2 * part + 1 in bfloat16, and what the rounding left in a second tile
__device__ __forceinline__ void store_split(uint8_t* hi, uint8_t* lo, int row, int part, const float (&v)[16])
{
#pragma unroll
    for (int q = 0; q < 2; ++q) {
        uint32_t h[4], r[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float a = v[q * 8 + 2 * i], b = v[q * 8 + 2 * i + 1];
            h[i] = pack_bf16(a, b);
            r[i] = pack_bf16(a - bf16_lo(h[i]), b - bf16_hi(h[i]));
        }
        const uint32_t at = at_piece(row, part * 2 + q);
        *reinterpret_cast<uint4*>(hi + at) = make_uint4(h[0], h[1], h[2], h[3]);
        *reinterpret_cast<uint4*>(lo + at) = make_uint4(r[0], r[1], r[2], r[3]);
    }
}

__device__ __forceinline__ void load_row(const uint8_t* tile, int row, int part, float (&v)[16])
{
#pragma unroll
    for (int q = 0; q < 2; ++q) {
        float x[8];
        unpack8(*reinterpret_cast<const uint4*>(tile + at_piece(row, part * 2 + q)), x);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[q * 8 + i] = x[i];
    }
}

__device__ __forceinline__ void tmem_ld16f(uint32_t taddr, float (&v)[16])
{
    tmem_ldn(taddr, reinterpret_cast<int32_t(&)[16]>(v));
}

// decays of a chunk of 32 heads: a warp takes four heads, a lane four tokens.  grid (chunks, heads / 32, batch)
__global__ void __launch_bounds__(256)
scan_decay_kernel(const ScanTcParams p)
{
    __shared__ float raw[kL][33];
    const int c = blockIdx.x, h0 = blockIdx.y * 32, b = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (p.step) {
        float v[kL / 8];                           // all loads in flight
#pragma unroll
        for (int i = 0; i < kL / 8; ++i) {
            const int t = c * kL + i * 8 + warp;
            v[i] = t < p.seq && h0 + lane < p.heads ? p.step[((long long)b * p.seq + t) * p.step_tok + h0 + lane] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < kL / 8; ++i) raw[i * 8 + warp][lane] = v[i];
        __syncthreads();
    }
    for (int k = 0; k < 4; ++k) {
        const int hl = warp * 4 + k, head = h0 + hl;
        if (head >= p.heads) break;
        const float decay = p.decay[head], bias = p.step ? p.step_bias[head] : 0.f;
        float l[4], w[4], lw[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            l[i] = 0.f;                         // tokens behind the end: no decay, no weight
            w[i] = 0.f;
            if (c * kL + lane * 4 + i < p.seq) {
                l[i] = fmaxf(log2f(decay), -150.f);
                w[i] = p.k_scale;
                if (p.step) {
                    const float dt = softplus_f(raw[lane * 4 + i][hl] + bias);
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
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            l[i] += before;
            lw[i] = l[i] - log2f(w[i]);                                 // no weight: +infinity
        }
        const float end = __shfl_sync(0xffffffffu, l[3], lane | 7);     // of the block of 32
        ChunkDecays* d = reinterpret_cast<ChunkDecays*>(p.decays) + ((long long)b * p.heads + head) * p.chunks + c;
        *reinterpret_cast<float4*>(&d->l[lane * 4]) = make_float4(l[0], l[1], l[2], l[3]);
        *reinterpret_cast<float4*>(&d->lw[lane * 4]) = make_float4(lw[0], lw[1], lw[2], lw[3]);
        if (lane < 24)
            *reinterpret_cast<float4*>(&d->col[lane * 4]) =
                make_float4(exp2_fast(end - lw[0]), exp2_fast(end - lw[1]), exp2_fast(end - lw[2]), exp2_fast(end - lw[3]));
    }
}

// OUT false: only the state that a segment builds from zero
template <bool OUT>
__global__ void __launch_bounds__(kScanThreads, 1)
scan_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                  const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmO, const ScanTcParams p)
{
    extern __shared__ __align__(1024) uint8_t raw[];
    uint8_t* base = (uint8_t*)(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    const int rows_s = p.segq * 64;                                       // rows of the state tiles
    const uint32_t bytes_q = OUT ? (uint32_t)p.segq * kSegB : 0u, stage_bytes = bytes_q + 3 * kSegB;
    const uint32_t bytes_s = (uint32_t)rows_s * 128u;
    // without outputs there is room for a third stage, and for a second pair of value tiles instead of the state's
    constexpr int kStages = OUT ? 2 : 3;
    const uint32_t tile_bytes = kStages * stage_bytes + (OUT ? 2 * kSegB + 2 * bytes_s : 4 * kSegB), vp_step = OUT ? 0u : 2 * kSegB;
    if (base + tile_bytes + sizeof(ScanTcShared<kStages>) > raw + p.smem_bytes[OUT]) {  // not the alignment the host counted on
        if (threadIdx.x == 0) *(volatile int*)p.error_flag = 1;
        return;
    }
    ScanTcShared<kStages>& s = *reinterpret_cast<ScanTcShared<kStages>*>(base + tile_bytes);
    uint8_t* vp = base + kStages * stage_bytes;                                 // scaled values: rounded, remainder
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
        for (int i = 0; i < kStages; ++i) {
            mbar_init(smem_u32(&s.qk_full[i]), 1);
            mbar_init(smem_u32(&s.qk_empty[i]), 1);
            mbar_init(smem_u32(&s.v_full[i]), 1);
            mbar_init(smem_u32(&s.v_empty[i]), OUT ? kElemWarps : 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&s.out_full[i]), kElemWarps);
            mbar_init(smem_u32(&s.vp_full[i]), kElemWarps);
            mbar_init(smem_u32(&s.ds_full[i]), 1);
        }
        mbar_init(smem_u32(&s.s_full), 1);
        mbar_init(smem_u32(&s.p_full), kElemWarps);
        mbar_init(smem_u32(&s.st_full), kElemWarps);
        mbar_init(smem_u32(&s.o_full), 2);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    if (warp == kElemWarps) tmem_alloc(smem_u32(&s.tmem), 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s.tmem;

    // stage of chunk c, and how often that stage has been used before
    auto stage_of = [](int c) { return OUT ? c & 1 : c % 3; };
    auto turn_of = [](int c) { return OUT ? c >> 1 : c / 3; };

    if (warp == kElemWarps + 1) {
        if (lane == 0) {
            const int hq = head / p.heads_per_qk;
            const ChunkDecays* decays = reinterpret_cast<const ChunkDecays*>(p.decays) + ((long long)b * p.heads + head) * p.chunks + c_begin;
            for (int c = 0; c < nc; ++c) {
                const int stage = stage_of(c), y = b * p.seq + (c_begin + c) * kL;
                const uint32_t free_phase = (uint32_t)(turn_of(c) & 1) ^ 1u, dst = smem0 + (uint32_t)stage * stage_bytes;
                if (!mbar_wait_polling(smem_u32(&s.v_empty[stage]), free_phase, abort_flag)) break;
                uint32_t bar = smem_u32(&s.v_full[stage]);
                mbar_expect_tx(bar, kSegB + (uint32_t)sizeof(ChunkDecays));
                tma_load_3d(dst + bytes_q + 2 * kSegB, &tmV, slice * kPT, head, y, bar);
                bulk_load(smem_u32(&s.d[stage]), decays + c, (uint32_t)sizeof(ChunkDecays), bar);
                if (!mbar_wait_polling(smem_u32(&s.qk_empty[stage]), free_phase, abort_flag)) break;
                bar = smem_u32(&s.qk_full[stage]);
                mbar_expect_tx(bar, bytes_q + 2 * kSegB);
                if (OUT)
                    for (int k = 0; k < p.segq; ++k) tma_load_3d(dst + (uint32_t)k * kSegB, &tmQ, k * 64, hq, y, bar);
                for (int k = 0; k < 2; ++k) tma_load_3d(dst + bytes_q + (uint32_t)k * kSegB, &tmK, k * 64, hq, y, bar);
            }
        }
    } else if (warp == kElemWarps || warp == kElemWarps + 3) {
        // the whole warp walks along, lane 0 issues
        const bool lead = lane == 0;
        const uint32_t idesc_qk = idesc_bf16(kL, kL), idesc_v = idesc_bf16(kL, kPT, true), idesc_s = idesc_bf16(kL, 2 * kPT, true);
        const uint32_t idesc_d = idesc_s | (1u << 15);                  // both operands with their tokens as rows
        const int steps = (p.n + 15) / 16;                              // of 16 state rows
        auto wait = [&](uint64_t* bar, int phase) {
            const bool ok = mbar_wait_polling(smem_u32(bar), (uint32_t)(phase & 1), abort_flag);
            tc_fence_after();
            return ok;
        };
        bool ok = true;
        if (warp == kElemWarps) {
            for (int c = 0; OUT && c <= nc && ok; ++c) {
                if (c > 0) {                                            // what the previous chunk's own tokens give
                    if (!(ok = wait(&s.v_full[(c - 1) & 1], (c - 1) >> 1) && wait(&s.p_full, c - 1))) break;
                    const uint64_t vd = smem_desc_mn_sw128(smem0 + (uint32_t)((c - 1) & 1) * stage_bytes + bytes_q + 2 * kSegB, kSegB);
                    if (lead) {
#pragma unroll
                        for (int k = 0; k < kL / 16; ++k)
                            umma_bf16_ts(tmem + kColO, tmem + kColP + (uint32_t)(k * 8), vd + (uint64_t)(k * 128), idesc_v, k ? 1u : 0u);
                        umma_commit(smem_u32(&s.o_full));
                    }
                }
                if (c == nc || !(ok = wait(&s.qk_full[c & 1], c >> 1))) break;
                const uint32_t q = smem0 + (uint32_t)(c & 1) * stage_bytes;
                const uint64_t ad = smem_desc_sw128(q), bd = smem_desc_sw128(q + bytes_q);
                if (lead) {                                             // the scores before have been read: p_full
#pragma unroll
                    for (int k = 0; k < 8; ++k)
                        if (k < steps) {
                            const uint64_t at = (uint64_t)((k >> 2) * (kSegB >> 4) + (k & 3) * 2);
                            umma_bf16(tmem + kColS, ad + at, bd + at, idesc_qk, k ? 1u : 0u);
                        }
                    umma_commit(smem_u32(&s.s_full));
                }
            }
        } else {
            for (int c = 0; c < nc; ++c) {
                const uint32_t q = smem0 + (uint32_t)stage_of(c) * stage_bytes;
                if (!wait(&s.qk_full[stage_of(c)], turn_of(c)) || !wait(&s.vp_full[c & 1], c >> 1)) break;
                const uint64_t vd = smem_desc_mn_sw128(smem_u32(vp) + (uint32_t)(c & 1) * vp_step, kSegB);
                const uint32_t d = tmem + kColD - (OUT ? 0u : (uint32_t)(c & 1) * 128u);
                const uint64_t kd = smem_desc_mn_sw128(q + bytes_q, kSegB);
                if (lead) {
#pragma unroll
                    for (int k = 0; k < kL / 16; ++k)
                        umma_bf16(d, kd + (uint64_t)(k * 128), vd + (uint64_t)(k * 128), idesc_d, k ? 1u : 0u);
                    umma_commit(smem_u32(&s.ds_full[c & 1]));
                    if (!OUT) {
                        umma_commit(smem_u32(&s.qk_empty[stage_of(c)]));
                        umma_commit(smem_u32(&s.v_empty[stage_of(c)]));
                    }
                }
                if (!OUT) continue;
                // the state's tile is published after the previous chunk's outputs have been read
                if (!wait(&s.st_full, c)) break;
                if (lead) {
#pragma unroll
                    for (int k = 0; k < 8; ++k)
                        if (k < steps)
                            umma_bf16(tmem + kColQS, smem_desc_sw128(q + (uint32_t)(k >> 2) * kSegB + (uint32_t)(k & 3) * 32u),
                                      smem_desc_mn_sw128(smem_u32(st) + (uint32_t)k * 2048u, bytes_s), idesc_s, k ? 1u : 0u);
                    umma_commit(smem_u32(&s.o_full));
                }
            }
        }
    } else if (warp == kElemWarps + 2) {
        if (OUT && lane == 0) {
            for (int c = 0; c < nc; ++c) {
                if (!mbar_wait_polling(smem_u32(&s.out_full[c & 1]), (uint32_t)((c >> 1) & 1), abort_flag)) break;
                const uint32_t tile = smem0 + (uint32_t)(c & 1) * stage_bytes;
                tma_store_4d(&tmO, slice * kPT, head, (c_begin + c) * kL, b, tile);
                bulk_commit();
                bulk_wait_read();
                mbar_arrive(smem_u32(&s.qk_empty[c & 1]));
            }
            bulk_wait_all();
        }
    } else {
        const int part = warp >> 2, quarter = warp & 3, row = quarter * 32 + lane;
        const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
        const int col0 = slice * kPT + part * 16;
        // this thread's 16 values of the state in global memory
        auto state_at = [&](bool own) {
            const long long sh = ((long long)b * p.heads + head) * p.segments + seg;
            return own ? p.state + ((slot * p.heads + head) * p.n + row) * p.p + col0 : p.seg_state + (sh * p.n + row) * p.p + col0;
        };
        float S[16];
        {
            const bool segmented = p.segments > 1, read = OUT && row < p.n && (segmented || p.start[b] != 0);
            const float* from = state_at(!segmented);
#pragma unroll
            for (int i = 0; i < 16; i += 8) {
                float v[8] = {};
                if (read && col0 + i < p.p) load8(from + i, v);
#pragma unroll
                for (int k = 0; k < 8; ++k) S[i + k] = v[k];
            }
        }
        auto arrive = [&](uint64_t* bar) {
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(bar));
        };
        auto publish = [&](uint64_t* bar) {                              // shared-memory tiles for the tensor core or TMA
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            arrive(bar);
        };
        auto wait = [&](uint64_t* bar, int phase) { return mbar_wait_polling(smem_u32(bar), (uint32_t)(phase & 1), abort_flag); };
        auto value_tile = [&](int c) { return base + (uint32_t)stage_of(c) * stage_bytes + bytes_q + 2 * kSegB; };
        // values scaled by what is left of them at the chunk's end
        float l_row = 0.f, l_end = 0.f, l_row_next, l_end_next;          // a stage may be refilled once its values are scaled
        auto scale_values = [&](int c) {
            float v[16];
            load_row(value_tile(c), row, part, v);
            l_row_next = s.d[stage_of(c)].l[row];
            l_end_next = s.d[stage_of(c)].l[kL - 1];
            const float f = exp2_fast(l_end_next - s.d[stage_of(c)].lw[row]);
#pragma unroll
            for (int i = 0; i < 16; ++i) v[i] *= f;
            uint8_t* dst = vp + (uint32_t)(c & 1) * vp_step;
            store_split(dst, dst + kSegB, row, part, v);
            publish(&s.vp_full[c & 1]);
        };
        if (OUT) {
            if (row < rows_s) store_split(st, st + bytes_s, row, part, S);
            publish(&s.st_full);
        }
        const float skip = p.skip ? p.skip[head] : 0.f;
        float total = 0.f;
        bool ok = wait(&s.v_full[0], 0);
        if (ok) scale_values(0);
        for (int c = 0; c < nc && ok; ++c) {
            const int stage = c & 1;
            l_row = l_row_next;
            l_end = l_end_next;
            if (OUT) {
                // what is left at each row of each column's weight, half of it while the scores are on their way
                const float f = part < quarter ? exp2_fast(l_row - s.d[stage].l[part * 32 + 31]) : 0.f;
                float g[16];
                auto factors = [&](int q) {
                    if (part < quarter) {
#pragma unroll
                        for (int i = 0; i < 16; i += 4) {
                            const float4 x = *reinterpret_cast<const float4*>(&s.d[stage].col[part * 32 + q * 16 + i]);
                            g[i] = f * x.x; g[i + 1] = f * x.y; g[i + 2] = f * x.z; g[i + 3] = f * x.w;
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; i += 4) {
                            const float4 x = *reinterpret_cast<const float4*>(&s.d[stage].lw[part * 32 + q * 16 + i]);
                            const int e = q * 16 + i;
                            g[i] = e <= lane ? exp2_fast(l_row - x.x) : 0.f;
                            g[i + 1] = e + 1 <= lane ? exp2_fast(l_row - x.y) : 0.f;
                            g[i + 2] = e + 2 <= lane ? exp2_fast(l_row - x.z) : 0.f;
                            g[i + 3] = e + 3 <= lane ? exp2_fast(l_row - x.w) : 0.f;
                        }
                    }
                };
                if (part <= quarter) factors(0);
                if (!(ok = wait(&s.s_full, c))) break;
                tc_fence_after();
                uint32_t w[16];
                if (part > quarter) {                                    // the block of columns lies behind every row
#pragma unroll
                    for (int i = 0; i < 16; ++i) w[i] = 0u;
                } else {
                    const uint32_t ts = tmem + kColS + lanes + (uint32_t)part * 32u;
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        float v[16];
                        tmem_ld16f(ts + (uint32_t)(q * 16), v);
                        if (q) factors(1);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 8; ++i) w[q * 8 + i] = pack_bf16(v[2 * i] * g[2 * i], v[2 * i + 1] * g[2 * i + 1]);
                    }
                }
                tmem_st16(tmem + kColP + lanes + (uint32_t)part * 16u, w);
                tmem_st_wait();
                arrive(&s.p_full);
            }
            auto next_values = [&] { return c + 1 == nc || wait(&s.v_full[stage_of(c + 1)], turn_of(c + 1)); };
            if (!OUT) {
                if (!(ok = next_values())) break;
                if (c + 1 < nc) scale_values(c + 1);
            }
            // the state behind the chunk
            if (!(ok = wait(&s.ds_full[stage], c >> 1))) break;
            tc_fence_after();
            {
                const uint32_t td = tmem + kColD - (OUT ? 0u : (uint32_t)stage * 128u) + lanes + (uint32_t)part * 16u;
                float d[16], r[16];
                tmem_ld16f(td, d);
                tmem_ld16f(td + 64u, r);
                const float f = exp2_fast(l_end);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i) S[i] = fmaf(f, S[i], d[i] + r[i]);
                total += l_end;
            }
            if (OUT && c + 1 < nc) {
                if (!(ok = next_values())) break;
                scale_values(c + 1);
            }
            if (OUT) {
                if (!(ok = wait(&s.o_full, c))) break;
                tc_fence_after();
                float o[16], x[16];
                tmem_ld16f(tmem + kColQS + lanes + (uint32_t)part * 16u, o);
                tmem_ld16f(tmem + kColQS + lanes + 64u + (uint32_t)part * 16u, x);
                const float f = exp2_fast(l_row);
                uint8_t* tile = base + (uint32_t)stage * stage_bytes;
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i) o[i] = f * (o[i] + x[i]);
                tmem_ld16f(tmem + kColO + lanes + (uint32_t)part * 16u, x);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i) o[i] += x[i];
                if (p.skip) {
                    load_row(value_tile(c), row, part, x);
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = fmaf(skip, x[i], o[i]);
                }
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&s.v_empty[stage]));
#pragma unroll
                for (int q = 0; q < 2; ++q)
                    *reinterpret_cast<uint4*>(tile + at_piece(row, part * 2 + q)) =
                        make_uint4(pack_bf16(o[q * 8], o[q * 8 + 1]), pack_bf16(o[q * 8 + 2], o[q * 8 + 3]),
                                   pack_bf16(o[q * 8 + 4], o[q * 8 + 5]), pack_bf16(o[q * 8 + 6], o[q * 8 + 7]));
                // the state's tile has been read
                if (c + 1 < nc && row < rows_s) store_split(st, st + bytes_s, row, part, S);
                publish(&s.out_full[stage]);
                if (lane == 0 && c + 1 < nc) mbar_arrive(smem_u32(&s.st_full));
            }
        }
        if ((!OUT || seg == p.segments - 1) && row < p.n) {
            float* to = state_at(OUT);
#pragma unroll
            for (int i = 0; i < 16; i += 8)
                if (col0 + i < p.p) {
                    float y[8];
#pragma unroll
                    for (int k = 0; k < 8; ++k) y[k] = S[i + k];
                    store8(to + i, y);
                }
        }
        if (!OUT && slice == 0 && threadIdx.x == 0) p.seg_decay[((long long)b * p.heads + head) * p.segments + seg] = total;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == kElemWarps) tmem_dealloc(tmem, 512);
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
    constexpr int B = 4;                           // segments whose states are loaded together
    for (int s0 = 0; s0 < p.segments; s0 += B) {
        float4 mine[B];
        float f[B];
#pragma unroll
        for (int k = 0; k < B; ++k)
            if (s0 + k < p.segments) {
                mine[k] = *reinterpret_cast<const float4*>(p.seg_state + (sh + s0 + k) * size + i);
                f[k] = exp2_fast(p.seg_decay[sh + s0 + k]);
            }
#pragma unroll
        for (int k = 0; k < B; ++k)
            if (s0 + k < p.segments) {
                *reinterpret_cast<float4*>(p.seg_state + (sh + s0 + k) * size + i) = run;
                run.x = fmaf(f[k], run.x, mine[k].x); run.y = fmaf(f[k], run.y, mine[k].y);
                run.z = fmaf(f[k], run.z, mine[k].z); run.w = fmaf(f[k], run.w, mine[k].w);
            }
    }
}

size_t scan_smem(int n, bool out)
{
    const size_t segq = (size_t)(n + 63) / 64;
    const size_t tiles = out ? 2 * (segq + 3) * kSegB + 2 * kSegB + 2 * segq * 64 * 128 : 3 * 3 * kSegB + 4 * kSegB;
    const size_t bytes = tiles + (out ? sizeof(ScanTcShared<2>) : sizeof(ScanTcShared<3>)) + 64;
    return bytes + 1024 < kScanSmemAll ? bytes + 1024 : kScanSmemAll;
}

long long scan_decay_floats(const zkfp_scan_args& a)
{
    return a.batch * a.heads * ((a.seq + kL - 1) / kL) * (long long)(sizeof(ChunkDecays) / sizeof(float));
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
    return scan_decay_floats(a) + (s > 1 ? a.batch * a.heads * s * ((long long)a.n * a.p + 1) : 0);
}

int launch_scan_tc(const zkfp_scan_args& a, cudaStream_t st)
{
    ScanTcParams p;
    p.decay = a.decay; p.step = a.step; p.step_bias = a.step_bias; p.skip = a.skip; p.state = a.state;
    p.start = a.start; p.slots = a.slots; p.step_tok = a.step_tok;
    p.n_slots = a.n_slots; p.seq = (int)a.seq; p.heads = (int)a.heads; p.heads_per_qk = a.heads_per_qk; p.n = a.n; p.p = a.p;
    p.segq = (a.n + 63) / 64;
    p.chunks = (p.seq + kL - 1) / kL;
    p.segments = scan_segments(a);
    p.chunks_per_segment = (p.chunks + p.segments - 1) / p.segments;
    if (!a.scratch || (uintptr_t)a.scratch & 15) return ZKDS_ERR_ARG;
    p.decays = a.scratch;
    p.seg_state = a.scratch + scan_decay_floats(a);
    p.seg_decay = p.segments > 1 ? p.seg_state + a.batch * a.heads * p.segments * (long long)a.n * a.p : nullptr;
    p.k_scale = a.k_scale;
    p.error_flag = fp_error_flag();
    if (!p.error_flag) return ZKDS_ERR_WORKSPACE;
    const uint64_t rows = (uint64_t)(a.batch * a.seq), hqk = (uint64_t)(a.heads / a.heads_per_qk);
    const uint64_t dqk[3] = {(uint64_t)a.n, hqk, rows}, dv[3] = {(uint64_t)a.p, (uint64_t)a.heads, rows};
    const uint64_t sq[2] = {(uint64_t)a.qk_head * 2, (uint64_t)a.q_tok * 2}, sk[2] = {(uint64_t)a.qk_head * 2, (uint64_t)a.k_tok * 2};
    const uint64_t sv[2] = {(uint64_t)a.v_head * 2, (uint64_t)a.v_tok * 2};
    const uint32_t box[3] = {64, 1, kL};
    // the sequence is a dimension of its own, so that a last chunk's rows behind its end are not stored
    const uint64_t dout[4] = {(uint64_t)a.p, (uint64_t)a.heads, (uint64_t)a.seq, (uint64_t)a.batch};
    const uint64_t so[3] = {(uint64_t)a.o_head * 2, (uint64_t)a.o_tok * 2, (uint64_t)(a.seq * a.o_tok) * 2};
    const uint32_t box_o[4] = {64, 1, kL, 1};
    CUtensorMap q, k, v, o;
    if (!fp_tensor_map(&q, a.q, 3, dqk, sq, box) || !fp_tensor_map(&k, a.k, 3, dqk, sk, box) || !fp_tensor_map(&v, a.v, 3, dv, sv, box) ||
        !fp_tensor_map(&o, a.out, 4, dout, so, box_o))
        return ZKDS_ERR_UNSUPPORTED;
    for (int i = 0; i < 2; ++i) p.smem_bytes[i] = (uint32_t)scan_smem(a.n, i);
    const dim3 grid((unsigned)((a.p + kPT - 1) / kPT), (unsigned)a.heads, (unsigned)(a.batch * p.segments));
    if (grid.z > 65535u) return ZKDS_ERR_UNSUPPORTED;
    scan_decay_kernel<<<dim3((unsigned)p.chunks, (unsigned)((a.heads + 31) / 32), (unsigned)a.batch), 256, 0, st>>>(p);
    int rc = fp_launched();
    if (rc != ZKDS_OK) return rc;
    if (p.segments > 1) {
        ZKDS_CUDA(cudaFuncSetAttribute(scan_chunk_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kScanSmemAll));
        scan_chunk_kernel<false><<<grid, kScanThreads, p.smem_bytes[0], st>>>(q, k, v, o, p);
        rc = fp_launched();
        if (rc != ZKDS_OK) return rc;
        scan_segments_kernel<<<dim3((unsigned)((a.n * a.p + 1023) / 1024), (unsigned)a.heads, (unsigned)a.batch), 256, 0, st>>>(p);
        rc = fp_launched();
        if (rc != ZKDS_OK) return rc;
    }
    ZKDS_CUDA(cudaFuncSetAttribute(scan_chunk_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kScanSmemAll));
    scan_chunk_kernel<true><<<grid, kScanThreads, p.smem_bytes[1], st>>>(q, k, v, o, p);
    return fp_launched();
}

}  // namespace zkds
