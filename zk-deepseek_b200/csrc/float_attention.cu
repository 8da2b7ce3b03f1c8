// Windowed softmax attention on the tensor cores, bfloat16 operands, 32-bit scores, weights and sums.
//
// attention_expanded_kernel (prefill): per-head keys [k1 | k2] and values.  A CTA owns one head and two tiles of 128
// query tokens; keys come in tiles of 128.  Tensor memory holds both score tiles and both output tiles; the bfloat16
// weights overwrite the scores they came from and feed the second product from tensor memory.  While one query tile is
// in its softmax the tensor core works for the other.  Keys come through a ring of 64-column segments (16 KB), so that
// the next tile starts to load as soon as the first segment of the current one has been used; values through whole
// tiles, two where they fit.
//   warp 0      TMA loads          warp 1      MMA issue
//   warps 2-9   softmax, tile 0    warps 10-17 softmax, tile 1: two threads share a query row, half of the columns each
// The running maximum only replaces the one in use when it has grown by more than 2^8; the output tile is then
// rescaled in place.  A commit covers every MMA issued before it, so "scores ready" also says that the output tile is
// free to be rescaled.
#include <cuda.h>

#include "float_common.cuh"
#include "tcgen05.cuh"

namespace zkds {

bool fp_tensor_map(CUtensorMap* map, const void* base, int rank, const uint64_t* dims, const uint64_t* strides_bytes,
                   const uint32_t* box);

namespace {

constexpr int kTile = 128;                     // query rows and keys per tile
constexpr uint32_t kSeg = kTile * 128;         // bytes of 128 rows x 64 bfloat16
constexpr int kThreadsAttn = 576;
constexpr int kMaxKeySlots = 8;
constexpr int kHeadGroup = 32;
constexpr size_t kSmemMax = 226 * 1024, kSmemAll = 227 * 1024;

__device__ __forceinline__ float exp2_approx(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct ExpandedParams {
    bf16* out;
    const bf16* gate;
    const int* start;
    long long o_head, o_tok, gate_tok, gate_head;
    float out_scale;
    int seq, heads, heads_per_kv, base, window;
    int d1, d2, dv, seg1, seg2, segv;          // segments of 64 columns
    int k_slots, v_stages;                     // ring of key segments, value tiles
    float scale_log2;                          // scale * log2(e)
    uint32_t smem_bytes;
    int* error_flag;
};

struct ExpandedShared {
    uint64_t q_full, k_full[kMaxKeySlots], k_empty[kMaxKeySlots], v_full[2], v_empty[2], s_full[2], p_full[2], o_full[2];
    float row_max[2][2][kTile];            // [query tile][column half][row]; at the end the row sums
    uint32_t tmem;
    int abort;
};

// key tiles of one block of query tiles: tile j covers positions lo + 128 j ..; tile g is active for first[g] .. last[g]
struct KeyTiles {
    int lo, n, first[2], last[2];
};

__device__ __forceinline__ KeyTiles key_tiles(const ExpandedParams& p, int t0, int start)
{
    KeyTiles k;
    const int lo0 = p.window > 0 ? start + t0 - p.window + 1 : 0;
    k.lo = lo0 > p.base ? lo0 : p.base;
    k.n = 0;
#pragma unroll
    for (int g = 0; g < 2; ++g) {
        const int r0 = t0 + g * kTile;
        if (r0 >= p.seq) { k.first[g] = 1; k.last[g] = 0; continue; }
        const int r1 = min(r0 + kTile, p.seq) - 1;
        const int lo = p.window > 0 ? max(start + r0 - p.window + 1, k.lo) : k.lo;
        k.first[g] = (lo - k.lo) / kTile;
        k.last[g] = (start + r1 - k.lo) / kTile;
        k.n = max(k.n, k.last[g] + 1);
    }
    return k;
}

__global__ void __launch_bounds__(kThreadsAttn, 1)
attention_expanded_kernel(const __grid_constant__ CUtensorMap tmQ1, const __grid_constant__ CUtensorMap tmQ2,
                          const __grid_constant__ CUtensorMap tmK1, const __grid_constant__ CUtensorMap tmK2,
                          const __grid_constant__ CUtensorMap tmV, const ExpandedParams p)
{
    // the tiles of the largest shapes leave less than a kilobyte, so the bookkeeping lies behind them in the same block
    extern __shared__ __align__(1024) uint8_t raw[];
    uint8_t* base = (uint8_t*)(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    const uint32_t tile_bytes = (uint32_t)(2 * (p.seg1 + p.seg2) + p.k_slots + p.v_stages * p.segv) * kSeg;
    if (base + tile_bytes + sizeof(ExpandedShared) > raw + p.smem_bytes) {      // not the alignment the host counted on
        if (threadIdx.x == 0) *(volatile int*)p.error_flag = 1;
        return;
    }
    ExpandedShared& s = *reinterpret_cast<ExpandedShared*>(base + tile_bytes);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // the longest blocks of a group of heads first: short tails, keys and values of the group stay in L2
    const int blocks = (p.seq + 2 * kTile - 1) / (2 * kTile), group0 = (int)blockIdx.x / (blocks * kHeadGroup) * kHeadGroup;
    const int in_group = (int)blockIdx.x - group0 * blocks, width = min(kHeadGroup, p.heads - group0);
    const int head = group0 + in_group % width, t0 = (blocks - 1 - in_group / width) * 2 * kTile;
    const int kv_head = head / p.heads_per_kv;
    const int start = p.start[0];
    const KeyTiles kt = key_tiles(p, t0, start);
    const int segq = p.seg1 + p.seg2;
    const uint32_t sQ = smem_u32(base), bytesQ = (uint32_t)segq * kSeg;
    const uint32_t sK = sQ + 2 * bytesQ, sV = sK + (uint32_t)p.k_slots * kSeg, bytesV = (uint32_t)p.segv * kSeg;
    volatile int* abort_flag = &s.abort;

    if (threadIdx.x == 0) {
        s.abort = 0;
        mbar_init(smem_u32(&s.q_full), 1);
        for (int i = 0; i < kMaxKeySlots; ++i) {
            mbar_init(smem_u32(&s.k_full[i]), 1);
            mbar_init(smem_u32(&s.k_empty[i]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&s.v_full[i]), 1);
            mbar_init(smem_u32(&s.v_empty[i]), 1);
        }
        for (int g = 0; g < 2; ++g) {
            mbar_init(smem_u32(&s.s_full[g]), 1);
            mbar_init(smem_u32(&s.p_full[g]), 8);
            mbar_init(smem_u32(&s.o_full[g]), 1);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    if (warp == 1) tmem_alloc(smem_u32(&s.tmem), 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s.tmem;

    if (warp == 0) {
        if (lane == 0) {
            const int tiles_q = t0 + kTile < p.seq ? 2 : 1;
            mbar_expect_tx(smem_u32(&s.q_full), (uint32_t)tiles_q * bytesQ);
            for (int g = 0; g < tiles_q; ++g) {
                for (int c = 0; c < p.seg1; ++c)
                    tma_load_3d(sQ + g * bytesQ + c * kSeg, &tmQ1, c * 64, head, t0 + g * kTile, smem_u32(&s.q_full));
                for (int c = 0; c < p.seg2; ++c)
                    tma_load_3d(sQ + g * bytesQ + (p.seg1 + c) * kSeg, &tmQ2, c * 64, head, t0 + g * kTile,
                                smem_u32(&s.q_full));
            }
            int ks = 0, vs = 0;
            uint32_t kp = 0, vp = 0;
            bool ok = true;
            for (int j = 0; j < kt.n && ok; ++j) {
                const int y = kt.lo - p.base + j * kTile;
                for (int c = 0; c < segq; ++c) {
                    if (!(ok = mbar_wait(smem_u32(&s.k_empty[ks]), kp ^ 1u, abort_flag))) break;
                    const uint32_t bar = smem_u32(&s.k_full[ks]), dst = sK + (uint32_t)ks * kSeg;
                    mbar_expect_tx(bar, kSeg);
                    if (c < p.seg1) tma_load_3d(dst, &tmK1, c * 64, kv_head, y, bar);
                    else tma_load_2d(dst, &tmK2, (c - p.seg1) * 64, y, bar);
                    if (++ks == p.k_slots) { ks = 0; kp ^= 1u; }
                }
                if (!ok || !mbar_wait(smem_u32(&s.v_empty[vs]), vp ^ 1u, abort_flag)) break;
                const uint32_t bar = smem_u32(&s.v_full[vs]), dst = sV + (uint32_t)vs * bytesV;
                mbar_expect_tx(bar, bytesV);
                for (int c = 0; c < p.segv; ++c) tma_load_3d(dst + c * kSeg, &tmV, c * 64, kv_head, y, bar);
                if (++vs == p.v_stages) { vs = 0; vp ^= 1u; }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = idesc_bf16(kTile, kTile), idesc_o = idesc_bf16(kTile, (p.dv + 15) & ~15, true);
            uint32_t pp[2] = {0, 0};
            int ks = 0, vs = 0;                           // ring slot of the key tile's first segment, value stage
            uint32_t kp = 0, vp = 0;
            // the score product of query tile g with the key tile at (ks, kp); `load` waits for its segments,
            // `release` hands each back after use
            auto scores = [&](int g, bool use, bool load, bool release) {
                const uint32_t a = sQ + (uint32_t)g * bytesQ, d = tmem + (uint32_t)g * kTile;
                int slot = ks;
                uint32_t phase = kp;
                for (int c = 0; c < segq; ++c) {
                    if (load) {
                        if (!mbar_wait(smem_u32(&s.k_full[slot]), phase, abort_flag)) return false;
                        tc_fence_after();
                    }
                    if (use) {
                        const int cols = c < p.seg1 ? p.d1 - c * 64 : p.d2 - (c - p.seg1) * 64;
                        const uint64_t ad = smem_desc_sw128(a + (uint32_t)c * kSeg), bd = smem_desc_sw128(sK + (uint32_t)slot * kSeg);
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            if (k * 16 < cols) umma_bf16(d, ad + (uint64_t)(k * 2), bd + (uint64_t)(k * 2), idesc_s, (c | k) ? 1u : 0u);
                    }
                    if (release) umma_commit(smem_u32(&s.k_empty[slot]));
                    if (++slot == p.k_slots) { slot = 0; phase ^= 1u; }
                }
                if (use) umma_commit(smem_u32(&s.s_full[g]));
                if (release) { ks = slot; kp = phase; }
                return true;
            };
            auto active = [&](int g, int j) {
                return g ? j >= kt.first[1] && j <= kt.last[1] : j >= kt.first[0] && j <= kt.last[0];
            };
            bool ok = mbar_wait(smem_u32(&s.q_full), 0, abort_flag);
            for (int j = -1; j < kt.n && ok; ++j) {
                if (j >= 0 && !(ok = mbar_wait(smem_u32(&s.v_full[vs]), vp, abort_flag))) break;
                for (int g = 0; g < 2 && ok; ++g) {
                    if (j >= 0 && active(g, j)) {
                        if (!(ok = mbar_wait(smem_u32(&s.p_full[g]), pp[g], abort_flag))) break;
                        pp[g] ^= 1u;
                        tc_fence_after();
                        const uint32_t a = tmem + (uint32_t)g * kTile, d = tmem + 256u + (uint32_t)g * kTile;
                        const uint64_t vd = smem_desc_mn_sw128(sV + (uint32_t)vs * bytesV, kSeg);
                        const bool opens = j == (g ? kt.first[1] : kt.first[0]);
#pragma unroll
                        for (int k = 0; k < kTile / 16; ++k)
                            umma_bf16_ts(d, a + (uint32_t)k * 8u, vd + (uint64_t)(k * 128), idesc_o, (!opens || k) ? 1u : 0u);
                        if (j == (g ? kt.last[1] : kt.last[0])) umma_commit(smem_u32(&s.o_full[g]));
                    }
                    if (j >= 0 && g == 1) umma_commit(smem_u32(&s.v_empty[vs]));
                    // every segment is waited for once and handed back once, also when no query tile uses it
                    if (j + 1 < kt.n) ok = scores(g, active(g, j + 1), g == 0, g == 1);
                }
                if (!ok) break;
                if (j >= 0 && ++vs == p.v_stages) { vs = 0; vp ^= 1u; }
            }
        }
    } else {
        const int g = (warp - 2) >> 3, half = ((warp - 2) >> 2) & 1, quarter = warp & 3, row = quarter * 32 + lane;
        const int t = t0 + g * kTile + row, pos = start + t, c0 = half * 64;
        const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
        const uint32_t tS = tmem + (uint32_t)g * kTile + lanes, tO = tmem + 256u + (uint32_t)g * kTile + lanes;
        const int o_begin = half * ((p.dv / 2 + 31) & ~31), o_end = half ? p.dv : min(p.dv, (p.dv / 2 + 31) & ~31);
        const int first_tile = g ? kt.first[1] : kt.first[0], last_tile = g ? kt.last[1] : kt.last[0];
        auto pair_sync = [&] { asm volatile("bar.sync %0, 64;" ::"r"(1 + g * 4 + quarter) : "memory"); };
        float m_used = -INFINITY, l = 0.f;
        uint32_t sp = 0;
        bool ok = true;
        for (int j = first_tile; j <= last_tile; ++j) {
            ok = mbar_wait(smem_u32(&s.s_full[g]), sp, abort_flag);
            sp ^= 1u;
            tc_fence_after();
            float v[2][32];
            tmem_ld32(tS + (uint32_t)c0, v[0]);
            tmem_ld32(tS + (uint32_t)c0 + 32u, v[1]);
            // visible columns of this row: c_lo .. c_hi
            const int c_hi = pos - (kt.lo + j * kTile), c_lo = p.window > 0 ? c_hi - p.window + 1 : -1;
            const bool masked = __any_sync(0xffffffffu, c_hi < kTile - 1 || c_lo > 0);
            tmem_ld_wait();
            if (masked) {
#pragma unroll
                for (int c = 0; c < 64; ++c)
                    if (c0 + c < c_lo || c0 + c > c_hi) v[c >> 5][c & 31] = -INFINITY;
            }
            float mp[8];                              // independent chains
#pragma unroll
            for (int i = 0; i < 8; ++i) mp[i] = v[0][i];
#pragma unroll
            for (int c = 8; c < 64; ++c) mp[c & 7] = fmaxf(mp[c & 7], v[c >> 5][c & 31]);
            const float mine = fmaxf(fmaxf(fmaxf(mp[0], mp[1]), fmaxf(mp[2], mp[3])),
                                     fmaxf(fmaxf(mp[4], mp[5]), fmaxf(mp[6], mp[7])));
            s.row_max[g][half][row] = mine;
            // also: both threads of every row have read their scores before either overwrites any of them
            pair_sync();
            const float m_new = fmaxf(m_used, fmaxf(mine, s.row_max[g][half ^ 1][row]) * p.scale_log2);
            if (j == first_tile) {
                m_used = m_new;
            } else if (__any_sync(0xffffffffu, m_new > m_used + 8.0f)) {     // the same rows, so the same decision in both warps
                const float f = m_used == -INFINITY ? 0.f : exp2_approx(m_used - m_new);
                for (int c = o_begin; c < o_end; c += 8) {
                    int32_t o[8];
                    tmem_ld8(tO + (uint32_t)c, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 8; ++i) o[i] = __float_as_int(__int_as_float(o[i]) * f);
                    tmem_st8(tO + (uint32_t)c, o);
                }
                l *= f;
                m_used = m_new;
            }
            const float m_sub = m_used == -INFINITY ? 0.f : m_used;
            float lp[4] = {};
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                uint32_t w[16];
#pragma unroll
                for (int i = 0; i < 32; ++i) v[q][i] = exp2_approx(fmaf(v[q][i], p.scale_log2, -m_sub));
#pragma unroll
                for (int i = 0; i < 32; ++i) lp[i & 3] += v[q][i];
#pragma unroll
                for (int i = 0; i < 16; ++i) w[i] = pack_bf16(v[q][2 * i], v[q][2 * i + 1]);
                tmem_st16(tS + (uint32_t)(half * 32 + q * 16), w);
            }
            l += (lp[0] + lp[1]) + (lp[2] + lp[3]);
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s.p_full[g]));
        }
        if (first_tile <= last_tile) {
            pair_sync();                              // the last maxima have been read
            s.row_max[g][half][row] = l;
            pair_sync();
            l += s.row_max[g][half ^ 1][row];
        }
        if (ok && first_tile <= last_tile && mbar_wait(smem_u32(&s.o_full[g]), 0, abort_flag)) {
            tc_fence_after();
            const float r = 1.0f / l;
            bf16* o = p.out + (long long)t * p.o_tok + head * p.o_head;
            const bf16* gate = p.gate ? p.gate + (long long)t * p.gate_tok + head * p.gate_head : nullptr;
            for (int c = o_begin; c < o_end; c += 8) {
                int32_t x[8];
                tmem_ld8(tO + (uint32_t)c, x);
                tmem_ld_wait();
                if (t < p.seq) {
                    float w[8];
#pragma unroll
                    for (int k = 0; k < 8; ++k) w[k] = __int_as_float(x[k]) * r;
                    if (gate) {
                        float z[8];
                        load8(gate + c, z);
#pragma unroll
                        for (int k = 0; k < 8; ++k) w[k] *= sigmoid_f(z[k]) * p.out_scale;
                    }
                    store8(o + c, w);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 1) tmem_dealloc(tmem, 512);
    if (threadIdx.x == 0 && s.abort) *(volatile int*)p.error_flag = 1;
}

size_t expanded_smem(const zkfp_attention_args& a, int& k_slots, int& v_stages)
{
    const size_t segq = (size_t)(a.d1 + 63) / 64 + (a.d2 + 63) / 64, segv = (a.dv + 63) / 64;
    const size_t fixed = sizeof(ExpandedShared) + 512, segs = (kSmemAll - fixed) / kSeg;
    if (segq > (size_t)kMaxKeySlots || 3 * segq + segv > segs) return 0;
    v_stages = 3 * segq + 2 * segv <= segs ? 2 : 1;
    const size_t left = segs - 2 * segq - v_stages * segv;
    k_slots = (int)(left < (size_t)kMaxKeySlots ? left : (size_t)kMaxKeySlots);
    const size_t bytes = kSeg * (2 * segq + k_slots + v_stages * segv) + fixed;
    return bytes + 1024 < kSmemAll ? bytes + 1024 : kSmemAll;
}

}  // namespace

bool attention_prefill_tc_takes(const zkfp_attention_args& a)
{
    int ks, vs;
    return a.dtype == ZKFP_BF16 && !a.shared && a.batch == 1 && a.dv <= 128 && a.keys > 0 &&
           a.keys < 0x40000000 && a.seq < 0x40000000 && expanded_smem(a, ks, vs) > 0 &&
           !((a.q_head | a.k1_tok | a.k1_head | a.k2_tok | a.v_tok | a.v_head | a.o_head) & 7) &&
           !(((uintptr_t)a.q | (uintptr_t)a.k1 | (uintptr_t)a.k2 | (uintptr_t)a.v | (uintptr_t)a.out) & 15);
}

int launch_attention_prefill_tc(const zkfp_attention_args& a, cudaStream_t st)
{
    ExpandedParams p;
    p.out = (bf16*)a.out; p.start = a.start; p.o_head = a.o_head;
    p.o_tok = a.o_tok ? a.o_tok : a.heads * a.o_head;
    p.gate = (const bf16*)a.gate; p.gate_tok = a.gate_tok; p.gate_head = a.gate_head; p.out_scale = a.out_scale;
    p.heads_per_kv = a.heads_per_kv > 1 ? a.heads_per_kv : 1;
    p.seq = (int)a.seq; p.heads = (int)a.heads; p.base = (int)a.base; p.window = a.window;
    p.d1 = a.d1; p.d2 = a.d2; p.dv = a.dv;
    p.seg1 = (a.d1 + 63) / 64; p.seg2 = (a.d2 + 63) / 64; p.segv = (a.dv + 63) / 64;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.error_flag = fp_error_flag();
    if (!p.error_flag) return ZKDS_ERR_WORKSPACE;
    const size_t smem = expanded_smem(a, p.k_slots, p.v_stages);
    CUtensorMap q1, q2, k1, k2, v;
    const uint64_t H = (uint64_t)a.heads, S = (uint64_t)a.seq, N = (uint64_t)a.keys;
    const uint64_t qs[2] = {(uint64_t)a.q_head * 2, (uint64_t)a.q_head * 2 * H};
    const uint64_t ks[2] = {(uint64_t)a.k1_head * 2, (uint64_t)a.k1_tok * 2}, k2s[1] = {(uint64_t)a.k2_tok * 2};
    const uint64_t vs[2] = {(uint64_t)a.v_head * 2, (uint64_t)a.v_tok * 2};
    const uint64_t dq1[3] = {(uint64_t)a.d1, H, S}, dq2[3] = {(uint64_t)(a.d2 ? a.d2 : 8), H, S};
    const uint64_t G = H / (uint64_t)p.heads_per_kv;
    const uint64_t dk1[3] = {(uint64_t)a.d1, G, N}, dk2[2] = {(uint64_t)(a.d2 ? a.d2 : 8), N}, dv[3] = {(uint64_t)a.dv, G, N};
    const uint32_t b3[3] = {64, 1, kTile}, b2[2] = {64, kTile};
    const bf16* q = (const bf16*)a.q;
    if (!fp_tensor_map(&q1, q, 3, dq1, qs, b3) || !fp_tensor_map(&q2, a.d2 ? q + a.d1 : q, 3, dq2, qs, b3) ||
        !fp_tensor_map(&k1, a.k1, 3, dk1, ks, b3) || !fp_tensor_map(&k2, a.k2, 2, dk2, k2s, b2) ||
        !fp_tensor_map(&v, a.v, 3, dv, vs, b3))
        return ZKDS_ERR_UNSUPPORTED;
    ZKDS_CUDA(cudaFuncSetAttribute(attention_expanded_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemAll));
    // more than half the shared memory: one CTA per SM, so the tensor-memory allocation never waits
    const size_t want = smem < 120 * 1024 ? 120 * 1024 : smem;
    p.smem_bytes = (uint32_t)want;
    const long long ctas = (a.seq + 2 * kTile - 1) / (2 * kTile) * a.heads;
    if (ctas > 0x7fffffffll) return ZKDS_ERR_UNSUPPORTED;
    attention_expanded_kernel<<<(unsigned)ctas, kThreadsAttn, want, st>>>(q1, q2, k1, k2, v, p);
    return fp_launched();
}

// ---- attention over the latents (decode) -------------------------------------------------------------------------
// Rows are (token, head) pairs, all heads read the same keys, and the values are the latent part of the keys.  A CTA
// takes 128 rows and one chunk of 64 keys: scores, softmax of the chunk, weighted sum; partial results go to scratch
// and latent_combine_kernel merges the chunks.  The key tile in shared memory serves both products (keys x latent as
// the K-major operand of the scores and as the N-major operand of the sum), so the cache is read once.  The
// weights take the place of the queries in shared memory and the sums that of the scores in tensor memory.
namespace {

constexpr int kChunk = 64;
constexpr uint32_t kSegC = kChunk * 128;       // bytes of 64 keys x 64 columns

struct LatentParams {
    const int* start;
    const int* slots;
    float* part;               // [batch][row tile][chunk][c][128]
    float* ml;                 // [batch][row tile][chunk][2][128]: maximum (log2 units), sum
    int rows, heads, seq, window, c, r, segc, segr, chunks, row_tiles, keys;
    float scale_log2;
    int* error_flag;
};

struct LatentShared {
    uint64_t q_full, k_full, s_full, p_full, o_full;
    uint32_t tmem;
    int abort;
};

// first chunk (in units of kChunk positions) and number of chunks of a row tile
__device__ __forceinline__ void chunk_range(int start, int row0, int rows, int heads, int window, int& first, int& n)
{
    const int last_row = min(row0 + kTile, rows) - 1;
    const int lo = window > 0 ? max(start + row0 / heads - window + 1, 0) : 0;
    const int hi = start + last_row / heads;
    first = lo / kChunk;
    n = hi / kChunk - first + 1;
}

__global__ void __launch_bounds__(192, 1)
attention_latent_kernel(const __grid_constant__ CUtensorMap tmQ1, const __grid_constant__ CUtensorMap tmQ2,
                        const __grid_constant__ CUtensorMap tmK1, const __grid_constant__ CUtensorMap tmK2,
                        const LatentParams p)
{
    extern __shared__ uint8_t raw[];
    __shared__ LatentShared s;
    const int b = blockIdx.z, row0 = blockIdx.y * kTile, start = p.start[b];
    int first, n;
    chunk_range(start, row0, p.rows, p.heads, p.window, first, n);
    if (start < 0 || start + p.seq > p.keys || n > p.chunks) {        // not a step of this cache
        if (threadIdx.x == 0) *(volatile int*)p.error_flag = 1;
        return;
    }
    if ((int)blockIdx.x >= n) return;
    const int j0 = (first + (int)blockIdx.x) * kChunk;
    uint8_t* base = (uint8_t*)(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, seg = p.segc + p.segr;
    const uint32_t sQ = smem_u32(base), sK = sQ + (uint32_t)seg * kSeg;
    volatile int* abort_flag = &s.abort;
    if (threadIdx.x == 0) {
        s.abort = 0;
        mbar_init(smem_u32(&s.q_full), 1);
        mbar_init(smem_u32(&s.k_full), 1);
        mbar_init(smem_u32(&s.s_full), 1);
        mbar_init(smem_u32(&s.p_full), 4);
        mbar_init(smem_u32(&s.o_full), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    if (warp == 1) tmem_alloc(smem_u32(&s.tmem), 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s.tmem;

    if (warp == 0) {
        if (lane == 0) {
            const uint32_t kb = smem_u32(&s.k_full), qb = smem_u32(&s.q_full);
            const int y = b * p.rows + row0, slot = p.slots ? p.slots[b] : b;
            mbar_expect_tx(kb, (uint32_t)seg * kSegC);
            mbar_expect_tx(qb, (uint32_t)seg * kSeg);
            for (int c = 0; c < seg; ++c) {
                const bool lat = c < p.segc;
                const int x = (lat ? c : c - p.segc) * 64;
                tma_load_3d(sK + (uint32_t)c * kSegC, lat ? &tmK1 : &tmK2, x, j0, slot, kb);
                tma_load_2d(sQ + (uint32_t)c * kSeg, lat ? &tmQ1 : &tmQ2, x, y, qb);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            bool ok = mbar_wait(smem_u32(&s.q_full), 0, abort_flag) && mbar_wait(smem_u32(&s.k_full), 0, abort_flag);
            if (ok) {
                tc_fence_after();
                const uint32_t idesc = idesc_bf16(kTile, kChunk);
                const int steps1 = (p.c + 15) / 16, steps2 = (p.r + 15) / 16;
                for (int k = 0; k < steps1 + steps2; ++k) {
                    const int kk = k < steps1 ? k : p.segc * 4 + (k - steps1);
                    umma_bf16(tmem, smem_desc_sw128(sQ + (uint32_t)(kk >> 2) * kSeg + (uint32_t)(kk & 3) * 32u),
                              smem_desc_sw128(sK + (uint32_t)(kk >> 2) * kSegC + (uint32_t)(kk & 3) * 32u), idesc,
                              k ? 1u : 0u);
                }
                umma_commit(smem_u32(&s.s_full));
                ok = mbar_wait(smem_u32(&s.p_full), 0, abort_flag);
            }
            if (ok) {
                tc_fence_after();
                for (int n0 = 0; n0 < p.c; n0 += 256) {
                    const int w = (min(p.c - n0, 256) + 15) & ~15;
                    const uint32_t idesc = idesc_bf16(kTile, w, true);
#pragma unroll
                    for (int k = 0; k < kChunk / 16; ++k)
                        umma_bf16(tmem + (uint32_t)n0, smem_desc_sw128(sQ + (uint32_t)k * 32u),
                                  smem_desc_mn_sw128(sK + (uint32_t)(n0 / 64) * kSegC + (uint32_t)k * 2048u, kSegC), idesc,
                                  k ? 1u : 0u);
                }
                umma_commit(smem_u32(&s.o_full));
            }
        }
    } else {
        const int quarter = warp & 3, row = quarter * 32 + lane, rr = row0 + row;
        const uint32_t tq = tmem + ((uint32_t)(quarter * 32) << 16);
        const bool row_ok = rr < p.rows;
        const int c_hi = start + rr / p.heads - j0, c_lo = p.window > 0 ? c_hi - p.window + 1 : 0;
        const long long tile = ((long long)b * p.row_tiles + blockIdx.y) * p.chunks + blockIdx.x;
        if (mbar_wait(smem_u32(&s.s_full), 0, abort_flag)) {
            tc_fence_after();
            float v[2][32];
            tmem_ld32(tq, v[0]);
            tmem_ld32(tq + 32u, v[1]);
            tmem_ld_wait();
            float m = -INFINITY, l = 0.f;
#pragma unroll
            for (int i = 0; i < 64; ++i) {
                float& x = v[i >> 5][i & 31];
                x = row_ok && i >= c_lo && i <= c_hi ? x * p.scale_log2 : -INFINITY;
                m = fmaxf(m, x);
            }
            const float m_sub = m == -INFINITY ? 0.f : m;
#pragma unroll
            for (int i = 0; i < 64; ++i) {
                float& x = v[i >> 5][i & 31];
                x = exp2_approx(x - m_sub);
                l += x;
            }
            // 128 bytes of bfloat16 weights per row, 16-byte pieces swizzled as TMA would have written them
            uint8_t* dst = base + row * 128;
#pragma unroll
            for (int q = 0; q < 8; ++q) {
                const float* x = &v[q >> 2][(q & 3) * 8];
                *reinterpret_cast<uint4*>(dst + ((q ^ (row & 7)) << 4)) =
                    make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s.p_full));
            if (row_ok) {
                p.ml[tile * 256 + row] = m;
                p.ml[tile * 256 + 128 + row] = l;
            }
            if (mbar_wait(smem_u32(&s.o_full), 0, abort_flag)) {
                tc_fence_after();
                float* out = p.part + tile * p.c * 128 + row;
                for (int c = 0; c < p.c; c += 32) {
                    tmem_ld32(tq + (uint32_t)c, v[0]);
                    tmem_ld_wait();
                    if (row_ok) {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (c + i < p.c) out[(long long)(c + i) * 128] = v[0][i];
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 1) tmem_dealloc(tmem, 512);
    if (threadIdx.x == 0 && s.abort) *(volatile int*)p.error_flag = 1;
}

// merges the chunks of 32 rows x 8 latent columns: the warps share the chunks.  grid (c / 8, row tiles * 4, batch)
__global__ void __launch_bounds__(256)
latent_combine_kernel(const LatentParams p, bf16* __restrict__ out, long long o_head)
{
    __shared__ float red[8][9][32];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, b = blockIdx.z, c0 = blockIdx.x * 8;
    const int rt = blockIdx.y >> 2, row = (blockIdx.y & 3) * 32 + lane, row0 = rt * kTile;
    if (row0 + (int)(blockIdx.y & 3) * 32 >= p.rows) return;
    int first, n;
    chunk_range(p.start[b], row0, p.rows, p.heads, p.window, first, n);
    if (p.start[b] < 0 || p.start[b] + p.seq > p.keys || n > p.chunks) return;
    const long long t0 = ((long long)b * p.row_tiles + rt) * p.chunks;
    const float* ml = p.ml + t0 * 256 + row;
    const bool row_ok = row0 + row < p.rows;
    float m = -INFINITY;
    if (row_ok)
#pragma unroll 4
        for (int i = warp; i < n; i += 8) m = fmaxf(m, ml[(long long)i * 256]);
    red[warp][0][lane] = m;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 8; ++k) m = fmaxf(m, red[k][0][lane]);
    __syncthreads();
    float acc[8] = {}, l = 0.f;
    if (row_ok) {
        const float* src = p.part + (t0 * p.c + c0) * 128 + row;
#pragma unroll 4
        for (int i = warp; i < n; i += 8) {
            const float w = exp2_approx(ml[(long long)i * 256] - m);
            l = fmaf(w, ml[(long long)i * 256 + 128], l);
#pragma unroll
            for (int k = 0; k < 8; ++k) acc[k] = fmaf(w, src[((long long)i * p.c + k) * 128], acc[k]);
        }
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) red[warp][k][lane] = acc[k];
    red[warp][8][lane] = l;
    __syncthreads();
    // thread (row, column): eight threads write the 16 bytes of a row
    const int rr = threadIdx.x >> 3, k = threadIdx.x & 7;
    float v = 0.f, sum = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
        v += red[w][k][rr];
        sum += red[w][8][rr];
    }
    const int r = row0 + (int)(blockIdx.y & 3) * 32 + rr;
    if (r < p.rows) out[((long long)b * p.rows + r) * o_head + c0 + k] = __float2bfloat16_rn(v / sum);
}

int latent_chunks(const zkfp_attention_args& a) { return (a.max_keys + kChunk - 1) / kChunk + 1; }

size_t latent_smem(const zkfp_attention_args& a)
{
    return 1024 + (size_t)((a.d1 + 63) / 64 + (a.d2 + 63) / 64) * (kSeg + kSegC);
}

}  // namespace

bool attention_decode_tc_takes(const zkfp_attention_args& a)
{
    return a.dtype == ZKFP_BF16 && a.shared && a.v == a.k1 && a.dv == a.d1 && a.v_tok == a.k1_tok && a.d1 <= 512 &&
           a.k2_tok == a.k1_tok && a.base == 0 && a.keys > 0 && a.max_keys > 0 && latent_smem(a) <= kSmemMax &&
           a.seq * a.heads < 0x1000000 && !((a.q_head | a.k1_tok | a.o_head | a.slot_stride) & 7) &&
           !(((uintptr_t)a.q | (uintptr_t)a.k1 | (uintptr_t)a.k2 | (uintptr_t)a.out) & 15);
}

long long attention_decode_scratch(const zkfp_attention_args& a)
{
    const long long row_tiles = (a.seq * a.heads + kTile - 1) / kTile;
    return a.batch * row_tiles * latent_chunks(a) * 128 * (a.d1 + 2);
}

int launch_attention_decode_tc(const zkfp_attention_args& a, cudaStream_t st)
{
    if (!a.scratch) return ZKDS_ERR_ARG;
    LatentParams p;
    p.start = a.start; p.slots = a.slots;
    p.rows = (int)(a.seq * a.heads); p.heads = (int)a.heads; p.seq = (int)a.seq; p.window = a.window;
    p.c = a.d1; p.r = a.d2; p.segc = (a.d1 + 63) / 64; p.segr = (a.d2 + 63) / 64;
    p.chunks = latent_chunks(a);
    p.keys = (int)a.keys;
    p.row_tiles = (p.rows + kTile - 1) / kTile;
    p.part = a.scratch;
    p.ml = a.scratch + (long long)a.batch * p.row_tiles * p.chunks * 128 * p.c;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.error_flag = fp_error_flag();
    if (!p.error_flag) return ZKDS_ERR_WORKSPACE;
    CUtensorMap q1, q2, k1, k2;
    const uint64_t rows = (uint64_t)(a.batch * p.rows), r = (uint64_t)(a.d2 ? a.d2 : 8);
    const uint64_t dq1[2] = {(uint64_t)a.d1, rows}, dq2[2] = {r, rows}, qs[1] = {(uint64_t)a.q_head * 2};
    // the slot extent only bounds the coordinate; slots are valid by construction
    const uint64_t dk1[3] = {(uint64_t)a.d1, (uint64_t)a.keys, 65536}, dk2[3] = {r, (uint64_t)a.keys, 65536};
    const uint64_t ks[2] = {(uint64_t)a.k1_tok * 2, (uint64_t)a.slot_stride * 2};
    const uint32_t bq[2] = {64, kTile}, bk[3] = {64, kChunk, 1};
    const bf16* q = (const bf16*)a.q;
    if (!fp_tensor_map(&q1, q, 2, dq1, qs, bq) || !fp_tensor_map(&q2, a.d2 ? q + a.d1 : q, 2, dq2, qs, bq) ||
        !fp_tensor_map(&k1, a.k1, 3, dk1, ks, bk) || !fp_tensor_map(&k2, a.d2 ? a.k2 : a.k1, 3, dk2, ks, bk))
        return ZKDS_ERR_UNSUPPORTED;
    ZKDS_CUDA(cudaFuncSetAttribute(attention_latent_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    const size_t smem = latent_smem(a) < 120 * 1024 ? 120 * 1024 : latent_smem(a);
    attention_latent_kernel<<<dim3((unsigned)p.chunks, (unsigned)p.row_tiles, (unsigned)a.batch), 192, smem, st>>>(q1, q2, k1,
                                                                                                             k2, p);
    int rc = fp_launched();
    if (rc != ZKDS_OK) return rc;
    latent_combine_kernel<<<dim3((unsigned)(p.c / 8), (unsigned)p.row_tiles * 4, (unsigned)a.batch), 256, 0, st>>>(
        p, (bf16*)a.out, a.o_head);
    return fp_launched();
}

}  // namespace zkds
