// tcgen05 attention in the latent space (decode steps and short portions of latent attention): every query head of a token attends to
// the SAME cached rows [latent | rotated key part | zeros], and the mean of their latents is the output.
//
// Many rows (short portions of prompts): the 128 MMA rows of a CTA are consecutive (token, head) pairs of one work item: rows of q are token-major, so they are one 2-D box.
// A tile of KT cached rows is loaded once into shared memory and is both operands: keys (K-major, all columns) and values (MN-major, up
// to 256 of the latent's columns; wider latents take one CTA per 256 columns).
//
//   warp 0   : TMA producer — Q once, then key tiles through the block table (ring of n_stages, SWIZZLE_128B)
//   warp 1   : TMEM allocator + tcgen05.mma issuer:  S = Q K^T,  O += P V  (P read from TMEM, where it replaces S)
//   warps 2-5: softmax, one thread per row: S to registers, mask, online maximum and sum in fp32, P (16-bit pairs) back over S
//
// S has two buffers, so Q K^T of the next tile runs under this tile's exponentials. O stays in TMEM over all tiles and is rescaled
// only when a row's running maximum grows by more than 2^8. The key range can be split over gridDim.z CTAs; the last one merges.
#include "hds_host.cuh"
#include "hds_ptx.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kLaThreads = 192, kLaRows = 128, kLaMaxStages = 8, kLaValues = 256;
constexpr size_t kLaSmemMax = 227 * 1024;

struct LatentArgs {
    void* out;                      // [T][heads][rank]
    const int32_t* block_tables;
    const hds_attn_item* items;
    int max_blocks_per_seq, heads, rank, panels, block_size, window, n_splits, n_stages, row_tiles;
    float scale_log2;
    int32_t* tickets;               // [units][4], zero between calls
    float* ws_ml;                   // [units][n_splits][128][2]
    float* ws_o;                    // [units][n_splits][128][256]
};

__device__ __forceinline__ float la_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <bool kBf16, int KT>
__global__ void __launch_bounds__(kLaThreads, 1)
paged_attn_latent_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv, const LatentArgs a) {
    constexpr uint32_t TMEM_COLS = 512;   // S: 2 x KT columns, O: up to 256
    constexpr uint32_t IDESC_QK = make_idesc_f16(128, KT, kBf16, false, false);
    constexpr int QPANEL = kLaRows * 128, KPANEL = KT * 128;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* q_sm = smem;
    uint8_t* kv_sm = q_sm + a.panels * QPANEL;
    uint64_t* bars = reinterpret_cast<uint64_t*>(kv_sm + static_cast<size_t>(a.n_stages) * a.panels * KPANEL);
    uint64_t *q_full = bars, *s_full = bars + 1 /*[2]*/, *p_full = bars + 3 /*[2]*/, *o_done = bars + 5, *kv_full = bars + 6,
             *kv_empty = kv_full + kLaMaxStages;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(kv_empty + kLaMaxStages);

    const uint32_t warp = warp_id(), lane = lane_id();
    pdl_enter();
    const int item_idx = static_cast<int>(blockIdx.x) / a.row_tiles, row_tile = static_cast<int>(blockIdx.x) % a.row_tiles;
    const hds_attn_item item = a.items[item_idx];
    const int row0 = row_tile * kLaRows, n_rows = min(kLaRows, item.n_q * a.heads - row0);    // live rows of this tile
    if (n_rows <= 0) return;
    const int v0 = blockIdx.y * kLaValues;                                 // first latent column of this CTA's output
    const int nv = min(kLaValues, ((a.rank + 63) & ~63) - v0);
    const int pos_lo = item.pos0 + row0 / a.heads, pos_hi = item.pos0 + (row0 + n_rows - 1) / a.heads;
    const int t_first = a.window > 0 ? max(0, pos_lo - a.window + 1) / KT : 0;
    const int live = pos_hi / KT + 1 - t_first;
    const int tps = (live + a.n_splits - 1) / a.n_splits, eff_splits = (live + tps - 1) / tps;
    const int split = blockIdx.z;
    if (split >= eff_splits) return;
    const int t0 = t_first + split * tps, n_tiles = min(tps, live - split * tps);

    if (warp == 0 && lane == 0) {
        prefetch_tmap(&tmap_q);
        prefetch_tmap(&tmap_kv);
        mbar_init(q_full, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(p_full + i, 4);
        }
        mbar_init(o_done, 1);
        for (int i = 0; i < a.n_stages; ++i) {
            mbar_init(kv_full + i, 1);
            mbar_init(kv_empty + i, 1);
        }
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc<TMEM_COLS>(tmem_slot);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, t_o = tmem + 2 * KT;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(q_full, a.panels * QPANEL);
            for (int p = 0; p < a.panels; ++p)
                tma_load_2d(q_sm + p * QPANEL, &tmap_q, q_full, p * 64, item.q_row0 * a.heads + row0, kEvictFirst);
            const int32_t* table = a.block_tables + static_cast<int64_t>(item.seq) * a.max_blocks_per_seq;
            uint32_t stage = 0, phase = 0;
            for (int i = 0; i < n_tiles; ++i) {
                const int first = (t0 + i) * KT;        // pages hold whole tiles
                mbar_wait(kv_empty + stage, phase ^ 1);
                mbar_expect_tx(kv_full + stage, a.panels * KPANEL);
                const int row = table[first / a.block_size] * a.block_size + first % a.block_size;
                uint8_t* dst = kv_sm + static_cast<size_t>(stage) * a.panels * KPANEL;
                for (int p = 0; p < a.panels; ++p) tma_load_2d(dst + p * KPANEL, &tmap_kv, kv_full + stage, p * 64, row, kEvictNormal);
                if (++stage == static_cast<uint32_t>(a.n_stages)) {
                    stage = 0;
                    phase ^= 1;
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_pv = make_idesc_f16(128, nv, kBf16, false, true);
            auto issue_qk = [&](int i, uint32_t stage) {
                const uint8_t* k = kv_sm + static_cast<size_t>(stage) * a.panels * KPANEL;
                for (int p = 0; p < a.panels; ++p) {
                    const uint64_t dq = make_desc_kmajor_sw128(smem_u32(q_sm + p * QPANEL)), dk = make_desc_kmajor_sw128(smem_u32(k + p * KPANEL));
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk) umma_f16_ss(tmem + (i & 1) * KT, dq + 2 * kk, dk + 2 * kk, IDESC_QK, (p > 0 || kk > 0) ? 1u : 0u);
                }
                umma_commit(s_full + (i & 1));
            };
            mbar_wait(q_full, 0);
            mbar_wait(kv_full, 0);
            tc_fence_after();
            issue_qk(0, 0);
            uint32_t stage = 0, phase = 0;
            for (int i = 0; i < n_tiles; ++i) {
                const bool wrap = stage + 1 == static_cast<uint32_t>(a.n_stages);
                const uint32_t nstage = wrap ? 0 : stage + 1, nphase = wrap ? phase ^ 1 : phase;
                if (i + 1 < n_tiles) {       // (over P of tile i - 1, whose product must be complete)
                    if (i > 0) mbar_wait(o_done, (i - 1) & 1);
                    mbar_wait(kv_full + nstage, nphase);
                    tc_fence_after();
                    issue_qk(i + 1, nstage);
                }
                mbar_wait(p_full + (i & 1), (i >> 1) & 1);
                tc_fence_after();
                const uint8_t* v = kv_sm + static_cast<size_t>(stage) * a.panels * KPANEL + (v0 / 64) * KPANEL;
#pragma unroll
                for (int kk = 0; kk < KT / 16; ++kk)
                    umma_f16_ts(t_o, tmem + (i & 1) * KT + kk * 8, make_desc_mnmajor_sw128(smem_u32(v + kk * 16 * 128), KPANEL), idesc_pv,
                                (i > 0 || kk > 0) ? 1u : 0u);
                umma_commit(o_done);
                umma_commit(kv_empty + stage);
                stage = nstage;
                phase = nphase;
            }
        }
    } else {
        const uint32_t quad = warp & 3;
        const int r = quad * 32 + lane;
        const int r_tok = (row0 + r) / a.heads, r_head = (row0 + r) % a.heads;
        const int q_pos = item.pos0 + r_tok;
        const bool quad_live = static_cast<int>(quad * 32) < n_rows, row_valid = r < n_rows;
        const uint32_t la = (quad * 32u) << 16;
        const int win_lo = a.window > 0 ? q_pos - a.window : -1;     // keys at or before this position are hidden
        float m_run = -INFINITY, l_run = 0.0f;
        for (int i = 0; i < n_tiles; ++i) {
            const int tok0 = (t0 + i) * KT;
            const uint32_t t_s = tmem + (i & 1) * KT + la;
            mbar_wait(s_full + (i & 1), (i >> 1) & 1);
            tc_fence_after();
            if (!quad_live) {      // no live row here: keep the barriers going
                if (i > 0) mbar_wait(o_done, (i - 1) & 1);
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(p_full + (i & 1));
                continue;
            }
            uint32_t sr[KT];
#pragma unroll
            for (int c = 0; c < KT; c += 32) tmem_ld_32x32(t_s + c, *reinterpret_cast<uint32_t(*)[32]>(&sr[c]));
            tmem_ld_wait();
            float tmax = -INFINITY;
            if (tok0 + KT - 1 > pos_lo || (a.window > 0 && tok0 <= pos_hi - a.window)) {
#pragma unroll
                for (int j = 0; j < KT; ++j) {
                    const float s = (tok0 + j <= q_pos && tok0 + j > win_lo) ? __uint_as_float(sr[j]) : -INFINITY;
                    sr[j] = __float_as_uint(s);
                    tmax = fmaxf(tmax, s);
                }
            } else {
#pragma unroll
                for (int j = 0; j < KT; ++j) tmax = fmaxf(tmax, __uint_as_float(sr[j]));
            }
            const float m_cand = fmaxf(m_run, tmax * a.scale_log2);
            const bool fresh = m_run == -INFINITY;
            const bool grow = m_cand > m_run + 8.0f || (fresh && m_cand != -INFINITY);
            const float m_new = grow ? m_cand : m_run;
            const float alpha = grow ? (fresh ? 0.0f : la_ex2(m_run - m_new)) : 1.0f;
            const float m_sub = m_new == -INFINITY ? 0.0f : m_new;
            float ps = 0.0f;
            uint32_t packed[KT / 2];
#pragma unroll
            for (int j = 0; j < KT; j += 2) {
                const float p0 = la_ex2(fmaf(__uint_as_float(sr[j]), a.scale_log2, -m_sub));
                const float p1 = la_ex2(fmaf(__uint_as_float(sr[j + 1]), a.scale_log2, -m_sub));
                ps += p0 + p1;
                packed[j >> 1] = pack2<kBf16>(p0, p1);
            }
            l_run = l_run * alpha + ps;
            m_run = m_new;
            if (i > 0) {
                mbar_wait(o_done, (i - 1) & 1);
                tc_fence_after();
                const bool rescale = grow && !fresh;
                if (__any_sync(0xffffffffu, rescale)) {
                    const float f = rescale ? alpha : 1.0f;
                    for (int c = 0; c < nv; c += 32) {
                        uint32_t o[32];
                        tmem_ld_32x32(t_o + la + c, o);
                        tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
                        tmem_st_32x32(t_o + la + c, o);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < KT / 2; c += 16) tmem_st_32x16(t_s + c, *reinterpret_cast<uint32_t(*)[16]>(&packed[c]));
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full + (i & 1));
        }
        mbar_wait(o_done, (n_tiles - 1) & 1);
        tc_fence_after();
        const int width = min(nv, a.rank - v0);              // output values of this CTA
        const int64_t out0 = (static_cast<int64_t>(item.q_row0) * a.heads + row0 + r) * a.rank + v0;
        const bool vec = (a.rank & 7) == 0;
        auto store32 = [&](int c, const float (&o)[32], float inv) {
            if (vec) {
#pragma unroll
                for (int j = 0; j < 32; j += 8)
                    if (c + j < width) {
                        uint4 v;
                        v.x = pack2<kBf16>(o[j] * inv, o[j + 1] * inv);
                        v.y = pack2<kBf16>(o[j + 2] * inv, o[j + 3] * inv);
                        v.z = pack2<kBf16>(o[j + 4] * inv, o[j + 5] * inv);
                        v.w = pack2<kBf16>(o[j + 6] * inv, o[j + 7] * inv);
                        st_v4(reinterpret_cast<char*>(a.out) + (out0 + c + j) * 2, v);
                    }
            } else {
#pragma unroll
                for (int j = 0; j < 32; ++j)
                    if (c + j < width) store_scalar<kBf16>(a.out, out0 + c + j, o[j] * inv);
            }
        };
        const int64_t unit = static_cast<int64_t>(blockIdx.x) * gridDim.y + blockIdx.y;
        const int64_t ws_row = (unit * a.n_splits + split) * kLaRows + r;
        if (quad_live) {
            const float inv = 1.0f / l_run;
            for (int c = 0; c < nv; c += 32) {
                uint32_t t[32];
                tmem_ld_32x32(t_o + la + c, t);
                tmem_ld_wait();
                float o[32];
#pragma unroll
                for (int j = 0; j < 32; ++j) o[j] = __uint_as_float(t[j]);
                if (!row_valid) continue;
                if (eff_splits == 1) {
                    store32(c, o, inv);
                } else {
                    float4* w = reinterpret_cast<float4*>(a.ws_o + ws_row * kLaValues + c);
#pragma unroll
                    for (int j = 0; j < 32; j += 4) __stcg(w + (j >> 2), make_float4(o[j], o[j + 1], o[j + 2], o[j + 3]));
                }
            }
            tc_fence_before();
            __syncwarp();
            if (eff_splits > 1) {
                if (row_valid) __stcg(reinterpret_cast<float2*>(a.ws_ml + ws_row * 2), make_float2(m_run, l_run));
                __threadfence();
                __syncwarp();
                int last = 0;
                if (lane == 0) last = atomicAdd(&a.tickets[unit * 4 + quad], 1) == eff_splits - 1;
                last = __shfl_sync(0xffffffffu, last, 0);
                if (last) {
                    __threadfence();
                    if (row_valid) {
                        const int64_t first = unit * a.n_splits * kLaRows + r;
                        float mx = -INFINITY, l = 0.0f;
                        for (int s = 0; s < eff_splits; ++s) mx = fmaxf(mx, __ldcg(a.ws_ml + (first + s * kLaRows) * 2));
                        for (int s = 0; s < eff_splits; ++s) {
                            const float2 ml = __ldcg(reinterpret_cast<const float2*>(a.ws_ml + (first + s * kLaRows) * 2));
                            l = fmaf(ml.x == -INFINITY ? 0.0f : la_ex2(ml.x - mx), ml.y, l);
                        }
                        for (int c = 0; c < nv; c += 32) {
                            float o[32];
#pragma unroll
                            for (int j = 0; j < 32; ++j) o[j] = 0.0f;
                            for (int s = 0; s < eff_splits; ++s) {
                                const float m = __ldcg(a.ws_ml + (first + s * kLaRows) * 2);
                                const float f = m == -INFINITY ? 0.0f : la_ex2(m - mx);
                                const float4* w = reinterpret_cast<const float4*>(a.ws_o + (first + s * kLaRows) * kLaValues + c);
#pragma unroll
                                for (int j = 0; j < 32; j += 4) {
                                    const float4 t = __ldcg(w + (j >> 2));
                                    o[j] = fmaf(f, t.x, o[j]);
                                    o[j + 1] = fmaf(f, t.y, o[j + 1]);
                                    o[j + 2] = fmaf(f, t.z, o[j + 2]);
                                    o[j + 3] = fmaf(f, t.w, o[j + 3]);
                                }
                            }
                            store32(c, o, 1.0f / l);
                        }
                    }
                    __syncwarp();
                    if (lane == 0) a.tickets[unit * 4 + quad] = 0;
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<TMEM_COLS>(tmem);
    }
}

// ---- few rows: decode steps ---------------------------------------------------------------------------------------------
// The same attention with the roles of the operands swapped: the 128 MMA rows are KEYS and the N columns are the item's (token, head)
// rows, so that a step whose heads do not fill 128 rows does not pay for them, and O^T [latent value, row] holds latents of any width
// at once. A tile of 128 cached rows is read once:  S^T = K Q^T,  O^T += V^T P^T  (V^T: the tile's first panels, MN-major).
//
//   warp 0   : TMA producer; every 64-column panel of a tile has its own barriers, so panels refill as soon as they are used up
//   warp 1   : TMEM, tcgen05.mma
//   warps 2-5: thread = key. Scores of a row lie across lanes: maxima by a transposing butterfly and shared memory, sums kept per
//              thread until the end; P^T to shared memory (K-major)
constexpr int kFwKeys = 128, kFwPanel = kFwKeys * 128, kFwMaxBars = 32;

struct FewArgs {
    LatentArgs l;
    int v_blocks;       // 128-value blocks of the latent
    int stage_panels;   // panels between two stages' bases
};

template <int N>
__host__ __device__ constexpr size_t fw_fixed_smem(int panels) {
    return 1024 + static_cast<size_t>(panels) * N * 128 /*Q*/ + 2 * N * 128 /*P*/ + (2 * 4 * N + 4 * N + 4 * N + 2 * N) * 4 + (8 + 2 * kFwMaxBars) * 8 + 16;
}

// key tiles that a row tile sees, and how they are split
struct FewTiles {
    int first, live, per, splits;
};
__device__ __forceinline__ FewTiles fw_tiles(const LatentArgs& a, int pos_lo, int pos_hi) {
    FewTiles t;
    t.first = a.window > 0 ? max(0, pos_lo - a.window + 1) / kFwKeys : 0;
    t.live = pos_hi / kFwKeys + 1 - t.first;
    t.per = (t.live + a.n_splits - 1) / a.n_splits;
    t.splits = (t.live + t.per - 1) / t.per;
    return t;
}

// v[0..31] of every lane -> lane n holds op over the lanes of v[n]
template <typename Op>
__device__ __forceinline__ float fw_transpose_reduce(float (&v)[32], uint32_t lane, Op op) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int j = 0; j < o; ++j) {
            const float send = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
            v[j] = op(keep, __shfl_xor_sync(0xffffffffu, send, o));
        }
    }
    return v[0];
}

template <bool kBf16, int N>
__global__ void __launch_bounds__(kLaThreads, 1)
paged_attn_latent_few_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv, const FewArgs f) {
    const LatentArgs& a = f.l;
    constexpr uint32_t TMEM_COLS = 512;    // S^T: 2 x N columns, O^T: N per 128 values
    constexpr uint32_t IDESC_QK = make_idesc_f16(128, N, kBf16, false, false);
    constexpr uint32_t IDESC_PV = make_idesc_f16(128, N, kBf16, true, false);
    constexpr int NP = N * 128;            // a panel of Q or P
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* kv_sm = smem;
    uint8_t* q_sm = kv_sm + static_cast<size_t>(a.n_stages) * f.stage_panels * kFwPanel;
    uint8_t* p_sm = q_sm + a.panels * NP;
    float* mx_s = reinterpret_cast<float*>(p_sm + 2 * NP);   // [2][4][N] maxima of 32 keys each
    float* m_s = mx_s + 2 * 4 * N;                           // [4][N] reference maxima, one copy per warp
    float* al_s = m_s + 4 * N;                               // [4][N] rescale factors; at the end sums
    int* pos_s = reinterpret_cast<int*>(al_s + 4 * N);       // [N] position of a row's query
    float* inv_s = reinterpret_cast<float*>(pos_s + N);      // [N]
    uint64_t* bars = reinterpret_cast<uint64_t*>(inv_s + N);
    uint64_t *q_full = bars, *s_full = bars + 1 /*[2]*/, *p_full = bars + 3, *o_done = bars + 4, *k_full = bars + 8, *k_empty = k_full + kFwMaxBars;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5);

    const uint32_t warp = warp_id(), lane = lane_id();
    pdl_enter();
    const int item_idx = static_cast<int>(blockIdx.x) / a.row_tiles, row_tile = static_cast<int>(blockIdx.x) % a.row_tiles;
    const hds_attn_item item = a.items[item_idx];
    const int row0 = row_tile * N, n_rows = min(N, item.n_q * a.heads - row0);
    if (n_rows <= 0) return;
    const int pos_lo = item.pos0 + row0 / a.heads, pos_hi = item.pos0 + (row0 + n_rows - 1) / a.heads;
    const FewTiles ft = fw_tiles(a, pos_lo, pos_hi);
    const int split = blockIdx.z, eff_splits = ft.splits;
    if (split >= eff_splits) return;
    const int t0 = ft.first + split * ft.per, n_tiles = min(ft.per, ft.live - split * ft.per);

    if (warp == 0 && lane == 0) {
        prefetch_tmap(&tmap_q);
        prefetch_tmap(&tmap_kv);
        mbar_init(q_full, 1);
        mbar_init(s_full, 1);
        mbar_init(s_full + 1, 1);
        mbar_init(p_full, 4);
        mbar_init(o_done, 1);
        for (int i = 0; i < a.n_stages * a.panels; ++i) {
            mbar_init(k_full + i, 1);
            mbar_init(k_empty + i, 1);
        }
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc<TMEM_COLS>(tmem_slot);
        tmem_relinquish();
    }
    for (int n = threadIdx.x; n < N; n += kLaThreads) pos_s[n] = item.pos0 + min(row0 + n, item.n_q * a.heads - 1) / a.heads;
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, t_o = tmem + 2 * N;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(q_full, a.panels * NP);
            for (int p = 0; p < a.panels; ++p) tma_load_2d(q_sm + p * NP, &tmap_q, q_full, p * 64, item.q_row0 * a.heads + row0, kEvictFirst);
            const int32_t* table = a.block_tables + static_cast<int64_t>(item.seq) * a.max_blocks_per_seq;
            const int last_blk = pos_hi / a.block_size;
            for (int i = 0; i < n_tiles; ++i) {
                const int st = i % a.n_stages;
                const uint32_t phase = (i / a.n_stages) & 1;
                int row[2];
#pragma unroll
                for (int g = 0; g < 2; ++g) {       // (behind the last page: that page again, masked)
                    const int pos = (t0 + i) * kFwKeys + g * 64;
                    row[g] = table[min(pos / a.block_size, last_blk)] * a.block_size + pos % a.block_size;
                }
                for (int p = 0; p < a.panels; ++p) {
                    uint64_t* full = k_full + st * a.panels + p;
                    mbar_wait(k_empty + st * a.panels + p, phase ^ 1);
                    mbar_expect_tx(full, kFwPanel);
                    uint8_t* dst = kv_sm + (static_cast<size_t>(st) * f.stage_panels + p) * kFwPanel;
                    tma_load_2d(dst, &tmap_kv, full, p * 64, row[0], kEvictNormal);
                    tma_load_2d(dst + kFwPanel / 2, &tmap_kv, full, p * 64, row[1], kEvictNormal);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            auto issue_qk = [&](int i) {
                const int st = i % a.n_stages;
                const uint8_t* k = kv_sm + static_cast<size_t>(st) * f.stage_panels * kFwPanel;
                for (int p = 0; p < a.panels; ++p) {
                    mbar_wait(k_full + st * a.panels + p, (i / a.n_stages) & 1);
                    tc_fence_after();
                    const uint64_t dk = make_desc_kmajor_sw128(smem_u32(k + p * kFwPanel)), dq = make_desc_kmajor_sw128(smem_u32(q_sm + p * NP));
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk) umma_f16_ss(tmem + (i & 1) * N, dk + 2 * kk, dq + 2 * kk, IDESC_QK, (p > 0 || kk > 0) ? 1u : 0u);
                    if (p >= 2 * f.v_blocks) umma_commit(k_empty + st * a.panels + p);      // no values in this panel
                }
                umma_commit(s_full + (i & 1));
            };
            const bool ahead = a.n_stages > 1;
            mbar_wait(q_full, 0);
            issue_qk(0);
            for (int i = 0; i < n_tiles; ++i) {
                if (ahead && i + 1 < n_tiles) issue_qk(i + 1);
                mbar_wait(p_full, i & 1);
                tc_fence_after();
                const int st = i % a.n_stages;
                const uint8_t* v = kv_sm + static_cast<size_t>(st) * f.stage_panels * kFwPanel;
                const uint64_t dp = make_desc_kmajor_sw128(smem_u32(p_sm));
                for (int b = 0; b < f.v_blocks; ++b) {
                    const uint64_t dv = make_desc_mnmajor_sw128(smem_u32(v + 2 * b * kFwPanel), kFwPanel);
#pragma unroll
                    for (int kk = 0; kk < kFwKeys / 16; ++kk)
                        umma_f16_ss(t_o + b * N, dv + kk * ((16 * 128) >> 4), dp + (kk >> 2) * (NP >> 4) + 2 * (kk & 3), IDESC_PV, (i > 0 || kk > 0) ? 1u : 0u);
                    umma_commit(k_empty + st * a.panels + 2 * b);
                    if (2 * b + 1 < a.panels) umma_commit(k_empty + st * a.panels + 2 * b + 1);
                }
                umma_commit(o_done);
                if (!ahead && i + 1 < n_tiles) issue_qk(i + 1);
            }
        }
    } else {
        const uint32_t quad = warp & 3;
        const int r = quad * 32 + lane;                  // key of the tile; later value of a block
        const uint32_t la = (quad * 32u) << 16;
        const int tid = threadIdx.x - 64;
        auto group_sync = [] { asm volatile("bar.sync 1, 128;" ::: "memory"); };
        float m_run[N / 32], l[N];                       // m_run: of rows lane, lane + 32
#pragma unroll
        for (int g = 0; g < N / 32; ++g) m_run[g] = -INFINITY;
#pragma unroll
        for (int n = 0; n < N; ++n) l[n] = 0.0f;
        uint8_t* p_key = p_sm + (r >> 6) * NP + (r & 7) * 2;
        const int chunk = (r & 63) >> 3;
        for (int i = 0; i < n_tiles; ++i) {
            const int tile0 = (t0 + i) * kFwKeys, key = tile0 + r;
            mbar_wait(s_full + (i & 1), (i >> 1) & 1);
            tc_fence_after();
            float s[N];
#pragma unroll
            for (int g = 0; g < N / 32; ++g) {
                uint32_t t[32];
                tmem_ld_32x32(tmem + (i & 1) * N + la + g * 32, t);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; ++j) s[g * 32 + j] = __uint_as_float(t[j]);
            }
            if (tile0 + kFwKeys - 1 > pos_lo || (a.window > 0 && tile0 <= pos_hi - a.window)) {
#pragma unroll
                for (int n = 0; n < N; ++n) {
                    const int q = pos_s[n];
                    if (key > q || (a.window > 0 && key <= q - a.window)) s[n] = -INFINITY;
                }
            }
            // ---- maxima of the rows over the tile's keys ----
            float* mx = mx_s + (i & 1) * 4 * N;
#pragma unroll
            for (int g = 0; g < N / 32; ++g) {
                float v[32];
#pragma unroll
                for (int j = 0; j < 32; ++j) v[j] = s[g * 32 + j];
                mx[quad * N + g * 32 + lane] = fw_transpose_reduce(v, lane, [](float x, float y) { return fmaxf(x, y); });
            }
            group_sync();
            bool any = false;
#pragma unroll
            for (int g = 0; g < N / 32; ++g) {
                const int n = g * 32 + lane;
                const float t = fmaxf(fmaxf(mx[n], mx[N + n]), fmaxf(mx[2 * N + n], mx[3 * N + n])) * a.scale_log2;
                const float cand = fmaxf(m_run[g], t);
                const bool fresh = m_run[g] == -INFINITY, grow = cand > m_run[g] + 8.0f || (fresh && cand != -INFINITY);
                const float m_new = grow ? cand : m_run[g];
                al_s[quad * N + n] = grow && !fresh ? la_ex2(m_run[g] - m_new) : 1.0f;
                m_s[quad * N + n] = m_new == -INFINITY ? 0.0f : m_new;
                any |= grow && !fresh;
                m_run[g] = m_new;
            }
            any = __any_sync(0xffffffffu, any);      // (the same for all four warps)
            __syncwarp();
            if (i > 0) {
                mbar_wait(o_done, (i - 1) & 1);      // P has been used, O is stable
                tc_fence_after();
                if (any) {
#pragma unroll
                    for (int n = 0; n < N; ++n) l[n] *= al_s[quad * N + n];
                    for (int b = 0; b < f.v_blocks; ++b)
#pragma unroll
                        for (int g = 0; g < N / 32; ++g) {
                            uint32_t t[32];
                            tmem_ld_32x32(t_o + la + b * N + g * 32, t);
                            tmem_ld_wait();
#pragma unroll
                            for (int j = 0; j < 32; ++j) t[j] = __float_as_uint(__uint_as_float(t[j]) * al_s[quad * N + g * 32 + j]);
                            tmem_st_32x32(t_o + la + b * N + g * 32, t);
                        }
                    tmem_st_wait();
                }
            }
#pragma unroll
            for (int n = 0; n < N; n += 4) {
                const float4 m = *reinterpret_cast<const float4*>(m_s + quad * N + n);
                const float pr[4] = {la_ex2(fmaf(s[n], a.scale_log2, -m.x)), la_ex2(fmaf(s[n + 1], a.scale_log2, -m.y)),
                                     la_ex2(fmaf(s[n + 2], a.scale_log2, -m.z)), la_ex2(fmaf(s[n + 3], a.scale_log2, -m.w))};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    l[n + e] += pr[e];
                    store_scalar<kBf16>(p_key + (n + e) * 128 + ((chunk ^ ((n + e) & 7)) << 4), 0, pr[e]);
                }
            }
            tc_fence_before();
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
        }
        // ---- sums over keys, then the rows' outputs ----
#pragma unroll
        for (int g = 0; g < N / 32; ++g) {
            float v[32];
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] = l[g * 32 + j];
            const float t = fw_transpose_reduce(v, lane, [](float x, float y) { return x + y; });
            __syncwarp();
            al_s[quad * N + g * 32 + lane] = t;
        }
        group_sync();
        const int64_t unit = blockIdx.x, slot = unit * a.n_splits + split;
        for (int n = tid; n < N; n += 128) {
            const float t = al_s[n] + al_s[N + n] + al_s[2 * N + n] + al_s[3 * N + n];
            inv_s[n] = 1.0f / t;
            if (eff_splits > 1) __stcg(reinterpret_cast<float2*>(a.ws_ml + (slot * kLaRows + n) * 2), make_float2(n / 32 == 0 ? m_run[0] : m_run[N / 32 - 1], t));
        }
        group_sync();
        mbar_wait(o_done, (n_tiles - 1) & 1);
        tc_fence_after();
        const int64_t out0 = (static_cast<int64_t>(item.q_row0) * a.heads + row0) * a.rank;
        const int width = f.v_blocks * 128;
        for (int b = 0; b < f.v_blocks; ++b) {
            const int d = b * 128 + r;
#pragma unroll
            for (int g = 0; g < N / 32; ++g) {
                uint32_t t[32];
                tmem_ld_32x32(t_o + la + b * N + g * 32, t);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    const int n = g * 32 + j;
                    if (n >= n_rows) continue;
                    if (eff_splits > 1) __stcg(a.ws_o + (slot * N + n) * width + d, __uint_as_float(t[j]));
                    else if (d < a.rank) store_scalar<kBf16>(a.out, out0 + static_cast<int64_t>(n) * a.rank + d, __uint_as_float(t[j]) * inv_s[n]);
                }
            }
        }
        tc_fence_before();
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<TMEM_COLS>(tmem);
    }
}

// Splits of a row meet: CTA = (row tile, row), thread = value of each 128-value block.
template <bool kBf16>
__global__ void __launch_bounds__(128) latent_merge_kernel(const FewArgs f, int tile_rows) {
    const LatentArgs& a = f.l;
    pdl_enter();
    const int unit = blockIdx.x, n = blockIdx.y;
    const hds_attn_item item = a.items[unit / a.row_tiles];
    const int row0 = unit % a.row_tiles * tile_rows, n_rows = min(tile_rows, item.n_q * a.heads - row0);
    if (n >= n_rows) return;
    const FewTiles ft = fw_tiles(a, item.pos0 + row0 / a.heads, item.pos0 + (row0 + n_rows - 1) / a.heads);
    if (ft.splits == 1) return;       // written by the attention kernel itself
    const int width = f.v_blocks * 128;
    float mx = -INFINITY, sum = 0.0f;
    for (int s = 0; s < ft.splits; ++s) mx = fmaxf(mx, a.ws_ml[((static_cast<int64_t>(unit) * a.n_splits + s) * kLaRows + n) * 2]);
    float o[5] = {};
#pragma unroll 4
    for (int s = 0; s < ft.splits; ++s) {
        const int64_t slot = static_cast<int64_t>(unit) * a.n_splits + s;
        const float2 ml = *reinterpret_cast<const float2*>(a.ws_ml + (slot * kLaRows + n) * 2);
        const float w = ml.x == -INFINITY ? 0.0f : la_ex2(ml.x - mx);
        sum = fmaf(w, ml.y, sum);
#pragma unroll
        for (int b = 0; b < 5; ++b)
            if (b < f.v_blocks) o[b] = fmaf(w, a.ws_o[(slot * tile_rows + n) * width + b * 128 + threadIdx.x], o[b]);
    }
    const int64_t out0 = (static_cast<int64_t>(item.q_row0) * a.heads + row0 + n) * a.rank;
#pragma unroll
    for (int b = 0; b < 5; ++b)
        if (b < f.v_blocks && b * 128 + static_cast<int>(threadIdx.x) < a.rank) store_scalar<kBf16>(a.out, out0 + b * 128 + threadIdx.x, o[b] / sum);
}

struct FewPlan {
    int n, stages, stage_panels;      // rows per CTA (0: not for this kernel)
};
static FewPlan fw_plan(int rows, int rank, int page_width) {
    const int panels = page_width / 64, v_blocks = (rank + 127) / 128, sp = panels > 2 * v_blocks ? panels : 2 * v_blocks;
    FewPlan p = {0, 0, sp};
    if (rows > 128 || v_blocks > 5) return p;
    for (int n = rows > 32 ? 64 : 32; n >= 32 && p.n == 0; n /= 2) {
        const size_t fixed = n == 64 ? fw_fixed_smem<64>(panels) : fw_fixed_smem<32>(panels);
        for (int st = 3; st >= 1; --st)
            if (st * panels <= kFwMaxBars && fixed + static_cast<size_t>(st) * sp * kFwPanel <= kLaSmemMax) {
                p.n = n;
                p.stages = st;
                break;
            }
    }
    return p;
}

static size_t la_smem(int panels, int kt, int stages) {
    return 1024 + static_cast<size_t>(panels) * 128 * 128 + static_cast<size_t>(stages) * panels * kt * 128 + 256;
}
// keys per tile: 64 when two such tiles fit beside Q, else 32
static int la_tile(int panels) { return la_smem(panels, 64, 2) <= kLaSmemMax ? 64 : la_smem(panels, 32, 2) <= kLaSmemMax ? 32 : 0; }

constexpr int kLaMaxUnits = 148;      // a split launch fills one wave of CTAs at most

template <bool kBf16, int N>
static int launch_few(const CUtensorMap& tq, const CUtensorMap& tk, const FewArgs& f, size_t smem, dim3 grid, cudaStream_t s) {
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!configured[dev & 63]) {
        HDS_CHECK_CUDA(cudaFuncSetAttribute(paged_attn_latent_few_kernel<kBf16, N>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                            static_cast<int>(kLaSmemMax)));
        configured[dev & 63] = true;
    }
    HDS_CHECK_CUDA(launch_kernel(paged_attn_latent_few_kernel<kBf16, N>, grid, dim3(kLaThreads), smem, s, tq, tk, f));
    if (f.l.n_splits > 1) HDS_CHECK_CUDA(launch_kernel(latent_merge_kernel<kBf16>, dim3(grid.x, N), dim3(128), 0, s, f, N));
    return HDS_OK;
}

template <bool kBf16, int KT>
static int launch_latent(const CUtensorMap& tq, const CUtensorMap& tk, LatentArgs& a, dim3 grid, cudaStream_t s) {
    a.n_stages = 2;
    while (a.n_stages < kLaMaxStages && la_smem(a.panels, KT, a.n_stages + 1) <= kLaSmemMax) ++a.n_stages;
    const size_t smem = la_smem(a.panels, KT, a.n_stages);
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!configured[dev & 63]) {
        HDS_CHECK_CUDA(cudaFuncSetAttribute(paged_attn_latent_kernel<kBf16, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                            static_cast<int>(kLaSmemMax)));
        configured[dev & 63] = true;
    }
    HDS_CHECK_CUDA(launch_kernel(paged_attn_latent_kernel<kBf16, KT>, grid, dim3(kLaThreads), smem, s, tq, tk, a));
    return HDS_OK;
}

}  // namespace hds

using namespace hds;

extern "C" int hds_paged_attention_latent_supported(int rank, int page_width) {
    return page_width % 64 == 0 && rank >= 1 && rank <= page_width && la_tile(page_width / 64) != 0 ? 1 : 0;
}

extern "C" int64_t hds_paged_attention_latent_workspace_bytes(void) {
    // per CTA: 128 rows of 256 values, or 64 rows of up to 640
    return 4096 + static_cast<int64_t>(kLaMaxUnits) * (kLaRows * 2 + 64 * 640) * 4;
}

extern "C" int hds_paged_attention_latent_ctas(int item_tokens, int heads, int rank, int page_width, int* tile_keys) {
    const FewPlan p = fw_plan(item_tokens * heads, rank, page_width);
    *tile_keys = p.n ? kFwKeys : la_tile(page_width / 64);
    return p.n ? (item_tokens * heads + p.n - 1) / p.n : (item_tokens * heads + kLaRows - 1) / kLaRows * ((rank + kLaValues - 1) / kLaValues);
}

extern "C" int hds_paged_attention_latent(const void* q, void* out, const void* pages, int64_t num_blocks, const int32_t* block_tables,
                                          int max_blocks_per_seq, const hds_attn_item* items, int n_items, int item_tokens, int T, int heads,
                                          int rank, int page_width, int block_size, float scale, int window, int n_splits, void* workspace,
                                          int64_t workspace_bytes, int dtype, void* stream) {
    HDS_REQUIRE(dtype == 0 || dtype == 1, "hds_paged_attention_latent: dtype 0 bf16 / 1 fp16");
    HDS_REQUIRE(hds_paged_attention_latent_supported(rank, page_width), "hds_paged_attention_latent: page rows of 64-value panels, up to 576 values");
    HDS_REQUIRE(block_size % 64 == 0 && heads >= 1 && window >= 0 && item_tokens >= 1, "hds_paged_attention_latent: pages of whole 64-token tiles");
    if (n_items == 0) return HDS_OK;
    LatentArgs a;
    memset(&a, 0, sizeof(a));
    a.out = out;
    a.block_tables = block_tables;
    a.items = items;
    a.max_blocks_per_seq = max_blocks_per_seq;
    a.heads = heads;
    a.rank = rank;
    a.panels = page_width / 64;
    a.block_size = block_size;
    a.window = window;
    a.scale_log2 = scale * 1.4426950408889634f;
    const FewPlan few = fw_plan(item_tokens * heads, rank, page_width);
    const int tile_rows = few.n ? few.n : kLaRows;
    a.row_tiles = (item_tokens * heads + tile_rows - 1) / tile_rows;
    const dim3 grid(n_items * a.row_tiles, few.n ? 1 : (rank + kLaValues - 1) / kLaValues, n_splits < 1 ? 1 : n_splits);
    a.n_splits = static_cast<int>(grid.z);
    if (a.n_splits > 1) {
        HDS_REQUIRE(static_cast<int64_t>(grid.x) * grid.y * grid.z <= kLaMaxUnits, "hds_paged_attention_latent: split launches of at most 148 CTAs");
        HDS_REQUIRE(workspace != nullptr && workspace_bytes >= hds_paged_attention_latent_workspace_bytes(),
                    "hds_paged_attention_latent: workspace too small");
        char* ws = static_cast<char*>(workspace);
        a.tickets = reinterpret_cast<int32_t*>(ws);
        a.ws_ml = reinterpret_cast<float*>(ws + 4096);
        a.ws_o = a.ws_ml + static_cast<int64_t>(kLaMaxUnits) * kLaRows * 2;
    }
    const int kt = few.n ? 64 : la_tile(a.panels);
    CUtensorMap tq, tk;
    int rc = make_tmap_2d_16b(&tq, q, page_width, static_cast<uint64_t>(T) * heads, static_cast<uint64_t>(page_width) * 2, 64, tile_rows, dtype == 0);
    if (rc) return rc;
    rc = make_tmap_2d_16b(&tk, pages, page_width, static_cast<uint64_t>(num_blocks) * block_size, static_cast<uint64_t>(page_width) * 2, 64, kt,
                          dtype == 0);
    if (rc) return rc;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (few.n) {
        FewArgs f;
        a.n_stages = few.stages;
        f.l = a;
        f.v_blocks = (rank + 127) / 128;
        f.stage_panels = few.stage_panels;
        const size_t smem = (few.n == 64 ? fw_fixed_smem<64>(a.panels) : fw_fixed_smem<32>(a.panels)) +
                            static_cast<size_t>(few.stages) * few.stage_panels * kFwPanel;
        if (few.n == 64) return dtype == 0 ? launch_few<true, 64>(tq, tk, f, smem, grid, s) : launch_few<false, 64>(tq, tk, f, smem, grid, s);
        return dtype == 0 ? launch_few<true, 32>(tq, tk, f, smem, grid, s) : launch_few<false, 32>(tq, tk, f, smem, grid, s);
    }
    if (kt == 64) return dtype == 0 ? launch_latent<true, 64>(tq, tk, a, grid, s) : launch_latent<false, 64>(tq, tk, a, grid, s);
    return dtype == 0 ? launch_latent<true, 32>(tq, tk, a, grid, s) : launch_latent<false, 32>(tq, tk, a, grid, s);
}
