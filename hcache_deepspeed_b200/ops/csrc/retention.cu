// Retention over a ragged batch, per head:  S <- decay S + v k^T,  o = S q  (q and k turned by position), then o / rms(o) * silu(gate).
// Sequences with one new token are stepped, and batches whose q and k still have to be turned scanned, by the kernels of
// linear_attention.cu. Prompts of bf16 models, whose projection has turned them already, run here on tcgen05, 128 tokens at a time. With S
// the state in front of a chunk and d the head's decay:
//
//   o_i = d^(i + 1) S q_i + sum_{j <= i} d^(i - j) (q_i . k_j) v_j          S <- d^n S + sum_j d^(n - 1 - j) v_j k_j^T
//
//   ret_state : per (sequence, head, 32 values): walks the chunks with the state in TMEM and leaves the state in front of every chunk in the
//               workspace; advances the state pool
//   ret_out   : per (chunk, head): scores, state and value products, norm and gate. Persistent blocks
//
// q, k and v enter products exactly as they are. Everything fp32 that becomes an operand (decayed values, decayed scores, the state) is a bf16
// value plus the bf16 rest, 16 significant bits; sums are fp32 in TMEM, the carried state is never rounded. A state in the workspace is N rows
// of P leading terms and P rests, which TMA reads as two tiles. Long batches run in segments, which bounds the workspace.
#include "linear_attention.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kRtTok = 128, kRtP = 128, kRtPanel = kRtTok * 128;       // a panel: 128 rows of 128 bytes
constexpr uint64_t kRtRows16 = (16 * 128) >> 4;     // 16 rows of a panel, in descriptor units

//: set when a wait ran out (a fault of the kernels' own protocol); read by hds_retention_status
__device__ int g_ret_stuck = 0;

// Wait for a phase; gives up after about a second, records it and never waits again.
__device__ __forceinline__ void rt_wait(uint64_t* bar, uint32_t parity, bool& stuck) {
    if (stuck || mbar_try_wait(bar, parity)) return;
    const long long t0 = clock64();
    for (uint32_t probes = 1; !mbar_try_wait(bar, parity); ++probes) {
        if ((probes & 1023u) == 0 && clock64() - t0 > (1ll << 31)) {
            stuck = true;
            g_ret_stuck = 1;
            return;
        }
    }
}
__device__ __forceinline__ float rt_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rt_rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rt_silu(float g) { return g * rt_rcp(1.0f + rt_ex2(g * -1.4426950408889634f)); }
__device__ __forceinline__ void rt_split(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - bf16_lo(hi), v1 - bf16_hi(hi));
}
__device__ __forceinline__ void rt_store32(void* p, const uint32_t (&v)[8]) {
    asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]),
                 "r"(v[5]), "r"(v[6]), "r"(v[7])
                 : "memory");
}
// 16-byte piece c (8 values) of row r in a swizzled panel
__device__ __forceinline__ uint4* rt_cell(uint8_t* panel, int r, int c) { return reinterpret_cast<uint4*>(panel + r * 128 + ((c ^ (r & 7)) << 4)); }

struct RetWs {
    uint16_t* s;        // [chunks][heads][N][2 P]: states in front of the chunks (see above), or nullptr: not wanted
    int c0, n;          // chunks [c0, c0 + n) of the batch
};
struct RetMaps {
    CUtensorMap q, k, v, s;     // [T][heads * N] twice, [T][heads * P]; [cells * N][2 P] rows of states
};

// ret_state: warp 0 loads keys, warp 1 issues products, 8 warps keep the chain (a thread: a key channel of the state, half of the 32
// columns), 8 warps decay values (a thread: a token, half of the columns), ahead of it. Between two products lies only the state's own
// decay; the state in front of a chunk is written out while the chunk's product runs.
constexpr int kRsP = 32, kRsThreads = 64 + 2 * 256, kRsStages = 4;
__host__ __device__ constexpr size_t rt_state_smem(int N) { return static_cast<size_t>(kRsStages * (N / 64) + 2 * 2) * kRtPanel + 1024; }

template <int N>
__global__ void __launch_bounds__(kRsThreads, 1) ret_state_kernel(const __grid_constant__ RetMaps maps, const LinArgs a, const RetWs ws) {
    constexpr int KP = N / 64;
    extern __shared__ uint8_t smem_raw[];
    __shared__ uint64_t k_full[kRsStages], k_free[kRsStages], w_full[2], w_free[2], s_ready, s_done;
    __shared__ uint32_t tmem_slot;
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int total = span_chunks(sp, kRtTok), base = first_chunk(a.spans, blockIdx.x, kRtTok);
    const int i0 = max(0, ws.c0 - base), n_chunks = min(total, ws.c0 + ws.n - base) - i0;       // those of the segment
    if (n_chunks <= 0) return;
    const int P = a.P, h = blockIdx.y, p0 = blockIdx.z * kRsP;
    uint8_t* k_sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));     // [stages]
    uint8_t* w_sm = k_sm + kRsStages * KP * kRtPanel;       // [2][leading terms, rests]: 32 of a panel's columns
    const uint32_t warp = warp_id(), lane = lane_id();
    bool stuck = false;
    if (threadIdx.x == 0) {
        for (int i = 0; i < kRsStages; ++i) {
            mbar_init(k_full + i, 1);
            mbar_init(k_free + i, 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(w_full + i, 8);
            mbar_init(w_free + i, 1);
        }
        mbar_init(&s_ready, 8);
        mbar_init(&s_done, 1);
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc<32>(&tmem_slot);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    if (warp == 0) {
        if (lane == 0) {
            for (int c = 0; c < n_chunks; ++c) {
                const int b = c % kRsStages;
                if (c >= kRsStages) rt_wait(k_free + b, (c / kRsStages - 1) & 1, stuck);
                mbar_expect_tx(k_full + b, KP * kRtPanel);
                for (int p = 0; p < KP; ++p)
                    tma_load_2d(k_sm + (b * KP + p) * kRtPanel, &maps.k, k_full + b, h * N + p * 64, sp.row0 + (i0 + c) * kRtTok, kEvictNormal);
            }
        }
    } else if (warp == 1) {
        const bool leader = elect_one();
        constexpr uint32_t idesc = make_idesc_f16(128, kRsP, true, true, true);     // S [N][32] += K^T V, both operands as they lie (tokens are rows)
        constexpr uint64_t PANEL = kRtPanel >> 4;
        const uint64_t d_k = make_desc_mnmajor_sw128(smem_u32(k_sm), kRtPanel), d_w = make_desc_mnmajor_sw128(smem_u32(w_sm), kRtPanel);
        for (int c = 0; c < n_chunks; ++c) {
            const int b = c & 1, kb = c % kRsStages;
            rt_wait(k_full + kb, (c / kRsStages) & 1, stuck);
            rt_wait(w_full + b, (c >> 1) & 1, stuck);
            rt_wait(&s_ready, c & 1, stuck);
            tc_fence_after();
            if (leader) {
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kRtTok / 16; ++kk)
                        umma_f16_ss(tmem, d_k + kb * KP * PANEL + kk * kRtRows16, d_w + (2 * b + t) * PANEL + kk * kRtRows16, idesc, 1u);
                umma_commit(&s_done);
                umma_commit(w_free + b);
                umma_commit(k_free + kb);
            }
            __syncwarp();
        }
    } else if (warp < 10) {
        const int quad = warp & 3, half = (warp - 2) >> 2, r = quad * 32 + lane, p = p0 + half * 16;
        const uint32_t t_s = tmem + (static_cast<uint32_t>(quad * 32) << 16) + half * 16;
        const bool mine = r < N && p < P;       // (P is a multiple of 16)
        const float ld = a.log2_decay[h];
        float* st = a.state + ((static_cast<int64_t>(sp.slot) * a.heads + h) * P + p) * N + r;
        uint32_t sw[16];
        for (int c = 0; c < n_chunks; ++c) {
            if (c == 0) {
#pragma unroll
                for (int j = 0; j < 16; ++j) sw[j] = __float_as_uint((sp.seen > 0 || i0 > 0) && mine ? st[static_cast<int64_t>(j) * N] : 0.0f);
            } else {
                rt_wait(&s_done, (c - 1) & 1, stuck);
                __syncwarp();
                tc_fence_after();
                tmem_ld_32x16(t_s, sw);
                tmem_ld_wait();
            }
            const float keep = rt_ex2(ld * static_cast<float>(min(kRtTok, sp.n - (i0 + c) * kRtTok)));
            uint32_t sc[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) sc[j] = __float_as_uint(__uint_as_float(sw[j]) * keep);
            tmem_st_32x16(t_s, sc);
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_ready);
            if (ws.s != nullptr && mine) {
                uint32_t hi[8], lo[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) rt_split(__uint_as_float(sw[2 * j]), __uint_as_float(sw[2 * j + 1]), hi[j], lo[j]);
                uint16_t* dst = ws.s + ((static_cast<int64_t>(base + i0 + c - ws.c0) * a.heads + h) * N + r) * 2 * P + p;
                rt_store32(dst, hi);        // whole sectors
                rt_store32(dst + P, lo);
            }
        }
        rt_wait(&s_done, (n_chunks - 1) & 1, stuck);
        __syncwarp();
        tc_fence_after();
        tmem_ld_32x16(t_s, sw);
        tmem_ld_wait();
        tc_fence_before();
        if (mine)
#pragma unroll
            for (int j = 0; j < 16; ++j) st[static_cast<int64_t>(j) * N] = __uint_as_float(sw[j]);
    } else {
        const int quad = warp & 3, half = (warp - 10) >> 2, r = quad * 32 + lane, p = p0 + half * 16;
        const float ld = a.log2_decay[h];
        constexpr int U = 3;        // chunks whose values are on their way
        uint4 x[U][2];
        auto fetch = [&](int c, uint4 (&v)[2]) {       // this token's values
            const int t = (i0 + c) * kRtTok + r;
            v[0] = v[1] = make_uint4(0, 0, 0, 0);
            if (c < n_chunks && t < sp.n && p < P) {
                const uint4* src = reinterpret_cast<const uint4*>(static_cast<const char*>(a.v) +
                                                                 (static_cast<int64_t>(sp.row0 + t) * a.ld + static_cast<int64_t>(h) * P + p) * 2);
                v[0] = ld_nc_v4(src);
                v[1] = ld_nc_v4(src + 1);
            }
        };
#pragma unroll
        for (int u = 0; u < U; ++u) fetch(u, x[u]);
        for (int c0 = 0; c0 < n_chunks; c0 += U) {
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int c = c0 + u;
                if (c >= n_chunks) break;
                const int n = min(kRtTok, sp.n - (i0 + c) * kRtTok);
                const float w = r < n ? a.k_scale * rt_ex2(ld * static_cast<float>(n - 1 - r)) : 0.0f;      // faded to the end of the chunk
                uint8_t* hi_p = w_sm + (c & 1) * 2 * kRtPanel;
                if (c > 1) rt_wait(w_free + (c & 1), ((c >> 1) - 1) & 1, stuck);
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    const uint4 v = x[u][g];
                    uint4 hi, lo;
                    rt_split(w * bf16_lo(v.x), w * bf16_hi(v.x), hi.x, lo.x);
                    rt_split(w * bf16_lo(v.y), w * bf16_hi(v.y), hi.y, lo.y);
                    rt_split(w * bf16_lo(v.z), w * bf16_hi(v.z), hi.z, lo.z);
                    rt_split(w * bf16_lo(v.w), w * bf16_hi(v.w), hi.w, lo.w);
                    *rt_cell(hi_p, r, half * 2 + g) = hi;
                    *rt_cell(hi_p + kRtPanel, r, half * 2 + g) = lo;
                }
                fence_proxy_async_smem();
                __syncwarp();
                if (lane == 0) mbar_arrive(w_full + (c & 1));
                fetch(c + U, x[u]);
            }
        }
    }
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<32>(tmem);
    }
}

// ret_out: warp 0 loads, warp 1 issues products, 16 warps form weights and outputs (a thread: a row and a quarter of its columns).
// q and k have two buffers, v and the state one (two of each up to 64 channels); scores and outputs have two places in TMEM, so that the
// products of one item run under the arithmetic of the other.
constexpr int kRtOutWarps = 16, kRtOutThreads = 64 + kRtOutWarps * 32;
__host__ __device__ constexpr int rt_stages(int N) { return N == 64 ? 2 : 1; }
__host__ __device__ constexpr size_t rt_out_smem(int N) {
    return static_cast<size_t>(2 * 2 * (N / 64) + rt_stages(N) * (2 + 2 * (N / 64))) * kRtPanel + 256 + 4 * kRtTok * 4;
}

struct RtItem {
    int row, n, h, p0, Pb, cell;
    bool fresh, valid;      // fresh: nothing in front, the state is zero
};
// Item number `index`: (chunk of the segment, head, block of values), by a whole warp.
__device__ __forceinline__ RtItem rt_item(const LinArgs& a, const RetWs& ws, int index, int blocks) {
    const int lane = threadIdx.x & 31, per = a.heads * blocks, local = index / per, rest = index - local * per;
    const int target = ws.c0 + local;
    int base = 0, seq = -1, chunk = 0;
    for (int s0 = 0; s0 < a.n_seqs && seq < 0; s0 += 32) {
        const int s = s0 + lane, mine = s < a.n_seqs ? span_chunks(a.spans[s], kRtTok) : 0;
        int incl = mine;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, target < base + incl);
        if (hit) {
            const int l = __ffs(hit) - 1;
            seq = s0 + l;
            chunk = target - base - __shfl_sync(0xffffffffu, incl - mine, l);
        }
        base += __shfl_sync(0xffffffffu, incl, 31);
    }
    RtItem it;
    it.valid = seq >= 0;
    const SsmSpan sp = a.spans[max(seq, 0)];
    it.row = sp.row0 + chunk * kRtTok;
    it.n = min(kRtTok, sp.n - chunk * kRtTok);
    it.fresh = sp.seen == 0 && chunk == 0;
    it.h = rest / blocks;
    it.p0 = (rest - it.h * blocks) * kRtP;
    it.Pb = min(kRtP, a.P - it.p0);
    it.cell = local * a.heads + it.h;
    return it;
}

template <int N>
__global__ void __launch_bounds__(kRtOutThreads, 1)
ret_out_kernel(const __grid_constant__ RetMaps maps, const LinArgs a, const RetWs ws, const int items, const int blocks) {
    constexpr int KP = N / 64, VS = rt_stages(N), SPANEL = N * 128;
    extern __shared__ __align__(1024) uint8_t smem[];       // (no room for alignment slack: the tiles need 1024-byte bases)
    pdl_enter();
    uint8_t* qk_sm = smem;                                  // [2][q, k]
    uint8_t* v_sm = qk_sm + 4 * KP * kRtPanel;              // [VS][2 panels]
    uint8_t* s_sm = v_sm + VS * 2 * kRtPanel;               // [VS][leading terms, rests][2 panels of N rows]
    uint64_t* bars = reinterpret_cast<uint64_t*>(s_sm + VS * 2 * KP * kRtPanel);     // two of each
    uint64_t *qk_full = bars, *qk_free = bars + 2, *v_full = bars + 4, *v_free = bars + 6, *s_full = bars + 8, *s_free = bars + 10,
             *sc_done = bars + 12, *y_done = bars + 14, *o_done = bars + 16, *a_full = bars + 18, *t_free = bars + 20;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 22);
    float* ss_s = reinterpret_cast<float*>(bars + 32);      // [4][128]
    const uint32_t warp = warp_id(), lane = lane_id();
    if ((smem_u32(smem) & 1023u) != 0u) {
        g_ret_stuck = 2;
        return;
    }
    if (threadIdx.x == 0) {
        for (int i = 0; i < 18; ++i) mbar_init(bars + i, 1);
        for (int i = 18; i < 22; ++i) mbar_init(bars + i, kRtOutWarps);
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc<512>(tmem_slot);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;       // twice: scores, then their two terms (per 16 tokens: 8 columns each); output
    bool stuck = false;
    const int stride = gridDim.x;

    if (warp == 0) {
        const bool leader = elect_one();
        int i = 0, si = 0;      // items; items with a state
        auto load_qk = [&](const RtItem& it, int k) {
            if (k > 1) rt_wait(qk_free + (k & 1), ((k >> 1) - 1) & 1, stuck);
            if (leader) {
                uint8_t* q = qk_sm + (k & 1) * 2 * KP * kRtPanel;
                mbar_expect_tx(qk_full + (k & 1), 2 * KP * kRtPanel);
                for (int p = 0; p < KP; ++p) {
                    tma_load_2d(q + p * kRtPanel, &maps.q, qk_full + (k & 1), it.h * N + p * 64, it.row, kEvictNormal);
                    tma_load_2d(q + (KP + p) * kRtPanel, &maps.k, qk_full + (k & 1), it.h * N + p * 64, it.row, kEvictNormal);
                }
            }
            __syncwarp();
        };
        RtItem it, next;
        next.valid = false;
        int at = blockIdx.x;
        if (at < items) next = rt_item(a, ws, at, blocks);
        if (next.valid) load_qk(next, 0);
        while (next.valid) {
            it = next;
            at += stride;
            next.valid = false;
            if (at < items) next = rt_item(a, ws, at, blocks);
            if (next.valid) load_qk(next, i + 1);
            if (!it.fresh) {
                const int b = si % VS;
                if (si >= VS) rt_wait(s_free + b, (si / VS - 1) & 1, stuck);
                if (leader) {
                    uint8_t* s = s_sm + b * 4 * SPANEL;
                    const int panels = (it.Pb + 63) >> 6;       // (columns past the head's own values are never used)
                    mbar_expect_tx(s_full + b, 2 * panels * SPANEL);
                    for (int t = 0; t < 2; ++t)
                        for (int p = 0; p < panels; ++p)
                            tma_load_2d(s + (2 * t + p) * SPANEL, &maps.s, s_full + b, t * a.P + it.p0 + p * 64, it.cell * N, kEvictFirst);
                }
                __syncwarp();
                ++si;
            }
            const int b = i % VS, panels = (it.Pb + 63) >> 6;
            if (i >= VS) rt_wait(v_free + b, (i / VS - 1) & 1, stuck);
            if (leader) {
                mbar_expect_tx(v_full + b, panels * kRtPanel);
                for (int p = 0; p < panels; ++p)
                    tma_load_2d(v_sm + (2 * b + p) * kRtPanel, &maps.v, v_full + b, it.h * a.P + it.p0 + p * 64, it.row, kEvictNormal);
            }
            __syncwarp();
            ++i;
        }
    } else if (warp == 1) {
        const bool leader = elect_one();
        constexpr uint64_t PANEL = kRtPanel >> 4;
        constexpr uint32_t IDESC_QK = make_idesc_f16(128, 128, true, false, false);
        const uint64_t d_qk = make_desc_kmajor_sw128(smem_u32(qk_sm)), d_s = make_desc_mnmajor_sw128(smem_u32(s_sm), SPANEL),
                       d_v = make_desc_mnmajor_sw128(smem_u32(v_sm), kRtPanel);
        int i = 0, si = 0;
        bool prev_fresh = false;
        int prev_pb = 0;
        auto values = [&](int k, bool fresh, int pb) {     // output += weights of item k times its values
            const int b = k & 1, vb = k % VS;
            rt_wait(v_full + vb, (k / VS) & 1, stuck);
            rt_wait(a_full + b, (k >> 1) & 1, stuck);
            tc_fence_after();
            const uint32_t t_a = tmem + b * 256;
            const uint32_t idesc = make_idesc_f16(128, pb, true, false, true);
            if (leader) {
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kRtTok / 16; ++kk)
                        umma_f16_ts(t_a + 128, t_a + kk * 16 + t * 8, d_v + 2 * vb * PANEL + kk * kRtRows16, idesc, (!fresh || t > 0 || kk > 0) ? 1u : 0u);
                umma_commit(o_done + b);
                umma_commit(v_free + vb);
            }
            __syncwarp();
        };
        for (int at = blockIdx.x; at < items; at += stride) {
            const RtItem it = rt_item(a, ws, at, blocks);
            if (!it.valid) break;
            const int b = i & 1;
            const uint32_t t_a = tmem + b * 256;
            const uint64_t dq = d_qk + b * 2 * KP * PANEL, dk = dq + KP * PANEL;
            rt_wait(qk_full + b, (i >> 1) & 1, stuck);
            if (i > 1) rt_wait(t_free + b, ((i >> 1) - 1) & 1, stuck);       // (its output has been read)
            tc_fence_after();
            if (leader) {
#pragma unroll
                for (int kk = 0; kk < N / 16; ++kk) {
                    const uint64_t o = (kk >> 2) * PANEL + 2 * (kk & 3);
                    umma_f16_ss(t_a, dq + o, dk + o, IDESC_QK, kk > 0 ? 1u : 0u);
                }
                umma_commit(sc_done + b);
            }
            __syncwarp();
            if (!it.fresh) {
                const int sb = si % VS;
                rt_wait(s_full + sb, (si / VS) & 1, stuck);
                tc_fence_after();
                const uint32_t idesc = make_idesc_f16(128, it.Pb, true, false, true);
                if (leader) {
#pragma unroll
                    for (int t = 0; t < 2; ++t)
#pragma unroll
                        for (int kk = 0; kk < N / 16; ++kk) {
                            const uint64_t o = (kk >> 2) * PANEL + 2 * (kk & 3);
                            umma_f16_ss(t_a + 128, dq + o, d_s + (2 * sb + t) * (2 * SPANEL >> 4) + kk * kRtRows16, idesc, (t > 0 || kk > 0) ? 1u : 0u);
                        }
                    umma_commit(y_done + b);
                    umma_commit(s_free + sb);
                }
                __syncwarp();
                ++si;
            }
            if (leader) umma_commit(qk_free + b);
            __syncwarp();
            if (i > 0) values(i - 1, prev_fresh, prev_pb);
            prev_fresh = it.fresh;
            prev_pb = it.Pb;
            ++i;
        }
        if (i > 0) values(i - 1, prev_fresh, prev_pb);
    } else {
        const int quad = warp & 3, part0 = (warp - 2) >> 2, r = quad * 32 + lane;
        const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
        int i = 0, yc[2] = {0, 0};      // items; those with a state, by place
        auto output = [&](const RtItem& it, int k) {
            const int b = k & 1, n_blocks = it.Pb >> 4;
            const bool live = r < it.n;
            const uint32_t t_y = tmem + b * 256 + 128 + la;
            const int64_t col = static_cast<int64_t>(it.h) * a.P + it.p0;
            uint4 gate[2][2];
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int blk = part0 + 4 * x;
                gate[x][0] = gate[x][1] = make_uint4(0, 0, 0, 0);
                if (!a.write_y && live && blk < n_blocks) {
                    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const char*>(a.gate) + ((it.row + r) * a.ld + col + blk * 16) * 2);
                    gate[x][0] = src[0];
                    gate[x][1] = src[1];
                }
            }
            rt_wait(o_done + b, (k >> 1) & 1, stuck);
            __syncwarp();
            tc_fence_after();
            float o[2][16], ss = 0.0f;
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int blk = part0 + 4 * x;
                uint32_t y[16];
                if (blk < n_blocks) {
                    tmem_ld_32x16(t_y + blk * 16, y);
                    tmem_ld_wait();
                }
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    o[x][j] = blk < n_blocks ? __uint_as_float(y[j]) : 0.0f;
                    ss = fmaf(o[x][j], o[x][j], ss);
                }
            }
            tc_fence_before();
            auto rows_sync = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + quad) : "memory"); };       // the four warps of these rows
            rows_sync();        // (the sums of the item before have been read)
            ss_s[part0 * kRtTok + r] = ss;
            __syncwarp();
            if (lane == 0) mbar_arrive(t_free + b);
            rows_sync();
            const float f = rsqrtf((ss_s[r] + ss_s[kRtTok + r] + ss_s[2 * kRtTok + r] + ss_s[3 * kRtTok + r]) / a.norm_cols + a.eps);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int blk = part0 + 4 * x;
                if (blk >= n_blocks || !live) continue;
                if (a.write_y) {
#pragma unroll
                    for (int j = 0; j < 16; j += 4)
                        *reinterpret_cast<float4*>(a.y + (it.row + r) * a.ld_y + col + blk * 16 + j) = make_float4(o[x][j], o[x][j + 1], o[x][j + 2], o[x][j + 3]);
                    continue;
                }
                const uint32_t gw[8] = {gate[x][0].x, gate[x][0].y, gate[x][0].z, gate[x][0].w, gate[x][1].x, gate[x][1].y, gate[x][1].z, gate[x][1].w};
                uint32_t res[8];
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    res[j] = pack_bf16(o[x][2 * j] * f * rt_silu(bf16_lo(gw[j])), o[x][2 * j + 1] * f * rt_silu(bf16_hi(gw[j])));
                char* dst = static_cast<char*>(a.out) + ((it.row + r) * a.ld_out + col + blk * 16) * 2;
                st_v4(dst, make_uint4(res[0], res[1], res[2], res[3]));
                st_v4(dst + 16, make_uint4(res[4], res[5], res[6], res[7]));
            }
        };
        RtItem prev;
        for (int at = blockIdx.x; at < items; at += stride) {
            const RtItem it = rt_item(a, ws, at, blocks);
            if (!it.valid) break;
            const int b = i & 1;
            const uint32_t t_a = tmem + b * 256 + la;
            const float ld = a.log2_decay[it.h], d = rt_ex2(ld);
            rt_wait(sc_done + b, (i >> 1) & 1, stuck);
            __syncwarp();
            tc_fence_after();
            // ---- scores, decayed, in place: 16 fp32 columns become 8 of leading terms and 8 of rests ----
#pragma unroll
            for (int part = part0; part < 8; part += 4) {
                const int j0 = part * 16;
                uint32_t m[16];
                if (j0 > quad * 32 + 31) {          // every column lies in the future
#pragma unroll
                    for (int j = 0; j < 16; ++j) m[j] = 0u;
                } else {
                    uint32_t x[16];
                    tmem_ld_32x16(t_a + j0, x);
                    tmem_ld_wait();
                    float v[16];
                    if (j0 + 15 > quad * 32) {      // the diagonal
#pragma unroll
                        for (int j = 0; j < 16; ++j) {
                            const int back = r - j0 - j;
                            v[j] = back < 0 ? 0.0f : __uint_as_float(x[j]) * (a.k_scale * rt_ex2(ld * static_cast<float>(back)));
                        }
                    } else {
                        float f = a.k_scale * rt_ex2(ld * static_cast<float>(r - j0 - 15));
#pragma unroll
                        for (int j = 15; j >= 0; --j) {
                            v[j] = __uint_as_float(x[j]) * f;
                            f *= d;
                        }
                    }
#pragma unroll
                    for (int j = 0; j < 8; ++j) rt_split(v[2 * j], v[2 * j + 1], m[j], m[8 + j]);
                }
                tmem_st_32x16(t_a + j0, m);
            }
            // ---- what the state gives, decayed, in place; the product with the values adds to it ----
            if (!it.fresh) {
                rt_wait(y_done + b, yc[b] & 1, stuck);
                ++yc[b];
                __syncwarp();
                tc_fence_after();
                const float g = rt_ex2(ld * static_cast<float>(r + 1));
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const int blk = part0 + 4 * x;
                    if (blk >= it.Pb >> 4) break;
                    uint32_t y[16];
                    tmem_ld_32x16(t_a + 128 + blk * 16, y);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; ++j) y[j] = __float_as_uint(__uint_as_float(y[j]) * g);
                    tmem_st_32x16(t_a + 128 + blk * 16, y);
                }
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(a_full + b);
            if (i > 0) output(prev, i - 1);
            prev = it;
            ++i;
        }
        if (i > 0) output(prev, i - 1);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<512>(tmem);
    }
}

static int64_t rt_cell_bytes(int heads, int P, int N) { return static_cast<int64_t>(heads) * N * P * 4; }

// Chunks of a segment: as many as 512 MiB of intermediate values hold.
static int64_t rt_segment(int64_t chunks, int heads, int P, int N) {
    const int64_t n = (int64_t(512) << 20) / rt_cell_bytes(heads, P, N);
    return n >= chunks ? chunks : n > 0 ? n : 1;
}

static bool rt_chunk_supported(const LinArgs& a, int dtype, const void* ws, int64_t ws_bytes) {
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    return dtype == 0 && a.freq == nullptr && (a.N == 64 || a.N == 128) && a.P % 16 == 0 && ws != nullptr && ws_bytes >= rt_cell_bytes(a.heads, a.P, a.N) &&
           (reinterpret_cast<uintptr_t>(ws) & 31) == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) && aligned(a.gate) && aligned(a.out) &&
           aligned(a.state) && aligned(a.y) && a.ld % 8 == 0 && a.ld_qk % 8 == 0 && a.ld_out % 8 == 0 && a.ld_y % 4 == 0;
}

template <int N>
static int rt_chunk_launch(const LinArgs& a, int n_multi, void* ws, int64_t ws_bytes, cudaStream_t s) {
    const int64_t bound = a.T / kRtTok + n_multi;           // at least as many as there are chunks
    const int64_t fits = ws_bytes / rt_cell_bytes(a.heads, a.P, N), seg = rt_segment(bound, a.heads, a.P, N);
    const int step = static_cast<int>(seg < fits ? seg : fits);
    RetMaps m;
    const uint64_t T = static_cast<uint64_t>(a.T), keys = static_cast<uint64_t>(a.heads) * N, vals = static_cast<uint64_t>(a.heads) * a.P;
    int rc = make_tmap_2d_16b(&m.q, a.q, keys, T, static_cast<uint64_t>(a.ld_qk) * 2, 64, kRtTok, true);
    if (!rc) rc = make_tmap_2d_16b(&m.k, a.k, keys, T, static_cast<uint64_t>(a.ld_qk) * 2, 64, kRtTok, true);
    if (!rc) rc = make_tmap_2d_16b(&m.v, a.v, vals, T, static_cast<uint64_t>(a.ld) * 2, 64, kRtTok, true);
    if (!rc) rc = make_tmap_2d_16b(&m.s, ws, 2 * static_cast<uint64_t>(a.P), static_cast<uint64_t>(step) * keys, 4 * static_cast<uint64_t>(a.P), 64, N, true);
    if (rc) return rc;
    auto chain = ret_state_kernel<N>;
    auto out = ret_out_kernel<N>;
    HDS_CHECK_CUDA(cudaFuncSetAttribute(chain, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(rt_state_smem(N))));
    HDS_CHECK_CUDA(cudaFuncSetAttribute(out, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(rt_out_smem(N))));
    const unsigned blocks = (a.P + kRtP - 1) / kRtP;
    const bool reads = a.out != nullptr || a.write_y;
    for (int64_t c0 = 0; c0 < bound; c0 += step) {
        RetWs w;
        w.s = reads ? static_cast<uint16_t*>(ws) : nullptr;
        w.c0 = static_cast<int>(c0);
        w.n = static_cast<int>(step < bound - c0 ? step : bound - c0);
        HDS_CHECK_CUDA(launch_kernel(chain, dim3(a.n_seqs, a.heads, (a.P + kRsP - 1) / kRsP), dim3(kRsThreads), rt_state_smem(N), s, m, a, w));
        if (reads) {
            const int items = w.n * a.heads * static_cast<int>(blocks), sms = sm_count();
            HDS_CHECK_CUDA(launch_kernel(out, dim3(items < sms ? items : sms), dim3(kRtOutThreads), rt_out_smem(N), s, m, a, w, items, static_cast<int>(blocks)));
        }
    }
    return HDS_OK;
}

}  // namespace hds

using namespace hds;

extern "C" int64_t hds_retention_workspace_bytes(int T, int n_seqs, int heads, int vdim, int dim) {
    if ((dim != 64 && dim != 128) || vdim % 16 != 0) return 0;
    const int64_t all = T / kRtTok + (n_seqs < T / 2 ? n_seqs : T / 2);
    return rt_segment(all > 0 ? all : 1, heads, vdim, dim) * rt_cell_bytes(heads, vdim, dim);
}

extern "C" int hds_retention_status(int* stuck) {
    HDS_CHECK_CUDA(cudaMemcpyFromSymbol(stuck, g_ret_stuck, sizeof(int)));
    return HDS_OK;
}

// Returns in *finished 1 when out holds the finished rows, 0 when y holds the read-outs (out still to be normed and gated).
extern "C" int hds_retention(const void* q, const void* k, int64_t ld_qk, const void* v, const void* gate, int64_t ld, const float* log2_decay,
                             const float* freq, const float* amp, float k_scale, int norm_cols, float* state, const int32_t* spans, int n_seqs,
                             int n_single, int T, int heads, int vdim, int dim, float* y, int64_t ld_y, void* out, int64_t ld_out, float eps,
                             void* workspace, int64_t workspace_bytes, int method, int* finished, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_retention: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(heads >= 1 && vdim >= 1 && vdim <= 8192 && dim >= 2 && dim <= 1024 && dim % 2 == 0, "hds_retention: heads of up to 1024 x 8192");
    HDS_REQUIRE(norm_cols >= 1 && norm_cols <= vdim, "hds_retention: 1 <= norm_cols <= vdim");
    HDS_REQUIRE(method >= 0 && method <= 2, "hds_retention: method 0 / 1 / 2");
    *finished = 1;
    if (T == 0 || n_seqs == 0) return HDS_OK;
    LinArgs a{q, k, v, gate, ld, nullptr, 0, nullptr, 0.0f, state, reinterpret_cast<const SsmSpan*>(spans), n_seqs, T, heads, vdim, dim,
              y, ld_y, out, ld_out, nullptr, eps, 0, norm_cols, 1.0f, k_scale, ld_qk, log2_decay, freq, amp};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    int rc = HDS_OK;
    if (n_seqs > n_single) {
        const bool chunked = rt_chunk_supported(a, dtype, workspace, workspace_bytes);
        HDS_REQUIRE(method != 2 || chunked, "hds_retention: the chunked form does not take this shape");
        if (chunked && method != 1) {
            if (vdim > kRtP && out != nullptr) {    // heads of several blocks: the norm takes a pass of its own
                *finished = 0;
                a.write_y = 1;
            }
            rc = dim == 64 ? rt_chunk_launch<64>(a, n_seqs - n_single, workspace, workspace_bytes, s)
                           : rt_chunk_launch<128>(a, n_seqs - n_single, workspace, workspace_bytes, s);
        } else {
            *finished = 0;
            a.write_y = 1;      // by every row of the batch: one norm finishes them all
            rc = lin_launch_scan(a, dtype, true, s);
        }
    }
    if (rc != HDS_OK || n_single == 0) return rc;
    return lin_launch_step(a, dtype, true, s);
}
