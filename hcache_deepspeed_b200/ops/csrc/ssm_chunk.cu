// Chunked state-space scan on the tensor cores (prompts). One CTA walks one head of one sequence in chunks of 128 tokens and
// carries the head's state in TMEM. With a_i the running sum of decay_rate * dt inside the chunk (log2 units):
//
//   CB  = C B^T                                                   [token, token]     tcgen05, both operands from the tiles
//   M   = CB * 2^(a_i - a_j) * dt_j  for j <= i (+ d for j = i)   fp32 in registers, written as two bf16 terms; 0 for j > i
//   y_i = (M x)_i + 2^(a_i) (C S)_i                               tcgen05 (M hi, M lo, S hi, S lo), combined in fp32
//   S  <- 2^(a_last) S + B^T (dt_j 2^(a_last - a_j) x_j)          tcgen05 into the fp32 state in TMEM (weighted x as two terms)
//
// x, B and C are 16-bit already (outputs of the convolution), so they enter exactly; everything fp32 that meets them in a
// product — M, the state, the weighted inputs — is split into a bf16 value and the bf16 rest, which keeps 16 significant
// bits of it, and accumulates in fp32. The carried state itself never leaves fp32.
//
//   warp 0     : TMA producer — C, B and x tiles (128 tokens x 64-column panels, SWIZZLE_128B)
//   warp 1     : TMEM allocation, tcgen05.mma issue
//   warps 2-9  : the state's chain — running sums, two-term copy of the state, weighted inputs
//   warps 10-17: M and the output                            (both groups: two threads per TMEM lane, one per column half)
//
// The chain of the state runs ahead of the other one: while M of chunk c is formed and multiplied, chunk c + 1 already updates
// the state. M replaces CB in TMEM (fp32 columns become the two bf16 terms) and is the A operand of its product from there.
// Accumulators: CB / M and C S twice, M x and the state once = all 512 TMEM columns.
#include "ssm.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kChTok = 128, kChThreads = 576, kChPanel = kChTok * 128;   // a panel: 128 rows of 128 bytes
constexpr int kChP = 64;                                                // head columns per CTA

constexpr size_t kChSmem = 2 * 2 * kChPanel /*C: two buffers*/ + 2 * 2 * kChPanel /*B: two buffers*/ + 2 * kChPanel /*x: two buffers*/ +
                           2 * kChPanel /*S hi, lo*/ + 2 * kChPanel /*W hi, lo*/ +
                           2 * 2 * kChTok * 4 /*a, b: two buffers*/ + 256;

__device__ __forceinline__ float ch_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// two values as packed bf16 pairs: leading terms and what they leave
__device__ __forceinline__ void ch_split(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - bf16_lo(hi), v1 - bf16_hi(hi));
}
// 16-byte chunk c (8 values) of row r in a 128-byte-swizzled panel
__device__ __forceinline__ uint4* ch_cell(uint8_t* panel, int r, int c) {
    return reinterpret_cast<uint4*>(panel + r * 128 + ((c ^ (r & 7)) << 4));
}

__global__ void __launch_bounds__(kChThreads, 1)
ssm_chunk_kernel(const __grid_constant__ CUtensorMap tmap_u, const SsmArgs a) {
    constexpr uint32_t kTmem = 512;
    constexpr uint32_t IDESC_CB = make_idesc_f16(128, 128, true, false, false);
    constexpr uint32_t IDESC_KN = make_idesc_f16(128, kChP, true, false, true);   // A K-major, B MN-major
    constexpr uint32_t IDESC_NN = make_idesc_f16(128, kChP, true, true, true);    // both MN-major

    extern __shared__ __align__(1024) uint8_t smem[];   // (no room for alignment slack: the tiles need 1024-byte bases)
    uint8_t* c_sm = smem;
    uint8_t* b_sm = c_sm + 4 * kChPanel;    // (C, B, x: two buffers each)
    uint8_t* x_sm = b_sm + 4 * kChPanel;
    uint8_t* s_sm = x_sm + 2 * kChPanel;    // hi, lo: rows = state index, 64 head columns
    uint8_t* w_sm = s_sm + 2 * kChPanel;    // hi, lo: rows = tokens, 64 head columns
    float* a_s = reinterpret_cast<float*>(w_sm + 2 * kChPanel);   // [2][128]: a_j
    float* b_s = a_s + 2 * kChTok;                                // [2][128]: a_j - log2(dt_j)
    uint64_t* bar = reinterpret_cast<uint64_t*>(b_s + 2 * kChTok);
    uint64_t *cb_full = bar + 23 /*[2]*/, *s_done = bar, *s_full = bar + 2, *w_full = bar + 3, *y_free = bar + 4, *st_done = bar + 5,
             *y_done = bar + 6, *x_full = bar + 7 /*[2] from here on*/, *x_empty = bar + 9, *ab_full = bar + 11, *ab_empty = bar + 13,
             *cb_done = bar + 15, *m_full = bar + 17, *cb_empty = bar + 19;
    float* warp_tot = reinterpret_cast<float*>(bar + 25);   // [2][4] sums of 32 tokens each
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(warp_tot + 8);

    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const uint32_t warp = warp_id(), lane = lane_id();
    const int h = blockIdx.y, p0 = blockIdx.z * kChP, N = a.N, P = a.P, H = a.heads;
    const int g = h / (H / a.groups), inner = a.inner();
    const int n_chunks = (sp.n + kChTok - 1) / kChTok;
    const int panels = (N + 63) / 64;

    if (warp == 0 && lane == 0) {
        prefetch_tmap(&tmap_u);
        mbar_init(s_done, 1);
        mbar_init(s_full, 8);
        mbar_init(w_full, 8);
        mbar_init(y_free, 8);
        mbar_init(st_done, 1);
        mbar_init(y_done, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(x_full + i, 1);
            mbar_init(x_empty + i, 1);
            mbar_init(ab_full + i, 4);
            mbar_init(ab_empty + i, 8);
            mbar_init(cb_done + i, 1);
            mbar_init(m_full + i, 8);
            mbar_init(cb_full + i, 1);
            mbar_init(cb_empty + i, 1);
        }
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc<kTmem>(tmem_slot);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const uint32_t t_cb = tmem /*[2]: CB, then M (per 16 tokens: 8 columns hi, 8 lo)*/, t_y1 = tmem + 256, t_y2 = tmem + 320 /*[2]*/, t_st = tmem + 448;

    if (warp == 0) {
        if (lane == 0) {
            for (int c = 0; c < n_chunks; ++c) {
                const int row = sp.row0 + c * kChTok;
                const int ph = c & 1;
                const uint32_t before = ((c >> 1) - 1) & 1;      // phase of what a two-buffer barrier saw two chunks ago
                if (c > 1) mbar_wait(cb_empty + ph, before);
                mbar_expect_tx(cb_full + ph, 2 * panels * kChPanel);
                for (int p = 0; p < panels; ++p) {
                    tma_load_2d(b_sm + (2 * ph + p) * kChPanel, &tmap_u, cb_full + ph, inner + g * N + p * 64, row, kEvictNormal);
                    tma_load_2d(c_sm + (2 * ph + p) * kChPanel, &tmap_u, cb_full + ph, inner + (a.groups + g) * N + p * 64, row, kEvictNormal);
                }
                if (c > 1) mbar_wait(x_empty + ph, before);
                mbar_expect_tx(x_full + ph, kChPanel);
                tma_load_2d(x_sm + ph * kChPanel, &tmap_u, x_full + ph, h * P + p0, row, kEvictNormal);
            }
        }
    } else if (warp == 1) {
        {   // the whole warp walks the schedule, one elected lane issues
            const bool leader = elect_one();
            // one thread issues every product: descriptors are formed once, a step only moves their address field (16-byte units)
            constexpr uint64_t PANEL = kChPanel >> 4, ROWS16 = (16 * 128) >> 4;
            const int k_steps = N / 16;
            const uint64_t d_c = make_desc_kmajor_sw128(smem_u32(c_sm)), d_s = make_desc_mnmajor_sw128(smem_u32(s_sm), kChPanel),
                           d_w = make_desc_mnmajor_sw128(smem_u32(w_sm), kChPanel);
            const uint64_t d_bk = make_desc_kmajor_sw128(smem_u32(b_sm)), d_bn = make_desc_mnmajor_sw128(smem_u32(b_sm), kChPanel),
                           d_x = make_desc_mnmajor_sw128(smem_u32(x_sm), kChPanel);
            auto m_times_x = [&](int c) {   // Y1 = M x
                const int ph = c & 1;
                mbar_wait(x_full + ph, (c >> 1) & 1);
                mbar_wait(m_full + ph, (c >> 1) & 1);
                if (c > 0) mbar_wait(y_free, ph ^ 1);     // Y1 (and Y2) of the chunk before have been read
                tc_fence_after();
                const uint32_t tm = t_cb + ph * 128;
                const uint64_t dx = d_x + ph * PANEL;
                if (leader) {
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kChTok / 16; ++kk)
                        umma_f16_ts(t_y1, tm + kk * 16 + t * 8, dx + kk * ROWS16, IDESC_KN, (t > 0 || kk > 0) ? 1u : 0u);
                umma_commit(y_done);
                umma_commit(x_empty + ph);
                }
                __syncwarp();
            };
            for (int c = 0; c < n_chunks; ++c) {
                const uint32_t ph = c & 1;
                const uint64_t dbk = d_bk + 2 * ph * PANEL, dbn = d_bn + 2 * ph * PANEL, dc = d_c + 2 * ph * PANEL;
                const uint32_t tc = t_cb + ph * 128, ty = t_y2 + ph * 64;
                // ---- CB = C B^T ---- (over M of chunk c - 2, whose product must be complete)
                if (c > 1) mbar_wait(y_done, ph);
                mbar_wait(cb_full + ph, (c >> 1) & 1);
                tc_fence_after();
                if (leader) {
#pragma unroll
                for (int kk = 0; kk < 8; ++kk)
                    if (kk < k_steps)
                        umma_f16_ss(tc, dc + (kk >> 2) * PANEL + 2 * (kk & 3), dbk + (kk >> 2) * PANEL + 2 * (kk & 3), IDESC_CB, kk > 0 ? 1u : 0u);
                umma_commit(cb_done + ph);
                }
                __syncwarp();
                if (c > 0) m_times_x(c - 1);
                // ---- S += B^T W ---- (S already scaled in place): the state's chain goes first
                mbar_wait(w_full, ph);
                tc_fence_after();
                if (leader) {
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kChTok / 16; ++kk)
                        umma_f16_ss(t_st, dbn + kk * ROWS16, d_w + t * PANEL + kk * ROWS16, IDESC_NN, 1u);
                umma_commit(st_done);
                }
                __syncwarp();
                // ---- Y2 = C S, with the state before the update (its two-term copy) ---- (Y2 of chunk c - 2 has been read: see above)
                mbar_wait(s_full, ph);
                tc_fence_after();
                if (leader) {
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < 8; ++kk)
                        if (kk < k_steps)
                            umma_f16_ss(ty, dc + (kk >> 2) * PANEL + 2 * (kk & 3), d_s + t * PANEL + kk * ROWS16, IDESC_KN, (t > 0 || kk > 0) ? 1u : 0u);
                umma_commit(s_done);
                umma_commit(cb_empty + ph);
                }
                __syncwarp();
            }
            m_times_x(n_chunks - 1);
        }
    } else if (warp < 10) {
        // ===================== the state's chain: thread = (token r of the chunk and state index, column half) =====================
        const int quad = warp & 3, half = (warp - 2) >> 2;
        const int r = quad * 32 + lane;
        const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
        const float rate = a.a[h] * 1.4426950408889634f;
        float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
        auto arrive = [&](uint64_t* b) {
            tc_fence_before();
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(b);
        };
        float dt_next = r < min(kChTok, sp.n) ? a.dt[static_cast<int64_t>(sp.row0 + r) * H + h] : 0.0f;
        for (int c = 0; c < n_chunks; ++c) {
            const uint32_t ph = c & 1;
            // ---- running log decays of the chunk (rows behind the end count nothing; both halves compute them) ----
            float dt;
            asm volatile("mov.b32 %0, %1;" : "=f"(dt) : "f"(dt_next));     // (keeps the wait for the load of a chunk ago down here)
            float run = rate * dt;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, run, o);
                if (static_cast<int>(lane) >= o) run += up;
            }
            float* tot = warp_tot + ph * 4;
            if (half == 0 && lane == 31) tot[quad] = run;
            asm volatile("bar.sync 1, 256;" ::: "memory");
            float a_last = 0.0f;
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                if (q == quad) run += a_last;
                a_last += tot[q];
            }
            const float b_mine = run - __log2f(dt);    // dt = 0 behind the end: infinite, its weights are zero
            if (half == 0) {
                if (c > 1) mbar_wait(ab_empty + ph, ((c >> 1) - 1) & 1);
                a_s[ph * kChTok + r] = run;
                b_s[ph * kChTok + r] = b_mine;
                __syncwarp();
                if (lane == 0) mbar_arrive(ab_full + ph);
            }
            const int next = (c + 1) * kChTok + r;
            dt_next = next < sp.n ? a.dt[static_cast<int64_t>(sp.row0 + next) * H + h] : 0.0f;
            const float keep = ch_ex2(a_last), wj = ch_ex2(a_last - b_mine);
            // ---- the state, scaled in place for its update (registers keep the unscaled values) ----
            uint32_t sw[32];
            if (c == 0) {
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    const int p = p0 + half * 32 + j;
                    sw[j] = __float_as_uint((sp.seen > 0 && p < P && r < N) ? st[static_cast<int64_t>(p) * N + r] : 0.0f);
                }
            } else {
                mbar_wait(st_done, ph ^ 1);
                tc_fence_after();
                tmem_ld_32x32(t_st + la + half * 32, sw);
                tmem_ld_wait();
            }
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                uint32_t sc[16];
#pragma unroll
                for (int j = 0; j < 16; ++j) sc[j] = __float_as_uint(__uint_as_float(sw[part * 16 + j]) * keep);
                tmem_st_32x16(t_st + la + half * 32 + part * 16, sc);
            }
            // ---- weighted inputs of the update ----
            mbar_wait(x_full + ph, (c >> 1) & 1);
            uint8_t* xt = x_sm + ph * kChPanel;
#pragma unroll
            for (int ch = 0; ch < 4; ++ch) {
                const uint4 x = *ch_cell(xt, r, half * 4 + ch);
                uint4 hi, lo;
                ch_split(wj * bf16_lo(x.x), wj * bf16_hi(x.x), hi.x, lo.x);
                ch_split(wj * bf16_lo(x.y), wj * bf16_hi(x.y), hi.y, lo.y);
                ch_split(wj * bf16_lo(x.z), wj * bf16_hi(x.z), hi.z, lo.z);
                ch_split(wj * bf16_lo(x.w), wj * bf16_hi(x.w), hi.w, lo.w);
                *ch_cell(w_sm, r, half * 4 + ch) = hi;
                *ch_cell(w_sm + kChPanel, r, half * 4 + ch) = lo;
            }
            tmem_st_wait();
            arrive(w_full);
            // ---- two-term copy of the state before the update, for C S ----
            if (c > 0) mbar_wait(s_done, ph ^ 1);     // (the previous copy has been multiplied)
#pragma unroll
            for (int ch = 0; ch < 4; ++ch) {
                uint4 hi, lo;
                ch_split(__uint_as_float(sw[8 * ch + 0]), __uint_as_float(sw[8 * ch + 1]), hi.x, lo.x);
                ch_split(__uint_as_float(sw[8 * ch + 2]), __uint_as_float(sw[8 * ch + 3]), hi.y, lo.y);
                ch_split(__uint_as_float(sw[8 * ch + 4]), __uint_as_float(sw[8 * ch + 5]), hi.z, lo.z);
                ch_split(__uint_as_float(sw[8 * ch + 6]), __uint_as_float(sw[8 * ch + 7]), hi.w, lo.w);
                *ch_cell(s_sm, r, half * 4 + ch) = hi;
                *ch_cell(s_sm + kChPanel, r, half * 4 + ch) = lo;
            }
            arrive(s_full);
        }
        mbar_wait(st_done, (n_chunks - 1) & 1);
        tc_fence_after();
        uint32_t sw[32];
        tmem_ld_32x32(t_st + la + half * 32, sw);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
            const int p = p0 + half * 32 + j;
            if (p < P && r < N) st[static_cast<int64_t>(p) * N + r] = __uint_as_float(sw[j]);
        }
        tc_fence_before();
    } else {
        // ===================== M and the output: thread = (token r of the chunk, column half) =====================
        const int quad = warp & 3, half = (warp - 10) >> 2;
        const int r = quad * 32 + lane;
        const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
        const float skip = a.d[h];
        auto output = [&](int c, float a_mine) {     // of chunk c
            mbar_wait(y_done, c & 1);
            tc_fence_after();
            const float grow = ch_ex2(a_mine);
            const bool live = r < min(kChTok, sp.n - c * kChTok);
            float* yo = a.y + static_cast<int64_t>(sp.row0 + c * kChTok + r) * inner + h * P + p0 + half * 32;
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                uint32_t y1[16], y2[16];
                tmem_ld_32x16(t_y1 + la + half * 32 + part * 16, y1);
                tmem_ld_32x16(t_y2 + (c & 1) * 64 + la + half * 32 + part * 16, y2);
                tmem_ld_wait();
                if (part == 1) {
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(y_free);
                }
#pragma unroll
                for (int ch = 0; ch < 2; ++ch) {
                    float o[8];
#pragma unroll
                    for (int j = 0; j < 8; ++j) o[j] = fmaf(grow, __uint_as_float(y2[8 * ch + j]), __uint_as_float(y1[8 * ch + j]));
                    const int col = part * 16 + ch * 8;
                    if (live && p0 + half * 32 + col < P) st_v8_f32(yo + col, o);      // P is a multiple of 8
                }
            }
            __syncwarp();
        };
        float a_prev = 0.0f;
        for (int c = 0; c < n_chunks; ++c) {
            const uint32_t ph = c & 1;
            mbar_wait(ab_full + ph, (c >> 1) & 1);
            const float a_mine = a_s[ph * kChTok + r];
            const float* bv = b_s + ph * kChTok;
            mbar_wait(cb_done + ph, (c >> 1) & 1);
            tc_fence_after();
            // in place, 16 columns at a time: 16 fp32 values become 8 columns of leading terms and 8 of what they leave
            const uint32_t t_m = t_cb + ph * 128 + la;
#pragma unroll 1
            for (int part = 0; part < 4; ++part) {
                const int jp = half * 64 + part * 16;
                uint32_t m[16];
                if (jp > quad * 32 + 16) {        // every column lies in the future
#pragma unroll
                    for (int j = 0; j < 16; ++j) m[j] = 0u;
                } else {
                    uint32_t cb[16];
                    tmem_ld_32x16(t_m + jp, cb);
                    tmem_ld_wait();
                    float v[16];
#pragma unroll
                    for (int j = 0; j < 16; j += 4) {
                        const float4 b = *reinterpret_cast<const float4*>(bv + jp + j);
                        v[j + 0] = __uint_as_float(cb[j + 0]) * ch_ex2(a_mine - b.x);
                        v[j + 1] = __uint_as_float(cb[j + 1]) * ch_ex2(a_mine - b.y);
                        v[j + 2] = __uint_as_float(cb[j + 2]) * ch_ex2(a_mine - b.z);
                        v[j + 3] = __uint_as_float(cb[j + 3]) * ch_ex2(a_mine - b.w);
                    }
                    if (jp >= quad * 32) {       // the diagonal: later columns out, the skip connection in
                        const int mine = r - jp;
#pragma unroll
                        for (int j = 0; j < 16; ++j) v[j] = j > mine ? 0.0f : j == mine ? v[j] + skip : v[j];
                    }
#pragma unroll
                    for (int j = 0; j < 8; ++j) ch_split(v[2 * j], v[2 * j + 1], m[j], m[8 + j]);
                }
                tmem_st_32x16(t_m + jp, m);
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
                mbar_arrive(ab_empty + ph);
                mbar_arrive(m_full + ph);
            }
            if (c > 0) output(c - 1, a_prev);
            a_prev = a_mine;
        }
        output(n_chunks - 1, a_prev);
        if (blockIdx.z == 0) ssm_save_conv_of_head<0>(a, sp, h, threadIdx.x - 320, 256);
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<kTmem>(tmem);
    }
}

bool ssm_chunk_supported(const SsmArgs& a, int dtype) {
    return dtype == 0 && a.N % 16 == 0 && a.N <= 128 && a.P % 8 == 0 && (a.P <= kChP || a.P % kChP == 0) && a.ld_u % 8 == 0 &&
           (reinterpret_cast<uintptr_t>(a.u) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.y) & 31) == 0;
}

int ssm_chunk_launch(const SsmArgs& a, int dtype, cudaStream_t s) {
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!configured[dev & 63]) {
        HDS_CHECK_CUDA(cudaFuncSetAttribute(ssm_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kChSmem)));
        configured[dev & 63] = true;
    }
    CUtensorMap tm;
    const int rc = make_tmap_2d_16b(&tm, a.u, static_cast<uint64_t>(a.channels()), static_cast<uint64_t>(a.T),
                                    static_cast<uint64_t>(a.ld_u) * 2, 64, kChTok, dtype == 0);
    if (rc) return rc;
    const dim3 grid(a.n_seqs, a.heads, (a.P + kChP - 1) / kChP);
    HDS_CHECK_CUDA(launch_kernel(ssm_chunk_kernel, grid, dim3(kChThreads), kChSmem, s, tm, a));
    return HDS_OK;
}

}  // namespace hds
