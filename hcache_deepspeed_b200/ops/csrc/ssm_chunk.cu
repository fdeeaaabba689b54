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
//   warp 0    : TMA producer — C, B and x tiles (128 tokens x 64-column panels, SWIZZLE_128B)
//   warp 1    : TMEM allocation, tcgen05.mma issue
//   warps 2-9 : running sums, operand generation and output; two threads per TMEM lane (column halves). Per chunk: sums, state
//               operand, weighted inputs (the state's own chain of products can start), then the PREVIOUS chunk's output (its
//               products have run meanwhile), then M.
#include "ssm.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kChTok = 128, kChThreads = 320, kChPanel = kChTok * 128;   // a panel: 128 rows of 128 bytes
constexpr int kChP = 64;                                                // head columns per CTA

constexpr size_t kChSmem = 2 * 2 * kChPanel /*C, B*/ + 2 * kChPanel /*x*/ + 4 * kChPanel /*M hi, lo*/ + 2 * kChPanel /*S hi, lo*/ +
                           2 * kChPanel /*W hi, lo*/ + 2 * kChTok * 4 /*a, b*/ + 256 + 1024;

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

    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* c_sm = smem;
    uint8_t* b_sm = c_sm + 2 * kChPanel;
    uint8_t* x_sm = b_sm + 2 * kChPanel;
    uint8_t* m_sm = x_sm + 2 * kChPanel;    // (x: two buffers)  M hi: panels 0, 1; lo: panels 2, 3
    uint8_t* s_sm = m_sm + 4 * kChPanel;    // hi, lo: rows = state index, 64 head columns
    uint8_t* w_sm = s_sm + 2 * kChPanel;    // hi, lo: rows = tokens, 64 head columns
    float* b_s = reinterpret_cast<float*>(w_sm + 2 * kChPanel);   // [128]: a_j - log2(dt_j)
    float* a_s = b_s + kChTok;                                    // [128]: a_j
    uint64_t* bar = reinterpret_cast<uint64_t*>(b_s + 2 * kChTok);
    uint64_t *cb_full = bar, *cb_empty = bar + 1, *x_full = bar + 2 /*[2]*/, *x_empty = bar + 4 /*[2]*/, *s_full = bar + 6,
             *w_full = bar + 7, *m_full = bar + 8, *cb_done = bar + 9, *st_done = bar + 10, *y_done = bar + 11;
    float* warp_tot = reinterpret_cast<float*>(bar + 12);   // [4] sums of 32 tokens each
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(warp_tot + 4);

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
        mbar_init(cb_full, 1);
        mbar_init(cb_empty, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(x_full + i, 1);
            mbar_init(x_empty + i, 1);
        }
        mbar_init(s_full, 8);
        mbar_init(w_full, 8);
        mbar_init(m_full, 8);
        mbar_init(cb_done, 1);
        mbar_init(st_done, 1);
        mbar_init(y_done, 1);
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
    const uint32_t t_cb = tmem, t_y1 = tmem + 128, t_y2 = tmem + 192, t_st = tmem + 256;

    if (warp == 0) {
        if (lane == 0) {
            for (int c = 0; c < n_chunks; ++c) {
                const int row = sp.row0 + c * kChTok;
                if (c > 0) mbar_wait(cb_empty, (c - 1) & 1);
                mbar_expect_tx(cb_full, 2 * panels * kChPanel);
                for (int p = 0; p < panels; ++p) {
                    tma_load_2d(b_sm + p * kChPanel, &tmap_u, cb_full, inner + g * N + p * 64, row, kEvictNormal);
                    tma_load_2d(c_sm + p * kChPanel, &tmap_u, cb_full, inner + (a.groups + g) * N + p * 64, row, kEvictNormal);
                }
                const int xb = c & 1;
                if (c > 1) mbar_wait(x_empty + xb, ((c >> 1) - 1) & 1);
                mbar_expect_tx(x_full + xb, kChPanel);
                tma_load_2d(x_sm + xb * kChPanel, &tmap_u, x_full + xb, h * P + p0, row, kEvictNormal);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            for (int c = 0; c < n_chunks; ++c) {
                const uint32_t ph = c & 1;
                // ---- CB = C B^T ---- (its accumulator was read before the previous chunk's M was complete)
                mbar_wait(cb_full, ph);
                tc_fence_after();
                for (int kk = 0; kk < N / 16; ++kk)
                    umma_f16_ss(t_cb, make_desc_kmajor_sw128(smem_u32(c_sm + (kk >> 2) * kChPanel)) + 2 * (kk & 3),
                                make_desc_kmajor_sw128(smem_u32(b_sm + (kk >> 2) * kChPanel)) + 2 * (kk & 3), IDESC_CB, kk > 0 ? 1u : 0u);
                umma_commit(cb_done);
                // ---- S += B^T W ---- (S already scaled in place)
                mbar_wait(w_full, ph);
                tc_fence_after();
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kChTok / 16; ++kk)
                        umma_f16_ss(t_st, make_desc_mnmajor_sw128(smem_u32(b_sm + kk * 16 * 128), kChPanel),
                                    make_desc_mnmajor_sw128(smem_u32(w_sm + t * kChPanel + kk * 16 * 128), kChPanel), IDESC_NN, 1u);
                // ---- Y2 = C S, with the state before the update (its two-term copy) ----
                mbar_wait(s_full, ph);
                tc_fence_after();
#pragma unroll
                for (int t = 0; t < 2; ++t)
                    for (int kk = 0; kk < N / 16; ++kk)
                        umma_f16_ss(t_y2, make_desc_kmajor_sw128(smem_u32(c_sm + (kk >> 2) * kChPanel)) + 2 * (kk & 3),
                                    make_desc_mnmajor_sw128(smem_u32(s_sm + t * kChPanel + kk * 16 * 128), kChPanel), IDESC_KN,
                                    (t > 0 || kk > 0) ? 1u : 0u);
                umma_commit(st_done);
                umma_commit(cb_empty);
                // ---- Y1 = M x ----
                mbar_wait(m_full, ph);
                tc_fence_after();
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kChTok / 16; ++kk)
                        umma_f16_ss(t_y1, make_desc_kmajor_sw128(smem_u32(m_sm + (2 * t + (kk >> 2)) * kChPanel)) + 2 * (kk & 3),
                                    make_desc_mnmajor_sw128(smem_u32(x_sm + (c & 1) * kChPanel + kk * 16 * 128), kChPanel), IDESC_KN, (t > 0 || kk > 0) ? 1u : 0u);
                umma_commit(y_done);
                umma_commit(x_empty + (c & 1));
            }
        }
    } else {
        const int quad = warp & 3, half = (warp - 2) >> 2;
        const int r = quad * 32 + lane;            // token of the chunk, or state index
        const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
        const float rate = a.a[h] * 1.4426950408889634f, skip = a.d[h];
        float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
        auto all_compute = [] { asm volatile("bar.sync 1, 256;" ::: "memory"); };
        auto arrive = [&](uint64_t* b) {
            tc_fence_before();
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(b);
        };
        // Output of chunk c, whose products are complete: my row's 32 columns, staged through this warp's 32 rows of the first
        // M panel of its half (free until M of the next chunk is written) so that a store instruction covers four whole rows.
        auto output = [&](int c, float a_mine) {
            mbar_wait(y_done, c & 1);
            tc_fence_after();
            uint32_t y1[32], y2[32];
            tmem_ld_32x32(t_y1 + la + half * 32, y1);
            tmem_ld_32x32(t_y2 + la + half * 32, y2);
            tmem_ld_wait();
            const float grow = ch_ex2(a_mine);
            uint8_t* stage = m_sm + half * kChPanel;
#pragma unroll
            for (int ch = 0; ch < 8; ++ch) {
                uint4 o;
                o.x = __float_as_uint(fmaf(grow, __uint_as_float(y2[4 * ch + 0]), __uint_as_float(y1[4 * ch + 0])));
                o.y = __float_as_uint(fmaf(grow, __uint_as_float(y2[4 * ch + 1]), __uint_as_float(y1[4 * ch + 1])));
                o.z = __float_as_uint(fmaf(grow, __uint_as_float(y2[4 * ch + 2]), __uint_as_float(y1[4 * ch + 2])));
                o.w = __float_as_uint(fmaf(grow, __uint_as_float(y2[4 * ch + 3]), __uint_as_float(y1[4 * ch + 3])));
                *ch_cell(stage, r, ch) = o;
            }
            __syncwarp();
            const int nt = min(kChTok, sp.n - c * kChTok);
            const int ch = lane & 7, col = p0 + half * 32 + 4 * ch;
            float* yo = a.y + static_cast<int64_t>(sp.row0 + c * kChTok) * inner + h * P + col;
#pragma unroll
            for (int it = 0; it < 8; ++it) {
                const int i = quad * 32 + it * 4 + (lane >> 3);
                if (i < nt && col < P) *reinterpret_cast<uint4*>(yo + static_cast<int64_t>(i) * inner) = *ch_cell(stage, i, ch);
            }
            __syncwarp();
        };
        float dt = half == 0 && r < min(kChTok, sp.n) ? a.dt[static_cast<int64_t>(sp.row0 + r) * H + h] : 0.0f;
        float a_prev = 0.0f;
        for (int c = 0; c < n_chunks; ++c) {
            const uint32_t ph = c & 1;
            // ---- running log decays of the chunk (first column half; rows behind the end count nothing) ----
            float run = rate * dt;
            if (half == 0) {
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const float up = __shfl_up_sync(0xffffffffu, run, o);
                    if (static_cast<int>(lane) >= o) run += up;
                }
                if (lane == 31) warp_tot[quad] = run;
            }
            all_compute();
            if (half == 0) {
                for (int q = 0; q < quad; ++q) run += warp_tot[q];
                b_s[r] = run - log2f(dt);      // dt = 0 behind the end: infinite, its weights are zero
                a_s[r] = run;
                const int next = (c + 1) * kChTok + r;
                dt = next < sp.n ? a.dt[static_cast<int64_t>(sp.row0 + next) * H + h] : 0.0f;
            }
            all_compute();
            const float a_last = a_s[kChTok - 1], a_mine = a_s[r];
            // ---- state: two-term copy for C S, scaled copy for the update ----
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
            for (int ch = 0; ch < 4; ++ch) {
                uint4 hi, lo;
                ch_split(__uint_as_float(sw[8 * ch + 0]), __uint_as_float(sw[8 * ch + 1]), hi.x, lo.x);
                ch_split(__uint_as_float(sw[8 * ch + 2]), __uint_as_float(sw[8 * ch + 3]), hi.y, lo.y);
                ch_split(__uint_as_float(sw[8 * ch + 4]), __uint_as_float(sw[8 * ch + 5]), hi.z, lo.z);
                ch_split(__uint_as_float(sw[8 * ch + 6]), __uint_as_float(sw[8 * ch + 7]), hi.w, lo.w);
                *ch_cell(s_sm, r, half * 4 + ch) = hi;
                *ch_cell(s_sm + kChPanel, r, half * 4 + ch) = lo;
            }
            const float keep = ch_ex2(a_last);
#pragma unroll
            for (int j = 0; j < 32; ++j) sw[j] = __float_as_uint(__uint_as_float(sw[j]) * keep);
            tmem_st_32x32(t_st + la + half * 32, sw);
            tmem_st_wait();
            // ---- weighted inputs of the state update ----
            mbar_wait(x_full + ph, (c >> 1) & 1);
            const float wj = ch_ex2(a_last - b_s[r]);
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
            // ---- the previous chunk's output: behind it, Y1 and Y2 may be overwritten ----
            arrive(w_full);
            if (c > 0) output(c - 1, a_prev);
            a_prev = a_mine;
            arrive(s_full);
            // ---- M: my row's 64 columns (all of them in the future for the upper right quarter) ----
            mbar_wait(cb_done, ph);
            tc_fence_after();
            uint8_t* m_hi = m_sm + half * kChPanel;
            uint8_t* m_lo = m_sm + (2 + half) * kChPanel;
#pragma unroll 1
            for (int part = 0; part < 2; ++part) {
                const int jp = half * 64 + part * 32;
                if (jp > quad * 32) {        // every column lies in the future
#pragma unroll
                    for (int ch = 0; ch < 4; ++ch) {
                        *ch_cell(m_hi, r, part * 4 + ch) = make_uint4(0, 0, 0, 0);
                        if (c == 0) *ch_cell(m_lo, r, part * 4 + ch) = make_uint4(0, 0, 0, 0);   // (never used for staging)
                    }
                    continue;
                }
                uint32_t cb[32];
                tmem_ld_32x32(t_cb + la + jp, cb);
                tmem_ld_wait();
                float v[32];
#pragma unroll
                for (int j = 0; j < 32; j += 4) {
                    const float4 b = *reinterpret_cast<const float4*>(b_s + jp + j);
                    v[j + 0] = __uint_as_float(cb[j + 0]) * ch_ex2(a_mine - b.x);
                    v[j + 1] = __uint_as_float(cb[j + 1]) * ch_ex2(a_mine - b.y);
                    v[j + 2] = __uint_as_float(cb[j + 2]) * ch_ex2(a_mine - b.z);
                    v[j + 3] = __uint_as_float(cb[j + 3]) * ch_ex2(a_mine - b.w);
                }
                if (jp == quad * 32) {       // the diagonal: later columns out, the skip connection in
#pragma unroll
                    for (int j = 0; j < 32; ++j) v[j] = j > static_cast<int>(lane) ? 0.0f : j == static_cast<int>(lane) ? v[j] + skip : v[j];
                }
#pragma unroll
                for (int ch = 0; ch < 4; ++ch) {
                    uint4 hi, lo;
                    ch_split(v[8 * ch + 0], v[8 * ch + 1], hi.x, lo.x);
                    ch_split(v[8 * ch + 2], v[8 * ch + 3], hi.y, lo.y);
                    ch_split(v[8 * ch + 4], v[8 * ch + 5], hi.z, lo.z);
                    ch_split(v[8 * ch + 6], v[8 * ch + 7], hi.w, lo.w);
                    *ch_cell(m_hi, r, part * 4 + ch) = hi;
                    *ch_cell(m_lo, r, part * 4 + ch) = lo;
                }
            }
            arrive(m_full);
        }
        output(n_chunks - 1, a_prev);
        // (all products are complete: the last commit tracks every one before it)
        uint32_t sw[32];
        tmem_ld_32x32(t_st + la + half * 32, sw);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
            const int p = p0 + half * 32 + j;
            if (p < P && r < N) st[static_cast<int64_t>(p) * N + r] = __uint_as_float(sw[j]);
        }
        if (blockIdx.z == 0) ssm_save_conv_of_head<0>(a, sp, h, threadIdx.x - 64, 256);
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
           (reinterpret_cast<uintptr_t>(a.u) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.y) & 15) == 0;
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
