// Gated delta rule of prompts on the tensor cores, 128 tokens at a time. With a_i the running sum of log2 decays inside a chunk, unit
// keys k and queries q, and S the state in front of the chunk, the recurrence of the whole chunk is one triangular system:
//
//   A_ij = beta_i 2^(a_i - a_j) (k_i . k_j)  for j < i                      (I + A) U = R
//   R_i  = beta_i (v_i - 2^(a_i) S^T k_i)                                   U_i: what token i writes along its key
//   o_i  = 2^(a_i) S^T q_i + sum_{j <= i} 2^(a_i - a_j) (q_i . k_j) U_j
//   S   <- 2^(a_last) S + sum_j 2^(a_last - a_j) k_j U_j^T
//
//   delta_prep  : per (chunk, head), independent of the state and so of all other chunks: decays, step sizes, norms, K K^T on tcgen05,
//                 and the inverse of I + A in fp32 (32 x 32 diagonal blocks by substitution, then blocks of 32 and 64 by products);
//                 stored as two bf16 terms
//   delta_chunk : per (sequence, head, 64 value columns), chunk after chunk with the fp32 state in TMEM
//
// k, q and v enter products as the convolution's 16-bit outputs, exactly; their norms are fp32 factors of rows and columns. Everything
// fp32 that becomes an operand (the state, R, U, the inverse, decayed scores) is a bf16 value plus the bf16 rest: 16 significant bits.
//
// delta_chunk's warps
//   0     : TMA producer — k (two buffers), q and v tiles
//   1     : TMEM allocation, tcgen05.mma issue
//   2-9   : the state's chain — two-term state, R, U
//   10-17 : inverse -> TMEM, decayed scores in TMEM, output                 (both groups: two threads per TMEM lane)
// The chain runs ahead: the output of a chunk is formed while the next one already solves for its U.
// TMEM: scores 128 columns, inverse 128, S^T k and then U 64, scores x U 64, S^T q 64, state 64.
#include "delta.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kDcTok = 128, kDcPanel = kDcTok * 128, kDcP = 64;
constexpr int kDcThreads = 576, kPrepThreads = 256, kPrepPitch = 132;
// the inverse in memory: 16 pieces of leading terms and 16 of rests, a piece = 8 neighbouring values of every row
constexpr int kInvPiece = kDcTok * 16;
constexpr int64_t kInvBytes = 32 * kInvPiece;

struct DeltaWs {
    uint8_t* inv;      // [chunks][heads][32 pieces][128 rows][16 B]
    float* a;          // [T][heads]: running log2 decay inside the token's chunk
    float* beta;       // [T][heads]
    float* rk;         // [T][groups]: 1 / |k|
    float* rq;         // [T][groups]: dim^-1/2 / |q|
};

__device__ __forceinline__ float dc_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// two values as packed bf16 pairs: leading terms and what they leave
__device__ __forceinline__ void dc_split(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - bf16_lo(hi), v1 - bf16_hi(hi));
}
__device__ __forceinline__ uint4* dc_cell(uint8_t* panel, int r, int c) {   // 16-byte chunk c of row r in a swizzled panel
    return reinterpret_cast<uint4*>(panel + r * 128 + ((c ^ (r & 7)) << 4));
}
__device__ __forceinline__ int dc_chunks(const SsmSpan& s) { return s.n > 1 ? (s.n + kDcTok - 1) / kDcTok : 0; }

// ---- per chunk and head -------------------------------------------------------------------------------------------------
constexpr size_t kPrepSmem = static_cast<size_t>(kDcTok) * kPrepPitch * 4 /*k panels, then A*/ + 3 * kDcTok * 4 + 64;
static_assert(2 * kDcPanel <= kDcTok * kPrepPitch * 4, "A replaces the key panels");

__global__ void __launch_bounds__(kPrepThreads, 3)
delta_prep_kernel(const __grid_constant__ CUtensorMap tmap_u, const SsmArgs a, const DeltaWs ws) {
    extern __shared__ __align__(1024) uint8_t smem[];
    uint8_t* k_sm = smem;                                           // two panels, until K K^T is done
    float* A = reinterpret_cast<float*>(smem);                      // [128][kPrepPitch]: A, then the inverse in place
    float* tmp = A + 64;                                            // products' intermediates: the quarter above the diagonal
    float* a_s = A + kDcTok * kPrepPitch;
    float* b_s = a_s + kDcTok;
    float* r_s = b_s + kDcTok;
    uint64_t* full = reinterpret_cast<uint64_t*>(r_s + kDcTok);
    uint64_t* done = full + 1;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
    __shared__ int where[2];                                        // sequence, chunk inside it
    __shared__ float warp_tot[4];
    pdl_enter();
    const int tid = threadIdx.x, h = blockIdx.y;
    const uint32_t warp = warp_id(), lane = lane_id();
    if (warp == 0) {        // which chunk is number blockIdx.x
        int base = 0, seq = -1, chunk = 0;
        for (int s0 = 0; s0 < a.n_seqs && seq < 0; s0 += 32) {
            const int s = s0 + static_cast<int>(lane);
            const int mine = s < a.n_seqs ? dc_chunks(a.spans[s]) : 0;
            int incl = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, o);
                if (static_cast<int>(lane) >= o) incl += up;
            }
            const unsigned hit = __ballot_sync(0xffffffffu, static_cast<int>(blockIdx.x) < base + incl);
            if (hit) {
                const int l = __ffs(hit) - 1;
                seq = s0 + l;
                chunk = static_cast<int>(blockIdx.x) - base - __shfl_sync(0xffffffffu, incl - mine, l);
            }
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (lane == 0) {
            where[0] = seq;
            where[1] = chunk;
        }
    }
    if (tid == 0) {
        prefetch_tmap(&tmap_u);
        mbar_init(full, 1);
        mbar_init(done, 1);
        fence_barrier_init();
    }
    __syncthreads();
    if (where[0] < 0) return;
    const SsmSpan sp = a.spans[where[0]];
    const int N = a.N, H = a.heads, g = h / (H / a.groups), inner = a.inner();
    const int row = sp.row0 + where[1] * kDcTok, n = min(kDcTok, sp.n - where[1] * kDcTok);
    if (warp == 1) {
        tmem_alloc<128>(tmem_slot);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const int panels = (N + 63) / 64;
    if (tid == 0) {
        mbar_expect_tx(full, panels * kDcPanel);
        for (int p = 0; p < panels; ++p) tma_load_2d(k_sm + p * kDcPanel, &tmap_u, full, inner + g * N + p * 64, row, kEvictNormal);
        mbar_wait(full, 0);
        tc_fence_after();
        constexpr uint32_t IDESC = make_idesc_f16(128, 128, true, false, false);
        const uint64_t d = make_desc_kmajor_sw128(smem_u32(k_sm));
        for (int kk = 0; kk < N / 16; ++kk) {
            const uint64_t dk = d + (kk >> 2) * (kDcPanel >> 4) + 2 * (kk & 3);
            umma_f16_ss(tmem, dk, dk, IDESC, kk > 0 ? 1u : 0u);
        }
        umma_commit(done);
    }
    __syncwarp();
    if (tid < kDcTok) {     // running decays and step sizes
        const bool live = tid < n;
        float run = live ? a.a[h] * 1.4426950408889634f * a.dt[static_cast<int64_t>(row + tid) * H + h] : 0.0f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (static_cast<int>(lane) >= o) run += up;
        }
        if (lane == 31) warp_tot[warp] = run;
        asm volatile("bar.sync 1, 128;" ::: "memory");
        for (uint32_t w = 0; w < warp; ++w) run += warp_tot[w];
        const float beta = live ? delta_beta<0>(a, row + tid, h) : 0.0f;
        a_s[tid] = run;
        b_s[tid] = beta;
        if (live) {
            ws.a[static_cast<int64_t>(row + tid) * H + h] = run;
            ws.beta[static_cast<int64_t>(row + tid) * H + h] = beta;
        }
    } else if (h % (H / a.groups) == 0) {      // the group's query norms
        const int t = tid - kDcTok;
        if (t < n) {
            const char* q = reinterpret_cast<const char*>(a.u) + (static_cast<int64_t>(row + t) * a.ld_u + inner + (a.groups + g) * N) * 2;
            float ss = 0.0f;
            for (int i = 0; i < N / 8; ++i) {
                const uint4 v = *reinterpret_cast<const uint4*>(q + i * 16);
                ss += bf16_lo(v.x) * bf16_lo(v.x) + bf16_hi(v.x) * bf16_hi(v.x) + bf16_lo(v.y) * bf16_lo(v.y) + bf16_hi(v.y) * bf16_hi(v.y) +
                      bf16_lo(v.z) * bf16_lo(v.z) + bf16_hi(v.z) * bf16_hi(v.z) + bf16_lo(v.w) * bf16_lo(v.w) + bf16_hi(v.w) * bf16_hi(v.w);
            }
            ws.rq[static_cast<int64_t>(row + t) * a.groups + g] = rsqrtf(static_cast<float>(N)) / sqrtf(ss + kUnitEps);
        }
    }
    // ---- K K^T -> norms (its diagonal) -> A ----
    const int quad = warp & 3, half = warp >> 2, r = quad * 32 + lane;
    mbar_wait(done, 0);
    tc_fence_after();
    const uint32_t t_row = tmem + (static_cast<uint32_t>(quad * 32) << 16);
    if (quad / 2 == half) {      // (uniform in a warp)
        uint32_t s[32];
        tmem_ld_32x32(t_row + quad * 32, s);
        tmem_ld_wait();
        float kk = 0.0f;
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (j == static_cast<int>(lane)) kk = __uint_as_float(s[j]);
        {
            const float rk = 1.0f / sqrtf(kk + kUnitEps);
            r_s[r] = rk;
            if (r < n && h % (H / a.groups) == 0) ws.rk[static_cast<int64_t>(row + r) * a.groups + g] = rk;
        }
    }
    __syncthreads();
    {
        const float f = r < n ? b_s[r] * r_s[r] : 0.0f, ar = a_s[r];
#pragma unroll 1
        for (int j0 = half * 64; j0 < half * 64 + 64; j0 += 16) {
            float* row_out = A + r * kPrepPitch + j0;
            if (j0 > quad * 32 + 31) {      // all above the diagonal
#pragma unroll
                for (int j = 0; j < 16; j += 4) *reinterpret_cast<float4*>(row_out + j) = make_float4(0.f, 0.f, 0.f, 0.f);
                continue;
            }
            uint32_t s[16];
            tmem_ld_32x16(t_row + j0, s);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; j += 4) {
                const float4 rk = *reinterpret_cast<const float4*>(r_s + j0 + j), aj = *reinterpret_cast<const float4*>(a_s + j0 + j);
                float4 v;
                v.x = j0 + j + 0 < r ? f * rk.x * dc_ex2(ar - aj.x) * __uint_as_float(s[j + 0]) : 0.0f;
                v.y = j0 + j + 1 < r ? f * rk.y * dc_ex2(ar - aj.y) * __uint_as_float(s[j + 1]) : 0.0f;
                v.z = j0 + j + 2 < r ? f * rk.z * dc_ex2(ar - aj.z) * __uint_as_float(s[j + 2]) : 0.0f;
                v.w = j0 + j + 3 < r ? f * rk.w * dc_ex2(ar - aj.w) * __uint_as_float(s[j + 3]) : 0.0f;
                *reinterpret_cast<float4*>(row_out + j) = v;
            }
        }
    }
    __syncthreads();
    // ---- diagonal 32 x 32 blocks of the inverse: lane = column, substitution down the rows ----
    if (warp < 4) {
        float* D = A + warp * 32 * kPrepPitch + warp * 32;
        float x[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
            float v0 = static_cast<int>(lane) == i ? 1.0f : 0.0f, v1 = 0.0f, v2 = 0.0f, v3 = 0.0f;
#pragma unroll
            for (int j = 0; j < i; j += 4) {
                const float4 l = *reinterpret_cast<const float4*>(D + i * kPrepPitch + j);      // (zero on and above the diagonal)
                v0 = fmaf(-l.x, x[j], v0);
                if (j + 1 < i) v1 = fmaf(-l.y, x[j + 1], v1);
                if (j + 2 < i) v2 = fmaf(-l.z, x[j + 2], v2);
                if (j + 3 < i) v3 = fmaf(-l.w, x[j + 3], v3);
            }
            x[i] = (v0 + v1) + (v2 + v3);
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 32; ++i) D[i * kPrepPitch + lane] = x[i];
    }
    __syncthreads();
    // ---- blocks below the diagonal: X21 = -X22 (A21 X11), sizes 32 then 64 ----
    {   // two 32 x 32 blocks at once: threads 0-127 and 128-255, 4 x 2 values each
        const int b = tid >> 7, t = tid & 127, i0 = (t >> 4) * 4, j0 = (t & 15) * 2;
        float* X11 = A + b * 64 * kPrepPitch + b * 64;
        float* X21 = X11 + 32 * kPrepPitch;
        float* X22 = X21 + 32;
        float* T1 = tmp + b * 32;
        for (int step = 0; step < 2; ++step) {
            float acc[4][2] = {};
            const float* L = step == 0 ? X21 : X22;
            const float* R = step == 0 ? X11 : T1;
#pragma unroll 2
            for (int k = 0; k < (step == 0 ? 32 : i0 + 4); k += 4) {      // (X22 is zero above its diagonal)
                float2 w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) w[e] = *reinterpret_cast<const float2*>(R + (k + e) * kPrepPitch + j0);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float4 l = *reinterpret_cast<const float4*>(L + (i0 + i) * kPrepPitch + k);
                    acc[i][0] = fmaf(l.x, w[0].x, acc[i][0]); acc[i][1] = fmaf(l.x, w[0].y, acc[i][1]);
                    acc[i][0] = fmaf(l.y, w[1].x, acc[i][0]); acc[i][1] = fmaf(l.y, w[1].y, acc[i][1]);
                    acc[i][0] = fmaf(l.z, w[2].x, acc[i][0]); acc[i][1] = fmaf(l.z, w[2].y, acc[i][1]);
                    acc[i][0] = fmaf(l.w, w[3].x, acc[i][0]); acc[i][1] = fmaf(l.w, w[3].y, acc[i][1]);
                }
            }
            if (step == 1) __syncthreads();
#pragma unroll
            for (int i = 0; i < 4; ++i)
                *reinterpret_cast<float2*>((step == 0 ? T1 : X21) + (i0 + i) * kPrepPitch + j0) =
                    step == 0 ? make_float2(acc[i][0], acc[i][1]) : make_float2(-acc[i][0], -acc[i][1]);
            __syncthreads();
        }
    }
    {
        const int i0 = (tid >> 4) * 4, j0 = (tid & 15) * 4;
        float* X21 = A + 64 * kPrepPitch;
        float* X22 = X21 + 64;
        for (int step = 0; step < 2; ++step) {
            float acc[4][4] = {};
            const float* L = step == 0 ? X21 : X22;
            const float* R = step == 0 ? A : tmp;
#pragma unroll 2
            for (int k = 0; k < (step == 0 ? 64 : i0 + 4); k += 4) {
                float4 w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) w[e] = *reinterpret_cast<const float4*>(R + (k + e) * kPrepPitch + j0);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float4 l4 = *reinterpret_cast<const float4*>(L + (i0 + i) * kPrepPitch + k);
                    const float l[4] = {l4.x, l4.y, l4.z, l4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        acc[i][0] = fmaf(l[e], w[e].x, acc[i][0]);
                        acc[i][1] = fmaf(l[e], w[e].y, acc[i][1]);
                        acc[i][2] = fmaf(l[e], w[e].z, acc[i][2]);
                        acc[i][3] = fmaf(l[e], w[e].w, acc[i][3]);
                    }
                }
            }
            if (step == 1) __syncthreads();
#pragma unroll
            for (int i = 0; i < 4; ++i)
                *reinterpret_cast<float4*>((step == 0 ? tmp : X21) + (i0 + i) * kPrepPitch + j0) =
                    step == 0 ? make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3])
                              : make_float4(-acc[i][0], -acc[i][1], -acc[i][2], -acc[i][3]);
            __syncthreads();
        }
    }
    // ---- two-term copy ----
    uint8_t* dst = ws.inv + (static_cast<int64_t>(blockIdx.x) * H + h) * kInvBytes;
    for (int e = tid; e < kDcTok * 16; e += kPrepThreads) {      // 8 values at a time
        const int i = e & (kDcTok - 1), p = e / kDcTok, c = p * 8;
        const float4 x = *reinterpret_cast<const float4*>(A + i * kPrepPitch + c), y = *reinterpret_cast<const float4*>(A + i * kPrepPitch + c + 4);
        uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
        if (i >= 64 || c < 64) {      // (the other quarter is zero and held intermediates)
            dc_split(x.x, x.y, hi.x, lo.x);
            dc_split(x.z, x.w, hi.y, lo.y);
            dc_split(y.x, y.y, hi.z, lo.z);
            dc_split(y.z, y.w, hi.w, lo.w);
        }
        *reinterpret_cast<uint4*>(dst + p * kInvPiece + i * 16) = hi;
        *reinterpret_cast<uint4*>(dst + (16 + p) * kInvPiece + i * 16) = lo;
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<128>(tmem);
    }
}

// ---- chunk after chunk --------------------------------------------------------------------------------------------------
constexpr size_t kDcSmem = 4 * kDcPanel /*k: two buffers*/ + 2 * kDcPanel /*q*/ + kDcPanel /*v*/ + 2 * kDcPanel /*S*/ + 2 * kDcPanel /*U*/ +
                           2 * kDcPanel /*R, then weighted U*/ + 2 * kDcTok * 4 + 256;

__global__ void __launch_bounds__(kDcThreads, 1)
delta_chunk_kernel(const __grid_constant__ CUtensorMap tmap_u, const SsmArgs a, const DeltaWs ws) {
    constexpr uint32_t kTmem = 512;
    constexpr uint32_t IDESC_CB = make_idesc_f16(128, 128, true, false, false);
    constexpr uint32_t IDESC_KN = make_idesc_f16(128, kDcP, true, false, true);   // A K-major, B MN-major
    constexpr uint32_t IDESC_NN = make_idesc_f16(128, kDcP, true, true, true);    // both MN-major

    extern __shared__ __align__(1024) uint8_t smem[];
    uint8_t* k_sm = smem;
    uint8_t* q_sm = k_sm + 4 * kDcPanel;
    uint8_t* v_sm = q_sm + 2 * kDcPanel;
    uint8_t* s_sm = v_sm + kDcPanel;       // hi, lo: rows = key dimension, 64 value columns
    uint8_t* u_sm = s_sm + 2 * kDcPanel;   // hi, lo: rows = tokens
    uint8_t* w_sm = u_sm + 2 * kDcPanel;   // hi, lo: rows = tokens
    float* b_s = reinterpret_cast<float*>(w_sm + 2 * kDcPanel);   // [2][128]: a_j - log2(1 / |k_j|)
    uint64_t* bar = reinterpret_cast<uint64_t*>(b_s + 2 * kDcTok);
    uint64_t *k_full = bar /*[2]*/, *k_empty = bar + 2 /*[2]*/, *q_full = bar + 4, *q_empty = bar + 5, *v_full = bar + 6, *v_empty = bar + 7,
             *cb_done = bar + 8, *s_full = bar + 9, *x_done = bar + 10, *r_full = bar + 11, *t_full = bar + 12, *u_done = bar + 13,
             *u_full = bar + 14, *st_done = bar + 15, *p_full = bar + 16, *y_done = bar + 17, *y_free = bar + 18;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar + 19);

    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const uint32_t warp = warp_id(), lane = lane_id();
    const int h = blockIdx.y, p0 = blockIdx.z * kDcP, N = a.N, P = a.P, H = a.heads;
    const int g = h / (H / a.groups), inner = a.inner();
    const int n_chunks = (sp.n + kDcTok - 1) / kDcTok;
    const int panels = (N + 63) / 64;

    if (warp == 0 && lane == 0) {
        prefetch_tmap(&tmap_u);
        for (int i = 0; i < 2; ++i) {
            mbar_init(k_full + i, 1);
            mbar_init(k_empty + i, 1);
        }
        mbar_init(q_full, 1);
        mbar_init(q_empty, 1);
        mbar_init(v_full, 1);
        mbar_init(v_empty, 8);
        mbar_init(cb_done, 1);
        mbar_init(s_full, 8);
        mbar_init(x_done, 1);
        mbar_init(r_full, 8);
        mbar_init(t_full, 8);
        mbar_init(u_done, 1);
        mbar_init(u_full, 8);
        mbar_init(st_done, 1);
        mbar_init(p_full, 8);
        mbar_init(y_done, 1);
        mbar_init(y_free, 8);
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
    const uint32_t t_cb = tmem /*scores, then decayed scores (per 16 tokens: 8 columns hi, 8 lo)*/, t_inv = tmem + 128 /*same layout*/,
                   t_xu = tmem + 256, t_y1 = tmem + 320, t_y2 = tmem + 384, t_st = tmem + 448;

    if (warp == 0) {
        if (lane == 0) {
            for (int c = 0; c < n_chunks; ++c) {
                const int row = sp.row0 + c * kDcTok, b = c & 1;
                if (c > 1) mbar_wait(k_empty + b, ((c >> 1) - 1) & 1);
                mbar_expect_tx(k_full + b, panels * kDcPanel);
                for (int p = 0; p < panels; ++p)
                    tma_load_2d(k_sm + (2 * b + p) * kDcPanel, &tmap_u, k_full + b, inner + g * N + p * 64, row, kEvictNormal);
                if (c > 0) mbar_wait(v_empty, (c - 1) & 1);
                mbar_expect_tx(v_full, kDcPanel);
                tma_load_2d(v_sm, &tmap_u, v_full, h * P + p0, row, kEvictNormal);
                if (c > 0) mbar_wait(q_empty, (c - 1) & 1);
                mbar_expect_tx(q_full, panels * kDcPanel);
                for (int p = 0; p < panels; ++p)
                    tma_load_2d(q_sm + p * kDcPanel, &tmap_u, q_full, inner + (a.groups + g) * N + p * 64, row, kEvictNormal);
            }
        }
    } else if (warp == 1) {
        const bool leader = elect_one();      // the whole warp walks the schedule, one elected lane issues
        constexpr uint64_t PANEL = kDcPanel >> 4, ROWS16 = (16 * 128) >> 4;
        const int k_steps = N / 16;
        const uint64_t d_k = make_desc_kmajor_sw128(smem_u32(k_sm)), d_kn = make_desc_mnmajor_sw128(smem_u32(k_sm), kDcPanel),
                       d_q = make_desc_kmajor_sw128(smem_u32(q_sm)), d_s = make_desc_mnmajor_sw128(smem_u32(s_sm), kDcPanel),
                       d_u = make_desc_mnmajor_sw128(smem_u32(u_sm), kDcPanel), d_w = make_desc_mnmajor_sw128(smem_u32(w_sm), kDcPanel);
        auto scores = [&](int c) {
            const uint64_t dk = d_k + 2 * (c & 1) * PANEL;
            if (leader) {
#pragma unroll
                for (int kk = 0; kk < 8; ++kk)
                    if (kk < k_steps)
                        umma_f16_ss(t_cb, d_q + (kk >> 2) * PANEL + 2 * (kk & 3), dk + (kk >> 2) * PANEL + 2 * (kk & 3), IDESC_CB, kk > 0 ? 1u : 0u);
                umma_commit(cb_done);
                umma_commit(q_empty);
            }
            __syncwarp();
        };
        // rows x state: both terms of the state
        auto times_state = [&](uint32_t d, uint64_t rows) {
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int kk = 0; kk < 8; ++kk)
                    if (kk < k_steps)
                        umma_f16_ss(d, rows + (kk >> 2) * PANEL + 2 * (kk & 3), d_s + t * PANEL + kk * ROWS16, IDESC_KN, (t > 0 || kk > 0) ? 1u : 0u);
        };
        // two-term matrix in TMEM x two-term rows: hi hi + hi lo + lo hi
        auto times_rows = [&](uint32_t d, uint32_t m, uint64_t rows) {
#pragma unroll
            for (int t = 0; t < 3; ++t)
#pragma unroll
                for (int kk = 0; kk < kDcTok / 16; ++kk)
                    umma_f16_ts(d, m + kk * 16 + (t == 2 ? 8 : 0), rows + (t == 1 ? PANEL : 0) + kk * ROWS16, IDESC_KN, (t > 0 || kk > 0) ? 1u : 0u);
        };
        for (int c = 0; c < n_chunks; ++c) {
            const uint32_t ph = c & 1;
            const uint64_t kb = 2 * (c & 1) * PANEL;
            mbar_wait(k_full + (c & 1), (c >> 1) & 1);
            mbar_wait(s_full, ph);
            tc_fence_after();
            if (leader) {
                times_state(t_xu, d_k + kb);
                umma_commit(x_done);
            }
            __syncwarp();
            if (c > 0) {      // scores x U of the chunk before, while R of this one is formed
                mbar_wait(p_full, ph ^ 1);
                tc_fence_after();
                if (leader) {
                    times_rows(t_y1, t_cb, d_u);
                    umma_commit(y_done);
                }
                __syncwarp();
            }
            mbar_wait(t_full, ph);
            mbar_wait(r_full, ph);
            tc_fence_after();
            if (leader) {
                times_rows(t_xu, t_inv, d_w);
                umma_commit(u_done);
            }
            __syncwarp();
            // (the outputs of the chunk before have been read, so its last product is complete: products of unlike shapes are not
            // ordered by themselves, and the scores below overwrite that product's operand)
            if (c > 0) mbar_wait(y_free, ph ^ 1);
            mbar_wait(q_full, ph);
            tc_fence_after();
            if (leader) times_state(t_y2, d_q);
            __syncwarp();
            scores(c);
            mbar_wait(u_full, ph);
            tc_fence_after();
            if (leader) {      // (the state has been scaled in place)
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int kk = 0; kk < kDcTok / 16; ++kk)
                        umma_f16_ss(t_st, d_kn + kb + kk * ROWS16, d_w + t * PANEL + kk * ROWS16, IDESC_NN, 1u);
                umma_commit(st_done);
                umma_commit(k_empty + (c & 1));
            }
            __syncwarp();
        }
        mbar_wait(p_full, (n_chunks - 1) & 1);
        tc_fence_after();
        if (leader) {
            times_rows(t_y1, t_cb, d_u);
            umma_commit(y_done);
        }
        __syncwarp();
    } else if (warp < 10) {
        // ===================== the state's chain: thread = (token r of the chunk and key dimension, column half) =====================
        const int quad = warp & 3, half = (warp - 2) >> 2;
        const int r = quad * 32 + lane;
        const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
        float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
        auto arrive = [&](uint64_t* b) {
            tc_fence_before();
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(b);
        };
        float a_last_n, a_r_n, beta_n, rk_n;      // of the next chunk, loaded a chunk ahead
        auto load_factors = [&](int c) {
            const int row = sp.row0 + c * kDcTok, n = min(kDcTok, sp.n - c * kDcTok);
            const int64_t th = static_cast<int64_t>(row + r) * H + h;
            a_last_n = __ldcg(ws.a + static_cast<int64_t>(row + n - 1) * H + h);
            a_r_n = r < n ? __ldcg(ws.a + th) : 0.0f;
            beta_n = r < n ? __ldcg(ws.beta + th) : 0.0f;
            rk_n = r < n ? __ldcg(ws.rk + static_cast<int64_t>(row + r) * a.groups + g) : 0.0f;
        };
        load_factors(0);
        for (int c = 0; c < n_chunks; ++c) {
            const uint32_t ph = c & 1;
            const bool live = r < min(kDcTok, sp.n - c * kDcTok);
            const float a_last = a_last_n, a_r = live ? a_r_n : a_last, beta = beta_n, rk = rk_n;
            const float keep = dc_ex2(a_last), from_state = dc_ex2(a_r) * rk, weight = dc_ex2(a_last - a_r) * rk;
            // ---- the state: two-term copy, then scaled in place for its update ----
            uint32_t sw[32];
            if (c == 0) {
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    const int p = p0 + half * 32 + j;
                    sw[j] = __float_as_uint((sp.seen > 0 && p < P && r < N) ? st[static_cast<int64_t>(p) * N + r] : 0.0f);
                }
            } else {
                mbar_wait(st_done, ph ^ 1);      // (and with it every product of the chunk before but the last)
                tc_fence_after();
                tmem_ld_32x32(t_st + la + half * 32, sw);
                tmem_ld_wait();
            }
#pragma unroll
            for (int ch = 0; ch < 4; ++ch) {
                uint4 hi, lo;
                dc_split(__uint_as_float(sw[8 * ch + 0]), __uint_as_float(sw[8 * ch + 1]), hi.x, lo.x);
                dc_split(__uint_as_float(sw[8 * ch + 2]), __uint_as_float(sw[8 * ch + 3]), hi.y, lo.y);
                dc_split(__uint_as_float(sw[8 * ch + 4]), __uint_as_float(sw[8 * ch + 5]), hi.z, lo.z);
                dc_split(__uint_as_float(sw[8 * ch + 6]), __uint_as_float(sw[8 * ch + 7]), hi.w, lo.w);
                *dc_cell(s_sm, r, half * 4 + ch) = hi;
                *dc_cell(s_sm + kDcPanel, r, half * 4 + ch) = lo;
            }
            arrive(s_full);
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                uint32_t sc[16];
#pragma unroll
                for (int j = 0; j < 16; ++j) sc[j] = __float_as_uint(__uint_as_float(sw[part * 16 + j]) * keep);
                tmem_st_32x16(t_st + la + half * 32 + part * 16, sc);
            }
            tmem_st_wait();
            // ---- R ----
            mbar_wait(v_full, ph);
            uint4 v[4];
#pragma unroll
            for (int ch = 0; ch < 4; ++ch) v[ch] = *dc_cell(v_sm, r, half * 4 + ch);
            mbar_wait(x_done, ph);
            tc_fence_after();
            uint32_t x[32];
            tmem_ld_32x32(t_xu + la + half * 32, x);
            tmem_ld_wait();
            if (c + 1 < n_chunks) load_factors(c + 1);
#pragma unroll
            for (int ch = 0; ch < 4; ++ch) {
                const uint32_t vv[4] = {v[ch].x, v[ch].y, v[ch].z, v[ch].w};
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float r0 = beta * (bf16_lo(vv[e]) - from_state * __uint_as_float(x[8 * ch + 2 * e]));
                    const float r1 = beta * (bf16_hi(vv[e]) - from_state * __uint_as_float(x[8 * ch + 2 * e + 1]));
                    dc_split(live ? r0 : 0.0f, live ? r1 : 0.0f, hi[e], lo[e]);
                }
                *dc_cell(w_sm, r, half * 4 + ch) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *dc_cell(w_sm + kDcPanel, r, half * 4 + ch) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            arrive(r_full);
            if (lane == 0) mbar_arrive(v_empty);      // (all of v has been used)
            // ---- U ----
            mbar_wait(u_done, ph);
            tc_fence_after();
            tmem_ld_32x32(t_xu + la + half * 32, x);
            tmem_ld_wait();
            if (c > 0) mbar_wait(y_done, ph ^ 1);      // U of the chunk before has been multiplied
#pragma unroll
            for (int ch = 0; ch < 4; ++ch) {
                uint32_t hi[4], lo[4], whi[4], wlo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float u0 = __uint_as_float(x[8 * ch + 2 * e]), u1 = __uint_as_float(x[8 * ch + 2 * e + 1]);
                    dc_split(u0, u1, hi[e], lo[e]);
                    dc_split(weight * u0, weight * u1, whi[e], wlo[e]);
                }
                *dc_cell(u_sm, r, half * 4 + ch) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *dc_cell(u_sm + kDcPanel, r, half * 4 + ch) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
                *dc_cell(w_sm, r, half * 4 + ch) = make_uint4(whi[0], whi[1], whi[2], whi[3]);
                *dc_cell(w_sm + kDcPanel, r, half * 4 + ch) = make_uint4(wlo[0], wlo[1], wlo[2], wlo[3]);
            }
            arrive(u_full);
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
        // ===================== inverse, decayed scores, output: thread = (token r of the chunk, column half) =====================
        const int quad = warp & 3, half = (warp - 10) >> 2;
        const int r = quad * 32 + lane;
        const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
        int first = 0;      // number of this sequence's first chunk
        for (int s = lane; s < static_cast<int>(blockIdx.x); s += 32) first += dc_chunks(a.spans[s]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) first += __shfl_xor_sync(0xffffffffu, first, o);
        auto output = [&](int c, float from_state) {
            mbar_wait(y_done, c & 1);
            tc_fence_after();
            const bool live = r < min(kDcTok, sp.n - c * kDcTok);
            float* yo = a.y + static_cast<int64_t>(sp.row0 + c * kDcTok + r) * inner + h * P + p0 + half * 32;
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                uint32_t y1[16], y2[16];
                tmem_ld_32x16(t_y1 + la + half * 32 + part * 16, y1);
                tmem_ld_32x16(t_y2 + la + half * 32 + part * 16, y2);
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
                    for (int j = 0; j < 8; ++j) o[j] = fmaf(from_state, __uint_as_float(y2[8 * ch + j]), __uint_as_float(y1[8 * ch + j]));
                    const int col = part * 16 + ch * 8;
                    if (live && p0 + half * 32 + col < P) st_v8_f32(yo + col, o);      // P is a multiple of 8
                }
            }
            __syncwarp();
        };
        // the inverse of chunk c: my row's 64 columns, 16 at a time
        auto load_inverse = [&](int c) {
            const uint8_t* src = ws.inv + (static_cast<int64_t>(first + c) * H + h) * kInvBytes + half * 8 * kInvPiece + r * 16;
            uint4 hi[8], lo[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                hi[i] = __ldcg(reinterpret_cast<const uint4*>(src + i * kInvPiece));      // (not through L1: the launch before wrote it)
                lo[i] = __ldcg(reinterpret_cast<const uint4*>(src + (16 + i) * kInvPiece));
            }
            if (c > 0) mbar_wait(u_done, (c - 1) & 1);
            tc_fence_after();
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t m[16] = {hi[2 * i].x, hi[2 * i].y, hi[2 * i].z, hi[2 * i].w, hi[2 * i + 1].x, hi[2 * i + 1].y, hi[2 * i + 1].z, hi[2 * i + 1].w,
                                        lo[2 * i].x, lo[2 * i].y, lo[2 * i].z, lo[2 * i].w, lo[2 * i + 1].x, lo[2 * i + 1].y, lo[2 * i + 1].z, lo[2 * i + 1].w};
                tmem_st_32x16(t_inv + la + half * 64 + i * 16, m);
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(t_full);
            __syncwarp();
        };
        float a_last_n, a_r_n, rk_n, rq_n;
        auto load_factors = [&](int c) {
            const int row = sp.row0 + c * kDcTok, n = min(kDcTok, sp.n - c * kDcTok);
            a_last_n = __ldcg(ws.a + static_cast<int64_t>(row + n - 1) * H + h);
            a_r_n = r < n ? __ldcg(ws.a + static_cast<int64_t>(row + r) * H + h) : 0.0f;
            rk_n = r < n ? __ldcg(ws.rk + static_cast<int64_t>(row + r) * a.groups + g) : 1.0f;
            rq_n = r < n ? __ldcg(ws.rq + static_cast<int64_t>(row + r) * a.groups + g) : 0.0f;
        };
        load_factors(0);
        load_inverse(0);
        for (int c = 0; c < n_chunks; ++c) {
            const uint32_t ph = c & 1;
            const float a_r = r < min(kDcTok, sp.n - c * kDcTok) ? a_r_n : a_last_n, rq = rq_n;
            if (half == 0) b_s[ph * kDcTok + r] = a_r - __log2f(rk_n);
            if (c + 1 < n_chunks) load_factors(c + 1);
            asm volatile("bar.sync 2, 256;" ::: "memory");     // b_s of this chunk is complete
            // ---- decayed scores, in place: 16 fp32 columns become 8 of leading terms and 8 of rests ----
            const float* bv = b_s + ph * kDcTok;
            mbar_wait(cb_done, ph);
            tc_fence_after();
            const uint32_t t_m = t_cb + la;
#pragma unroll 1
            for (int part = 0; part < 4; ++part) {
                const int jp = half * 64 + part * 16;
                uint32_t m[16];
                if (jp > quad * 32 + 31) {        // every column lies in the future
#pragma unroll
                    for (int j = 0; j < 16; ++j) m[j] = 0u;
                } else {
                    uint32_t cb[16];
                    tmem_ld_32x16(t_m + jp, cb);
                    tmem_ld_wait();
                    const int mine = r - jp;
                    float v[16];
#pragma unroll
                    for (int j = 0; j < 16; j += 4) {
                        const float4 b = *reinterpret_cast<const float4*>(bv + jp + j);
                        v[j + 0] = __uint_as_float(cb[j + 0]) * rq * dc_ex2(a_r - b.x);
                        v[j + 1] = __uint_as_float(cb[j + 1]) * rq * dc_ex2(a_r - b.y);
                        v[j + 2] = __uint_as_float(cb[j + 2]) * rq * dc_ex2(a_r - b.z);
                        v[j + 3] = __uint_as_float(cb[j + 3]) * rq * dc_ex2(a_r - b.w);
                    }
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = j > mine ? 0.0f : v[j];
#pragma unroll
                    for (int j = 0; j < 8; ++j) dc_split(v[2 * j], v[2 * j + 1], m[j], m[8 + j]);
                }
                tmem_st_32x16(t_m + jp, m);
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
            __syncwarp();
            if (c + 1 < n_chunks) load_inverse(c + 1);
            output(c, dc_ex2(a_r) * rq);
        }
        if (blockIdx.z == 0) ssm_save_conv_of_head<0>(a, sp, h, threadIdx.x - 320, 256);
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<kTmem>(tmem);
    }
}

static int64_t dc_align(int64_t x) { return (x + 255) & ~int64_t(255); }
static int64_t dc_slots(int T, int n_seqs) { return T / kDcTok + n_seqs; }

int64_t delta_chunk_workspace(int T, int n_seqs, int heads, int groups) {
    return dc_slots(T, n_seqs) * heads * kInvBytes + 2 * dc_align(static_cast<int64_t>(T) * heads * 4) + 2 * dc_align(static_cast<int64_t>(T) * groups * 4);
}

bool delta_chunk_supported(const SsmArgs& a, int n_multi, int dtype, int64_t ws_bytes) {
    return dtype == 0 && a.N % 16 == 0 && a.N <= 128 && a.P % 8 == 0 && (a.P <= kDcP || a.P % kDcP == 0) && a.ld_u % 8 == 0 &&
           (reinterpret_cast<uintptr_t>(a.u) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.y) & 31) == 0 &&
           ws_bytes >= delta_chunk_workspace(a.T, n_multi, a.heads, a.groups);
}

int delta_chunk_launch(const SsmArgs& a, int n_multi, int dtype, void* workspace, cudaStream_t s) {
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!configured[dev & 63]) {
        HDS_CHECK_CUDA(cudaFuncSetAttribute(delta_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kPrepSmem)));
        HDS_CHECK_CUDA(cudaFuncSetAttribute(delta_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kDcSmem)));
        configured[dev & 63] = true;
    }
    DeltaWs ws;
    uint8_t* p = static_cast<uint8_t*>(workspace);
    const int64_t per_head = dc_align(static_cast<int64_t>(a.T) * a.heads * 4), per_group = dc_align(static_cast<int64_t>(a.T) * a.groups * 4);
    const int64_t slots = dc_slots(a.T, n_multi);
    ws.inv = p;
    p += slots * a.heads * kInvBytes;
    ws.a = reinterpret_cast<float*>(p);
    ws.beta = reinterpret_cast<float*>(p + per_head);
    ws.rk = reinterpret_cast<float*>(p + 2 * per_head);
    ws.rq = reinterpret_cast<float*>(p + 2 * per_head + per_group);
    CUtensorMap tm;
    const int rc = make_tmap_2d_16b(&tm, a.u, static_cast<uint64_t>(a.channels()), static_cast<uint64_t>(a.T),
                                    static_cast<uint64_t>(a.ld_u) * 2, 64, kDcTok, dtype == 0);
    if (rc) return rc;
    HDS_CHECK_CUDA(launch_kernel(delta_prep_kernel, dim3(static_cast<unsigned>(slots), a.heads), dim3(kPrepThreads), kPrepSmem, s, tm, a, ws));
    HDS_CHECK_CUDA(launch_kernel(delta_chunk_kernel, dim3(a.n_seqs, a.heads, (a.P + kDcP - 1) / kDcP), dim3(kDcThreads), kDcSmem, s, tm, a, ws));
    return HDS_OK;
}

}  // namespace hds
