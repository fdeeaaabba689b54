// Retention over a ragged batch, per head:  S <- decay S + v k^T,  o = S q  (q and k turned by position), then o / rms(o) * silu(gate).
// Sequences with one new token are stepped, and fp32 / fp16 models and odd sizes scanned, by the kernels of linear_attention.cu. Prompts of
// bf16 models run here on tcgen05, 128 tokens at a time. With S the state in front of a chunk and d the head's decay:
//
//   o_i = d^(i + 1) S q_i + sum_{j <= i} d^(i - j) (q_i . k_j) v_j          S <- d^n S + sum_j d^(n - 1 - j) v_j k_j^T
//
//   ret_local : per (chunk, head): what the chunk's tokens add to the state. Independent of other chunks
//   ret_chain : states in front of every chunk, in place of those sums; advances the state pool. A plain stream along the chunks
//   ret_out   : per (chunk, head): scores, state and value products, norm and gate
//
// v enters products exactly as it is. Everything fp32 that becomes an operand (turned q and k, decayed keys and scores, the state) is a bf16
// value plus the bf16 rest, 16 significant bits; sums are fp32 in TMEM, the carried state is never rounded. A thread turns runs of
// consecutive tokens: one sine and cosine of its first position, then a step by the pair's own angle per token (runs of 64 at most).
// The sums are [P][N] rows of 32-byte groups (8 values); a state takes their place as 8 leading terms and 8 rests, the 16-byte pieces of
// swizzled operand rows. Long batches run in segments, which bounds the workspace.
#include "linear_attention.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kRtTok = 128, kRtThreads = 256, kRtP = 128, kRtPanel = kRtTok * 128;       // a panel: 128 rows of 128 bytes

//: set when a wait ran out (a fault of the kernel's own protocol); read by hds_retention_status
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
__device__ __forceinline__ void rt_split(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - bf16_lo(hi), v1 - bf16_hi(hi));
}
// byte of column c (of 64-column panels) in row r of a 128-byte-swizzled tile
__device__ __forceinline__ uint32_t rt_byte(int r, int c) {
    return static_cast<uint32_t>((c >> 6) * kRtPanel + r * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4) + (c & 7) * 2);
}
__device__ __forceinline__ void rt_copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// Which tokens and columns a thread turns: columns c, c + 1 and their partners half a row behind, tokens t0 .. t0 + run - 1.
struct RtPlace {
    int c, t0, run;
};
__device__ __forceinline__ RtPlace rt_place(int N) {
    const int lanes = N >> 2, runs = kRtThreads / lanes, run = (kRtTok + runs - 1) / runs, u = threadIdx.x / lanes;
    RtPlace p;
    p.c = (threadIdx.x - u * lanes) * 2;
    p.t0 = u < runs ? u * run : kRtTok;
    p.run = run;
    return p;
}

// Rows of q or k of one head (fp32 once turned) -> two operand tiles. weight(t): factor of token t. Tokens from n on are zeros.
// RUN: tokens per run where that is known (8 loads in flight at a time otherwise).
template <int RUN, typename F>
__device__ __forceinline__ void rt_turn(const LinArgs& a, const void* x, int64_t row, int64_t head_col, int N, int n, float pos0, uint8_t* hi_t,
                                        uint8_t* lo_t, F weight) {
    const RtPlace p = rt_place(N);
    if (p.t0 >= kRtTok) return;
    const int half = N >> 1;
    const char* src = static_cast<const char*>(x) + ((row + p.t0) * a.ld + head_col + p.c) * 2;
    float s0, c0, s1, c1, fs0, fc0, fs1, fc1;
    const float f0 = a.freq[p.c], f1 = a.freq[p.c + 1];
    rope_sincos((pos0 + p.t0) * f0, &s0, &c0);
    rope_sincos((pos0 + p.t0) * f1, &s1, &c1);
    rope_sincos(f0, &fs0, &fc0);
    rope_sincos(f1, &fs1, &fc1);
    if (a.amp != nullptr) {
        s0 *= a.amp[p.c]; c0 *= a.amp[p.c];
        s1 *= a.amp[p.c + 1]; c1 *= a.amp[p.c + 1];
    }
    constexpr int U = RUN > 0 ? RUN : 8;
    for (int b = 0; b < (RUN > 0 ? RUN : p.run); b += U) {
        uint32_t u[U], v[U];
#pragma unroll
        for (int i = 0; i < U; ++i) {
            u[i] = v[i] = 0u;
            if (b + i < p.run && p.t0 + b + i < n) {
                const char* at = src + static_cast<int64_t>(b + i) * a.ld * 2;
                u[i] = *reinterpret_cast<const uint32_t*>(at);
                v[i] = *reinterpret_cast<const uint32_t*>(at + half * 2);
            }
        }
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int t = p.t0 + b + i;
            if (b + i >= p.run || t >= kRtTok) break;
            const float w = weight(t);
            const float x0 = bf16_lo(u[i]), x1 = bf16_hi(u[i]), y0 = bf16_lo(v[i]), y1 = bf16_hi(v[i]);
            uint32_t hi, lo;
            rt_split(w * (x0 * c0 - y0 * s0), w * (x1 * c1 - y1 * s1), hi, lo);
            uint32_t at = rt_byte(t, p.c);
            *reinterpret_cast<uint32_t*>(hi_t + at) = hi;
            *reinterpret_cast<uint32_t*>(lo_t + at) = lo;
            rt_split(w * (y0 * c0 + x0 * s0), w * (y1 * c1 + x1 * s1), hi, lo);
            at = rt_byte(t, p.c + half);
            *reinterpret_cast<uint32_t*>(hi_t + at) = hi;
            *reinterpret_cast<uint32_t*>(lo_t + at) = lo;
            const float n0 = c0 * fc0 - s0 * fs0, n1 = c1 * fc1 - s1 * fs1;
            s0 = s0 * fc0 + c0 * fs0;
            s1 = s1 * fc1 + c1 * fs1;
            c0 = n0;
            c1 = n1;
        }
    }
}

struct RetWs {
    float* s;           // [chunks][heads][P][N]: sums, then states (see above)
    int c0, n;          // chunks [c0, c0 + n) of the batch
};

__host__ __device__ constexpr int rt_panels(int cols) { return (cols + 63) / 64; }
// k (two terms) and v
__host__ __device__ constexpr size_t rt_local_smem(int N) { return static_cast<size_t>(2 * rt_panels(N) + 2) * kRtPanel + 1024; }

// NT: the number of key channels where it is known, 0: any
template <int NT>
__global__ void __launch_bounds__(kRtThreads, 2)
ret_local_kernel(const __grid_constant__ CUtensorMap tmap_v, const LinArgs a, const RetWs ws) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ ChunkPlace place;
    __shared__ uint64_t v_full, done;
    __shared__ uint32_t tmem_slot;
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kRtTok, ws.c0 + blockIdx.x, &place)) return;
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int N = NT > 0 ? NT : a.N, P = a.P, h = blockIdx.y, p0 = blockIdx.z * kRtP, Pb = min(kRtP, P - p0);
    const int t0 = place.chunk * kRtTok, n = min(kRtTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0;
    uint8_t* k_hi = smem;
    uint8_t* k_lo = k_hi + rt_panels(N) * kRtPanel;
    uint8_t* v_sm = k_lo + rt_panels(N) * kRtPanel;
    const uint32_t warp = warp_id(), lane = lane_id();
    bool stuck = false;
    if (threadIdx.x == 0) {
        prefetch_tmap(&tmap_v);
        mbar_init(&v_full, 1);
        mbar_init(&done, 1);
        fence_barrier_init();
        const int panels = rt_panels(Pb);
        mbar_expect_tx(&v_full, panels * kRtPanel);
        for (int p = 0; p < panels; ++p) tma_load_2d(v_sm + p * kRtPanel, &tmap_v, &v_full, h * P + p0 + p * 64, static_cast<int>(row), kEvictNormal);
    }
    if (warp == 1) {
        tmem_alloc<128>(&tmem_slot);
        tmem_relinquish();
    }
    const float ld = a.log2_decay[h], last = static_cast<float>(n - 1);
    rt_turn<NT == 128 ? 16 : NT == 64 ? 8 : 0>(a, a.k, row, static_cast<int64_t>(h) * N, N, n, static_cast<float>(place.span.seen + t0), k_hi, k_lo,
                                               [&](int t) { return a.k_scale * rt_ex2(ld * fmaxf(last - t, 0.0f)); });
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    if (threadIdx.x == 0) {      // sums [P][N] = V^T K, both operands as they lie (tokens are rows)
        rt_wait(&v_full, 0, stuck);
        tc_fence_after();
        const uint32_t idesc = make_idesc_f16(128, N, true, true, true);
        const uint64_t dv = make_desc_mnmajor_sw128(smem_u32(v_sm), kRtPanel);
        constexpr uint64_t ROWS16 = (16 * 128) >> 4;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const uint64_t dk = make_desc_mnmajor_sw128(smem_u32(t ? k_lo : k_hi), kRtPanel);
#pragma unroll
            for (int kk = 0; kk < kRtTok / 16; ++kk) umma_f16_ss(tmem, dv + kk * ROWS16, dk + kk * ROWS16, idesc, (t > 0 || kk > 0) ? 1u : 0u);
        }
        umma_commit(&done);
    }
    __syncwarp();
    rt_wait(&done, 0, stuck);
    __syncwarp();
    tc_fence_after();
    const int quad = warp & 3, half = warp >> 2, p = quad * 32 + lane;
    float* out = ws.s + ((static_cast<int64_t>(blockIdx.x) * a.heads + h) * P + p0 + p) * N;
    for (int b = half; b < N >> 4; b += 2) {
        uint32_t r[16];
        tmem_ld_32x16(tmem + (static_cast<uint32_t>(quad * 32) << 16) + b * 16, r);
        tmem_ld_wait();
        if (p < Pb) {
#pragma unroll
            for (int g = 0; g < 2; ++g) {
                float o[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) o[j] = __uint_as_float(r[8 * g + j]);
                st_v8_f32(out + b * 16 + g * 8, o);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<128>(tmem);
    }
}

// A thread keeps eight state values along the chunks of a sequence that lie in the segment; loads run ahead of the stores.
__global__ void __launch_bounds__(kRtThreads) ret_chain_kernel(const LinArgs a, const RetWs ws) {
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int total = span_chunks(sp, kRtTok), base = first_chunk(a.spans, blockIdx.x, kRtTok);
    const int i0 = max(0, ws.c0 - base), i1 = min(total, ws.c0 + ws.n - base);
    const int h = blockIdx.y, PN = a.P * a.N, e = (blockIdx.z * kRtThreads + threadIdx.x) * 8;
    if (i0 >= i1 || e >= PN) return;
    float* st = a.state + (static_cast<int64_t>(sp.slot) * a.heads + h) * PN + e;
    float4 S = make_float4(0.f, 0.f, 0.f, 0.f), R = S;
    if (sp.seen > 0 || i0 > 0) {
        S = *reinterpret_cast<const float4*>(st);
        R = *reinterpret_cast<const float4*>(st + 4);
    }
    const float ld = a.log2_decay[h], keep = rt_ex2(ld * kRtTok), keep_last = rt_ex2(ld * (sp.n - (total - 1) * kRtTok));
    const int64_t step = static_cast<int64_t>(a.heads) * PN;
    float* s = ws.s + (base + i0 - ws.c0) * step + static_cast<int64_t>(h) * PN + e;
    constexpr int U = 4;
    float4 x[U], y[U];
    const float* sl = s;
    auto load = [&](int j, bool live) {
        if (!live) return;
        x[j] = __ldcg(reinterpret_cast<const float4*>(sl));
        y[j] = __ldcg(reinterpret_cast<const float4*>(sl + 4));
        sl += step;
    };
    const int n = i1 - i0;
#pragma unroll
    for (int j = 0; j < U; ++j) load(j, j < n);
    for (int i = 0; i < n; i += U) {
#pragma unroll
        for (int j = 0; j < U; ++j) {
            if (i + j >= n) break;
            uint4 hi, lo;
            rt_split(S.x, S.y, hi.x, lo.x);
            rt_split(S.z, S.w, hi.y, lo.y);
            rt_split(R.x, R.y, hi.z, lo.z);
            rt_split(R.z, R.w, hi.w, lo.w);
            reinterpret_cast<uint4*>(s)[0] = hi;
            reinterpret_cast<uint4*>(s)[1] = lo;
            s += step;
            const float f = i0 + i + j == total - 1 ? keep_last : keep;
            S = make_float4(fmaf(f, S.x, x[j].x), fmaf(f, S.y, x[j].y), fmaf(f, S.z, x[j].z), fmaf(f, S.w, x[j].w));
            R = make_float4(fmaf(f, R.x, y[j].x), fmaf(f, R.y, y[j].y), fmaf(f, R.z, y[j].z), fmaf(f, R.w, y[j].w));
            load(j, i + j + U < n);
        }
    }
    *reinterpret_cast<float4*>(st) = S;
    *reinterpret_cast<float4*>(st + 4) = R;
}

// q, k and the state (two terms each) and v. Up to 64 key channels two blocks share an SM: the state takes the place of the keys, once
// those have been multiplied.
__host__ __device__ constexpr bool rt_shares(int N) { return N <= 64; }
__host__ __device__ constexpr size_t rt_out_smem(int N) {
    const int p = rt_panels(N);
    return static_cast<size_t>((rt_shares(N) ? 4 : 6) * p + 2) * kRtPanel + 1024;
}

template <int NT>
__global__ void __launch_bounds__(kRtThreads, NT == 64 ? 2 : 1)
ret_out_kernel(const __grid_constant__ CUtensorMap tmap_v, const LinArgs a, const RetWs ws) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ ChunkPlace place;
    __shared__ uint64_t v_full, s_done, y_done, o_done;
    __shared__ uint32_t tmem_slot;
    __shared__ float ss_s[2][kRtTok];
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kRtTok, ws.c0 + blockIdx.x, &place)) return;
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int N = NT > 0 ? NT : a.N, P = a.P, h = blockIdx.y, p0 = blockIdx.z * kRtP, Pb = min(kRtP, P - p0);
    const int t0 = place.chunk * kRtTok, n = min(kRtTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0;
    const int tile = rt_panels(N) * kRtPanel;
    uint8_t* q_hi = smem;
    uint8_t* q_lo = q_hi + tile;
    uint8_t* k_hi = q_lo + tile;
    uint8_t* k_lo = k_hi + tile;
    uint8_t* s_hi = rt_shares(N) ? k_hi : k_lo + tile;
    uint8_t* s_lo = s_hi + tile;
    uint8_t* v_sm = s_lo + tile;
    const uint32_t warp = warp_id(), lane = lane_id();
    const bool fresh = place.span.seen == 0 && place.chunk == 0;        // (nothing in front: the state is zero)
    bool stuck = false;
    if (threadIdx.x == 0) {
        prefetch_tmap(&tmap_v);
        mbar_init(&v_full, 1);
        mbar_init(&s_done, 1);
        mbar_init(&y_done, 1);
        mbar_init(&o_done, 1);
        fence_barrier_init();
        const int panels = rt_panels(Pb);
        mbar_expect_tx(&v_full, panels * kRtPanel);
        for (int p = 0; p < panels; ++p) tma_load_2d(v_sm + p * kRtPanel, &tmap_v, &v_full, h * P + p0 + p * 64, static_cast<int>(row), kEvictNormal);
    }
    if (warp == 1) {
        tmem_alloc<256>(&tmem_slot);
        tmem_relinquish();
    }
    auto fetch_state = [&]() {
        const char* src = reinterpret_cast<const char*>(ws.s + ((static_cast<int64_t>(blockIdx.x) * a.heads + h) * P + p0) * N);
        const int groups = N >> 3;
        for (int e = threadIdx.x; e < Pb * groups; e += kRtThreads) {
            const int r = e / groups, at = rt_byte(r, (e - r * groups) * 8);
            rt_copy16(s_hi + at, src + static_cast<int64_t>(e) * 32);
            rt_copy16(s_lo + at, src + static_cast<int64_t>(e) * 32 + 16);
        }
    };
    if (!fresh && !rt_shares(N)) fetch_state();
    const float ld = a.log2_decay[h], pos0 = static_cast<float>(place.span.seen + t0);
    constexpr int RUN = NT == 128 ? 16 : NT == 64 ? 8 : 0;
    rt_turn<RUN>(a, a.k, row, static_cast<int64_t>(h) * N, N, n, pos0, k_hi, k_lo, [&](int) { return a.k_scale; });
    rt_turn<RUN>(a, a.q, row, static_cast<int64_t>(h) * N, N, n, pos0, q_hi, q_lo, [&](int) { return 1.0f; });
    if (!rt_shares(N)) asm volatile("cp.async.wait_all;" ::: "memory");
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t t_a = tmem_slot, t_y = t_a + 128;        // scores, then their two terms (per 16 tokens: 8 columns each); output
    constexpr uint64_t PANEL = kRtPanel >> 4, ROWS16 = (16 * 128) >> 4;
    // the three products of two operands of two terms each that matter
    auto three = [&](uint32_t d, const uint8_t* x_hi, const uint8_t* x_lo, const uint8_t* y_hi, const uint8_t* y_lo, uint32_t idesc) {
        const uint64_t dx[2] = {make_desc_kmajor_sw128(smem_u32(x_hi)), make_desc_kmajor_sw128(smem_u32(x_lo))};
        const uint64_t dy[2] = {make_desc_kmajor_sw128(smem_u32(y_hi)), make_desc_kmajor_sw128(smem_u32(y_lo))};
#pragma unroll
        for (int t = 0; t < 3; ++t)
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
                if (kk < N >> 4) {
                    const uint64_t at = (kk >> 2) * PANEL + 2 * (kk & 3);
                    umma_f16_ss(d, dx[t == 2] + at, dy[t == 1] + at, idesc, (t > 0 || kk > 0) ? 1u : 0u);
                }
    };
    if (threadIdx.x == 0) {
        three(t_a, q_hi, q_lo, k_hi, k_lo, make_idesc_f16(128, 128, true, false, false));
        umma_commit(&s_done);
        if (!fresh && !rt_shares(N)) {
            three(t_y, q_hi, q_lo, s_hi, s_lo, make_idesc_f16(128, Pb, true, false, false));
            umma_commit(&y_done);
        }
    }
    __syncwarp();
    const int quad = warp & 3, half = warp >> 2, r = quad * 32 + lane;
    const uint32_t la = static_cast<uint32_t>(quad * 32) << 16;
    rt_wait(&s_done, 0, stuck);
    __syncwarp();
    tc_fence_after();
    if (!fresh && rt_shares(N)) {
        fetch_state();
        asm volatile("cp.async.wait_all;" ::: "memory");
        fence_proxy_async_smem();
        __syncthreads();
        if (threadIdx.x == 0) {
            three(t_y, q_hi, q_lo, s_hi, s_lo, make_idesc_f16(128, Pb, true, false, false));
            umma_commit(&y_done);
        }
        __syncwarp();
    }
    // ---- scores, decayed, in place: 16 fp32 columns become 8 of leading terms and 8 of rests ----
    const float d = rt_ex2(ld);
#pragma unroll 1
    for (int part = 0; part < 4; ++part) {
        const int j0 = half * 64 + part * 16;
        uint32_t m[16];
        if (j0 > quad * 32 + 31) {          // every column lies in the future
#pragma unroll
            for (int j = 0; j < 16; ++j) m[j] = 0u;
        } else {
            uint32_t x[16];
            tmem_ld_32x16(t_a + la + j0, x);
            tmem_ld_wait();
            float v[16];
            if (j0 + 15 > quad * 32) {      // the diagonal
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    const int back = r - j0 - j;
                    v[j] = back < 0 ? 0.0f : __uint_as_float(x[j]) * rt_ex2(ld * back);
                }
            } else {
                float f = rt_ex2(ld * (r - j0 - 15));
#pragma unroll
                for (int j = 15; j >= 0; --j) {
                    v[j] = __uint_as_float(x[j]) * f;
                    f *= d;
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) rt_split(v[2 * j], v[2 * j + 1], m[j], m[8 + j]);
        }
        tmem_st_32x16(t_a + la + j0, m);
    }
    // ---- what the state gives, decayed, in place; the scores' product adds to it ----
    const int blocks = Pb >> 4;
    if (!fresh) {
        rt_wait(&y_done, 0, stuck);
        __syncwarp();
        tc_fence_after();
        const float g = rt_ex2(ld * (r + 1));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int b = half + 2 * i;
            if (b >= blocks) break;
            uint32_t x[16];
            tmem_ld_32x16(t_y + la + b * 16, x);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) x[j] = __float_as_uint(__uint_as_float(x[j]) * g);
            tmem_st_32x16(t_y + la + b * 16, x);
        }
    }
    tmem_st_wait();
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0) {
        rt_wait(&v_full, 0, stuck);
        tc_fence_after();
        const uint32_t idesc = make_idesc_f16(128, Pb, true, false, true);
        const uint64_t dv = make_desc_mnmajor_sw128(smem_u32(v_sm), kRtPanel);
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int kk = 0; kk < kRtTok / 16; ++kk)
                umma_f16_ts(t_y, t_a + kk * 16 + t * 8, dv + kk * ROWS16, idesc, (!fresh || t > 0 || kk > 0) ? 1u : 0u);
        umma_commit(&o_done);
    }
    __syncwarp();
    const bool live = r < n;
    const int64_t col = static_cast<int64_t>(h) * P + p0;
    uint4 gate[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int b = half + 2 * i;
        gate[i][0] = gate[i][1] = make_uint4(0, 0, 0, 0);
        if (!a.write_y && live && b < blocks) {
            const uint4* src = reinterpret_cast<const uint4*>(static_cast<const char*>(a.gate) + ((row + r) * a.ld + col + b * 16) * 2);
            gate[i][0] = src[0];
            gate[i][1] = src[1];
        }
    }
    rt_wait(&o_done, 0, stuck);
    __syncwarp();
    tc_fence_after();
    float o[4][16], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int b = half + 2 * i;
        if (b >= blocks) break;
        uint32_t x[16];
        tmem_ld_32x16(t_y + la + b * 16, x);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; ++j) {
            o[i][j] = __uint_as_float(x[j]);
            ss = fmaf(o[i][j], o[i][j], ss);
        }
    }
    ss_s[half][r] = ss;
    tc_fence_before();
    __syncthreads();
    const float f = rsqrtf((ss_s[0][r] + ss_s[1][r]) / a.norm_cols + a.eps);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int b = half + 2 * i;
        if (b >= blocks || !live) break;
        if (a.write_y) {
#pragma unroll
            for (int j = 0; j < 16; j += 4)
                *reinterpret_cast<float4*>(a.y + (row + r) * a.ld_y + col + b * 16 + j) = make_float4(o[i][j], o[i][j + 1], o[i][j + 2], o[i][j + 3]);
            continue;
        }
        const uint32_t* gw = reinterpret_cast<const uint32_t*>(gate[i]);
        const float* w = a.norm_w + col + b * 16;
        uint32_t res[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const float2 nw = *reinterpret_cast<const float2*>(w + 2 * j);
            res[j] = pack_bf16(o[i][2 * j] * f * nw.x * ssm_silu<0>(bf16_lo(gw[j])), o[i][2 * j + 1] * f * nw.y * ssm_silu<0>(bf16_hi(gw[j])));
        }
        char* dst = static_cast<char*>(a.out) + ((row + r) * a.ld_out + col + b * 16) * 2;
        st_v4(dst, make_uint4(res[0], res[1], res[2], res[3]));
        st_v4(dst + 16, make_uint4(res[4], res[5], res[6], res[7]));
    }
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc<256>(t_a);
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
    return dtype == 0 && a.N % 16 == 0 && a.N <= 128 && a.P % 16 == 0 && ws != nullptr && ws_bytes >= rt_cell_bytes(a.heads, a.P, a.N) &&
           (reinterpret_cast<uintptr_t>(ws) & 31) == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) && aligned(a.gate) && aligned(a.out) &&
           aligned(a.state) && aligned(a.y) && a.ld % 8 == 0 && a.ld_out % 8 == 0 && a.ld_y % 4 == 0;
}

template <int NT>
static int rt_chunk_launch_as(const LinArgs& a, const CUtensorMap& tv, int64_t bound, int step, void* ws, cudaStream_t s) {
    auto local = ret_local_kernel<NT>;
    auto out = ret_out_kernel<NT>;
    HDS_CHECK_CUDA(cudaFuncSetAttribute(local, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(rt_local_smem(a.N))));
    HDS_CHECK_CUDA(cudaFuncSetAttribute(out, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(rt_out_smem(a.N))));
    const unsigned blocks = (a.P + kRtP - 1) / kRtP;
    for (int64_t c0 = 0; c0 < bound; c0 += step) {
        RetWs w;
        w.s = static_cast<float*>(ws);
        w.c0 = static_cast<int>(c0);
        w.n = static_cast<int>(step < bound - c0 ? step : bound - c0);
        const dim3 grid(w.n, a.heads, blocks), block(kRtThreads);
        HDS_CHECK_CUDA(launch_kernel(local, grid, block, rt_local_smem(a.N), s, tv, a, w));
        HDS_CHECK_CUDA(launch_kernel(ret_chain_kernel, dim3(a.n_seqs, a.heads, (a.P * a.N / 8 + kRtThreads - 1) / kRtThreads), block, 0, s, a, w));
        if (a.out != nullptr || a.write_y) HDS_CHECK_CUDA(launch_kernel(out, grid, block, rt_out_smem(a.N), s, tv, a, w));
    }
    return HDS_OK;
}

static int rt_chunk_launch(const LinArgs& a, int n_multi, void* ws, int64_t ws_bytes, cudaStream_t s) {
    const int64_t bound = a.T / kRtTok + n_multi;           // at least as many as there are chunks
    const int64_t fits = ws_bytes / rt_cell_bytes(a.heads, a.P, a.N), seg = rt_segment(bound, a.heads, a.P, a.N);
    const int step = static_cast<int>(seg < fits ? seg : fits);
    CUtensorMap tv;      // columns of all heads' values; a box that reaches past them reads zeros
    const int rc = make_tmap_2d_16b(&tv, a.v, static_cast<uint64_t>(a.heads) * a.P, static_cast<uint64_t>(a.T), static_cast<uint64_t>(a.ld) * 2, 64, kRtTok, true);
    if (rc) return rc;
    return a.N == 128 ? rt_chunk_launch_as<128>(a, tv, bound, step, ws, s)
           : a.N == 64 ? rt_chunk_launch_as<64>(a, tv, bound, step, ws, s)
                       : rt_chunk_launch_as<0>(a, tv, bound, step, ws, s);
}

}  // namespace hds

using namespace hds;

extern "C" int64_t hds_retention_workspace_bytes(int T, int n_seqs, int heads, int vdim, int dim) {
    if (dim % 16 != 0 || dim > 128 || vdim % 16 != 0) return 0;
    const int64_t all = T / kRtTok + (n_seqs < T / 2 ? n_seqs : T / 2);
    return rt_segment(all > 0 ? all : 1, heads, vdim, dim) * rt_cell_bytes(heads, vdim, dim);
}

extern "C" int hds_retention_status(int* stuck) {
    HDS_CHECK_CUDA(cudaMemcpyFromSymbol(stuck, g_ret_stuck, sizeof(int)));
    return HDS_OK;
}

// Returns in *finished 1 when out holds the finished rows, 0 when y holds the read-outs (out still to be normed and gated).
extern "C" int hds_retention(const void* q, const void* k, const void* v, const void* gate, int64_t ld, const float* log2_decay,
                             const float* freq, const float* amp, float k_scale, int norm_cols, float* state, const int32_t* spans, int n_seqs,
                             int n_single, int T, int heads, int vdim, int dim, float* y, int64_t ld_y, void* out, int64_t ld_out,
                             const float* norm_w, float eps, void* workspace, int64_t workspace_bytes, int method, int* finished, int dtype,
                             void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_retention: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(heads >= 1 && vdim >= 1 && vdim <= 8192 && dim >= 2 && dim <= 1024 && dim % 2 == 0, "hds_retention: heads of up to 1024 x 8192");
    HDS_REQUIRE(norm_cols >= 1 && norm_cols <= vdim, "hds_retention: 1 <= norm_cols <= vdim");
    HDS_REQUIRE(method >= 0 && method <= 2, "hds_retention: method 0 / 1 / 2");
    *finished = 1;
    if (T == 0 || n_seqs == 0) return HDS_OK;
    LinArgs a{q, k, v, gate, ld, nullptr, 0, nullptr, 0.0f, state, reinterpret_cast<const SsmSpan*>(spans), n_seqs, T, heads, vdim, dim,
              y, ld_y, out, ld_out, norm_w, eps, 0, norm_cols, 1.0f, k_scale, log2_decay, freq, amp};
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
            rc = rt_chunk_launch(a, n_seqs - n_single, workspace, workspace_bytes, s);
        } else {
            *finished = 0;
            a.write_y = 1;      // by every row of the batch: one norm finishes them all
            rc = lin_launch_scan(a, dtype, true, s);
        }
    }
    if (rc != HDS_OK || n_single == 0) return rc;
    return lin_launch_step(a, dtype, true, s);
}
