// Gated linear attention of prompts on the tensor cores, 64 tokens at a time. With b_t the running sum of a chunk's log2 decays (per key
// channel, the token's own included) and S the state in front of the chunk:
//
//   o_t = (q_t 2^(b_t)) S + sum_{s <= t} (sum_n q_tn k_sn 2^(b_tn - b_sn)) v_s         S <- 2^(b_last) S + sum_s v_s (k_s 2^(b_last - b_s))^T
//
//   lin_local : per (chunk, head): running sums of the decays, and what the chunk's tokens add to the state. Independent of other chunks
//   lin_chain : states in front of every chunk, in place of those sums; advances the state pool. A plain stream along the chunks
//   lin_out   : per (chunk, head): the outputs, normed and gated
//
// Scores come in 16 x 16 blocks. Keys are taken relative to the last token of their block (never grown), queries relative to that same
// token: in blocks below the diagonal never grown either, on it by the decay of 16 tokens at most. Where that exceeds 2^100 the
// block's scores are summed one by one.
//
// Everything fp32 that becomes an operand (decayed q and k, scores, the state) is a bf16 value plus the bf16 rest, 16 significant bits;
// v enters exactly as it is. The tensor work is a small part of the kernels' time, so it is plain warp-level products (mma.sync), whose
// operands are decayed in registers on the way from shared memory. The state's sums are stored as accumulators hold them, and the
// states as operands take them: a thread's 16 bytes are columns 2t, 2t + 1, 2t + 8, 2t + 9 of 16 (of a state: leading terms, then rests).
// Long batches run in segments, which bounds the workspace. (Segments whose intermediate values stay in the L2 cache were slower:
// 64 MiB 270 us, one segment of 195 MiB 243 us for 4096 tokens x 32 heads of 128 x 128; their waves of blocks are too few.)
#include "linear_attention.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kLkTok = 64, kLkThreads = 256, kLkWarps = kLkThreads / 32, kLkP = 128;
constexpr float kLkRange = 100.0f;

struct LinWs {
    float* s;           // [chunks][heads][P][N]: sums, then states (see above)
    float* b;           // [chunks][heads][64][N]: running sums of the log2 decays
    int c0, n;          // chunks [c0, c0 + n) of the batch
};

__device__ __forceinline__ float lk_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
constexpr float kLkLog2e = 1.4426950408889634f;
// log2 of the logistic function of x / log2(e)
__device__ __forceinline__ float lk_log2_sigmoid(float x) { return fminf(x, 0.0f) - __log2f(1.0f + lk_ex2(-fabsf(x))); }
__device__ __forceinline__ void lk_split(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - bf16_lo(hi), v1 - bf16_hi(hi));
}
__device__ __forceinline__ void lk_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lk_ldsm_t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lk_ldsm(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}

__device__ __forceinline__ void lk_copy16(void* dst, const void* src, bool live) {     // (not live: zeros)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void lk_copies_done() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ void lk_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void lk_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }

// eight values, each times 2^w, split into two terms
__device__ __forceinline__ void lk_decay8(uint4 k, const float (&w)[8], uint4& hi, uint4& lo) {
    lk_split(bf16_lo(k.x) * lk_ex2(w[0]), bf16_hi(k.x) * lk_ex2(w[1]), hi.x, lo.x);
    lk_split(bf16_lo(k.y) * lk_ex2(w[2]), bf16_hi(k.y) * lk_ex2(w[3]), hi.y, lo.y);
    lk_split(bf16_lo(k.z) * lk_ex2(w[4]), bf16_hi(k.z) * lk_ex2(w[5]), hi.z, lo.z);
    lk_split(bf16_lo(k.w) * lk_ex2(w[6]), bf16_hi(k.w) * lk_ex2(w[7]), hi.w, lo.w);
}
__device__ __forceinline__ void lk_get8(const float* p, float (&w)[8]) {
    const float4 x = *reinterpret_cast<const float4*>(p), y = *reinterpret_cast<const float4*>(p + 4);
    w[0] = x.x; w[1] = x.y; w[2] = x.z; w[3] = x.w;
    w[4] = y.x; w[5] = y.y; w[6] = y.z; w[7] = y.w;
}

// rows of `width` 16-bit values (a multiple of 8) -> shared rows `pitch` values apart; rows past n are zeros
__device__ __forceinline__ void lk_load(const void* src, int64_t row, int64_t ld, int64_t col, int n, int width, __nv_bfloat16* dst, int pitch) {
    const int vecs = width >> 3;
    for (int e = threadIdx.x; e < kLkTok * vecs; e += kLkThreads) {
        const int t = e / vecs, c = (e - t * vecs) * 8;
        lk_copy16(dst + t * pitch + c, reinterpret_cast<const char*>(src) + ((row + min(t, n - 1)) * ld + col + c) * 2, t < n);
    }
}

__host__ __device__ inline int lk_pitch16(int w) { return w + 8; }

inline size_t lk_local_smem(int N) {
    return static_cast<size_t>(kLkTok) * (2 * lk_pitch16(N) * 2 + lk_pitch16(kLkP) * 2) + 4 * static_cast<size_t>(N) * 4;
}

// NT: the number of key channels where it is known, 0: any; R: pairs of channels x 16 tokens per thread (N <= 128 * R)
template <int NT, int R>
__global__ void __launch_bounds__(kLkThreads, R == 1 ? 3 : 2) lin_local_kernel(const LinArgs a, const LinWs ws) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ ChunkPlace place;
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kLkTok, ws.c0 + blockIdx.x, &place)) return;
    const int N = NT > 0 ? NT : a.N, P = a.P, h = blockIdx.y, p_base = blockIdx.z * kLkP, Pb = min(kLkP, P - p_base);
    const int t0 = place.chunk * kLkTok, n = min(kLkTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0;
    const int kp = lk_pitch16(N), vp = lk_pitch16(kLkP);
    __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(smem);
    __nv_bfloat16* klo = khi + kLkTok * kp;
    __nv_bfloat16* v = klo + kLkTok * kp;
    float* part = reinterpret_cast<float*>(v + kLkTok * vp);        // [4][N]: decays of 16 tokens
    lk_load(a.v, row, a.ld, static_cast<int64_t>(h) * P + p_base, n, Pb, v, vp);
    // a thread's tokens: loads first, then logarithms and their running sums in registers
    const int half = N >> 1;
    uint32_t k[R][16];
    float2 b[R][16];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int u = threadIdx.x + r * kLkThreads, s = u / half * 16, c = (u % half) * 2;
        if (s >= kLkTok) continue;
        uint32_t z[16];
        const char* pz = static_cast<const char*>(a.z) + ((row + s) * a.ld_z + static_cast<int64_t>(h) * N + c) * 2;
        const char* pk = static_cast<const char*>(a.k) + ((row + s) * a.ld + static_cast<int64_t>(h) * N + c) * 2;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            z[i] = k[r][i] = 0;
            if (s + i < n) {
                z[i] = *reinterpret_cast<const uint32_t*>(pz + i * a.ld_z * 2);
                k[r][i] = *reinterpret_cast<const uint32_t*>(pk + i * a.ld * 2);
            }
        }
        float2 bias = *reinterpret_cast<const float2*>(a.bias + static_cast<int64_t>(h) * N + c);
        bias.x *= kLkLog2e;
        bias.y *= kLkLog2e;
        const float floor = -200.0f / a.inv_tau;
        float2 sum = make_float2(0.0f, 0.0f);
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            if (s + i < n) {        // (tokens past the last one do not decay and add nothing)
                sum.x = fmaf(lk_log2_sigmoid(fmaxf(fmaf(bf16_lo(z[i]), kLkLog2e, bias.x), floor)), a.inv_tau, sum.x);
                sum.y = fmaf(lk_log2_sigmoid(fmaxf(fmaf(bf16_hi(z[i]), kLkLog2e, bias.y), floor)), a.inv_tau, sum.y);
            }
            b[r][i] = sum;
        }
        *reinterpret_cast<float2*>(part + u / half * N + c) = sum;
    }
    __syncthreads();
    const int64_t cell = static_cast<int64_t>(blockIdx.x) * a.heads + h;
#pragma unroll
    for (int r = 0; r < R; ++r) {       // keys, each faded to the end of the chunk
        const int u = threadIdx.x + r * kLkThreads, s = u / half * 16, c = (u % half) * 2;
        if (s >= kLkTok) continue;
        float2 last = make_float2(0.0f, 0.0f), before = last;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            if (16 * x == s) before = last;
            const float2 y = *reinterpret_cast<const float2*>(part + x * N + c);
            last.x += y.x;
            last.y += y.y;
        }
        float* g = ws.b + (cell * kLkTok + s) * N + c;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            const float2 x = make_float2(before.x + b[r][i].x, before.y + b[r][i].y);
            if (blockIdx.z == 0) *reinterpret_cast<float2*>(g + static_cast<int64_t>(i) * N) = x;
            uint32_t hi, lo;
            lk_split(bf16_lo(k[r][i]) * lk_ex2(last.x - x.x), bf16_hi(k[r][i]) * lk_ex2(last.y - x.y), hi, lo);
            *reinterpret_cast<uint32_t*>(khi + (s + i) * kp + c) = hi;
            *reinterpret_cast<uint32_t*>(klo + (s + i) * kp + c) = lo;
        }
    }
    lk_copies_done();
    __syncthreads();
    // sums [P][N] = V^T K: units of 16 rows x 32 columns
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int groups = (N + 31) >> 5, units = (Pb >> 4) * groups;
    const int tr = (lane & 7) + ((lane & 16) ? 8 : 0), tc = (lane & 8) ? 8 : 0;     // transposed A: token, column
    const int br = (lane & 7) + ((lane & 8) ? 8 : 0), bc = (lane & 16) ? 8 : 0;     // transposed B: token, column
    float* out = ws.s + cell * P * N;
    for (int u = warp; u < units; u += kLkWarps) {
        const int p0 = u / groups * 16, n0 = u % groups * 32;
        float acc[4][4] = {};
#pragma unroll
        for (int ks = 0; ks < kLkTok; ks += 16) {
            uint32_t av[4], hi[4], lo[4];
            lk_ldsm_t(av, v + (ks + tr) * vp + p0 + tc);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                if (n0 + 16 * j >= N) break;
                const int at = (ks + br) * kp + n0 + 16 * j + bc;
                lk_ldsm_t(hi, khi + at);
                lk_ldsm_t(lo, klo + at);
                lk_mma(acc[2 * j], av, hi[0], hi[1]);
                lk_mma(acc[2 * j + 1], av, hi[2], hi[3]);
                lk_mma(acc[2 * j], av, lo[0], lo[1]);
                lk_mma(acc[2 * j + 1], av, lo[2], lo[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            if (n0 + 16 * j >= N) break;
            float* o = out + static_cast<int64_t>(p_base + p0 + (lane >> 2)) * N + n0 + 16 * j + (lane & 3) * 4;
            *reinterpret_cast<float4*>(o) = make_float4(acc[2 * j][0], acc[2 * j][1], acc[2 * j + 1][0], acc[2 * j + 1][1]);
            *reinterpret_cast<float4*>(o + 8 * static_cast<int64_t>(N)) = make_float4(acc[2 * j][2], acc[2 * j][3], acc[2 * j + 1][2], acc[2 * j + 1][3]);
        }
    }
}

// A thread keeps four state values along the chunks of a sequence that lie in the segment; loads run a step ahead of the stores.
__global__ void __launch_bounds__(kLkThreads) lin_chain_kernel(const LinArgs a, const LinWs ws) {
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int total = span_chunks(sp, kLkTok), base = first_chunk(a.spans, blockIdx.x, kLkTok);
    const int i0 = max(0, ws.c0 - base), i1 = min(total, ws.c0 + ws.n - base);
    const int h = blockIdx.y, N = a.N, e = (blockIdx.z * kLkThreads + threadIdx.x) * 4;
    if (i0 >= i1 || e >= a.P * N) return;
    const int p = e / N, c = ((e - p * N) & ~15) + ((e & 15) >> 1);      // columns c, c + 1, c + 8, c + 9
    float* st = a.state + (static_cast<int64_t>(sp.slot) * a.heads + h) * a.P * N + p * N + c;
    float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
    if (sp.seen > 0 || i0 > 0) {
        const float2 x = *reinterpret_cast<const float2*>(st), y = *reinterpret_cast<const float2*>(st + 8);
        S = make_float4(x.x, x.y, y.x, y.y);
    }
    const int64_t s_step = static_cast<int64_t>(a.heads) * a.P * N, d_step = static_cast<int64_t>(a.heads) * kLkTok * N;
    float* s = ws.s + (base + i0 - ws.c0) * s_step + static_cast<int64_t>(h) * a.P * N + e;
    const float* d = ws.b + (base + i0 - ws.c0) * d_step + (static_cast<int64_t>(h) * kLkTok + kLkTok - 1) * N + c;
    constexpr int U = 4;
    float4 x[U];
    float2 f[U], f8[U];
    int n = i1 - i0;                    // chunks not done yet; the loads are U chunks ahead
    const float* sl = s;
    auto load = [&](int j, bool live) {
        if (!live) return;
        x[j] = __ldcg(reinterpret_cast<const float4*>(sl));
        f[j] = *reinterpret_cast<const float2*>(d);
        f8[j] = *reinterpret_cast<const float2*>(d + 8);
        sl += s_step;
        d += d_step;
    };
    auto step = [&](int j) {
        uint4 o;
        lk_split(S.x, S.y, o.x, o.z);
        lk_split(S.z, S.w, o.y, o.w);
        *reinterpret_cast<uint4*>(s) = o;
        s += s_step;
        S = make_float4(fmaf(lk_ex2(f[j].x), S.x, x[j].x), fmaf(lk_ex2(f[j].y), S.y, x[j].y), fmaf(lk_ex2(f8[j].x), S.z, x[j].z),
                        fmaf(lk_ex2(f8[j].y), S.w, x[j].w));
    };
#pragma unroll
    for (int j = 0; j < U; ++j) load(j, j < n);
    for (; n >= 2 * U; n -= U) {
#pragma unroll
        for (int j = 0; j < U; ++j) {
            step(j);
            load(j, true);
        }
    }
#pragma unroll
    for (int j = 0; j < U; ++j) {
        if (j < n) step(j);
        load(j, U + j < n);
    }
#pragma unroll
    for (int j = 0; j < U; ++j)
        if (U + j < n) step(j);
    *reinterpret_cast<float2*>(st) = make_float2(S.x, S.y);
    *reinterpret_cast<float2*>(st + 8) = make_float2(S.z, S.w);
}

constexpr int kLkAp = 24, kLkAb = 16 * kLkAp;       // a block of scores: 16 rows, their pitch

// Shared memory of lin_out: running sums, q, and a region that holds first the queries decayed from the chunk's start (two terms) and the
// state's stages (16 key channels of 128 rows each), then the decayed keys (two terms) and the scores, at last the values.
constexpr int kLkStages = 3, kLkStage = kLkP * 16 * 4;
__host__ __device__ constexpr int lk_terms_bytes(int N) { return 2 * kLkTok * (N + 8) * 2; }
inline size_t lk_out_smem(int N) {
    const int keys = lk_terms_bytes(N) > kLkTok * lk_pitch16(kLkP) * 2 ? lk_terms_bytes(N) : kLkTok * lk_pitch16(kLkP) * 2;
    const int second = keys + 2 * 10 * kLkAb * 2, first = lk_terms_bytes(N) + kLkStages * kLkStage;
    return static_cast<size_t>(kLkTok) * (lk_pitch16(N) * 4 + lk_pitch16(N) * 2) + (first > second ? first : second);
}

// two neighbouring values of a row, decayed relative to a reference
__device__ __forceinline__ void lk_pair(const __nv_bfloat16* x, const float* b, float2 r, uint32_t& hi, uint32_t& lo) {
    const uint32_t w = *reinterpret_cast<const uint32_t*>(x);
    const float2 d = *reinterpret_cast<const float2*>(b);
    lk_split(bf16_lo(w) * lk_ex2(d.x - r.x), bf16_hi(w) * lk_ex2(d.y - r.y), hi, lo);
}

// NT: as above; kWhole: values in whole blocks of 128
template <int NT, bool kWhole>
__global__ void __launch_bounds__(kLkThreads, 2) lin_out_kernel(const LinArgs a, const LinWs ws) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ ChunkPlace place;
    __shared__ float sq_s[2][kLkTok];
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kLkTok, ws.c0 + blockIdx.x, &place)) return;
    const int N = NT > 0 ? NT : a.N, P = a.P, h = blockIdx.y, p_base = blockIdx.z * kLkP, Pb = kWhole ? kLkP : min(kLkP, P - p_base);
    const int t0 = place.chunk * kLkTok, n = min(kLkTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0;
    const int bp = lk_pitch16(N), kp = lk_pitch16(N), vp = lk_pitch16(kLkP);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c2 = (lane & 3) * 2;
    float* b = reinterpret_cast<float*>(smem);
    __nv_bfloat16* q = reinterpret_cast<__nv_bfloat16*>(b + kLkTok * bp);
    uint8_t* region = reinterpret_cast<uint8_t*>(q + kLkTok * kp);
    __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(region);
    __nv_bfloat16* klo = khi + kLkTok * kp;
    __nv_bfloat16* v = khi;
    __nv_bfloat16* ahi = reinterpret_cast<__nv_bfloat16*>(region + max(lk_terms_bytes(N), kLkTok * lk_pitch16(kLkP) * 2));
    uint8_t* ring = region + lk_terms_bytes(N);
    __nv_bfloat16* alo = ahi + 10 * kLkAb;
    const int64_t cell = static_cast<int64_t>(blockIdx.x) * a.heads + h;
    const bool fresh = place.span.seen == 0 && place.chunk == 0;        // (nothing in front: the state is zero)
    // ---- everything the block reads from far away is on its way before anything is waited for -------------------------------
    {
        const float* src = ws.b + cell * kLkTok * N;
        for (int e = threadIdx.x; e < kLkTok * (N >> 2); e += kLkThreads) {
            const int t = e / (N >> 2), c = (e - t * (N >> 2)) * 4;
            lk_copy16(b + t * bp + c, src + 4 * e, true);
        }
    }
    lk_load(a.q, row, a.ld, static_cast<int64_t>(h) * N, n, N, q, kp);
    lk_commit();
    const int stages = fresh ? 0 : N >> 4;
    auto stage_in = [&](int s) {       // (a group each, empty ones at the end: the counts of what is waited for stay the same)
        if (s < stages) {
            const float* src = ws.s + (cell * P + p_base) * N + 16 * s;
            for (int e = threadIdx.x; e < Pb * 4; e += kLkThreads)
                lk_copy16(ring + s % kLkStages * kLkStage + e * 16, src + static_cast<int64_t>(e >> 2) * N + (e & 3) * 4, true);
        }
        lk_commit();
    };
#pragma unroll
    for (int s = 0; s < kLkStages - 1; ++s) stage_in(s);
    // ---- what the state gives: rows 16 i.. of warp pair i, 64 of the columns each -------------------------------------------
    const int i = warp & 3, half = warp >> 2, pc = half * 64;
    const int nt = kWhole ? 8 : max(0, min(8, (Pb - pc) >> 3));         // blocks of 8 columns (an even number)
    float acc[8][4] = {};
    if (!fresh) {
        lk_wait<kLkStages - 1>();           // sums and q have landed
        __syncthreads();
        for (int e = threadIdx.x; e < kLkTok * (N >> 3); e += kLkThreads) {
            const int t = e / (N >> 3), c = (e - t * (N >> 3)) * 8;
            float w[8];
            uint4 hi, lo;
            lk_get8(b + t * bp + c, w);
            lk_decay8(*reinterpret_cast<const uint4*>(q + t * kp + c), w, hi, lo);
            *reinterpret_cast<uint4*>(khi + t * kp + c) = hi;
            *reinterpret_cast<uint4*>(klo + t * kp + c) = lo;
        }
        const int at = (16 * i + (lane & 15)) * kp + (lane >> 4) * 8;        // A: row, column
        for (int s = 0; s < stages; ++s) {
            lk_wait<kLkStages - 2>();       // stage s (and all in front of it) has landed
            __syncthreads();                // for everybody; and everybody is done with the stage that the next load replaces
            stage_in(s + kLkStages - 1);
            uint32_t qh[4], ql[4];
            lk_ldsm(qh, khi + at + 16 * s);
            lk_ldsm(ql, klo + at + 16 * s);
            const uint4* S = reinterpret_cast<const uint4*>(ring + s % kLkStages * kLkStage) + (pc + g) * 4 + (lane & 3);
            uint4 x[8];
#pragma unroll
            for (int t = 0; t < 8; ++t) x[t] = t < nt ? S[t * 32] : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int t = 0; t < 8; ++t) lk_mma(acc[t], qh, x[t].x, x[t].y);
#pragma unroll
            for (int t = 0; t < 8; ++t) lk_mma(acc[t], qh, x[t].z, x[t].w);
#pragma unroll
            for (int t = 0; t < 8; ++t) lk_mma(acc[t], ql, x[t].x, x[t].y);
        }
    }
    // ---- keys, each faded to the end of its block of 16 ------------------------------------------------------------------------
    lk_copies_done();
    __syncthreads();
    for (int e0 = threadIdx.x; e0 < kLkTok * (N >> 3); e0 += 2 * kLkThreads) {
        uint4 k[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int e = e0 + x * kLkThreads, t = e / (N >> 3), c = (e - t * (N >> 3)) * 8;
            k[x] = make_uint4(0, 0, 0, 0);
            if (t < n) k[x] = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(a.k) + ((row + t) * a.ld + static_cast<int64_t>(h) * N + c) * 2);
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int e = e0 + x * kLkThreads, t = e / (N >> 3), c = (e - t * (N >> 3)) * 8;
            if (t >= kLkTok) break;
            float w[8], end[8];
            uint4 hi, lo;
            lk_get8(b + t * bp + c, w);
            lk_get8(b + (t | 15) * bp + c, end);
#pragma unroll
            for (int y = 0; y < 8; ++y) w[y] = end[y] - w[y];
            lk_decay8(k[x], w, hi, lo);
            *reinterpret_cast<uint4*>(khi + t * kp + c) = hi;
            *reinterpret_cast<uint4*>(klo + t * kp + c) = lo;
        }
    }
    __syncthreads();
    uint4 vr[4];        // this thread's share of the values, on its way during the scores
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        const int e = threadIdx.x + x * kLkThreads, t = e / (Pb >> 3), c = (e - t * (Pb >> 3)) * 8;
        vr[x] = make_uint4(0, 0, 0, 0);
        if (t < n) vr[x] = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(a.v) + ((row + t) * a.ld + static_cast<int64_t>(h) * P + p_base + c) * 2);
    }
    const int nr = (lane & 7) + ((lane & 16) ? 8 : 0), nc = (lane & 8) ? 8 : 0;     // B from rows of keys: key, column
    // ---- scores of the 10 blocks (i, j) on and below the diagonal: a warp makes whole blocks -------------------------------
    for (int blk = warp; blk < 10; blk += kLkWarps) {
        int i = 0, j = blk;
        while (j > i) j -= ++i;
        // (blocks past the last token hold zeros; their rows are never stored and their columns meet zero weights)
        const float* ref = b + (16 * j + 15) * bp;
        bool slow = false;
        if (i == j) {
            for (int c = lane; c < N; c += 32) slow |= b[16 * i * bp + c] - ref[c] > kLkRange;
            slow = __any_sync(0xffffffffu, slow);
        }
        float sc[2][4] = {};
        if (!slow) {
            const __nv_bfloat16* qr = q + (16 * i + g) * kp + c2;
            const float* bq = b + (16 * i + g) * bp + c2;
#pragma unroll 2
            for (int ks = 0; ks < N; ks += 16) {
                const float2 r0 = *reinterpret_cast<const float2*>(ref + ks + c2), r8 = *reinterpret_cast<const float2*>(ref + ks + 8 + c2);
                uint32_t qh[4], ql[4], kh[4], kl[4];
                lk_ldsm(kh, khi + (16 * j + nr) * kp + ks + nc);
                lk_ldsm(kl, klo + (16 * j + nr) * kp + ks + nc);
                lk_pair(qr + ks, bq + ks, r0, qh[0], ql[0]);
                lk_pair(qr + ks + 8 * kp, bq + ks + 8 * bp, r0, qh[1], ql[1]);
                lk_pair(qr + ks + 8, bq + ks + 8, r8, qh[2], ql[2]);
                lk_pair(qr + ks + 8 + 8 * kp, bq + ks + 8 + 8 * bp, r8, qh[3], ql[3]);
#pragma unroll
                for (int t = 0; t < 2; ++t) {
                    lk_mma(sc[t], qh, kh[2 * t], kh[2 * t + 1]);
                    lk_mma(sc[t], qh, kl[2 * t], kl[2 * t + 1]);
                    lk_mma(sc[t], ql, kh[2 * t], kh[2 * t + 1]);
                }
            }
        } else {
            for (int e = 0; e < 8; ++e) {           // this lane's places of the accumulator
                const int t = 16 * i + g + (e & 2 ? 8 : 0), s = 16 * i + (e & 4 ? 8 : 0) + c2 + (e & 1);
                float sum = 0.0f;
                if (s <= t && t < n)
                    for (int c = 0; c < N; ++c)
                        sum = fmaf(__bfloat162float(q[t * kp + c]) * load_any<0>(a.k, (row + s) * a.ld + static_cast<int64_t>(h) * N + c),
                                   lk_ex2(b[t * bp + c] - b[s * bp + c]), sum);
                sc[e >> 2][e & 3] = sum;
            }
        }
        if (i == j) {
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (8 * t + c2 + (e & 1) > g + (e & 2 ? 8 : 0)) sc[t][e] = 0.0f;
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int at = blk * kLkAb + (g + (e ? 8 : 0)) * kLkAp + 8 * t + c2;
                uint32_t hi, lo;
                lk_split(sc[t][e], sc[t][e + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(ahi + at) = hi;
                *reinterpret_cast<uint32_t*>(alo + at) = lo;
            }
    }
    __syncthreads();        // all scores are there, the keys have been used
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        const int e = threadIdx.x + x * kLkThreads, t = e / (Pb >> 3), c = (e - t * (Pb >> 3)) * 8;
        if (t < kLkTok) *reinterpret_cast<uint4*>(v + t * vp + c) = vr[x];
    }
    // gates of this thread's outputs, on their way during the last products
    uint32_t gate[2][8];
    const int64_t col = static_cast<int64_t>(h) * P + p_base + pc + c2;
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            gate[x][t] = 0;
            if (!a.write_y && t < nt && 16 * i + g + 8 * x < n)
                gate[x][t] = *reinterpret_cast<const uint32_t*>(reinterpret_cast<const char*>(a.gate) + ((row + 16 * i + g + 8 * x) * a.ld + col + 8 * t) * 2);
        }
    __syncthreads();
    {
        const int ar = (lane & 7) + ((lane & 8) ? 8 : 0), ac = (lane & 16) ? 8 : 0;
        const int br = (lane & 7) + ((lane & 8) ? 8 : 0), bc = (lane & 16) ? 8 : 0;
        for (int j = 0; j <= i; ++j) {
            uint32_t ah[4], al[4];
            const int at = (i * (i + 1) / 2 + j) * kLkAb + ar * kLkAp + ac;
            lk_ldsm(ah, ahi + at);
            lk_ldsm(al, alo + at);
#pragma unroll
            for (int t = 0; t < 8; t += 2)
                if (t < nt) {
                    uint32_t vv[4];
                    lk_ldsm_t(vv, v + (16 * j + br) * vp + pc + 8 * t + bc);
                    lk_mma(acc[t], ah, vv[0], vv[1]);
                    lk_mma(acc[t + 1], ah, vv[2], vv[3]);
                    lk_mma(acc[t], al, vv[0], vv[1]);
                    lk_mma(acc[t + 1], al, vv[2], vv[3]);
                }
        }
    }
    // ---- norm over the head (its columns lie in this block), gate --------------------------------------------------------------
    const float scale = rsqrtf(static_cast<float>(N)), inv_p = 1.0f / P;
    float2 nw[8];
#pragma unroll
    for (int t = 0; t < 8; ++t) nw[t] = !a.write_y && t < nt ? *reinterpret_cast<const float2*>(a.norm_w + col + 8 * t) : make_float2(0.0f, 0.0f);
    float ss0 = 0.0f, ss8 = 0.0f;
#pragma unroll
    for (int t = 0; t < 8; ++t) {
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[t][e] *= scale;
        ss0 += acc[t][0] * acc[t][0] + acc[t][1] * acc[t][1];
        ss8 += acc[t][2] * acc[t][2] + acc[t][3] * acc[t][3];
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
        ss0 += __shfl_xor_sync(0xffffffffu, ss0, o);
        ss8 += __shfl_xor_sync(0xffffffffu, ss8, o);
    }
    if ((lane & 3) == 0) {
        sq_s[half][16 * i + g] = ss0;
        sq_s[half][16 * i + g + 8] = ss8;
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int t = 16 * i + g + 8 * x;
        if (t >= n) continue;
        const float r = rsqrtf((sq_s[0][t] + sq_s[1][t]) * inv_p + a.eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (j >= nt) continue;
            const float v0 = acc[j][2 * x], v1 = acc[j][2 * x + 1];
            if (a.write_y) {
                *reinterpret_cast<float2*>(a.y + (row + t) * a.ld_y + col + 8 * j) = make_float2(v0, v1);
            } else {
                const uint32_t gw = gate[x][j];
                const float2 w = nw[j];
                *reinterpret_cast<uint32_t*>(reinterpret_cast<char*>(a.out) + ((row + t) * a.ld_out + col + 8 * j) * 2) =
                    pack_bf16(v0 * r * w.x * ssm_silu<0>(bf16_lo(gw)), v1 * r * w.y * ssm_silu<0>(bf16_hi(gw)));
            }
        }
    }
}

// bytes of one (chunk, all heads)
static int64_t lk_cell_bytes(int heads, int P, int N) { return static_cast<int64_t>(heads) * N * (P + kLkTok) * 4; }

// Chunks of a segment: as many as 512 MiB of intermediate values hold.
static int64_t lk_segment(int64_t chunks, int heads, int P, int N) {
    const int64_t n = (int64_t(512) << 20) / lk_cell_bytes(heads, P, N);
    return n >= chunks ? chunks : n > 0 ? n : 1;
}

int64_t lin_chunk_workspace(int T, int n_seqs, int heads, int P, int N) {
    if (N % 16 != 0 || N > 256 || P % 16 != 0) return 0;
    const int64_t all = T / kLkTok + (n_seqs < T / 2 ? n_seqs : T / 2);
    return lk_segment(all > 0 ? all : 1, heads, P, N) * lk_cell_bytes(heads, P, N);
}

bool lin_chunk_supported(const LinArgs& a, int dtype, const void* ws, int64_t ws_bytes) {
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    return dtype == 0 && a.N % 16 == 0 && a.N <= 256 && a.P % 16 == 0 && ws != nullptr && ws_bytes >= lk_cell_bytes(a.heads, a.P, a.N) &&
           aligned(a.q) && aligned(a.k) && aligned(a.v) && aligned(a.z) && aligned(a.gate) && aligned(a.out) && aligned(ws) && aligned(a.state) &&
           a.ld % 8 == 0 && a.ld_z % 8 == 0 && a.ld_out % 8 == 0 && a.ld_y % 2 == 0;
}

int lin_chunk_launch(const LinArgs& a, int n_multi, void* ws, int64_t ws_bytes, cudaStream_t s) {
    const int64_t bound = a.T / kLkTok + n_multi;           // at least as many as there are chunks
    const int64_t fits = ws_bytes / lk_cell_bytes(a.heads, a.P, a.N), seg = lk_segment(bound, a.heads, a.P, a.N);
    const int step = static_cast<int>(seg < fits ? seg : fits);
    const bool whole = a.P % kLkP == 0;
    auto local = a.N == 128 ? lin_local_kernel<128, 1> : a.N == 64 ? lin_local_kernel<64, 1> : a.N <= 128 ? lin_local_kernel<0, 1> : lin_local_kernel<0, 2>;
    auto out = a.N == 128 && whole ? lin_out_kernel<128, true> : a.N == 64 && whole ? lin_out_kernel<64, true> : lin_out_kernel<0, false>;
    HDS_CHECK_CUDA(cudaFuncSetAttribute(local, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(lk_local_smem(a.N))));
    HDS_CHECK_CUDA(cudaFuncSetAttribute(out, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(lk_out_smem(a.N))));
    const unsigned blocks = (a.P + kLkP - 1) / kLkP;
    for (int c0 = 0; c0 < bound; c0 += step) {
        LinWs w;
        w.c0 = c0;
        w.n = static_cast<int>(step < bound - c0 ? step : bound - c0);
        w.s = static_cast<float*>(ws);
        w.b = w.s + static_cast<int64_t>(w.n) * a.heads * a.P * a.N;
        const dim3 grid(w.n, a.heads, blocks), block(kLkThreads);
        HDS_CHECK_CUDA(launch_kernel(local, grid, block, lk_local_smem(a.N), s, a, w));
        HDS_CHECK_CUDA(launch_kernel(lin_chain_kernel, dim3(a.n_seqs, a.heads, (a.P * a.N / 4 + kLkThreads - 1) / kLkThreads), block, 0, s, a, w));
        if (a.out != nullptr || a.write_y)
            HDS_CHECK_CUDA(launch_kernel(out, grid, block, lk_out_smem(a.N), s, a, w));
    }
    return HDS_OK;
}

}  // namespace hds
