// Gated linear attention of prompts on the tensor cores, 64 tokens at a time. With b_t the running sum of a chunk's log2 decays (per key
// channel, the token's own included) and S the state in front of the chunk:
//
//   o_t = (q_t 2^(b_t)) S + sum_{s <= t} (sum_n q_tn k_sn 2^(b_tn - b_sn)) v_s         S <- 2^(b_last) S + sum_s v_s (k_s 2^(b_last - b_s))^T
//
//   lin_local : per (chunk, head): what its tokens add to the state, and the chunk's whole decay. Independent of all other chunks
//   lin_chain : states in front of every chunk, in place of those sums; advances the state pool. A plain stream along the chunks
//   lin_out   : per (chunk, head): the outputs, normed and gated
//
// No exponent is ever positive by more than a few tokens' decays: the scores of 16 x 16 blocks are products of q and k each taken relative to
// a token between them; inside a block on the diagonal that is its 8th token, and where decays are too strong even for that
// (2^50 in 8 tokens) its scores are summed one by one.
//
// Everything fp32 that becomes an operand (decayed q and k, scores, the state) is a bf16 value plus the bf16 rest, 16 significant bits;
// v enters exactly as it is. The tensor work is a tenth of the kernels' memory time, so it is plain warp-level products
// (mma.sync): operands are decayed in registers on the way from shared memory and need no second staging.
#include "linear_attention.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kLkTok = 64, kLkThreads = 256, kLkWarps = kLkThreads / 32, kLkP = 128;
constexpr float kLkRange = 50.0f;

struct LinWs {
    float* s;           // [chunks][heads][P][N]: sums, then states
    float* d;           // [chunks][heads][N]: 2^(b_last)
    int c0, n;          // chunks [c0, c0 + n) of the batch
};

__device__ __forceinline__ float lk_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
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

// rows of `width` 16-bit values (a multiple of 8) -> shared rows `pitch` values apart; rows past n are zeros
__device__ __forceinline__ void lk_load(const void* src, int64_t row, int64_t ld, int64_t col, int n, int width, __nv_bfloat16* dst, int pitch) {
    const int vecs = width >> 3;
    for (int e = threadIdx.x; e < kLkTok * vecs; e += kLkThreads) {
        const int t = e / vecs, c = (e - t * vecs) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (t < n) v = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(src) + ((row + t) * ld + col + c) * 2);
        *reinterpret_cast<uint4*>(dst + t * pitch + c) = v;
    }
}

// Running sums of the chunk's log2 decays, b [64][pitch]; tokens past n do not decay. `part` [kLkThreads] scratch. All threads; synchronised.
__device__ __forceinline__ void lk_decays(const LinArgs& a, int64_t row, int n, int h, float* b, int pitch, float* part) {
    const int N = a.N, vecs = N >> 3;
    for (int e = threadIdx.x; e < kLkTok * vecs; e += kLkThreads) {
        const int t = e / vecs, c = (e - t * vecs) * 8;
        float l[8] = {};
        if (t < n) {
            const uint4 z = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(a.z) + ((row + t) * a.ld_z + h * N + c) * 2);
            const uint32_t w[4] = {z.x, z.y, z.z, z.w};
            const float* bias = a.bias + h * N + c;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                l[2 * i] = lin_log2_decay<0>(bf16_lo(w[i]) + bias[2 * i], a.inv_tau);
                l[2 * i + 1] = lin_log2_decay<0>(bf16_hi(w[i]) + bias[2 * i + 1], a.inv_tau);
            }
        }
        float4* o = reinterpret_cast<float4*>(b + t * pitch + c);
        o[0] = make_float4(l[0], l[1], l[2], l[3]);
        o[1] = make_float4(l[4], l[5], l[6], l[7]);
    }
    __syncthreads();
    int parts = 1;                              // threads per channel
    while (parts < 8 && 2 * parts * N <= kLkThreads) parts *= 2;
    const int len = kLkTok / parts, p = threadIdx.x / N, c = threadIdx.x - p * N;
    if (p < parts) {
        float s = 0.0f;
        for (int t = p * len; t < (p + 1) * len; ++t) s += b[t * pitch + c];
        part[p * N + c] = s;
    }
    __syncthreads();
    if (p < parts) {
        float s = 0.0f;
        for (int q = 0; q < p; ++q) s += part[q * N + c];
        for (int t = p * len; t < (p + 1) * len; ++t) {
            s += b[t * pitch + c];
            b[t * pitch + c] = s;
        }
    }
    __syncthreads();
}

__host__ __device__ inline int lk_pitch16(int w) { return w + 8; }
__host__ __device__ inline int lk_pitch32(int w) { return w + 8; }

inline size_t lk_local_smem(int N) {
    return static_cast<size_t>(kLkTok) * (lk_pitch32(N) * 4 + 2 * lk_pitch16(N) * 2 + lk_pitch16(kLkP) * 2) + kLkThreads * 4;
}

__global__ void __launch_bounds__(kLkThreads) lin_local_kernel(const LinArgs a, const LinWs ws) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ ChunkPlace place;
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kLkTok, ws.c0 + blockIdx.x, &place)) return;
    const int N = a.N, P = a.P, h = blockIdx.y, p_base = blockIdx.z * kLkP, Pb = min(kLkP, P - p_base);
    const int t0 = place.chunk * kLkTok, n = min(kLkTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0;
    const int bp = lk_pitch32(N), kp = lk_pitch16(N), vp = lk_pitch16(kLkP);
    float* b = reinterpret_cast<float*>(smem);
    __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(b + kLkTok * bp);
    __nv_bfloat16* klo = khi + kLkTok * kp;
    __nv_bfloat16* v = klo + kLkTok * kp;
    float* part = reinterpret_cast<float*>(v + kLkTok * vp);
    lk_load(a.v, row, a.ld, static_cast<int64_t>(h) * P + p_base, n, Pb, v, vp);
    lk_decays(a, row, n, h, b, bp, part);
    // keys, each faded to the end of the chunk
    const float* last = b + (kLkTok - 1) * bp;
    for (int e = threadIdx.x; e < kLkTok * (N >> 2); e += kLkThreads) {
        const int t = e / (N >> 2), c = (e - t * (N >> 2)) * 4;
        uint2 k = make_uint2(0, 0);
        if (t < n) k = *reinterpret_cast<const uint2*>(reinterpret_cast<const char*>(a.k) + ((row + t) * a.ld + static_cast<int64_t>(h) * N + c) * 2);
        const float4 x = *reinterpret_cast<const float4*>(b + t * bp + c), y = *reinterpret_cast<const float4*>(last + c);
        uint2 hi, lo;
        lk_split(bf16_lo(k.x) * lk_ex2(y.x - x.x), bf16_hi(k.x) * lk_ex2(y.y - x.y), hi.x, lo.x);
        lk_split(bf16_lo(k.y) * lk_ex2(y.z - x.z), bf16_hi(k.y) * lk_ex2(y.w - x.w), hi.y, lo.y);
        *reinterpret_cast<uint2*>(khi + t * kp + c) = hi;
        *reinterpret_cast<uint2*>(klo + t * kp + c) = lo;
    }
    const int64_t cell = static_cast<int64_t>(blockIdx.x) * a.heads + h;
    if (blockIdx.z == 0)
        for (int c = threadIdx.x; c < N; c += kLkThreads) ws.d[cell * N + c] = lk_ex2(last[c]);
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
                lk_ldsm_t(hi, khi + (ks + br) * kp + n0 + 16 * j + bc);
                lk_ldsm_t(lo, klo + (ks + br) * kp + n0 + 16 * j + bc);
                lk_mma(acc[2 * j], av, hi[0], hi[1]);
                lk_mma(acc[2 * j + 1], av, hi[2], hi[3]);
                lk_mma(acc[2 * j], av, lo[0], lo[1]);
                lk_mma(acc[2 * j + 1], av, lo[2], lo[3]);
            }
        }
        const int g = lane >> 2, c = (lane & 3) * 2;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (n0 + 8 * j >= N) break;
            float* o = out + static_cast<int64_t>(p_base + p0 + g) * N + n0 + 8 * j + c;
            *reinterpret_cast<float2*>(o) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(o + 8 * static_cast<int64_t>(N)) = make_float2(acc[j][2], acc[j][3]);
        }
    }
}

// A thread keeps four neighbouring state values along the chunks of a sequence that lie in the segment.
__global__ void __launch_bounds__(kLkThreads) lin_chain_kernel(const LinArgs a, const LinWs ws) {
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int total = span_chunks(sp, kLkTok), base = first_chunk(a.spans, blockIdx.x, kLkTok);
    const int i0 = max(0, ws.c0 - base), i1 = min(total, ws.c0 + ws.n - base);
    const int h = blockIdx.y, e = (blockIdx.z * kLkThreads + threadIdx.x) * 4;
    if (i0 >= i1 || e >= a.P * a.N) return;
    const int c = e % a.N;
    float4* st = reinterpret_cast<float4*>(a.state + (static_cast<int64_t>(sp.slot) * a.heads + h) * a.P * a.N + e);
    float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
    if (sp.seen > 0 || i0 > 0) S = *st;
    const int64_t s_step = static_cast<int64_t>(a.heads) * a.P * a.N, d_step = static_cast<int64_t>(a.heads) * a.N;
    float* s = ws.s + (base + i0 - ws.c0) * s_step + static_cast<int64_t>(h) * a.P * a.N + e;
    const float* d = ws.d + (base + i0 - ws.c0) * d_step + static_cast<int64_t>(h) * a.N + c;
    constexpr int U = 4;
    for (int i = i0; i < i1; i += U) {
        float4 x[U], f[U];
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const int k = min(j, i1 - 1 - i);
            x[j] = *reinterpret_cast<const float4*>(s + k * s_step);
            f[j] = *reinterpret_cast<const float4*>(d + k * d_step);
        }
#pragma unroll
        for (int j = 0; j < U; ++j) {
            if (i + j >= i1) break;
            *reinterpret_cast<float4*>(s + j * s_step) = S;
            S = make_float4(fmaf(f[j].x, S.x, x[j].x), fmaf(f[j].y, S.y, x[j].y), fmaf(f[j].z, S.z, x[j].z), fmaf(f[j].w, S.w, x[j].w));
        }
        s += U * s_step;
        d += U * d_step;
    }
    *st = S;
}

constexpr int kLkAp = kLkTok + 8;       // pitch of the scores

inline size_t lk_out_smem(int N) {
    return static_cast<size_t>(kLkTok) * (lk_pitch32(N) * 4 + 2 * lk_pitch16(N) * 2 + lk_pitch16(kLkP) * 2 + 2 * kLkAp * 2) +
           kLkThreads * 4;
}

// two neighbouring decayed values of row r: x 2^(b - ref)
__device__ __forceinline__ void lk_pair(const __nv_bfloat16* x, const float* b, float r0, float r1, float sign, uint32_t& hi, uint32_t& lo) {
    const uint32_t w = *reinterpret_cast<const uint32_t*>(x);
    const float2 d = *reinterpret_cast<const float2*>(b);
    lk_split(bf16_lo(w) * lk_ex2(sign * (d.x - r0)), bf16_hi(w) * lk_ex2(sign * (d.y - r1)), hi, lo);
}

__global__ void __launch_bounds__(kLkThreads, 2) lin_out_kernel(const LinArgs a, const LinWs ws) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ ChunkPlace place;
    __shared__ float sq_s[2][kLkTok];
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kLkTok, ws.c0 + blockIdx.x, &place)) return;
    const int N = a.N, P = a.P, h = blockIdx.y, p_base = blockIdx.z * kLkP, Pb = min(kLkP, P - p_base);
    const int t0 = place.chunk * kLkTok, n = min(kLkTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0;
    const int bp = lk_pitch32(N), kp = lk_pitch16(N), vp = lk_pitch16(kLkP);
    float* b = reinterpret_cast<float*>(smem);
    __nv_bfloat16* q = reinterpret_cast<__nv_bfloat16*>(b + kLkTok * bp);
    __nv_bfloat16* k = q + kLkTok * kp;
    __nv_bfloat16* v = k + kLkTok * kp;
    __nv_bfloat16* ahi = v + kLkTok * vp;
    __nv_bfloat16* alo = ahi + kLkTok * kLkAp;
    float* part = reinterpret_cast<float*>(alo + kLkTok * kLkAp);
    lk_load(a.q, row, a.ld, static_cast<int64_t>(h) * N, n, N, q, kp);
    lk_load(a.k, row, a.ld, static_cast<int64_t>(h) * N, n, N, k, kp);
    lk_load(a.v, row, a.ld, static_cast<int64_t>(h) * P + p_base, n, Pb, v, vp);
    lk_decays(a, row, n, h, b, bp, part);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c2 = (lane & 3) * 2;
    // ---- scores of the 10 blocks (i, j) on and below the diagonal: a warp makes whole blocks -------------------------------
    for (int blk = warp; blk < 10; blk += kLkWarps) {
        int i = 0, j = blk;
        while (j > i) j -= ++i;
        // (blocks past the last token hold zeros; their rows are never stored and their columns meet zero weights)
        const float* ref = b + (i == j ? 16 * i + 7 : 16 * i - 1) * bp;
        bool slow = false;
        if (i == j) {
            for (int c = lane; c < N; c += 32)
                slow |= b[16 * i * bp + c] - ref[c] > kLkRange || ref[c] - b[(16 * i + 15) * bp + c] > kLkRange;
            slow = __any_sync(0xffffffffu, slow);
        }
        float acc[2][4] = {};
        if (!slow) {
            const __nv_bfloat16* qr = q + (16 * i + g) * kp + c2;
            const __nv_bfloat16* kr = k + (16 * j + g) * kp + c2;
            const float* bq = b + (16 * i + g) * bp + c2;
            const float* bk = b + (16 * j + g) * bp + c2;
            for (int ks = 0; ks < N; ks += 16) {
                const float2 r0 = *reinterpret_cast<const float2*>(ref + ks + c2), r8 = *reinterpret_cast<const float2*>(ref + ks + 8 + c2);
                uint32_t qh[4], ql[4], kh[4], kl[4];
                lk_pair(qr + ks, bq + ks, r0.x, r0.y, 1.0f, qh[0], ql[0]);
                lk_pair(qr + ks + 8 * kp, bq + ks + 8 * bp, r0.x, r0.y, 1.0f, qh[1], ql[1]);
                lk_pair(qr + ks + 8, bq + ks + 8, r8.x, r8.y, 1.0f, qh[2], ql[2]);
                lk_pair(qr + ks + 8 + 8 * kp, bq + ks + 8 + 8 * bp, r8.x, r8.y, 1.0f, qh[3], ql[3]);
                lk_pair(kr + ks, bk + ks, r0.x, r0.y, -1.0f, kh[0], kl[0]);
                lk_pair(kr + ks + 8, bk + ks + 8, r8.x, r8.y, -1.0f, kh[1], kl[1]);
                lk_pair(kr + ks + 8 * kp, bk + ks + 8 * bp, r0.x, r0.y, -1.0f, kh[2], kl[2]);
                lk_pair(kr + ks + 8 + 8 * kp, bk + ks + 8 + 8 * bp, r8.x, r8.y, -1.0f, kh[3], kl[3]);
#pragma unroll
                for (int t = 0; t < 2; ++t) {
                    lk_mma(acc[t], qh, kh[2 * t], kh[2 * t + 1]);
                    lk_mma(acc[t], qh, kl[2 * t], kl[2 * t + 1]);
                    lk_mma(acc[t], ql, kh[2 * t], kh[2 * t + 1]);
                }
            }
        } else {
            for (int e = 0; e < 8; ++e) {           // this lane's places of the accumulator
                const int t = 16 * i + g + (e & 2 ? 8 : 0), s = 16 * i + (e & 4 ? 8 : 0) + c2 + (e & 1);
                float sum = 0.0f;
                if (s <= t)
                    for (int c = 0; c < N; ++c)
                        sum = fmaf(__bfloat162float(q[t * kp + c]) * __bfloat162float(k[s * kp + c]), lk_ex2(b[t * bp + c] - b[s * bp + c]), sum);
                acc[e >> 2][e & 3] = sum;
            }
        }
        if (i == j) {
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (8 * t + c2 + (e & 1) > g + (e & 2 ? 8 : 0)) acc[t][e] = 0.0f;
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int at = (16 * i + g + (e ? 8 : 0)) * kLkAp + 16 * j + 8 * t + c2;
                uint32_t hi, lo;
                lk_split(acc[t][e], acc[t][e + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(ahi + at) = hi;
                *reinterpret_cast<uint32_t*>(alo + at) = lo;
            }
    }
    // ---- what the state gives: rows 16 i.. of warp pair i, 64 of the columns each -------------------------------------------
    const int i = warp & 3, half = warp >> 2, pc = half * 64;
    const int nt = max(0, min(8, (Pb - pc) >> 3));         // blocks of 8 columns (an even number)
    float acc[8][4] = {};
    const float* S = ws.s + ((static_cast<int64_t>(blockIdx.x) * a.heads + h) * P + p_base + pc + g) * N + c2;
    const bool fresh = place.span.seen == 0 && place.chunk == 0;        // (nothing in front: the state is zero)
    if (!fresh && nt > 0 && 16 * i < n) {
        const __nv_bfloat16* qr = q + (16 * i + g) * kp + c2;
        const float* bq = b + (16 * i + g) * bp + c2;
        for (int ks = 0; ks < N; ks += 16) {
            uint32_t qh[4], ql[4];
            float2 s0[8], s8[8];
#pragma unroll
            for (int t = 0; t < 8; ++t)
                if (t < nt) {
                    const float* p = S + static_cast<int64_t>(8 * t) * N + ks;
                    s0[t] = *reinterpret_cast<const float2*>(p);
                    s8[t] = *reinterpret_cast<const float2*>(p + 8);
                }
            lk_pair(qr + ks, bq + ks, 0.0f, 0.0f, 1.0f, qh[0], ql[0]);
            lk_pair(qr + ks + 8 * kp, bq + ks + 8 * bp, 0.0f, 0.0f, 1.0f, qh[1], ql[1]);
            lk_pair(qr + ks + 8, bq + ks + 8, 0.0f, 0.0f, 1.0f, qh[2], ql[2]);
            lk_pair(qr + ks + 8 + 8 * kp, bq + ks + 8 + 8 * bp, 0.0f, 0.0f, 1.0f, qh[3], ql[3]);
#pragma unroll
            for (int t = 0; t < 8; ++t)
                if (t < nt) {
                    uint32_t h0, l0, h1, l1;
                    lk_split(s0[t].x, s0[t].y, h0, l0);
                    lk_split(s8[t].x, s8[t].y, h1, l1);
                    lk_mma(acc[t], qh, h0, h1);
                    lk_mma(acc[t], qh, l0, l1);
                    lk_mma(acc[t], ql, h0, h1);
                }
        }
    }
    __syncthreads();        // all scores are there
    {
        const int ar = (lane & 7) + ((lane & 8) ? 8 : 0), ac = (lane & 16) ? 8 : 0;
        const int br = (lane & 7) + ((lane & 8) ? 8 : 0), bc = (lane & 16) ? 8 : 0;
        for (int j = 0; j <= i; ++j) {
            uint32_t ah[4], al[4];
            lk_ldsm(ah, ahi + (16 * i + ar) * kLkAp + 16 * j + ac);
            lk_ldsm(al, alo + (16 * i + ar) * kLkAp + 16 * j + ac);
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
    const float scale = rsqrtf(static_cast<float>(N));
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
        const float r = 1.0f / sqrtf((sq_s[0][t] + sq_s[1][t]) / P + a.eps);
        const int64_t col = static_cast<int64_t>(h) * P + p_base + pc + c2;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (j >= nt) break;
            const float v0 = acc[j][2 * x], v1 = acc[j][2 * x + 1];
            if (a.write_y) {
                *reinterpret_cast<float2*>(a.y + (row + t) * a.ld_y + col + 8 * j) = make_float2(v0, v1);
            } else {
                const uint32_t gw = *reinterpret_cast<const uint32_t*>(reinterpret_cast<const char*>(a.gate) + ((row + t) * a.ld + col + 8 * j) * 2);
                const float2 w = *reinterpret_cast<const float2*>(a.norm_w + col + 8 * j);
                *reinterpret_cast<uint32_t*>(reinterpret_cast<char*>(a.out) + ((row + t) * a.ld_out + col + 8 * j) * 2) =
                    pack_bf16(v0 * r * w.x * ssm_silu<0>(bf16_lo(gw)), v1 * r * w.y * ssm_silu<0>(bf16_hi(gw)));
            }
        }
    }
}

// chunks whose states a workspace of this size holds
static int64_t lk_cell_bytes(int heads, int P, int N) { return static_cast<int64_t>(heads) * N * (P + 1) * 4; }

int64_t lin_chunk_workspace(int T, int n_seqs, int heads, int P, int N) {
    if (N % 16 != 0 || N > 256 || P % 16 != 0) return 0;
    const int64_t cell = lk_cell_bytes(heads, P, N), all = T / kLkTok + (n_seqs < T / 2 ? n_seqs : T / 2), cap = (int64_t(1) << 29) / cell;
    return (all < cap ? (all > 0 ? all : 1) : (cap > 0 ? cap : 1)) * cell;
}

bool lin_chunk_supported(const LinArgs& a, int dtype, const void* ws, int64_t ws_bytes) {
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    return dtype == 0 && a.N % 16 == 0 && a.N <= 256 && a.P % 16 == 0 && ws != nullptr && ws_bytes >= lk_cell_bytes(a.heads, a.P, a.N) &&
           aligned(a.q) && aligned(a.k) && aligned(a.v) && aligned(a.z) && aligned(a.gate) && aligned(a.out) && aligned(ws) &&
           a.ld % 8 == 0 && a.ld_z % 8 == 0 && a.ld_out % 8 == 0 && a.ld_y % 2 == 0;
}

int lin_chunk_launch(const LinArgs& a, int n_multi, void* ws, int64_t ws_bytes, cudaStream_t s) {
    const int64_t cap = ws_bytes / lk_cell_bytes(a.heads, a.P, a.N);
    const int bound = a.T / kLkTok + n_multi;           // at least as many as there are chunks
    HDS_CHECK_CUDA(cudaFuncSetAttribute(lin_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(lk_local_smem(a.N))));
    HDS_CHECK_CUDA(cudaFuncSetAttribute(lin_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(lk_out_smem(a.N))));
    const unsigned blocks = (a.P + kLkP - 1) / kLkP;
    for (int c0 = 0; c0 < bound; c0 += static_cast<int>(cap < bound ? cap : bound)) {
        LinWs w;
        w.c0 = c0;
        w.n = static_cast<int>(cap < bound - c0 ? cap : bound - c0);
        w.s = static_cast<float*>(ws);
        w.d = w.s + static_cast<int64_t>(w.n) * a.heads * a.P * a.N;
        const dim3 grid(w.n, a.heads, blocks), block(kLkThreads);
        HDS_CHECK_CUDA(launch_kernel(lin_local_kernel, grid, block, lk_local_smem(a.N), s, a, w));
        HDS_CHECK_CUDA(launch_kernel(lin_chain_kernel, dim3(a.n_seqs, a.heads, (a.P * a.N / 4 + kLkThreads - 1) / kLkThreads), block, 0, s, a, w));
        if (a.out != nullptr || a.write_y) HDS_CHECK_CUDA(launch_kernel(lin_out_kernel, grid, block, lk_out_smem(a.N), s, a, w));
    }
    return HDS_OK;
}

}  // namespace hds
