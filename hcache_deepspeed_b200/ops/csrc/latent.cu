// Latent attention around its attention kernels.
//
//   latent_append : behind the layer's input projection [q heads | latent | rotated key part]: rotates the queries' rotated part on
//                   the way to the dense q rows, RMS-norms the latent, rotates the shared key part and writes both into the
//                   token's page row [latent | key part | zeros]. Statistics and angles in fp32.
//   head_matmul   : out[t][h][n] = sum_k x[t][h][k] w[h][k][n], fp32 accumulation: takes queries to the latent space (and copies
//                   their rotated part behind), and mean latents to values. One CTA = 16 tokens of one head
//                   and 64 columns; x is broadcast from shared memory.
#include <type_traits>
#include "hds_host.cuh"
#include "hds_ptx.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

template <int DT>
__device__ __forceinline__ void put(void* base, int64_t idx, float v) {
    if constexpr (DT == 2) reinterpret_cast<float*>(base)[idx] = v;
    else store_scalar<DT == 0>(base, idx, v);
}
template <int DT>
__device__ __forceinline__ void angle_sincos(float x, float* s, float* c) {
    if constexpr (DT == 2) sincosf(x, s, c);
    else rope_sincos(x, s, c);
}

constexpr int kApThreads = 256;

// grid (T, 2): y = 0 the queries, y = 1 the cached row. Adjacent pairs are rotated, so a pair of values is the unit of work.
template <int DT>
__global__ void __launch_bounds__(kApThreads)
latent_append_kernel(const void* __restrict__ proj, int64_t ld, void* __restrict__ q_out, void* __restrict__ pages,
                     const int32_t* __restrict__ tok_pos, const int32_t* __restrict__ tok_slot, int heads, int dim, int rot, int hw,
                     int rank, int width, const float* __restrict__ freq, const float* __restrict__ norm_w, float eps) {
    __shared__ float red[kApThreads / 32];
    __shared__ float cs[2][512];      // cos, sin of this token's angles
    pdl_enter();
    const int64_t t = blockIdx.x;
    const float pos = static_cast<float>(tok_pos[t]);
    const bool cached = blockIdx.y == 1;
    for (int i = threadIdx.x; i < rot / 2; i += kApThreads) angle_sincos<DT>(pos * freq[i], &cs[1][i], &cs[0][i]);
    __syncthreads();
    const int64_t base = t * ld;
    if (!cached) {
        if (q_out == nullptr) return;
        const int half = hw / 2, p0 = dim, p1 = dim + rot;      // (dim may be odd: values are handled one by one then)
        if ((dim & 1) == 0) {
            for (int e = threadIdx.x; e < heads * half; e += kApThreads) {
                const int h = e / half, c = e % half * 2;
                const int64_t src = base + h * hw + c;
                float u = load_any<DT>(proj, src), v = load_any<DT>(proj, src + 1);
                if (c >= p0 && c < p1) {
                    const float co = cs[0][(c - p0) >> 1], si = cs[1][(c - p0) >> 1];
                    const float x = u * co - v * si;
                    v = v * co + u * si;
                    u = x;
                }
                const int64_t dst = (t * heads + h) * hw + c;
                put<DT>(q_out, dst, u);
                put<DT>(q_out, dst + 1, v);
            }
        } else {
            for (int e = threadIdx.x; e < heads * hw; e += kApThreads) {
                const int h = e / hw, c = e % hw;
                float v = load_any<DT>(proj, base + h * hw + c);
                if (c >= p0 && c < p1) {
                    const int i = (c - p0) >> 1;
                    const bool second = (c - p0) & 1;
                    const float w = load_any<DT>(proj, base + h * hw + (second ? c - 1 : c + 1));
                    v = second ? v * cs[0][i] + w * cs[1][i] : v * cs[0][i] - w * cs[1][i];
                }
                put<DT>(q_out, (t * heads + h) * hw + c, v);
            }
        }
        return;
    }
    if (pages == nullptr) return;
    const int slot = tok_slot[t];
    if (slot < 0) return;
    const int64_t src = base + static_cast<int64_t>(heads) * hw, dst = static_cast<int64_t>(slot) * width;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < rank; c += kApThreads) {
        const float v = load_any<DT>(proj, src + c);
        ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.0f;
#pragma unroll
    for (int w = 0; w < kApThreads / 32; ++w) ss += red[w];
    const float r = 1.0f / sqrtf(ss / rank + eps);
    for (int c = threadIdx.x; c < width; c += kApThreads) {
        float v = 0.0f;
        if (c < rank) {
            v = load_any<DT>(proj, src + c) * r * norm_w[c];
        } else if (c < rank + rot) {
            const int i = (c - rank) >> 1;
            const bool second = (c - rank) & 1;
            const float a = load_any<DT>(proj, src + c), b = load_any<DT>(proj, src + (second ? c - 1 : c + 1));
            v = second ? a * cs[0][i] + b * cs[1][i] : a * cs[0][i] - b * cs[1][i];
        }
        put<DT>(pages, dst + c, v);
    }
}

constexpr int kHmTok = 16, kHmCols = 64, kHmSlices = 8, kHmBatch = 16, kHmThreads = kHmCols / 2 * kHmSlices;

// Warp = one of kHmSlices equal parts of K, lane = two neighbouring columns of the CTA's 64; the parts' sums meet in shared memory.
// A thread has kHmBatch weights in flight, the first ones before the kernel in front has finished. Tokens of sequences that bring
// more than `limit` tokens are left alone.
template <int DT>
__global__ void __launch_bounds__(kHmThreads)
head_matmul_kernel(const void* __restrict__ x, int64_t ld_x, int in_width, const void* __restrict__ w, void* __restrict__ out,
                   int64_t ld_out, int out_width, const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ spans, int limit,
                   int T, int K, int N, int copy) {
    extern __shared__ float sm[];
    float* x_s = sm;                      // [K][kHmTok]
    float* part = sm + K * kHmTok;        // [kHmSlices][kHmTok][kHmCols]
    __shared__ int live[kHmTok];
    const int t0 = blockIdx.x * kHmTok, h = blockIdx.y, n0 = blockIdx.z * kHmCols, tid = threadIdx.x;
    const int slice = tid >> 5, n = n0 + 2 * (tid & 31);
    const int per = (K + kHmSlices - 1) / kHmSlices, k0 = min(K, slice * per), k1 = min(K, k0 + per);
    const bool two = n + 1 < N, pair = two && (N & 1) == 0;
    const int64_t wh = static_cast<int64_t>(h) * K * N + n;
    using W = typename std::conditional<DT == 2, float2, uint32_t>::type;
    W q[kHmBatch];
    auto load = [&](int k) {
#pragma unroll
        for (int i = 0; i < kHmBatch; ++i) {
            const bool ok = k + i < k1 && n < N;
            const int64_t wi = wh + static_cast<int64_t>(k + i) * N;
            if constexpr (DT == 2) {
                q[i] = make_float2(ok ? reinterpret_cast<const float*>(w)[wi] : 0.0f, ok && two ? reinterpret_cast<const float*>(w)[wi + 1] : 0.0f);
            } else {
                const uint16_t* p = reinterpret_cast<const uint16_t*>(w) + wi;
                q[i] = !ok ? 0u : pair ? *reinterpret_cast<const uint32_t*>(p) : (p[0] | (two ? static_cast<uint32_t>(p[1]) << 16 : 0u));
            }
        }
    };
    load(k0);
    pdl_enter();
    int any = 0;
    if (tid < kHmTok) {
        live[tid] = t0 + tid < T && spans[4 * tok_seq[t0 + tid] + 1] <= limit;
        any = live[tid];
    }
    if (!__syncthreads_or(any)) return;
    if (DT != 2 && (K & 7) == 0 && (in_width & 7) == 0 && (ld_x & 7) == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0) {
        const int kv = K / 8;
#pragma unroll 4
        for (int e = tid; e < kv * kHmTok; e += kHmThreads) {      // lanes: tokens, so that the transposed stores spread over the banks
            const int i = e % kHmTok, k = e / kHmTok * 8;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (live[i]) v = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(x) +
                                                            (static_cast<int64_t>(t0 + i) * ld_x + static_cast<int64_t>(h) * in_width + k) * 2);
            float* d = x_s + k * kHmTok + i;
            d[0 * kHmTok] = unpack_lo<DT == 0>(v.x); d[1 * kHmTok] = unpack_hi<DT == 0>(v.x);
            d[2 * kHmTok] = unpack_lo<DT == 0>(v.y); d[3 * kHmTok] = unpack_hi<DT == 0>(v.y);
            d[4 * kHmTok] = unpack_lo<DT == 0>(v.z); d[5 * kHmTok] = unpack_hi<DT == 0>(v.z);
            d[6 * kHmTok] = unpack_lo<DT == 0>(v.w); d[7 * kHmTok] = unpack_hi<DT == 0>(v.w);
        }
    } else
    for (int e = tid; e < K * kHmTok; e += kHmThreads) {
        const int i = e / K, k = e % K;
        x_s[k * kHmTok + i] = live[i] ? load_any<DT>(x, static_cast<int64_t>(t0 + i) * ld_x + static_cast<int64_t>(h) * in_width + k) : 0.0f;
    }
    __syncthreads();
    float a[kHmTok][2];
#pragma unroll
    for (int i = 0; i < kHmTok; ++i) a[i][0] = a[i][1] = 0.0f;
    for (int k = k0; k < k1; k += kHmBatch) {
        if (k > k0) load(k);
#pragma unroll
        for (int j = 0; j < kHmBatch; ++j) {
            if (k + j >= k1) break;
            float w0, w1;
            if constexpr (DT == 2) {
                w0 = q[j].x;
                w1 = q[j].y;
            } else {
                w0 = unpack_lo<DT == 0>(q[j]);
                w1 = unpack_hi<DT == 0>(q[j]);
            }
            const float4* xk = reinterpret_cast<const float4*>(x_s + (k + j) * kHmTok);
#pragma unroll
            for (int i = 0; i < kHmTok / 4; ++i) {
                const float4 v = xk[i];
                a[4 * i + 0][0] = fmaf(v.x, w0, a[4 * i + 0][0]); a[4 * i + 0][1] = fmaf(v.x, w1, a[4 * i + 0][1]);
                a[4 * i + 1][0] = fmaf(v.y, w0, a[4 * i + 1][0]); a[4 * i + 1][1] = fmaf(v.y, w1, a[4 * i + 1][1]);
                a[4 * i + 2][0] = fmaf(v.z, w0, a[4 * i + 2][0]); a[4 * i + 2][1] = fmaf(v.z, w1, a[4 * i + 2][1]);
                a[4 * i + 3][0] = fmaf(v.w, w0, a[4 * i + 3][0]); a[4 * i + 3][1] = fmaf(v.w, w1, a[4 * i + 3][1]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < kHmTok; ++i)
        *reinterpret_cast<float2*>(part + (slice * kHmTok + i) * kHmCols + 2 * (tid & 31)) = make_float2(a[i][0], a[i][1]);
    __syncthreads();
    for (int e = tid; e < kHmTok * kHmCols; e += kHmThreads) {
        const int i = e / kHmCols, c = e % kHmCols;
        float s = 0.0f;
#pragma unroll
        for (int z = 0; z < kHmSlices; ++z) s += part[(z * kHmTok + i) * kHmCols + c];
        if (live[i] && n0 + c < N) put<DT>(out, static_cast<int64_t>(t0 + i) * ld_out + static_cast<int64_t>(h) * out_width + n0 + c, s);
    }
    if (blockIdx.z != 0) return;
    // behind the product: `copy` input values that follow the first K, then zeros
    const int rest = out_width - N;
    for (int e = tid; e < kHmTok * rest; e += kHmThreads) {
        const int i = e / rest, c = e % rest;
        if (!live[i]) continue;
        const float v = c < copy ? load_any<DT>(x, static_cast<int64_t>(t0 + i) * ld_x + static_cast<int64_t>(h) * in_width + K + c) : 0.0f;
        put<DT>(out, static_cast<int64_t>(t0 + i) * ld_out + static_cast<int64_t>(h) * out_width + N + c, v);
    }
}

}  // namespace hds

using namespace hds;

extern "C" int hds_latent_append(const void* proj, int64_t ld, void* q_out, void* pages, const int32_t* tok_pos, const int32_t* tok_slot,
                                 int T, int heads, int dim, int rot_dim, int head_width, int rank, int page_width, const float* freq,
                                 const float* norm_w, float eps, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_latent_append: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(rot_dim % 2 == 0 && rot_dim <= 1024 && dim + rot_dim <= head_width && head_width % 2 == 0 && rank + rot_dim <= page_width,
                "hds_latent_append: an even rotated part of at most 1024 values that fits the head and the page row");
    if (T == 0) return HDS_OK;
    const dim3 grid(T, 2), block(kApThreads);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
#define HDS_LA(DT)                                                                                                              \
    HDS_CHECK_CUDA(launch_kernel(latent_append_kernel<DT>, grid, block, 0, s, proj, ld, q_out, pages, tok_pos, tok_slot, heads, dim, \
                                 rot_dim, head_width, rank, page_width, freq, norm_w, eps))
    if (dtype == 0) HDS_LA(0);
    else if (dtype == 1) HDS_LA(1);
    else HDS_LA(2);
#undef HDS_LA
    return HDS_OK;
}

extern "C" int hds_head_matmul(const void* x, int64_t ld_x, int in_width, const void* w, void* out, int64_t ld_out, int out_width,
                               const int32_t* tok_seq, const int32_t* spans, int limit, int T, int heads, int K, int N, int copy, int dtype,
                               void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_head_matmul: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(K >= 1 && N >= 1 && N + copy <= out_width && K + copy <= in_width, "hds_head_matmul: the product fits its rows");
    if (T == 0) return HDS_OK;
    const size_t smem = (static_cast<size_t>(K) * kHmTok + kHmSlices * kHmTok * kHmCols) * 4;
    HDS_REQUIRE(smem <= 220 * 1024, "hds_head_matmul: inner size up to 2900");
    const dim3 grid((T + kHmTok - 1) / kHmTok, heads, (N + kHmCols - 1) / kHmCols), block(kHmThreads);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
#define HDS_HM(DT)                                                                                                             \
    do {                                                                                                                       \
        if (smem > 40 * 1024)                                                                                                  \
            HDS_CHECK_CUDA(cudaFuncSetAttribute(head_matmul_kernel<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize,            \
                                                static_cast<int>(smem)));                                                      \
        HDS_CHECK_CUDA(launch_kernel(head_matmul_kernel<DT>, grid, block, smem, s, x, ld_x, in_width, w, out, ld_out, out_width, \
                                     tok_seq, spans, limit, T, K, N, copy));                                                   \
    } while (0)
    if (dtype == 0) HDS_HM(0);
    else if (dtype == 1) HDS_HM(1);
    else HDS_HM(2);
#undef HDS_HM
    return HDS_OK;
}
