// What lies between a layer's projections and its attention where the GEMM's epilogue cannot do it: all of q, and all of k, normed at
// once before the heads are rotated; values mixed with those that another layer cached of the same token.
//
//   attention_append : [q heads | k heads | v heads] rows -> q rows and K / V pages
//   mix_cached       : the value rows of a layer's pages, in place (behind the fused projection of prompts)
//
// Heads are D values wide (their rows were reordered at load): value c < D / 2 is rotated with value D / 2 + c by pos * freq[c];
// values that are not rotated have frequency zero. bf16, fp16 and fp32.
#include "hds_host.cuh"
#include "hds_ptx.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

struct AppendArgs {
    const void* qkv;
    int64_t ld;
    void* q_out;                // [T][n_q * D]
    void* cache;                // [blocks][2][n_kv][bs][D]
    const int32_t* tok_pos;
    const int32_t* tok_slot;    // negative: nothing is cached
    const float* freq;          // [D / 2] or nullptr
    const float* amp;           // [D / 2] factors of sines and cosines, or nullptr
    const float* q_norm;        // [n_q * D] and [n_kv * D], or nullptr
    const float* k_norm;
    int q_cols, k_cols;         // values the two means are taken over (padding excluded)
    float eps;
    const void* first;          // pages whose values are mixed in, heads D1 wide, or nullptr
    int D1;
    const float* share;
    int n_q, n_kv, D, bs;
};

constexpr int kAaThreads = 256;

// V consecutive values as fp32: V = 4 everywhere (heads are multiples of 8 values)
template <int DT>
__device__ __forceinline__ float4 aa_load(const void* p, int64_t i) {
    if constexpr (DT == 2) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
    else {
        const uint2 q = *reinterpret_cast<const uint2*>(reinterpret_cast<const char*>(p) + i * 2);
        return make_float4(unpack_lo<DT == 0>(q.x), unpack_hi<DT == 0>(q.x), unpack_lo<DT == 0>(q.y), unpack_hi<DT == 0>(q.y));
    }
}
template <int DT>
__device__ __forceinline__ void aa_store(void* p, int64_t i, float4 v) {
    if constexpr (DT == 2) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = v;
    else *reinterpret_cast<uint2*>(reinterpret_cast<char*>(p) + i * 2) = make_uint2(pack2<DT == 0>(v.x, v.y), pack2<DT == 0>(v.z, v.w));
}
template <int DT>
__device__ __forceinline__ void aa_sincos(float x, float* s, float* c) {
    if constexpr (DT == 2) sincosf(x, s, c);
    else rope_sincos(x, s, c);
}
__device__ __forceinline__ float4 aa_mix(float4 own, float4 other, float share) {
    const float keep = 1.0f - share;
    return make_float4(keep * own.x + share * other.x, keep * own.y + share * other.y, keep * own.z + share * other.z,
                       keep * own.w + share * other.w);
}

__device__ __forceinline__ void aa_two_sums(float& a, float& b, float* red) {
    a = warp_sum(a);
    b = warp_sum(b);
    if ((threadIdx.x & 31) == 0) {
        red[threadIdx.x >> 5] = a;
        red[8 + (threadIdx.x >> 5)] = b;
    }
    __syncthreads();
    a = b = 0.0f;
#pragma unroll
    for (int w = 0; w < kAaThreads / 32; ++w) {
        a += red[w];
        b += red[8 + w];
    }
}

// One CTA per token.
template <int DT>
__global__ void __launch_bounds__(kAaThreads) attention_append_kernel(const AppendArgs a) {
    extern __shared__ float cs[];      // [D / 2] cosines, [D / 2] sines
    __shared__ float red[16];
    pdl_enter();
    const int64_t t = blockIdx.x;
    const int D = a.D, half = D >> 1, hv = half >> 2;      // hv: vectors of half a head
    const int slot = a.tok_slot[t];
    const int64_t row = t * a.ld;
    if (a.freq != nullptr) {
        const float pos = static_cast<float>(a.tok_pos[t]);
        for (int c = threadIdx.x; c < half; c += kAaThreads) {
            float s, co;
            aa_sincos<DT>(pos * a.freq[c], &s, &co);
            const float m = a.amp != nullptr ? a.amp[c] : 1.0f;
            cs[half + c] = s * m;
            cs[c] = co * m;
        }
    }
    float rq = 1.0f, rk = 1.0f;
    if (a.k_norm != nullptr) {
        float sq = 0.0f, sk = 0.0f;
        for (int e = threadIdx.x * 4; e < (a.n_q + a.n_kv) * D; e += kAaThreads * 4) {
            const float4 v = aa_load<DT>(a.qkv, row + e);
            const float s = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            if (e < a.n_q * D) sq += s;
            else sk += s;
        }
        aa_two_sums(sq, sk, red);
        rq = 1.0f / sqrtf(sq / a.q_cols + a.eps);
        rk = 1.0f / sqrtf(sk / a.k_cols + a.eps);
    }
    __syncthreads();
    const int64_t blk = slot < 0 ? 0 : slot / a.bs, off = slot < 0 ? 0 : slot % a.bs;
    auto page = [&](int which, int h) { return (((blk * 2 + which) * a.n_kv + h) * a.bs + off) * D; };
    // queries and keys: a unit is 4 values of a head's first half and their partners
    for (int u = threadIdx.x; u < (a.n_q + a.n_kv) * hv; u += kAaThreads) {
        const int h = u / hv, c = (u - h * hv) * 4;
        const bool is_q = h < a.n_q;
        if (!is_q && slot < 0) continue;
        const int64_t e = row + static_cast<int64_t>(h) * D + c;
        float4 x = aa_load<DT>(a.qkv, e), y = aa_load<DT>(a.qkv, e + half);
        if (a.k_norm != nullptr) {
            const float r = is_q ? rq : rk;
            const float* w = (is_q ? a.q_norm + h * D : a.k_norm + (h - a.n_q) * D) + c;
            const float4 wx = *reinterpret_cast<const float4*>(w), wy = *reinterpret_cast<const float4*>(w + half);
            x = make_float4(x.x * r * wx.x, x.y * r * wx.y, x.z * r * wx.z, x.w * r * wx.w);
            y = make_float4(y.x * r * wy.x, y.y * r * wy.y, y.z * r * wy.z, y.w * r * wy.w);
        }
        if (a.freq != nullptr) {
            const float4 co = *reinterpret_cast<const float4*>(cs + c), si = *reinterpret_cast<const float4*>(cs + half + c);
            const float4 x0 = x;
            x = make_float4(x.x * co.x - y.x * si.x, x.y * co.y - y.y * si.y, x.z * co.z - y.z * si.z, x.w * co.w - y.w * si.w);
            y = make_float4(y.x * co.x + x0.x * si.x, y.y * co.y + x0.y * si.y, y.z * co.z + x0.z * si.z, y.w * co.w + x0.w * si.w);
        }
        void* dst = is_q ? a.q_out : a.cache;
        const int64_t o = is_q ? (t * a.n_q + h) * D + c : page(0, h - a.n_q) + c;
        aa_store<DT>(dst, o, x);
        aa_store<DT>(dst, o + half, y);
    }
    if (slot < 0 || a.n_kv == 0) return;
    const float share = a.first != nullptr ? *a.share : 0.0f;
    for (int u = threadIdx.x * 4; u < a.n_kv * D; u += kAaThreads * 4) {
        const int h = u / D, c = u - h * D;
        float4 v = aa_load<DT>(a.qkv, row + static_cast<int64_t>(a.n_q + a.n_kv) * D + u);
        if (a.first != nullptr) {
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
            if (c < a.D1) o = aa_load<DT>(a.first, (((blk * 2 + 1) * a.n_kv + h) * a.bs + off) * a.D1 + c);
            v = aa_mix(v, o, share);
        }
        aa_store<DT>(a.cache, page(1, h) + c, v);
    }
}

template <int DT>
__global__ void __launch_bounds__(kAaThreads)
mix_cached_kernel(void* __restrict__ cache, const void* __restrict__ first, const int32_t* __restrict__ tok_slot, const float* __restrict__ share,
                  int64_t units, int n_kv, int D, int D1, int bs) {
    pdl_enter();
    const int64_t u = static_cast<int64_t>(blockIdx.x) * kAaThreads + threadIdx.x;
    if (u >= units) return;
    const int vecs = n_kv * D / 4;
    const int64_t t = u / vecs;
    const int e = static_cast<int>(u - t * vecs) * 4, h = e / D, c = e - h * D;
    const int slot = tok_slot[t];
    if (slot < 0) return;
    const int64_t r = ((static_cast<int64_t>(slot / bs) * 2 + 1) * n_kv + h) * bs + slot % bs;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < D1) o = aa_load<DT>(first, r * D1 + c);
    aa_store<DT>(cache, r * D + c, aa_mix(aa_load<DT>(cache, r * D + c), o, *share));
}

}  // namespace hds

using namespace hds;

extern "C" int hds_attention_append(const void* qkv, int64_t ld_qkv, void* q_out, void* kv_cache_layer, const int32_t* tok_pos,
                                    const int32_t* tok_slot, int T, int n_q_heads, int n_kv_heads, int head_dim, int block_size,
                                    const float* freq, const float* amp, const float* q_norm, const float* k_norm, int q_cols, int k_cols, float eps,
                                    const void* first, int first_dim, const float* share, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_attention_append: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(head_dim >= 8 && head_dim % 8 == 0 && head_dim <= 8192 && ld_qkv % 4 == 0, "hds_attention_append: heads of 8-value multiples");
    HDS_REQUIRE((reinterpret_cast<uintptr_t>(qkv) & 7) == 0, "hds_attention_append: aligned rows");
    HDS_REQUIRE(k_norm == nullptr || (k_cols > 0 && q_cols > 0 && (q_norm != nullptr || n_q_heads == 0)), "hds_attention_append: norms of q and k");
    HDS_REQUIRE(first == nullptr || (share != nullptr && first_dim % 4 == 0), "hds_attention_append: a share for the mixed values");
    if (T == 0) return HDS_OK;
    HDS_REQUIRE(n_kv_heads == 0 || kv_cache_layer != nullptr, "hds_attention_append: pages for the keys and values");
    const AppendArgs a{qkv, ld_qkv, q_out, kv_cache_layer, tok_pos, tok_slot, freq, amp, q_norm, k_norm, q_cols, k_cols, eps,
                       first, first_dim, share, n_q_heads, n_kv_heads, head_dim, block_size};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const size_t smem = static_cast<size_t>(head_dim) * 4;
    if (dtype == 0) HDS_CHECK_CUDA(launch_kernel(attention_append_kernel<0>, dim3(T), dim3(kAaThreads), smem, s, a));
    else if (dtype == 1) HDS_CHECK_CUDA(launch_kernel(attention_append_kernel<1>, dim3(T), dim3(kAaThreads), smem, s, a));
    else HDS_CHECK_CUDA(launch_kernel(attention_append_kernel<2>, dim3(T), dim3(kAaThreads), smem, s, a));
    return HDS_OK;
}

extern "C" int hds_mix_cached_values(void* kv_cache_layer, const void* first, int first_dim, const int32_t* tok_slot, const float* share, int T,
                                     int n_kv_heads, int head_dim, int block_size, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_mix_cached_values: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(head_dim % 8 == 0 && first_dim % 4 == 0, "hds_mix_cached_values: heads of 8-value multiples");
    if (T == 0) return HDS_OK;
    const int64_t units = static_cast<int64_t>(T) * (n_kv_heads * head_dim / 4);
    const dim3 grid(static_cast<unsigned>((units + kAaThreads - 1) / kAaThreads));
    cudaStream_t s = static_cast<cudaStream_t>(stream);
#define HDS_MIX(DT)                                                                                                               \
    HDS_CHECK_CUDA(launch_kernel(mix_cached_kernel<DT>, grid, dim3(kAaThreads), 0, s, kv_cache_layer, first, tok_slot, share, units, \
                                 n_kv_heads, head_dim, first_dim, block_size))
    if (dtype == 0) HDS_MIX(0);
    else if (dtype == 1) HDS_MIX(1);
    else HDS_MIX(2);
#undef HDS_MIX
    return HDS_OK;
}
