// Paged attention and KV append for what the tensor-core kernels do not take: fp32 operands, head sizes above 128, and pages of
// one plane whose rows are keys and (their first values) values at once.
// Plain fp32 arithmetic, one warp per (token, query head): lanes hold keys while scores are formed and head dims while values
// are accumulated. Correctness first; the 16-bit kernels (attention_prefill.cu, attention_splitkv.cu) carry the fast path.
#include "hds_host.cuh"
#include "hds_ptx.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kGenWarps = 4;
constexpr int kGenMaxDims = 16;   // value dims per lane: values of up to 512 (kWideDims: 2048)
constexpr int kWideDims = 64;

template <int DT>
__device__ __forceinline__ void store_any(void* base, int64_t idx, float v) {
    if constexpr (DT == 2) reinterpret_cast<float*>(base)[idx] = v;
    else store_scalar<DT == 0>(base, idx, v);
}

// Keys a query at position p sees: [0, keep_first) and (p - window, p] (window 0: all up to p), walked as two ranges. DV: size of
// a value (and of an output head); v_plane: elements from a key row to its value row (0: the same row). Sequences that bring more
// than `limit` tokens are skipped.
template <int DT, int DIMS>
__global__ void __launch_bounds__(kGenWarps * 32)
paged_attn_generic_kernel(const void* __restrict__ q, void* __restrict__ out, int64_t ld_out, const void* __restrict__ cache,
                          const int32_t* __restrict__ tables, int table_stride, const int32_t* __restrict__ tok_seq,
                          const int32_t* __restrict__ tok_pos, int n_units, int n_q, int n_kv, int D, int bs, float scale,
                          int window, int keep_first, int DV, int64_t v_plane, const int32_t* __restrict__ spans, int limit, const AttnOptions opt) {
    extern __shared__ float q_s[];   // [warps][D]
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * kGenWarps + warp;
    if (unit >= n_units) return;
    const int64_t t = unit / n_q;
    const int head = unit % n_q;
    const int kvh = head / (n_q / n_kv);
    if (spans != nullptr && spans[4 * tok_seq[t] + 1] > limit) return;
    const int pos = tok_pos[t];
    const int planes = v_plane > 0 ? 2 : 1;
    const int32_t* table = tables + static_cast<int64_t>(tok_seq[t]) * table_stride;
    float* qw = q_s + warp * D;
    for (int c = lane; c < D; c += 32) qw[c] = load_any<DT>(q, (t * n_q + head) * D + c) * scale;
    __syncwarp();
    float acc[DIMS];
#pragma unroll
    for (int i = 0; i < DIMS; ++i) acc[i] = 0.0f;
    const bool sigmoid = opt.sigmoid_bias != nullptr;      // sigmoid weights: no maximum, no denominator
    const float bias = sigmoid ? opt.sigmoid_bias[head] : 0.0f;
    float m = sigmoid ? 0.0f : -INFINITY, l = 0.0f;
    const int lo = window > 0 ? max(0, pos - window + 1) : 0;
    const int keep_end = min(keep_first, lo);      // the kept range ends where the window takes over
    for (int range = 0; range < 2; ++range) {
        const int j0 = range == 0 ? 0 : lo, j1 = range == 0 ? keep_end : pos + 1;
        for (int b = j0; b < j1; b += 32) {
            const int j = b + lane;
            float s = -INFINITY;
            int64_t vrow = 0;
            if (j < j1) {
                const int blk = table[j / bs], off = j % bs;
                const int64_t krow = ((static_cast<int64_t>(blk) * planes * n_kv + kvh) * bs + off) * D;
                vrow = krow + v_plane;
                s = 0.0f;
                for (int c = 0; c < D; ++c) s = fmaf(qw[c], load_any<DT>(cache, krow + c), s);
                if (opt.softcap > 0.0f) s = opt.softcap * tanhf(s / opt.softcap);
            }
            const float m_new = sigmoid ? 0.0f : fmaxf(m, warp_max(s));
            const float keep = m == -INFINITY ? 0.0f : expf(m - m_new);
            const float p = j >= j1 ? 0.0f : sigmoid ? 1.0f / (1.0f + expf(-(s + bias))) : expf(s - m_new);
            l = l * keep + warp_sum(p);
            m = m_new;
#pragma unroll
            for (int i = 0; i < DIMS; ++i) acc[i] *= keep;
            const int n = min(32, j1 - b);
            for (int k = 0; k < n; ++k) {
                const float pk = __shfl_sync(0xffffffffu, p, k);
                const int64_t vr = __shfl_sync(0xffffffffu, vrow, k);
#pragma unroll
                for (int i = 0; i < DIMS; ++i) {
                    const int c = lane + 32 * i;
                    if (c < DV) acc[i] = fmaf(pk, load_any<DT>(cache, vr + c), acc[i]);
                }
            }
        }
    }
    if (sigmoid) l = 1.0f;
    else if (opt.sink != nullptr) l += expf(opt.sink[head] - m);
#pragma unroll
    for (int i = 0; i < DIMS; ++i) {
        const int c = lane + 32 * i;
        if (c >= DV) continue;
        float o = acc[i] / l;
        if (opt.gate != nullptr) o /= 1.0f + expf(-load_any<DT>(opt.gate, t * opt.gate_ld + head * DV + c));
        store_any<DT>(out, t * ld_out + head * DV + c, o);
    }
}

// dense [T, (n_q + 2 n_kv) * D] -> q rows and the tokens' K / V page rows; copies bytes of `elem` per value
template <typename E>
__global__ void kv_append_generic_kernel(const E* __restrict__ qkv, int64_t ld, E* __restrict__ q_out, E* __restrict__ cache,
                                         const int32_t* __restrict__ tok_slot, int n_q, int n_kv, int D, int bs) {
    pdl_enter();
    const int64_t t = blockIdx.x;
    const int slot = tok_slot[t];
    for (int e = threadIdx.x; e < (n_q + 2 * n_kv) * D; e += blockDim.x) {
        const int h = e / D, c = e % D;
        const E v = qkv[t * ld + e];
        if (h < n_q) {
            q_out[(t * n_q + h) * D + c] = v;
        } else if (slot >= 0) {
            const int kv = h - n_q;
            const int which = kv >= n_kv, kvh = which ? kv - n_kv : kv;
            const int64_t blk = slot / bs, off = slot % bs;
            cache[(((blk * 2 + which) * n_kv + kvh) * bs + off) * D + c] = v;
        }
    }
}

}  // namespace hds

using namespace hds;

extern "C" int hds_paged_attention_generic(const void* q, void* out, int64_t ld_out, const void* kv_cache_layer,
                                           const int32_t* block_tables, int max_blocks_per_seq, const int32_t* tok_seq,
                                           const int32_t* tok_pos, int T, int n_q_heads, int n_kv_heads, int head_dim,
                                           int block_size, float scale, int window, int keep_first, int value_dim,
                                           const int32_t* spans, int limit, int dtype, void* stream) {
    const AttnOptions opt = attn_take_options();
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_paged_attention_generic: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(head_dim >= 1 && value_dim <= head_dim && (value_dim > 0 ? value_dim : head_dim) <= 32 * kWideDims && head_dim <= 2816,
                "hds_paged_attention_generic: values up to 2048, keys up to 2816");
    HDS_REQUIRE(n_kv_heads > 0 && n_q_heads % n_kv_heads == 0, "hds_paged_attention_generic: n_q_heads % n_kv_heads != 0");
    HDS_REQUIRE(window >= 0 && keep_first >= 0, "hds_paged_attention_generic: window and keep_first >= 0");
    if (T == 0) return HDS_OK;
    const int units = T * n_q_heads;
    const int dv = value_dim > 0 ? value_dim : head_dim;
    const int64_t v_plane = value_dim > 0 ? 0 : static_cast<int64_t>(n_kv_heads) * block_size * head_dim;
    const dim3 grid((units + kGenWarps - 1) / kGenWarps), block(kGenWarps * 32);
    const size_t smem = static_cast<size_t>(kGenWarps) * head_dim * 4;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
#define HDS_GEN(DT)                                                                                                          \
    if (dv <= 32 * kGenMaxDims)                                                                                               \
        HDS_CHECK_CUDA(launch_kernel(paged_attn_generic_kernel<DT, kGenMaxDims>, grid, block, smem, s, q, out, ld_out,        \
                                     kv_cache_layer, block_tables, max_blocks_per_seq, tok_seq, tok_pos, units, n_q_heads,    \
                                     n_kv_heads, head_dim, block_size, scale, window, keep_first, dv, v_plane, spans, limit, opt)); \
    else                                                                                                                      \
        HDS_CHECK_CUDA(launch_kernel(paged_attn_generic_kernel<DT, kWideDims>, grid, block, smem, s, q, out, ld_out,          \
                                     kv_cache_layer, block_tables, max_blocks_per_seq, tok_seq, tok_pos, units, n_q_heads,    \
                                     n_kv_heads, head_dim, block_size, scale, window, keep_first, dv, v_plane, spans, limit, opt))
    if (dtype == 0) { HDS_GEN(0); }
    else if (dtype == 1) { HDS_GEN(1); }
    else { HDS_GEN(2); }
#undef HDS_GEN
    return HDS_OK;
}

extern "C" int hds_kv_append_generic(const void* qkv, int64_t ld_qkv, void* q_out, void* kv_cache_layer, const int32_t* tok_slot,
                                     int T, int n_q_heads, int n_kv_heads, int head_dim, int block_size, int elem_bytes,
                                     void* stream) {
    HDS_REQUIRE(elem_bytes == 2 || elem_bytes == 4, "hds_kv_append_generic: 2- or 4-byte elements");
    if (T == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (elem_bytes == 4)
        HDS_CHECK_CUDA(launch_kernel(kv_append_generic_kernel<uint32_t>, dim3(T), dim3(256), 0, s,
                                     static_cast<const uint32_t*>(qkv), ld_qkv, static_cast<uint32_t*>(q_out),
                                     static_cast<uint32_t*>(kv_cache_layer), tok_slot, n_q_heads, n_kv_heads, head_dim, block_size));
    else
        HDS_CHECK_CUDA(launch_kernel(kv_append_generic_kernel<uint16_t>, dim3(T), dim3(256), 0, s,
                                     static_cast<const uint16_t*>(qkv), ld_qkv, static_cast<uint16_t*>(q_out),
                                     static_cast<uint16_t*>(kv_cache_layer), tok_slot, n_q_heads, n_kv_heads, head_dim, block_size));
    return HDS_OK;
}
