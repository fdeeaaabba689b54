// Mixture-of-experts routing kernels for the ragged forward (tensor-parallel experts, no expert parallelism):
//
//   top-k gating  : softmax over the expert logits of each token, k rounds of arg-max (ties -> lower index), optionally of the
//                   scores plus a per-expert bias; optional renormalisation of the k scores, a factor on them, one atomic per
//                   (token, choice) to claim a row inside the expert. Sigmoid scores (each expert by itself) likewise; or the
//                   bias joins the logits, which choose as they are
//   offsets       : per-expert row ranges padded to the GEMM's 128-row tile (so no A tile straddles two experts);
//                   re-zeroes the counters for the next layer
//   scatter       : copies each token's activation row (optionally times the choice's score) to its k expert rows, records the row
//                   index per choice
//   gather        : out[t] += sum_j score[t, j] * y[row(t, j)]   (fp32, straight into the pending residual delta)
//
// The expert GEMMs in between are ONE grouped tcgen05 launch each (gemm_core.cuh, GemmArgs::group_pad_off).
// Role in the reference: ragged_ops/top_k_gating/top_k_gating_cuda.cu:14-87, moe_scatter/moe_scatter_cuda.cu:22-150,
// moe_gather/moe_gather_cuda.cu:21-112, cutlass_ops/moe_gemm (external library).
#include "hds_host.cuh"
#include "hds_ptx.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kGateThreads = 128;
constexpr int kMoeMaxK = 64;
constexpr int kMoeRowPad = 128;
// softmax scores (+ bias) choose; sigmoids do; softmax scores of logits + bias, chosen by those
enum MoeScores : int { MOE_SOFTMAX = 0, MOE_SIGMOID = 1, MOE_BIASED = 2 };

template <int DT>
__global__ void __launch_bounds__(kGateThreads)
moe_topk_gating_kernel(void* __restrict__ logits, int64_t ld, int E, int k, int normalize, int kind, const float* __restrict__ bias,
                       float scale, int clear, float* __restrict__ scores, int32_t* __restrict__ expert_ids, int32_t* __restrict__ offsets,
                       int32_t* __restrict__ counts) {
    extern __shared__ float probs[];  // [E] scores, [E] what chooses
    float* choice = probs + E;
    __shared__ float red_v[kGateThreads / 32];
    __shared__ int red_i[kGateThreads / 32];
    __shared__ float sel_v[kMoeMaxK];
    __shared__ int sel_i[kMoeMaxK];
    pdl_enter();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bool sigmoid = kind == MOE_SIGMOID, biased = kind == MOE_BIASED;
    float mx = -INFINITY;
    for (int e = tid; e < E; e += kGateThreads) {
        float v = load_any<DT>(logits, static_cast<int64_t>(t) * ld + e);
        if (biased) v += bias[e];
        probs[e] = v;
        mx = fmaxf(mx, v);
        if (DT == 2 && clear) reinterpret_cast<float*>(logits)[static_cast<int64_t>(t) * ld + e] = 0.0f;
    }
    mx = warp_max(mx);
    if (lane == 0) red_v[warp] = mx;
    __syncthreads();
    mx = red_v[0];
#pragma unroll
    for (int w = 1; w < kGateThreads / 32; ++w) mx = fmaxf(mx, red_v[w]);
    __syncthreads();
    float sum = 0.0f;
    for (int e = tid; e < E; e += kGateThreads) {
        if (sigmoid || biased) choice[e] = probs[e];    // (logits choose as scores do, and still where those are all 1 or 0)
        const float p = sigmoid ? 1.0f / (1.0f + expf(-probs[e])) : expf(probs[e] - mx);
        probs[e] = p;
        sum += p;
    }
    sum = warp_sum(sum);
    if (lane == 0) red_v[warp] = sum;
    __syncthreads();
    sum = 0.0f;
#pragma unroll
    for (int w = 0; w < kGateThreads / 32; ++w) sum += red_v[w];
    const float inv = sigmoid ? 1.0f : 1.0f / sum;
    for (int e = tid; e < E; e += kGateThreads)
        if (biased) continue;
        else if (bias != nullptr) choice[e] = fmaf(probs[e], inv, bias[e]);
        else if (!sigmoid) choice[e] = probs[e];
    __syncthreads();
    for (int j = 0; j < k; ++j) {
        float bv = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = tid; e < E; e += kGateThreads) {
            const float p = choice[e];
            if (p > bv || (p == bv && e < bi)) {
                bv = p;
                bi = e;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) {
                bv = ov;
                bi = oi;
            }
        }
        if (lane == 0) {
            red_v[warp] = bv;
            red_i[warp] = bi;
        }
        __syncthreads();
        if (tid == 0) {
            for (int w = 1; w < kGateThreads / 32; ++w) {
                if (red_v[w] > bv || (red_v[w] == bv && red_i[w] < bi)) {
                    bv = red_v[w];
                    bi = red_i[w];
                }
            }
            sel_v[j] = probs[bi] * inv;
            sel_i[j] = bi;
            choice[bi] = -INFINITY;  // taken
        }
        __syncthreads();
    }
    if (tid < k) {
        float s = sel_v[tid];
        if (normalize) {
            float tot = 0.0f;
            for (int j = 0; j < k; ++j) tot += sel_v[j];
            s /= tot;
        }
        const int e = sel_i[tid];
        scores[static_cast<int64_t>(t) * k + tid] = s * scale;
        expert_ids[static_cast<int64_t>(t) * k + tid] = e;
        offsets[static_cast<int64_t>(t) * k + tid] = atomicAdd(&counts[e], 1);
    }
}

// Expert choice by a table of token ids: the same outputs as the gating kernel, every choice with weight 1 / k. Ids outside
// the vocabulary take row 0 (their rows are never read).
__global__ void moe_table_route_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ table, int vocab, int T, int k,
                                       float* __restrict__ scores, int32_t* __restrict__ expert_ids,
                                       int32_t* __restrict__ offsets, int32_t* __restrict__ counts) {
    pdl_enter();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= T * k) return;
    const int id = ids[c / k];
    const int e = table[static_cast<int64_t>(id >= 0 && id < vocab ? id : 0) * k + c % k];
    scores[c] = 1.0f / k;
    expert_ids[c] = e;
    offsets[c] = atomicAdd(&counts[e], 1);
}

// out[t] = base[t] + sum_j score[t, j] * y[row(t, j)]: stores, base optional, scores too (1); `accumulate`: out itself is the base. DT: type of y
// and base.
template <int DT>
__global__ void moe_combine_kernel(const void* __restrict__ y, int64_t ldy, const int32_t* __restrict__ mapped_slots,
                                   const float* __restrict__ scores, const void* __restrict__ base, int64_t ldb,
                                   float* __restrict__ out, int64_t ldo, int H, int k, int accumulate) {
    pdl_enter();
    const int64_t t = blockIdx.x;
    auto add8 = [](const void* p, int64_t idx, float s, float (&v)[8]) {
        if constexpr (DT == 2) {
            const float4* q = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + idx);
            const float4 x = q[0], y = q[1];
            v[0] = fmaf(s, x.x, v[0]); v[1] = fmaf(s, x.y, v[1]); v[2] = fmaf(s, x.z, v[2]); v[3] = fmaf(s, x.w, v[3]);
            v[4] = fmaf(s, y.x, v[4]); v[5] = fmaf(s, y.y, v[5]); v[6] = fmaf(s, y.z, v[6]); v[7] = fmaf(s, y.w, v[7]);
        } else {
            const uint4 x = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(p) + idx * 2);
            v[0] = fmaf(s, unpack_lo<DT == 0>(x.x), v[0]); v[1] = fmaf(s, unpack_hi<DT == 0>(x.x), v[1]);
            v[2] = fmaf(s, unpack_lo<DT == 0>(x.y), v[2]); v[3] = fmaf(s, unpack_hi<DT == 0>(x.y), v[3]);
            v[4] = fmaf(s, unpack_lo<DT == 0>(x.z), v[4]); v[5] = fmaf(s, unpack_hi<DT == 0>(x.z), v[5]);
            v[6] = fmaf(s, unpack_lo<DT == 0>(x.w), v[6]); v[7] = fmaf(s, unpack_hi<DT == 0>(x.w), v[7]);
        }
    };
    for (int c = threadIdx.x * 8; c < H; c += blockDim.x * 8) {
        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (base != nullptr) add8(base, t * ldb + c, 1.0f, v);
        for (int j = 0; j < k; ++j) add8(y, static_cast<int64_t>(mapped_slots[t * k + j]) * ldy + c, scores == nullptr ? 1.0f : scores[t * k + j], v);
        float4* o = reinterpret_cast<float4*>(out + t * ldo + c);
        if (accumulate) {
            const float4 p = o[0], q = o[1];
            v[0] += p.x; v[1] += p.y; v[2] += p.z; v[3] += p.w;
            v[4] += q.x; v[5] += q.y; v[6] += q.z; v[7] += q.w;
        }
        o[0] = make_float4(v[0], v[1], v[2], v[3]);
        o[1] = make_float4(v[4], v[5], v[6], v[7]);
    }
}

__global__ void moe_offsets_kernel(int32_t* __restrict__ counts, int32_t* __restrict__ pad_off, int E) {
    pdl_enter();
    if (threadIdx.x == 0 && blockIdx.x == 0) {
        int acc = 0;
        pad_off[0] = 0;
        for (int e = 0; e < E; ++e) {
            acc += (counts[e] + kMoeRowPad - 1) / kMoeRowPad * kMoeRowPad;
            pad_off[e + 1] = acc;
            counts[e] = 0;
        }
    }
}

// DT: type of the rows where they are weighted (0 bf16, 1 fp16, 2 fp32); without weights H, ldx and lds count 16-bit units of any type
template <int DT>
__global__ void moe_scatter_scaled_kernel(const void* __restrict__ x, int64_t ldx, void* __restrict__ xs, int64_t lds,
                                          const int32_t* __restrict__ expert_ids, const int32_t* __restrict__ offsets,
                                          const int32_t* __restrict__ pad_off, const float* __restrict__ scores,
                                          int32_t* __restrict__ mapped_slots, int H, int k) {
    pdl_enter();
    const int t = blockIdx.x, j = blockIdx.y;
    const int64_t c = static_cast<int64_t>(t) * k + j;
    const int slot = pad_off[expert_ids[c]] + offsets[c];
    const float s = scores[c];
    if (threadIdx.x == 0) mapped_slots[c] = slot;
    const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(x) + static_cast<int64_t>(t) * ldx * 2);
    uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<char*>(xs) + static_cast<int64_t>(slot) * lds * 2);
    auto times = [&](uint32_t v) {
        if constexpr (DT == 2) return __float_as_uint(__uint_as_float(v) * s);
        else return pack2<DT == 0>(unpack_lo<DT == 0>(v) * s, unpack_hi<DT == 0>(v) * s);
    };
    for (int i = threadIdx.x; i < (H >> 3); i += blockDim.x) {
        const uint4 v = src[i];
        dst[i] = make_uint4(times(v.x), times(v.y), times(v.z), times(v.w));
    }
}

__global__ void moe_scatter_kernel(const void* __restrict__ x, int64_t ldx, void* __restrict__ xs, int64_t lds,
                                   const int32_t* __restrict__ expert_ids, const int32_t* __restrict__ offsets,
                                   const int32_t* __restrict__ pad_off, int32_t* __restrict__ mapped_slots, int H, int k) {
    pdl_enter();
    const int t = blockIdx.x, j = blockIdx.y;
    const int64_t c = static_cast<int64_t>(t) * k + j;
    const int slot = pad_off[expert_ids[c]] + offsets[c];
    if (threadIdx.x == 0) mapped_slots[c] = slot;
    const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(x) + static_cast<int64_t>(t) * ldx * 2);
    uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<char*>(xs) + static_cast<int64_t>(slot) * lds * 2);
    for (int i = threadIdx.x; i < (H >> 3); i += blockDim.x) dst[i] = src[i];
}

template <bool kBf16>
__global__ void moe_gather_kernel(const void* __restrict__ y, int64_t ldy, const int32_t* __restrict__ mapped_slots,
                                  const float* __restrict__ scores, float* __restrict__ out, int64_t ldo, int H, int k) {
    pdl_enter();
    const int t = blockIdx.x;
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
        float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        for (int j = 0; j < k; ++j) {
            const int slot = mapped_slots[static_cast<int64_t>(t) * k + j];
            const float s = scores[static_cast<int64_t>(t) * k + j];
            const uint4 q = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(y) +
                                                            (static_cast<int64_t>(slot) * ldy + v * 8) * 2);
            acc[0] += s * unpack_lo<kBf16>(q.x); acc[1] += s * unpack_hi<kBf16>(q.x);
            acc[2] += s * unpack_lo<kBf16>(q.y); acc[3] += s * unpack_hi<kBf16>(q.y);
            acc[4] += s * unpack_lo<kBf16>(q.z); acc[5] += s * unpack_hi<kBf16>(q.z);
            acc[6] += s * unpack_lo<kBf16>(q.w); acc[7] += s * unpack_hi<kBf16>(q.w);
        }
        float4* o = reinterpret_cast<float4*>(out + static_cast<int64_t>(t) * ldo + v * 8);
        float4 a = o[0], b = o[1];
        a.x += acc[0]; a.y += acc[1]; a.z += acc[2]; a.w += acc[3];
        b.x += acc[4]; b.y += acc[5]; b.z += acc[6]; b.w += acc[7];
        o[0] = a;
        o[1] = b;
    }
}

}  // namespace hds

using namespace hds;

extern "C" int hds_moe_topk_gating(void* logits, int64_t ld_logits, int T, int E, int k, int normalize, int kind, const float* bias,
                                   float scale, int clear, int logits_dtype, float* scores, int32_t* expert_ids, int32_t* offsets,
                                   int32_t* counts, void* stream) {
    HDS_REQUIRE(E >= 1 && E <= 4096, "hds_moe_topk_gating: 1..4096 experts");
    HDS_REQUIRE(k >= 1 && k <= kMoeMaxK && k <= E, "hds_moe_topk_gating: top_k must be in 1..64 and <= experts");
    HDS_REQUIRE(logits_dtype >= 0 && logits_dtype <= 2, "hds_moe_topk_gating: logits dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(kind >= 0 && kind <= 2 && (kind != 2 || bias != nullptr), "hds_moe_topk_gating: kind 0 / 1 / 2, the last with a bias");
    HDS_REQUIRE(!clear || logits_dtype == 2, "hds_moe_topk_gating: only fp32 logits are cleared");
    if (T == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const size_t smem = 2 * static_cast<size_t>(E) * sizeof(float);
    cudaError_t rc;
    if (logits_dtype == 0)
        rc = launch_kernel(moe_topk_gating_kernel<0>, dim3(T), dim3(kGateThreads), smem, s, logits, ld_logits, E, k,
                           normalize, kind, bias, scale, clear, scores, expert_ids, offsets, counts);
    else if (logits_dtype == 1)
        rc = launch_kernel(moe_topk_gating_kernel<1>, dim3(T), dim3(kGateThreads), smem, s, logits, ld_logits, E, k,
                           normalize, kind, bias, scale, clear, scores, expert_ids, offsets, counts);
    else
        rc = launch_kernel(moe_topk_gating_kernel<2>, dim3(T), dim3(kGateThreads), smem, s, logits, ld_logits, E, k,
                           normalize, kind, bias, scale, clear, scores, expert_ids, offsets, counts);
    HDS_CHECK_CUDA(rc);
    return HDS_OK;
}

extern "C" int hds_moe_scatter(const void* x, int64_t ldx, void* xs, int64_t ld_xs, const int32_t* expert_ids,
                               const int32_t* offsets, int32_t* counts, int32_t* pad_off, int32_t* mapped_slots, int T,
                               int E, int k, int H, const float* scores, int dtype, void* stream) {
    HDS_REQUIRE(H % 8 == 0 && ldx % 8 == 0 && ld_xs % 8 == 0, "hds_moe_scatter: H and strides must be multiples of 8");
    if (T == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    HDS_CHECK_CUDA(launch_kernel(moe_offsets_kernel, dim3(1), dim3(32), 0, s, counts, pad_off, E));
    const dim3 grid(T, k), block(H / 8 >= 256 ? 256 : 128);
    const int32_t* off = pad_off;
    if (scores == nullptr)
        HDS_CHECK_CUDA(launch_kernel(moe_scatter_kernel, grid, block, 0, s, x, ldx, xs, ld_xs, expert_ids, offsets, off, mapped_slots, H, k));
    else if (dtype == 0)
        HDS_CHECK_CUDA(launch_kernel(moe_scatter_scaled_kernel<0>, grid, block, 0, s, x, ldx, xs, ld_xs, expert_ids, offsets, off, scores, mapped_slots, H, k));
    else if (dtype == 1)
        HDS_CHECK_CUDA(launch_kernel(moe_scatter_scaled_kernel<1>, grid, block, 0, s, x, ldx, xs, ld_xs, expert_ids, offsets, off, scores, mapped_slots, H, k));
    else
        HDS_CHECK_CUDA(launch_kernel(moe_scatter_scaled_kernel<2>, grid, block, 0, s, x, ldx, xs, ld_xs, expert_ids, offsets, off, scores, mapped_slots, H, k));
    return HDS_OK;
}

extern "C" int hds_moe_gather(const void* y, int64_t ldy, const int32_t* mapped_slots, const float* scores, float* out,
                              int64_t ldo, int T, int k, int H, int dtype, void* stream) {
    HDS_REQUIRE(H % 8 == 0 && ldy % 8 == 0 && ldo % 4 == 0, "hds_moe_gather: H / strides must be vector aligned");
    HDS_REQUIRE(dtype == 0 || dtype == 1, "hds_moe_gather: dtype must be 0 (bf16) or 1 (fp16)");
    if (T == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const dim3 block(H / 8 >= 256 ? 256 : 128);
    if (dtype == 0)
        HDS_CHECK_CUDA(launch_kernel(moe_gather_kernel<true>, dim3(T), block, 0, s, y, ldy, mapped_slots, scores, out, ldo, H, k));
    else
        HDS_CHECK_CUDA(launch_kernel(moe_gather_kernel<false>, dim3(T), block, 0, s, y, ldy, mapped_slots, scores, out, ldo, H, k));
    return HDS_OK;
}

extern "C" int64_t hds_moe_padded_rows(int T, int E, int k) {
    // every expert's range is rounded up to the 128-row GEMM tile
    return (static_cast<int64_t>(T) * k + static_cast<int64_t>(E) * (kMoeRowPad - 1)) / kMoeRowPad * kMoeRowPad + kMoeRowPad;
}

extern "C" int hds_moe_table_route(const int32_t* ids, const int32_t* table, int vocab, int T, int E, int k, float* scores,
                                   int32_t* expert_ids, int32_t* offsets, int32_t* counts, void* stream) {
    HDS_REQUIRE(E >= 1 && k >= 1 && k <= E && vocab >= 1, "hds_moe_table_route: 1 <= top_k <= experts, vocab >= 1");
    if (T == 0) return HDS_OK;
    HDS_CHECK_CUDA(launch_kernel(moe_table_route_kernel, dim3((T * k + 255) / 256), dim3(256), 0, static_cast<cudaStream_t>(stream),
                                 ids, table, vocab, T, k, scores, expert_ids, offsets, counts));
    return HDS_OK;
}

extern "C" int hds_moe_combine(const void* y, int64_t ldy, const int32_t* mapped_slots, const float* scores, const void* base,
                               int64_t ldb, float* out, int64_t ldo, int T, int k, int H, int accumulate, int dtype, void* stream) {
    HDS_REQUIRE(H % 8 == 0 && ldy % 8 == 0 && ldo % 4 == 0 && (base == nullptr || ldb % 8 == 0), "hds_moe_combine: rows of 8-value vectors");
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_moe_combine: dtype 0 bf16 / 1 fp16 / 2 fp32");
    if (T == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const dim3 block(H / 8 >= 512 ? 512 : H / 8 >= 256 ? 256 : 128);
    if (dtype == 0)
        HDS_CHECK_CUDA(launch_kernel(moe_combine_kernel<0>, dim3(T), block, 0, s, y, ldy, mapped_slots, scores, base, ldb, out, ldo, H, k, accumulate));
    else if (dtype == 1)
        HDS_CHECK_CUDA(launch_kernel(moe_combine_kernel<1>, dim3(T), block, 0, s, y, ldy, mapped_slots, scores, base, ldb, out, ldo, H, k, accumulate));
    else
        HDS_CHECK_CUDA(launch_kernel(moe_combine_kernel<2>, dim3(T), block, 0, s, y, ldy, mapped_slots, scores, base, ldb, out, ldo, H, k, accumulate));
    return HDS_OK;
}
