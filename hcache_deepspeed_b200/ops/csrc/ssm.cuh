// Shared pieces of the kernels with recurrent state (state-space mixers, delta rules): arguments, the sequences of a ragged batch,
// the inner steps. A delta rule uses the same columns, x = v, B = k, C = q, and has one more per head behind dt (its step input).
#pragma once
#include "hds_host.cuh"
#include "hds_ptx.cuh"

namespace hds {

// One sequence of the batch: first row, new tokens, tokens seen before, slot in the state pools.
struct SsmSpan {
    int32_t row0, n, seen, slot;
};

struct SsmArgs {
    const void* proj;        // [T][ld_proj]: z (inner) | x (inner) | B (groups * N) | C (groups * N) | dt (heads) [| step (heads)]
    int64_t ld_proj;
    const float* conv_w;     // [taps][channels]
    const float* conv_b;     // [channels]
    const float* dt_bias;    // [heads]
    const float* a;          // [heads]: the (negative) decay rates
    const float* d;          // [heads]
    float* state;            // [slots][heads][P][N]
    float* conv_state;       // [slots][taps][channels], ring by position % taps
    const SsmSpan* spans;
    int n_seqs, T;
    int heads, P, N, groups, taps;
    void* u;                 // [T][ld_u]: convolved x | B | C
    int64_t ld_u;
    float* dt;               // [T][heads]: step sizes
    float* y;                // [T][heads * P]
    __host__ __device__ int inner() const { return heads * P; }
    __host__ __device__ int channels() const { return heads * P + 2 * groups * N; }
};

template <int DT>
__device__ __forceinline__ void ssm_store(void* base, int64_t idx, float v) {
    if constexpr (DT == 2) reinterpret_cast<float*>(base)[idx] = v;
    else store_scalar<DT == 0>(base, idx, v);
}
// a value as the activation type holds it
template <int DT>
__device__ __forceinline__ float ssm_round(float v) {
    if constexpr (DT == 0) return __bfloat162float(__float2bfloat16_rn(v));
    if constexpr (DT == 1) return __half2float(__float2half_rn(v));
    return v;
}
// (fast intrinsics where the result is rounded to 16 bits anyway)
template <int DT>
__device__ __forceinline__ float ssm_silu(float v) {
    return DT == 2 ? v / (1.0f + expf(-v)) : __fdividef(v, 1.0f + __expf(-v));
}
__device__ __forceinline__ float ssm_softplus(float v) { return v > 20.0f ? v : log1pf(expf(v)); }

// Latest inputs of a sequence's convolution channels [c0, c1) -> the ring (all threads of the block).
template <int DT>
__device__ __forceinline__ void ssm_save_conv(const SsmArgs& a, const SsmSpan& s, int c0, int c1, int tid, int n_threads) {
    const int C = a.channels(), width = c1 - c0;
    const int k = min(s.n, a.taps);
    for (int e = tid; e < k * width; e += n_threads) {
        const int i = s.n - k + e / width, c = c0 + e % width;
        a.conv_state[(static_cast<int64_t>(s.slot) * a.taps + (s.seen + i) % a.taps) * C + c] =
            load_any<DT>(a.proj, static_cast<int64_t>(s.row0 + i) * a.ld_proj + a.inner() + c);
    }
}
// The part of it that belongs to one head: its x channels, and for the first head of a group the group's B and C.
template <int DT>
__device__ __forceinline__ void ssm_save_conv_of_head(const SsmArgs& a, const SsmSpan& s, int head, int tid, int n_threads) {
    ssm_save_conv<DT>(a, s, head * a.P, (head + 1) * a.P, tid, n_threads);
    const int per = a.heads / a.groups;
    if (head % per == 0) {
        const int b = a.inner() + head / per * a.N;
        ssm_save_conv<DT>(a, s, b, b + a.N, tid, n_threads);
        ssm_save_conv<DT>(a, s, b + a.groups * a.N, b + a.groups * a.N + a.N, tid, n_threads);
    }
}

// convolution + silu of all sequences with several new tokens into u, softplus(dt + bias) into dt (ssm.cu)
int ssm_conv_launch(const SsmArgs& a, int dtype, cudaStream_t s);
bool ssm_chunk_supported(const SsmArgs& a, int dtype);
int ssm_chunk_launch(const SsmArgs& a, int dtype, cudaStream_t s);

}  // namespace hds
