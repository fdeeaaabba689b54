// Shared pieces of the linear attention kernels (linear_attention.cu, linear_chunk.cu, retention.cu).
#pragma once
#include "recurrent.cuh"

namespace hds {

struct LinArgs {
    const void* q;          // [T][ld_qk]: heads * N columns each of q, k; [T][ld]: heads * P of v, gate
    const void* k;
    const void* v;
    const void* gate;
    int64_t ld;
    const void* z;          // [T][ld_z]: heads * N inputs of the decays, without their bias
    int64_t ld_z;
    const float* bias;      // [heads * N]
    float inv_tau;
    float* state;           // [slots][heads][P][N]
    const SsmSpan* spans;
    int n_seqs, T, heads, P, N;
    float* y;               // [T][ld_y] read-outs, where they are not finished at once
    int64_t ld_y;
    void* out;              // [T][ld_out], or nullptr: the state alone
    int64_t ld_out;
    const float* norm_w;    // [heads * P], or nullptr: ones
    float eps;
    int write_y;            // steps leave read-outs in y instead of finished rows in out
    int norm_cols;          // values of a head that its norm averages over
    float q_scale, k_scale;
    int64_t ld_qk;              // of q and k
    // retention: a constant decay per head instead of z; q and k are turned by position (freq nullptr: they have been)
    const float* log2_decay;    // [heads]
    const float* freq;          // [N / 2] or nullptr
    const float* amp;           // [N / 2] or nullptr
};

template <int DT>
__device__ __forceinline__ void lin_sincos(float x, float* s, float* c) {
    if constexpr (DT == 2) sincosf(x, s, c);
    else rope_sincos(x, s, c);
}

// sine and cosine of pair c at a position
template <int DT>
__device__ __forceinline__ void lin_turn(const LinArgs& a, float pos, int c, float* s, float* co) {
    *s = 0.0f;
    *co = 1.0f;
    if (a.freq == nullptr) return;
    lin_sincos<DT>(pos * a.freq[c], s, co);
    if (a.amp != nullptr) {
        *s *= a.amp[c];
        *co *= a.amp[c];
    }
}

// values c and N / 2 + c of a head's row, turned
template <int DT>
__device__ __forceinline__ float2 lin_turned(const LinArgs& a, const void* x, int64_t head_row, int c, float s, float co) {
    const float u = load_any<DT>(x, head_row + c), v = load_any<DT>(x, head_row + (a.N >> 1) + c);
    return make_float2(u * co - v * s, v * co + u * s);
}

// log2 of sigmoid(x)^(1 / tau); below 2^-200 a decay is zero to everything behind it
template <int DT>
__device__ __forceinline__ float lin_log2_decay(float x, float inv_tau) {
    constexpr float kLog2e = 1.4426950408889634f;
    float l;
    if constexpr (DT == 2) l = (fminf(x, 0.0f) - log1pf(expf(-fabsf(x)))) * kLog2e;
    else l = fminf(x, 0.0f) * kLog2e - __log2f(1.0f + __expf(-fabsf(x)));
    return fmaxf(l * inv_tau, -200.0f);
}

// token by token (linear_attention.cu): sequences with one new token; with several, which leave their read-outs in y
int lin_launch_step(const LinArgs& a, int dtype, bool retention, cudaStream_t s);
int lin_launch_scan(const LinArgs& a, int dtype, bool retention, cudaStream_t s);

bool lin_chunk_supported(const LinArgs& a, int dtype, const void* ws, int64_t ws_bytes);
int lin_chunk_launch(const LinArgs& a, int n_multi, void* ws, int64_t ws_bytes, cudaStream_t s);
int64_t lin_chunk_workspace(int T, int n_seqs, int heads, int P, int N);

}  // namespace hds
