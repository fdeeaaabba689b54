// Shared pieces of the gated delta rule kernels (delta.cu, delta_chunk.cu). Arguments are those of the state-space kernels:
// x = v, B = k, C = q, dt = softplus of the decay input, and the step input behind dt in the projections.
#pragma once
#include "ssm.cuh"

namespace hds {

constexpr float kUnitEps = 1e-6f;   // under the root that makes queries and keys unit vectors

struct DeltaArgs {
    SsmArgs s;              // (d and conv skip unused)
    void* out;              // normed and gated output rows, or nullptr: y only
    int64_t ld_out;
    const float* norm_w;    // [heads * P]
    float eps;
};

// columns of the projections behind the convolution's: decay input, step input
template <int DT>
__device__ __forceinline__ float delta_beta(const SsmArgs& a, int64_t row, int h) {
    const float b = load_any<DT>(a.proj, row * a.ld_proj + a.inner() + a.channels() + a.heads + h);
    return 1.0f / (1.0f + expf(-b));
}

// n_multi: sequences of the batch that bring several tokens
bool delta_chunk_supported(const SsmArgs& a, int n_multi, int dtype, int64_t ws_bytes);
int delta_chunk_launch(const SsmArgs& a, int n_multi, int dtype, void* ws, cudaStream_t s);
int64_t delta_chunk_workspace(int T, int n_seqs, int heads, int groups);

}  // namespace hds
