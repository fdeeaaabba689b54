// fp32 GEMM  D[M,N] = A[M,K] * W[N,K]^T  in plain FFMA (no reduced-precision matrix mode), with the epilogues of the 16-bit
// kernels: store + activation, gated (interleaved gate / up rows), accumulate, and grouped rows for expert stacks. It serves
// models run entirely in fp32; a 64 x 64 tile per CTA, 4 x 4 outputs per thread.
#include "gemm_core.cuh"
#include "hds_host.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

struct GemmF32Args {
    const float* A;
    int64_t lda;
    const float* W;
    int64_t ldw;
    float* out;
    int64_t ldo;
    int M, N, K, epilogue, act;
    float limit;
    const int32_t* group_off;   // as GemmArgs::group_pad_off
    int n_groups;
    const float* bias;          // [N] or nullptr
};

__device__ __forceinline__ float act_f32(float x, int act) {
    if (act == ACT_SILU) return x / (1.0f + expf(-x));
    if (act == ACT_RELU) return fmaxf(x, 0.0f);
    if (act == ACT_RELU2) return fmaxf(x, 0.0f) * fmaxf(x, 0.0f);
    if (act == ACT_GELU) return 0.5f * x * (1.0f + erff(x * 0.70710678118654752f));
    if (act == ACT_GELU_TANH) return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
    return x;
}

constexpr int kF32Tile = 64, kF32K = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Args g) {
    __shared__ float as[kF32K][kF32Tile + 4], ws[kF32K][kF32Tile + 4];
    pdl_enter();
    const int m0 = blockIdx.y * kF32Tile, n0 = blockIdx.x * kF32Tile;
    const float* W = g.W;
    if (g.group_off != nullptr) {   // ranges are multiples of 128 rows: a 64-row tile never straddles two groups
        if (m0 >= g.group_off[g.n_groups]) return;
        int e = 0;
        while (e + 1 < g.n_groups && g.group_off[e + 1] <= m0) ++e;
        W += static_cast<int64_t>(e) * g.N * g.ldw;
    }
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < g.K; k0 += kF32K) {
        for (int e = threadIdx.x; e < kF32Tile * kF32K; e += 256) {
            const int r = e / kF32K, k = e % kF32K;
            as[k][r] = (m0 + r < g.M && k0 + k < g.K) ? g.A[static_cast<int64_t>(m0 + r) * g.lda + k0 + k] : 0.0f;
            ws[k][r] = (n0 + r < g.N && k0 + k < g.K) ? W[static_cast<int64_t>(n0 + r) * g.ldw + k0 + k] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kF32K; ++k) {
            float a[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = as[k][ty * 4 + i];
                w[i] = ws[k][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= g.M) continue;
        float* row = g.out + static_cast<int64_t>(m) * g.ldo;
        if (g.epilogue == EPI_GATED) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + tx * 4 + j;
                if (n + 1 >= g.N) continue;
                float a = acc[i][j], u = acc[i][j + 1];
                if (g.act == ACT_SWIGLU_CLAMPED) {
                    a = fminf(a, g.limit);
                    u = fminf(fmaxf(u, -g.limit), g.limit) + 1.0f;
                    a = a / (1.0f + expf(-kClampedGluAlpha * a));
                } else {
                    a = act_f32(a, g.act);
                }
                row[n >> 1] = a * u;
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int n = n0 + tx * 4 + j;
                if (n >= g.N) continue;
                if (g.bias != nullptr) acc[i][j] += g.bias[n];
                if (g.epilogue == EPI_RED_F32) row[n] += acc[i][j];
                else row[n] = act_f32(acc[i][j], g.act);
            }
        }
    }
}

}  // namespace hds

using namespace hds;

extern "C" int hds_gemm_f32(const float* A, int64_t lda, const float* W, int64_t ldw, int M, int N, int K, int epilogue, int act,
                            float limit, float* out, int64_t ldo, const int32_t* group_off, int n_groups, const float* bias, void* stream) {
    HDS_REQUIRE(epilogue == EPI_STORE || epilogue == EPI_GATED || epilogue == EPI_RED_F32, "hds_gemm_f32: epilogue 0 / 1 / 2");
    HDS_REQUIRE(epilogue != EPI_GATED || N % 2 == 0, "hds_gemm_f32: gated epilogue needs an even N");
    HDS_REQUIRE(group_off == nullptr || M % 128 == 0, "hds_gemm_f32: grouped rows come in multiples of 128");
    HDS_REQUIRE(bias == nullptr || (epilogue != EPI_GATED && group_off == nullptr), "hds_gemm_f32: a bias goes with plain rows");
    if (M == 0 || N == 0) return HDS_OK;
    GemmF32Args g{A, lda, W, ldw, out, ldo, M, N, K, epilogue, act, limit, group_off, n_groups, bias};
    const dim3 grid((N + kF32Tile - 1) / kF32Tile, (M + kF32Tile - 1) / kF32Tile);
    HDS_REQUIRE(grid.y <= 65535, "hds_gemm_f32: too many rows");
    HDS_CHECK_CUDA(launch_kernel(gemm_f32_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), g));
    return HDS_OK;
}
