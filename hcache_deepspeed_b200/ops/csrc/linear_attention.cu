// Gated linear attention over a ragged batch, per head:  S <- S diag(alpha) + v k^T,  o = S q dim^-1/2, with a decay per key channel,
// alpha = s(z + bias)^(1 / tau) (s the logistic function), then o / rms(o) * weight * silu(gate). The state is kept as [vdim][dim].
// Retention (kRet) has one constant decay per head and turns q and k by position on the way in.
//
//   lin_step : sequences with one new token (decode), norm and gate included
//   lin_scan : sequences with several, token by token in fp32 (fp32 models, and shapes the chunked form does not take)
//   the chunked form (linear_chunk.cu): prompts of bf16 models on the tensor cores
#include "linear_attention.cuh"
#include <math.h>
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kLsThreads = 256, kLsWarps = kLsThreads / 32;

// CTA = (sequence, head). NV > 0: state rows of up to 128 * NV values (a multiple of 4) as float4, R rows in flight per warp; 0: any.
template <int DT, int NV, bool kRet>
__global__ void __launch_bounds__(kLsThreads) lin_step_kernel(const LinArgs a) {
    extern __shared__ float sm[];
    __shared__ float red[kLsWarps];
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n != 1) return;
    const int h = blockIdx.y, N = a.N, P = a.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* q_s = sm;            // [N]
    float* k_s = q_s + N;       // [N]
    float* d_s = k_s + N;       // [N] decays
    float* o_s = d_s + N;       // [P] values, then outputs
    const int64_t row = sp.row0;
    const bool carry = sp.seen > 0;
    float* st = a.state + (static_cast<int64_t>(sp.slot) * a.heads + h) * P * N;
    constexpr int R = NV == 1 ? 8 : NV == 2 ? 4 : 2;
    float4 S[NV > 0 ? R : 1][NV > 0 ? NV : 1];
    auto load_rows = [&](int p0) {
#pragma unroll
        for (int r = 0; r < (NV > 0 ? R : 0); ++r)
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int n = (lane + 32 * j) * 4;
                S[r][j] = carry && p0 + r < P && n < N ? __ldcs(reinterpret_cast<const float4*>(st + static_cast<int64_t>(p0 + r) * N + n))
                                                       : make_float4(0.f, 0.f, 0.f, 0.f);
            }
    };
    if constexpr (NV > 0) load_rows(warp * R);
    const float keep = kRet ? exp2f(a.log2_decay[h]) : 0.0f;
    if constexpr (kRet) {
        const float pos = static_cast<float>(sp.seen);
        for (int c = threadIdx.x; c < N >> 1; c += kLsThreads) {
            float s, co;
            lin_turn<DT>(a, pos, c, &s, &co);
            const int64_t at = row * a.ld_qk + h * N;
            const float2 q = lin_turned<DT>(a, a.q, at, c, s, co), k = lin_turned<DT>(a, a.k, at, c, s, co);
            q_s[c] = q.x * a.q_scale;
            q_s[c + (N >> 1)] = q.y * a.q_scale;
            k_s[c] = k.x * a.k_scale;
            k_s[c + (N >> 1)] = k.y * a.k_scale;
        }
    } else {
        for (int n = threadIdx.x; n < N; n += kLsThreads) {
            q_s[n] = load_any<DT>(a.q, row * a.ld_qk + h * N + n) * a.q_scale;
            k_s[n] = load_any<DT>(a.k, row * a.ld_qk + h * N + n) * a.k_scale;
            d_s[n] = exp2f(lin_log2_decay<DT>(load_any<DT>(a.z, row * a.ld_z + h * N + n) + a.bias[h * N + n], a.inv_tau));
        }
    }
    for (int p = threadIdx.x; p < P; p += kLsThreads) o_s[p] = load_any<DT>(a.v, row * a.ld + h * P + p);
    __syncthreads();
    float ss = 0.0f;
    if constexpr (NV > 0) {
        for (int p0 = warp * R; p0 < P; p0 += kLsWarps * R) {
            if (p0 != warp * R) load_rows(p0);
            float sq[R] = {}, v[R];
#pragma unroll
            for (int r = 0; r < R; ++r) v[r] = p0 + r < P ? o_s[p0 + r] : 0.0f;
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int n = (lane + 32 * j) * 4;
                if (n >= N) continue;
                const float4 q = *reinterpret_cast<const float4*>(q_s + n), k = *reinterpret_cast<const float4*>(k_s + n),
                             d = kRet ? make_float4(keep, keep, keep, keep) : *reinterpret_cast<const float4*>(d_s + n);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    float4 x = S[r][j];
                    x.x = fmaf(v[r], k.x, d.x * x.x); x.y = fmaf(v[r], k.y, d.y * x.y);
                    x.z = fmaf(v[r], k.z, d.z * x.z); x.w = fmaf(v[r], k.w, d.w * x.w);
                    sq[r] += x.x * q.x + x.y * q.y + x.z * q.z + x.w * q.w;
                    if (p0 + r < P) __stcs(reinterpret_cast<float4*>(st + static_cast<int64_t>(p0 + r) * N + n), x);
                }
            }
            float mine = 0.0f;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float o = warp_sum(sq[r]);
                if (lane == r) mine = o;
            }
            if (lane < R && p0 + lane < P) {
                o_s[p0 + lane] = mine;       // (a row's value has been read by its own warp)
                ss = fmaf(mine, mine, ss);
            }
        }
    } else {
        for (int p = warp; p < P; p += kLsWarps) {
            float sq = 0.0f;
            const float v = o_s[p];
            float* r = st + static_cast<int64_t>(p) * N;
            for (int n = lane; n < N; n += 32) {
                const float x = fmaf(v, k_s[n], carry ? (kRet ? keep : d_s[n]) * r[n] : 0.0f);
                r[n] = x;
                sq = fmaf(x, q_s[n], sq);
            }
            sq = warp_sum(sq);
            __syncwarp();
            if (lane == 0) {
                o_s[p] = sq;
                ss = fmaf(sq, sq, ss);
            }
        }
    }
    if (a.write_y) {
        __syncthreads();
        for (int p = threadIdx.x; p < P; p += kLsThreads) a.y[row * a.ld_y + h * P + p] = o_s[p];
        return;
    }
    if (a.out == nullptr) return;
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.0f;
#pragma unroll
    for (int w = 0; w < kLsWarps; ++w) ss += red[w];
    const float r = 1.0f / sqrtf(ss / a.norm_cols + a.eps);
    for (int p = threadIdx.x; p < P; p += kLsThreads) {
        const float g = load_any<DT>(a.gate, row * a.ld + h * P + p);
        ssm_store<DT>(a.out, row * a.ld_out + h * P + p, o_s[p] * r * (a.norm_w != nullptr ? a.norm_w[h * P + p] : 1.0f) * ssm_silu<DT>(g));
    }
}

// CTA = (sequence, head, 16 rows): a warp keeps 4 rows, NL state values of each per lane.
constexpr int kLcWarps = 4, kLcRows = 4, kLcP = kLcWarps * kLcRows, kLcTok = 16;

template <int DT, int NL, bool kRet>
__global__ void __launch_bounds__(kLcWarps * 32) lin_scan_kernel(const LinArgs a) {
    extern __shared__ float sm[];
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int h = blockIdx.y, p0 = blockIdx.z * kLcP, N = a.N, P = a.P;
    float* k_s = sm;                        // [tok][N]
    float* q_s = k_s + kLcTok * N;
    float* d_s = q_s + kLcTok * N;
    float* v_s = d_s + kLcTok * N;          // [tok][kLcP]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float keep = kRet ? exp2f(a.log2_decay[h]) : 0.0f;
    float S[kLcRows][NL];
    float* st = a.state + (static_cast<int64_t>(sp.slot) * a.heads + h) * P * N;
#pragma unroll
    for (int r = 0; r < kLcRows; ++r)
#pragma unroll
        for (int j = 0; j < NL; ++j) {
            const int p = p0 + warp * kLcRows + r, n = lane + 32 * j;
            S[r][j] = (sp.seen > 0 && p < P && n < N) ? st[static_cast<int64_t>(p) * N + n] : 0.0f;
        }
    for (int t0 = 0; t0 < sp.n; t0 += kLcTok) {
        const int nt = min(kLcTok, sp.n - t0);
        const int64_t row = sp.row0 + t0;
        __syncthreads();
        if constexpr (kRet) {
            const int half = N >> 1;
            for (int e = threadIdx.x; e < nt * half; e += blockDim.x) {
                const int t = e / half, c = e - t * half;
                const int64_t at = (row + t) * a.ld_qk + h * N;
                float s, co;
                lin_turn<DT>(a, static_cast<float>(sp.seen + t0 + t), c, &s, &co);
                const float2 q = lin_turned<DT>(a, a.q, at, c, s, co), k = lin_turned<DT>(a, a.k, at, c, s, co);
                q_s[t * N + c] = q.x * a.q_scale;
                q_s[t * N + half + c] = q.y * a.q_scale;
                k_s[t * N + c] = k.x * a.k_scale;
                k_s[t * N + half + c] = k.y * a.k_scale;
            }
        }
        for (int e = threadIdx.x; !kRet && e < nt * N; e += blockDim.x) {
            const int t = e / N, n = e - t * N;
            const int64_t at = (row + t) * a.ld_qk + h * N + n;
            k_s[e] = load_any<DT>(a.k, at) * a.k_scale;
            q_s[e] = load_any<DT>(a.q, at) * a.q_scale;
            d_s[e] = exp2f(lin_log2_decay<DT>(load_any<DT>(a.z, (row + t) * a.ld_z + h * N + n) + a.bias[h * N + n], a.inv_tau));
        }
        for (int e = threadIdx.x; e < nt * kLcP; e += blockDim.x) {
            const int p = p0 + e % kLcP;
            v_s[e] = p < P ? load_any<DT>(a.v, (row + e / kLcP) * a.ld + h * P + p) : 0.0f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            float sq[kLcRows] = {};
#pragma unroll
            for (int j = 0; j < NL; ++j) {
                const int n = lane + 32 * j;
                const float k = n < N ? k_s[t * N + n] : 0.0f, q = n < N ? q_s[t * N + n] : 0.0f, d = kRet ? keep : n < N ? d_s[t * N + n] : 0.0f;
#pragma unroll
                for (int r = 0; r < kLcRows; ++r) {
                    S[r][j] = fmaf(v_s[t * kLcP + warp * kLcRows + r], k, d * S[r][j]);
                    sq[r] = fmaf(S[r][j], q, sq[r]);
                }
            }
#pragma unroll
            for (int r = 0; r < kLcRows; ++r) {
                const float o = warp_sum(sq[r]);
                const int p = p0 + warp * kLcRows + r;
                if (lane == r && p < P) a.y[(row + t) * a.ld_y + h * P + p] = o;
            }
        }
    }
#pragma unroll
    for (int r = 0; r < kLcRows; ++r)
#pragma unroll
        for (int j = 0; j < NL; ++j) {
            const int p = p0 + warp * kLcRows + r, n = lane + 32 * j;
            if (p < P && n < N) st[static_cast<int64_t>(p) * N + n] = S[r][j];
        }
}

template <int DT, bool kRet>
static int launch_step(const LinArgs& a, cudaStream_t s) {
    const dim3 grid(a.n_seqs, a.heads), block(kLsThreads);
    const size_t smem = (3 * static_cast<size_t>(a.N) + a.P) * 4;
#define HDS_LS(NV) HDS_CHECK_CUDA(launch_kernel(lin_step_kernel<DT, NV, kRet>, grid, block, smem, s, a))
    if (a.N % 4 != 0 || a.N > 512) HDS_LS(0);
    else if (a.N <= 128) HDS_LS(1);
    else if (a.N <= 256) HDS_LS(2);
    else HDS_LS(4);
#undef HDS_LS
    return HDS_OK;
}

template <int DT, bool kRet>
static int launch_scan(const LinArgs& a, cudaStream_t s) {
    const dim3 grid(a.n_seqs, a.heads, (a.P + kLcP - 1) / kLcP), block(kLcWarps * 32);
    const size_t smem = static_cast<size_t>(kLcTok) * (3 * a.N + kLcP) * 4;
#define HDS_LC(NL)                                                                                                                                \
    do {                                                                                                                                          \
        HDS_CHECK_CUDA(cudaFuncSetAttribute(lin_scan_kernel<DT, NL, kRet>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem))); \
        HDS_CHECK_CUDA(launch_kernel(lin_scan_kernel<DT, NL, kRet>, grid, block, smem, s, a));                                                    \
    } while (0)
    if (a.N <= 32) HDS_LC(1);
    else if (a.N <= 64) HDS_LC(2);
    else if (a.N <= 128) HDS_LC(4);
    else if (a.N <= 256) HDS_LC(8);
    else if (a.N <= 512) HDS_LC(16);
    else HDS_LC(32);
#undef HDS_LC
    return HDS_OK;
}

template <bool kRet>
static int launch_tokens(bool step, const LinArgs& a, int dtype, cudaStream_t s) {
    if (step) return dtype == 0 ? launch_step<0, kRet>(a, s) : dtype == 1 ? launch_step<1, kRet>(a, s) : launch_step<2, kRet>(a, s);
    return dtype == 0 ? launch_scan<0, kRet>(a, s) : dtype == 1 ? launch_scan<1, kRet>(a, s) : launch_scan<2, kRet>(a, s);
}
int lin_launch_step(const LinArgs& a, int dtype, bool retention, cudaStream_t s) {
    return retention ? launch_tokens<true>(true, a, dtype, s) : launch_tokens<false>(true, a, dtype, s);
}
int lin_launch_scan(const LinArgs& a, int dtype, bool retention, cudaStream_t s) {
    return retention ? launch_tokens<true>(false, a, dtype, s) : launch_tokens<false>(false, a, dtype, s);
}

}  // namespace hds

using namespace hds;

extern "C" int64_t hds_linear_attention_workspace_bytes(int T, int n_seqs, int heads, int vdim, int dim) {
    return lin_chunk_workspace(T, n_seqs, heads, vdim, dim);
}

// Returns 1 when out holds the finished rows, 0 when y holds the read-outs of the rows (out still to be normed and gated).
extern "C" int hds_linear_attention(const void* q, const void* k, const void* v, const void* gate, int64_t ld, const void* z, int64_t ld_z,
                                    const float* bias, float inv_tau, float* state, const int32_t* spans, int n_seqs, int n_single, int T,
                                    int heads, int vdim, int dim, float* y, int64_t ld_y, void* out, int64_t ld_out, const float* norm_w,
                                    float eps, void* workspace, int64_t workspace_bytes, int method, int* finished, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_linear_attention: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(heads >= 1 && vdim >= 1 && vdim <= 8192 && dim >= 1 && dim <= 1024, "hds_linear_attention: heads of up to 1024 x 8192");
    HDS_REQUIRE(method >= 0 && method <= 2, "hds_linear_attention: method 0 / 1 / 2");
    *finished = 1;
    if (T == 0 || n_seqs == 0) return HDS_OK;
    LinArgs a{q, k, v, gate, ld, z, ld_z, bias, inv_tau, state, reinterpret_cast<const SsmSpan*>(spans), n_seqs, T, heads, vdim, dim,
              y, ld_y, out, ld_out, norm_w, eps, 0, vdim, 1.0f / sqrtf(static_cast<float>(dim)), 1.0f, ld, nullptr, nullptr, nullptr};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const int n_multi = n_seqs - n_single;
    int rc = HDS_OK;
    if (n_multi > 0) {
        const bool chunked = lin_chunk_supported(a, dtype, workspace, workspace_bytes);
        HDS_REQUIRE(method != 2 || chunked, "hds_linear_attention: the chunked form does not take this shape");
        if (chunked && method != 1) {
            if (vdim > 128 && out != nullptr) {     // heads of several blocks: the norm takes a pass of its own
                *finished = 0;
                a.write_y = 1;
            }
            rc = lin_chunk_launch(a, n_multi, workspace, workspace_bytes, s);
        } else {
            *finished = 0;
            a.write_y = 1;      // by every row of the batch: one norm finishes them all
            rc = lin_launch_scan(a, dtype, false, s);
        }
    }
    if (rc != HDS_OK || n_single == 0) return rc;
    return lin_launch_step(a, dtype, false, s);
}
