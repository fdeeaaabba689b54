// Gated delta rule over a ragged batch, per head:  S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q,
// with unit keys and queries (q also times dim^-1/2) that the value heads of a group share, behind a short causal convolution.
//
//   delta_scan : sequences with several new tokens, token by token in fp32 (fp32 models, and shapes the chunked kernel does not
//                take); rows of S^T live in registers, tokens are staged through shared memory
//   delta_step : sequences with ONE new token (decode): convolution, unit vectors, decay, step size, state update, read-out, and
//                (when every sequence of the batch brings one token) the norm and gate behind, in one kernel
//   (the convolution of prompts is the state-space mixers' kernel, ssm.cu; delta_chunk.cu holds the tensor-core form of the scan)
//
// The state is kept as [vdim][dim]: its rows are independent of one another. With the old state's products a = S^T k and b = S^T q
// a row needs one pass:  u = beta (v - g a),  S <- g S + u k,  o = g b + u (k.q).  A sequence at position 0 starts from zero.
#include "delta.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kDsWarps = 4, kDsRows = 4, kDsP = kDsWarps * kDsRows, kDsTok = 16;

// CTA = (sequence, head, 16 rows): a warp keeps 4 rows, NL state values of each per lane.
template <int DT, int NL>
__global__ void __launch_bounds__(kDsWarps * 32) delta_scan_kernel(const SsmArgs a) {
    extern __shared__ float sm[];
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int h = blockIdx.y, p0 = blockIdx.z * kDsP, N = a.N, P = a.P, H = a.heads;
    const int g = h / (H / a.groups), inner = a.inner();
    float* k_s = sm;                        // [tok][N] unit keys
    float* q_s = k_s + kDsTok * N;          // [tok][N] unit queries, scaled
    float* v_s = q_s + kDsTok * N;          // [tok][kDsP]
    float* e_s = v_s + kDsTok * kDsP;       // [tok] decay
    float* b_s = e_s + kDsTok;              // [tok] step size
    float* d_s = b_s + kDsTok;              // [tok] k.q
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float rate = a.a[h], q_scale = rsqrtf(static_cast<float>(N));
    float S[kDsRows][NL];
    float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
#pragma unroll
    for (int r = 0; r < kDsRows; ++r)
#pragma unroll
        for (int j = 0; j < NL; ++j) {
            const int p = p0 + warp * kDsRows + r, n = lane + 32 * j;
            S[r][j] = (sp.seen > 0 && p < P && n < N) ? st[static_cast<int64_t>(p) * N + n] : 0.0f;
        }
    for (int t0 = 0; t0 < sp.n; t0 += kDsTok) {
        const int nt = min(kDsTok, sp.n - t0);
        const int64_t row = sp.row0 + t0;
        __syncthreads();
        for (int t = warp; t < nt; t += kDsWarps) {      // a warp makes one token's vectors
            const int64_t base = (row + t) * a.ld_u + inner + g * N;
            float kk = 0.0f, qq = 0.0f, kq = 0.0f;
            for (int n = lane; n < N; n += 32) {
                const float k = load_any<DT>(a.u, base + n), q = load_any<DT>(a.u, base + a.groups * N + n);
                kk = fmaf(k, k, kk);
                qq = fmaf(q, q, qq);
                kq = fmaf(k, q, kq);
                k_s[t * N + n] = k;
                q_s[t * N + n] = q;
            }
            const float rk = 1.0f / sqrtf(warp_sum(kk) + kUnitEps), rq = q_scale / sqrtf(warp_sum(qq) + kUnitEps);
            kq = warp_sum(kq);
            for (int n = lane; n < N; n += 32) {
                k_s[t * N + n] *= rk;
                q_s[t * N + n] *= rq;
            }
            if (lane == 0) {
                e_s[t] = expf(rate * a.dt[(row + t) * H + h]);
                b_s[t] = delta_beta<DT>(a, row + t, h);
                d_s[t] = kq * rk * rq;
            }
        }
        for (int e = threadIdx.x; e < nt * kDsP; e += blockDim.x) {
            const int p = p0 + e % kDsP;
            v_s[e] = p < P ? load_any<DT>(a.u, (row + e / kDsP) * a.ld_u + h * P + p) : 0.0f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float dec = e_s[t], beta = b_s[t], kq = d_s[t];
            float sk[kDsRows] = {}, sq[kDsRows] = {}, u[kDsRows];
#pragma unroll
            for (int j = 0; j < NL; ++j) {
                const int n = lane + 32 * j;
                const float k = n < N ? k_s[t * N + n] : 0.0f, q = n < N ? q_s[t * N + n] : 0.0f;
#pragma unroll
                for (int r = 0; r < kDsRows; ++r) {
                    sk[r] = fmaf(S[r][j], k, sk[r]);
                    sq[r] = fmaf(S[r][j], q, sq[r]);
                }
            }
#pragma unroll
            for (int r = 0; r < kDsRows; ++r) {
                const int p = p0 + warp * kDsRows + r;
                u[r] = beta * (v_s[t * kDsP + warp * kDsRows + r] - dec * warp_sum(sk[r]));
                const float o = fmaf(dec, warp_sum(sq[r]), u[r] * kq);
                if (lane == r && p < P) a.y[(row + t) * inner + h * P + p] = o;
            }
#pragma unroll
            for (int j = 0; j < NL; ++j) {
                const int n = lane + 32 * j;
                const float k = n < N ? k_s[t * N + n] : 0.0f;
#pragma unroll
                for (int r = 0; r < kDsRows; ++r) S[r][j] = fmaf(u[r], k, dec * S[r][j]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < kDsRows; ++r)
#pragma unroll
        for (int j = 0; j < NL; ++j) {
            const int p = p0 + warp * kDsRows + r, n = lane + 32 * j;
            if (p < P && n < N) st[static_cast<int64_t>(p) * N + n] = S[r][j];
        }
    if (blockIdx.z == 0) ssm_save_conv_of_head<DT>(a, sp, h, threadIdx.x, blockDim.x);
}

// ---- one token per sequence --------------------------------------------------------------------------------------
constexpr int kDtThreads = 256, kDtWarps = kDtThreads / 32;

__device__ __forceinline__ float dt_block_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int w = 0; w < kDtWarps; ++w) t += red[w];
    __syncthreads();
    return t;
}

// CTA = (sequence, head). NV > 0: rows of N = a multiple of 4 up to 128 * NV values as float4 in registers, R rows in flight per
// warp, the first ones loaded before the convolution; NV = 0: any N, two passes over a row.
template <int DT, int NV>
__global__ void __launch_bounds__(kDtThreads) delta_step_kernel(const DeltaArgs d) {
    extern __shared__ float sm[];
    __shared__ float red[kDtWarps];
    const SsmArgs& a = d.s;
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n != 1) return;
    const int h = blockIdx.y, N = a.N, P = a.P, H = a.heads, C = a.channels(), inner = a.inner(), taps = a.taps;
    const int per = H / a.groups, g = h / per;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* k_s = sm;           // [N]
    float* q_s = k_s + N;      // [N]
    float* v_s = q_s + N;      // [P], then the outputs
    const int64_t row = sp.row0;
    const int pos = sp.seen;
    const bool carry = pos > 0;
    float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
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
    float* ring = a.conv_state + static_cast<int64_t>(sp.slot) * taps * C;
    float kk = 0.0f, qq = 0.0f;
    for (int e = threadIdx.x; e < 2 * N + P; e += kDtThreads) {
        const int c = e < N ? inner + g * N + e : e < 2 * N ? inner + a.groups * N + g * N + (e - N) : h * P + (e - 2 * N);
        const float x = load_any<DT>(a.proj, row * a.ld_proj + inner + c);
        float v = 0.0f;
        for (int k = 0; k + 1 < taps; ++k) {
            const int p = pos - (taps - 1) + k;
            if (p >= 0) v = fmaf(ring[static_cast<int64_t>(p % taps) * C + c], a.conv_w[static_cast<int64_t>(k) * C + c], v);
        }
        v = fmaf(x, a.conv_w[static_cast<int64_t>(taps - 1) * C + c], v);
        v = ssm_round<DT>(ssm_silu<DT>(v));
        sm[e] = v;
        if (e < N) kk = fmaf(v, v, kk);
        else if (e < 2 * N) qq = fmaf(v, v, qq);
        // the ring entry of this position is read by nobody in this launch
        if (e >= 2 * N || h % per == 0) ring[static_cast<int64_t>(pos % taps) * C + c] = x;
    }
    const float beta = delta_beta<DT>(a, row, h);
    const float dt = ssm_softplus(load_any<DT>(a.proj, row * a.ld_proj + inner + C + h) + a.dt_bias[h]);
    const float dec = expf(a.a[h] * dt);
    kk = dt_block_sum(kk, red);
    qq = dt_block_sum(qq, red);
    const float rk = 1.0f / sqrtf(kk + kUnitEps), rq = rsqrtf(static_cast<float>(N)) / sqrtf(qq + kUnitEps);
    float kq = 0.0f;
    for (int n = threadIdx.x; n < N; n += kDtThreads) {
        const float k = k_s[n] * rk, q = q_s[n] * rq;
        k_s[n] = k;
        q_s[n] = q;
        kq = fmaf(k, q, kq);
    }
    kq = dt_block_sum(kq, red);
    float ss = 0.0f;
    if constexpr (NV > 0) {
        for (int p0 = warp * R; p0 < P; p0 += kDtWarps * R) {
            if (p0 != warp * R) load_rows(p0);
            float sk[R] = {}, sq[R] = {};
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int n = (lane + 32 * j) * 4;
                if (n >= N) continue;
                const float4 k = *reinterpret_cast<const float4*>(k_s + n), q = *reinterpret_cast<const float4*>(q_s + n);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    sk[r] += S[r][j].x * k.x + S[r][j].y * k.y + S[r][j].z * k.z + S[r][j].w * k.w;
                    sq[r] += S[r][j].x * q.x + S[r][j].y * q.y + S[r][j].z * q.z + S[r][j].w * q.w;
                }
            }
            float mine = 0.0f;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float u = beta * ((p0 + r < P ? v_s[p0 + r] : 0.0f) - dec * warp_sum(sk[r]));
                const float o = fmaf(dec, warp_sum(sq[r]), u * kq);
                if (lane == r) mine = o;
                sk[r] = u;
            }
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int n = (lane + 32 * j) * 4;
                if (n >= N) continue;
                const float4 k = *reinterpret_cast<const float4*>(k_s + n);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    if (p0 + r >= P) continue;
                    float4 v = S[r][j];
                    v.x = fmaf(sk[r], k.x, dec * v.x); v.y = fmaf(sk[r], k.y, dec * v.y);
                    v.z = fmaf(sk[r], k.z, dec * v.z); v.w = fmaf(sk[r], k.w, dec * v.w);
                    __stcs(reinterpret_cast<float4*>(st + static_cast<int64_t>(p0 + r) * N + n), v);
                }
            }
            __syncwarp();
            if (lane < R && p0 + lane < P) {      // (only this warp reads v of these rows)
                v_s[p0 + lane] = mine;
                ss = fmaf(mine, mine, ss);
            }
        }
    } else {
        for (int p = warp; p < P; p += kDtWarps) {
            float* q = st + static_cast<int64_t>(p) * N;
            float sk = 0.0f, sq = 0.0f;
            for (int n = lane; n < N; n += 32) {
                const float S0 = carry ? q[n] : 0.0f;
                sk = fmaf(S0, k_s[n], sk);
                sq = fmaf(S0, q_s[n], sq);
            }
            const float u = beta * (v_s[p] - dec * warp_sum(sk));
            const float o = fmaf(dec, warp_sum(sq), u * kq);
            for (int n = lane; n < N; n += 32) q[n] = fmaf(u, k_s[n], carry ? dec * q[n] : 0.0f);
            __syncwarp();
            if (lane == 0) {
                v_s[p] = o;
                ss = fmaf(o, o, ss);
            }
        }
    }
    if (d.out == nullptr) {
        __syncthreads();
        for (int p = threadIdx.x; p < P; p += kDtThreads) a.y[row * inner + h * P + p] = v_s[p];
        return;
    }
    const float r = 1.0f / sqrtf(dt_block_sum(ss, red) / P + d.eps);
    for (int p = threadIdx.x; p < P; p += kDtThreads) {
        const float z = load_any<DT>(a.proj, row * a.ld_proj + h * P + p);
        ssm_store<DT>(d.out, row * d.ld_out + h * P + p, v_s[p] * r * d.norm_w[h * P + p] * ssm_silu<DT>(z));
    }
}

template <int DT>
static int launch_scan(const SsmArgs& a, cudaStream_t s) {
    const dim3 grid(a.n_seqs, a.heads, (a.P + kDsP - 1) / kDsP), block(kDsWarps * 32);
    const size_t smem = (static_cast<size_t>(kDsTok) * (2 * a.N + kDsP) + 3 * kDsTok) * 4;
#define HDS_SCAN(NL)                                                                                                          \
    do {                                                                                                                      \
        if (smem > 48 * 1024)                                                                                                 \
            HDS_CHECK_CUDA(cudaFuncSetAttribute(delta_scan_kernel<DT, NL>, cudaFuncAttributeMaxDynamicSharedMemorySize,        \
                                                static_cast<int>(smem)));                                                     \
        HDS_CHECK_CUDA(launch_kernel(delta_scan_kernel<DT, NL>, grid, block, smem, s, a));                                    \
    } while (0)
    if (a.N <= 32) HDS_SCAN(1);
    else if (a.N <= 64) HDS_SCAN(2);
    else if (a.N <= 128) HDS_SCAN(4);
    else if (a.N <= 256) HDS_SCAN(8);
    else HDS_SCAN(16);
#undef HDS_SCAN
    return HDS_OK;
}

template <int DT>
static int launch_step(const DeltaArgs& d, cudaStream_t s) {
    const SsmArgs& a = d.s;
    const dim3 grid(a.n_seqs, a.heads), block(kDtThreads);
    const size_t smem = static_cast<size_t>(2 * a.N + a.P) * 4;
    if (a.N % 4 != 0 || a.N > 512) HDS_CHECK_CUDA(launch_kernel(delta_step_kernel<DT, 0>, grid, block, smem, s, d));
    else if (a.N <= 128) HDS_CHECK_CUDA(launch_kernel(delta_step_kernel<DT, 1>, grid, block, smem, s, d));
    else if (a.N <= 256) HDS_CHECK_CUDA(launch_kernel(delta_step_kernel<DT, 2>, grid, block, smem, s, d));
    else HDS_CHECK_CUDA(launch_kernel(delta_step_kernel<DT, 4>, grid, block, smem, s, d));
    return HDS_OK;
}

}  // namespace hds

using namespace hds;

extern "C" int64_t hds_delta_workspace_bytes(int T, int n_seqs, int heads, int groups) { return delta_chunk_workspace(T, n_seqs, heads, groups); }

extern "C" int hds_delta_rule(const void* proj, int64_t ld_proj, const float* conv_w, const float* conv_b, const float* dt_bias,
                              const float* decay_rate, float* state, float* conv_state, const int32_t* spans, int n_seqs, int n_single,
                              int T, int heads, int vdim, int dim, int groups, int taps, void* u, int64_t ld_u, float* dt, float* y,
                              void* out, int64_t ld_out, const float* norm_w, float eps, void* workspace, int64_t workspace_bytes,
                              int method, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_delta_rule: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(heads >= 1 && groups >= 1 && heads % groups == 0, "hds_delta_rule: heads % groups != 0");
    HDS_REQUIRE(dim >= 1 && dim <= 512 && vdim >= 1 && vdim <= 2048, "hds_delta_rule: dim up to 512, vdim up to 2048");
    HDS_REQUIRE(taps >= 1, "hds_delta_rule: at least one convolution tap");
    HDS_REQUIRE(method >= 0 && method <= 2, "hds_delta_rule: method 0 auto / 1 scan / 2 chunked");
    if (n_seqs == 0 || T == 0) return HDS_OK;
    DeltaArgs d;
    memset(&d, 0, sizeof(d));
    SsmArgs& a = d.s;
    a.proj = proj; a.ld_proj = ld_proj;
    a.conv_w = conv_w; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a = decay_rate;
    a.state = state; a.conv_state = conv_state;
    a.spans = reinterpret_cast<const SsmSpan*>(spans);
    a.n_seqs = n_seqs; a.T = T;
    a.heads = heads; a.P = vdim; a.N = dim; a.groups = groups; a.taps = taps;
    a.u = u; a.ld_u = ld_u; a.dt = dt; a.y = y;
    d.out = n_single == n_seqs ? out : nullptr;      // mixed batches: norm and gate of all rows behind this call
    d.ld_out = ld_out; d.norm_w = norm_w; d.eps = eps;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    int rc = HDS_OK;
    if (n_single < n_seqs) {
        if ((rc = ssm_conv_launch(a, dtype, s))) return rc;
        const bool chunk = method != 1 && delta_chunk_supported(a, n_seqs - n_single, dtype, workspace_bytes);
        HDS_REQUIRE(method != 2 || chunk, "hds_delta_rule: the chunked kernel does not take this shape");
        rc = chunk ? delta_chunk_launch(a, n_seqs - n_single, dtype, workspace, s)
             : dtype == 0 ? launch_scan<0>(a, s) : dtype == 1 ? launch_scan<1>(a, s) : launch_scan<2>(a, s);
        if (rc) return rc;
    }
    if (n_single > 0) rc = dtype == 0 ? launch_step<0>(d, s) : dtype == 1 ? launch_step<1>(d, s) : launch_step<2>(d, s);
    return rc;
}
