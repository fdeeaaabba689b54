// State-space (Mamba-2) mixer over a ragged batch:  S <- exp(a dt) S + dt x B^T,   y = S C + d x   per head, with a short
// causal convolution in front of x, B and C.
//
//   ssm_conv   : sequences with several new tokens: convolution + silu into u[T][x|B|C], step sizes into dt[T][heads]
//   ssm_scan   : those sequences token by token, fp32, any shape (fp32 models, and shapes the chunked kernel does not take);
//                state rows live in registers, tokens are staged through shared memory
//   ssm_step   : sequences with ONE new token (decode): convolution, step size, decay, state update and read-out in one kernel
//   (ssm_chunk.cu holds the tensor-core form of the scan for prompts)
//
// State and step sizes are fp32 throughout. A sequence at position 0 starts from zero whatever its slot holds.
#include "ssm.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kConvRows = 16;      // rows of the batch per block
constexpr int kConvThreads = 256;

// Thread = VEC neighbouring channels, walking kConvRows rows with the last TAPS - 1 inputs in registers. TAPS 0: any number of
// taps, inputs re-read. Blocks whose rows all belong to one sequence load them up front (VEC 4). Blocks behind the channel
// blocks compute step sizes.
template <int DT, int TAPS, int VEC>
__global__ void __launch_bounds__(kConvThreads) ssm_conv_kernel(const SsmArgs a, int channel_blocks) {
    pdl_enter();
    const int r_begin = blockIdx.x * kConvRows, r_end = min(a.T, r_begin + kConvRows);
    int s = 0;
    {   // the sequence of the first row (rows of the batch are in sequence order)
        int lo = 0, hi = a.n_seqs;
        while (hi - lo > 1) {
            const int mid = (lo + hi) >> 1;
            if (a.spans[mid].row0 <= r_begin) lo = mid;
            else hi = mid;
        }
        s = lo;
    }
    const int C = a.channels(), inner = a.inner();
    if (static_cast<int>(blockIdx.y) >= channel_blocks) {
        const int dt_col = inner + C;
        for (int e = threadIdx.x; e < (r_end - r_begin) * a.heads; e += kConvThreads) {
            const int64_t r = r_begin + e / a.heads;
            const int h = e % a.heads;
            a.dt[r * a.heads + h] = ssm_softplus(load_any<DT>(a.proj, r * a.ld_proj + dt_col + h) + a.dt_bias[h]);
        }
        return;
    }
    const int c = (blockIdx.y * kConvThreads + threadIdx.x) * VEC;
    if (c >= C) return;
    const int taps = TAPS > 0 ? TAPS : a.taps;
    float w[TAPS > 0 ? TAPS : 1][VEC], b[VEC], win[TAPS > 1 ? TAPS - 1 : 1][VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
        b[v] = a.conv_b[c + v];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) w[k][v] = a.conv_w[static_cast<int64_t>(k) * C + c + v];
    }
    auto input = [&](const SsmSpan& sp, int i, int v) -> float {   // input of token i of the span (i < 0: an earlier one)
        if (i >= 0) return load_any<DT>(a.proj, static_cast<int64_t>(sp.row0 + i) * a.ld_proj + inner + c + v);
        const int p = sp.seen + i;
        return p >= 0 ? a.conv_state[(static_cast<int64_t>(sp.slot) * taps + p % taps) * C + c + v] : 0.0f;
    };
    SsmSpan sp = a.spans[s];
    bool fresh = true;
    if constexpr (TAPS > 1 && VEC == 4 && DT != 2) {
        if (sp.n > 1 && r_end - r_begin == kConvRows && r_end <= sp.row0 + sp.n) {
            const char* src = reinterpret_cast<const char*>(a.proj) + (static_cast<int64_t>(r_begin) * a.ld_proj + inner + c) * 2;
            uint2 q[kConvRows];
#pragma unroll
            for (int i = 0; i < kConvRows; ++i) q[i] = *reinterpret_cast<const uint2*>(src + static_cast<int64_t>(i) * a.ld_proj * 2);
#pragma unroll
            for (int k = 0; k + 1 < TAPS; ++k)
#pragma unroll
                for (int v = 0; v < VEC; ++v) win[k][v] = input(sp, r_begin - sp.row0 - (TAPS - 1) + k, v);
            char* dst = reinterpret_cast<char*>(a.u) + (static_cast<int64_t>(r_begin) * a.ld_u + c) * 2;
#pragma unroll
            for (int i = 0; i < kConvRows; ++i) {
                const float x[4] = {unpack_lo<DT == 0>(q[i].x), unpack_hi<DT == 0>(q[i].x), unpack_lo<DT == 0>(q[i].y), unpack_hi<DT == 0>(q[i].y)};
                float o[4];
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    o[v] = b[v];
#pragma unroll
                    for (int k = 0; k + 1 < TAPS; ++k) o[v] = fmaf(win[k][v], w[k][v], o[v]);
                    o[v] = fmaf(x[v], w[TAPS - 1][v], o[v]);
#pragma unroll
                    for (int k = 0; k + 2 < TAPS; ++k) win[k][v] = win[k + 1][v];
                    win[TAPS - 2][v] = x[v];
                    o[v] = ssm_silu<DT>(o[v]);
                }
                uint2 p;
                p.x = pack2<DT == 0>(o[0], o[1]);
                p.y = pack2<DT == 0>(o[2], o[3]);
                *reinterpret_cast<uint2*>(dst + static_cast<int64_t>(i) * a.ld_u * 2) = p;
            }
            return;
        }
    }
    for (int r = r_begin; r < r_end; ++r) {
        while (r >= sp.row0 + sp.n) {
            sp = a.spans[++s];
            fresh = true;
        }
        if (sp.n == 1) continue;   // the step kernel's
        const int i = r - sp.row0;
        float out[VEC];
        if constexpr (TAPS > 0) {
            if (fresh) {
#pragma unroll
                for (int k = 0; k + 1 < TAPS; ++k)
#pragma unroll
                    for (int v = 0; v < VEC; ++v) win[k][v] = input(sp, i - (TAPS - 1) + k, v);
                fresh = false;
            }
            float x[VEC];
            if constexpr (VEC == 2 && DT != 2) {
                const uint32_t q = *reinterpret_cast<const uint32_t*>(reinterpret_cast<const char*>(a.proj) +
                                                                      (static_cast<int64_t>(r) * a.ld_proj + inner + c) * 2);
                x[0] = unpack_lo<DT == 0>(q);
                x[1] = unpack_hi<DT == 0>(q);
            } else {
#pragma unroll
                for (int v = 0; v < VEC; ++v) x[v] = input(sp, i, v);
            }
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                out[v] = b[v];
#pragma unroll
                for (int k = 0; k + 1 < TAPS; ++k) out[v] = fmaf(win[k][v], w[k][v], out[v]);
                out[v] = fmaf(x[v], w[TAPS - 1][v], out[v]);
#pragma unroll
                for (int k = 0; k + 2 < TAPS; ++k) win[k][v] = win[k + 1][v];
                if (TAPS > 1) win[TAPS > 1 ? TAPS - 2 : 0][v] = x[v];
            }
        } else {
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                out[v] = b[v];
                for (int k = 0; k < taps; ++k)
                    out[v] = fmaf(input(sp, i - (taps - 1) + k, v), a.conv_w[static_cast<int64_t>(k) * C + c + v], out[v]);
            }
        }
        if constexpr (VEC == 2 && DT != 2) {
            *reinterpret_cast<uint32_t*>(reinterpret_cast<char*>(a.u) + (static_cast<int64_t>(r) * a.ld_u + c) * 2) =
                pack2<DT == 0>(ssm_silu<DT>(out[0]), ssm_silu<DT>(out[1]));
        } else {
#pragma unroll
            for (int v = 0; v < VEC; ++v) ssm_store<DT>(a.u, static_cast<int64_t>(r) * a.ld_u + c + v, ssm_silu<DT>(out[v]));
        }
    }
}

// ---- token-by-token scan ------------------------------------------------------------------------------------------
constexpr int kScanWarps = 4, kScanRows = 4, kScanP = kScanWarps * kScanRows, kScanTok = 16;

// CTA = (sequence, head, 16 rows of the head's state): a warp keeps 4 rows, NL state values of each per lane.
template <int DT, int NL>
__global__ void __launch_bounds__(kScanWarps * 32) ssm_scan_kernel(const SsmArgs a) {
    extern __shared__ float sm[];
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n <= 1) return;
    const int h = blockIdx.y, p0 = blockIdx.z * kScanP, N = a.N, P = a.P, H = a.heads;
    const int g = h / (H / a.groups), inner = a.inner();
    float* b_s = sm;                         // [tok][N]
    float* c_s = b_s + kScanTok * N;
    float* x_s = c_s + kScanTok * N;         // [tok][kScanP]
    float* e_s = x_s + kScanTok * kScanP;    // [tok]: decay
    float* t_s = e_s + kScanTok;             // [tok]: step size
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float decay_rate = a.a[h], dh = a.d[h];
    float S[kScanRows][NL];
    float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
#pragma unroll
    for (int r = 0; r < kScanRows; ++r)
#pragma unroll
        for (int j = 0; j < NL; ++j) {
            const int p = p0 + warp * kScanRows + r, n = lane + 32 * j;
            S[r][j] = (sp.seen > 0 && p < P && n < N) ? st[static_cast<int64_t>(p) * N + n] : 0.0f;
        }
    for (int t0 = 0; t0 < sp.n; t0 += kScanTok) {
        const int nt = min(kScanTok, sp.n - t0);
        const int64_t row = sp.row0 + t0;
        __syncthreads();
        for (int e = threadIdx.x; e < nt * N; e += blockDim.x) {
            const int64_t base = (row + e / N) * a.ld_u + inner + g * N + e % N;
            b_s[e] = load_any<DT>(a.u, base);
            c_s[e] = load_any<DT>(a.u, base + a.groups * N);
        }
        for (int e = threadIdx.x; e < nt * kScanP; e += blockDim.x) {
            const int p = p0 + e % kScanP;
            x_s[e] = p < P ? load_any<DT>(a.u, (row + e / kScanP) * a.ld_u + h * P + p) : 0.0f;
        }
        if (threadIdx.x < nt) {
            const float dt = a.dt[(row + threadIdx.x) * H + h];
            t_s[threadIdx.x] = dt;
            e_s[threadIdx.x] = expf(decay_rate * dt);
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float dec = e_s[t], dt = t_s[t];
            float y[kScanRows], xv[kScanRows];
#pragma unroll
            for (int r = 0; r < kScanRows; ++r) {
                xv[r] = x_s[t * kScanP + warp * kScanRows + r];
                y[r] = 0.0f;
            }
#pragma unroll
            for (int j = 0; j < NL; ++j) {
                const int n = lane + 32 * j;
                const float bn = n < N ? b_s[t * N + n] : 0.0f, cn = n < N ? c_s[t * N + n] : 0.0f;
#pragma unroll
                for (int r = 0; r < kScanRows; ++r) {
                    S[r][j] = fmaf(dt * xv[r], bn, dec * S[r][j]);
                    y[r] = fmaf(S[r][j], cn, y[r]);
                }
            }
#pragma unroll
            for (int r = 0; r < kScanRows; ++r) {
                y[r] = warp_sum(y[r]);
                const int p = p0 + warp * kScanRows + r;
                if (lane == r && p < P) a.y[(row + t) * inner + h * P + p] = fmaf(dh, xv[r], y[r]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < kScanRows; ++r)
#pragma unroll
        for (int j = 0; j < NL; ++j) {
            const int p = p0 + warp * kScanRows + r, n = lane + 32 * j;
            if (p < P && n < N) st[static_cast<int64_t>(p) * N + n] = S[r][j];
        }
    if (blockIdx.z == 0) ssm_save_conv_of_head<DT>(a, sp, h, threadIdx.x, blockDim.x);
}

// ---- one token per sequence --------------------------------------------------------------------------------------
constexpr int kStepThreads = 128;

// CTA = (sequence, head). The convolution of the head's x channels and its group's B and C is redone per head (a few taps);
// VEC4: state rows are read and written as float4 (N a multiple of 4).
template <int DT, bool VEC4>
__global__ void __launch_bounds__(kStepThreads) ssm_step_kernel(const SsmArgs a) {
    extern __shared__ float sm[];
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    if (sp.n != 1) return;
    const int h = blockIdx.y, N = a.N, P = a.P, H = a.heads, C = a.channels(), inner = a.inner(), taps = a.taps;
    const int per = H / a.groups, g = h / per;
    float* b_s = sm;           // [N]
    float* c_s = b_s + N;      // [N]
    float* x_s = c_s + N;      // [P]
    const int64_t row = sp.row0;
    const int pos = sp.seen;
    float* ring = a.conv_state + static_cast<int64_t>(sp.slot) * taps * C;
    for (int e = threadIdx.x; e < 2 * N + P; e += kStepThreads) {
        const int c = e < N ? inner + g * N + e : e < 2 * N ? inner + a.groups * N + g * N + (e - N) : h * P + (e - 2 * N);
        const float x = load_any<DT>(a.proj, row * a.ld_proj + inner + c);
        float v = a.conv_b[c];
        for (int k = 0; k + 1 < taps; ++k) {
            const int p = pos - (taps - 1) + k;
            if (p >= 0) v = fmaf(ring[static_cast<int64_t>(p % taps) * C + c], a.conv_w[static_cast<int64_t>(k) * C + c], v);
        }
        v = fmaf(x, a.conv_w[static_cast<int64_t>(taps - 1) * C + c], v);
        sm[e] = ssm_round<DT>(ssm_silu<DT>(v));
        // the ring entry of this position is read by nobody in this launch
        if (e >= 2 * N || h % per == 0) ring[static_cast<int64_t>(pos % taps) * C + c] = x;
    }
    const float dt = ssm_softplus(load_any<DT>(a.proj, row * a.ld_proj + inner + C + h) + a.dt_bias[h]);
    const float dec = expf(a.a[h] * dt), dh = a.d[h];
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* st = a.state + (static_cast<int64_t>(sp.slot) * H + h) * P * N;
    const bool carry = pos > 0;
    constexpr int R = 4;       // rows in flight per warp
    for (int p0 = warp * R; p0 < P; p0 += R * (kStepThreads / 32)) {
        float y[R] = {0.f, 0.f, 0.f, 0.f}, w[R];
#pragma unroll
        for (int r = 0; r < R; ++r) w[r] = p0 + r < P ? dt * x_s[p0 + r] : 0.0f;
        if constexpr (VEC4) {
            for (int n = lane * 4; n < N; n += 128) {
                float4 S[R];
#pragma unroll
                for (int r = 0; r < R; ++r)
                    S[r] = carry && p0 + r < P ? __ldcs(reinterpret_cast<const float4*>(st + static_cast<int64_t>(p0 + r) * N + n))
                                               : make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 b = *reinterpret_cast<const float4*>(b_s + n), c = *reinterpret_cast<const float4*>(c_s + n);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    S[r].x = fmaf(w[r], b.x, dec * S[r].x); S[r].y = fmaf(w[r], b.y, dec * S[r].y);
                    S[r].z = fmaf(w[r], b.z, dec * S[r].z); S[r].w = fmaf(w[r], b.w, dec * S[r].w);
                    y[r] += S[r].x * c.x + S[r].y * c.y + S[r].z * c.z + S[r].w * c.w;
                    if (p0 + r < P) __stcs(reinterpret_cast<float4*>(st + static_cast<int64_t>(p0 + r) * N + n), S[r]);
                }
            }
        } else {
            for (int n = lane; n < N; n += 32) {
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    if (p0 + r >= P) continue;
                    float* q = st + static_cast<int64_t>(p0 + r) * N + n;
                    const float S = fmaf(w[r], b_s[n], carry ? dec * *q : 0.0f);
                    y[r] = fmaf(S, c_s[n], y[r]);
                    *q = S;
                }
            }
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            y[r] = warp_sum(y[r]);
            if (lane == r && p0 + r < P) a.y[row * inner + h * P + p0 + r] = fmaf(dh, x_s[p0 + r], y[r]);
        }
    }
}

template <int DT>
static int launch_conv(const SsmArgs& a, cudaStream_t s) {
    const int C = a.channels();
    const bool pair = C % 2 == 0 && a.inner() % 2 == 0 && a.ld_u % 2 == 0 && a.ld_proj % 2 == 0 &&
                      (reinterpret_cast<uintptr_t>(a.proj) & 3) == 0;
    const bool quad = DT != 2 && a.taps == 4 && C % 4 == 0 && a.inner() % 4 == 0 && a.ld_u % 4 == 0 && a.ld_proj % 4 == 0 &&
                      (reinterpret_cast<uintptr_t>(a.proj) & 7) == 0;
    const int vec = quad ? 4 : pair ? 2 : 1;
    const int cb = (C / vec + kConvThreads - 1) / kConvThreads;
    const dim3 grid((a.T + kConvRows - 1) / kConvRows, cb + 1);
    if (quad) HDS_CHECK_CUDA(launch_kernel(ssm_conv_kernel<DT, 4, DT == 2 ? 1 : 4>, grid, dim3(kConvThreads), 0, s, a, cb));
    else if (a.taps == 4 && pair) HDS_CHECK_CUDA(launch_kernel(ssm_conv_kernel<DT, 4, 2>, grid, dim3(kConvThreads), 0, s, a, cb));
    else if (a.taps == 4) HDS_CHECK_CUDA(launch_kernel(ssm_conv_kernel<DT, 4, 1>, grid, dim3(kConvThreads), 0, s, a, cb));
    else if (pair) HDS_CHECK_CUDA(launch_kernel(ssm_conv_kernel<DT, 0, 2>, grid, dim3(kConvThreads), 0, s, a, cb));
    else HDS_CHECK_CUDA(launch_kernel(ssm_conv_kernel<DT, 0, 1>, grid, dim3(kConvThreads), 0, s, a, cb));
    return HDS_OK;
}

int ssm_conv_launch(const SsmArgs& a, int dtype, cudaStream_t s) {
    return dtype == 0 ? launch_conv<0>(a, s) : dtype == 1 ? launch_conv<1>(a, s) : launch_conv<2>(a, s);
}

template <int DT>
static int launch_scan(const SsmArgs& a, cudaStream_t s) {
    const dim3 grid(a.n_seqs, a.heads, (a.P + kScanP - 1) / kScanP), block(kScanWarps * 32);
    const size_t smem = (static_cast<size_t>(kScanTok) * (2 * a.N + kScanP) + 2 * kScanTok) * 4;
#define HDS_SCAN(NL)                                                                                                          \
    do {                                                                                                                      \
        if (smem > 48 * 1024)                                                                                                 \
            HDS_CHECK_CUDA(cudaFuncSetAttribute(ssm_scan_kernel<DT, NL>, cudaFuncAttributeMaxDynamicSharedMemorySize,          \
                                                static_cast<int>(smem)));                                                     \
        HDS_CHECK_CUDA(launch_kernel(ssm_scan_kernel<DT, NL>, grid, block, smem, s, a));                                      \
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
static int launch_step(const SsmArgs& a, cudaStream_t s) {
    const dim3 grid(a.n_seqs, a.heads);
    const size_t smem = static_cast<size_t>(2 * a.N + a.P) * 4;
    if (a.N % 4 == 0) HDS_CHECK_CUDA(launch_kernel(ssm_step_kernel<DT, true>, grid, dim3(kStepThreads), smem, s, a));
    else HDS_CHECK_CUDA(launch_kernel(ssm_step_kernel<DT, false>, grid, dim3(kStepThreads), smem, s, a));
    return HDS_OK;
}

template <int DT>
static int run(const SsmArgs& a, int n_single, bool allow_chunk, cudaStream_t s) {
    int rc = HDS_OK;
    if (n_single < a.n_seqs) {
        if ((rc = launch_conv<DT>(a, s))) return rc;
        rc = allow_chunk && ssm_chunk_supported(a, DT) ? ssm_chunk_launch(a, DT, s) : launch_scan<DT>(a, s);
        if (rc) return rc;
    }
    if (n_single > 0) rc = launch_step<DT>(a, s);
    return rc;
}

}  // namespace hds

using namespace hds;

extern "C" int hds_state_space(const void* proj, int64_t ld_proj, const float* conv_w, const float* conv_b, const float* dt_bias,
                               const float* decay_rate, const float* skip, float* state, float* conv_state, const int32_t* spans,
                               int n_seqs, int n_single, int T, int heads, int vdim, int state_size, int groups, int taps, void* u,
                               int64_t ld_u, float* dt, float* y, int method, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_state_space: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(heads >= 1 && groups >= 1 && heads % groups == 0, "hds_state_space: heads % groups != 0");
    HDS_REQUIRE(state_size >= 1 && state_size <= 512 && vdim >= 1 && vdim <= 2048, "hds_state_space: state up to 512, head size up to 2048");
    HDS_REQUIRE(taps >= 1, "hds_state_space: at least one convolution tap");
    HDS_REQUIRE(method >= 0 && method <= 2, "hds_state_space: method 0 auto / 1 scan / 2 chunked");
    if (n_seqs == 0 || T == 0) return HDS_OK;
    SsmArgs a;
    memset(&a, 0, sizeof(a));
    a.proj = proj; a.ld_proj = ld_proj;
    a.conv_w = conv_w; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a = decay_rate; a.d = skip;
    a.state = state; a.conv_state = conv_state;
    a.spans = reinterpret_cast<const SsmSpan*>(spans);
    a.n_seqs = n_seqs; a.T = T;
    a.heads = heads; a.P = vdim; a.N = state_size; a.groups = groups; a.taps = taps;
    a.u = u; a.ld_u = ld_u; a.dt = dt; a.y = y;
    HDS_REQUIRE(method != 2 || ssm_chunk_supported(a, dtype), "hds_state_space: the chunked kernel does not take this shape");
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == 0) return run<0>(a, n_single, method != 1, s);
    if (dtype == 1) return run<1>(a, n_single, method != 1, s);
    return run<2>(a, n_single, method != 1, s);
}
