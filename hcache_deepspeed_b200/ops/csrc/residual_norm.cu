// Norms of stacks that keep the residual stream in fp32.
//
//   norm_residual : one pass per sublayer boundary. The previous sublayer's output d (16-bit, or the fp32 partial sums of a
//                   split-K GEMM, cleared while being read) is itself RMS-normed and weighted, added to the fp32 stream, and
//                   the stream is RMS-normed for the next sublayer:
//                       x += f d / rms(f d) * post;   out = x / rms(x) * gamma
//                   (no post weight: x += f d). One CTA per row; the row stays in registers between the two reductions.
//                   A second output may be normed, weighted and added in the same pass; the stream's norm may be taken over
//                   equal consecutive parts of a row, each by itself.
//   gated_norm    : out = rms(y * silu(z)) * weight * scale over `groups` equal parts of a row (state-space mixers), or
//                   rms(y) * weight * scale * silu(z) (delta rules)
//   embed_f32     : embedding rows into the fp32 stream, optionally RMS-normed on the way
#include "hds_host.cuh"
#include "hds_ptx.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

// two sums at once; red: 2 * THREADS / 32 floats
template <int THREADS>
__device__ __forceinline__ void block_sums_t(float& a, float& b, float* red) {
    a = warp_sum(a);
    b = warp_sum(b);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    if (l == 0) {
        red[w] = a;
        red[THREADS / 32 + w] = b;
    }
    __syncthreads();
    a = warp_sum(l < THREADS / 32 ? red[l] : 0.0f);
    b = warp_sum(l < THREADS / 32 ? red[THREADS / 32 + l] : 0.0f);
}

template <int THREADS>
__device__ __forceinline__ float block_sum_t(float v, float* red) {
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    if (l == 0) red[w] = v;
    __syncthreads();
    float t = l < THREADS / 32 ? red[l] : 0.0f;
    t = warp_sum(t);
    __syncthreads();
    return t;
}

// four consecutive values of a row; DT 0 bf16, 1 fp16, 2 fp32
template <int DT>
__device__ __forceinline__ float4 load4(const void* base, int64_t idx) {
    if constexpr (DT == 2) {
        return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(base) + idx);
    } else {
        const uint2 q = *reinterpret_cast<const uint2*>(reinterpret_cast<const char*>(base) + idx * 2);
        return make_float4(unpack_lo<DT == 0>(q.x), unpack_hi<DT == 0>(q.x), unpack_lo<DT == 0>(q.y), unpack_hi<DT == 0>(q.y));
    }
}
template <int DT>
__device__ __forceinline__ void store4(void* base, int64_t idx, float4 v) {
    if constexpr (DT == 2) {
        *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + idx) = v;
    } else {
        uint2 q;
        q.x = pack2<DT == 0>(v.x, v.y);
        q.y = pack2<DT == 0>(v.z, v.w);
        *reinterpret_cast<uint2*>(reinterpret_cast<char*>(base) + idx * 2) = q;
    }
}

// `cols`: values a row's mean is taken over; `padded` >= cols: row width, zeros behind the values. DELTA 0 none, 1 fp32
// (cleared after being read), 2 the output's type. kTwo: a second output of the same kind. groups > 1: the last norm is taken over
// that many equal parts of the `cols` values (dynamic shared memory: groups * (THREADS / 32 + 1) floats).
template <int THREADS, int VPT, int DT, int DELTA, bool kPost, bool kTwo>
__global__ void __launch_bounds__(THREADS)
norm_residual_kernel(float* __restrict__ x, void* delta, float factor, const float* __restrict__ post,
                     const float* __restrict__ gamma, void* __restrict__ out, int64_t ld, int cols, int padded, float eps,
                     int store_x, int groups, void* delta2, const float* __restrict__ post2) {
    __shared__ float red[THREADS / 32], red2[kTwo ? THREADS / 16 : 1];
    extern __shared__ float group_s[];
    pdl_enter();
    const int64_t row = static_cast<int64_t>(blockIdx.x) * ld;
    const int nvec = padded >> 2;
    float4 v[VPT], d[VPT], d2[kTwo ? VPT : 1];
    float ss = 0.0f, ss2 = 0.0f;
    auto take = [&](void* from, int c) {
        if constexpr (DELTA == 1) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(from) + row + 4 * c);
        else return load4<DT>(from, row + 4 * c);
    };
    // (a store right behind the load of the same line, while that is still on its way, costs several times the transfer: clear later)
    auto clear = [&](void* from, int c) {
        if constexpr (DELTA == 1) *reinterpret_cast<float4*>(reinterpret_cast<float*>(from) + row + 4 * c) = make_float4(0.f, 0.f, 0.f, 0.f);
    };
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * THREADS;
        v[i] = d[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < nvec) {
            v[i] = *reinterpret_cast<const float4*>(x + row + 4 * c);
            if constexpr (DELTA != 0) d[i] = take(delta, c);
            if constexpr (kTwo) {
                d2[i] = take(delta2, c);
                ss2 += d2[i].x * d2[i].x + d2[i].y * d2[i].y + d2[i].z * d2[i].z + d2[i].w * d2[i].w;
            }
            if constexpr (DELTA != 0) {
                d[i].x *= factor; d[i].y *= factor; d[i].z *= factor; d[i].w *= factor;
                if constexpr (kPost) ss += d[i].x * d[i].x + d[i].y * d[i].y + d[i].z * d[i].z + d[i].w * d[i].w;
            }
        }
    }
    if constexpr (DELTA != 0) {
        float r = 1.0f;
        float r2 = 0.0f;
        if constexpr (kTwo) {
            block_sums_t<THREADS>(ss, ss2, red2);
            r = 1.0f / sqrtf(ss / cols + eps);
            r2 = 1.0f / sqrtf(ss2 / cols + eps);
        } else if constexpr (kPost) {
            r = 1.0f / sqrtf(block_sum_t<THREADS>(ss, red) / cols + eps);
        }
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + i * THREADS;
            if (c < nvec) {
                float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
                if constexpr (kPost) w = *reinterpret_cast<const float4*>(post + 4 * c);
                v[i].x += d[i].x * r * w.x; v[i].y += d[i].y * r * w.y;
                v[i].z += d[i].z * r * w.z; v[i].w += d[i].w * r * w.w;
                if constexpr (kTwo) {
                    const float4 u = *reinterpret_cast<const float4*>(post2 + 4 * c);
                    v[i].x += d2[i].x * r2 * u.x; v[i].y += d2[i].y * r2 * u.y;
                    v[i].z += d2[i].z * r2 * u.z; v[i].w += d2[i].w * r2 * u.w;
                }
                if (store_x) *reinterpret_cast<float4*>(x + row + 4 * c) = v[i];
                clear(delta, c);
                if constexpr (kTwo) clear(delta2, c);
            }
        }
    }
    if (groups > 1) {
        const int part = cols / groups, warp = threadIdx.x >> 5;
        float* r_s = group_s + groups * (THREADS / 32);
        for (int g = 0; g < groups; ++g) {
            const int g0 = g * part, g1 = g0 + part;
            float s = 0.0f;
#pragma unroll
            for (int i = 0; i < VPT; ++i) {
                const int e = 4 * (threadIdx.x + i * THREADS);
                if (e + 3 < g0 || e >= g1) continue;
                s += (e >= g0 ? v[i].x * v[i].x : 0.0f) + (e + 1 >= g0 && e + 1 < g1 ? v[i].y * v[i].y : 0.0f) +
                     (e + 2 >= g0 && e + 2 < g1 ? v[i].z * v[i].z : 0.0f) + (e + 3 < g1 ? v[i].w * v[i].w : 0.0f);
            }
            s = warp_sum(s);
            if ((threadIdx.x & 31) == 0) group_s[g * (THREADS / 32) + warp] = s;
        }
        __syncthreads();
        for (int g = threadIdx.x; g < groups; g += THREADS) {
            float s = 0.0f;
            for (int w = 0; w < THREADS / 32; ++w) s += group_s[g * (THREADS / 32) + w];
            r_s[g] = 1.0f / sqrtf(s / part + eps);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + i * THREADS, e = 4 * c;
            if (c < nvec) {
                const float4 w = *reinterpret_cast<const float4*>(gamma + e);
                auto of = [&](int x) { return r_s[min(x / part, groups - 1)]; };    // (past the values: zeros)
                const float r0 = of(e);
                if ((part & 3) == 0)
                    store4<DT>(out, row + e, make_float4(v[i].x * r0 * w.x, v[i].y * r0 * w.y, v[i].z * r0 * w.z, v[i].w * r0 * w.w));
                else
                    store4<DT>(out, row + e, make_float4(v[i].x * r0 * w.x, v[i].y * of(e + 1) * w.y, v[i].z * of(e + 2) * w.z,
                                                         v[i].w * of(e + 3) * w.w));
            }
        }
        return;
    }
    ss = 0.0f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float r = 1.0f / sqrtf(block_sum_t<THREADS>(ss, red) / cols + eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * THREADS;
        if (c < nvec) {
            const float4 w = *reinterpret_cast<const float4*>(gamma + 4 * c);
            store4<DT>(out, row + 4 * c, make_float4(v[i].x * r * w.x, v[i].y * r * w.y, v[i].z * r * w.z, v[i].w * r * w.w));
        }
    }
}

template <int DT, int DELTA, bool kPost, bool kTwo = false>
static int launch_norm_residual(float* x, void* delta, float factor, const float* post, const float* gamma, void* out, int64_t ld,
                                int rows, int cols, int padded, float eps, int store_x, int groups, void* delta2, const float* post2,
                                cudaStream_t s) {
    const int nvec = padded / 4;
#define HDS_NR(TH, V)                                                                                                       \
    HDS_CHECK_CUDA(launch_kernel(norm_residual_kernel<TH, V, DT, DELTA, kPost, kTwo>, dim3(rows), dim3(TH),                        \
                                 groups > 1 ? sizeof(float) * groups * (TH / 32 + 1) : 0, s, x, delta, factor, post, gamma, out, ld, \
                                 cols, padded, eps, store_x, groups, delta2, post2))
    if (nvec <= 128) HDS_NR(128, 1);
    else if (nvec <= 256) HDS_NR(256, 1);
    else if (nvec <= 512) HDS_NR(512, 1);
    else if (nvec <= 1024) HDS_NR(512, 2);
    else if (nvec <= 2048) HDS_NR(512, 4);
    else if (nvec <= 8192) HDS_NR(1024, 8);
    else {
        set_error("hds_norm_residual: rows wider than 32768 are unsupported");
        return HDS_ERR_UNSUPPORTED;
    }
#undef HDS_NR
    return HDS_OK;
}

template <int DT>
__device__ __forceinline__ float gate_silu(float b) {
    return DT == 2 ? b / (1.0f + expf(-b)) : __fdividef(b, 1.0f + __expf(-b));
}

// One warp per (row, part) of up to 128 * VPT values (a multiple of 4), all in registers.
template <int DT, int VPT>
__global__ void __launch_bounds__(256)
gated_norm_warp_kernel(const float* __restrict__ y, int64_t ld_y, const void* __restrict__ z, int64_t ld_z, const float* __restrict__ w,
                       void* __restrict__ out, int64_t ld_out, int rows, int groups, int part, float eps, float scale, int gate_after) {
    pdl_enter();
    const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= rows * groups) return;
    const int64_t t = unit / groups;
    const int c0 = unit % groups * part;
    float4 g[VPT], b[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = (lane + 32 * i) * 4;
        g[i] = b[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < part) {
            g[i] = *reinterpret_cast<const float4*>(y + t * ld_y + c0 + c);
            b[i] = load4<DT>(z, t * ld_z + c0 + c);
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        b[i] = make_float4(gate_silu<DT>(b[i].x), gate_silu<DT>(b[i].y), gate_silu<DT>(b[i].z), gate_silu<DT>(b[i].w));
        if (!gate_after) {
            g[i].x *= b[i].x; g[i].y *= b[i].y; g[i].z *= b[i].z; g[i].w *= b[i].w;
            b[i] = make_float4(1.f, 1.f, 1.f, 1.f);
        }
        ss += g[i].x * g[i].x + g[i].y * g[i].y + g[i].z * g[i].z + g[i].w * g[i].w;
    }
    const float r = scale / sqrtf(warp_sum(ss) / part + eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = (lane + 32 * i) * 4;
        if (c < part) {
            const float4 ww = *reinterpret_cast<const float4*>(w + c0 + c);
            store4<DT>(out, t * ld_out + c0 + c, make_float4(g[i].x * r * ww.x * b[i].x, g[i].y * r * ww.y * b[i].y,
                                                                 g[i].z * r * ww.z * b[i].z, g[i].w * r * ww.w * b[i].w));
        }
    }
}

template <int DT>
static cudaError_t launch_gated_norm_warp(const float* y, int64_t ld_y, const void* z, int64_t ld_z, const float* w, void* out, int64_t ld_out,
                                          int rows, int groups, int part, float eps, float scale, int gate_after, cudaStream_t s) {
    const dim3 grid((static_cast<int64_t>(rows) * groups + 7) / 8), block(256);
#define HDS_GNW(V) \
    return launch_kernel(gated_norm_warp_kernel<DT, V>, grid, block, 0, s, y, ld_y, z, ld_z, w, out, ld_out, rows, groups, part, eps, scale, \
                         gate_after)
    if (part <= 128) HDS_GNW(1);
    if (part <= 256) HDS_GNW(2);
    if (part <= 512) HDS_GNW(4);
    HDS_GNW(8);
#undef HDS_GNW
}

// One CTA per (row, part). y fp32, z in the I/O type; any part size.
template <int DT>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ y, int64_t ld_y, const void* __restrict__ z, int64_t ld_z,
                  const float* __restrict__ w, void* __restrict__ out, int64_t ld_out, int part, float eps, float scale, int gate_after) {
    extern __shared__ float vals[];
    __shared__ float red[8];
    pdl_enter();
    const int64_t t = blockIdx.x;
    const int c0 = blockIdx.y * part;
    float ss = 0.0f;
    const bool vec = !gate_after && (part & 3) == 0 && (ld_y & 3) == 0 && (ld_z & 3) == 0 && (ld_out & 3) == 0;
    if (vec) {
        for (int c = threadIdx.x * 4; c < part; c += 1024) {
            const float4 a = *reinterpret_cast<const float4*>(y + t * ld_y + c0 + c);
            const float4 b = load4<DT>(z, t * ld_z + c0 + c);
            float4 g;
            g.x = a.x * gate_silu<DT>(b.x);
            g.y = a.y * gate_silu<DT>(b.y);
            g.z = a.z * gate_silu<DT>(b.z);
            g.w = a.w * gate_silu<DT>(b.w);
            *reinterpret_cast<float4*>(vals + c) = g;
            ss += g.x * g.x + g.y * g.y + g.z * g.z + g.w * g.w;
        }
    } else {
        for (int c = threadIdx.x; c < part; c += 256) {
            const float b = load_any<DT>(z, t * ld_z + c0 + c);
            const float g = gate_after ? y[t * ld_y + c0 + c] : y[t * ld_y + c0 + c] * gate_silu<DT>(b);
            vals[c] = g;
            ss += g * g;
        }
    }
    const float r = scale / sqrtf(block_sum_t<256>(ss, red) / part + eps);
    if (vec) {
        for (int c = threadIdx.x * 4; c < part; c += 1024) {
            const float4 g = *reinterpret_cast<const float4*>(vals + c);
            const float4 ww = *reinterpret_cast<const float4*>(w + c0 + c);
            store4<DT>(out, t * ld_out + c0 + c, make_float4(g.x * r * ww.x, g.y * r * ww.y, g.z * r * ww.z, g.w * r * ww.w));
        }
    } else {
        for (int c = threadIdx.x; c < part; c += 256) {
            float v = vals[c] * r * w[c0 + c];
            if (gate_after) v *= gate_silu<DT>(load_any<DT>(z, t * ld_z + c0 + c));
            if constexpr (DT == 2) reinterpret_cast<float*>(out)[t * ld_out + c0 + c] = v;
            else store_scalar<DT == 0>(out, t * ld_out + c0 + c, v);
        }
    }
}

template <int DT>
__global__ void embed_f32_kernel(const int32_t* __restrict__ ids, const void* __restrict__ W, float* __restrict__ out, int H, int vocab, float scale) {
    pdl_enter();
    const int64_t t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    for (int c = threadIdx.x * 4; c < H; c += blockDim.x * 4) {
        const float4 v = ok ? load4<DT>(W, static_cast<int64_t>(id) * H + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        *reinterpret_cast<float4*>(out + t * H + c) = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
    }
}

// the same, each row then divided by its root mean square over `cols` and weighted
template <int DT>
__global__ void __launch_bounds__(256)
embed_norm_f32_kernel(const int32_t* __restrict__ ids, const void* __restrict__ W, const float* __restrict__ gamma,
                      float* __restrict__ out, int H, int vocab, int cols, float eps) {
    __shared__ float red[8];
    pdl_enter();
    const int64_t t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    float ss = 0.0f;
    for (int c = threadIdx.x * 4; c < H; c += 1024) {
        const float4 v = ok ? load4<DT>(W, static_cast<int64_t>(id) * H + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float r = 1.0f / sqrtf(block_sum_t<256>(ss, red) / cols + eps);
    for (int c = threadIdx.x * 4; c < H; c += 1024) {
        const float4 v = ok ? load4<DT>(W, static_cast<int64_t>(id) * H + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 g = *reinterpret_cast<const float4*>(gamma + c);
        *reinterpret_cast<float4*>(out + t * H + c) = make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w);
    }
}

}  // namespace hds

using namespace hds;

extern "C" int hds_norm_residual(float* x, void* delta, int delta_is_f32, float factor, const float* post, const float* gamma,
                                 void* out, int64_t ld, int rows, int cols, int padded, float eps, int store_x, int groups, void* delta2,
                                 const float* post2, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_norm_residual: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(padded % 4 == 0 && ld % 4 == 0 && cols <= padded && padded <= ld, "hds_norm_residual: rows of 4-value vectors");
    HDS_REQUIRE(groups >= 1 && groups <= 256 && cols % groups == 0, "hds_norm_residual: 1..256 equal parts");
    HDS_REQUIRE(delta2 == nullptr || (delta != nullptr && post != nullptr && post2 != nullptr),
                "hds_norm_residual: a second output comes behind a first one, both with weights");
    if (rows == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const int mode = delta == nullptr ? 0 : delta_is_f32 ? 1 : 2;
#define HDS_NR_ARGS x, delta, factor, post, gamma, out, ld, rows, cols, padded, eps, store_x, groups, delta2, post2, s
#define HDS_NR_DT(DT)                                                                               \
    return mode == 0         ? launch_norm_residual<DT, 0, false>(HDS_NR_ARGS)                       \
           : post == nullptr ? (mode == 1 ? launch_norm_residual<DT, 1, false>(HDS_NR_ARGS)          \
                                          : launch_norm_residual<DT, 2, false>(HDS_NR_ARGS))         \
           : delta2 != nullptr ? (mode == 1 ? launch_norm_residual<DT, 1, true, true>(HDS_NR_ARGS)   \
                                            : launch_norm_residual<DT, 2, true, true>(HDS_NR_ARGS))  \
           : mode == 1       ? launch_norm_residual<DT, 1, true>(HDS_NR_ARGS)                        \
                             : launch_norm_residual<DT, 2, true>(HDS_NR_ARGS)
    if (dtype == 0) { HDS_NR_DT(0); }
    if (dtype == 1) { HDS_NR_DT(1); }
    HDS_NR_DT(2);
#undef HDS_NR_DT
#undef HDS_NR_ARGS
}

extern "C" int hds_gated_norm(const float* y, int64_t ld_y, const void* z, int64_t ld_z, const float* w, void* out, int64_t ld_out,
                              int rows, int cols, int groups, float eps, float scale, int gate_after, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_gated_norm: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(groups >= 1 && cols % groups == 0 && cols / groups <= 12000, "hds_gated_norm: equal parts of at most 12000 values");
    if (rows == 0) return HDS_OK;
    const int part = cols / groups;
    const size_t smem = static_cast<size_t>(part) * 4;
    const dim3 grid(rows, groups);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const uintptr_t al = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(z) * 2 |
                         reinterpret_cast<uintptr_t>(out) * 2;   // 16-byte vectors of fp32, 8-byte ones of the 16-bit types
    if (part % 4 == 0 && part <= 1024 && ld_y % 4 == 0 && ld_z % 4 == 0 && ld_out % 4 == 0 && (al & 15) == 0 && dtype != 2) {
        HDS_CHECK_CUDA(dtype == 0 ? launch_gated_norm_warp<0>(y, ld_y, z, ld_z, w, out, ld_out, rows, groups, part, eps, scale, gate_after, s)
                                  : launch_gated_norm_warp<1>(y, ld_y, z, ld_z, w, out, ld_out, rows, groups, part, eps, scale, gate_after, s));
        return HDS_OK;
    }
    if (dtype == 0)
        HDS_CHECK_CUDA(launch_kernel(gated_norm_kernel<0>, grid, dim3(256), smem, s, y, ld_y, z, ld_z, w, out, ld_out, part, eps, scale, gate_after));
    else if (dtype == 1)
        HDS_CHECK_CUDA(launch_kernel(gated_norm_kernel<1>, grid, dim3(256), smem, s, y, ld_y, z, ld_z, w, out, ld_out, part, eps, scale, gate_after));
    else
        HDS_CHECK_CUDA(launch_kernel(gated_norm_kernel<2>, grid, dim3(256), smem, s, y, ld_y, z, ld_z, w, out, ld_out, part, eps, scale, gate_after));
    return HDS_OK;
}

extern "C" int hds_embed_f32(const int32_t* ids, const void* W, const float* gamma, float* out, int T, int H, int vocab, int cols, float eps,
                             float scale, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_embed_f32: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(H % 4 == 0, "hds_embed_f32: rows of 4-value vectors");
    if (T == 0) return HDS_OK;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    HDS_REQUIRE(gamma == nullptr || scale == 1.0f, "hds_embed_f32: a norm or a factor");
    if (gamma != nullptr) {
        if (dtype == 0) HDS_CHECK_CUDA(launch_kernel(embed_norm_f32_kernel<0>, dim3(T), dim3(256), 0, s, ids, W, gamma, out, H, vocab, cols, eps));
        else if (dtype == 1) HDS_CHECK_CUDA(launch_kernel(embed_norm_f32_kernel<1>, dim3(T), dim3(256), 0, s, ids, W, gamma, out, H, vocab, cols, eps));
        else HDS_CHECK_CUDA(launch_kernel(embed_norm_f32_kernel<2>, dim3(T), dim3(256), 0, s, ids, W, gamma, out, H, vocab, cols, eps));
        return HDS_OK;
    }
    if (dtype == 0) HDS_CHECK_CUDA(launch_kernel(embed_f32_kernel<0>, dim3(T), dim3(256), 0, s, ids, W, out, H, vocab, scale));
    else if (dtype == 1) HDS_CHECK_CUDA(launch_kernel(embed_f32_kernel<1>, dim3(T), dim3(256), 0, s, ids, W, out, H, vocab, scale));
    else HDS_CHECK_CUDA(launch_kernel(embed_f32_kernel<2>, dim3(T), dim3(256), 0, s, ids, W, out, H, vocab, scale));
    return HDS_OK;
}
