// minGRU over a ragged batch, element by element:  S <- (1 - s(z)) S + s(z) c,  out = S * silu(g), with s the logistic function and
// c = u + 1/2 where u >= 0, s(u) where u < 0. z and u have biases; everything up to the state is fp32.
//
//   gru_step  : sequences with one new token (decode)
//   gru_local : what 32 tokens do to a state: S -> A S + B, per element
//   gru_chain : states in front of every chunk, from the (A, B) of the chunks before it; advances the state pool
//   gru_out   : the tokens of a chunk from the state in front of it
// The gates depend on the token alone, so only gru_chain walks along a sequence, a step per 32 tokens.
#include <type_traits>

#include "recurrent.cuh"
#include "../../../include/hds_b200.h"

namespace hds {

constexpr int kGruTok = 32, kGruThreads = 128;

struct GruArgs {
    const void* proj;       // [T][ld]: z | u | output gate (C each)
    int64_t ld;
    const float* bias;      // [2 * C]: of z, of u
    float* state;           // [slots][C]
    const SsmSpan* spans;
    int n_seqs, C;
    void* out;              // [T][ld_out] or nullptr
    int64_t ld_out;
    float4* a;              // [chunks][C / 4]: A, then (gru_chain) the state in front
    float4* b;
};

// four neighbouring values as they are stored, and as fp32
template <int DT>
struct GruRaw {
    typename std::conditional<DT == 2, float4, uint2>::type v;
    __device__ __forceinline__ void load(const void* p, int64_t i) {
        v = *reinterpret_cast<const decltype(v)*>(reinterpret_cast<const char*>(p) + i * (DT == 2 ? 4 : 2));
    }
    __device__ __forceinline__ float4 get() const {
        if constexpr (DT == 2) return v;
        else return make_float4(unpack_lo<DT == 0>(v.x), unpack_hi<DT == 0>(v.x), unpack_lo<DT == 0>(v.y), unpack_hi<DT == 0>(v.y));
    }
};
template <int DT>
__device__ __forceinline__ float gru_sigmoid(float v) {
    return DT == 2 ? 1.0f / (1.0f + expf(-v)) : __fdividef(1.0f, 1.0f + __expf(-v));
}
// gates of one value: kept share of the state, and what is added. 16-bit inputs: both sigmoids from one reciprocal (inputs below -40,
// whose sigmoid is zero to any state, count as -40 so that the product of the denominators stays finite).
template <int DT>
__device__ __forceinline__ void gru_gate(float z, float u, float& keep, float& add) {
    float s, c;
    if constexpr (DT == 2) {
        s = gru_sigmoid<2>(z);
        c = gru_sigmoid<2>(u);
    } else {
        const float a = 1.0f + __expf(-fmaxf(z, -40.0f)), b = 1.0f + __expf(-fmaxf(u, -40.0f)), r = __fdividef(1.0f, a * b);
        s = r * b;
        c = r * a;
    }
    keep = 1.0f - s;
    add = s * (u >= 0.0f ? u + 0.5f : c);
}
template <int DT>
__device__ __forceinline__ void gru_gates(float4 z, float4 u, float4 bz, float4 bu, float4& keep, float4& add) {
    gru_gate<DT>(z.x + bz.x, u.x + bu.x, keep.x, add.x);
    gru_gate<DT>(z.y + bz.y, u.y + bu.y, keep.y, add.y);
    gru_gate<DT>(z.z + bz.z, u.z + bu.z, keep.z, add.z);
    gru_gate<DT>(z.w + bz.w, u.w + bu.w, keep.w, add.w);
}
__device__ __forceinline__ float4 gru_fma(float4 a, float4 s, float4 b) {
    return make_float4(fmaf(a.x, s.x, b.x), fmaf(a.y, s.y, b.y), fmaf(a.z, s.z, b.z), fmaf(a.w, s.w, b.w));
}
template <int DT>
__device__ __forceinline__ void gru_emit(const GruArgs& a, int64_t row, int c, float4 s, float4 g) {
    const float4 o = make_float4(s.x * g.x * gru_sigmoid<DT>(g.x), s.y * g.y * gru_sigmoid<DT>(g.y), s.z * g.z * gru_sigmoid<DT>(g.z),
                                 s.w * g.w * gru_sigmoid<DT>(g.w));
    if constexpr (DT == 2) *reinterpret_cast<float4*>(reinterpret_cast<float*>(a.out) + row * a.ld_out + c) = o;
    else *reinterpret_cast<uint2*>(reinterpret_cast<char*>(a.out) + (row * a.ld_out + c) * 2) =
             make_uint2(pack2<DT == 0>(o.x, o.y), pack2<DT == 0>(o.z, o.w));
}

template <int DT>
__global__ void __launch_bounds__(kGruThreads) gru_step_kernel(const GruArgs a) {
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    const int c = (blockIdx.y * kGruThreads + threadIdx.x) * 4;
    if (sp.n != 1 || c >= a.C) return;
    float4* st = reinterpret_cast<float4*>(a.state + static_cast<int64_t>(sp.slot) * a.C + c);
    const int64_t at = static_cast<int64_t>(sp.row0) * a.ld + c;
    GruRaw<DT> z, u, g;
    z.load(a.proj, at);
    u.load(a.proj, at + a.C);
    g.load(a.proj, at + 2 * a.C);
    float4 keep, add, S = make_float4(0.f, 0.f, 0.f, 0.f);
    if (sp.seen > 0) S = *st;
    gru_gates<DT>(z.get(), u.get(), *reinterpret_cast<const float4*>(a.bias + c), *reinterpret_cast<const float4*>(a.bias + a.C + c), keep, add);
    S = gru_fma(keep, S, add);
    *st = S;
    if (a.out != nullptr) gru_emit<DT>(a, sp.row0, c, S, g.get());
}

// kOut false: (A, B) of the chunk; true: its outputs from the state in front
template <int DT, bool kOut>
__global__ void __launch_bounds__(kGruThreads) gru_chunk_kernel(const GruArgs a) {
    __shared__ ChunkPlace place;
    pdl_enter();
    if (!find_chunk(a.spans, a.n_seqs, kGruTok, blockIdx.x, &place)) return;
    const int c = (blockIdx.y * kGruThreads + threadIdx.x) * 4;
    if (c >= a.C) return;
    const int t0 = place.chunk * kGruTok, n = min(kGruTok, place.span.n - t0);
    const int64_t row = place.span.row0 + t0, cell = static_cast<int64_t>(blockIdx.x) * (a.C / 4) + c / 4;
    const float4 bz = *reinterpret_cast<const float4*>(a.bias + c), bu = *reinterpret_cast<const float4*>(a.bias + a.C + c);
    float4 A = make_float4(1.f, 1.f, 1.f, 1.f), S = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (kOut) S = a.a[cell];
    constexpr int U = 4;        // tokens loaded ahead of those being worked on
    GruRaw<DT> z[U], u[U], g[kOut ? U : 1];
    auto load = [&](int t, int i) {
        const int64_t at = (row + min(t, n - 1)) * a.ld + c;
        z[i].load(a.proj, at);
        u[i].load(a.proj, at + a.C);
        if constexpr (kOut) g[i].load(a.proj, at + 2 * a.C);
    };
#pragma unroll
    for (int i = 0; i < U; ++i) load(i, i);
    for (int t = 0; t < n; t += U) {
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const GruRaw<DT> zi = z[i], ui = u[i], gi = g[kOut ? i : 0];
            load(t + i + U, i);
            if (t + i < n) {
                float4 keep, add;
                gru_gates<DT>(zi.get(), ui.get(), bz, bu, keep, add);
                S = gru_fma(keep, S, add);
                if constexpr (kOut) gru_emit<DT>(a, row + t + i, c, S, gi.get());
                else A = make_float4(A.x * keep.x, A.y * keep.y, A.z * keep.z, A.w * keep.w);
            }
        }
    }
    if constexpr (!kOut) {
        a.a[cell] = A;
        a.b[cell] = S;
    }
}

// One value per thread; the loads of 16 chunks run ahead of the chain.
__global__ void __launch_bounds__(kGruThreads) gru_chain_kernel(const GruArgs a) {
    pdl_enter();
    const SsmSpan sp = a.spans[blockIdx.x];
    const int c = blockIdx.y * kGruThreads + threadIdx.x;
    if (sp.n <= 1 || c >= a.C) return;
    const int n = span_chunks(sp, kGruTok);
    float* st = a.state + static_cast<int64_t>(sp.slot) * a.C + c;
    float S = sp.seen > 0 ? *st : 0.0f;
    const int64_t cell = static_cast<int64_t>(first_chunk(a.spans, blockIdx.x, kGruTok)) * a.C + c;
    float* pa = reinterpret_cast<float*>(a.a) + cell;
    const float* pb = reinterpret_cast<const float*>(a.b) + cell;
    constexpr int U = 16;
    float A[U], B[U];
    auto load = [&](int i, int j) {
        const int64_t at = static_cast<int64_t>(min(i, n - 1)) * a.C;
        A[j] = __ldcg(pa + at);
        B[j] = __ldcg(pb + at);
    };
#pragma unroll
    for (int j = 0; j < U; ++j) load(j, j);
    for (int i = 0; i < n; i += U) {
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const float aj = A[j], bj = B[j];
            load(i + j + U, j);
            if (i + j < n) {
                pa[static_cast<int64_t>(i + j) * a.C] = S;
                S = fmaf(aj, S, bj);
            }
        }
    }
    *st = S;
}

template <int DT>
static int launch_gru(const GruArgs& a, int n_single, int T, cudaStream_t s) {
    const unsigned blocks = (a.C / 4 + kGruThreads - 1) / kGruThreads;
    const dim3 block(kGruThreads);
    const int n_multi = a.n_seqs - n_single;
    if (n_multi > 0) {
        const dim3 grid(T / kGruTok + n_multi, blocks);      // (at least as many as there are chunks)
        HDS_CHECK_CUDA(launch_kernel(gru_chunk_kernel<DT, false>, grid, block, 0, s, a));
        HDS_CHECK_CUDA(launch_kernel(gru_chain_kernel, dim3(a.n_seqs, (a.C + kGruThreads - 1) / kGruThreads), block, 0, s, a));
        if (a.out != nullptr) HDS_CHECK_CUDA(launch_kernel(gru_chunk_kernel<DT, true>, grid, block, 0, s, a));
    }
    if (n_single > 0) HDS_CHECK_CUDA(launch_kernel(gru_step_kernel<DT>, dim3(a.n_seqs, blocks), block, 0, s, a));
    return HDS_OK;
}

}  // namespace hds

using namespace hds;

extern "C" int64_t hds_gru_workspace_bytes(int T, int n_seqs, int width) {
    return static_cast<int64_t>(T / kGruTok + n_seqs) * width * 2 * 4;
}

extern "C" int hds_gru(const void* proj, int64_t ld_proj, const float* bias, float* state, const int32_t* spans, int n_seqs, int n_single, int T,
                       int width, void* out, int64_t ld_out, void* workspace, int64_t workspace_bytes, int dtype, void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_gru: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(width > 0 && width % 4 == 0 && ld_proj % 4 == 0 && ld_out % 4 == 0, "hds_gru: rows of 4-value vectors");
    HDS_REQUIRE(((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(out)) & (dtype == 2 ? 15 : 7)) == 0, "hds_gru: aligned rows");
    if (T == 0 || n_seqs == 0) return HDS_OK;
    HDS_REQUIRE(n_single == n_seqs || (workspace != nullptr && workspace_bytes >= hds_gru_workspace_bytes(T, n_seqs - n_single, width)),
                "hds_gru: workspace too small");
    float4* ws = static_cast<float4*>(workspace);
    const GruArgs a{proj, ld_proj, bias, state, reinterpret_cast<const SsmSpan*>(spans), n_seqs, width, out, ld_out,
                    ws, ws == nullptr ? nullptr : ws + static_cast<int64_t>(T / kGruTok + n_seqs - n_single) * (width / 4)};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == 0) return launch_gru<0>(a, n_single, T, s);
    if (dtype == 1) return launch_gru<1>(a, n_single, T, s);
    return launch_gru<2>(a, n_single, T, s);
}
