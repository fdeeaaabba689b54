// Retention over a ragged batch, per head:  S <- decay S + v k^T,  o = S q  (q and k turned by position), then o / rms(o) * silu(gate).
#include "linear_attention.cuh"
#include "../../../include/hds_b200.h"

using namespace hds;

extern "C" int64_t hds_retention_workspace_bytes(int T, int n_seqs, int heads, int vdim, int dim) { return 0; }

// Returns in *finished 1 when out holds the finished rows, 0 when y holds the read-outs (out still to be normed and gated).
extern "C" int hds_retention(const void* q, const void* k, const void* v, const void* gate, int64_t ld, const float* log2_decay,
                             const float* freq, const float* amp, float k_scale, int norm_cols, float* state, const int32_t* spans, int n_seqs,
                             int n_single, int T, int heads, int vdim, int dim, float* y, int64_t ld_y, void* out, int64_t ld_out,
                             const float* norm_w, float eps, void* workspace, int64_t workspace_bytes, int method, int* finished, int dtype,
                             void* stream) {
    HDS_REQUIRE(dtype >= 0 && dtype <= 2, "hds_retention: dtype 0 bf16 / 1 fp16 / 2 fp32");
    HDS_REQUIRE(heads >= 1 && vdim >= 1 && vdim <= 8192 && dim >= 2 && dim <= 1024 && dim % 2 == 0, "hds_retention: heads of up to 1024 x 8192");
    HDS_REQUIRE(norm_cols >= 1 && norm_cols <= vdim, "hds_retention: 1 <= norm_cols <= vdim");
    HDS_REQUIRE(method >= 0 && method <= 2, "hds_retention: method 0 / 1 / 2");
    *finished = 1;
    if (T == 0 || n_seqs == 0) return HDS_OK;
    LinArgs a{q, k, v, gate, ld, nullptr, 0, nullptr, 0.0f, state, reinterpret_cast<const SsmSpan*>(spans), n_seqs, T, heads, vdim, dim,
              y, ld_y, out, ld_out, norm_w, eps, 0, norm_cols, 1.0f, k_scale, log2_decay, freq, amp};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    int rc = HDS_OK;
    if (n_seqs > n_single) {
        *finished = 0;
        a.write_y = 1;      // by every row of the batch: one norm finishes them all
        rc = lin_launch_scan(a, dtype, true, s);
    }
    if (rc != HDS_OK || n_single == 0) return rc;
    return lin_launch_step(a, dtype, true, s);
}
