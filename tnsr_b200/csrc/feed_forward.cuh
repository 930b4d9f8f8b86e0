// Feed-forwards of models described layer by layer and the grouped product they and the recurrent gates use.
#pragma once

#include "common.cuh"

namespace tb {

// ---- products of row groups with a matrix each -----------------------------------
// Rows offsets[g] .. offsets[g + 1] of a [rows, k] times w[g] [n, k] transposed -> out [rows, n].
struct GroupedGemm {
    const void* a = nullptr;
    const void* w = nullptr;              // [groups, n, k]
    void* out = nullptr;
    const uint32_t* offsets = nullptr;    // [groups + 1] on the device; nullptr: rows / groups rows each
    uint32_t groups = 0, rows = 0, n = 0, k = 0;
    int activation = ACT_NONE;
    int out_dtype = TNSR_B200_F32;
    int* d_status = nullptr;
    int engine = 0;                       // 0: tcgen05 where the shape allows it, 1: CUDA cores
};
// dtype: element type of a and w.
int launch_gemm_grouped(const GroupedGemm& g, int dtype, cudaStream_t stream);

// ---- PolyNorm ---------------------------------------------------------------------
// out[r] = a N(z) + b N(z^2) + c N(z^3) + e, N(v) = v / sqrt(mean(v^2) + eps) over the row; act = {a, b, c, e} on the device.
// Columns [width, out_cols) are zeroed.
int launch_polynorm(const void* z, const float* act, void* out, uint32_t rows, uint32_t width, uint32_t out_ld, uint32_t out_cols,
                    float eps, int dtype, cudaStream_t stream);

// ---- mixture of experts --------------------------------------------------------------
// x += layer_scale * sum over the chosen experts (see tnsr_b200_experts), then optionally the next norm of x.
struct Experts {
    const float* logits = nullptr;        // [rows, logits_ld]
    const float* correction = nullptr;    // [experts + identity]
    const void* h = nullptr;              // [rows, d]
    const void* up = nullptr;             // [experts, ff, d]
    const void* down = nullptr;           // [experts, d, ff]
    float* x = nullptr;                   // [rows, d]
    const float* layer_scale = nullptr;   // [d] or nullptr
    const float* norm_w = nullptr;        // [d], with norm_out
    void* norm_out = nullptr;             // [rows, d] or nullptr; may be h
    void* workspace = nullptr;
    uint64_t workspace_bytes = 0;
    uint32_t* chosen = nullptr;           // [rows, top] or nullptr
    float* weights = nullptr;             // [rows, top] or nullptr
    int* d_status = nullptr;
    uint32_t rows = 0, logits_ld = 0, d = 0, ff = 0, experts = 0, identity = 0, top = 0;
    float router_scale = 1.0f, norm_offset = 0.0f, eps = 0.0f;
    int engine = 0;
    // Set `router` to have launch_experts also norm x into h and form the router logits (steps of few rows, see
    // experts_fused_router); `logits` is not read then.
    const void* router = nullptr;         // [experts + identity, d]
    const float* router_norm = nullptr;   // [d]
    const float* partials = nullptr;      // partial sums of a split product, added to x first (launch_layernorm_fold)
    uint32_t parts = 0, split_rows = 0;   // at most 4
};
constexpr uint32_t kMaxExperts = 1024;    // experts and identity experts together
constexpr uint32_t kMaxTop = 32;
bool experts_fused_router(const Experts& e);
uint64_t experts_workspace_bytes(uint32_t rows, uint32_t d, uint32_t ff, uint32_t experts, uint32_t top, int dtype);
// Routing, both grouped products and the gather between them; the result stays in the workspace.
int launch_experts(const Experts& e, int dtype, cudaStream_t stream);
// The other half: x += layer_scale * weighted sum, and the norm if norm_out is set.
int launch_experts_combine(const Experts& e, int dtype, cudaStream_t stream);

}  // namespace tb
