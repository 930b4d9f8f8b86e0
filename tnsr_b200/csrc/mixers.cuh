// Sequence mixers of models described layer by layer: launchers shared by layer_stack.cu and the operator tests.
// Every kernel exists for bf16 activations (the serving path) and f32 (everything in 32-bit); norms, scores, angles,
// decays, step sizes and the recurrent state are f32 in both.
#pragma once

#include "common.cuh"

namespace tb {

constexpr uint32_t kMaxConvTaps = 16;

// Where the rows of a step stand: row r belongs to session r / chunk and to position pos(session) + r % chunk.
struct StepPlace {
    uint32_t sessions = 0, chunk = 0;
    uint32_t position = 0;                  // used when d_position == nullptr
    const uint32_t* d_position = nullptr;   // device scalar, or one entry per session (position_stride 1)
    uint32_t position_stride = 0;
#ifdef __CUDACC__
    __device__ __forceinline__ uint32_t pos(uint32_t session) const {
        return d_position ? d_position[session * position_stride] : position;
    }
#endif
};

// Convolution inputs of a session live in a ring of `taps` rows indexed by position modulo taps.  A single-token step
// reads the taps - 1 older rows and overwrites the oldest one, so reader and writer never meet; longer chunks write the
// ring in a launch of their own (launch_conv_ring) after every reader is done.  A row of a negative position is zero
// and is never read from memory, so a session that starts at position 0 needs no clearing.
int launch_conv_ring(const void* rows, uint32_t ld, uint32_t channels, uint32_t taps, void* ring, const StepPlace& place,
                     int dtype, cudaStream_t stream);

// ---- attention ------------------------------------------------------------------
// Projected rows [q | k | v] -> convolution over time -> per-head RMS norm of q and k -> rotation -> q rows and cache rows.
struct AttentionPrep {
    const void* proj = nullptr;        // [rows, ld], channels q | k | v
    uint32_t ld = 0;
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0;
    const float* conv_w = nullptr;     // [channels, taps], last column = current token
    const float* q_norm = nullptr;     // [dim]
    const float* k_norm = nullptr;
    float eps = 0.0f;
    uint32_t rotary_dims = 0;
    const float2* rotation = nullptr;  // [position][rotary_dims / 2] (cos, sin)
    void* ring = nullptr;              // [sessions, taps, channels]
    void* q = nullptr;                 // [rows, heads * dim]
    void* k_cache = nullptr;           // [sessions, capacity, kv_heads * dim]
    void* v_cache = nullptr;           // [sessions, capacity, kv_heads * vdim]
    uint32_t capacity = 0;
    KvPaging paging;
};
int launch_attention_prep(const AttentionPrep& a, const StepPlace& place, int dtype, cudaStream_t stream);

// Grouped-query causal attention with capped scores and a sigmoid gate per head:
// out[row, h * vdim ..] = sigmoid(gate[row, h]) * softmax(cap(q . k * scale)) . v ; columns [heads * vdim, out_cols) are zeroed.
struct GroupedAttention {
    const void* q = nullptr;
    const void* k_cache = nullptr;
    const void* v_cache = nullptr;
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, capacity = 0;
    float scale = 0.0f, softcap = 0.0f;   // softcap 0: scores as they are
    const float* gate = nullptr;          // [rows, gate_ld], nullptr: no gate
    uint32_t gate_ld = 0;
    void* out = nullptr;
    uint32_t out_ld = 0, out_cols = 0;
    KvPaging paging;
    void* workspace = nullptr;            // grouped_attention_workspace_bytes(), zeroed once
    uint64_t workspace_bytes = 0;
    int engine = 0;                       // 0: best kernel for the shape, 1: one warp per (row, head)
};
uint64_t grouped_attention_workspace_bytes(uint32_t sessions, uint32_t heads, uint32_t kv_heads, uint32_t vdim);
int launch_grouped_attention(const GroupedAttention& a, const StepPlace& place, int dtype, cudaStream_t stream);

// ---- mamba2 ---------------------------------------------------------------------
struct Mamba2 {
    const void* proj = nullptr;        // [rows, ld], channels z (inner) | x (inner) | B (groups * state) | C (groups * state)
    uint32_t ld = 0;
    const float* dt = nullptr;         // [rows, dt_ld] projected step sizes, before bias and softplus
    uint32_t dt_ld = 0;
    uint32_t heads = 0, vdim = 0, state = 0, groups = 0, norm_groups = 0, taps = 0;
    const float* conv_w = nullptr;     // [inner + 2 groups * state, taps]
    const float* conv_b = nullptr;
    const float* dt_bias = nullptr;    // [heads]
    const float* a_log = nullptr;
    const float* d_skip = nullptr;
    const float* norm_w = nullptr;     // [inner]
    float eps = 0.0f;
    void* ring = nullptr;              // [sessions, taps, inner + 2 groups * state]
    float* ssm = nullptr;              // [sessions, heads, state, vdim]
    void* xbc = nullptr;               // [rows, inner + 2 groups * state] scratch (chunks of two tokens and more)
    void* gated = nullptr;             // [rows, inner] scratch: y * silu(z)
    void* out = nullptr;               // [rows, out_ld]; columns [inner, out_cols) are zeroed
    uint32_t out_ld = 0, out_cols = 0;
    int engine = 0;                    // 0: best kernel for the shape, 1: token by token
};
bool mamba2_supported(uint32_t heads, uint32_t vdim, uint32_t state);
int launch_mamba2(const Mamba2& m, const StepPlace& place, int dtype, cudaStream_t stream);

}  // namespace tb
