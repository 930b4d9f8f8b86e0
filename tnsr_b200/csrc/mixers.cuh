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
// conv_w == nullptr: rotation alone (no convolution, no norm, no ring), in either layout.
struct AttentionPrep {
    const void* proj = nullptr;        // [rows, ld], channels q | k | v
    uint32_t ld = 0;
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0;
    const float* conv_w = nullptr;     // [channels, taps], last column = current token
    const float* q_norm = nullptr;     // [dim]
    const float* k_norm = nullptr;
    float eps = 0.0f;
    uint32_t rotary_dims = 0;
    uint32_t rotary_layout = TNSR_B200_ROTARY_INTERLEAVED;   // halves: without a convolution only
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
// out[row, h * vdim ..] = gain * sigmoid(gate[row, h]) * softmax(cap(q . k * scale)) . v ; columns [heads * vdim, out_cols)
// are zeroed.  window > 0: a query at i sees keys i - window + 1 .. i.  score_kind SIGMOID: the weight of a
// visible key is sigmoid(q . k * scale + head_bias[h]), and no sum divides the result (softcap does not apply).
struct GroupedAttention {
    const void* q = nullptr;
    const void* k_cache = nullptr;
    const void* v_cache = nullptr;
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, capacity = 0;
    float scale = 0.0f, softcap = 0.0f;   // softcap 0: scores as they are
    float gain = 1.0f;
    uint32_t window = 0, score_kind = TNSR_B200_SCORE_SOFTMAX;
    const float* head_bias = nullptr;     // [heads], sigmoid scores
    const float* gate = nullptr;          // [rows, gate_ld], nullptr: no gate
    uint32_t gate_ld = 0;
    void* out = nullptr;
    uint32_t out_ld = 0, out_cols = 0;
    KvPaging paging;
    void* workspace = nullptr;            // grouped_attention_workspace_bytes(), zeroed once
    uint64_t workspace_bytes = 0;
    int* d_status = nullptr;              // device status word (a bounded wait of the tcgen05 kernel gave up), may be null
    int engine = 0;                       // 0: best kernel for the shape, 1: one warp per (row, head), 2: not the tcgen05 kernel
};
uint64_t grouped_attention_workspace_bytes(uint32_t dim, uint32_t vdim);
int launch_grouped_attention(const GroupedAttention& a, const StepPlace& place, int dtype, cudaStream_t stream);

// Many rows, heads of 64, position on the host: the tcgen05 kernel of prefill_tc.cu.
bool grouped_attention_tc_eligible(const GroupedAttention& a, const StepPlace& place);
int launch_grouped_attention_tc(const GroupedAttention& a, const StepPlace& place, cudaStream_t stream);

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
    void* xbc = nullptr;               // [rows, inner + 2 groups * state] scratch: convolved x | B | C
    void* gated = nullptr;             // [rows, inner] scratch: y * silu(z)
    void* out = nullptr;               // [rows, out_ld]; columns [inner, out_cols) are zeroed
    uint32_t out_ld = 0, out_cols = 0;
    int engine = 0;                    // 0: best kernel for the shape, 1: token by token
};
bool mamba2_supported(uint32_t heads, uint32_t vdim, uint32_t state);
int launch_mamba2(const Mamba2& m, const StepPlace& place, int dtype, cudaStream_t stream);

// ---- convolution alone ------------------------------------------------------------
// out = [silu](conv(rows) + bias), reading and updating the session's ring.  Output channels may be cut into parts of
// `part` channels, each a matrix [rows, part] of its own.
struct ShortConv {
    const void* rows = nullptr;        // [rows, ld]
    uint32_t ld = 0, channels = 0, taps = 0, part = 0;   // part: channels, or a divisor of it
    const float* w = nullptr;          // [channels, taps]
    const float* b = nullptr;
    void* ring = nullptr;              // [sessions, taps, channels]
    void* out = nullptr;               // [channels / part][rows][part]
    bool silu = false;
};
int launch_short_conv(const ShortConv& c, const StepPlace& place, int dtype, cudaStream_t stream);

// ---- HGRN2 ------------------------------------------------------------------------
// f = l + (1 - l) sigmoid(f_raw + b);  S <- diag(f) S + (1 - f) v^T;  o = S^T silu(q);  out = gain * norm_w * o / rms(o)
struct Hgrn2 {
    const void* q = nullptr;           // [rows, ld], before silu
    const void* v = nullptr;           // [rows, ld]
    uint32_t ld = 0;
    const float* f = nullptr;          // [rows, f_ld], before bias and sigmoid
    uint32_t f_ld = 0;
    uint32_t heads = 0, dim = 0, vdim = 0;
    const float* f_bias = nullptr;     // [heads * dim]
    const float* lower = nullptr;      // [heads * dim]
    const float* norm_w = nullptr;     // [vdim]
    float eps = 0.0f, gain = 1.0f;
    float* state = nullptr;            // [sessions, heads, dim, vdim]
    float* raw = nullptr;              // [rows, heads * vdim] scratch, used when vdim > HGRN2_FUSED_VDIM
    void* out = nullptr;               // [rows, out_ld]; columns [heads * vdim, out_cols) are zeroed
    uint32_t out_ld = 0, out_cols = 0;
    int engine = 0;                    // 0: best kernel for the shape, 1: token by token
};
constexpr uint32_t HGRN2_FUSED_VDIM = 128;   // value width up to which the kernels norm their own output
bool hgrn2_supported(uint32_t heads, uint32_t dim, uint32_t vdim);
int launch_hgrn2(const Hgrn2& m, const StepPlace& place, int dtype, cudaStream_t stream);

// ---- real-gated linear recurrent unit ------------------------------------------------
struct Rglru {
    const void* proj = nullptr;        // [rows, ld]: y (after gelu) from column 0, x from column x_col
    uint32_t ld = 0, x_col = 0;
    uint32_t width = 0, blocks = 0, taps = 0;
    const float* conv_w = nullptr;     // [width, taps]
    const float* conv_b = nullptr;
    const void* gate_w = nullptr;      // [blocks, 2 n, n]: rows of r, then of i; n = width / blocks
    const float* r_bias = nullptr;     // [width]
    const float* i_bias = nullptr;
    const float* lambda = nullptr;     // [width]
    void* ring = nullptr;              // [sessions, taps, width]
    float* state = nullptr;            // [sessions, width]
    void* u = nullptr;                 // [blocks, rows, n] scratch: convolved x
    float* gates = nullptr;            // [blocks, rows, 2 n] scratch
    void* out = nullptr;               // [rows, out_ld]; columns [width, out_cols) are zeroed
    uint32_t out_ld = 0, out_cols = 0;
    int* d_status = nullptr;
};
int launch_rglru(const Rglru& m, const StepPlace& place, int dtype, cudaStream_t stream);

// ---- device helpers ----------------------------------------------------------------
#ifdef __CUDACC__
__device__ __forceinline__ float full_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
// Two neighbouring channels as f32; one access when `vec` (even address), else element by element (`second`: the second
// one exists).
template <typename T>
__device__ __forceinline__ float2 load_pair(const T* p, bool vec, bool second);
template <>
__device__ __forceinline__ float2 load_pair<float>(const float* p, bool vec, bool second) {
    if (vec) return *reinterpret_cast<const float2*>(p);
    return make_float2(p[0], second ? p[1] : 0.0f);
}
template <>
__device__ __forceinline__ float2 load_pair<bf16>(const bf16* p, bool vec, bool second) {
    if (vec) return bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(p));
    return make_float2(__bfloat162float(p[0]), second ? __bfloat162float(p[1]) : 0.0f);
}
template <typename T>
__device__ __forceinline__ void store_pair(T* p, float2 v, bool vec, bool second);
template <>
__device__ __forceinline__ void store_pair<float>(float* p, float2 v, bool vec, bool second) {
    if (vec) { *reinterpret_cast<float2*>(p) = v; return; }
    p[0] = v.x;
    if (second) p[1] = v.y;
}
template <>
__device__ __forceinline__ void store_pair<bf16>(bf16* p, float2 v, bool vec, bool second) {
    if (vec) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v.x, v.y); return; }
    p[0] = __float2bfloat16_rn(v.x);
    if (second) p[1] = __float2bfloat16_rn(v.y);
}

// Warp-level tensor-core pieces shared by the grouped attention and the chunked scan: ldmatrix, mma.sync m16n8k16
// (bf16 operands, f32 accumulators), 16-byte asynchronous copies.
__device__ __forceinline__ uint32_t mx_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mx_cp16(void* dst, const void* src, bool real) {
    const uint32_t bytes = real ? 16u : 0u;   // zero-fill when the source is outside
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mx_smem(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mx_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void mx_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void mx_ldsm(uint32_t addr, uint32_t* r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mx_ldsm_t(uint32_t addr, uint32_t* r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mx_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float mx_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float mx_rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// silu by one exponential and one reciprocal of the special-function unit (for results that are stored as bf16).
__device__ __forceinline__ float mx_silu(float x) { return x * mx_rcp(1.0f + mx_ex2(-1.4426950408889634f * x)); }
// x = hi + lo with both halves bf16: two products with an exact bf16 operand then carry 16 bits of x.
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(x, y);
    const float2 h = bf16x2_to_f32(hi);
    lo = pack_bf16x2(x - h.x, y - h.y);
}
#endif  // __CUDACC__

}  // namespace tb
