// extern "C" wrappers of the individual kernels (operator-level entry points of
// include/tnsr_b200.h).  They queue work on the caller's stream and never
// synchronise or allocate.
#include "common.cuh"
#include "feed_forward.cuh"
#include "mixers.cuh"

using namespace tb;

namespace {
inline cudaStream_t as_stream(void* s) { return reinterpret_cast<cudaStream_t>(s); }
inline int bad(const char* msg) {
    set_thread_error(msg);
    return TNSR_B200_ERR_INVALID_ARGUMENT;
}
}  // namespace

extern "C" {

int tnsr_b200_embedding(const void* token_table, const void* position_table, const uint32_t* ids, float* out,
                        uint32_t rows, uint32_t chunk, uint32_t position0, uint32_t vocab, uint32_t width, int dtype,
                        int* d_status, void* stream) {
    if (!token_table || !position_table || !ids || !out) return bad("embedding: null pointer");
    if (dtype != TNSR_B200_F32 && dtype != TNSR_B200_BF16) return bad("embedding: dtype must be f32 or bf16");
    if (chunk == 0 || width == 0) return bad("embedding: chunk and width must be non-zero");
    return launch_embedding(token_table, position_table, ids, out, rows, chunk, position0, nullptr, vocab, width, dtype,
                            d_status, as_stream(stream));
}

int tnsr_b200_layernorm(const float* x, const float* weight, const float* bias, void* out, uint32_t rows, uint32_t width,
                        float epsilon, int out_dtype, int strict, void* stream) {
    if (!x || !weight || !bias || !out) return bad("layernorm: null pointer");
    if (width == 0 || !(epsilon > 0.0f)) return bad("layernorm: width and epsilon must be positive");
    if (out_dtype != TNSR_B200_F32 && out_dtype != TNSR_B200_BF16) return bad("layernorm: bad output dtype");
    return launch_layernorm(x, weight, bias, out, rows, width, epsilon, out_dtype, strict != 0, as_stream(stream));
}

int tnsr_b200_gemm_f32_strict(const float* a, const float* b, const float* bias, float* out, uint32_t m, uint32_t k,
                              uint32_t n, int b_transposed, void* stream) {
    if (!a || !b || !out) return bad("gemm_f32_strict: null pointer");
    GemmEpilogue ep;
    ep.bias = bias;
    return launch_gemm_strict(a, b, out, n, m, k, n, b_transposed != 0, ep, as_stream(stream));
}

int tnsr_b200_gemm_bf16(const void* a, const void* bt, const float* bias, const float* residual, void* out, uint32_t m,
                        uint32_t n, uint32_t k, int activation, int out_dtype, void* stream) {
    return tnsr_b200_gemm_bf16_ws(a, bt, bias, residual, out, m, n, k, activation, out_dtype, nullptr, 0, stream);
}

uint64_t tnsr_b200_gemm_workspace(void) { return gemm_skinny_workspace_bytes(); }

int tnsr_b200_gemm_bf16_ws(const void* a, const void* bt, const float* bias, const float* residual, void* out, uint32_t m,
                           uint32_t n, uint32_t k, int activation, int out_dtype, void* workspace, uint64_t workspace_bytes,
                           void* stream) {
    if (!a || !bt || !out) return bad("gemm_bf16: null pointer");
    if (out_dtype != TNSR_B200_F32 && out_dtype != TNSR_B200_BF16) return bad("gemm_bf16: bad output dtype");
    if (activation < -1 || activation > TNSR_B200_ACT_GELU_TANH || activation == TNSR_B200_ACT_SWIGLU)
        return bad("gemm_bf16: activation must be -1, RELU, GELU or GELU_TANH");
    if (residual && out_dtype != TNSR_B200_F32) return bad("gemm_bf16: a residual needs f32 output");
    GemmEpilogue ep;
    ep.bias = bias;
    ep.residual = residual;
    ep.ldr = n;
    ep.activation = activation;
    ep.out_dtype = out_dtype;
    if (workspace) {
        if (workspace_bytes < gemm_skinny_workspace_bytes() || (reinterpret_cast<uintptr_t>(workspace) & 15))
            return bad("gemm_bf16_ws: workspace too small or not 16-byte aligned");
        ep.skinny_ws = workspace;
        ep.skinny_ws_bytes = workspace_bytes;
    }
    return launch_gemm_bf16((const bf16*)a, (const bf16*)bt, out, n, m, n, k, GEMM_PLAIN, ep, nullptr, nullptr,
                            as_stream(stream));
}

int tnsr_b200_transpose_bf16(const void* in, void* out, uint32_t k, uint32_t n, void* stream) {
    if (!in || !out) return bad("transpose_bf16: null pointer");
    return launch_transpose_bf16((const bf16*)in, (bf16*)out, k, n, as_stream(stream));
}

int tnsr_b200_swiglu(const void* gate, const void* up, void* out, uint64_t elems, void* stream) {
    if (!gate || !up || !out) return bad("swiglu: null pointer");
    return launch_swiglu((const bf16*)gate, (const bf16*)up, (bf16*)out, elems, as_stream(stream));
}

int tnsr_b200_pack_gate_up(const void* w_gate, const void* w_up, const float* b_gate, const float* b_up, void* w_out,
                           float* b_out, uint32_t d, uint32_t f, void* stream) {
    if (!w_gate || !w_up || !w_out) return bad("pack_gate_up: null pointer");
    return launch_pack_gate_up((const bf16*)w_gate, (const bf16*)w_up, b_gate, b_up, (bf16*)w_out, b_out, d, f,
                               as_stream(stream));
}

int tnsr_b200_swiglu_mlp(const void* x, const void* w_gate_up_t, const float* b_gate_up, const void* w_down_t,
                         const float* b_down, void* hidden, void* out, uint32_t rows, uint32_t d, uint32_t f, void* stream) {
    if (!x || !w_gate_up_t || !w_down_t || !hidden || !out) return bad("swiglu_mlp: null pointer");
    if (f % 16 != 0) {
        set_thread_error("swiglu_mlp: feed-forward width must be a multiple of 16");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    GemmEpilogue eg;
    eg.bias = b_gate_up;
    eg.out_dtype = TNSR_B200_BF16;
    int rc = launch_gemm_bf16((const bf16*)x, (const bf16*)w_gate_up_t, hidden, f, rows, 2 * f, d, GEMM_SWIGLU, eg, nullptr,
                              nullptr, as_stream(stream));
    if (rc) return rc;
    GemmEpilogue ed;
    ed.bias = b_down;
    ed.out_dtype = TNSR_B200_BF16;
    return launch_gemm_bf16((const bf16*)hidden, (const bf16*)w_down_t, out, d, rows, d, f, GEMM_PLAIN, ed, nullptr, nullptr,
                            as_stream(stream));
}

uint64_t tnsr_b200_decode_attention_workspace(uint32_t batch, uint32_t capacity, uint32_t heads, uint32_t head_dim) {
    return decode_attention_workspace_bytes(batch, capacity, heads, head_dim);
}

int tnsr_b200_decode_attention(const void* q, const void* k_cache, const void* v_cache, const uint32_t* lengths, void* out,
                               void* workspace, uint64_t workspace_bytes, uint32_t batch, uint32_t capacity, uint32_t heads,
                               uint32_t head_dim, void* stream) {
    if (!q || !k_cache || !v_cache || !lengths || !out || !workspace) return bad("decode_attention: null pointer");
    // nothing may be written before the size is known to fit (the status word below lives inside the workspace)
    if (workspace_bytes < decode_attention_workspace_bytes(batch, capacity, heads, head_dim) || workspace_bytes < 256)
        return bad("decode_attention: workspace smaller than tnsr_b200_decode_attention_workspace() asks for");
    // bytes 64..67 of the workspace hold the kernel's status word
    int* d_status = reinterpret_cast<int*>(reinterpret_cast<uint8_t*>(workspace) + 64);
    cudaError_t e = cudaMemsetAsync(d_status, 0, 4, as_stream(stream));
    if (e != cudaSuccess) {
        set_thread_error(std::string("decode_attention: ") + cudaGetErrorString(e));
        return TNSR_B200_ERR_CUDA;
    }
    return launch_decode_attention((const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, lengths, (bf16*)out, workspace,
                                   workspace_bytes, batch, capacity, heads, head_dim, d_status, as_stream(stream));
}

int tnsr_b200_prefill_attention(const void* q, const void* k_cache, const void* v_cache, void* out, uint32_t batch,
                                uint32_t chunk, uint32_t position, uint32_t capacity, uint32_t heads, uint32_t head_dim,
                                void* stream) {
    if (!q || !k_cache || !v_cache || !out) return bad("prefill_attention: null pointer");
    if ((uint64_t)position + chunk > capacity) return bad("prefill_attention: position + chunk exceeds the capacity");
    if (prefill_attention_supported(head_dim))
        return launch_prefill_attention((const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, batch, chunk,
                                        position, nullptr, capacity, heads, head_dim, nullptr, as_stream(stream));
    return launch_attention_generic((const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, batch, chunk,
                                    position, nullptr, capacity, heads, head_dim, as_stream(stream));
}

int tnsr_b200_sample_top_k(const float* logits, uint32_t* out, uint32_t rows, uint32_t vocab, float temperature,
                           uint32_t top_k, uint64_t seed, uint32_t step, uint32_t first_session, void* stream) {
    if (!logits || !out) return bad("sample_top_k: null pointer");
    return launch_sample_top_k(logits, out, rows, vocab, vocab, temperature, top_k, seed, nullptr, 0, step, first_session,
                               as_stream(stream));
}

int tnsr_b200_argmax(const float* logits, uint32_t* out, uint32_t rows, uint32_t vocab, void* stream) {
    if (!logits || !out || vocab == 0) return bad("argmax: null pointer or empty vocabulary");
    return launch_argmax(logits, out, rows, vocab, vocab, as_stream(stream));
}

int tnsr_b200_rmsnorm(const float* x, const float* weight, float offset, void* out, uint32_t rows, uint32_t width,
                      float epsilon, int out_dtype, void* stream) {
    if (!x || !weight || !out) return bad("rmsnorm: null pointer");
    if (width == 0 || !(epsilon > 0.0f)) return bad("rmsnorm: width and epsilon must be positive");
    if (out_dtype != TNSR_B200_F32 && out_dtype != TNSR_B200_BF16) return bad("rmsnorm: bad output dtype");
    return launch_rmsnorm(x, weight, offset, out, rows, width, epsilon, out_dtype, as_stream(stream));
}

uint64_t tnsr_b200_grouped_attention_workspace(uint32_t dim, uint32_t vdim) { return grouped_attention_workspace_bytes(dim, vdim); }

static StepPlace step_place(const tnsr_b200_place* p) {
    StepPlace place;
    place.sessions = p->sessions;
    place.chunk = p->chunk;
    place.position = p->position;
    place.d_position = p->d_positions;
    place.position_stride = p->d_positions ? 1u : 0u;
    return place;
}

int tnsr_b200_grouped_attention(const tnsr_b200_grouped_attention_args* args, const tnsr_b200_place* place, void* stream) {
    if (!args || !place || !args->q || !args->k_cache || !args->v_cache || !args->out) return bad("grouped_attention: null pointer");
    if (args->dtype != TNSR_B200_F32 && args->dtype != TNSR_B200_BF16) return bad("grouped_attention: dtype must be f32 or bf16");
    if (args->score_kind > TNSR_B200_SCORE_SIGMOID) return bad("grouped_attention: unknown score kind");
    if (args->heads == 0 || args->dim == 0 || args->vdim == 0 || args->capacity == 0 || args->out_ld < args->out_cols ||
        args->out_cols < args->heads * args->vdim)
        return bad("grouped_attention: sizes must be positive and the output row must hold every head");
    if (!place->d_positions && (uint64_t)place->position + place->chunk > args->capacity) return bad("grouped_attention: the chunk ends past the capacity");
    GroupedAttention a;
    a.q = args->q; a.k_cache = args->k_cache; a.v_cache = args->v_cache;
    a.heads = args->heads; a.kv_heads = args->kv_heads; a.dim = args->dim; a.vdim = args->vdim; a.capacity = args->capacity;
    a.scale = args->scale; a.softcap = args->softcap; a.gate = args->gate; a.gate_ld = args->gate_ld;
    a.out = args->out; a.out_ld = args->out_ld; a.out_cols = args->out_cols;
    a.d_status = args->d_status; a.workspace = args->workspace; a.workspace_bytes = args->workspace_bytes; a.engine = args->engine;
    a.head_bias = args->head_bias; a.window = args->window; a.score_kind = args->score_kind; a.gain = args->gain != 0.0f ? args->gain : 1.0f;
    return launch_grouped_attention(a, step_place(place), args->dtype, as_stream(stream));
}

int tnsr_b200_mamba2(const tnsr_b200_mamba2_args* args, const tnsr_b200_place* place, void* stream) {
    if (!args || !place || !args->proj || !args->dt || !args->conv_w || !args->conv_b || !args->dt_bias || !args->a_log || !args->d_skip ||
        !args->norm_w || !args->ring || !args->ssm || !args->xbc || !args->gated || !args->out)
        return bad("mamba2: null pointer");
    if (args->dtype != TNSR_B200_F32 && args->dtype != TNSR_B200_BF16) return bad("mamba2: dtype must be f32 or bf16");
    if (args->groups == 0 || args->heads == 0 || args->heads % args->groups || args->norm_groups == 0 ||
        (args->heads * args->vdim) % args->norm_groups || args->out_ld < args->out_cols || args->out_cols < args->heads * args->vdim)
        return bad("mamba2: groups must divide heads, norm_groups the width, and the output row must hold every head");
    Mamba2 m;
    m.proj = args->proj; m.ld = args->ld; m.dt = args->dt; m.dt_ld = args->dt_ld;
    m.heads = args->heads; m.vdim = args->vdim; m.state = args->state; m.groups = args->groups; m.norm_groups = args->norm_groups; m.taps = args->taps;
    m.conv_w = args->conv_w; m.conv_b = args->conv_b; m.dt_bias = args->dt_bias; m.a_log = args->a_log; m.d_skip = args->d_skip; m.norm_w = args->norm_w;
    m.eps = args->eps; m.ring = args->ring; m.ssm = args->ssm; m.xbc = args->xbc; m.gated = args->gated;
    m.out = args->out; m.out_ld = args->out_ld; m.out_cols = args->out_cols; m.engine = args->engine;
    return launch_mamba2(m, step_place(place), args->dtype, as_stream(stream));
}

static bool two_types(int32_t dtype) { return dtype == TNSR_B200_F32 || dtype == TNSR_B200_BF16; }

int tnsr_b200_rotary(const tnsr_b200_rotary_args* args, const tnsr_b200_place* place, void* stream) {
    if (!args || !place || !args->proj || !args->q || !args->k_cache || !args->v_cache || (args->rotary_dims && !args->rotation)) return bad("rotary: null pointer");
    if (!two_types(args->dtype) || args->rotary_layout > TNSR_B200_ROTARY_HALVES) return bad("rotary: bad dtype or layout");
    if (args->heads == 0 || args->kv_heads == 0 || args->dim == 0 || args->vdim == 0 || args->rotary_dims > args->dim || args->rotary_dims % 2 ||
        args->ld < args->heads * args->dim + args->kv_heads * (args->dim + args->vdim))
        return bad("rotary: sizes must be positive, rotated dimensions even and the rows must hold q, k and v");
    if (!place->d_positions && (uint64_t)place->position + place->chunk > args->capacity) return bad("rotary: the chunk ends past the capacity");
    AttentionPrep p;
    p.proj = args->proj; p.ld = args->ld; p.heads = args->heads; p.kv_heads = args->kv_heads; p.dim = args->dim; p.vdim = args->vdim;
    p.rotary_dims = args->rotary_dims; p.rotary_layout = args->rotary_layout; p.rotation = (const float2*)args->rotation;
    p.q = args->q; p.k_cache = args->k_cache; p.v_cache = args->v_cache; p.capacity = args->capacity;
    return launch_attention_prep(p, step_place(place), args->dtype, as_stream(stream));
}

int tnsr_b200_hgrn2(const tnsr_b200_hgrn2_args* args, const tnsr_b200_place* place, void* stream) {
    if (!args || !place || !args->q || !args->v || !args->f || !args->f_bias || !args->lower || !args->norm_w || !args->state || !args->out)
        return bad("hgrn2: null pointer");
    if (!two_types(args->dtype)) return bad("hgrn2: dtype must be f32 or bf16");
    if (args->heads == 0 || args->dim == 0 || args->vdim == 0 || args->f_ld < args->heads * args->dim || args->out_ld < args->out_cols ||
        args->out_cols < args->heads * args->vdim)
        return bad("hgrn2: sizes must be positive and the rows must hold every head");
    Hgrn2 m;
    m.q = args->q; m.v = args->v; m.ld = args->ld; m.f = args->f; m.f_ld = args->f_ld; m.heads = args->heads; m.dim = args->dim; m.vdim = args->vdim;
    m.f_bias = args->f_bias; m.lower = args->lower; m.norm_w = args->norm_w; m.eps = args->eps; m.gain = args->gain; m.state = args->state; m.raw = args->raw;
    m.out = args->out; m.out_ld = args->out_ld; m.out_cols = args->out_cols; m.engine = args->engine;
    return launch_hgrn2(m, step_place(place), args->dtype, as_stream(stream));
}

int tnsr_b200_rglru(const tnsr_b200_rglru_args* args, const tnsr_b200_place* place, void* stream) {
    if (!args || !place || !args->proj || !args->gate_w || !args->conv_w || !args->conv_b || !args->r_bias || !args->i_bias || !args->lambda ||
        !args->ring || !args->state || !args->u || !args->gates || !args->out)
        return bad("rglru: null pointer");
    if (!two_types(args->dtype)) return bad("rglru: dtype must be f32 or bf16");
    if (args->width == 0 || args->x_col < args->width || args->ld < args->x_col + args->width || args->out_ld < args->out_cols || args->out_cols < args->width)
        return bad("rglru: the rows must hold y, x and the output");
    Rglru m;
    m.proj = args->proj; m.ld = args->ld; m.x_col = args->x_col; m.width = args->width; m.blocks = args->blocks; m.taps = args->taps;
    m.conv_w = args->conv_w; m.conv_b = args->conv_b; m.gate_w = args->gate_w; m.r_bias = args->r_bias; m.i_bias = args->i_bias; m.lambda = args->lambda;
    m.ring = args->ring; m.state = args->state; m.u = args->u; m.gates = args->gates; m.out = args->out; m.out_ld = args->out_ld; m.out_cols = args->out_cols;
    m.d_status = args->d_status;
    return launch_rglru(m, step_place(place), args->dtype, as_stream(stream));
}

int tnsr_b200_polynorm(const void* z, const float* act, void* out, uint32_t rows, uint32_t width, uint32_t out_ld, uint32_t out_cols, float epsilon,
                       int dtype, void* stream) {
    if (!z || !act || !out) return bad("polynorm: null pointer");
    if (!two_types(dtype) || width == 0 || out_cols < width || out_ld < out_cols || !(epsilon > 0.0f)) return bad("polynorm: bad dtype, sizes or epsilon");
    return launch_polynorm(z, act, out, rows, width, out_ld, out_cols, epsilon, dtype, as_stream(stream));
}

int tnsr_b200_gemm_grouped(const void* a, const void* w, void* out, const uint32_t* offsets, uint32_t groups, uint32_t rows, uint32_t n, uint32_t k,
                           int activation, int dtype, int out_dtype, int engine, int* d_status, void* stream) {
    if (!a || !w || !out) return bad("gemm_grouped: null pointer");
    if (!two_types(dtype) || !two_types(out_dtype)) return bad("gemm_grouped: dtype must be f32 or bf16");
    GroupedGemm g;
    g.a = a; g.w = w; g.out = out; g.offsets = offsets; g.groups = groups; g.rows = rows; g.n = n; g.k = k; g.activation = activation;
    g.out_dtype = out_dtype; g.d_status = d_status; g.engine = engine;
    return launch_gemm_grouped(g, dtype, as_stream(stream));
}

uint64_t tnsr_b200_experts_workspace(uint32_t rows, uint32_t d, uint32_t ff, uint32_t experts, uint32_t top, int dtype) {
    return experts_workspace_bytes(rows, d, ff, experts, top, dtype);
}

int tnsr_b200_experts(const tnsr_b200_experts_args* args, void* stream) {
    if (!args || !args->logits || !args->correction || !args->h || !args->up || !args->down || !args->x || !args->workspace ||
        (args->norm_out && !args->norm_w))
        return bad("experts: null pointer");
    if (!two_types(args->dtype)) return bad("experts: dtype must be f32 or bf16");
    if (args->d == 0 || args->ff == 0 || args->logits_ld < args->experts + args->identity_experts) return bad("experts: bad sizes");
    Experts e;
    e.logits = args->logits; e.correction = args->correction; e.h = args->h; e.up = args->up; e.down = args->down; e.x = args->x;
    e.layer_scale = args->layer_scale; e.norm_w = args->norm_w; e.norm_out = args->norm_out; e.workspace = args->workspace;
    e.workspace_bytes = args->workspace_bytes; e.chosen = args->chosen; e.weights = args->weights; e.d_status = args->d_status; e.rows = args->rows;
    e.logits_ld = args->logits_ld; e.d = args->d; e.ff = args->ff; e.experts = args->experts; e.identity = args->identity_experts; e.top = args->top;
    e.router_scale = args->router_scale; e.norm_offset = args->norm_offset; e.eps = args->eps; e.engine = args->engine;
    int rc = launch_experts(e, args->dtype, as_stream(stream));
    return rc ? rc : launch_experts_combine(e, args->dtype, as_stream(stream));
}

}  // extern "C"
