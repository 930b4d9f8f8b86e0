// Sessions of models that are described layer by layer (tnsr_b200_decoder_create_stack).  The handle, its stream, token
// staging, page table, sampler, captured steps and entry points are those of decoder.cu; this file holds what such a
// model adds: packed weights, one cache or state per layer, and the step.
//
// Everything that reads a norm's rows is one product (column ranges routed by the epilogue), everything that a mixer adds
// to the residual another, whatever the mixer is.  Parallel blocks, where the feed-forward reads the mixer's rows:
//   norm -> [projections | up] -> mixer -> [mixer output | activated up] . [W_o | W_down]^T added to the residual
// Sequential blocks, with a layer scale s (a factor per output column of the product):
//   norm1 -> [projections] -> mixer -> mixer output . W_o^T s1 added to the residual
//   norm2 -> feed-forward (dense: up, activation, down s2 added; experts: router, grouped products, weighted sum s2 added
//            by the kernel that also forms the next norm)
// Two mixers side by side are column ranges of the same two products; their gains are applied where they write.
#include <algorithm>
#include <cmath>
#include <cstring>

#include "decoder.cuh"
#include "feed_forward.cuh"
#include "mixers.cuh"

namespace tb {

struct StackWeights {
    float* norm = nullptr;
    void* w_in = nullptr;        // [n_in, d]: projections | f32 tail (gates or step sizes) | up
    float* b_in = nullptr;       // [n_in]
    void* w_out = nullptr;       // [d, k_out]: W_o | 0 | W_down | 0
    float* conv_w = nullptr;     // [channels, taps]
    float* conv_b = nullptr;     // mamba2
    float *q_norm = nullptr, *k_norm = nullptr;                                   // attention
    float *dt_bias = nullptr, *a_log = nullptr, *d_skip = nullptr, *norm_w = nullptr;   // mamba2 (norm_w also hgrn2)
    float *head_bias = nullptr, *f_bias = nullptr, *lower = nullptr;              // sigmoid attention, hgrn2
    float *r_bias = nullptr, *i_bias = nullptr, *lambda = nullptr;                // rglru
    void* gate_w = nullptr;      // rglru: [blocks, 2 part, part]
    // sequential blocks
    float *scale1 = nullptr, *norm2 = nullptr, *scale2 = nullptr;
    void *w_up = nullptr, *w_down = nullptr;     // [k_ff, d], [d, k_ff]; experts: [experts, ff, d], [experts, d, ff]
    float* act = nullptr;        // polynorm
    void* router = nullptr;      // [experts + identity, d]
    float* correction = nullptr;
};

struct StackLayer {
    tnsr_b200_layer cfg;
    uint32_t owner = 0;          // layer whose tensors it uses
    uint32_t channels = 0;       // convolved channels
    uint32_t proj = 0;           // projection channels (mamba2: z before the convolved ones)
    uint32_t proj_cols = 0, tail_cols = 0, up_cols = 0, mixer_cols = 0;   // column ranges, padded
    uint32_t mixer_width = 0;    // columns the mixer writes
    uint32_t n_in = 0, k_out = 0;
    uint32_t rec_q_col = 0, rec_v_col = 0, rec_col = 0;   // hgrn2: its q and v among the projections, its output
    uint32_t x_col = 0;          // rglru: x behind y
    uint32_t k_ff = 0;           // sequential dense feed-forward: K of its second product
    const float2* rotation = nullptr;
    void *k_cache = nullptr, *v_cache = nullptr, *ring = nullptr;
    float* ssm = nullptr;
    uint64_t k_elems = 0, v_elems = 0, ring_elems = 0, ssm_elems = 0;
};

// Where the values of one parameter go: rows [row0, row0 + rows) of the stored matrix into a packed operand (`dst` with
// pitch ld at (dst_row, dst_col)), or, with ld == 0, a plain f32 copy.
struct StackPiece {
    void* dst = nullptr;
    uint32_t row0 = 0, rows = 0, dst_row = 0, dst_col = 0, ld = 0;
};
struct StackParam {
    uint32_t rows = 0, cols = 0;
    std::vector<StackPiece> pieces;
    uint64_t elems() const { return (uint64_t)rows * cols; }
};

struct RotationTable {
    tnsr_b200_layer key;
    float2* table;
};

struct StackCache {
    void* ptr;
    uint64_t elems;
    int dtype;
};

struct LayerStack {
    float embedding_scale = 1.0f, norm_offset = 0.0f;
    std::vector<tnsr_b200_layer> desc;
    std::vector<StackLayer> layers;
    std::vector<StackWeights> weights;   // by owner
    std::vector<StackParam> params;
    std::vector<RotationTable> rotations;
    std::vector<StackCache> caches;
    void *embed = nullptr, *head = nullptr;
    float* final_norm = nullptr;
    // activations
    void* proj = nullptr;     // [rows, proj_cols]
    float* tail = nullptr;    // [rows, tail_cols]
    void* cat = nullptr;      // [rows, k_out]: mixer output | activated up
    void* q = nullptr;        // [rows, heads * dim]
    void* xbc = nullptr;      // [rows, channels] of mamba2 layers
    void* gated = nullptr;    // [rows, inner]
    void* attention_ws = nullptr;
    uint64_t attention_ws_bytes = 0;
    float* raw = nullptr;     // [rows, rec_heads * rec_vdim] of hgrn2 with wide heads
    void* u = nullptr;        // [rows, width] of rglru
    float* gates = nullptr;   // [rows, 2 width]
    void* ff_z = nullptr;     // [rows, ff]: up before polynorm
    void* ff_act = nullptr;   // [rows, k_ff]
    float* router = nullptr;  // [rows, experts + identity]
    void* experts_ws = nullptr;
    uint64_t experts_ws_bytes = 0;
};

namespace {

uint32_t round_up(uint32_t x, uint32_t to) { return (x + to - 1) / to * to; }

bool same_rotation(const tnsr_b200_layer& a, const tnsr_b200_layer& b) {
    return a.rotary_dims == b.rotary_dims && a.rotary_base == b.rotary_base && a.rotary_factor == b.rotary_factor &&
           a.rotary_low == b.rotary_low && a.rotary_high == b.rotary_high && a.rotary_original == b.rotary_original;
}

// Angular frequencies of the rotated pairs.  With a scaling factor, slow pairs (wavelength above original / low) turn
// `factor` times slower, fast ones (below original / high) keep their frequency, and those between are blended.
std::vector<double> rotary_frequencies(const tnsr_b200_layer& l) {
    std::vector<double> f(l.rotary_dims / 2);
    const double two_pi = 6.283185307179586476925286766559;
    for (uint32_t i = 0; i < f.size(); ++i) {
        f[i] = std::pow(l.rotary_base, -2.0 * i / l.rotary_dims);
        if (l.rotary_factor <= 0.0) continue;
        const double wavelength = two_pi / f[i];
        if (wavelength < l.rotary_original / l.rotary_high) continue;
        if (wavelength > l.rotary_original / l.rotary_low) {
            f[i] /= l.rotary_factor;
        } else {
            const double s = (l.rotary_original / wavelength - l.rotary_low) / (l.rotary_high - l.rotary_low);
            f[i] = (1.0 - s) * f[i] / l.rotary_factor + s * f[i];
        }
    }
    return f;
}

// table[p][i] = (cos, sin)(p * frequency_i); the angle is formed and reduced in f64, so that its error does not grow
// with the position.
__global__ void rotation_table_kernel(const double* __restrict__ freq, float2* __restrict__ table, uint32_t positions, uint32_t pairs) {
    const uint64_t total = (uint64_t)positions * pairs;
    for (uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (uint64_t)gridDim.x * blockDim.x) {
        double s, c;
        sincos((double)(i / pairs) * freq[i % pairs], &s, &c);
        table[i] = make_float2((float)c, (float)s);
    }
}

int make_rotation(tnsr_b200_decoder* dec, const tnsr_b200_layer& l, const float2** out) {
    *out = nullptr;
    const uint32_t pairs = l.rotary_dims / 2;
    if (pairs == 0) return TNSR_B200_OK;
    for (const RotationTable& r : dec->stack->rotations)
        if (same_rotation(r.key, l)) { *out = r.table; return TNSR_B200_OK; }
    const std::vector<double> f = rotary_frequencies(l);
    double* d_freq = nullptr;
    float2* table = nullptr;
    int rc;
    if ((rc = dev_alloc(dec, (void**)&d_freq, pairs * sizeof(double), false))) return rc;
    if ((rc = dev_alloc(dec, (void**)&table, (size_t)dec->cfg.capacity * pairs * sizeof(float2), false))) return rc;
    CU(dec, cudaMemcpyAsync(d_freq, f.data(), pairs * sizeof(double), cudaMemcpyHostToDevice, dec->stream));
    rotation_table_kernel<<<(unsigned)std::min<uint64_t>(ceil_div64((uint64_t)dec->cfg.capacity * pairs, 256), 148 * 16), 256, 0,
                            dec->stream>>>(d_freq, table, dec->cfg.capacity, pairs);
    count_launch();
    RUN(dec, check_launch("rotation_table"));
    CU(dec, cudaStreamSynchronize(dec->stream));
    dev_free(dec, d_freq);
    dec->stack->rotations.push_back({l, table});
    *out = table;
    return TNSR_B200_OK;
}

uint32_t owner_of(const std::vector<tnsr_b200_layer>& desc, uint32_t i) {
    for (size_t hops = 0; desc[i].weights_of >= 0 && hops < desc.size(); ++hops) i = (uint32_t)desc[i].weights_of;
    return i;
}

bool attends(const tnsr_b200_layer& l) { return l.mixer == TNSR_B200_MIXER_ATTENTION || l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2; }
bool sequential(const tnsr_b200_layer& l) { return l.block_form == TNSR_B200_BLOCK_SEQUENTIAL; }
bool convolves(const tnsr_b200_layer& l) { return l.mixer != TNSR_B200_MIXER_ATTENTION_HGRN2; }

// Derived sizes of a layer.  Ranges of the first product start at multiples of 32 columns; what is inside one range starts
// at multiples of 8, so that 16-byte accesses stay possible.
void lay_out(StackLayer& L) {
    const tnsr_b200_layer& c = L.cfg;
    L.mixer_width = c.heads * c.vdim;
    L.tail_cols = round_up(c.heads, 32);
    switch (c.mixer) {
        case TNSR_B200_MIXER_ATTENTION:
            L.proj = L.channels = c.heads * c.dim + c.kv_heads * (c.dim + c.vdim);
            break;
        case TNSR_B200_MIXER_MAMBA2:
            L.channels = L.mixer_width + 2 * c.groups * c.state;
            L.proj = L.mixer_width + L.channels;
            break;
        case TNSR_B200_MIXER_ATTENTION_HGRN2:
            L.rec_q_col = round_up(c.heads * c.dim + c.kv_heads * (c.dim + c.vdim), 8);
            L.rec_v_col = round_up(L.rec_q_col + c.rec_heads * c.rec_dim, 8);
            L.proj = L.rec_v_col + c.rec_heads * c.rec_vdim;
            L.tail_cols = round_up(c.rec_heads * c.rec_dim, 32);
            L.rec_col = round_up(L.mixer_width, 8);
            L.mixer_width = L.rec_col + c.rec_heads * c.rec_vdim;
            break;
        default:
            L.x_col = round_up(c.width, 32);
            L.channels = c.width;
            L.proj = 2 * L.x_col;
            L.tail_cols = 0;
            L.mixer_width = c.width;
    }
    L.proj_cols = round_up(L.proj, 32);
    // the second product's K: a multiple of 64 (its k-blocks), the activated up starting at a 32-column boundary
    const bool with_up = !sequential(c) && c.feed_forward;
    L.mixer_cols = round_up(L.mixer_width, with_up ? 32 : 64);
    L.k_out = round_up(L.mixer_cols + (with_up ? c.feed_forward : 0), 64);
    L.up_cols = L.k_out - L.mixer_cols;
    L.n_in = L.proj_cols + L.tail_cols + L.up_cols;
    L.k_ff = round_up(c.feed_forward, 64);
}

}  // namespace

int stack_check(const tnsr_b200_config* c, const tnsr_b200_stack* st, std::string& why) {
    auto bad = [&](const char* m) { why = m; return TNSR_B200_ERR_INVALID_ARGUMENT; };
    if (!c || !st || !st->layers) return bad("null configuration");
    if (c->vocab_size == 0 || c->embed_dim == 0 || st->num_layers == 0 || c->num_layers != st->num_layers ||
        !(c->layer_norm_epsilon > 0.0f) || !std::isfinite(c->layer_norm_epsilon))
        return bad("invalid model configuration");
    if (c->weight_dtype > TNSR_B200_BF16 || c->kv_dtype != c->weight_dtype) return bad("a described model keeps its caches in the weights' type");
    if (c->logits_mode > TNSR_B200_LOGITS_NONE || c->prefill_mode > TNSR_B200_PREFILL_SCALAR) return bad("invalid enum value in configuration");
    if (c->batch == 0) return bad("decoder batch size must be non-zero");
    if (c->capacity == 0 || c->capacity > c->max_sequence_length) return bad("decoder capacity must fit the model context");
    if (c->kv_page_rows) {
        if (c->kv_page_rows % 16 != 0 || c->capacity % c->kv_page_rows != 0)
            return bad("paged K/V needs a page size that is a multiple of 16 rows and divides the capacity");
    } else if (c->kv_pool_pages) {
        return bad("kv_pool_pages without kv_page_rows");
    }
    if ((uint64_t)c->batch * c->capacity > 0xffffffffull) return bad("decoder cache size overflow");
    for (uint32_t i = 0; i < st->num_layers; ++i) {
        const tnsr_b200_layer& l = st->layers[i];
        if (l.mixer > TNSR_B200_MIXER_RGLRU) return bad("unknown mixer");
        if (convolves(l) && (l.conv_taps == 0 || l.conv_taps > kMaxConvTaps)) return bad("layer: 1..16 convolution taps are needed");
        if (l.mixer != TNSR_B200_MIXER_RGLRU && (l.heads == 0 || l.vdim == 0)) return bad("layer: heads and vdim are needed");
        if (attends(l)) {
            if (l.kv_heads == 0 || l.heads % l.kv_heads || l.dim == 0 || l.dim > 256 || l.vdim > 256 || l.rotary_dims > l.dim || l.rotary_dims % 2)
                return bad("attention layer: kv_heads must divide heads, widths are at most 256, rotated dimensions even");
            if (!(l.rotary_dims == 0 || l.rotary_base > 0.0) || !std::isfinite(l.score_scale) || l.score_softcap < 0.0) return bad("attention layer: invalid constants");
            if (l.rotary_factor > 0.0 && !(l.rotary_high > l.rotary_low && l.rotary_low > 0.0)) return bad("attention layer: invalid rotary scaling");
            if (l.rotary_layout > TNSR_B200_ROTARY_HALVES || l.score_kind > TNSR_B200_SCORE_SIGMOID) return bad("attention layer: unknown rotary layout or score kind");
            if (l.mixer == TNSR_B200_MIXER_ATTENTION && (l.rotary_layout || l.window || l.score_kind))
                return bad("attention layer: windows, sigmoid scores and the rotation of halves belong to attention beside a recurrence");
        }
        if (l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2 &&
            (l.rec_vdim > 0xffffu || !hgrn2_supported(l.rec_heads, l.rec_dim, l.rec_vdim) || !std::isfinite(l.attention_gain) || !std::isfinite(l.recurrent_gain)))
            return bad("hgrn2 half: heads and widths are needed, the state has at most 256 rows");
        if (l.mixer == TNSR_B200_MIXER_MAMBA2) {
            if (l.state == 0 || l.groups == 0 || l.heads % l.groups || l.norm_groups == 0 || (l.heads * l.vdim) % l.norm_groups)
                return bad("mamba2 layer: groups must divide heads and norm_groups their total width");
            if (!mamba2_supported(l.heads, l.vdim, l.state)) return bad("mamba2 layer: the state has at most 256 rows");
        }
        if (l.mixer == TNSR_B200_MIXER_RGLRU && (l.width == 0 || l.blocks == 0 || l.width % l.blocks || l.blocks > 1024)) return bad("rglru layer: blocks (at most 1024) must divide the width");
        if (l.block_form > TNSR_B200_BLOCK_SEQUENTIAL || l.feed_forward_kind > TNSR_B200_FF_EXPERTS) return bad("unknown block form or feed-forward");
        if (!sequential(l) && l.feed_forward_kind != TNSR_B200_FF_GELU_TANH) return bad("parallel blocks have the gelu feed-forward");
        if (l.feed_forward && l.feed_forward_kind == TNSR_B200_FF_EXPERTS &&
            (l.experts == 0 || (uint64_t)l.experts + l.identity_experts > kMaxExperts || l.top == 0 || l.top > kMaxTop || l.top > l.experts + l.identity_experts ||
             !std::isfinite(l.router_scale)))
            return bad("experts: 1..1024 of them, at most 32 chosen");
        if (l.weights_of >= 0) {
            if ((uint32_t)l.weights_of >= st->num_layers || (uint32_t)l.weights_of == i) return bad("weights_of names no other layer");
            // follow the chain: it must end at a layer with tensors, and sizes must agree
            uint32_t j = i, hops = 0;
            while (st->layers[j].weights_of >= 0 && hops++ <= st->num_layers) {
                j = (uint32_t)st->layers[j].weights_of;
                if (j >= st->num_layers) return bad("weights_of names no other layer");
            }
            if (st->layers[j].weights_of >= 0) return bad("weights_of forms a loop");
            const tnsr_b200_layer& o = st->layers[j];
            if (o.mixer != l.mixer || o.heads != l.heads || o.vdim != l.vdim || o.conv_taps != l.conv_taps || o.feed_forward != l.feed_forward ||
                o.block_form != l.block_form || o.feed_forward_kind != l.feed_forward_kind || o.experts != l.experts || o.identity_experts != l.identity_experts ||
                (attends(l) && (o.kv_heads != l.kv_heads || o.dim != l.dim || o.score_kind != l.score_kind)) ||
                (l.mixer == TNSR_B200_MIXER_MAMBA2 && (o.state != l.state || o.groups != l.groups)) ||
                (l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2 && (o.rec_heads != l.rec_heads || o.rec_dim != l.rec_dim || o.rec_vdim != l.rec_vdim)) ||
                (l.mixer == TNSR_B200_MIXER_RGLRU && (o.width != l.width || o.blocks != l.blocks)))
                return bad("weights_of: the two layers have different sizes");
        }
    }
    return TNSR_B200_OK;
}

int stack_create(tnsr_b200_decoder* dec, const tnsr_b200_stack* st) {
    LayerStack* S = new (std::nothrow) LayerStack();
    if (!S) return fail(dec, TNSR_B200_ERR_OUT_OF_MEMORY, "host allocation failed");
    dec->stack = S;
    const tnsr_b200_config& c = dec->cfg;
    const uint64_t d = c.embed_dim;
    const size_t e = elt(dec);
    const int dtype = dec->bf16_path ? TNSR_B200_BF16 : TNSR_B200_F32;
    S->embedding_scale = (float)st->embedding_scale;
    S->norm_offset = (float)st->norm_offset;
    S->desc.assign(st->layers, st->layers + st->num_layers);
    S->layers.resize(st->num_layers);
    S->weights.resize(st->num_layers);
    int rc;
    auto matrix = [&](uint32_t rows, uint32_t cols, std::vector<StackPiece> pieces) {
        StackParam p;
        p.rows = rows; p.cols = cols; p.pieces = std::move(pieces);
        S->params.push_back(std::move(p));
    };
    auto vector_param = [&](uint32_t rows, uint32_t cols, float* dst) { matrix(rows, cols, {StackPiece{dst, 0, rows, 0, 0, 0}}); };
    if ((rc = dev_alloc(dec, &S->embed, (size_t)c.vocab_size * d * e, true))) return rc;
    if ((rc = dev_alloc(dec, &S->head, (size_t)c.vocab_size * d * e, true))) return rc;
    if ((rc = dev_alloc(dec, (void**)&S->final_norm, d * 4, true))) return rc;
    matrix(c.vocab_size, (uint32_t)d, {StackPiece{S->embed, 0, c.vocab_size, 0, 0, (uint32_t)d}});
    matrix(c.vocab_size, (uint32_t)d, {StackPiece{S->head, 0, c.vocab_size, 0, 0, (uint32_t)d}});
    vector_param(1, (uint32_t)d, S->final_norm);
    for (uint32_t i = 0; i < st->num_layers; ++i) {
        StackLayer& L = S->layers[i];
        L.cfg = st->layers[i];
        L.owner = owner_of(S->desc, i);
        lay_out(L);
        const tnsr_b200_layer& l = L.cfg;
        if (L.owner == i) {
            StackWeights& W = S->weights[i];
            const uint32_t D = (uint32_t)d, inner = l.heads * l.vdim;
            auto floats = [&](float** p, size_t n) { return dev_alloc(dec, (void**)p, n * 4, true); };
            if ((rc = floats(&W.norm, d))) return rc;
            if ((rc = dev_alloc(dec, &W.w_in, (size_t)L.n_in * d * e, true))) return rc;
            if ((rc = floats(&W.b_in, L.n_in))) return rc;
            if ((rc = dev_alloc(dec, &W.w_out, (size_t)d * L.k_out * e, true))) return rc;
            if (convolves(l))
                if ((rc = floats(&W.conv_w, (size_t)L.channels * l.conv_taps))) return rc;
            vector_param(1, D, W.norm);
            auto rows_of_w_in = [&](uint32_t rows, uint32_t at) { matrix(rows, D, {StackPiece{W.w_in, 0, rows, at, 0, D}}); };
            auto cols_of_w_out = [&](uint32_t cols, uint32_t at) { matrix(D, cols, {StackPiece{W.w_out, 0, D, 0, at, L.k_out}}); };
            const uint32_t nq = l.heads * l.dim, nk = l.kv_heads * l.dim, nv = l.kv_heads * l.vdim;
            if (l.mixer == TNSR_B200_MIXER_ATTENTION) {
                if ((rc = floats(&W.q_norm, l.dim))) return rc;
                if ((rc = floats(&W.k_norm, l.dim))) return rc;
                rows_of_w_in(nq, 0);
                vector_param(1, nq, W.b_in);
                rows_of_w_in(nk, nq);
                vector_param(1, nk, W.b_in + nq);
                rows_of_w_in(nv, nq + nk);
                vector_param(1, nv, W.b_in + nq + nk);
                vector_param(1, l.dim, W.q_norm);
                vector_param(1, l.dim, W.k_norm);
                vector_param(nq, l.conv_taps, W.conv_w);
                vector_param(nk, l.conv_taps, W.conv_w + (size_t)nq * l.conv_taps);
                vector_param(nv, l.conv_taps, W.conv_w + (size_t)(nq + nk) * l.conv_taps);
                rows_of_w_in(l.heads, L.proj_cols);
                cols_of_w_out(inner, 0);
            } else if (l.mixer == TNSR_B200_MIXER_MAMBA2) {
                if ((rc = floats(&W.conv_b, L.channels))) return rc;
                if ((rc = floats(&W.dt_bias, l.heads))) return rc;
                if ((rc = floats(&W.a_log, l.heads))) return rc;
                if ((rc = floats(&W.d_skip, l.heads))) return rc;
                if ((rc = floats(&W.norm_w, inner))) return rc;
                matrix(L.proj + l.heads, D, {StackPiece{W.w_in, 0, L.proj, 0, 0, D}, StackPiece{W.w_in, L.proj, l.heads, L.proj_cols, 0, D}});
                vector_param(L.channels, l.conv_taps, W.conv_w);
                vector_param(1, L.channels, W.conv_b);
                vector_param(1, l.heads, W.dt_bias);
                vector_param(1, l.heads, W.a_log);
                vector_param(1, l.heads, W.d_skip);
                vector_param(1, inner, W.norm_w);
                cols_of_w_out(inner, 0);
            } else if (l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2) {
                const uint32_t rk = l.rec_heads * l.rec_dim, rv = l.rec_heads * l.rec_vdim;
                if ((rc = floats(&W.f_bias, rk))) return rc;
                if ((rc = floats(&W.lower, rk))) return rc;
                if ((rc = floats(&W.norm_w, l.rec_vdim))) return rc;
                rows_of_w_in(nq, 0);
                rows_of_w_in(nk, nq);
                rows_of_w_in(nv, nq + nk);
                if (l.score_kind == TNSR_B200_SCORE_SIGMOID) {
                    if ((rc = floats(&W.head_bias, l.heads))) return rc;
                    vector_param(1, l.heads, W.head_bias);
                }
                cols_of_w_out(inner, 0);
                rows_of_w_in(rk, L.rec_q_col);
                rows_of_w_in(rk, L.proj_cols);
                vector_param(1, rk, W.f_bias);
                vector_param(1, rk, W.lower);
                rows_of_w_in(rv, L.rec_v_col);
                vector_param(1, l.rec_vdim, W.norm_w);
                cols_of_w_out(rv, L.rec_col);
            } else {
                const uint32_t part = l.width / l.blocks;
                if ((rc = floats(&W.conv_b, l.width))) return rc;
                if ((rc = floats(&W.r_bias, l.width))) return rc;
                if ((rc = floats(&W.i_bias, l.width))) return rc;
                if ((rc = floats(&W.lambda, l.width))) return rc;
                if ((rc = dev_alloc(dec, &W.gate_w, (size_t)2 * l.width * part * e, true))) return rc;
                rows_of_w_in(l.width, 0);
                vector_param(1, l.width, W.b_in);
                rows_of_w_in(l.width, L.x_col);
                vector_param(1, l.width, W.b_in + L.x_col);
                vector_param(l.width, l.conv_taps, W.conv_w);
                vector_param(1, l.width, W.conv_b);
                for (uint32_t which = 0; which < 2; ++which) {     // r, then i: [blocks, part, part] into every block's half
                    std::vector<StackPiece> pieces;
                    for (uint32_t b = 0; b < l.blocks; ++b) pieces.push_back(StackPiece{W.gate_w, b * part, part, (2 * b + which) * part, 0, part});
                    matrix(l.width, part, pieces);
                    vector_param(1, l.width, which ? W.i_bias : W.r_bias);
                }
                vector_param(1, l.width, W.lambda);
                cols_of_w_out(l.width, 0);
            }
            const uint32_t ff = l.feed_forward;
            if (!sequential(l)) {
                if (ff) {
                    rows_of_w_in(ff, L.proj_cols + L.tail_cols);
                    cols_of_w_out(ff, L.mixer_cols);
                }
            } else {
                if ((rc = floats(&W.scale1, d))) return rc;
                vector_param(1, D, W.scale1);
            }
            if (sequential(l) && ff) {
                if ((rc = floats(&W.norm2, d))) return rc;
                if ((rc = floats(&W.scale2, d))) return rc;
                vector_param(1, D, W.norm2);
                if (l.feed_forward_kind == TNSR_B200_FF_EXPERTS) {
                    const uint32_t total = l.experts + l.identity_experts;
                    if ((rc = dev_alloc(dec, &W.w_up, (size_t)l.experts * ff * d * e, true))) return rc;
                    if ((rc = dev_alloc(dec, &W.w_down, (size_t)l.experts * ff * d * e, true))) return rc;
                    if ((rc = dev_alloc(dec, &W.router, (size_t)round_up(total, 32) * d * e, true))) return rc;     // whole column blocks
                    if ((rc = floats(&W.correction, total))) return rc;
                    for (uint32_t x = 0; x < l.experts; ++x) {
                        matrix(ff, D, {StackPiece{W.w_up, 0, ff, x * ff, 0, D}});
                        matrix(D, ff, {StackPiece{W.w_down, 0, D, x * D, 0, ff}});
                    }
                    matrix(total, D, {StackPiece{W.router, 0, total, 0, 0, D}});
                    vector_param(1, total, W.correction);
                } else {
                    if ((rc = dev_alloc(dec, &W.w_up, (size_t)L.k_ff * d * e, true))) return rc;
                    if ((rc = dev_alloc(dec, &W.w_down, (size_t)L.k_ff * d * e, true))) return rc;
                    matrix(ff, D, {StackPiece{W.w_up, 0, ff, 0, 0, D}});
                    matrix(D, ff, {StackPiece{W.w_down, 0, D, 0, 0, L.k_ff}});
                    if (l.feed_forward_kind == TNSR_B200_FF_POLYNORM) {
                        if ((rc = floats(&W.act, 4))) return rc;
                        vector_param(1, 4, W.act);
                    }
                }
                vector_param(1, D, W.scale2);
            }
        }
        // a cache or state of its own, also for a layer that shares its tensors
        if (attends(l)) {
            const uint64_t rows = dec->paged ? (uint64_t)dec->pool_pages * dec->page_rows : (uint64_t)c.batch * c.capacity;
            L.k_elems = rows * l.kv_heads * l.dim;
            L.v_elems = rows * l.kv_heads * l.vdim;
            if ((rc = dev_alloc(dec, &L.k_cache, L.k_elems * e, true))) return rc;
            if ((rc = dev_alloc(dec, &L.v_cache, L.v_elems * e, true))) return rc;
            if ((rc = make_rotation(dec, l, &L.rotation))) return rc;
            S->caches.push_back({L.k_cache, L.k_elems, dtype});
            S->caches.push_back({L.v_cache, L.v_elems, dtype});
            S->attention_ws_bytes = std::max(S->attention_ws_bytes, grouped_attention_workspace_bytes(l.dim, l.vdim));
        }
        if (convolves(l)) {
            L.ring_elems = (uint64_t)c.batch * l.conv_taps * L.channels;
            if ((rc = dev_alloc(dec, &L.ring, L.ring_elems * e, true))) return rc;
            S->caches.push_back({L.ring, L.ring_elems, dtype});
        }
        L.ssm_elems = l.mixer == TNSR_B200_MIXER_MAMBA2 ? (uint64_t)c.batch * l.heads * l.state * l.vdim
                    : l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2 ? (uint64_t)c.batch * l.rec_heads * l.rec_dim * l.rec_vdim
                    : l.mixer == TNSR_B200_MIXER_RGLRU ? (uint64_t)c.batch * l.width : 0;
        if (L.ssm_elems) {
            if ((rc = dev_alloc(dec, (void**)&L.ssm, L.ssm_elems * 4, true))) return rc;
            S->caches.push_back({L.ssm, L.ssm_elems, TNSR_B200_F32});
        }
    }
    if (S->attention_ws_bytes)
        if ((rc = dev_alloc(dec, &S->attention_ws, S->attention_ws_bytes, true))) return rc;
    // single-token steps of few rows divide K of a layer's second product; the next norm adds the partial sums
    if (dec->bf16_path && c.batch <= 256 && layernorm_fold_supported(c.embed_dim)) {
        dec->split_rows = (c.batch + 31) / 32 * 32 + 32;
        if ((rc = dev_alloc(dec, (void**)&dec->split_ws, (size_t)4 * dec->split_rows * d * sizeof(float), true))) return rc;
    }
    return TNSR_B200_OK;
}

void stack_destroy(tnsr_b200_decoder* dec) {
    delete dec->stack;   // device memory is on the handle's list
    dec->stack = nullptr;
}

uint32_t stack_param_count(const tnsr_b200_decoder* dec) { return (uint32_t)dec->stack->params.size(); }
uint64_t stack_param_elems(const tnsr_b200_decoder* dec, uint32_t index) {
    return index < dec->stack->params.size() ? dec->stack->params[index].elems() : 0;
}

int stack_upload(tnsr_b200_decoder* dec, uint32_t index, const float* host) {
    const StackParam& p = dec->stack->params[index];
    const size_t bytes = p.elems() * 4;
    cudaStream_t st = dec->stream;
    if (p.pieces.size() == 1 && p.pieces[0].ld == 0) {
        CU(dec, cudaMemcpyAsync(p.pieces[0].dst, host, bytes, cudaMemcpyHostToDevice, st));
        CU(dec, cudaStreamSynchronize(st));   // `host` is pageable and not retained
        return TNSR_B200_OK;
    }
    if (bytes > dec->d_stage_bytes) {
        CU(dec, cudaStreamSynchronize(st));
        dev_free(dec, dec->d_stage);
        dec->d_stage = nullptr;
        dec->d_stage_bytes = 0;
        int rc = dev_alloc(dec, (void**)&dec->d_stage, bytes, false);
        if (rc) return rc;
        dec->d_stage_bytes = bytes;
    }
    CU(dec, cudaMemcpyAsync(dec->d_stage, host, bytes, cudaMemcpyHostToDevice, st));
    for (const StackPiece& q : p.pieces)
        RUN(dec, launch_pack_rows(dec->d_stage + (size_t)q.row0 * p.cols, q.dst, dec->bf16_path ? TNSR_B200_BF16 : TNSR_B200_F32,
                                  q.rows, p.cols, q.dst_row, q.dst_col, q.ld, st));
    CU(dec, cudaStreamSynchronize(st));
    return TNSR_B200_OK;
}

int stack_reset(tnsr_b200_decoder* dec) {
    for (const StackCache& t : dec->stack->caches)
        CU(dec, cudaMemsetAsync(t.ptr, 0, t.elems * (t.dtype == TNSR_B200_BF16 ? 2 : 4), dec->stream));
    if (dec->stack->attention_ws) CU(dec, cudaMemsetAsync(dec->stack->attention_ws, 0, dec->stack->attention_ws_bytes, dec->stream));
    return TNSR_B200_OK;
}

uint32_t stack_cache_count(const tnsr_b200_decoder* dec) { return (uint32_t)dec->stack->caches.size(); }
bool stack_cache(const tnsr_b200_decoder* dec, uint32_t index, void** ptr, uint64_t* elems, int* dtype) {
    if (index >= dec->stack->caches.size()) return false;
    const StackCache& t = dec->stack->caches[index];
    *ptr = t.ptr; *elems = t.elems; *dtype = t.dtype;
    return true;
}

int stack_alloc_rows(tnsr_b200_decoder* dec, uint32_t rows) {
    LayerStack* S = dec->stack;
    const size_t e = elt(dec);
    uint64_t proj = 0, tail = 0, cat = 0, q = 0, xbc = 0, gated = 0, raw = 0, u = 0, ff_z = 0, ff_act = 0, router = 0, experts = 0;
    for (const StackLayer& L : S->layers) {
        const tnsr_b200_layer& l = L.cfg;
        proj = std::max<uint64_t>(proj, L.proj_cols);
        tail = std::max<uint64_t>(tail, L.tail_cols);
        cat = std::max<uint64_t>(cat, L.k_out);
        if (attends(l)) q = std::max<uint64_t>(q, (uint64_t)l.heads * l.dim);
        if (l.mixer == TNSR_B200_MIXER_MAMBA2) {
            xbc = std::max<uint64_t>(xbc, L.channels);
            gated = std::max<uint64_t>(gated, L.mixer_width);
        }
        if (l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2 && l.rec_vdim > HGRN2_FUSED_VDIM) raw = std::max<uint64_t>(raw, (uint64_t)l.rec_heads * l.rec_vdim);
        if (l.mixer == TNSR_B200_MIXER_RGLRU) u = std::max<uint64_t>(u, l.width);
        if (!sequential(l) || !l.feed_forward) continue;
        if (l.feed_forward_kind == TNSR_B200_FF_EXPERTS) {
            router = std::max<uint64_t>(router, round_up(l.experts + l.identity_experts, 32));
            experts = std::max(experts, experts_workspace_bytes(rows, dec->cfg.embed_dim, l.feed_forward, l.experts, l.top, dec->bf16_path ? TNSR_B200_BF16 : TNSR_B200_F32));
        } else {
            ff_z = std::max<uint64_t>(ff_z, l.feed_forward);
            ff_act = std::max<uint64_t>(ff_act, L.k_ff);
        }
    }
    S->experts_ws_bytes = experts;
    struct { void** p; uint64_t bytes; } want[] = {{&S->proj, proj * e * rows}, {(void**)&S->tail, tail * 4 * rows}, {&S->cat, cat * e * rows},
                                                   {&S->q, q * e * rows}, {&S->xbc, xbc * e * rows}, {&S->gated, gated * e * rows},
                                                   {(void**)&S->raw, raw * 4 * rows}, {&S->u, u * e * rows}, {(void**)&S->gates, 2 * u * 4 * rows},
                                                   {&S->ff_z, ff_z * e * rows}, {&S->ff_act, ff_act * e * rows}, {(void**)&S->router, router * 4 * rows},
                                                   {&S->experts_ws, experts}};
    for (auto& w : want) {
        dev_free(dec, *w.p);
        *w.p = nullptr;
        if (w.bytes == 0) continue;
        int rc = dev_alloc(dec, w.p, w.bytes, false);
        if (rc) return rc;
    }
    return TNSR_B200_OK;
}

int stack_step(tnsr_b200_decoder* dec, const uint32_t* d_tokens, uint32_t chunk, uint32_t position, const uint32_t* d_position,
               bool ragged, uint32_t logit_rows, uint32_t* fused_ids) {
    LayerStack* S = dec->stack;
    const tnsr_b200_config& c = dec->cfg;
    const uint32_t d = c.embed_dim, B = c.batch, rows = B * chunk;
    const float eps = c.layer_norm_epsilon;
    const bool bf = dec->bf16_path;
    const int dtype = bf ? TNSR_B200_BF16 : TNSR_B200_F32;
    const size_t e = elt(dec);
    cudaStream_t st = dec->stream;
    StepPlace place;
    place.sessions = B; place.chunk = chunk; place.position = position; place.d_position = d_position;
    place.position_stride = ragged ? 1u : 0u;
    KvPaging pg;
    if (dec->paged) { pg.table = dec->d_table; pg.page_rows = dec->page_rows; pg.pages_per_session = dec->pps; }
    RUN(dec, launch_embedding(S->embed, nullptr, d_tokens, dec->h, rows, chunk, position, d_position, c.vocab_size, d, dtype,
                              dec->d_status, st, place.position_stride, S->embedding_scale));
    const bool splitk = bf && chunk == 1 && dec->split_ws;
    const bool plain_prefill = chunk > 1 && c.prefill_mode == TNSR_B200_PREFILL_SCALAR;
    // what the next norm has to finish first: partial sums of a split product, or the weighted sum of experts
    uint32_t pending = 0;
    Experts experts;
    bool pending_experts = false;
    auto norm = [&](const float* w) -> int {
        const uint32_t parts = pending;
        pending = 0;
        if (pending_experts) {
            pending_experts = false;
            experts.norm_w = w;
            experts.norm_out = dec->n;
            RUN(dec, launch_experts_combine(experts, dtype, st));
        } else if (parts)
            RUN(dec, launch_rmsnorm_fold(dec->h, dec->split_ws, parts, dec->split_rows, w, S->norm_offset, dec->n, rows, d, eps, st));
        else
            RUN(dec, launch_rmsnorm(dec->h, w, S->norm_offset, dec->n, rows, d, eps, dtype, st));
        return TNSR_B200_OK;
    };
    // residual += scale * (a [rows, k] . w [d, k]^T)
    auto add_product = [&](const void* a, const void* w, uint32_t k, const float* scale) -> int {
        GemmEpilogue eo;
        eo.residual = dec->h; eo.ldr = d; eo.out_dtype = TNSR_B200_F32; eo.scale = scale;
        if (!bf) {
            RUN(dec, launch_gemm_strict((const float*)a, (const float*)w, dec->h, d, rows, k, d, true, eo, st));
            return TNSR_B200_OK;
        }
        const uint32_t split = splitk ? gemm_split_k((const bf16*)a, (const bf16*)w, rows, d, k) : 0;
        if (split) { eo.split_k = split; eo.split_partials = dec->split_ws; eo.split_rows = dec->split_rows; }
        RUN(dec, launch_gemm_bf16((const bf16*)a, (const bf16*)w, dec->h, d, rows, d, k, GEMM_PLAIN, eo, nullptr, dec->d_status, st));
        pending = split;
        return TNSR_B200_OK;
    };
    // out [rows, n] = act(norm rows . w [n, d]^T)
    auto product = [&](const void* w, uint32_t n, void* out, uint32_t ld, int activation, int out_dtype) -> int {
        GemmEpilogue ep;
        ep.activation = activation; ep.out_dtype = out_dtype;
        if (bf && out_dtype == TNSR_B200_BF16 && n % 32 == 0 && rows > 16) {     // one column range: its epilogue is the faster one for a short K
            GemmSegments one;
            one.count = 1;
            one.s[0].out = out; one.s[0].ld = ld; one.s[0].activation = activation;
            RUN(dec, launch_gemm_segments((const bf16*)dec->n, (const bf16*)w, rows, n, d, nullptr, one, dec->d_status, st));
        } else if (bf) RUN(dec, launch_gemm_bf16((const bf16*)dec->n, (const bf16*)w, out, ld, rows, n, d, GEMM_PLAIN, ep, nullptr, dec->d_status, st));
        else RUN(dec, launch_gemm_strict((const float*)dec->n, (const float*)w, out, ld, rows, d, n, true, ep, st));
        return TNSR_B200_OK;
    };
    int rc;
    for (StackLayer& L : S->layers) {
        const StackWeights& W = S->weights[L.owner];
        const tnsr_b200_layer& l = L.cfg;
        if ((rc = norm(W.norm))) return rc;
        // ---- first product: column ranges and where they go ----
        GemmSegments seg;
        auto range = [&](void* out, uint32_t col0, uint32_t ld, int out_dtype, int activation) {
            GemmSegment& g = seg.s[seg.count++];
            g.out = out; g.col0 = col0; g.ld = ld; g.out_dtype = out_dtype; g.activation = activation;
        };
        if (l.mixer == TNSR_B200_MIXER_RGLRU) {
            range(S->proj, 0, L.proj_cols, dtype, ACT_GELU_TANH);
            range((uint8_t*)S->proj + (size_t)L.x_col * e, L.x_col, L.proj_cols, dtype, ACT_NONE);
        } else {
            range(S->proj, 0, L.proj_cols, dtype, ACT_NONE);
            range(S->tail, L.proj_cols, L.tail_cols, TNSR_B200_F32, ACT_NONE);
        }
        if (L.up_cols && !sequential(l)) range((uint8_t*)S->cat + (size_t)L.mixer_cols * e, L.proj_cols + L.tail_cols, L.k_out, dtype, ACT_GELU_TANH);
        if (bf) {
            RUN(dec, launch_gemm_segments((const bf16*)dec->n, (const bf16*)W.w_in, rows, L.n_in, d, W.b_in, seg, dec->d_status, st));
        } else {
            for (uint32_t i = 0; i < seg.count; ++i) {
                const GemmSegment& g = seg.s[i];
                GemmEpilogue ep;
                ep.bias = W.b_in + g.col0; ep.activation = g.activation;
                RUN(dec, launch_gemm_strict((const float*)dec->n, (const float*)W.w_in + (size_t)g.col0 * d, g.out, g.ld, rows, d,
                                            (i + 1 < seg.count ? seg.s[i + 1].col0 : L.n_in) - g.col0, true, ep, st));
            }
        }
        // ---- mixer ----
        if (attends(l)) {
            AttentionPrep p;
            p.proj = S->proj; p.ld = L.proj_cols;
            p.heads = l.heads; p.kv_heads = l.kv_heads; p.dim = l.dim; p.vdim = l.vdim; p.taps = l.conv_taps;
            p.conv_w = W.conv_w; p.q_norm = W.q_norm; p.k_norm = W.k_norm; p.eps = eps;
            p.rotary_dims = l.rotary_dims; p.rotary_layout = l.rotary_layout; p.rotation = L.rotation;
            p.ring = L.ring; p.q = S->q; p.k_cache = L.k_cache; p.v_cache = L.v_cache; p.capacity = c.capacity; p.paging = pg;
            RUN(dec, launch_attention_prep(p, place, dtype, st));
            if (chunk > 1 && convolves(l)) RUN(dec, launch_conv_ring(S->proj, L.proj_cols, L.channels, l.conv_taps, L.ring, place, dtype, st));
            GroupedAttention a;
            a.q = S->q; a.k_cache = L.k_cache; a.v_cache = L.v_cache;
            a.heads = l.heads; a.kv_heads = l.kv_heads; a.dim = l.dim; a.vdim = l.vdim; a.capacity = c.capacity;
            a.scale = (float)l.score_scale; a.softcap = (float)l.score_softcap;
            a.out = S->cat; a.out_ld = L.k_out; a.out_cols = L.mixer_cols;
            if (l.mixer == TNSR_B200_MIXER_ATTENTION) {
                a.gate = S->tail; a.gate_ld = L.tail_cols;
            } else {
                a.window = l.window; a.score_kind = l.score_kind; a.head_bias = W.head_bias; a.gain = (float)l.attention_gain;
                a.out_cols = L.rec_col;
            }
            a.paging = pg;
            a.d_status = dec->d_status;
            a.workspace = S->attention_ws; a.workspace_bytes = S->attention_ws_bytes;
            a.engine = plain_prefill ? 1 : 0;
            RUN(dec, launch_grouped_attention(a, place, dtype, st));
        }
        if (l.mixer == TNSR_B200_MIXER_ATTENTION_HGRN2) {
            Hgrn2 m;
            m.q = (const uint8_t*)S->proj + (size_t)L.rec_q_col * e; m.v = (const uint8_t*)S->proj + (size_t)L.rec_v_col * e; m.ld = L.proj_cols;
            m.f = S->tail; m.f_ld = L.tail_cols; m.heads = l.rec_heads; m.dim = l.rec_dim; m.vdim = l.rec_vdim;
            m.f_bias = W.f_bias; m.lower = W.lower; m.norm_w = W.norm_w; m.eps = eps; m.gain = (float)l.recurrent_gain;
            m.state = L.ssm; m.raw = S->raw;
            m.out = (uint8_t*)S->cat + (size_t)L.rec_col * e; m.out_ld = L.k_out; m.out_cols = L.mixer_cols - L.rec_col;
            m.engine = plain_prefill ? 1 : 0;
            RUN(dec, launch_hgrn2(m, place, dtype, st));
        } else if (l.mixer == TNSR_B200_MIXER_RGLRU) {
            Rglru m;
            m.proj = S->proj; m.ld = L.proj_cols; m.x_col = L.x_col; m.width = l.width; m.blocks = l.blocks; m.taps = l.conv_taps;
            m.conv_w = W.conv_w; m.conv_b = W.conv_b; m.gate_w = W.gate_w; m.r_bias = W.r_bias; m.i_bias = W.i_bias; m.lambda = W.lambda;
            m.ring = L.ring; m.state = L.ssm; m.u = S->u; m.gates = S->gates;
            m.out = S->cat; m.out_ld = L.k_out; m.out_cols = L.mixer_cols; m.d_status = dec->d_status;
            RUN(dec, launch_rglru(m, place, dtype, st));
        } else if (l.mixer == TNSR_B200_MIXER_MAMBA2) {
            Mamba2 m;
            m.proj = S->proj; m.ld = L.proj_cols; m.dt = S->tail; m.dt_ld = L.tail_cols;
            m.heads = l.heads; m.vdim = l.vdim; m.state = l.state; m.groups = l.groups; m.norm_groups = l.norm_groups; m.taps = l.conv_taps;
            m.conv_w = W.conv_w; m.conv_b = W.conv_b; m.dt_bias = W.dt_bias; m.a_log = W.a_log; m.d_skip = W.d_skip; m.norm_w = W.norm_w;
            m.eps = eps; m.ring = L.ring; m.ssm = L.ssm; m.xbc = S->xbc; m.gated = S->gated;
            m.out = S->cat; m.out_ld = L.k_out; m.out_cols = L.mixer_cols;
            m.engine = plain_prefill ? 1 : 0;
            RUN(dec, launch_mamba2(m, place, dtype, st));
        }
        if ((rc = add_product(S->cat, W.w_out, L.k_out, W.scale1))) return rc;
        if (!sequential(l) || !l.feed_forward) continue;
        // ---- feed-forward of a sequential block ----
        if (l.feed_forward_kind != TNSR_B200_FF_EXPERTS)
            if ((rc = norm(W.norm2))) return rc;
        if (l.feed_forward_kind == TNSR_B200_FF_EXPERTS) {
            const uint32_t logit_cols = round_up(l.experts + l.identity_experts, 32);
            experts = Experts();
            experts.logits = S->router; experts.logits_ld = logit_cols; experts.correction = W.correction;
            experts.h = dec->n; experts.up = W.w_up; experts.down = W.w_down; experts.x = dec->h; experts.layer_scale = W.scale2;
            experts.workspace = S->experts_ws; experts.workspace_bytes = S->experts_ws_bytes; experts.d_status = dec->d_status;
            experts.rows = rows; experts.d = d; experts.ff = l.feed_forward; experts.experts = l.experts; experts.identity = l.identity_experts;
            experts.top = l.top; experts.router_scale = (float)l.router_scale; experts.norm_offset = S->norm_offset; experts.eps = eps;
            if (chunk == 1) {       // few rows: norm and router in the choosing kernel
                experts.router = W.router; experts.router_norm = W.norm2;
                experts.partials = dec->split_ws; experts.parts = pending; experts.split_rows = dec->split_rows;
            }
            if (experts_fused_router(experts)) {
                pending = 0;
            } else {
                experts.router = nullptr;
                if ((rc = norm(W.norm2))) return rc;
                if ((rc = product(W.router, logit_cols, S->router, logit_cols, ACT_NONE, TNSR_B200_F32))) return rc;
            }
            RUN(dec, launch_experts(experts, dtype, st));
            pending_experts = true;
        } else {
            if (l.feed_forward_kind == TNSR_B200_FF_POLYNORM) {
                if ((rc = product(W.w_up, l.feed_forward, S->ff_z, l.feed_forward, ACT_NONE, dtype))) return rc;
                RUN(dec, launch_polynorm(S->ff_z, W.act, S->ff_act, rows, l.feed_forward, L.k_ff, L.k_ff, eps, dtype, st));
            } else if ((rc = product(W.w_up, L.k_ff, S->ff_act, L.k_ff, ACT_GELU_TANH, dtype))) {
                return rc;
            }
            if ((rc = add_product(S->ff_act, W.w_down, L.k_ff, W.scale2))) return rc;
        }
    }
    if (logit_rows != rows && pending_experts) {
        pending_experts = false;
        experts.norm_out = nullptr;
        RUN(dec, launch_experts_combine(experts, dtype, st));
    }
    if (logit_rows != rows) {
        RUN(dec, launch_gather_last_rows(dec->h, dec->hl, B, chunk, d, st));
        RUN(dec, launch_rmsnorm(dec->hl, S->final_norm, S->norm_offset, dec->n, logit_rows, d, eps, dtype, st));
    } else if ((rc = norm(S->final_norm))) {
        return rc;
    }
    if (fused_ids) {
        RUN(dec, launch_lm_head_argmax((const bf16*)dec->n, (const bf16*)S->head, logit_rows, c.vocab_size, d, dec->lm_candidates, fused_ids,
                                       dec->d_status, st));
        return TNSR_B200_OK;
    }
    GemmEpilogue el;
    if (bf)
        RUN(dec, launch_gemm_bf16((const bf16*)dec->n, (const bf16*)S->head, dec->logits, c.vocab_size, logit_rows, c.vocab_size, d,
                                  GEMM_PLAIN, el, nullptr, dec->d_status, st));
    else
        RUN(dec, launch_gemm_strict((const float*)dec->n, (const float*)S->head, dec->logits, c.vocab_size, logit_rows, d, c.vocab_size,
                                    true, el, st));
    return TNSR_B200_OK;
}

}  // namespace tb
