// Sessions of models that are described layer by layer (tnsr_b200_decoder_create_stack).  The handle, its stream, token
// staging, page table, sampler, captured steps and entry points are those of decoder.cu; this file holds what such a
// model adds: packed weights, one cache or state per layer, and the step.
//
// Mixer and feed-forward of a layer read the same normalised rows and are added to the residual together, so a layer
// is two products around its mixer whatever the mixer is:
//   norm -> [all projections and the feed-forward's up, one product, column ranges routed by the epilogue]
//        -> mixer -> [mixer output | activated up] . [W_o | W_down]^T added to the residual, one product
#include <algorithm>
#include <cmath>
#include <cstring>

#include "decoder.cuh"
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
    float *dt_bias = nullptr, *a_log = nullptr, *d_skip = nullptr, *norm_w = nullptr;   // mamba2
};

struct StackLayer {
    tnsr_b200_layer cfg;
    uint32_t owner = 0;          // layer whose tensors it uses
    uint32_t channels = 0;       // convolved channels
    uint32_t proj = 0;           // projection channels (mamba2: z before the convolved ones)
    uint32_t proj_cols = 0, tail_cols = 0, up_cols = 0, mixer_cols = 0;   // column ranges, padded
    uint32_t mixer_width = 0;    // heads * vdim
    uint32_t n_in = 0, k_out = 0;
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

// Derived sizes of a layer.
void lay_out(StackLayer& L) {
    const tnsr_b200_layer& c = L.cfg;
    L.mixer_width = c.heads * c.vdim;
    if (c.mixer == TNSR_B200_MIXER_ATTENTION) {
        L.channels = c.heads * c.dim + c.kv_heads * (c.dim + c.vdim);
        L.proj = L.channels;
    } else {
        L.channels = L.mixer_width + 2 * c.groups * c.state;
        L.proj = L.mixer_width + L.channels;
    }
    L.proj_cols = round_up(L.proj, 32);
    L.tail_cols = round_up(c.heads, 32);
    // the second product's K: a multiple of 64 (its k-blocks), the activated up starting at a 32-column boundary
    L.mixer_cols = round_up(L.mixer_width, c.feed_forward ? 32 : 64);
    L.k_out = round_up(L.mixer_cols + c.feed_forward, 64);
    L.up_cols = L.k_out - L.mixer_cols;
    L.n_in = L.proj_cols + L.tail_cols + L.up_cols;
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
        if (l.heads == 0 || l.vdim == 0 || l.conv_taps == 0 || l.conv_taps > kMaxConvTaps) return bad("layer: heads, vdim and 1..16 convolution taps are needed");
        if (l.mixer == TNSR_B200_MIXER_ATTENTION) {
            if (l.kv_heads == 0 || l.heads % l.kv_heads || l.dim == 0 || l.dim > 256 || l.vdim > 256 || l.rotary_dims > l.dim || l.rotary_dims % 2)
                return bad("attention layer: kv_heads must divide heads, widths are at most 256, rotated dimensions even");
            if (!(l.rotary_dims == 0 || l.rotary_base > 0.0) || !std::isfinite(l.score_scale) || l.score_softcap < 0.0) return bad("attention layer: invalid constants");
            if (l.rotary_factor > 0.0 && !(l.rotary_high > l.rotary_low && l.rotary_low > 0.0)) return bad("attention layer: invalid rotary scaling");
        } else if (l.mixer == TNSR_B200_MIXER_MAMBA2) {
            if (l.state == 0 || l.groups == 0 || l.heads % l.groups || l.norm_groups == 0 || (l.heads * l.vdim) % l.norm_groups)
                return bad("mamba2 layer: groups must divide heads and norm_groups their total width");
            if (!mamba2_supported(l.heads, l.vdim, l.state)) return bad("mamba2 layer: the state has at most 256 rows");
        } else {
            return bad("unknown mixer");
        }
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
                (l.mixer == TNSR_B200_MIXER_ATTENTION ? (o.kv_heads != l.kv_heads || o.dim != l.dim) : (o.state != l.state || o.groups != l.groups)))
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
        const bool attention = l.mixer == TNSR_B200_MIXER_ATTENTION;
        if (L.owner == i) {
            StackWeights& W = S->weights[i];
            const uint32_t D = (uint32_t)d;
            if ((rc = dev_alloc(dec, (void**)&W.norm, d * 4, true))) return rc;
            if ((rc = dev_alloc(dec, &W.w_in, (size_t)L.n_in * d * e, true))) return rc;
            if ((rc = dev_alloc(dec, (void**)&W.b_in, (size_t)L.n_in * 4, true))) return rc;
            if ((rc = dev_alloc(dec, &W.w_out, (size_t)d * L.k_out * e, true))) return rc;
            if ((rc = dev_alloc(dec, (void**)&W.conv_w, (size_t)L.channels * l.conv_taps * 4, true))) return rc;
            vector_param(1, D, W.norm);
            auto rows_of_w_in = [&](uint32_t rows, uint32_t at) { matrix(rows, D, {StackPiece{W.w_in, 0, rows, at, 0, D}}); };
            if (attention) {
                const uint32_t nq = l.heads * l.dim, nk = l.kv_heads * l.dim, nv = l.kv_heads * l.vdim;
                if ((rc = dev_alloc(dec, (void**)&W.q_norm, l.dim * 4, true))) return rc;
                if ((rc = dev_alloc(dec, (void**)&W.k_norm, l.dim * 4, true))) return rc;
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
            } else {
                if ((rc = dev_alloc(dec, (void**)&W.conv_b, (size_t)L.channels * 4, true))) return rc;
                if ((rc = dev_alloc(dec, (void**)&W.dt_bias, l.heads * 4, true))) return rc;
                if ((rc = dev_alloc(dec, (void**)&W.a_log, l.heads * 4, true))) return rc;
                if ((rc = dev_alloc(dec, (void**)&W.d_skip, l.heads * 4, true))) return rc;
                if ((rc = dev_alloc(dec, (void**)&W.norm_w, (size_t)L.mixer_width * 4, true))) return rc;
                matrix(L.proj + l.heads, D, {StackPiece{W.w_in, 0, L.proj, 0, 0, D}, StackPiece{W.w_in, L.proj, l.heads, L.proj_cols, 0, D}});
                vector_param(L.channels, l.conv_taps, W.conv_w);
                vector_param(1, L.channels, W.conv_b);
                vector_param(1, l.heads, W.dt_bias);
                vector_param(1, l.heads, W.a_log);
                vector_param(1, l.heads, W.d_skip);
                vector_param(1, L.mixer_width, W.norm_w);
            }
            matrix(D, L.mixer_width, {StackPiece{W.w_out, 0, D, 0, 0, L.k_out}});
            if (l.feed_forward) {
                rows_of_w_in(l.feed_forward, L.proj_cols + L.tail_cols);
                matrix(D, l.feed_forward, {StackPiece{W.w_out, 0, D, 0, L.mixer_cols, L.k_out}});
            }
        }
        // a cache or state of its own, also for a layer that shares its tensors
        L.ring_elems = (uint64_t)c.batch * l.conv_taps * L.channels;
        if ((rc = dev_alloc(dec, &L.ring, L.ring_elems * e, true))) return rc;
        if (attention) {
            const uint64_t rows = dec->paged ? (uint64_t)dec->pool_pages * dec->page_rows : (uint64_t)c.batch * c.capacity;
            L.k_elems = rows * l.kv_heads * l.dim;
            L.v_elems = rows * l.kv_heads * l.vdim;
            if ((rc = dev_alloc(dec, &L.k_cache, L.k_elems * e, true))) return rc;
            if ((rc = dev_alloc(dec, &L.v_cache, L.v_elems * e, true))) return rc;
            if ((rc = make_rotation(dec, l, &L.rotation))) return rc;
            S->caches.push_back({L.k_cache, L.k_elems, dtype});
            S->caches.push_back({L.v_cache, L.v_elems, dtype});
            S->caches.push_back({L.ring, L.ring_elems, dtype});
            S->attention_ws_bytes = std::max(S->attention_ws_bytes, grouped_attention_workspace_bytes(l.dim, l.vdim));
        } else {
            L.ssm_elems = (uint64_t)c.batch * l.heads * l.state * l.vdim;
            if ((rc = dev_alloc(dec, (void**)&L.ssm, L.ssm_elems * 4, true))) return rc;
            S->caches.push_back({L.ring, L.ring_elems, dtype});
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
    uint64_t proj = 0, tail = 0, cat = 0, q = 0, xbc = 0, gated = 0;
    for (const StackLayer& L : S->layers) {
        proj = std::max<uint64_t>(proj, L.proj_cols);
        tail = std::max<uint64_t>(tail, L.tail_cols);
        cat = std::max<uint64_t>(cat, L.k_out);
        if (L.cfg.mixer == TNSR_B200_MIXER_ATTENTION) {
            q = std::max<uint64_t>(q, (uint64_t)L.cfg.heads * L.cfg.dim);
        } else {
            xbc = std::max<uint64_t>(xbc, L.channels);
            gated = std::max<uint64_t>(gated, L.mixer_width);
        }
    }
    struct { void** p; uint64_t bytes; } want[] = {{&S->proj, proj * e}, {(void**)&S->tail, tail * 4}, {&S->cat, cat * e},
                                                   {&S->q, q * e}, {&S->xbc, xbc * e}, {&S->gated, gated * e}};
    for (auto& w : want) {
        dev_free(dec, *w.p);
        *w.p = nullptr;
        if (w.bytes == 0) continue;
        int rc = dev_alloc(dec, w.p, w.bytes * rows, false);
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
    uint32_t pending = 0;   // partial sums of the previous layer's second product
    auto norm = [&](const float* w) -> int {
        const uint32_t parts = pending;
        pending = 0;
        if (parts)
            RUN(dec, launch_rmsnorm_fold(dec->h, dec->split_ws, parts, dec->split_rows, w, S->norm_offset, dec->n, rows, d, eps, st));
        else
            RUN(dec, launch_rmsnorm(dec->h, w, S->norm_offset, dec->n, rows, d, eps, dtype, st));
        return TNSR_B200_OK;
    };
    int rc;
    for (StackLayer& L : S->layers) {
        const StackWeights& W = S->weights[L.owner];
        const tnsr_b200_layer& l = L.cfg;
        if ((rc = norm(W.norm))) return rc;
        uint8_t* up_out = (uint8_t*)S->cat + (size_t)L.mixer_cols * e;
        if (bf) {
            GemmSegments seg;
            seg.s[0].out = S->proj; seg.s[0].ld = L.proj_cols;
            seg.s[1].out = S->tail; seg.s[1].ld = L.tail_cols; seg.s[1].col0 = L.proj_cols; seg.s[1].out_dtype = TNSR_B200_F32;
            seg.s[2].out = up_out; seg.s[2].ld = L.k_out; seg.s[2].col0 = L.proj_cols + L.tail_cols; seg.s[2].activation = ACT_GELU_TANH;
            seg.count = L.up_cols ? 3 : 2;
            RUN(dec, launch_gemm_segments((const bf16*)dec->n, (const bf16*)W.w_in, rows, L.n_in, d, W.b_in, seg, dec->d_status, st));
        } else {
            const float* n = (const float*)dec->n;
            const float* w = (const float*)W.w_in;
            GemmEpilogue ep;
            ep.bias = W.b_in;
            RUN(dec, launch_gemm_strict(n, w, S->proj, L.proj_cols, rows, d, L.proj_cols, true, ep, st));
            ep.bias = nullptr;
            RUN(dec, launch_gemm_strict(n, w + (size_t)L.proj_cols * d, S->tail, L.tail_cols, rows, d, L.tail_cols, true, ep, st));
            ep.activation = ACT_GELU_TANH;
            if (L.up_cols)
                RUN(dec, launch_gemm_strict(n, w + (size_t)(L.proj_cols + L.tail_cols) * d, up_out, L.k_out, rows, d, L.up_cols, true, ep, st));
        }
        if (l.mixer == TNSR_B200_MIXER_ATTENTION) {
            AttentionPrep p;
            p.proj = S->proj; p.ld = L.proj_cols;
            p.heads = l.heads; p.kv_heads = l.kv_heads; p.dim = l.dim; p.vdim = l.vdim; p.taps = l.conv_taps;
            p.conv_w = W.conv_w; p.q_norm = W.q_norm; p.k_norm = W.k_norm; p.eps = eps;
            p.rotary_dims = l.rotary_dims; p.rotation = L.rotation;
            p.ring = L.ring; p.q = S->q; p.k_cache = L.k_cache; p.v_cache = L.v_cache; p.capacity = c.capacity; p.paging = pg;
            RUN(dec, launch_attention_prep(p, place, dtype, st));
            if (chunk > 1) RUN(dec, launch_conv_ring(S->proj, L.proj_cols, L.channels, l.conv_taps, L.ring, place, dtype, st));
            GroupedAttention a;
            a.q = S->q; a.k_cache = L.k_cache; a.v_cache = L.v_cache;
            a.heads = l.heads; a.kv_heads = l.kv_heads; a.dim = l.dim; a.vdim = l.vdim; a.capacity = c.capacity;
            a.scale = (float)l.score_scale; a.softcap = (float)l.score_softcap;
            a.gate = S->tail; a.gate_ld = L.tail_cols;
            a.out = S->cat; a.out_ld = L.k_out; a.out_cols = L.mixer_cols;
            a.paging = pg;
            a.d_status = dec->d_status;
            a.workspace = S->attention_ws; a.workspace_bytes = S->attention_ws_bytes;
            a.engine = chunk > 1 && c.prefill_mode == TNSR_B200_PREFILL_SCALAR ? 1 : 0;
            RUN(dec, launch_grouped_attention(a, place, dtype, st));
        } else {
            Mamba2 m;
            m.proj = S->proj; m.ld = L.proj_cols; m.dt = S->tail; m.dt_ld = L.tail_cols;
            m.heads = l.heads; m.vdim = l.vdim; m.state = l.state; m.groups = l.groups; m.norm_groups = l.norm_groups; m.taps = l.conv_taps;
            m.conv_w = W.conv_w; m.conv_b = W.conv_b; m.dt_bias = W.dt_bias; m.a_log = W.a_log; m.d_skip = W.d_skip; m.norm_w = W.norm_w;
            m.eps = eps; m.ring = L.ring; m.ssm = L.ssm; m.xbc = S->xbc; m.gated = S->gated;
            m.out = S->cat; m.out_ld = L.k_out; m.out_cols = L.mixer_cols;
            m.engine = chunk > 1 && c.prefill_mode == TNSR_B200_PREFILL_SCALAR ? 1 : 0;
            RUN(dec, launch_mamba2(m, place, dtype, st));
        }
        GemmEpilogue eo;
        eo.residual = dec->h; eo.ldr = d; eo.out_dtype = TNSR_B200_F32;
        if (bf) {
            const uint32_t split = splitk ? gemm_split_k((const bf16*)S->cat, (const bf16*)W.w_out, rows, d, L.k_out) : 0;
            if (split) { eo.split_k = split; eo.split_partials = dec->split_ws; eo.split_rows = dec->split_rows; }
            RUN(dec, launch_gemm_bf16((const bf16*)S->cat, (const bf16*)W.w_out, dec->h, d, rows, d, L.k_out, GEMM_PLAIN, eo, nullptr,
                                      dec->d_status, st));
            pending = split;
        } else {
            RUN(dec, launch_gemm_strict((const float*)S->cat, (const float*)W.w_out, dec->h, d, rows, L.k_out, d, true, eo, st));
        }
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
