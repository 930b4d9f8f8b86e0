// The session object behind tnsr_b200_decoder_* as its translation units share it: the handle itself, the error and
// allocation helpers, and the steps of models that are described layer by layer (layer_stack.cu).
#pragma once

#include <memory>
#include <string>
#include <vector>

#include "common.cuh"

namespace tb {

constexpr uint32_t kNoPage = 0xffffffffu;

struct Buffer {
    void* ptr = nullptr;
    size_t bytes = 0;
};

enum ParamKind { P_TOK, P_POS, P_VEC, P_QKV_W, P_QKV_B, P_O_W, P_FF_IN_W, P_FF_IN_B, P_FF_OUT_W, P_GATE_W, P_GATE_B, P_UP_W, P_UP_B };

struct ParamInfo {
    ParamKind kind;
    uint64_t elems;
    uint32_t rows, cols;  // [rows, cols] as the reference stores it ([in, out] for matrices)
    uint32_t layer;
    uint32_t slot;        // 0/1/2 = q/k/v for QKV params
    void* dev = nullptr;  // where the values live (f32 path: as given; bf16 path: see upload)
};

struct Layer {
    // f32 path: the reference layout, f32.  bf16 path: matrices are [out, in] bf16.
    void *wq = nullptr, *wk = nullptr, *wv = nullptr, *wo = nullptr;
    float *bq = nullptr, *bk = nullptr, *bv = nullptr, *bo = nullptr;
    float *ln1w = nullptr, *ln1b = nullptr, *ln2w = nullptr, *ln2b = nullptr;
    void *w_in = nullptr, *w_out = nullptr, *w_gate = nullptr, *w_up = nullptr;
    float *b_in = nullptr, *b_out = nullptr, *b_gate = nullptr, *b_up = nullptr;
    // bf16 path fused forms
    bf16* wqkv = nullptr;  // [3d, d]
    float* bqkv = nullptr; // [3d]
    bf16* wgu = nullptr;   // packed [2f, d] when f % 16 == 0
    float* bgu = nullptr;  // packed [2f]
    void *kcache = nullptr, *vcache = nullptr;
};

struct LayerStack;   // a model described layer by layer (layer_stack.cu)

}  // namespace tb

using namespace tb;

struct tnsr_b200_decoder {
    tnsr_b200_config cfg;
    cudaStream_t stream = nullptr;
    bool bf16_path = false, kv_bf16 = false, swiglu = false, fused_gu = false;
    bool failed = false;
    std::string error;
    std::vector<ParamInfo> params;
    std::vector<Layer> layers;
    void *tok = nullptr, *pos = nullptr;
    float *fnw = nullptr, *fnb = nullptr;
    std::vector<void*> allocations;
    // activations (grow with the chunk)
    uint32_t rows_cap = 0, logit_rows_cap = 0;
    float* h = nullptr;      // residual stream [rows, d] f32
    void* n = nullptr;       // normalised rows: f32 (strict) or bf16
    void* q = nullptr;       // queries: f32 (strict) or bf16
    void* att = nullptr;     // attention output: f32 (strict) or bf16
    void* ff = nullptr;      // FFN hidden [rows, f]
    void* ff2 = nullptr;     // second FFN buffer (up projection) when gate/up are not fused
    float* hl = nullptr;     // last rows [batch, d] f32
    float* logits = nullptr; // [logit_rows, vocab]
    uint32_t* d_tokens = nullptr;
    uint32_t tokens_cap = 0;
    uint32_t* d_argmax = nullptr;
    int* d_status = nullptr;
    void* attn_ws = nullptr;
    // a single-token step may be divided into up to kMaxParts session ranges on as many streams (see step_bf16):
    // range 0 runs on `stream` with `attn_ws`, range i > 0 on side_stream[i - 1] with side_ws[i - 1]
    void* side_ws[3] = {nullptr, nullptr, nullptr};
    // partial sums of the split-K projections of an undivided single-token step: [4][split_rows][d] f32
    float* split_ws = nullptr;
    uint32_t split_rows = 0;
    uint32_t split_pending = 0;   // partial sums of the last layer's down projection, for the final LayerNorm to add
    uint64_t attn_ws_bytes = 0;
    cudaStream_t side_stream[3] = {nullptr, nullptr, nullptr};   // forked from and joined to `stream` by events
    cudaEvent_t ev_fork = nullptr, ev_join[3] = {nullptr, nullptr, nullptr};
    uint32_t parts = 1;
    // small batches: one persistent kernel per layer between the attention scans (decode_tail.cu); its barrier words
    void* tail_ws = nullptr;
    bool use_tail = true;
    // paged K/V: every cache tensor is a pool [pool_pages, page_rows, d]; h_table[s * pps + i] is the pool page of
    // session s's i-th page, kNoPage while unassigned (the device copy is refreshed before the step that needs it)
    bool paged = false;
    uint32_t page_rows = 0, pool_pages = 0, pps = 0;
    std::vector<uint32_t> h_table_shadow;   // the table as the host knows it
    std::vector<uint32_t> free_pages;       // stack of unassigned pool pages
    uint32_t* h_table = nullptr;            // pinned copy used for the upload
    uint32_t* d_table = nullptr;
    bool table_dirty = false;
    // next-token sampling instead of the greedy pick (temperature <= 0: greedy)
    float sample_temperature = 0.0f;
    uint32_t sample_top_k = 0;
    uint64_t sample_seed = 0;
    uint32_t* d_positions = nullptr;   // [batch] per-session positions of a ragged step
    uint32_t* h_positions = nullptr;   // pinned staging for them
    // pinned staging
    uint32_t* h_tokens = nullptr;
    uint32_t* h_argmax = nullptr;
    int* h_status = nullptr;
    float* h_stage = nullptr;  // upload staging (pinned)
    size_t h_stage_bytes = 0;
    float* d_stage = nullptr;  // upload staging (device, f32)
    size_t d_stage_bytes = 0;
    std::vector<float> host_bqkv, host_bgu;
    bool profile_attention = false;
    KernelTimer attention_timer;
    void* lm_candidates = nullptr;  // per (session, vocabulary tile) greedy candidates of the fused LM head
    // single-token steps are replayed from a captured CUDA graph; the position lives in d_pos
    uint32_t* d_pos = nullptr;
    struct StepGraph {
        const uint32_t* tokens;
        uint32_t* argmax;
        cudaGraphExec_t exec;
        uint64_t kernels;
    };
    std::vector<StepGraph> graphs;
    bool use_graphs = true;
    bool use_pdl = true;
    bool stepped_once = false;  // a plain (uncaptured) single-token step has run: buffers and attributes are set
    // set: the model is described layer by layer; `params`, `layers` and the buffers above that only the GPT steps use stay empty
    LayerStack* stack = nullptr;
};

namespace tb {

inline int fail(tnsr_b200_decoder* dec, int code, const std::string& msg) {
    if (dec) dec->error = msg;
    set_thread_error(msg);
    return code;
}

inline int cuda_fail(tnsr_b200_decoder* dec, cudaError_t e, const char* what) {
    std::string msg = std::string(what) + ": " + cudaGetErrorString(e);
    int code = (e == cudaErrorMemoryAllocation) ? TNSR_B200_ERR_OUT_OF_MEMORY : TNSR_B200_ERR_CUDA;
    if (dec && code == TNSR_B200_ERR_CUDA) dec->failed = true;
    cudaGetLastError();
    return fail(dec, code, msg);
}

#define CU(dec, call)                                                   \
    do {                                                                \
        cudaError_t e__ = (call);                                       \
        if (e__ != cudaSuccess) return cuda_fail(dec, e__, #call);      \
    } while (0)

#define RUN(dec, call)                                                  \
    do {                                                                \
        int rc__ = (call);                                              \
        if (rc__ != TNSR_B200_OK) {                                     \
            (dec)->error = thread_error();                              \
            if (rc__ == TNSR_B200_ERR_CUDA) (dec)->failed = true;       \
            return rc__;                                                \
        }                                                               \
    } while (0)

inline void drop_graphs(tnsr_b200_decoder* dec) {
    for (auto& g : dec->graphs) cudaGraphExecDestroy(g.exec);
    dec->graphs.clear();
}

inline int dev_alloc(tnsr_b200_decoder* dec, void** out, size_t bytes, bool zero) {
    if (bytes == 0) bytes = 16;
    void* p = nullptr;
    cudaError_t e = cudaMalloc(&p, bytes);
    if (e != cudaSuccess) return cuda_fail(dec, e, "cudaMalloc");
    dec->allocations.push_back(p);
    if (zero) {
        e = cudaMemsetAsync(p, 0, bytes, dec->stream);
        if (e != cudaSuccess) return cuda_fail(dec, e, "cudaMemsetAsync");
    }
    *out = p;
    return TNSR_B200_OK;
}

inline void dev_free(tnsr_b200_decoder* dec, void* p) {
    if (!p) return;
    for (size_t i = 0; i < dec->allocations.size(); ++i)
        if (dec->allocations[i] == p) {
            dec->allocations.erase(dec->allocations.begin() + i);
            break;
        }
    cudaFree(p);
}

inline size_t elt(const tnsr_b200_decoder* dec) { return dec->bf16_path ? 2 : 4; }
inline size_t kv_elt(const tnsr_b200_decoder* dec) { return dec->kv_bf16 ? 2 : 4; }

inline bool mul_overflow(uint64_t a, uint64_t b, uint64_t* out) { return __builtin_mul_overflow(a, b, out); }

// ---- models described layer by layer (layer_stack.cu) -------------------------
int stack_check(const tnsr_b200_config* config, const tnsr_b200_stack* desc, std::string& why);
int stack_create(tnsr_b200_decoder* dec, const tnsr_b200_stack* desc);   // parameters, weights, caches and states
void stack_destroy(tnsr_b200_decoder* dec);
uint32_t stack_param_count(const tnsr_b200_decoder* dec);
uint64_t stack_param_elems(const tnsr_b200_decoder* dec, uint32_t index);
int stack_upload(tnsr_b200_decoder* dec, uint32_t index, const float* host);
int stack_reset(tnsr_b200_decoder* dec);                                  // queues zeroing of every cache and state
int stack_alloc_rows(tnsr_b200_decoder* dec, uint32_t rows);             // (re)allocates the activation buffers for `rows` rows
// One step: embedding, all layers, final norm, and logits or (fused_ids) greedy ids.
int stack_step(tnsr_b200_decoder* dec, const uint32_t* d_tokens, uint32_t chunk, uint32_t position, const uint32_t* d_position,
               bool ragged, uint32_t logit_rows, uint32_t* fused_ids);
uint32_t stack_cache_count(const tnsr_b200_decoder* dec);
// Cache or state tensor `index`: its device address, elements and element type (tnsr_b200_dtype).
bool stack_cache(const tnsr_b200_decoder* dec, uint32_t index, void** ptr, uint64_t* elems, int* dtype);

}  // namespace tb
