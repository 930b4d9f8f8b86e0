// The attention mixer of models described layer by layer: projections pass a short causal convolution, q and k an RMS
// norm per head and a rotation, and grouped-query attention runs on capped scores with a sigmoid gate per head.
//
//  * attention_prep_kernel     one warp per (head unit, run of tokens): the convolution slides over the run in
//                              registers, so every projected value is read once; q rows and cache rows come out.
//  * attention_rotary_kernel   the same without convolution and norm: rotation (either layout) of q and k, cache rows.
//  * grouped_attention_rows    one warp per (session, head, query), keys in order: f32 sessions, and every shape the
//                              tensor-core kernels (grouped_attention.cu) leave out.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

__device__ __forceinline__ float mx_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// NP: channel pairs per lane (a head unit has at most 64 NP channels).  TAPS: compiled window length; shorter filters are
// padded with zero weights at the old end and never touch the padded rows.
template <typename T, int NP, int TAPS>
__global__ void __launch_bounds__(128)
attention_prep_kernel(AttentionPrep a, StepPlace place, uint32_t run, uint32_t runs, uint32_t total, uint32_t vec) {
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t task = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (task >= total) return;
    const uint32_t units = a.heads + 2 * a.kv_heads;
    const uint32_t unit = task % units, r = (task / units) % runs, s = task / (units * runs);
    const uint32_t nq = a.heads * a.dim, nk = a.kv_heads * a.dim;
    const uint32_t channels = nq + nk + a.kv_heads * a.vdim;
    const uint32_t which = unit < a.heads ? 0u : unit < a.heads + a.kv_heads ? 1u : 2u;
    const uint32_t head = which == 0 ? unit : which == 1 ? unit - a.heads : unit - a.heads - a.kv_heads;
    const uint32_t width = which == 2 ? a.vdim : a.dim;
    const uint32_t ch0 = which == 0 ? head * a.dim : which == 1 ? nq + head * a.dim : nq + nk + head * a.vdim;
    const T* rows = reinterpret_cast<const T*>(a.proj) + (size_t)s * place.chunk * a.ld + ch0;
    T* ring = reinterpret_cast<T*>(a.ring) + (size_t)s * a.taps * channels + ch0;
    const uint32_t p0 = place.pos(s);
    const uint32_t t0 = r * run, t1 = min(place.chunk, t0 + run);

    float2 w[TAPS][NP], nw[NP], win[TAPS][NP];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const uint32_t c = 2 * (lane + 32 * i);
        const bool first = c < width, second = c + 1 < width;
        nw[i] = make_float2(1.0f, 1.0f);
        if (which < 2 && first) {
            const float* g = which == 0 ? a.q_norm : a.k_norm;
            nw[i] = make_float2(g[c], second ? g[c + 1] : 0.0f);
        }
        const float* cw = a.conv_w + (size_t)(ch0 + c) * a.taps;
        if (TAPS == 4 && a.taps == 4) {
            const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            const float4 x = first ? *reinterpret_cast<const float4*>(cw) : zero, y = second ? *reinterpret_cast<const float4*>(cw + 4) : zero;
            w[0][i] = make_float2(x.x, y.x);
            w[TAPS > 1 ? 1 : 0][i] = make_float2(x.y, y.y);
            w[TAPS > 2 ? 2 : 0][i] = make_float2(x.z, y.z);
            w[TAPS > 3 ? 3 : 0][i] = make_float2(x.w, y.w);
        } else {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                const int src = j - (TAPS - (int)a.taps);
                w[j][i].x = src >= 0 && first ? cw[src] : 0.0f;
                w[j][i].y = src >= 0 && second ? cw[a.taps + src] : 0.0f;
            }
        }
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            // the window holds tokens t - TAPS + 1 .. t; before the first token: t0 - TAPS + 1 .. t0 - 1 in slots 1 ..
            win[j][i] = make_float2(0.0f, 0.0f);
            const int t = (int)t0 - TAPS + j;      // token that slot j holds before the first shift
            if (j > 0 && (int)t0 - t < (int)a.taps && first) {
                const long long pos = (long long)p0 + t;
                if (t >= 0) win[j][i] = load_pair<T>(rows + (size_t)t * a.ld + c, vec, second);
                else if (pos >= 0) win[j][i] = load_pair<T>(ring + (size_t)(pos % a.taps) * channels + c, vec, second);
            }
        }
    }
    const uint32_t pairs = a.rotary_dims / 2;
    // a few tokens' inputs and angles are asked for together, so that their round trips overlap
    constexpr uint32_t AHEAD = NP == 1 ? 4 : NP == 2 ? 2 : 1;
    for (uint32_t tb = t0; tb < t1; tb += AHEAD) {
        float2 next[AHEAD][NP], angle[AHEAD][NP];
#pragma unroll
        for (uint32_t u = 0; u < AHEAD; ++u)
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const uint32_t pi = lane + 32 * i, c = 2 * pi;
                const bool there = tb + u < t1;
                next[u][i] = there && c < width ? load_pair<T>(rows + (size_t)(tb + u) * a.ld + c, vec, c + 1 < width) : make_float2(0.0f, 0.0f);
                angle[u][i] = there && which < 2 && pi < pairs ? a.rotation[(size_t)(p0 + tb + u) * pairs + pi] : make_float2(1.0f, 0.0f);
            }
#pragma unroll
        for (uint32_t u = 0; u < AHEAD; ++u) {
            const uint32_t t = tb + u;
            if (t >= t1) break;
            float2 y[NP];
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < NP; ++i) {
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) win[j][i] = win[j + 1][i];
                win[TAPS - 1][i] = next[u][i];
                y[i] = make_float2(0.0f, 0.0f);
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    y[i].x = fmaf(w[j][i].x, win[j][i].x, y[i].x);
                    y[i].y = fmaf(w[j][i].y, win[j][i].y, y[i].y);
                }
                ss = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, ss));
            }
            const uint32_t pos = p0 + t;
            if (place.chunk == 1) {
                // the slot of this position held the oldest row, which no single-token step reads
#pragma unroll
                for (int i = 0; i < NP; ++i) {
                    const uint32_t c = 2 * (lane + 32 * i);
                    if (c < width) store_pair<T>(ring + (size_t)(pos % a.taps) * channels + c, win[TAPS - 1][i], vec, c + 1 < width);
                }
            }
            if (which < 2) {
                const float inv = rsqrtf(mx_warp_sum(ss) / (float)width + a.eps);
#pragma unroll
                for (int i = 0; i < NP; ++i) {
                    const float2 v = make_float2(y[i].x * (inv * nw[i].x), y[i].y * (inv * nw[i].y)), cs = angle[u][i];
                    // pairs past the rotated dimensions have the angle zero
                    y[i] = make_float2(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y);
                }
            }
            T* dst;
            if (which == 0) dst = reinterpret_cast<T*>(a.q) + ((size_t)s * place.chunk + t) * nq + head * a.dim;
            else {
                const size_t row = kv_row(a.paging, s, pos, a.capacity);
                dst = which == 1 ? reinterpret_cast<T*>(a.k_cache) + row * nk + head * a.dim
                                 : reinterpret_cast<T*>(a.v_cache) + row * ((size_t)a.kv_heads * a.vdim) + head * a.vdim;
            }
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const uint32_t c = 2 * (lane + 32 * i);
                if (c < width) store_pair<T>(dst + c, y[i], vec, c + 1 < width);
            }
        }
    }
}

// The same for bf16 heads of whole 16-byte groups and at most four taps: a lane owns eight channels, LPU lanes a head unit,
// so that a warp serves 32 / LPU units at once; rows travel four tokens ahead of their use (the kernel lives on bytes in
// flight), angles one.
template <int LPU>
__global__ void __launch_bounds__(128, 4)
attention_prep_wide_kernel(AttentionPrep a, StepPlace place, uint32_t run, uint32_t runs, uint32_t total) {
    constexpr uint32_t AHEAD = 4;
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, sub = lane % LPU;
    const uint32_t task = (blockIdx.x * 4 + (threadIdx.x >> 5)) * (32 / LPU) + lane / LPU;
    const bool live_task = task < total;                       // idle groups take part in the shuffles
    const uint32_t units = a.heads + 2 * a.kv_heads;
    const uint32_t tk = live_task ? task : 0;
    const uint32_t unit = tk % units, r = (tk / units) % runs, s = tk / (units * runs);
    const uint32_t nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, channels = nq + nk + nv;
    const uint32_t which = unit < a.heads ? 0u : unit < a.heads + a.kv_heads ? 1u : 2u;
    const uint32_t head = which == 0 ? unit : which == 1 ? unit - a.heads : unit - a.heads - a.kv_heads;
    const uint32_t width = which == 2 ? a.vdim : a.dim;
    const uint32_t c = sub * 8, ch = (which == 0 ? head * a.dim : which == 1 ? nq + head * a.dim : nq + nk + head * a.vdim) + c;
    const bool mine = live_task && c < width;
    const uint32_t p0 = place.pos(s);
    const uint32_t t0 = r * run, n = mine ? min(place.chunk - t0, run) : 0u;     // this group's tokens: t0 .. t0 + n - 1
    const bf16* rows = reinterpret_cast<const bf16*>(a.proj) + ((size_t)s * place.chunk + t0) * a.ld + ch;
    bf16* ring = reinterpret_cast<bf16*>(a.ring) + (size_t)s * a.taps * channels + ch;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    uint4 next[AHEAD];
#pragma unroll
    for (uint32_t i = 0; i < AHEAD; ++i) next[i] = i < n ? *reinterpret_cast<const uint4*>(rows + (size_t)i * a.ld) : zero;
    uint4 win[4];
#pragma unroll
    for (int j = 1; j < 4; ++j) {           // slot j: token t0 - 4 + j until the first shift
        win[j] = zero;
        const uint32_t lag = 4 - j;
        if (mine && lag < a.taps) {
            if (t0 >= lag) win[j] = *reinterpret_cast<const uint4*>(rows - (size_t)lag * a.ld);
            else if (p0 + t0 >= lag) win[j] = *reinterpret_cast<const uint4*>(ring + (size_t)((p0 + t0 - lag) % a.taps) * channels);
        }
    }
    float w[4][8], nw[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        nw[e] = mine && which < 2 ? (which == 0 ? a.q_norm : a.k_norm)[c + e] : 1.0f;
        const float* cw = a.conv_w + (size_t)(ch + e) * a.taps;
        if (a.taps == 4) {
            const float4 x = mine ? *reinterpret_cast<const float4*>(cw) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            w[0][e] = x.x; w[1][e] = x.y; w[2][e] = x.z; w[3][e] = x.w;
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) { const int src = j - (4 - (int)a.taps); w[j][e] = mine && src >= 0 ? cw[src] : 0.0f; }
        }
    }
    const uint32_t pairs = a.rotary_dims / 2;
    const bool turns = which < 2 && c < a.rotary_dims;
    const float4* angles = reinterpret_cast<const float4*>(a.rotation + (size_t)(p0 + t0) * pairs + c / 2);
    const uint32_t angle_ld = pairs / 2;
    const float4 still = make_float4(1.0f, 0.0f, 1.0f, 0.0f);      // no rotation
    float4 ang[2];
    ang[0] = turns && n > 0 ? __ldg(angles) : still;
    ang[1] = turns && n > 0 ? __ldg(angles + 1) : still;
    bf16* dst = which == 0 ? reinterpret_cast<bf16*>(a.q) + ((size_t)s * place.chunk + t0) * nq + head * a.dim + c
              : which == 1 ? reinterpret_cast<bf16*>(a.k_cache) + head * a.dim + c : reinterpret_cast<bf16*>(a.v_cache) + head * a.vdim + c;
    const uint32_t dst_ld = which == 0 ? nq : which == 1 ? nk : nv;
    const float inv_width = 1.0f / (float)width;
    for (uint32_t u0 = 0; u0 < run; u0 += AHEAD) {      // the same trip count for every group of the warp: they shuffle together
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i) {
            const uint32_t u = u0 + i;
            const bool here = u < n;
            win[0] = win[1]; win[1] = win[2]; win[2] = win[3]; win[3] = next[i];
            next[i] = u + AHEAD < n ? *reinterpret_cast<const uint4*>(rows + (size_t)(u + AHEAD) * a.ld) : zero;
            const float4 now[2] = {ang[0], ang[1]};
            if (turns && u + 1 < n) {
                ang[0] = __ldg(angles + (size_t)(u + 1) * angle_ld);
                ang[1] = __ldg(angles + (size_t)(u + 1) * angle_ld + 1);
            }
            float y[8] = {};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const uint32_t words[4] = {win[j].x, win[j].y, win[j].z, win[j].w};
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const float2 f = bf16x2_to_f32(words[q]);
                    y[2 * q] = fmaf(w[j][2 * q], f.x, y[2 * q]);
                    y[2 * q + 1] = fmaf(w[j][2 * q + 1], f.y, y[2 * q + 1]);
                }
            }
            if (place.chunk == 1 && here) *reinterpret_cast<uint4*>(ring + (size_t)((p0 + t0) % a.taps) * channels) = win[3];
            float ss = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(y[e], y[e], ss);
#pragma unroll
            for (int o = LPU / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float inv = which < 2 ? rsqrtf(fmaf(ss, inv_width, a.eps)) : 1.0f;
            uint32_t out[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float cs = q & 1 ? now[q >> 1].z : now[q >> 1].x, sn = q & 1 ? now[q >> 1].w : now[q >> 1].y;
                const float a0 = y[2 * q] * (inv * nw[2 * q]), a1 = y[2 * q + 1] * (inv * nw[2 * q + 1]);
                out[q] = pack_bf16x2(a0 * cs - a1 * sn, a1 * cs + a0 * sn);
            }
            if (here) {
                const size_t row = which == 0 ? u : kv_row(a.paging, s, p0 + t0 + u, a.capacity);
                *reinterpret_cast<uint4*>(dst + row * dst_ld) = make_uint4(out[0], out[1], out[2], out[3]);
            }
        }
    }
}

static bool prep_wide_fits(const AttentionPrep& a) {
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    return a.taps <= 4 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld % 8 == 0 && a.rotary_dims % 8 == 0 &&
           aligned(a.proj) && aligned(a.ring) && aligned(a.q) && aligned(a.k_cache) && aligned(a.v_cache) && aligned(a.conv_w) && aligned(a.rotation);
}

template <typename T, int NP>
static void prep_taps(const AttentionPrep& a, const StepPlace& place, uint32_t run, uint32_t runs, uint32_t total, uint32_t vec,
                      cudaStream_t stream) {
    const dim3 grid(ceil_div(total, 4)), block(128);
    if (a.taps <= 4) launch_kernel(attention_prep_kernel<T, NP, 4>, grid, block, 0, stream, a, place, run, runs, total, vec);
    else launch_kernel(attention_prep_kernel<T, NP, kMaxConvTaps>, grid, block, 0, stream, a, place, run, runs, total, vec);
}

template <typename T>
static void prep_width(const AttentionPrep& a, const StepPlace& place, uint32_t run, uint32_t runs, uint32_t total, cudaStream_t stream) {
    const uint32_t width = std::max(a.dim, a.vdim);
    // pairs move as one access when every head starts at an even channel of an even row
    const uint32_t vec = a.dim % 2 == 0 && a.vdim % 2 == 0 && a.ld % 2 == 0;
    if (width <= 64) prep_taps<T, 1>(a, place, run, runs, total, vec, stream);
    else if (width <= 128) prep_taps<T, 2>(a, place, run, runs, total, vec, stream);
    else prep_taps<T, 4>(a, place, run, runs, total, vec, stream);
}

// ---- rotation alone --------------------------------------------------------------------------------
// A thread owns EPT rotated pairs (or 2 EPT plain channels) of one head of one row: with EPT 8 in the layout of halves,
// 16 bytes of the first half and 16 bytes of the second.  Heads of q, k and v are units of one row; a unit has `tasks`
// threads.  VEC: 16-byte accesses (bf16, EPT 8) or single elements (EPT 1).
template <typename T, int EPT>
__global__ void __launch_bounds__(256)
attention_rotary_kernel(AttentionPrep a, StepPlace place, uint32_t tasks, uint64_t total) {
    pdl_wait();
    pdl_trigger();
    const uint64_t id = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (id >= total) return;
    const uint32_t units = a.heads + 2 * a.kv_heads;
    const uint32_t task = (uint32_t)(id % tasks), unit = (uint32_t)(id / tasks % units);
    const uint32_t row = (uint32_t)(id / ((uint64_t)tasks * units)), s = row / place.chunk, t = row % place.chunk;
    const uint32_t nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    const uint32_t which = unit < a.heads ? 0u : unit < a.heads + a.kv_heads ? 1u : 2u;
    const uint32_t head = which == 0 ? unit : which == 1 ? unit - a.heads : unit - a.heads - a.kv_heads;
    const uint32_t width = which == 2 ? a.vdim : a.dim, turned = which == 2 ? 0u : a.rotary_dims, half = turned / 2;
    const uint32_t pos = place.pos(s) + t;
    const T* src = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.ld + (which == 0 ? head * a.dim : which == 1 ? nq + head * a.dim : nq + nk + head * a.vdim);
    T* dst;
    if (which == 0) {
        dst = reinterpret_cast<T*>(a.q) + (size_t)row * nq + head * a.dim;
    } else {
        const size_t kr = kv_row(a.paging, s, pos, a.capacity);
        dst = which == 1 ? reinterpret_cast<T*>(a.k_cache) + kr * nk + head * a.dim : reinterpret_cast<T*>(a.v_cache) + kr * nv + head * a.vdim;
    }
    // tasks [0, half / EPT) turn pairs; the rest copies channels from `turned` on, 2 EPT at a time
    const uint32_t pair_tasks = half / EPT;
    if (task < pair_tasks) {
        const uint32_t i0 = task * EPT;
        const float2* angle = a.rotation + (size_t)pos * half + i0;
        const bool halves = a.rotary_layout == TNSR_B200_ROTARY_HALVES;
        const uint32_t c0 = halves ? i0 : 2 * i0, c1 = halves ? i0 + half : 2 * i0 + EPT;
        if (EPT == 8) {
            const uint4 x4 = *reinterpret_cast<const uint4*>(src + c0), y4 = *reinterpret_cast<const uint4*>(src + c1);
            const uint32_t x[4] = {x4.x, x4.y, x4.z, x4.w}, y[4] = {y4.x, y4.y, y4.z, y4.w};
            uint32_t ox[4], oy[4];
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                const float2 u = bf16x2_to_f32(x[w]), v = bf16x2_to_f32(y[w]);
                if (halves) {        // word w: pairs 2w and 2w + 1, u from the first half, v from the second
                    const float4 cs = __ldg(reinterpret_cast<const float4*>(angle) + w);
                    ox[w] = pack_bf16x2(u.x * cs.x - v.x * cs.y, u.y * cs.z - v.y * cs.w);
                    oy[w] = pack_bf16x2(v.x * cs.x + u.x * cs.y, v.y * cs.z + u.y * cs.w);
                } else {             // word w of the first 16 bytes: pair w; of the second: pair 4 + w
                    const float2 ca = __ldg(angle + w), cb = __ldg(angle + 4 + w);
                    ox[w] = pack_bf16x2(u.x * ca.x - u.y * ca.y, u.y * ca.x + u.x * ca.y);
                    oy[w] = pack_bf16x2(v.x * cb.x - v.y * cb.y, v.y * cb.x + v.x * cb.y);
                }
            }
            *reinterpret_cast<uint4*>(dst + c0) = make_uint4(ox[0], ox[1], ox[2], ox[3]);
            *reinterpret_cast<uint4*>(dst + c1) = make_uint4(oy[0], oy[1], oy[2], oy[3]);
        } else {
            const float2 cs = *angle;
            const float u = to_f32(src[c0]), v = to_f32(src[c1]);
            dst[c0] = from_f32<T>(u * cs.x - v * cs.y);
            dst[c1] = from_f32<T>(v * cs.x + u * cs.y);
        }
        return;
    }
    const uint32_t c = turned + (task - pair_tasks) * 2 * EPT;
    if (EPT == 8) {
#pragma unroll
        for (int i = 0; i < 2; ++i)
            if (c + 8 * i < width) *reinterpret_cast<uint4*>(dst + c + 8 * i) = *reinterpret_cast<const uint4*>(src + c + 8 * i);
    } else {
#pragma unroll
        for (int i = 0; i < 2; ++i)
            if (c + i < width) dst[c + i] = src[c + i];
    }
}

static int launch_attention_rotary(const AttentionPrep& a, const StepPlace& place, int dtype, cudaStream_t stream) {
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool wide = dtype == TNSR_B200_BF16 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld % 8 == 0 && a.rotary_dims % 16 == 0 && aligned(a.proj) &&
                      aligned(a.q) && aligned(a.k_cache) && aligned(a.v_cache) && aligned(a.rotation);
    const uint32_t ept = wide ? 8 : 1;
    const uint32_t tasks = std::max(a.rotary_dims / 2 / ept + ceil_div(a.dim - a.rotary_dims, 2 * ept), ceil_div(a.vdim, 2 * ept));
    const uint64_t total = (uint64_t)place.sessions * place.chunk * (a.heads + 2 * a.kv_heads) * tasks;
    if (ceil_div64(total, 256) > 0x7fffffffull) { set_thread_error("attention: too many rows for one launch"); return TNSR_B200_ERR_UNSUPPORTED; }
    const dim3 grid((uint32_t)ceil_div64(total, 256)), block(256);
    if (wide) launch_kernel(attention_rotary_kernel<bf16, 8>, grid, block, 0, stream, a, place, tasks, total);
    else if (dtype == TNSR_B200_BF16) launch_kernel(attention_rotary_kernel<bf16, 1>, grid, block, 0, stream, a, place, tasks, total);
    else launch_kernel(attention_rotary_kernel<float, 1>, grid, block, 0, stream, a, place, tasks, total);
    count_launch();
    return check_launch("attention_rotary");
}

int launch_attention_prep(const AttentionPrep& a, const StepPlace& place, int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    if (!a.conv_w && a.dim <= 256 && a.vdim <= 256 && a.rotary_dims <= a.dim && a.rotary_dims % 2 == 0) return launch_attention_rotary(a, place, dtype, stream);
    if (a.rotary_layout != TNSR_B200_ROTARY_INTERLEAVED || a.dim > 256 || a.vdim > 256 || a.taps == 0 || a.taps > kMaxConvTaps || a.rotary_dims > a.dim || a.rotary_dims % 2) {
        set_thread_error("attention: head widths up to 256, 1..16 convolution taps (behind one the interleaved rotation), an even number of rotated dimensions");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    const uint32_t run = std::min(place.chunk, 32u), runs = ceil_div(place.chunk, run);
    const uint64_t total = (uint64_t)place.sessions * runs * (a.heads + 2 * a.kv_heads);
    if (total > 0x7fffffffull) { set_thread_error("attention: too many rows for one launch"); return TNSR_B200_ERR_UNSUPPORTED; }
    if (dtype == TNSR_B200_BF16 && prep_wide_fits(a)) {
        const uint32_t width = std::max(a.dim, a.vdim);
        auto grid = [&](uint32_t lanes) { return dim3((uint32_t)ceil_div64(total, 4 * (32 / lanes))); };
        if (width <= 64) launch_kernel(attention_prep_wide_kernel<8>, grid(8), dim3(128), 0, stream, a, place, run, runs, (uint32_t)total);
        else if (width <= 128) launch_kernel(attention_prep_wide_kernel<16>, grid(16), dim3(128), 0, stream, a, place, run, runs, (uint32_t)total);
        else launch_kernel(attention_prep_wide_kernel<32>, grid(32), dim3(128), 0, stream, a, place, run, runs, (uint32_t)total);
    } else if (dtype == TNSR_B200_BF16) prep_width<bf16>(a, place, run, runs, (uint32_t)total, stream);
    else prep_width<float>(a, place, run, runs, (uint32_t)total, stream);
    count_launch();
    return check_launch("attention_prep");
}

// ---- convolution inputs of a multi-token chunk into the session's ring ---------------------
template <typename T>
__global__ void __launch_bounds__(256)
conv_ring_kernel(const T* __restrict__ rows, uint32_t ld, uint32_t channels, uint32_t taps, T* __restrict__ ring, StepPlace place) {
    pdl_wait();
    pdl_trigger();
    const uint32_t s = blockIdx.y, keep = min(place.chunk, taps);
    const uint32_t p0 = place.pos(s);
    for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < keep * channels; i += gridDim.x * blockDim.x) {
        const uint32_t t = place.chunk - keep + i / channels, c = i % channels;
        ring[((size_t)s * taps + (p0 + t) % taps) * channels + c] = rows[((size_t)s * place.chunk + t) * ld + c];
    }
}

int launch_conv_ring(const void* rows, uint32_t ld, uint32_t channels, uint32_t taps, void* ring, const StepPlace& place,
                     int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    if (place.sessions > 65535u) { set_thread_error("convolution: too many sessions for one launch"); return TNSR_B200_ERR_UNSUPPORTED; }
    const dim3 grid(std::min(ceil_div(std::min(place.chunk, taps) * channels, 256u), 64u), place.sessions);
    if (dtype == TNSR_B200_BF16)
        launch_kernel(conv_ring_kernel<bf16>, grid, dim3(256), 0, stream, (const bf16*)rows, ld, channels, taps, (bf16*)ring, place);
    else
        launch_kernel(conv_ring_kernel<float>, grid, dim3(256), 0, stream, (const float*)rows, ld, channels, taps, (float*)ring, place);
    count_launch();
    return check_launch("conv_ring");
}

// ---- one warp per (session, head, query) -----------------------------------------------------
constexpr int GR_SLOTS = 8;   // widths up to 256: lane owns columns lane, lane + 32, ...

template <typename T>
__global__ void __launch_bounds__(128)
grouped_attention_rows_kernel(GroupedAttention a, StepPlace place, uint32_t total) {
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t task = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (task >= total) return;
    const uint32_t t = task % place.chunk, h = (task / place.chunk) % a.heads, s = task / (place.chunk * a.heads);
    const uint32_t g = h / (a.heads / a.kv_heads);
    const size_t row = (size_t)s * place.chunk + t;
    const T* qr = reinterpret_cast<const T*>(a.q) + row * ((size_t)a.heads * a.dim) + (size_t)h * a.dim;
    const T* kb = reinterpret_cast<const T*>(a.k_cache) + (size_t)g * a.dim;
    const T* vb = reinterpret_cast<const T*>(a.v_cache) + (size_t)g * a.vdim;
    const size_t k_ld = (size_t)a.kv_heads * a.dim, v_ld = (size_t)a.kv_heads * a.vdim;
    const uint32_t keys = min(place.pos(s) + t + 1, a.capacity), first = a.window && keys > a.window ? keys - a.window : 0u;
    const bool sigmoid = a.score_kind == TNSR_B200_SCORE_SIGMOID;
    const float bias = sigmoid && a.head_bias ? a.head_bias[h] : 0.0f;
    float q[GR_SLOTS], acc[GR_SLOTS];
#pragma unroll
    for (int i = 0; i < GR_SLOTS; ++i) {
        const uint32_t c = lane + 32 * i;
        q[i] = c < a.dim ? to_f32(qr[c]) : 0.0f;
        acc[i] = 0.0f;
    }
    float m = -INFINITY, l = 0.0f;
    for (uint32_t j = first; j < keys; ++j) {
        const size_t kr = kv_row(a.paging, s, j, a.capacity);
        float part = 0.0f;
#pragma unroll
        for (int i = 0; i < GR_SLOTS; ++i) {
            const uint32_t c = lane + 32 * i;
            if (c < a.dim) part = fmaf(q[i], to_f32(kb[kr * k_ld + c]), part);
        }
        float sc = mx_warp_sum(part) * a.scale;
        if (sigmoid) {
            const float p = 1.0f / (1.0f + expf(-(sc + bias)));
#pragma unroll
            for (int i = 0; i < GR_SLOTS; ++i) {
                const uint32_t c = lane + 32 * i;
                if (c < a.vdim) acc[i] = fmaf(p, to_f32(vb[kr * v_ld + c]), acc[i]);
            }
            continue;
        }
        if (a.softcap > 0.0f) sc = a.softcap * tanhf(sc / a.softcap);
        const float m_new = fmaxf(m, sc);
        const float corr = expf(m - m_new), p = expf(sc - m_new);
        l = l * corr + p;
#pragma unroll
        for (int i = 0; i < GR_SLOTS; ++i) {
            const uint32_t c = lane + 32 * i;
            if (c < a.vdim) acc[i] = fmaf(acc[i], corr, p * to_f32(vb[kr * v_ld + c]));
        }
        m = m_new;
    }
    const float gate = a.gain * (a.gate ? 1.0f / (1.0f + expf(-a.gate[row * a.gate_ld + h])) : 1.0f);
    if (sigmoid) l = 1.0f;
    T* orow = reinterpret_cast<T*>(a.out) + row * a.out_ld;
#pragma unroll
    for (int i = 0; i < GR_SLOTS; ++i) {
        const uint32_t c = lane + 32 * i;
        if (c < a.vdim) orow[(size_t)h * a.vdim + c] = from_f32<T>(acc[i] / l * gate);
    }
    if (h + 1 == a.heads)
        for (uint32_t c = a.heads * a.vdim + lane; c < a.out_cols; c += 32) orow[c] = from_f32<T>(0.0f);
}

int launch_grouped_attention_rows(const GroupedAttention& a, const StepPlace& place, int dtype, cudaStream_t stream) {
    const uint64_t total = (uint64_t)place.sessions * place.chunk * a.heads;
    if (total > 0x7fffffffull) { set_thread_error("attention: too many rows for one launch"); return TNSR_B200_ERR_UNSUPPORTED; }
    if (dtype == TNSR_B200_BF16)
        launch_kernel(grouped_attention_rows_kernel<bf16>, dim3((unsigned)ceil_div64(total, 4)), dim3(128), 0, stream, a, place, (uint32_t)total);
    else
        launch_kernel(grouped_attention_rows_kernel<float>, dim3((unsigned)ceil_div64(total, 4)), dim3(128), 0, stream, a, place, (uint32_t)total);
    count_launch();
    return check_launch("grouped_attention_rows");
}

}  // namespace tb
