// Feed-forwards of models described layer by layer.
//
//  * polynorm_kernel        W_down p(W_up h): the three normalised powers of a row, one pass for the sums, one for the values.
//  * expert routing         softmax of the router logits, the `top` largest corrected scores, weights (a warp per row); the
//                           chosen (row, expert) pairs are sorted by expert by counting -- per block of 256 rows, then over
//                           blocks -- and their rows gathered; a step of at most 256 rows sorts in its one routing block.
//                           Single-token steps: norm, router logits and choice in one block per row, and a gather that
//                           counts places itself.
//  * products               gemm_grouped.cu: up with relu^2, down.
//  * experts_combine_kernel x += layer_scale * (weighted expert rows + weighted h of identity experts), in slot order, and
//                           the next norm of the row: deterministic, and one trip of the residual row.
// Routing, norms and sums are f32 in both precisions.
#include <algorithm>

#include "feed_forward.cuh"
#include "mixers.cuh"

namespace tb {

__device__ __forceinline__ float ff_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// ---- PolyNorm ----------------------------------------------------------------------------------------
// One block per row.  VEC: 16-byte accesses of bf16 rows, kept in registers up to PN_KEEP chunks per thread.
constexpr uint32_t PN_THREADS = 256;
constexpr int PN_KEEP = 4;

struct PolySums { float s2, s4, s6; };
__device__ __forceinline__ void pn_add(PolySums& s, float z) {
    const float z2 = z * z, z4 = z2 * z2;
    s.s2 += z2;
    s.s4 += z4;
    s.s6 = fmaf(z4, z2, s.s6);
}
__device__ __forceinline__ PolySums pn_total(PolySums s) {
    __shared__ float red[3][PN_THREADS / 32];
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    s.s2 = ff_warp_sum(s.s2); s.s4 = ff_warp_sum(s.s4); s.s6 = ff_warp_sum(s.s6);
    if (lane == 0) { red[0][warp] = s.s2; red[1][warp] = s.s4; red[2][warp] = s.s6; }
    __syncthreads();
    PolySums t = {0.0f, 0.0f, 0.0f};
#pragma unroll
    for (uint32_t i = 0; i < PN_THREADS / 32; ++i) { t.s2 += red[0][i]; t.s4 += red[1][i]; t.s6 += red[2][i]; }
    return t;
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(PN_THREADS)
polynorm_kernel(const T* __restrict__ z, const float* __restrict__ act, T* __restrict__ out, uint32_t width, uint32_t out_ld, uint32_t out_cols,
                float eps) {
    pdl_wait();
    pdl_trigger();
    const size_t row = blockIdx.x;
    const T* in = z + row * width;
    T* o = out + row * out_ld;
    const float a = act[0], b = act[1], c = act[2], e = act[3];
    PolySums s = {0.0f, 0.0f, 0.0f};
    const uint32_t chunks = width / 8;
    uint4 keep[VEC ? PN_KEEP : 1];
    if (VEC) {
        auto add = [&](uint4 q) {
            const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) { const float2 f = bf16x2_to_f32(w[i]); pn_add(s, f.x); pn_add(s, f.y); }
        };
#pragma unroll
        for (int i = 0; i < (VEC ? PN_KEEP : 1); ++i) {
            const uint32_t k = threadIdx.x + i * PN_THREADS;
            keep[i] = k < chunks ? reinterpret_cast<const uint4*>(in)[k] : make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int i = 0; i < (VEC ? PN_KEEP : 1); ++i) add(keep[i]);
        for (uint32_t k = threadIdx.x + PN_KEEP * PN_THREADS; k < chunks; k += PN_THREADS) add(reinterpret_cast<const uint4*>(in)[k]);
    } else {
        for (uint32_t k = threadIdx.x; k < width; k += PN_THREADS) pn_add(s, to_f32(in[k]));
    }
    s = pn_total(s);
    const float inv_n = 1.0f / (float)width;
    const float fa = a * rsqrtf(fmaf(s.s2, inv_n, eps)), fb = b * rsqrtf(fmaf(s.s4, inv_n, eps)), fc = c * rsqrtf(fmaf(s.s6, inv_n, eps));
    auto value = [&](float x) { return fmaf(x, fmaf(x, fmaf(x, fc, fb), fa), e); };
    if (VEC) {
        auto put = [&](uint32_t k, uint4 q) {
            const uint32_t w[4] = {q.x, q.y, q.z, q.w};
            uint32_t r[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { const float2 f = bf16x2_to_f32(w[i]); r[i] = pack_bf16x2(value(f.x), value(f.y)); }
            reinterpret_cast<uint4*>(o)[k] = make_uint4(r[0], r[1], r[2], r[3]);
        };
#pragma unroll
        for (int i = 0; i < (VEC ? PN_KEEP : 1); ++i) {
            const uint32_t k = threadIdx.x + i * PN_THREADS;
            if (k < chunks) put(k, keep[i]);
        }
        for (uint32_t k = threadIdx.x + PN_KEEP * PN_THREADS; k < chunks; k += PN_THREADS) put(k, reinterpret_cast<const uint4*>(in)[k]);
    } else {
        for (uint32_t k = threadIdx.x; k < width; k += PN_THREADS) o[k] = from_f32<T>(value(to_f32(in[k])));
    }
    for (uint32_t k = width + threadIdx.x; k < out_cols; k += PN_THREADS) o[k] = from_f32<T>(0.0f);
}

// Rows of whole 16-byte chunks up to 4096 columns, many of them: a warp per row, the row in registers.
constexpr int PN_WARP_CHUNKS = 16;
template <int CHUNKS>
__global__ void __launch_bounds__(128)
polynorm_warp_kernel(const bf16* __restrict__ z, const float* __restrict__ act, bf16* __restrict__ out, uint32_t rows, uint32_t width, uint32_t out_ld,
                     uint32_t out_cols, float eps) {
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, row = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (row >= rows) return;
    const uint4* in = reinterpret_cast<const uint4*>(z + (size_t)row * width);
    uint4* o = reinterpret_cast<uint4*>(out + (size_t)row * out_ld);
    const uint32_t chunks = width / 8;
    uint4 keep[CHUNKS];
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) keep[i] = lane + 32 * i < chunks ? in[lane + 32 * i] : make_uint4(0u, 0u, 0u, 0u);
    PolySums s = {0.0f, 0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) {
        const uint32_t w[4] = {keep[i].x, keep[i].y, keep[i].z, keep[i].w};
#pragma unroll
        for (int k = 0; k < 4; ++k) { const float2 f = bf16x2_to_f32(w[k]); pn_add(s, f.x); pn_add(s, f.y); }
    }
    s.s2 = ff_warp_sum(s.s2); s.s4 = ff_warp_sum(s.s4); s.s6 = ff_warp_sum(s.s6);
    const float inv_n = 1.0f / (float)width;
    const float fa = act[0] * rsqrtf(fmaf(s.s2, inv_n, eps)), fb = act[1] * rsqrtf(fmaf(s.s4, inv_n, eps)), fc = act[2] * rsqrtf(fmaf(s.s6, inv_n, eps));
    const float e = act[3];
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) {
        if (lane + 32 * i >= chunks) continue;
        const uint32_t w[4] = {keep[i].x, keep[i].y, keep[i].z, keep[i].w};
        uint32_t r[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = bf16x2_to_f32(w[k]);
            r[k] = pack_bf16x2(fmaf(f.x, fmaf(f.x, fmaf(f.x, fc, fb), fa), e), fmaf(f.y, fmaf(f.y, fmaf(f.y, fc, fb), fa), e));
        }
        o[lane + 32 * i] = make_uint4(r[0], r[1], r[2], r[3]);
    }
    for (uint32_t k = width + lane; k < out_cols; k += 32) out[(size_t)row * out_ld + k] = __float2bfloat16_rn(0.0f);
}

int launch_polynorm(const void* z, const float* act, void* out, uint32_t rows, uint32_t width, uint32_t out_ld, uint32_t out_cols,
                    float eps, int dtype, cudaStream_t stream) {
    if (rows == 0) return TNSR_B200_OK;
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool vec = dtype == TNSR_B200_BF16 && width % 8 == 0 && out_ld % 8 == 0 && aligned(z) && aligned(out);
    if (vec && width <= PN_WARP_CHUNKS * 256 && !t_single_token_step) {     // few rows: a block per row has more loads in flight
        const dim3 grid(ceil_div(rows, 4u)), block(128);
        if (width <= 1024) launch_kernel(polynorm_warp_kernel<4>, grid, block, 0, stream, (const bf16*)z, act, (bf16*)out, rows, width, out_ld, out_cols, eps);
        else if (width <= 2048) launch_kernel(polynorm_warp_kernel<8>, grid, block, 0, stream, (const bf16*)z, act, (bf16*)out, rows, width, out_ld, out_cols, eps);
        else if (width <= 3072) launch_kernel(polynorm_warp_kernel<12>, grid, block, 0, stream, (const bf16*)z, act, (bf16*)out, rows, width, out_ld, out_cols, eps);
        else launch_kernel(polynorm_warp_kernel<16>, grid, block, 0, stream, (const bf16*)z, act, (bf16*)out, rows, width, out_ld, out_cols, eps);
    } else if (vec)
        launch_kernel(polynorm_kernel<bf16, true>, dim3(rows), dim3(PN_THREADS), 0, stream, (const bf16*)z, act, (bf16*)out, width, out_ld, out_cols, eps);
    else if (dtype == TNSR_B200_BF16)
        launch_kernel(polynorm_kernel<bf16, false>, dim3(rows), dim3(PN_THREADS), 0, stream, (const bf16*)z, act, (bf16*)out, width, out_ld, out_cols, eps);
    else
        launch_kernel(polynorm_kernel<float, false>, dim3(rows), dim3(PN_THREADS), 0, stream, (const float*)z, act, (float*)out, width, out_ld, out_cols, eps);
    count_launch();
    return check_launch("polynorm");
}

// ---- routing ---------------------------------------------------------------------------------------------
constexpr uint32_t MR_ROWS = 256, MR_THREADS = 1024;

struct RouteParams {
    const float* logits;
    const float* correction;
    uint32_t rows, logits_ld, experts, total, top;
    float scale;
    float* weights;        // [rows, top]
    uint32_t* place;       // [rows, top]: expert while routing (kMaxExperts and above: identity), then the row in expert order
    uint32_t* rank;        // [rows, top]: place among the pairs of the same block and expert
    uint32_t* counts;      // [blocks, experts], then first row of the block's pairs of that expert
    uint32_t* offsets;     // [experts + 1]
    uint32_t* chosen;      // may be null
    float* weights_out;    // may be null
};
constexpr uint32_t kIdentityPlace = 0xffffffffu;

// Exclusive sum of counts[0 .. n) into out[0 .. n], by one warp.
__device__ __forceinline__ void mr_scan(const uint32_t* counts, uint32_t* out, uint32_t n, uint32_t lane) {
    uint32_t base = 0;
    for (uint32_t e0 = 0; e0 < n; e0 += 32) {
        const uint32_t e = e0 + lane, c = e < n ? counts[e] : 0u;
        uint32_t x = c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const uint32_t y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= (uint32_t)o) x += y;
        }
        if (e < n) out[e] = base + x - c;
        base += __shfl_sync(0xffffffffu, x, 31);
    }
    if (lane == 0) out[n] = base;
}

// Routing of one row by a warp: lane k < top receives the k-th chosen expert and its weight.  NV: scores per lane.
template <int NV>
__device__ __forceinline__ void mr_route(const float* z, const float* __restrict__ correction, uint32_t n, uint32_t top, float scale, uint32_t lane,
                                         uint32_t& mine_e, float& mine_w) {
    float s[NV], c[NV];
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const uint32_t e = lane + 32 * i;
        s[i] = e < n ? z[e] : -INFINITY;
        c[i] = e < n ? correction[e] : 0.0f;
        mx = fmaxf(mx, s[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) { s[i] = lane + 32 * i < n ? expf(s[i] - mx) : 0.0f; sum += s[i]; }
    sum = ff_warp_sum(sum);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        s[i] /= sum;
        c[i] = lane + 32 * i < n ? s[i] + c[i] : -INFINITY;
    }
    float total = 0.0f, mine_s = 0.0f;
    mine_e = 0;
    for (uint32_t k = 0; k < top; ++k) {
        // largest corrected score, lowest index among equal ones
        float best = -INFINITY;
        uint32_t best_e = 0xffffffffu;
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (c[i] > best || (c[i] == best && best_e == 0xffffffffu)) { best = c[i]; best_e = lane + 32 * i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const uint32_t oe = __shfl_xor_sync(0xffffffffu, best_e, o);
            if (ob > best || (ob == best && oe < best_e)) { best = ob; best_e = oe; }
        }
        best_e = min(best_e, n - 1);       // a row of NaN logits still routes inside the table
        float best_s = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (lane + 32 * i == best_e) { c[i] = -INFINITY; best_s = s[i]; }
        best_s = __shfl_sync(0xffffffffu, best_s, best_e & 31);
        total += best_s;
        if (lane == k) { mine_s = best_s; mine_e = best_e; }
    }
    mine_w = mine_s / (total + 1e-20f) * scale;
}

// One block serves MR_ROWS rows, a warp per row at a time.
template <int NV>
__global__ void __launch_bounds__(MR_THREADS)
experts_route_kernel(RouteParams P) {
    __shared__ uint32_t hist[kMaxExperts], first[kMaxExperts + 1];
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (uint32_t e = threadIdx.x; e < P.experts; e += MR_THREADS) hist[e] = 0;
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    const uint32_t row0 = blockIdx.x * MR_ROWS, row1 = min(P.rows, row0 + MR_ROWS);
    for (uint32_t row = row0 + warp; row < row1; row += MR_THREADS / 32) {
        uint32_t mine_e;
        float w;
        mr_route<NV>(P.logits + (size_t)row * P.logits_ld, P.correction, P.total, P.top, P.scale, lane, mine_e, w);
        if (lane < P.top) {
            const size_t slot = (size_t)row * P.top + lane;
            P.weights[slot] = w;
            if (P.chosen) P.chosen[slot] = mine_e;
            if (P.weights_out) P.weights_out[slot] = w;
            const bool real = mine_e < P.experts;
            P.place[slot] = real ? mine_e : kIdentityPlace;
            if (real) P.rank[slot] = atomicAdd(hist + mine_e, 1u);
        }
    }
    __syncthreads();
    if (gridDim.x > 1) {
        for (uint32_t e = threadIdx.x; e < P.experts; e += MR_THREADS) P.counts[(size_t)blockIdx.x * P.experts + e] = hist[e];
        return;
    }
    // a single block knows everything
    if (warp == 0) mr_scan(hist, first, P.experts, lane);
    __syncthreads();
    for (uint32_t e = threadIdx.x; e <= P.experts; e += MR_THREADS) {
        P.offsets[e] = first[e];
        if (e < P.experts) P.counts[e] = first[e];
    }
}

// Several blocks: counts become first rows.  A warp per expert adds over blocks, 32 at a time.
__global__ void __launch_bounds__(MR_THREADS)
experts_offsets_kernel(uint32_t* counts, uint32_t* offsets, uint32_t blocks, uint32_t experts) {
    __shared__ uint32_t total[kMaxExperts], first[kMaxExperts + 1];
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (uint32_t e = warp; e < experts; e += MR_THREADS / 32) {
        uint32_t base = 0;
        for (uint32_t b0 = 0; b0 < blocks; b0 += 32) {
            const uint32_t b = b0 + lane;
            const uint32_t c = b < blocks ? counts[(size_t)b * experts + e] : 0u;
            uint32_t x = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const uint32_t y = __shfl_up_sync(0xffffffffu, x, o);
                if (lane >= (uint32_t)o) x += y;
            }
            if (b < blocks) counts[(size_t)b * experts + e] = base + x - c;
            base += __shfl_sync(0xffffffffu, x, 31);
        }
        if (lane == 0) total[e] = base;
    }
    __syncthreads();
    if (warp == 0) mr_scan(total, first, experts, lane);
    __syncthreads();
    for (uint32_t e = threadIdx.x; e <= experts; e += MR_THREADS) offsets[e] = first[e];
    for (uint32_t e = warp; e < experts; e += MR_THREADS / 32)
        for (uint32_t b = lane; b < blocks; b += 32) counts[(size_t)b * experts + e] += first[e];
}

// A warp per (row, slot): fixes its place and copies the row there.
template <typename V>
__global__ void __launch_bounds__(256)
experts_gather_kernel(const V* __restrict__ h, V* __restrict__ out, uint32_t* __restrict__ place, const uint32_t* __restrict__ rank,
                      const uint32_t* __restrict__ counts, uint32_t pairs, uint32_t top, uint32_t experts, uint32_t words) {
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, pair = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (pair >= pairs) return;
    const uint32_t row = pair / top, e = place[pair];
    if (e == kIdentityPlace) return;
    const uint32_t at = counts[(size_t)(row / MR_ROWS) * experts + e] + rank[pair];
    if (at >= pairs) return;
    __syncwarp();
    if (lane == 0) place[pair] = at;
    const V* src = h + (size_t)row * words;
    V* dst = out + (size_t)at * words;
    constexpr uint32_t AHEAD = 4;
    for (uint32_t c = lane; c < words; c += 32 * AHEAD) {
        V v[AHEAD];
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i) if (c + 32 * i < words) v[i] = src[c + 32 * i];
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i) if (c + 32 * i < words) dst[c + 32 * i] = v[i];
    }
}

// ---- single-token steps: norm, router and choice of a row in one block ------------------------------------------
// The row is completed first when a split product left partial sums (see launch_layernorm_fold), then normalised; its router
// logits are dot products of the normalised row in shared memory with the router's rows.
constexpr uint32_t EX_THREADS = 256;
struct ChooseParams {
    float* x;
    const float* partials;
    uint32_t parts, split_rows;
    const float* norm_w;
    float norm_offset, eps;
    void* h;                   // [rows, d]
    const void* router;        // [total, d]
    RouteParams route;
    uint32_t d;
};

template <typename T, int NV>
__global__ void __launch_bounds__(EX_THREADS)
experts_choose_kernel(ChooseParams P) {
    extern __shared__ __align__(16) float row_s[];       // [d]
    __shared__ float z[NV * 32], red[EX_THREADS / 32];
    pdl_wait();
    pdl_trigger();
    const uint32_t row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, d = P.d;
    float* xr = P.x + (size_t)row * d;
    float ss = 0.0f;
    for (uint32_t c = threadIdx.x; c < d; c += EX_THREADS) {
        float v = xr[c], p[4];
#pragma unroll
        for (uint32_t i = 0; i < 4; ++i) p[i] = i < P.parts ? P.partials[((size_t)i * P.split_rows + row) * d + c] : 0.0f;
#pragma unroll
        for (uint32_t i = 0; i < 4; ++i) v += p[i];
        if (P.parts) xr[c] = v;
        row_s[c] = v;
        ss = fmaf(v, v, ss);
    }
    ss = ff_warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float sum = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < EX_THREADS / 32; ++i) sum += red[i];
    const float inv = rsqrtf(sum / (float)d + P.eps);
    T* h = reinterpret_cast<T*>(P.h) + (size_t)row * d;
    for (uint32_t c = threadIdx.x; c < d; c += EX_THREADS) {
        const T v = from_f32<T>(row_s[c] * inv * (P.norm_offset + P.norm_w[c]));
        h[c] = v;
        row_s[c] = to_f32(v);
    }
    __syncthreads();
    const T* w = reinterpret_cast<const T*>(P.router);
    constexpr uint32_t WARPS = EX_THREADS / 32, SIDE = 4;          // a warp forms SIDE dot products side by side
    for (uint32_t e0 = warp; e0 < P.route.total; e0 += WARPS * SIDE) {
        float acc[SIDE] = {};
        if (sizeof(T) == 2 && d % 8 == 0) {
#pragma unroll 2
            for (uint32_t c = lane; c < d / 8; c += 32) {
                uint4 q[SIDE];
#pragma unroll
                for (uint32_t i = 0; i < SIDE; ++i)
                    q[i] = e0 + i * WARPS < P.route.total ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)(e0 + i * WARPS) * d) + c) : make_uint4(0u, 0u, 0u, 0u);
                const float4 a = *reinterpret_cast<const float4*>(row_s + 8 * c), b = *reinterpret_cast<const float4*>(row_s + 8 * c + 4);
                const float hv[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
                for (uint32_t i = 0; i < SIDE; ++i) {
                    const uint32_t words[4] = {q[i].x, q[i].y, q[i].z, q[i].w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float2 f = bf16x2_to_f32(words[j]);
                        acc[i] = fmaf(f.x, hv[2 * j], fmaf(f.y, hv[2 * j + 1], acc[i]));
                    }
                }
            }
        } else {
            for (uint32_t c = lane; c < d; c += 32)
#pragma unroll
                for (uint32_t i = 0; i < SIDE; ++i)
                    if (e0 + i * WARPS < P.route.total) acc[i] = fmaf(to_f32(w[(size_t)(e0 + i * WARPS) * d + c]), row_s[c], acc[i]);
        }
#pragma unroll
        for (uint32_t i = 0; i < SIDE; ++i) {
            const float v = ff_warp_sum(acc[i]);
            if (lane == 0 && e0 + i * WARPS < P.route.total) z[e0 + i * WARPS] = v;
        }
    }
    __syncthreads();
    if (warp != 0) return;
    uint32_t mine_e;
    float weight;
    mr_route<NV>(z, P.route.correction, P.route.total, P.route.top, P.route.scale, lane, mine_e, weight);
    if (lane < P.route.top) {
        const size_t slot = (size_t)row * P.route.top + lane;
        P.route.weights[slot] = weight;
        P.route.rank[slot] = mine_e;
    }
}

// The gather of few pairs: a pair's place is the number of pairs with a smaller expert, or the same one and a smaller index;
// every block counts for its eight pairs, the first one also makes the group offsets.
template <typename V>
__global__ void __launch_bounds__(256)
experts_gather_few_kernel(const V* __restrict__ h, V* __restrict__ out, uint32_t* __restrict__ place, const uint32_t* __restrict__ ids,
                          uint32_t* __restrict__ offsets, uint32_t pairs, uint32_t top, uint32_t experts, uint32_t words) {
    __shared__ uint32_t before[8][8], hist[kMaxExperts], first[kMaxExperts + 1];
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, pair0 = blockIdx.x * 8;
    uint32_t mine[8], count[8];
#pragma unroll
    for (uint32_t i = 0; i < 8; ++i) { mine[i] = pair0 + i < pairs ? ids[pair0 + i] : 0u; count[i] = 0; }
    const bool lists = blockIdx.x == 0;
    if (lists) {
        for (uint32_t e = threadIdx.x; e < experts; e += 256) hist[e] = 0;
        __syncthreads();
    }
    for (uint32_t p = threadIdx.x; p < pairs; p += 256) {
        const uint32_t e = ids[p];
        if (lists && e < experts) atomicAdd(hist + e, 1u);
#pragma unroll
        for (uint32_t i = 0; i < 8; ++i) count[i] += e < mine[i] || (e == mine[i] && p < pair0 + i) ? 1u : 0u;
    }
#pragma unroll
    for (uint32_t i = 0; i < 8; ++i) {
        count[i] = __reduce_add_sync(0xffffffffu, count[i]);
        if (lane == 0) before[warp][i] = count[i];
    }
    __syncthreads();
    if (lists) {
        if (warp == 0) mr_scan(hist, first, experts, lane);
        __syncthreads();
        for (uint32_t e = threadIdx.x; e <= experts; e += 256) offsets[e] = first[e];
    }
    const uint32_t pair = pair0 + warp;
    if (pair >= pairs) return;
    uint32_t at = 0;
#pragma unroll
    for (uint32_t w = 0; w < 8; ++w) at += before[w][warp];
    const bool real = ids[pair] < experts;      // identity experts have the largest ids: they count before nobody real
    if (lane == 0) place[pair] = real ? at : kIdentityPlace;
    if (!real) return;
    const V* src = h + (size_t)(pair / top) * words;
    V* dst = out + (size_t)at * words;
    for (uint32_t c = lane; c < words; c += 32) dst[c] = src[c];
}

// One block per row.  VEC: four columns per access, the row in registers up to 4 * 256 * EC_KEEP columns.
constexpr uint32_t EC_THREADS = 256;
constexpr int EC_KEEP = 4;

template <typename T, bool VEC>
__global__ void __launch_bounds__(EC_THREADS)
experts_combine_kernel(float* __restrict__ x, const T* __restrict__ y, const T* h, const uint32_t* __restrict__ place,
                       const float* __restrict__ weights, const float* __restrict__ layer_scale, const float* __restrict__ norm_w, T* norm_out,
                       uint32_t pairs, uint32_t top, uint32_t d, float norm_offset, float eps) {
    __shared__ uint32_t s_place[kMaxTop];
    __shared__ float s_weight[kMaxTop], red[EC_THREADS / 32];
    pdl_wait();
    pdl_trigger();
    const size_t row = blockIdx.x;
    if (threadIdx.x < top) {
        s_place[threadIdx.x] = place[row * top + threadIdx.x];
        s_weight[threadIdx.x] = weights[row * top + threadIdx.x];
    }
    __syncthreads();
    float* xr = x + row * d;
    const T* hr = h + row * d;
    float ss = 0.0f;
    constexpr int W = VEC ? 4 : 1, KEEP = VEC ? EC_KEEP : 1;
    const uint32_t n = d / W;
    auto load = [&](const T* p, float* v) {
        if (VEC && sizeof(T) == 2) {
            const uint2 q = *reinterpret_cast<const uint2*>(p);
            const float2 a = bf16x2_to_f32(q.x), b = bf16x2_to_f32(q.y);
            v[0] = a.x; v[W > 1 ? 1 : 0] = a.y; v[W > 2 ? 2 : 0] = b.x; v[W > 3 ? 3 : 0] = b.y;
        } else {
#pragma unroll
            for (int i = 0; i < W; ++i) v[i] = to_f32(p[i]);
        }
    };
    // x + scale * sum, columns W c ..
    auto value = [&](uint32_t c, float* v) {
        float acc[W] = {};
        for (uint32_t k = 0; k < top; ++k) {
            const uint32_t at = s_place[k];
            float t[W];
            load(at < pairs ? y + (size_t)at * d + (size_t)c * W : hr + (size_t)c * W, t);
#pragma unroll
            for (int i = 0; i < W; ++i) acc[i] = fmaf(s_weight[k], t[i], acc[i]);
        }
#pragma unroll
        for (int i = 0; i < W; ++i) {
            const float f = layer_scale ? layer_scale[c * W + i] : 1.0f;
            v[i] = fmaf(f, acc[i], xr[c * W + i]);
            ss = fmaf(v[i], v[i], ss);
        }
        if (VEC) *reinterpret_cast<float4*>(xr + c * W) = make_float4(v[0], v[W > 1 ? 1 : 0], v[W > 2 ? 2 : 0], v[W > 3 ? 3 : 0]);
        else xr[c] = v[0];
    };
    float keep[KEEP][W];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const uint32_t c = threadIdx.x + i * EC_THREADS;
        if (c < n) value(c, keep[i]);
    }
    for (uint32_t c = threadIdx.x + KEEP * EC_THREADS; c < n; c += EC_THREADS) { float v[W]; value(c, v); }
    if (!norm_out) return;
    ss = ff_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();      // also: every read of h is done before norm_out (possibly the same row) is written
    float sum = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < EC_THREADS / 32; ++i) sum += red[i];
    const float inv = rsqrtf(sum / (float)d + eps);
    T* o = norm_out + row * d;
    auto put = [&](uint32_t c, const float* v) {
        float r[W];
#pragma unroll
        for (int i = 0; i < W; ++i) r[i] = v[i] * inv * (norm_offset + norm_w[c * W + i]);
        if (VEC && sizeof(T) == 2) *reinterpret_cast<uint2*>(o + c * W) = make_uint2(pack_bf16x2(r[0], r[W > 1 ? 1 : 0]), pack_bf16x2(r[W > 2 ? 2 : 0], r[W > 3 ? 3 : 0]));
        else {
#pragma unroll
            for (int i = 0; i < W; ++i) o[c * W + i] = from_f32<T>(r[i]);
        }
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const uint32_t c = threadIdx.x + i * EC_THREADS;
        if (c < n) put(c, keep[i]);
    }
    for (uint32_t c = threadIdx.x + KEEP * EC_THREADS; c < n; c += EC_THREADS) {
        float v[W];
#pragma unroll
        for (int i = 0; i < W; ++i) v[i] = xr[c * W + i];      // written by this thread above
        put(c, v);
    }
}

// Many rows of at most 1024 columns: a warp per row.
template <typename T>
__global__ void __launch_bounds__(128)
experts_combine_warp_kernel(float* __restrict__ x, const T* __restrict__ y, const T* h, const uint32_t* __restrict__ place,
                            const float* __restrict__ weights, const float* __restrict__ layer_scale, const float* __restrict__ norm_w, T* norm_out,
                            uint32_t rows, uint32_t top, uint32_t d, float norm_offset, float eps) {
    constexpr int KEEP = 8;
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, row = blockIdx.x * 4 + (threadIdx.x >> 5), n = d / 4, pairs = rows * top;
    if (row >= rows) return;
    auto load = [&](const T* p) {
        if (sizeof(T) == 2) {
            const uint2 q = *reinterpret_cast<const uint2*>(p);
            const float2 a = bf16x2_to_f32(q.x), b = bf16x2_to_f32(q.y);
            return make_float4(a.x, a.y, b.x, b.y);
        }
        return *reinterpret_cast<const float4*>(p);
    };
    const uint32_t my_place = lane < top ? place[(size_t)row * top + lane] : 0u;
    const float my_weight = lane < top ? weights[(size_t)row * top + lane] : 0.0f;
    float4* xr = reinterpret_cast<float4*>(x + (size_t)row * d);
    float4 v[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) v[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    for (uint32_t k = 0; k < top; ++k) {
        const uint32_t at = __shfl_sync(0xffffffffu, my_place, k);
        const float w = __shfl_sync(0xffffffffu, my_weight, k);
        const T* src = at < pairs ? y + (size_t)at * d : h + (size_t)row * d;
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
            const uint32_t c = lane + 32 * i;
            if (c >= n) continue;
            const float4 t = load(src + 4 * c);
            v[i] = make_float4(fmaf(w, t.x, v[i].x), fmaf(w, t.y, v[i].y), fmaf(w, t.z, v[i].z), fmaf(w, t.w, v[i].w));
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const uint32_t c = lane + 32 * i;
        if (c >= n) continue;
        const float4 f = layer_scale ? reinterpret_cast<const float4*>(layer_scale)[c] : make_float4(1.0f, 1.0f, 1.0f, 1.0f), old = xr[c];
        v[i] = make_float4(fmaf(f.x, v[i].x, old.x), fmaf(f.y, v[i].y, old.y), fmaf(f.z, v[i].z, old.z), fmaf(f.w, v[i].w, old.w));
        xr[c] = v[i];
        ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
    }
    if (!norm_out) return;
    const float inv = rsqrtf(ff_warp_sum(ss) / (float)d + eps);      // behind it every lane has read its part of h
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const uint32_t c = lane + 32 * i;
        if (c >= n) continue;
        const float4 w = reinterpret_cast<const float4*>(norm_w)[c];
        const float4 r = make_float4(v[i].x * inv * (norm_offset + w.x), v[i].y * inv * (norm_offset + w.y), v[i].z * inv * (norm_offset + w.z),
                                     v[i].w * inv * (norm_offset + w.w));
        T* o = norm_out + (size_t)row * d + 4 * c;
        if (sizeof(T) == 2) *reinterpret_cast<uint2*>(o) = make_uint2(pack_bf16x2(r.x, r.y), pack_bf16x2(r.z, r.w));
        else *reinterpret_cast<float4*>(o) = r;
    }
}

namespace {

struct ExpertsLayout {
    uint64_t weights, place, rank, counts, offsets, rows_in, hidden, rows_out, bytes;
};
ExpertsLayout experts_layout(uint64_t rows, uint64_t d, uint64_t ff, uint64_t experts, uint64_t top, int dtype) {
    const uint64_t e = dtype == TNSR_B200_BF16 ? 2 : 4, pairs = rows * top, blocks = ceil_div64(rows, MR_ROWS);
    ExpertsLayout L;
    uint64_t at = 0;
    auto take = [&](uint64_t bytes) { const uint64_t p = at; at += (bytes + 255) / 256 * 256; return p; };
    L.weights = take(pairs * 4);
    L.place = take(pairs * 4);
    L.rank = take(pairs * 4);
    L.counts = take(blocks * experts * 4);
    L.offsets = take((experts + 1) * 4);
    L.rows_in = take(pairs * d * e);
    L.hidden = take(pairs * ff * e);
    L.rows_out = take(pairs * d * e);
    L.bytes = at;
    return L;
}

int experts_fail(const char* m, int code) {
    set_thread_error(m);
    return code;
}

}  // namespace

uint64_t experts_workspace_bytes(uint32_t rows, uint32_t d, uint32_t ff, uint32_t experts, uint32_t top, int dtype) {
    return experts_layout(rows, d, ff, experts, top, dtype).bytes;
}

// Most pairs of a step whose gather counts places itself.
constexpr uint32_t EX_FEW_PAIRS = 8192;

bool experts_fused_router(const Experts& E) {
    return E.router && (uint64_t)E.rows * E.top <= EX_FEW_PAIRS && E.d <= 8192 && !E.chosen && !E.weights;
}

int launch_experts(const Experts& E, int dtype, cudaStream_t stream) {
    const uint32_t total = E.experts + E.identity;
    if (E.experts == 0 || total > kMaxExperts || E.top == 0 || E.top > kMaxTop || E.top > total)
        return experts_fail("experts: 1..1024 experts, at most 32 of them chosen", TNSR_B200_ERR_UNSUPPORTED);
    if (E.rows == 0) return TNSR_B200_OK;
    const uint64_t pairs = (uint64_t)E.rows * E.top;
    if (pairs > 0x7fffffffull) return experts_fail("experts: too many rows for one launch", TNSR_B200_ERR_UNSUPPORTED);
    const ExpertsLayout L = experts_layout(E.rows, E.d, E.ff, E.experts, E.top, dtype);
    if (!E.workspace || E.workspace_bytes < L.bytes || reinterpret_cast<uintptr_t>(E.workspace) % 256)
        return experts_fail("experts: workspace too small or not aligned", TNSR_B200_ERR_INVALID_ARGUMENT);
    uint8_t* ws = (uint8_t*)E.workspace;
    const bool bf = dtype == TNSR_B200_BF16;
    RouteParams R;
    R.logits = E.logits; R.correction = E.correction; R.rows = E.rows; R.logits_ld = E.logits_ld; R.experts = E.experts; R.total = total;
    R.top = E.top; R.scale = E.router_scale;
    R.weights = (float*)(ws + L.weights); R.place = (uint32_t*)(ws + L.place); R.rank = (uint32_t*)(ws + L.rank);
    R.counts = (uint32_t*)(ws + L.counts); R.offsets = (uint32_t*)(ws + L.offsets);
    R.chosen = E.chosen; R.weights_out = E.weights;
    const size_t row_bytes = E.d * (bf ? 2 : 4);
    const dim3 pair_grid((uint32_t)ceil_div64(pairs, 8));
    const bool wide_rows = row_bytes % 16 == 0 && reinterpret_cast<uintptr_t>(E.h) % 16 == 0;
    int rc;
    if (E.router) {
        if (!experts_fused_router(E)) return experts_fail("experts: the step has too many rows for the fused router", TNSR_B200_ERR_UNSUPPORTED);
        ChooseParams P;
        P.x = E.x; P.partials = E.partials; P.parts = E.parts; P.split_rows = E.split_rows; P.norm_w = E.router_norm; P.norm_offset = E.norm_offset;
        P.eps = E.eps; P.h = const_cast<void*>(E.h); P.router = E.router; P.route = R; P.d = E.d;
        const size_t smem = E.d * sizeof(float);
        auto choose = [&](auto kernel) { launch_kernel(kernel, dim3(E.rows), dim3(EX_THREADS), smem, stream, P); };
        if (bf) {
            if (total <= 64) choose(experts_choose_kernel<bf16, 2>);
            else if (total <= 256) choose(experts_choose_kernel<bf16, 8>);
            else choose(experts_choose_kernel<bf16, 32>);
        } else {
            if (total <= 64) choose(experts_choose_kernel<float, 2>);
            else if (total <= 256) choose(experts_choose_kernel<float, 8>);
            else choose(experts_choose_kernel<float, 32>);
        }
        count_launch();
        if ((rc = check_launch("experts_choose"))) return rc;
        if (wide_rows)
            launch_kernel(experts_gather_few_kernel<uint4>, pair_grid, dim3(256), 0, stream, (const uint4*)E.h, (uint4*)(ws + L.rows_in), R.place, R.rank,
                          R.offsets, (uint32_t)pairs, E.top, E.experts, (uint32_t)(row_bytes / 16));
        else
            launch_kernel(experts_gather_few_kernel<uint16_t>, pair_grid, dim3(256), 0, stream, (const uint16_t*)E.h, (uint16_t*)(ws + L.rows_in), R.place,
                          R.rank, R.offsets, (uint32_t)pairs, E.top, E.experts, (uint32_t)(row_bytes / 2));
    } else {
        const uint32_t blocks = ceil_div(E.rows, MR_ROWS);
        if (total <= 64) launch_kernel(experts_route_kernel<2>, dim3(blocks), dim3(MR_THREADS), 0, stream, R);
        else if (total <= 256) launch_kernel(experts_route_kernel<8>, dim3(blocks), dim3(MR_THREADS), 0, stream, R);
        else launch_kernel(experts_route_kernel<32>, dim3(blocks), dim3(MR_THREADS), 0, stream, R);
        count_launch();
        if ((rc = check_launch("experts_route"))) return rc;
        if (blocks > 1) {
            launch_kernel(experts_offsets_kernel, dim3(1), dim3(MR_THREADS), 0, stream, R.counts, R.offsets, blocks, E.experts);
            count_launch();
            if ((rc = check_launch("experts_offsets"))) return rc;
        }
        if (wide_rows)
            launch_kernel(experts_gather_kernel<uint4>, pair_grid, dim3(256), 0, stream, (const uint4*)E.h, (uint4*)(ws + L.rows_in), R.place, R.rank, R.counts,
                          (uint32_t)pairs, E.top, E.experts, (uint32_t)(row_bytes / 16));
        else
            launch_kernel(experts_gather_kernel<uint16_t>, pair_grid, dim3(256), 0, stream, (const uint16_t*)E.h, (uint16_t*)(ws + L.rows_in), R.place, R.rank,
                          R.counts, (uint32_t)pairs, E.top, E.experts, (uint32_t)(row_bytes / 2));
    }
    count_launch();
    if ((rc = check_launch("experts_gather"))) return rc;
    GroupedGemm g;
    g.a = ws + L.rows_in; g.w = E.up; g.out = ws + L.hidden; g.offsets = R.offsets; g.groups = E.experts; g.rows = (uint32_t)pairs;
    g.n = E.ff; g.k = E.d; g.activation = ACT_RELU_SQUARED; g.out_dtype = dtype; g.d_status = E.d_status; g.engine = E.engine;
    if ((rc = launch_gemm_grouped(g, dtype, stream))) return rc;
    g.a = ws + L.hidden; g.w = E.down; g.out = ws + L.rows_out; g.n = E.d; g.k = E.ff; g.activation = ACT_NONE;
    return launch_gemm_grouped(g, dtype, stream);
}

int launch_experts_combine(const Experts& E, int dtype, cudaStream_t stream) {
    if (E.rows == 0) return TNSR_B200_OK;
    const ExpertsLayout L = experts_layout(E.rows, E.d, E.ff, E.experts, E.top, dtype);
    const uint8_t* ws = (const uint8_t*)E.workspace;
    const uint32_t* place = (const uint32_t*)(ws + L.place);
    const float* weights = (const float*)(ws + L.weights);
    const uint32_t pairs = E.rows * E.top;
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool vec = E.d % 4 == 0 && aligned(E.x) && aligned(E.h) && aligned(E.norm_out) && aligned(E.layer_scale) && aligned(E.norm_w);
    if (vec && E.d <= 1024 && E.rows >= 2048) {
        const dim3 grid(ceil_div(E.rows, 4u)), block(128);
        if (dtype == TNSR_B200_BF16)
            launch_kernel(experts_combine_warp_kernel<bf16>, grid, block, 0, stream, E.x, (const bf16*)(ws + L.rows_out), (const bf16*)E.h, place, weights,
                          E.layer_scale, E.norm_w, (bf16*)E.norm_out, E.rows, E.top, E.d, E.norm_offset, E.eps);
        else
            launch_kernel(experts_combine_warp_kernel<float>, grid, block, 0, stream, E.x, (const float*)(ws + L.rows_out), (const float*)E.h, place, weights,
                          E.layer_scale, E.norm_w, (float*)E.norm_out, E.rows, E.top, E.d, E.norm_offset, E.eps);
    } else if (dtype == TNSR_B200_BF16 && vec)
        launch_kernel(experts_combine_kernel<bf16, true>, dim3(E.rows), dim3(EC_THREADS), 0, stream, E.x, (const bf16*)(ws + L.rows_out), (const bf16*)E.h,
                      place, weights, E.layer_scale, E.norm_w, (bf16*)E.norm_out, pairs, E.top, E.d, E.norm_offset, E.eps);
    else if (dtype == TNSR_B200_BF16)
        launch_kernel(experts_combine_kernel<bf16, false>, dim3(E.rows), dim3(EC_THREADS), 0, stream, E.x, (const bf16*)(ws + L.rows_out), (const bf16*)E.h,
                      place, weights, E.layer_scale, E.norm_w, (bf16*)E.norm_out, pairs, E.top, E.d, E.norm_offset, E.eps);
    else if (vec)
        launch_kernel(experts_combine_kernel<float, true>, dim3(E.rows), dim3(EC_THREADS), 0, stream, E.x, (const float*)(ws + L.rows_out), (const float*)E.h,
                      place, weights, E.layer_scale, E.norm_w, (float*)E.norm_out, pairs, E.top, E.d, E.norm_offset, E.eps);
    else
        launch_kernel(experts_combine_kernel<float, false>, dim3(E.rows), dim3(EC_THREADS), 0, stream, E.x, (const float*)(ws + L.rows_out), (const float*)E.h,
                      place, weights, E.layer_scale, E.norm_w, (float*)E.norm_out, pairs, E.top, E.d, E.norm_offset, E.eps);
    count_launch();
    return check_launch("experts_combine");
}

}  // namespace tb
