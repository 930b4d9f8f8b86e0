// The recurrent block with a real-gated linear recurrent unit, between its projections:
//     u = conv(x),  r = sigmoid(R u + b),  i = sigmoid(I u + b)   (block-diagonal R, I)
//     log a = -8 r softplus(lambda),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S y
//
// The convolution writes u in the layout [blocks][rows][part], in which the gates are one grouped product with a [2 part,
// part] matrix per block (r rows, then i rows), f32 out.
//  * rglru_scan_kernel   many tokens: a block owns a strip of channels of one session; its 16 warps take consecutive
//                        segments of 8 tokens each, which are scanned side by side from zero, joined through shared memory
//                        (each segment is S -> A S + H) and finished from registers: every value is read once.
//  * rglru_step_kernel   single-token steps.
// Gates, decays and the state are f32 in both precisions; 1 - a^2 is formed as -expm1(2 log a).
#include <algorithm>

#include "feed_forward.cuh"
#include "mixers.cuh"

namespace tb {

__device__ __forceinline__ float rg_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

struct RgChannel { float r_bias, i_bias, rate; };      // rate = -8 softplus(lambda)
__device__ __forceinline__ RgChannel rg_channel(const Rglru& m, uint32_t c) { return {m.r_bias[c], m.i_bias[c], -8.0f * softplus(m.lambda[c])}; }
// One token: decay a and what is written, b.
__device__ __forceinline__ void rg_token(const RgChannel& ch, float r_raw, float i_raw, float u, float& a, float& b) {
    const float log_a = rg_sigmoid(r_raw + ch.r_bias) * ch.rate;
    a = expf(log_a);
    b = sqrtf(-expm1f(2.0f * log_a)) * rg_sigmoid(i_raw + ch.i_bias) * u;
}

constexpr uint32_t RG_WARPS = 16, RG_SEG = 8;

// VEC channels per lane (two when parts, pitches and pointers are even).
template <typename T, int VEC>
__global__ void __launch_bounds__(RG_WARPS * 32)
rglru_scan_kernel(Rglru m, StepPlace place) {
    constexpr uint32_t STRIP = 32 * VEC;
    __shared__ float seg_a[2][RG_WARPS][STRIP], seg_h[2][RG_WARPS][STRIP];
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, s = blockIdx.y;
    const uint32_t c = blockIdx.x * STRIP + lane * VEC;
    const bool live = c < m.width;
    const uint32_t part = m.width / m.blocks, rows = place.sessions * place.chunk;
    const uint32_t cc = live ? c : 0, blk = cc / part, local = cc % part;
    const size_t row0 = (size_t)s * place.chunk;
    const float* gates = m.gates + ((size_t)blk * rows + row0) * 2 * part + local;
    const T* u = reinterpret_cast<const T*>(m.u) + ((size_t)blk * rows + row0) * part + local;
    const T* y = reinterpret_cast<const T*>(m.proj) + row0 * m.ld + cc;
    T* out = reinterpret_cast<T*>(m.out) + row0 * m.out_ld + cc;
    RgChannel ch[VEC];
    float carry[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        ch[e] = rg_channel(m, cc + e);
        carry[e] = place.pos(s) > 0 ? m.state[(size_t)s * m.width + cc + e] : 0.0f;
    }
    uint32_t buf = 0;
    for (uint32_t t0 = 0; t0 < place.chunk; t0 += RG_WARPS * RG_SEG, buf ^= 1) {
        const uint32_t first = t0 + warp * RG_SEG;
        float a[RG_SEG][VEC], b[RG_SEG][VEC], yy[RG_SEG][VEC], uu[RG_SEG][VEC];
#pragma unroll
        for (uint32_t i = 0; i < RG_SEG; ++i) {
            const uint32_t t = first + i;
            const bool here = live && t < place.chunk;
            if (VEC == 2) {
                const float2 z = make_float2(0.0f, 0.0f);
                const float2 r = here ? *reinterpret_cast<const float2*>(gates + (size_t)t * 2 * part) : z;
                const float2 g = here ? *reinterpret_cast<const float2*>(gates + (size_t)t * 2 * part + part) : z;
                const float2 uv = here ? load_pair<T>(u + (size_t)t * part, true, true) : z, yv = here ? load_pair<T>(y + (size_t)t * m.ld, true, true) : z;
                a[i][0] = r.x; a[i][VEC - 1] = r.y; b[i][0] = g.x; b[i][VEC - 1] = g.y;
                uu[i][0] = uv.x; uu[i][VEC - 1] = uv.y; yy[i][0] = yv.x; yy[i][VEC - 1] = yv.y;
            } else {
                a[i][0] = here ? gates[(size_t)t * 2 * part] : 0.0f;
                b[i][0] = here ? gates[(size_t)t * 2 * part + part] : 0.0f;
                uu[i][0] = here ? to_f32(u[(size_t)t * part]) : 0.0f;
                yy[i][0] = here ? to_f32(y[(size_t)t * m.ld]) : 0.0f;
            }
        }
        float A[VEC], H[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) { A[e] = 1.0f; H[e] = 0.0f; }
#pragma unroll
        for (uint32_t i = 0; i < RG_SEG; ++i)
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                if (first + i < place.chunk) rg_token(ch[e], a[i][e], b[i][e], uu[i][e], a[i][e], b[i][e]);
                else { a[i][e] = 1.0f; b[i][e] = 0.0f; }
                A[e] *= a[i][e];
                H[e] = fmaf(a[i][e], H[e], b[i][e]);
            }
#pragma unroll
        for (int e = 0; e < VEC; ++e) { seg_a[buf][warp][lane * VEC + e] = A[e]; seg_h[buf][warp][lane * VEC + e] = H[e]; }
        __syncthreads();       // the other buffer is rewritten only after the next barrier
        float S[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float x = carry[e];
            S[e] = x;
#pragma unroll
            for (uint32_t w = 0; w < RG_WARPS; ++w) {
                if (w == warp) S[e] = x;
                x = fmaf(seg_a[buf][w][lane * VEC + e], x, seg_h[buf][w][lane * VEC + e]);
            }
            carry[e] = x;
        }
#pragma unroll
        for (uint32_t i = 0; i < RG_SEG; ++i) {
            const uint32_t t = first + i;
            float o[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) { S[e] = fmaf(a[i][e], S[e], b[i][e]); o[e] = S[e] * yy[i][e]; }
            if (!live || t >= place.chunk) continue;
            if (VEC == 2) store_pair<T>(out + (size_t)t * m.out_ld, make_float2(o[0], o[VEC - 1]), true, true);
            else out[(size_t)t * m.out_ld] = from_f32<T>(o[0]);
        }
    }
    if (warp == 0 && live)
#pragma unroll
        for (int e = 0; e < VEC; ++e) m.state[(size_t)s * m.width + c + e] = carry[e];
    if (blockIdx.x == 0 && m.out_cols > m.width) {
        const uint32_t pad = m.out_cols - m.width;
        for (uint64_t i = threadIdx.x; i < (uint64_t)pad * place.chunk; i += blockDim.x)
            reinterpret_cast<T*>(m.out)[(row0 + i / pad) * m.out_ld + m.width + i % pad] = from_f32<T>(0.0f);
    }
}

// A thread per (session, channel); channels past the width zero the padding of the output row.
template <typename T>
__global__ void __launch_bounds__(128)
rglru_step_kernel(Rglru m, StepPlace place) {
    pdl_wait();
    pdl_trigger();
    const uint32_t c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
    if (c >= m.out_cols) return;
    T* out = reinterpret_cast<T*>(m.out) + (size_t)s * m.out_ld;
    if (c >= m.width) { out[c] = from_f32<T>(0.0f); return; }
    const uint32_t part = m.width / m.blocks, blk = c / part, local = c % part;
    const size_t at = (size_t)blk * place.sessions + s;
    const float old = m.state[(size_t)s * m.width + c];
    const float r = m.gates[at * 2 * part + local], i = m.gates[at * 2 * part + part + local];
    const float u = to_f32(reinterpret_cast<const T*>(m.u)[at * part + local]), y = to_f32(reinterpret_cast<const T*>(m.proj)[(size_t)s * m.ld + c]);
    float a, b;
    rg_token(rg_channel(m, c), r, i, u, a, b);
    const float S = fmaf(a, place.pos(s) > 0 ? old : 0.0f, b);
    m.state[(size_t)s * m.width + c] = S;
    out[c] = from_f32<T>(S * y);
}

template <typename T>
static void rglru_typed(const Rglru& m, const StepPlace& place, cudaStream_t stream) {
    if (place.chunk == 1) {
        launch_kernel(rglru_step_kernel<T>, dim3(ceil_div(m.out_cols, 128u), place.sessions), dim3(128), 0, stream, m, place);
        return;
    }
    auto even = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % (2 * sizeof(T)) == 0; };
    const uint32_t part = m.width / m.blocks;
    const bool pairs = part % 2 == 0 && m.ld % 2 == 0 && m.out_ld % 2 == 0 && even(m.proj) && even(m.u) && even(m.out) &&
                       reinterpret_cast<uintptr_t>(m.gates) % 8 == 0;
    if (pairs) launch_kernel(rglru_scan_kernel<T, 2>, dim3(ceil_div(m.width, 64u), place.sessions), dim3(RG_WARPS * 32), 0, stream, m, place);
    else launch_kernel(rglru_scan_kernel<T, 1>, dim3(ceil_div(m.width, 32u), place.sessions), dim3(RG_WARPS * 32), 0, stream, m, place);
}

int launch_rglru(const Rglru& m, const StepPlace& place, int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    if (m.width == 0 || m.blocks == 0 || m.width % m.blocks || m.out_cols < m.width || place.sessions > 65535u) {
        set_thread_error("rglru: blocks must divide the width, at most 65535 sessions");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    const bool bf = dtype == TNSR_B200_BF16;
    const uint32_t part = m.width / m.blocks, rows = place.sessions * place.chunk;
    ShortConv c;
    c.rows = (const uint8_t*)m.proj + (size_t)m.x_col * (bf ? 2 : 4);
    c.ld = m.ld; c.channels = m.width; c.part = part; c.taps = m.taps; c.w = m.conv_w; c.b = m.conv_b; c.ring = m.ring; c.out = m.u;
    int rc;
    if ((rc = launch_short_conv(c, place, dtype, stream))) return rc;
    if ((uint64_t)m.blocks * rows > 0x7fffffffull) { set_thread_error("rglru: too many rows for one launch"); return TNSR_B200_ERR_UNSUPPORTED; }
    GroupedGemm g;
    g.a = m.u; g.w = m.gate_w; g.out = m.gates; g.groups = m.blocks; g.rows = m.blocks * rows; g.n = 2 * part; g.k = part;
    g.out_dtype = TNSR_B200_F32; g.d_status = m.d_status;
    if ((rc = launch_gemm_grouped(g, dtype, stream))) return rc;
    if (bf) rglru_typed<bf16>(m, place, stream); else rglru_typed<float>(m, place, stream);
    count_launch();
    return check_launch("rglru");
}

}  // namespace tb
