// The recurrent block with a real-gated linear recurrent unit, between its projections:
//     u = conv(x),  r = sigmoid(R u + b),  i = sigmoid(I u + b)   (block-diagonal R, I)
//     log a = -8 r softplus(lambda),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S y
//
// The convolution writes u in the layout [blocks][rows][part], in which the gates are one grouped product with a [2 part,
// part] matrix per block (r rows, then i rows), f32 out.
//  * rglru_scan_kernel   many tokens: a block owns a strip of channels of one session; its 16 warps take consecutive
//                        segments of 8 tokens each, which are scanned side by side from zero, joined through shared memory
//                        (each segment is S -> A S + H) and finished from registers: every value is read once.
//  * rglru_fused_step_kernel  single-token steps, bf16, parts of a multiple of 32 channels up to 256: convolution, both gates
//                        and the recurrence of a part for 16 sessions in one block.  The gates of a part need its own
//                        channels only, so nothing passes between blocks.
//  * rglru_step_kernel   the recurrence of the other single-token steps.
// Gates, decays and the state are f32 in both precisions; 1 - a^2 is formed as -expm1(2 log a).
#include <algorithm>

#include "feed_forward.cuh"
#include "mixers.cuh"

namespace tb {

__device__ __forceinline__ float rg_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

constexpr float RG_LOG2E = 1.4426950408889634f;
struct RgChannel { float r_bias, i_bias, rate; };      // rate = -8 softplus(lambda)
__device__ __forceinline__ RgChannel rg_channel(const Rglru& m, uint32_t c) { return {m.r_bias[c], m.i_bias[c], -8.0f * softplus(m.lambda[c])}; }
// One token: decay a and what is written, b.
template <typename T>
__device__ __forceinline__ void rg_token(const RgChannel& ch, float r_raw, float i_raw, float u, float& a, float& b);
// The bf16 path: exponentials, reciprocals and roots of the special-function unit, all in f32.  1 - a^2 loses its digits as a
// comes close to one; for t = -2 log a below 1/4 it is 1 - exp(-t) by its Taylor series (next term below 2e-6 of it).
template <>
__device__ __forceinline__ void rg_token<bf16>(const RgChannel& ch, float r_raw, float i_raw, float u, float& a, float& b) {
    const float r = mx_rcp(1.0f + mx_ex2(-RG_LOG2E * (r_raw + ch.r_bias))), i = mx_rcp(1.0f + mx_ex2(-RG_LOG2E * (i_raw + ch.i_bias)));
    const float log_a = r * ch.rate, t = -2.0f * log_a;
    a = mx_ex2(RG_LOG2E * log_a);
    const float series = t * fmaf(t, fmaf(t, fmaf(t, fmaf(t, 1.0f / 120.0f, -1.0f / 24.0f), 1.0f / 6.0f), -0.5f), 1.0f);
    const float w = t < 0.25f ? series : fmaf(-a, a, 1.0f);
    float root;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(w));
    b = root * i * u;
}
template <>
__device__ __forceinline__ void rg_token<float>(const RgChannel& ch, float r_raw, float i_raw, float u, float& a, float& b) {
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
                if (first + i < place.chunk) rg_token<T>(ch[e], a[i][e], b[i][e], uu[i][e], a[i][e], b[i][e]);
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
    rg_token<T>(rg_channel(m, c), r, i, u, a, b);
    const float S = fmaf(a, place.pos(s) > 0 ? old : 0.0f, b);
    m.state[(size_t)s * m.width + c] = S;
    out[c] = from_f32<T>(S * y);
}

// Block = (part, 16 sessions).  u of the part goes to shared memory in bf16 and is the A operand of mma.sync; the gate matrix
// is read from global memory as its B operand.  Of every 32 k values a lane loads eight consecutive ones (16 bytes): both
// operands use the same order of k, so the sum does not notice.
constexpr uint32_t RF_SESSIONS = 16, RF_MAX_PART = 256;
__global__ void __launch_bounds__(256)
rglru_fused_step_kernel(Rglru m, StepPlace place) {
    constexpr uint32_t PITCH = RF_MAX_PART + 8;                 // elements
    __shared__ __align__(16) bf16 su[RF_SESSIONS * PITCH];
    pdl_wait();
    pdl_trigger();
    const uint32_t part = m.width / m.blocks, blk = blockIdx.x, c_first = blk * part, s0 = blockIdx.y * RF_SESSIONS;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
    const bf16* proj = reinterpret_cast<const bf16*>(m.proj);
    bf16* ring = reinterpret_cast<bf16*>(m.ring);
    // ---- convolution of two neighbouring channels per thread and turn; the slot of this position held the oldest row ----
    for (uint32_t i = threadIdx.x; i < RF_SESSIONS * part / 2; i += 256) {
        const uint32_t r = i / (part / 2), c = i % (part / 2) * 2, ch = c_first + c, s = s0 + r;
        float2 y = make_float2(0.0f, 0.0f);
        if (s < place.sessions) {
            const uint32_t pos = place.pos(s);
            const uint32_t now = *reinterpret_cast<const uint32_t*>(proj + (size_t)s * m.ld + m.x_col + ch);
            uint32_t* slots = reinterpret_cast<uint32_t*>(ring + (size_t)s * m.taps * m.width + ch);
            const float *w0 = m.conv_w + (size_t)ch * m.taps, *w1 = w0 + m.taps;
            y = make_float2(m.conv_b[ch], m.conv_b[ch + 1]);
            for (uint32_t j = 0; j < m.taps; ++j) {
                const uint32_t lag = m.taps - 1 - j;
                const uint32_t q = lag == 0 ? now : pos >= lag ? slots[(size_t)((pos - lag) % m.taps) * (m.width / 2)] : 0u;
                const float2 v = bf16x2_to_f32(q);
                y.x = fmaf(w0[j], v.x, y.x);
                y.y = fmaf(w1[j], v.y, y.y);
            }
            slots[(size_t)(pos % m.taps) * (m.width / 2)] = now;
        }
        *reinterpret_cast<uint32_t*>(su + r * PITCH + c) = pack_bf16x2(y.x, y.y);
    }
    __syncthreads();
    // ---- gates and recurrence, eight channels per warp and turn ----
    const bf16* w = reinterpret_cast<const bf16*>(m.gate_w) + (size_t)blk * 2 * part * part;
    for (uint32_t n0 = warp * 8; n0 < part; n0 += 64) {
        float gr[4] = {0.0f, 0.0f, 0.0f, 0.0f}, gi[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        const bf16 *wr = w + (size_t)(n0 + g8) * part + t4 * 8, *wi = wr + (size_t)part * part;
#pragma unroll 4
        for (uint32_t k0 = 0; k0 < part; k0 += 32) {
            const uint4 br = __ldg(reinterpret_cast<const uint4*>(wr + k0)), bi = __ldg(reinterpret_cast<const uint4*>(wi + k0));
            const uint4 lo = *reinterpret_cast<const uint4*>(su + g8 * PITCH + k0 + t4 * 8), hi = *reinterpret_cast<const uint4*>(su + (g8 + 8) * PITCH + k0 + t4 * 8);
            const uint32_t a0[4] = {lo.x, hi.x, lo.y, hi.y}, a1[4] = {lo.z, hi.z, lo.w, hi.w};
            mx_mma(gr, a0, br.x, br.y);
            mx_mma(gi, a0, bi.x, bi.y);
            mx_mma(gr, a1, br.z, br.w);
            mx_mma(gi, a1, bi.z, bi.w);
        }
        const uint32_t c = n0 + t4 * 2, ch = c_first + c;
        const RgChannel ca = rg_channel(m, ch), cb = rg_channel(m, ch + 1);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const uint32_t r = g8 + half * 8, s = s0 + r;
            if (s >= place.sessions) continue;
            float2* state = reinterpret_cast<float2*>(m.state + (size_t)s * m.width + ch);
            const float2 old = place.pos(s) > 0 ? *state : make_float2(0.0f, 0.0f);
            const float2 y = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(proj + (size_t)s * m.ld + ch));
            const float2 u = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(su + r * PITCH + c));
            float a, b;
            float2 S;
            rg_token<bf16>(ca, gr[2 * half], gi[2 * half], u.x, a, b);
            S.x = fmaf(a, old.x, b);
            rg_token<bf16>(cb, gr[2 * half + 1], gi[2 * half + 1], u.y, a, b);
            S.y = fmaf(a, old.y, b);
            *state = S;
            *reinterpret_cast<uint32_t*>(reinterpret_cast<bf16*>(m.out) + (size_t)s * m.out_ld + ch) = pack_bf16x2(S.x * y.x, S.y * y.y);
        }
    }
    if (blk == 0 && m.out_cols > m.width) {
        const uint32_t pad = m.out_cols - m.width;
        for (uint32_t i = threadIdx.x; i < pad * RF_SESSIONS; i += 256) {
            const uint32_t s = s0 + i / pad;
            if (s < place.sessions) reinterpret_cast<bf16*>(m.out)[(size_t)s * m.out_ld + m.width + i % pad] = __float2bfloat16_rn(0.0f);
        }
    }
}

static bool rglru_fused_fits(const Rglru& m) {
    auto aligned = [](const void* p, uint32_t to) { return reinterpret_cast<uintptr_t>(p) % to == 0; };
    const uint32_t part = m.width / m.blocks;
    return part % 32 == 0 && part <= RF_MAX_PART && m.taps >= 1 && m.taps <= kMaxConvTaps && m.x_col % 2 == 0 && m.ld % 2 == 0 && m.out_ld % 2 == 0 &&
           aligned(m.proj, 4) && aligned(m.ring, 4) && aligned(m.out, 4) && aligned(m.state, 8) && aligned(m.gate_w, 16);
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
    if (bf && place.chunk == 1 && rglru_fused_fits(m)) {
        launch_kernel(rglru_fused_step_kernel, dim3(m.blocks, ceil_div(place.sessions, RF_SESSIONS)), dim3(256), 0, stream, m, place);
        count_launch();
        return check_launch("rglru_fused_step");
    }
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
