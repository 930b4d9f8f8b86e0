// The recurrent block with a real-gated linear recurrent unit, between its projections:
//     u = conv(x),  r = sigmoid(R u + b),  i = sigmoid(I u + b)   (block-diagonal R, I)
//     log a = -8 r softplus(lambda),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S y
//
// The convolution writes u in the layout [blocks][rows][part], in which the gates are one grouped product with a [2 part,
// part] matrix per block (r rows, then i rows), f32 out.
//  * rglru_scan_kernel   many tokens: a block owns a strip of channels of one session; its eight warps take consecutive
//                        segments of 8 tokens each, which are scanned side by side from zero, joined through shared memory
//                        (each segment is S -> A S + H) and finished from registers: every value is read once.
//  * rglru_fused_step_kernel  single-token steps, bf16, parts of a multiple of 32 channels up to 256: convolution, both gates
//                        and the recurrence in one launch.  The gates of a part need its own channels only, so nothing
//                        passes between parts.
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

constexpr uint32_t RG_WARPS = 8, RG_SEG = 8;

// VEC channels per lane: two when parts, pitches and pointers are even.  y stays as it was stored until it is used.
template <typename T, int VEC>
struct RgRaw { typedef T type; };
template <>
struct RgRaw<bf16, 2> { typedef uint32_t type; };
template <>
struct RgRaw<float, 2> { typedef float2 type; };
__device__ __forceinline__ float2 rg_values(uint32_t v) { return bf16x2_to_f32(v); }
__device__ __forceinline__ float2 rg_values(float2 v) { return v; }
__device__ __forceinline__ float2 rg_values(bf16 v) { return make_float2(__bfloat162float(v), 0.0f); }
__device__ __forceinline__ float2 rg_values(float v) { return make_float2(v, 0.0f); }

template <typename T, int VEC>
__global__ void __launch_bounds__(RG_WARPS * 32, 3)
rglru_scan_kernel(Rglru m, StepPlace place) {
    constexpr uint32_t STRIP = 32 * VEC;
    typedef typename RgRaw<T, VEC>::type Raw;
    __shared__ float4 seg[2][RG_WARPS][32];          // per lane: A of its channels, H of its channels
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
        float a[RG_SEG][VEC], b[RG_SEG][VEC];
        Raw yy[RG_SEG], uu[RG_SEG];
#pragma unroll
        for (uint32_t i = 0; i < RG_SEG; ++i) {
            const uint32_t t = first + i;
            const bool here = live && t < place.chunk;
            const Raw* up = reinterpret_cast<const Raw*>(u + (size_t)t * part);
            const Raw* yp = reinterpret_cast<const Raw*>(y + (size_t)t * m.ld);
            uu[i] = here ? *up : Raw();
            yy[i] = here ? *yp : Raw();
            if (VEC == 2) {
                const float2 z = make_float2(0.0f, 0.0f);
                const float2 r = here ? *reinterpret_cast<const float2*>(gates + (size_t)t * 2 * part) : z;
                const float2 g = here ? *reinterpret_cast<const float2*>(gates + (size_t)t * 2 * part + part) : z;
                a[i][0] = r.x; a[i][VEC - 1] = r.y; b[i][0] = g.x; b[i][VEC - 1] = g.y;
            } else {
                a[i][0] = here ? gates[(size_t)t * 2 * part] : 0.0f;
                b[i][0] = here ? gates[(size_t)t * 2 * part + part] : 0.0f;
            }
        }
        float A[VEC], H[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) { A[e] = 1.0f; H[e] = 0.0f; }
#pragma unroll
        for (uint32_t i = 0; i < RG_SEG; ++i) {
            const float2 uv = rg_values(uu[i]);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                if (first + i < place.chunk) rg_token<T>(ch[e], a[i][e], b[i][e], e ? uv.y : uv.x, a[i][e], b[i][e]);
                else { a[i][e] = 1.0f; b[i][e] = 0.0f; }
                A[e] *= a[i][e];
                H[e] = fmaf(a[i][e], H[e], b[i][e]);
            }
        }
        seg[buf][warp][lane] = make_float4(A[0], A[VEC - 1], H[0], H[VEC - 1]);
        __syncthreads();       // the other buffer is rewritten only after the next barrier
        float S[VEC];
#pragma unroll
        for (uint32_t w = 0; w < RG_WARPS; ++w) {
            const float4 q = seg[buf][w][lane];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                if (w == warp) S[e] = carry[e];
                carry[e] = e ? fmaf(q.y, carry[e], q.w) : fmaf(q.x, carry[e], q.z);
            }
        }
#pragma unroll
        for (uint32_t i = 0; i < RG_SEG; ++i) {
            const uint32_t t = first + i;
            const float2 yv = rg_values(yy[i]);
            float o[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) { S[e] = fmaf(a[i][e], S[e], b[i][e]); o[e] = S[e] * (e ? yv.y : yv.x); }
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

// Block = (8 output channels of a part per warp, 16 sessions).  u of the whole part goes to shared memory in bf16
// (every block of a part makes it; the ring slot they all write held the oldest row, which nobody reads) and is the A operand
// of mma.sync; the gate rows are the B operand.  Of every 32 k values a lane takes eight consecutive ones (16 bytes): both
// operands use the same order of k, so the sum does not notice.  Everything the block needs is asked for before the first use:
// the weights even before the previous kernel has finished.
constexpr uint32_t RF_SESSIONS = 16, RF_MAX_PART = 256, RF_MAX_WARPS = 16;
template <int KS>      // part / 32, rounded up to 2, 4 or 8
__global__ void __launch_bounds__(RF_MAX_WARPS * 32)
rglru_fused_step_kernel(Rglru m, StepPlace place) {
    constexpr uint32_t PITCH = KS * 32 + 8;                 // elements
    __shared__ __align__(16) bf16 su[RF_SESSIONS * PITCH];
    const uint32_t part = m.width / m.blocks, outs = blockDim.x / 4, subs = part / outs, blk = blockIdx.x / subs, c_first = blk * part, s0 = blockIdx.y * RF_SESSIONS;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t n0 = blockIdx.x % subs * outs + warp * 8;
    uint4 br[KS], bi[KS];
    {
        const bf16* wr = reinterpret_cast<const bf16*>(m.gate_w) + (size_t)blk * 2 * part * part + (size_t)(n0 + g8) * part + t4 * 8;
        const bf16* wi = wr + (size_t)part * part;
#pragma unroll
        for (int i = 0; i < KS; ++i) {
            const bool there = i * 32 < part;
            br[i] = there ? __ldg(reinterpret_cast<const uint4*>(wr + i * 32)) : make_uint4(0u, 0u, 0u, 0u);
            bi[i] = there ? __ldg(reinterpret_cast<const uint4*>(wi + i * 32)) : make_uint4(0u, 0u, 0u, 0u);
        }
    }
    const uint32_t c = n0 + t4 * 2, ch = c_first + c;
    const RgChannel ca = rg_channel(m, ch), cb = rg_channel(m, ch + 1);
    pdl_wait();
    pdl_trigger();
    const bf16* proj = reinterpret_cast<const bf16*>(m.proj);
    bf16* ring = reinterpret_cast<bf16*>(m.ring);
    float2 old[2], y[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const uint32_t s = s0 + g8 + half * 8;
        const bool here = s < place.sessions;
        old[half] = here && place.pos(s) > 0 ? *reinterpret_cast<const float2*>(m.state + (size_t)s * m.width + ch) : make_float2(0.0f, 0.0f);
        y[half] = here ? bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(proj + (size_t)s * m.ld + ch)) : make_float2(0.0f, 0.0f);
    }
    // ---- convolution: a thread owns two neighbouring channels and asks for eight sessions' rows at a time ----
    const uint32_t pairs = part / 2, groups = blockDim.x / pairs, group = threadIdx.x / pairs, cc = threadIdx.x % pairs * 2, x = c_first + cc;
    if (group < groups) {
        constexpr uint32_t AT_ONCE = 8, LAGS = 3;          // rows up to LAGS back travel together, older ones one by one
        const float *w0 = m.conv_w + (size_t)x * m.taps + m.taps - 1, *w1 = w0 + m.taps;       // of the current token; lag l at [-l]
        const float2 bias = make_float2(m.conv_b[x], m.conv_b[x + 1]), wn = make_float2(*w0, *w1);
        float2 wl[LAGS];
#pragma unroll
        for (uint32_t l = 0; l < LAGS; ++l) wl[l] = l + 1 < m.taps ? make_float2(w0[-(int)l - 1], w1[-(int)l - 1]) : make_float2(0.0f, 0.0f);
        for (uint32_t r0 = group; r0 < RF_SESSIONS; r0 += AT_ONCE * groups) {
            uint32_t now[AT_ONCE], back[LAGS][AT_ONCE], pos[AT_ONCE];
#pragma unroll
            for (uint32_t k = 0; k < AT_ONCE; ++k) {
                const uint32_t r = r0 + k * groups, s = s0 + r;
                const bool here = r < RF_SESSIONS && s < place.sessions;
                pos[k] = here ? place.pos(s) : 0u;
                now[k] = here ? *reinterpret_cast<const uint32_t*>(proj + (size_t)s * m.ld + m.x_col + x) : 0u;
                const uint32_t slot = pos[k] % m.taps;
#pragma unroll
                for (uint32_t l = 1; l <= LAGS; ++l) {
                    const uint32_t at = slot >= l ? slot - l : slot + m.taps - l;
                    back[l - 1][k] = here && l < m.taps && pos[k] >= l
                                         ? *reinterpret_cast<const uint32_t*>(ring + ((size_t)s * m.taps + at) * m.width + x) : 0u;
                }
            }
#pragma unroll
            for (uint32_t k = 0; k < AT_ONCE; ++k) {
                const uint32_t r = r0 + k * groups, s = s0 + r;
                if (r >= RF_SESSIONS) continue;
                const float2 f = bf16x2_to_f32(now[k]);
                float2 v = make_float2(fmaf(wn.x, f.x, bias.x), fmaf(wn.y, f.y, bias.y));
#pragma unroll
                for (uint32_t l = 0; l < LAGS; ++l) {
                    const float2 g = bf16x2_to_f32(back[l][k]);
                    v.x = fmaf(wl[l].x, g.x, v.x);
                    v.y = fmaf(wl[l].y, g.y, v.y);
                }
                if (s < place.sessions) {
                    const uint32_t slot = pos[k] % m.taps;
                    for (uint32_t l = LAGS + 1; l < m.taps && l <= pos[k]; ++l) {
                        const uint32_t at = slot >= l ? slot - l : slot + m.taps - l;
                        const float2 g = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(ring + ((size_t)s * m.taps + at) * m.width + x));
                        v.x = fmaf(w0[-(int)l], g.x, v.x);
                        v.y = fmaf(w1[-(int)l], g.y, v.y);
                    }
                    *reinterpret_cast<uint32_t*>(ring + ((size_t)s * m.taps + slot) * m.width + x) = now[k];
                }
                *reinterpret_cast<uint32_t*>(su + r * PITCH + cc) = pack_bf16x2(v.x, v.y);
            }
        }
    }
    __syncthreads();
    // ---- gates and recurrence ----
    float gr[4] = {0.0f, 0.0f, 0.0f, 0.0f}, gi[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < KS; ++i) {
        if (i * 32 >= part) continue;
        const uint4 lo = *reinterpret_cast<const uint4*>(su + g8 * PITCH + i * 32 + t4 * 8), hi = *reinterpret_cast<const uint4*>(su + (g8 + 8) * PITCH + i * 32 + t4 * 8);
        const uint32_t a0[4] = {lo.x, hi.x, lo.y, hi.y}, a1[4] = {lo.z, hi.z, lo.w, hi.w};
        mx_mma(gr, a0, br[i].x, br[i].y);
        mx_mma(gi, a0, bi[i].x, bi[i].y);
        mx_mma(gr, a1, br[i].z, br[i].w);
        mx_mma(gi, a1, bi[i].z, bi[i].w);
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const uint32_t r = g8 + half * 8, s = s0 + r;
        if (s >= place.sessions) continue;
        const float2 u = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(su + r * PITCH + c));
        float a, b;
        float2 S;
        rg_token<bf16>(ca, gr[2 * half], gi[2 * half], u.x, a, b);
        S.x = fmaf(a, old[half].x, b);
        rg_token<bf16>(cb, gr[2 * half + 1], gi[2 * half + 1], u.y, a, b);
        S.y = fmaf(a, old[half].y, b);
        *reinterpret_cast<float2*>(m.state + (size_t)s * m.width + ch) = S;
        *reinterpret_cast<uint32_t*>(reinterpret_cast<bf16*>(m.out) + (size_t)s * m.out_ld + ch) = pack_bf16x2(S.x * y[half].x, S.y * y[half].y);
    }
    if (blockIdx.x == 0 && m.out_cols > m.width) {
        const uint32_t pad = m.out_cols - m.width;
        for (uint32_t i = threadIdx.x; i < pad * RF_SESSIONS; i += blockDim.x) {
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
        // as many output channels per block as leave every SM a block: blocks of a part repeat its convolution
        const uint32_t tiles = ceil_div(place.sessions, RF_SESSIONS);
        uint32_t outs = 32;
        while (outs * 2 <= 8 * RF_MAX_WARPS && part % (outs * 2) == 0 && m.width / (outs * 2) * tiles >= 128) outs *= 2;
        const dim3 grid(m.width / outs, tiles), block(outs * 4);
        if (part <= 64) launch_kernel(rglru_fused_step_kernel<2>, grid, block, 0, stream, m, place);
        else if (part <= 128) launch_kernel(rglru_fused_step_kernel<4>, grid, block, 0, stream, m, place);
        else launch_kernel(rglru_fused_step_kernel<8>, grid, block, 0, stream, m, place);
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
