// The mamba2 (state-space duality) mixer of models described layer by layer.  Per head an f32 state S [state, vdim]:
//     S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t
// with x, B, C behind a causal convolution and silu, dt behind softplus, then y * silu(z) and an RMS norm in groups.
//
//  * short_conv_kernel         convolution (+ silu), sliding window in registers (single-token steps also update the ring)
//  * ssd_token_kernel          token by token with the state in registers: single-token steps (the state makes one trip
//                              through HBM), short chunks, f32 sessions
//  * gated_norm_kernel         the grouped RMS norm of y * silu(z)
// The chunked tensor-core scan of long chunks is in ssd_scan.cu.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

int launch_ssd_scan(const Mamba2& m, const StepPlace& place, cudaStream_t stream);   // ssd_scan.cu

// Shortest chunk that takes the chunked tensor-core scan; below it the token kernel's few steps are cheaper.
constexpr uint32_t SSD_SCAN_MIN_TOKENS = 16;

// silu of an activation that is stored in T: bf16 results come from the hardware exponential, f32 ones from expf.
template <typename T>
__device__ __forceinline__ float act_silu(float x);
template <>
__device__ __forceinline__ float act_silu<float>(float x) { return full_silu(x); }
template <>
__device__ __forceinline__ float act_silu<bf16>(float x) { return mx_silu(x); }

// ---- convolution (+ silu) --------------------------------------------------------------------
// A thread owns two neighbouring channels of a run of tokens.
template <typename T, int TAPS, bool SILU>
__global__ void __launch_bounds__(128)
short_conv_kernel(const T* __restrict__ rows, uint32_t ld, uint32_t channels, uint32_t taps, const float* __restrict__ conv_w,
                  const float* __restrict__ conv_b, T* __restrict__ ring, T* __restrict__ out, uint32_t part, StepPlace place,
                  uint32_t run, uint32_t vec) {
    pdl_wait();
    pdl_trigger();
    const uint32_t c = 2 * (blockIdx.x * blockDim.x + threadIdx.x);
    if (c >= channels) return;
    const bool second = c + 1 < channels;
    const uint32_t s = blockIdx.z, t0 = blockIdx.y * run, t1 = min(place.chunk, t0 + run);
    const uint32_t p0 = place.pos(s);
    const T* in = rows + (size_t)s * place.chunk * ld + c;
    // output parts of `part` channels, each [rows, part]; the two channels of a thread may lie in different ones
    const size_t part_elems = (size_t)place.sessions * place.chunk * part;
    T* dst = out + c / part * part_elems + (size_t)s * place.chunk * part + c % part;
    T* dst1 = out + (c + 1) / part * part_elems + (size_t)s * place.chunk * part + (c + 1) % part;
    auto put = [&](uint32_t t, float2 y) {
        if (SILU) y = make_float2(act_silu<T>(y.x), act_silu<T>(y.y));
        if (vec) { store_pair<T>(dst + (size_t)t * part, y, true, true); return; }
        dst[(size_t)t * part] = from_f32<T>(y.x);
        if (second) dst1[(size_t)t * part] = from_f32<T>(y.y);
    };
    float2 w[TAPS], win[TAPS];
    const float* cw = conv_w + (size_t)c * taps;
    if (TAPS == 4 && taps == 4) {
        const float4 x = *reinterpret_cast<const float4*>(cw), y = second ? *reinterpret_cast<const float4*>(cw + 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        w[0] = make_float2(x.x, y.x);
        w[TAPS > 1 ? 1 : 0] = make_float2(x.y, y.y);
        w[TAPS > 2 ? 2 : 0] = make_float2(x.z, y.z);
        w[TAPS > 3 ? 3 : 0] = make_float2(x.w, y.w);
    } else {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const int src = j - (TAPS - (int)taps);
            w[j] = make_float2(src >= 0 ? cw[src] : 0.0f, src >= 0 && second ? cw[taps + src] : 0.0f);
        }
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        win[j] = make_float2(0.0f, 0.0f);
        const int t = (int)t0 - TAPS + j;
        if (j > 0 && (int)t0 - t < (int)taps) {
            const long long pos = (long long)p0 + t;
            if (t >= 0) win[j] = load_pair<T>(in + (size_t)t * ld, vec, second);
            else if (pos >= 0) win[j] = load_pair<T>(ring + ((size_t)s * taps + pos % taps) * channels + c, vec, second);
        }
    }
    const float2 b = make_float2(conv_b[c], second ? conv_b[c + 1] : 0.0f);
    if (place.chunk == 1) {
        // the slot of this position held the oldest row, which no single-token step reads
        const float2 now = load_pair<T>(in, vec, second);
        float2 y = b;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const float2 u = j + 1 < TAPS ? win[j + 1] : now;
            y.x = fmaf(w[j].x, u.x, y.x);
            y.y = fmaf(w[j].y, u.y, y.y);
        }
        put(0, y);
        store_pair<T>(ring + ((size_t)s * taps + p0 % taps) * channels + c, now, vec, second);
        return;
    }
    // rows are asked for eight at a time, so that their round trips overlap
    constexpr uint32_t AHEAD = 8;
    for (uint32_t t = t0; t < t1; t += AHEAD) {
        float2 next[AHEAD];
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i)
            next[i] = t + i < t1 ? load_pair<T>(in + (size_t)(t + i) * ld, vec, second) : make_float2(0.0f, 0.0f);
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; ++j) win[j] = win[j + 1];
            win[TAPS - 1] = next[i];
            float2 y = b;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) { y.x = fmaf(w[j].x, win[j].x, y.x); y.y = fmaf(w[j].y, win[j].y, y.y); }
            if (t + i < t1) put(t + i, y);
        }
    }
}

template <typename T, bool SILU>
static void short_conv_typed(const ShortConv& c, const StepPlace& place, cudaStream_t stream) {
    const uint32_t run = std::min(place.chunk, 32u);
    const dim3 grid(ceil_div(ceil_div(c.channels, 2u), 128u), ceil_div(place.chunk, run), place.sessions);
    auto even = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % (2 * sizeof(T)) == 0; };
    const uint32_t vec = c.channels % 2 == 0 && c.ld % 2 == 0 && c.part % 2 == 0 && even(c.rows) && even(c.ring) && even(c.out);
    if (c.taps <= 4)
        launch_kernel(short_conv_kernel<T, 4, SILU>, grid, dim3(128), 0, stream, (const T*)c.rows, c.ld, c.channels, c.taps, c.w, c.b, (T*)c.ring,
                      (T*)c.out, c.part, place, run, vec);
    else
        launch_kernel(short_conv_kernel<T, kMaxConvTaps, SILU>, grid, dim3(128), 0, stream, (const T*)c.rows, c.ld, c.channels, c.taps, c.w, c.b,
                      (T*)c.ring, (T*)c.out, c.part, place, run, vec);
}

int launch_short_conv(const ShortConv& c, const StepPlace& place, int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    if (c.taps == 0 || c.taps > kMaxConvTaps || c.part == 0 || c.channels % c.part || place.sessions > 65535u || ceil_div(place.chunk, 32u) > 65535u) {
        set_thread_error("convolution: 1..16 taps, parts that divide the channels, at most 65535 sessions");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    const bool bf = dtype == TNSR_B200_BF16;
    if (bf && c.silu) short_conv_typed<bf16, true>(c, place, stream);
    else if (bf) short_conv_typed<bf16, false>(c, place, stream);
    else if (c.silu) short_conv_typed<float, true>(c, place, stream);
    else short_conv_typed<float, false>(c, place, stream);
    count_launch();
    int rc = check_launch("short_conv");
    if (rc) return rc;
    return place.chunk > 1 ? launch_conv_ring(c.rows, c.ld, c.channels, c.taps, c.ring, place, dtype, stream) : TNSR_B200_OK;
}

// ---- token by token ----------------------------------------------------------------------------
// Block = (slice of at most 64 columns of the state, head, session).  A thread owns VEC neighbouring columns of every
// (256 / (width / VEC))-th row of its slice; everything a token needs besides the state (x, B, C, step, gate input) is
// asked for together with the state, one memory round trip per step.
constexpr uint32_t SSD_THREADS = 256, SSD_SLICE = 64, SSD_MAX_STATE = 256;

template <typename T, int ROWS, int VEC>
__global__ void __launch_bounds__(SSD_THREADS, ROWS * VEC <= 32 ? 4 : 2)
ssd_token_kernel(Mamba2 m, StepPlace place) {
    __shared__ float sb[SSD_MAX_STATE], sc[SSD_MAX_STATE], sx[SSD_SLICE], red[SSD_THREADS * VEC];
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x;
    const uint32_t p_first = blockIdx.x * SSD_SLICE, h = blockIdx.y, s = blockIdx.z;
    const uint32_t width = min(SSD_SLICE, m.vdim - p_first);
    const uint32_t across = width / VEC, ng = SSD_THREADS / across;     // threads along a row, row groups
    const uint32_t p = (tid % across) * VEC, k = tid / across;
    const bool live = k < ng;
    const uint32_t inner = m.heads * m.vdim, gn = m.groups * m.state, channels = inner + 2 * gn;
    const uint32_t group = h / (m.heads / m.groups);
    const uint32_t p0 = place.pos(s);
    float* state = m.ssm + (((size_t)s * m.heads + h) * m.state) * m.vdim + p_first + p;
    float S[ROWS][VEC];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const uint32_t n = k + ng * i;
        const bool have = live && n < m.state && p0 > 0;
        if (VEC == 4) {
            const float4 v = have ? *reinterpret_cast<const float4*>(state + (size_t)n * m.vdim) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            S[i][0] = v.x; S[i][VEC > 1 ? 1 : 0] = v.y; S[i][VEC > 2 ? 2 : 0] = v.z; S[i][VEC > 3 ? 3 : 0] = v.w;
        } else {
            S[i][0] = have ? state[(size_t)n * m.vdim] : 0.0f;
        }
    }
    const T* xbc = reinterpret_cast<const T*>(m.xbc) + (size_t)s * place.chunk * channels;
    const T* zrow = reinterpret_cast<const T*>(m.proj) + (size_t)s * place.chunk * m.ld + h * m.vdim + p_first;
    const float a_log = m.a_log[h], dt_bias = m.dt_bias[h], skip = m.d_skip[h];
    for (uint32_t t = 0; t < place.chunk; ++t) {
        const size_t row = (size_t)s * place.chunk + t;
        const float dt_raw = m.dt[row * m.dt_ld + h];
        const float z = tid < width ? to_f32(zrow[(size_t)t * m.ld + tid]) : 0.0f;
        if (tid < m.state) {
            sb[tid] = to_f32(xbc[(size_t)t * channels + inner + group * m.state + tid]);
            sc[tid] = to_f32(xbc[(size_t)t * channels + inner + gn + group * m.state + tid]);
        }
        if (tid < width) sx[tid] = to_f32(xbc[(size_t)t * channels + h * m.vdim + p_first + tid]);
        const float dt = softplus(dt_raw + dt_bias);
        const float decay = expf(-expf(a_log) * dt);
        __syncthreads();
        float acc[VEC], xdt[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) { acc[e] = 0.0f; xdt[e] = live ? dt * sx[p + e] : 0.0f; }
        if (live) {
#pragma unroll
            for (int i = 0; i < ROWS; ++i) {
                const uint32_t n = k + ng * i;
                if (n < m.state) {
                    const float b = sb[n], c = sc[n];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        S[i][e] = fmaf(S[i][e], decay, b * xdt[e]);
                        acc[e] = fmaf(S[i][e], c, acc[e]);
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) red[k * width + p + e] = acc[e];
        }
        __syncthreads();
        if (tid < width) {
            float y = skip * sx[tid];
            for (uint32_t j = 0; j < ng; ++j) y += red[j * width + tid];
            reinterpret_cast<T*>(m.gated)[row * inner + h * m.vdim + p_first + tid] = from_f32<T>(y * act_silu<T>(z));
        }
        if (t + 1 < place.chunk) __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const uint32_t n = k + ng * i;
        if (!(live && n < m.state)) continue;
        if (VEC == 4)
            *reinterpret_cast<float4*>(state + (size_t)n * m.vdim) = make_float4(S[i][0], S[i][VEC > 1 ? 1 : 0], S[i][VEC > 2 ? 2 : 0], S[i][VEC > 3 ? 3 : 0]);
        else
            state[(size_t)n * m.vdim] = S[i][0];
    }
}

template <typename T>
static void ssd_token(const Mamba2& m, const StepPlace& place, cudaStream_t stream) {
    const dim3 grid(ceil_div(m.vdim, SSD_SLICE), m.heads, place.sessions), block(SSD_THREADS);
    const uint32_t width = std::min(m.vdim, SSD_SLICE);
    if (m.vdim % 4 == 0 && reinterpret_cast<uintptr_t>(m.ssm) % 16 == 0) {
        const uint32_t rows = ceil_div(m.state, SSD_THREADS / (width / 4));
        if (rows <= 2) launch_kernel(ssd_token_kernel<T, 2, 4>, grid, block, 0, stream, m, place);
        else if (rows <= 4) launch_kernel(ssd_token_kernel<T, 4, 4>, grid, block, 0, stream, m, place);
        else if (rows <= 8) launch_kernel(ssd_token_kernel<T, 8, 4>, grid, block, 0, stream, m, place);
        else launch_kernel(ssd_token_kernel<T, 16, 4>, grid, block, 0, stream, m, place);
        return;
    }
    const uint32_t rows = ceil_div(m.state, SSD_THREADS / width);
    if (rows <= 8) launch_kernel(ssd_token_kernel<T, 8, 1>, grid, block, 0, stream, m, place);
    else if (rows <= 32) launch_kernel(ssd_token_kernel<T, 32, 1>, grid, block, 0, stream, m, place);
    else launch_kernel(ssd_token_kernel<T, 64, 1>, grid, block, 0, stream, m, place);
}

bool mamba2_supported(uint32_t heads, uint32_t vdim, uint32_t state) {
    return heads > 0 && heads <= 65535u && vdim > 0 && state > 0 && state <= SSD_MAX_STATE;
}

// ---- grouped RMS norm ------------------------------------------------------------------------------
// One block per (row, norm group): any width.  Parts of whole 16-byte chunks up to 2048 values take a warp each and stay in
// registers between the sum and the scaling (gated_norm_warp_kernel).
template <typename T>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const T* __restrict__ gated, const float* __restrict__ w, T* __restrict__ out, uint32_t inner, uint32_t groups,
                  uint32_t out_ld, uint32_t out_cols, float eps) {
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    const size_t row = blockIdx.x;
    const uint32_t part = inner / groups, c0 = blockIdx.y * part;
    const T* in = gated + row * inner + c0;
    float ss = 0.0f;
    for (uint32_t c = threadIdx.x; c < part; c += blockDim.x) { const float v = to_f32(in[c]); ss = fmaf(v, v, ss); }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float sum = 0.0f;
    for (uint32_t i = 0; i < blockDim.x / 32; ++i) sum += red[i];
    const float inv = rsqrtf(sum / (float)part + eps);
    T* o = out + row * out_ld + c0;
    for (uint32_t c = threadIdx.x; c < part; c += blockDim.x) o[c] = from_f32<T>(to_f32(in[c]) * inv * w[c0 + c]);
    if (blockIdx.y == 0)
        for (uint32_t c = inner + threadIdx.x; c < out_cols; c += blockDim.x) out[row * out_ld + c] = from_f32<T>(0.0f);
}

constexpr uint32_t GN_VEC = 8;   // 16-byte chunks per lane: parts of up to 2048 values, one warp each
__global__ void __launch_bounds__(128)
gated_norm_warp_kernel(const bf16* __restrict__ gated, const float* __restrict__ w, bf16* __restrict__ out, uint32_t rows, uint32_t inner,
                       uint32_t groups, uint32_t out_ld, uint32_t out_cols, float eps) {
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, task = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (task >= rows * groups) return;
    const uint32_t row = task / groups, grp = task % groups, part = inner / groups, chunks = part / 8, c0 = grp * part;
    const uint4* in = reinterpret_cast<const uint4*>(gated + (size_t)row * inner + c0);
    float v[GN_VEC][8], ss = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < GN_VEC; ++i) {
        const uint32_t c = lane + 32 * i;
        const uint4 q = c < chunks ? in[c] : make_uint4(0u, 0u, 0u, 0u);
        const uint32_t words[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = bf16x2_to_f32(words[k]);
            v[i][2 * k] = f.x;
            v[i][2 * k + 1] = f.y;
            ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss));
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = rsqrtf(ss / (float)part + eps);
    uint4* o = reinterpret_cast<uint4*>(out + (size_t)row * out_ld + c0);
#pragma unroll
    for (uint32_t i = 0; i < GN_VEC; ++i) {
        const uint32_t c = lane + 32 * i;
        if (c >= chunks) continue;
        const float4 w0 = *reinterpret_cast<const float4*>(w + c0 + c * 8), w1 = *reinterpret_cast<const float4*>(w + c0 + c * 8 + 4);
        o[c] = make_uint4(pack_bf16x2(v[i][0] * inv * w0.x, v[i][1] * inv * w0.y), pack_bf16x2(v[i][2] * inv * w0.z, v[i][3] * inv * w0.w),
                          pack_bf16x2(v[i][4] * inv * w1.x, v[i][5] * inv * w1.y), pack_bf16x2(v[i][6] * inv * w1.z, v[i][7] * inv * w1.w));
    }
    if (grp == 0)
        for (uint32_t c = inner + lane; c < out_cols; c += 32) out[(size_t)row * out_ld + c] = __float2bfloat16_rn(0.0f);
}

int launch_mamba2(const Mamba2& m, const StepPlace& place, int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    const uint32_t inner = m.heads * m.vdim, channels = inner + 2 * m.groups * m.state, rows = place.sessions * place.chunk;
    if (!mamba2_supported(m.heads, m.vdim, m.state) || m.taps == 0 || m.taps > kMaxConvTaps || place.sessions > 65535u ||
        ceil_div(place.chunk, 32u) > 65535u || m.norm_groups > 65535u) {
        set_thread_error("mamba2: at most 256 state rows, 16 convolution taps, 65535 sessions");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    const bool bf = dtype == TNSR_B200_BF16;
    int rc;
    ShortConv c;
    c.rows = (const uint8_t*)m.proj + (size_t)inner * (bf ? 2 : 4);
    c.ld = m.ld; c.channels = c.part = channels; c.taps = m.taps; c.w = m.conv_w; c.b = m.conv_b; c.ring = m.ring; c.out = m.xbc; c.silu = true;
    if ((rc = launch_short_conv(c, place, dtype, stream))) return rc;
    if (bf && m.engine == 0 && place.chunk >= SSD_SCAN_MIN_TOKENS) {
        if ((rc = launch_ssd_scan(m, place, stream))) return rc;
    } else {
        if (bf) ssd_token<bf16>(m, place, stream); else ssd_token<float>(m, place, stream);
        count_launch();
        if ((rc = check_launch("ssd_token"))) return rc;
    }
    const dim3 grid(rows, m.norm_groups);
    const uint32_t part = inner / m.norm_groups;
    const bool warp_norm = bf && part % 8 == 0 && part <= GN_VEC * 256 && m.out_ld % 8 == 0 && inner % 8 == 0 &&
                           (reinterpret_cast<uintptr_t>(m.gated) | reinterpret_cast<uintptr_t>(m.out) | reinterpret_cast<uintptr_t>(m.norm_w)) % 16 == 0;
    if (warp_norm)
        launch_kernel(gated_norm_warp_kernel, dim3(ceil_div(rows * m.norm_groups, 4)), dim3(128), 0, stream, (const bf16*)m.gated, m.norm_w, (bf16*)m.out,
                      rows, inner, m.norm_groups, m.out_ld, m.out_cols, m.eps);
    else if (bf)
        launch_kernel(gated_norm_kernel<bf16>, grid, dim3(256), 0, stream, (const bf16*)m.gated, m.norm_w, (bf16*)m.out, inner, m.norm_groups,
                      m.out_ld, m.out_cols, m.eps);
    else
        launch_kernel(gated_norm_kernel<float>, grid, dim3(256), 0, stream, (const float*)m.gated, m.norm_w, (float*)m.out, inner,
                      m.norm_groups, m.out_ld, m.out_cols, m.eps);
    count_launch();
    return check_launch("gated_norm");
}

}  // namespace tb
