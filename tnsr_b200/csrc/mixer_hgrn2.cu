// HGRN2: linear attention in which every channel writes the share that it forgets.  Per head an f32 state S [dim, vdim]:
//     f = l + (1 - l) sigmoid(f_raw + b),   S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,   o_t = S_t^T silu(q_t)
// then an RMS norm of o per head.  1 - f is formed as (1 - l) sigmoid(-(f_raw + b)), so that a gate close to one writes
// what it should.
//
//  * hgrn2_token_kernel   token by token with the state in registers: single-token steps (the state makes one trip through
//                         HBM), short chunks, f32 sessions
//  * head_norm_kernel     the norm of heads wider than HGRN2_FUSED_VDIM (the others leave the kernels normed)
// The chunked tensor-core scan of long chunks is in hgrn2_scan.cu.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

int launch_hgrn2_scan(const Hgrn2& m, const StepPlace& place, cudaStream_t stream);   // hgrn2_scan.cu

// Shortest chunk that takes the chunked scan; below it the token kernel's few steps are cheaper.
constexpr uint32_t HG_SCAN_MIN_TOKENS = 16;
constexpr uint32_t HG_THREADS = 256, HG_MAX_DIM = 256, HG_SLICE = HGRN2_FUSED_VDIM;

// Block = (slice of at most HG_SLICE columns of the state, head, session).  A thread owns VEC neighbouring columns of every
// (256 / (width / VEC))-th row; what a token needs besides the state is asked for together with it.
template <typename T, int ROWS, int VEC>
__global__ void __launch_bounds__(HG_THREADS, ROWS * VEC <= 32 ? 4 : ROWS * VEC <= 64 ? 2 : 1)
hgrn2_token_kernel(Hgrn2 m, StepPlace place) {
    __shared__ float sf[HG_MAX_DIM], sk[HG_MAX_DIM], sq[HG_MAX_DIM], sv[HG_SLICE], red[HG_THREADS * VEC], ssum[HG_SLICE / 32];
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x;
    const uint32_t c_first = blockIdx.x * HG_SLICE, h = blockIdx.y, s = blockIdx.z;
    const uint32_t width = min(HG_SLICE, m.vdim - c_first);
    const uint32_t across = width / VEC, ng = HG_THREADS / across;      // threads along a row, row groups
    const uint32_t c = (tid % across) * VEC, k = tid / across;
    const bool live = k < ng;
    const uint32_t p0 = place.pos(s);
    float* state = m.state + (((size_t)s * m.heads + h) * m.dim) * m.vdim + c_first + c;
    float S[ROWS][VEC];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const uint32_t n = k + ng * i;
        const bool have = live && n < m.dim && p0 > 0;
        if (VEC == 4) {
            const float4 v = have ? *reinterpret_cast<const float4*>(state + (size_t)n * m.vdim) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            S[i][0] = v.x; S[i][VEC > 1 ? 1 : 0] = v.y; S[i][VEC > 2 ? 2 : 0] = v.z; S[i][VEC > 3 ? 3 : 0] = v.w;
        } else {
            S[i][0] = have ? state[(size_t)n * m.vdim] : 0.0f;
        }
    }
    const bool fused = m.vdim <= HGRN2_FUSED_VDIM;
    const float lower = tid < m.dim ? m.lower[h * m.dim + tid] : 0.0f, bias = tid < m.dim ? m.f_bias[h * m.dim + tid] : 0.0f;
    const float nw = fused && tid < width ? m.norm_w[tid] * m.gain : 0.0f;
    for (uint32_t t = 0; t < place.chunk; ++t) {
        const size_t row = (size_t)s * place.chunk + t;
        if (tid < m.dim) {
            const float z = m.f[row * m.f_ld + h * m.dim + tid] + bias;
            const float q = to_f32(reinterpret_cast<const T*>(m.q)[row * m.ld + h * m.dim + tid]);
            const float e = expf(-fabsf(z)), big = 1.0f / (1.0f + e), small = e * big;      // sigmoid(|z|), sigmoid(-|z|)
            sf[tid] = lower + (1.0f - lower) * (z >= 0.0f ? big : small);
            sk[tid] = (1.0f - lower) * (z >= 0.0f ? small : big);
            sq[tid] = full_silu(q);
        }
        if (tid < width) sv[tid] = to_f32(reinterpret_cast<const T*>(m.v)[row * m.ld + h * m.vdim + c_first + tid]);
        __syncthreads();
        if (live) {
            float acc[VEC], v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) { acc[e] = 0.0f; v[e] = sv[c + e]; }
#pragma unroll
            for (int i = 0; i < ROWS; ++i) {
                const uint32_t n = k + ng * i;
                if (n < m.dim) {
                    const float f = sf[n], w = sk[n], q = sq[n];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        S[i][e] = fmaf(S[i][e], f, w * v[e]);
                        acc[e] = fmaf(S[i][e], q, acc[e]);
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) red[k * width + c + e] = acc[e];
        }
        __syncthreads();
        float o = 0.0f;
        if (tid < width)
            for (uint32_t j = 0; j < ng; ++j) o += red[j * width + tid];
        if (!fused) {
            if (tid < width) m.raw[row * ((size_t)m.heads * m.vdim) + h * m.vdim + c_first + tid] = o;
            if (t + 1 < place.chunk) __syncthreads();
            continue;
        }
        if (tid < HG_SLICE) {
            float ss = o * o;
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
            if ((tid & 31) == 0) ssum[tid >> 5] = ss;
        }
        __syncthreads();
        if (tid < width) {
            float total = 0.0f;
#pragma unroll
            for (uint32_t i = 0; i < HG_SLICE / 32; ++i) total += ssum[i];
            T* out = reinterpret_cast<T*>(m.out) + row * m.out_ld;
            out[h * m.vdim + tid] = from_f32<T>(o * rsqrtf(total / (float)m.vdim + m.eps) * nw);
        }
        if (h + 1 == m.heads)
            for (uint32_t i = m.heads * m.vdim + tid; i < m.out_cols; i += HG_THREADS) reinterpret_cast<T*>(m.out)[row * m.out_ld + i] = from_f32<T>(0.0f);
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const uint32_t n = k + ng * i;
        if (!(live && n < m.dim)) continue;
        if (VEC == 4)
            *reinterpret_cast<float4*>(state + (size_t)n * m.vdim) = make_float4(S[i][0], S[i][VEC > 1 ? 1 : 0], S[i][VEC > 2 ? 2 : 0], S[i][VEC > 3 ? 3 : 0]);
        else
            state[(size_t)n * m.vdim] = S[i][0];
    }
}

template <typename T>
static void hgrn2_token(const Hgrn2& m, const StepPlace& place, cudaStream_t stream) {
    const dim3 grid(ceil_div(m.vdim, HG_SLICE), m.heads, place.sessions), block(HG_THREADS);
    const uint32_t width = std::min(m.vdim, HG_SLICE);
    if (m.vdim % 4 == 0 && reinterpret_cast<uintptr_t>(m.state) % 16 == 0) {
        const uint32_t rows = ceil_div(m.dim, HG_THREADS / (width / 4));
        if (rows <= 2) launch_kernel(hgrn2_token_kernel<T, 2, 4>, grid, block, 0, stream, m, place);
        else if (rows <= 4) launch_kernel(hgrn2_token_kernel<T, 4, 4>, grid, block, 0, stream, m, place);
        else if (rows <= 8) launch_kernel(hgrn2_token_kernel<T, 8, 4>, grid, block, 0, stream, m, place);
        else if (rows <= 16) launch_kernel(hgrn2_token_kernel<T, 16, 4>, grid, block, 0, stream, m, place);
        else launch_kernel(hgrn2_token_kernel<T, 32, 4>, grid, block, 0, stream, m, place);
        return;
    }
    const uint32_t rows = ceil_div(m.dim, HG_THREADS / width);
    if (rows <= 8) launch_kernel(hgrn2_token_kernel<T, 8, 1>, grid, block, 0, stream, m, place);
    else if (rows <= 32) launch_kernel(hgrn2_token_kernel<T, 32, 1>, grid, block, 0, stream, m, place);
    else launch_kernel(hgrn2_token_kernel<T, 128, 1>, grid, block, 0, stream, m, place);
}

bool hgrn2_supported(uint32_t heads, uint32_t dim, uint32_t vdim) {
    return heads > 0 && heads <= 65535u && vdim > 0 && dim > 0 && dim <= HG_MAX_DIM;
}

// ---- norm of wide heads: a block per (row, head) -----------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
head_norm_kernel(const float* __restrict__ raw, const float* __restrict__ w, T* __restrict__ out, uint32_t heads, uint32_t vdim, uint32_t out_ld,
                 uint32_t out_cols, float eps, float gain) {
    __shared__ float red[4];
    pdl_wait();
    pdl_trigger();
    const size_t row = blockIdx.x;
    const uint32_t h = blockIdx.y;
    const float* in = raw + (row * heads + h) * vdim;
    float ss = 0.0f;
    for (uint32_t c = threadIdx.x; c < vdim; c += 128) ss = fmaf(in[c], in[c], ss);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    const float inv = rsqrtf((red[0] + red[1] + red[2] + red[3]) / (float)vdim + eps) * gain;
    T* o = out + row * out_ld;
    for (uint32_t c = threadIdx.x; c < vdim; c += 128) o[h * vdim + c] = from_f32<T>(in[c] * inv * w[c]);
    if (h + 1 == heads)
        for (uint32_t c = heads * vdim + threadIdx.x; c < out_cols; c += 128) o[c] = from_f32<T>(0.0f);
}

int launch_hgrn2(const Hgrn2& m, const StepPlace& place, int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    const bool fused = m.vdim <= HGRN2_FUSED_VDIM, bf = dtype == TNSR_B200_BF16;
    if (!hgrn2_supported(m.heads, m.dim, m.vdim) || place.sessions > 65535u || (!fused && !m.raw)) {
        set_thread_error("hgrn2: at most 256 state rows, 65535 heads and sessions, scratch for wide heads");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    int rc;
    if (bf && m.engine == 0 && place.chunk >= HG_SCAN_MIN_TOKENS) {
        if ((rc = launch_hgrn2_scan(m, place, stream))) return rc;
    } else {
        if (bf) hgrn2_token<bf16>(m, place, stream); else hgrn2_token<float>(m, place, stream);
        count_launch();
        if ((rc = check_launch("hgrn2_token"))) return rc;
    }
    if (fused) return TNSR_B200_OK;
    const dim3 grid(place.sessions * place.chunk, m.heads);
    if (bf) launch_kernel(head_norm_kernel<bf16>, grid, dim3(128), 0, stream, m.raw, m.norm_w, (bf16*)m.out, m.heads, m.vdim, m.out_ld, m.out_cols, m.eps, m.gain);
    else launch_kernel(head_norm_kernel<float>, grid, dim3(128), 0, stream, m.raw, m.norm_w, (float*)m.out, m.heads, m.vdim, m.out_ld, m.out_cols, m.eps, m.gain);
    count_launch();
    return check_launch("head_norm");
}

}  // namespace tb
