// Chunked scan of the mamba2 mixer on the warp-level tensor cores (bf16 x, B, C; everything else f32).
//
// Within a chunk of 64 tokens, with c_i the running sum of the log decays:
//     y_i = exp(c_i) C_i S_in + sum_{j <= i} (C_i . B_j) exp(c_i - c_j) dt_j x_j + D x_i
//     S_out = exp(c_63) S_in + sum_j B_j (exp(c_63 - c_j) dt_j x_j)^T
// A CTA owns the whole sequence of one (session, head, slice of the state's columns) and carries S in accumulator
// registers from chunk to chunk; columns of S do not couple, so slices are independent.  Four warps: 16 token rows each
// for y, a quarter of the state's rows each for S.  Factors that are f32 -- the decayed weights, the state, the weighted
// inputs -- enter the products as two bf16 halves (split_bf16x2), so that they keep 16 bits.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

constexpr int SC_Q = 64;          // tokens per chunk
constexpr float SC_LOG2E = 1.4426950408889634f;

template <int NP, int PT>
struct ScanShape {
    static constexpr uint32_t BP = NP * 2 + 16, XP = PT * 2 + 16;     // row pitches: conflict-free ldmatrix
    static constexpr uint32_t B_BYTES = SC_Q * BP, X_BYTES = SC_Q * XP, S_BYTES = NP * XP;
    static constexpr uint32_t BYTES = 2 * B_BYTES + 3 * X_BYTES + 2 * S_BYTES;
};

// NP: state rows padded to a multiple of 64, PT: columns of the slice (padded).
template <int NP, int PT>
__global__ void __launch_bounds__(128, NP <= 128 ? 2 : 1)
ssd_scan_kernel(Mamba2 m, StepPlace place, uint32_t vec) {
    using S = ScanShape<NP, PT>;
    constexpr int MT = NP / 64;                 // 16-row tiles of the state per warp
    extern __shared__ __align__(16) uint8_t smem[];
    uint8_t* sb = smem;
    uint8_t* sc = sb + S::B_BYTES;
    uint8_t* sx = sc + S::B_BYTES;
    uint8_t* sxh = sx + S::X_BYTES;
    uint8_t* sxl = sxh + S::X_BYTES;
    uint8_t* ssh = sxl + S::X_BYTES;
    uint8_t* ssl = ssh + S::S_BYTES;
    __shared__ float s_cum[SC_Q], s_dt[SC_Q];   // running log2 decay, step size
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t p_first = blockIdx.x * PT, h = blockIdx.y, s = blockIdx.z;
    const uint32_t width = min((uint32_t)PT, m.vdim - p_first);
    const uint32_t inner = m.heads * m.vdim, gn = m.groups * m.state, channels = inner + 2 * gn;
    const uint32_t group = h / (m.heads / m.groups);
    pdl_wait();
    pdl_trigger();
    const uint32_t p0 = place.pos(s);
    const float a2 = -expf(m.a_log[h]) * SC_LOG2E, dt_bias = m.dt_bias[h], skip = m.d_skip[h];
    const size_t row_base = (size_t)s * place.chunk;
    const bf16* xbc = reinterpret_cast<const bf16*>(m.xbc) + row_base * channels;
    float* state = m.ssm + (((size_t)s * m.heads + h) * m.state) * m.vdim + p_first;

    // S: rows n = (warp * MT + mt) * 16 + g8 (+ 8), columns nt * 8 + t4 * 2 (+ 1)
    float acc[MT][PT / 8][4];
    auto state_rows = [&](int mt, int half) { return (uint32_t)((warp * MT + mt) * 16) + g8 + half * 8; };
    auto store_state_tiles = [&]() {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < PT / 8; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t hi, lo;
                    split_bf16x2(acc[mt][nt][2 * half], acc[mt][nt][2 * half + 1], hi, lo);
                    const uint32_t off = state_rows(mt, half) * S::XP + (nt * 8 + t4 * 2) * 2;
                    *reinterpret_cast<uint32_t*>(ssh + off) = hi;
                    *reinterpret_cast<uint32_t*>(ssl + off) = lo;
                }
    };
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < PT / 8; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t n = state_rows(mt, e >> 1), p = nt * 8 + t4 * 2 + (e & 1);
                acc[mt][nt][e] = p0 > 0 && n < m.state && p < width ? state[(size_t)n * m.vdim + p] : 0.0f;
            }
    store_state_tiles();

    // one operand tile: 64 rows of `w` channels from channel c0 on, rows past the chunk's end and channels past w are zero
    auto load_tile = [&](uint8_t* dst, uint32_t pitch, uint32_t padded, uint32_t c0, uint32_t w, uint32_t t0) {
        const uint32_t live = min((uint32_t)SC_Q, place.chunk - t0);
        if (vec) {
            const uint32_t ch = padded / 8;
            for (uint32_t i = tid; i < SC_Q * ch; i += 128) {
                const uint32_t r = i / ch, c = (i % ch) * 8;
                const bool real = r < live && c < w;
                mx_cp16(dst + r * pitch + c * 2, real ? xbc + (size_t)(t0 + r) * channels + c0 + c : xbc, real);
            }
        } else {
            for (uint32_t i = tid; i < SC_Q * padded; i += 128) {
                const uint32_t r = i / padded, c = i % padded;
                *reinterpret_cast<bf16*>(dst + r * pitch + c * 2) =
                    r < live && c < w ? xbc[(size_t)(t0 + r) * channels + c0 + c] : __float2bfloat16_rn(0.0f);
            }
        }
    };

    for (uint32_t t0 = 0; t0 < place.chunk; t0 += SC_Q) {
        load_tile(sb, S::BP, NP, inner + group * m.state, m.state, t0);
        load_tile(sc, S::BP, NP, inner + gn + group * m.state, m.state, t0);
        load_tile(sx, S::XP, PT, h * m.vdim + p_first, width, t0);
        mx_commit();
        if (warp == 0) {
            // steps and running log decays of tokens 2 lane, 2 lane + 1; tokens past the end have step 0
            float dt[2], d2[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const uint32_t t = t0 + 2 * lane + i;
                dt[i] = 0.0f;
                if (t < place.chunk) {
                    const float u = m.dt[(row_base + t) * m.dt_ld + h] + dt_bias;
                    dt[i] = u > 20.0f ? u : log1pf(expf(u));
                }
                d2[i] = a2 * dt[i];
            }
            float sum = d2[0] + d2[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= (uint32_t)o) sum += up;
            }
            s_cum[2 * lane + 1] = sum;
            s_cum[2 * lane] = sum - d2[1];
            s_dt[2 * lane] = dt[0];
            s_dt[2 * lane + 1] = dt[1];
        }
        mx_wait<0>();
        __syncthreads();
        const float last = s_cum[SC_Q - 1];
        // inputs weighted for the state at the end of the chunk
        for (uint32_t i = tid; i < SC_Q * (PT / 2); i += 128) {
            const uint32_t r = i / (PT / 2), c = (i % (PT / 2)) * 2;
            const float w = mx_ex2(last - s_cum[r]) * s_dt[r];
            const float2 x = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(sx + r * S::XP + c * 2));
            uint32_t hi, lo;
            split_bf16x2(x.x * w, x.y * w, hi, lo);
            *reinterpret_cast<uint32_t*>(sxh + r * S::XP + c * 2) = hi;
            *reinterpret_cast<uint32_t*>(sxl + r * S::XP + c * 2) = lo;
        }
        // ---- C . B^T (columns up to the warp's own rows) and C . S_in ----
        const uint32_t i0 = warp * 16 + g8, i1 = i0 + 8;
        const float cum0 = s_cum[i0], cum1 = s_cum[i1];
        float gm[SC_Q / 8][4], y[PT / 8][4];
#pragma unroll
        for (int i = 0; i < SC_Q / 8; ++i) gm[i][0] = gm[i][1] = gm[i][2] = gm[i][3] = 0.0f;
#pragma unroll
        for (int i = 0; i < PT / 8; ++i) y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.0f;
        const uint32_t a_addr = mx_smem(sc) + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::BP + (lane >> 4) * 16;
        const uint32_t b_off = ((lane & 7) + (lane >> 4) * 8) * S::BP + ((lane >> 3) & 1) * 16;
        const uint32_t t_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::XP + (lane >> 4) * 16;   // transposed [k][n] tiles
        const uint32_t sb_a = mx_smem(sb), ssh_a = mx_smem(ssh), ssl_a = mx_smem(ssl), sx_a = mx_smem(sx);
#pragma unroll
        for (int kk = 0; kk < NP / 16; ++kk) {
            uint32_t ca[4], bb[4];
            mx_ldsm(a_addr + kk * 32, ca);
#pragma unroll
            for (int n = 0; n < SC_Q / 16; ++n) {
                if ((uint32_t)n > warp) continue;
                mx_ldsm(sb_a + b_off + n * 16 * S::BP + kk * 32, bb);
                mx_mma(gm[2 * n], ca, bb[0], bb[1]);
                mx_mma(gm[2 * n + 1], ca, bb[2], bb[3]);
            }
#pragma unroll
            for (int n = 0; n < PT / 16; ++n) {
                mx_ldsm_t(ssh_a + t_off + kk * 16 * S::XP + n * 32, bb);
                mx_mma(y[2 * n], ca, bb[0], bb[1]);
                mx_mma(y[2 * n + 1], ca, bb[2], bb[3]);
                mx_ldsm_t(ssl_a + t_off + kk * 16 * S::XP + n * 32, bb);
                mx_mma(y[2 * n], ca, bb[0], bb[1]);
                mx_mma(y[2 * n + 1], ca, bb[2], bb[3]);
            }
        }
        const float e0 = mx_ex2(cum0), e1 = mx_ex2(cum1);
#pragma unroll
        for (int i = 0; i < PT / 8; ++i) { y[i][0] *= e0; y[i][1] *= e0; y[i][2] *= e1; y[i][3] *= e1; }
        // ---- decayed weights times x ----
#pragma unroll
        for (int kk = 0; kk < SC_Q / 16; ++kk) {
            if ((uint32_t)kk > warp) continue;
            uint32_t hi[4], lo[4], bb[4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const uint32_t j = (2 * kk + n) * 8 + t4 * 2;
                const float cj0 = s_cum[j], cj1 = s_cum[j + 1], dj0 = s_dt[j], dj1 = s_dt[j + 1];
                const float* v = gm[2 * kk + n];
                const float w0 = j <= i0 ? v[0] * mx_ex2(cum0 - cj0) * dj0 : 0.0f;
                const float w1 = j + 1 <= i0 ? v[1] * mx_ex2(cum0 - cj1) * dj1 : 0.0f;
                const float w2 = j <= i1 ? v[2] * mx_ex2(cum1 - cj0) * dj0 : 0.0f;
                const float w3 = j + 1 <= i1 ? v[3] * mx_ex2(cum1 - cj1) * dj1 : 0.0f;
                split_bf16x2(w0, w1, hi[2 * n], lo[2 * n]);
                split_bf16x2(w2, w3, hi[2 * n + 1], lo[2 * n + 1]);
            }
#pragma unroll
            for (int n = 0; n < PT / 16; ++n) {
                mx_ldsm_t(sx_a + t_off + kk * 16 * S::XP + n * 32, bb);
                mx_mma(y[2 * n], hi, bb[0], bb[1]);
                mx_mma(y[2 * n + 1], hi, bb[2], bb[3]);
                mx_mma(y[2 * n], lo, bb[0], bb[1]);
                mx_mma(y[2 * n + 1], lo, bb[2], bb[3]);
            }
        }
        // ---- skip, gate, store ----
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const uint32_t r = half ? i1 : i0, t = t0 + r;
            if (t >= place.chunk) continue;
            const bf16* z = reinterpret_cast<const bf16*>(m.proj) + (row_base + t) * m.ld + h * m.vdim + p_first;
            bf16* out = reinterpret_cast<bf16*>(m.gated) + (row_base + t) * inner + h * m.vdim + p_first;
#pragma unroll
            for (int nt = 0; nt < PT / 8; ++nt) {
                const uint32_t c = nt * 8 + t4 * 2;
                if (c >= width) continue;
                const float2 x = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(sx + r * S::XP + c * 2));
                const bool second = c + 1 < width;
                const float2 zz = load_pair<bf16>(z + c, vec, second);
                const float v0 = fmaf(skip, x.x, y[nt][2 * half]), v1 = fmaf(skip, x.y, y[nt][2 * half + 1]);
                store_pair<bf16>(out + c, make_float2(v0 * fast_silu(zz.x), v1 * fast_silu(zz.y)), vec, second);
            }
        }
        __syncthreads();     // weighted inputs are in place; the state tiles have been read
        // ---- state at the end of the chunk ----
        const float el = mx_ex2(last);
        const uint32_t bt_off = ((lane & 7) + (lane >> 4) * 8) * S::BP + ((lane >> 3) & 1) * 16;   // B^T: rows n from [token][n] tiles
        const uint32_t sxh_a = mx_smem(sxh), sxl_a = mx_smem(sxl);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < PT / 8; ++nt) { acc[mt][nt][0] *= el; acc[mt][nt][1] *= el; acc[mt][nt][2] *= el; acc[mt][nt][3] *= el; }
#pragma unroll
        for (int kk = 0; kk < SC_Q / 16; ++kk) {
            uint32_t ba[MT][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) mx_ldsm_t(sb_a + bt_off + kk * 16 * S::BP + (warp * MT + mt) * 32, ba[mt]);
#pragma unroll
            for (int n = 0; n < PT / 16; ++n) {
                uint32_t xh[4], xl[4];
                mx_ldsm_t(sxh_a + t_off + kk * 16 * S::XP + n * 32, xh);
                mx_ldsm_t(sxl_a + t_off + kk * 16 * S::XP + n * 32, xl);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    mx_mma(acc[mt][2 * n], ba[mt], xh[0], xh[1]);
                    mx_mma(acc[mt][2 * n + 1], ba[mt], xh[2], xh[3]);
                    mx_mma(acc[mt][2 * n], ba[mt], xl[0], xl[1]);
                    mx_mma(acc[mt][2 * n + 1], ba[mt], xl[2], xl[3]);
                }
            }
        }
        store_state_tiles();
        __syncthreads();     // every tile may be refilled
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < PT / 8; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t n = state_rows(mt, e >> 1), p = nt * 8 + t4 * 2 + (e & 1);
                if (n < m.state && p < width) state[(size_t)n * m.vdim + p] = acc[mt][nt][e];
            }
}

template <int NP, int PT>
static int launch_scan(const Mamba2& m, const StepPlace& place, uint32_t vec, cudaStream_t stream) {
    static bool configured[64] = {};
    const uint32_t bytes = ScanShape<NP, PT>::BYTES;
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64 || !configured[dev]) {
        if (cudaFuncSetAttribute(ssd_scan_kernel<NP, PT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
            return check_launch("ssd_scan attribute");
        if (dev >= 0 && dev < 64) configured[dev] = true;
    }
    launch_kernel(ssd_scan_kernel<NP, PT>, dim3(ceil_div(m.vdim, (uint32_t)PT), m.heads, place.sessions), dim3(128), bytes, stream, m, place, vec);
    count_launch();
    return check_launch("ssd_scan");
}

// Rows of xbc hold the convolved x | B | C of every token of the chunk.
int launch_ssd_scan(const Mamba2& m, const StepPlace& place, cudaStream_t stream) {
    const uint32_t inner = m.heads * m.vdim;
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const uint32_t vec = m.vdim % 8 == 0 && m.state % 8 == 0 && m.ld % 2 == 0 && inner % 8 == 0 && aligned(m.xbc) && aligned(m.proj) && aligned(m.gated);
    const bool narrow = m.vdim <= 32;
    if (m.state <= 64) return narrow ? launch_scan<64, 32>(m, place, vec, stream) : launch_scan<64, 64>(m, place, vec, stream);
    if (m.state <= 128) return narrow ? launch_scan<128, 32>(m, place, vec, stream) : launch_scan<128, 64>(m, place, vec, stream);
    return launch_scan<256, 32>(m, place, vec, stream);
}

}  // namespace tb
