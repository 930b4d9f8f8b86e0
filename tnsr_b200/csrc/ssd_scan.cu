// Chunked scan of the mamba2 mixer on the warp-level tensor cores (bf16 x, B, C; everything else f32).
//
// Within a chunk of 64 tokens, with c_i the running sum of the log decays:
//     y_i = exp(c_i) C_i S_in + sum_{j <= i} (C_i . B_j) exp(c_i - c_j) dt_j x_j + D x_i
//     S_out = exp(c_63) S_in + sum_j B_j (exp(c_63 - c_j) dt_j x_j)^T
// A CTA owns the whole sequence of one (session, head, 64 columns of the state) and carries S from chunk to chunk; columns
// of S do not couple, so each of its four warps owns 16 of them.  A warp keeps S transposed in accumulator registers
// (rows = its columns, from x^T . B): in that layout the accumulators of S^T are, register by register, the B operand of
// C . S, so the state never passes through shared memory.  The decayed weights (C B^T with the decays applied) are made
// once per CTA, 16 token rows per warp, and shared.  Three CTAs per SM (states up to 128 rows) hide each other's waits; the
// next chunk's C is asked for as soon as the current one is used up, its B and x at the end of the chunk.
//
// Factors that are f32 -- the decayed weights, the state, the weighted inputs -- enter the products as two bf16 halves
// (split_bf16x2), so that they keep 16 bits.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

constexpr int SC_Q = 64;          // tokens per chunk
constexpr uint32_t SC_P = 64;     // columns of the state per CTA, 16 per warp
constexpr float SC_LOG2E = 1.4426950408889634f;

template <int NP>
struct ScanShape {
    static constexpr uint32_t BP = NP * 2 + 16, XP = SC_P * 2 + 16, WP = SC_Q * 2 + 16;   // row pitches: conflict-free ldmatrix
    static constexpr uint32_t B_BYTES = SC_Q * BP, X_BYTES = SC_Q * XP, W_BYTES = SC_Q * WP;
    static constexpr uint32_t STAGE = 2 * B_BYTES + X_BYTES;          // B, C, x of one chunk
    static constexpr uint32_t BYTES = STAGE + 2 * W_BYTES;
};

// NP: state rows padded to a multiple of 64.
template <int NP>
__global__ void __launch_bounds__(128, NP <= 128 ? 3 : 1)
ssd_scan_kernel(Mamba2 m, StepPlace place, uint32_t vec) {
    using S = ScanShape<NP>;
    constexpr int NT = NP / 8;                  // 8-row tiles of the state
    extern __shared__ __align__(16) uint8_t smem[];
    uint8_t* swh = smem + S::STAGE;
    uint8_t* swl = swh + S::W_BYTES;
    __shared__ float s_cum[2][SC_Q], s_dt[2][SC_Q];   // running log2 decay, step size
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t p_first = blockIdx.x * SC_P, h = blockIdx.y, s = blockIdx.z;
    const uint32_t width = min(SC_P, m.vdim - p_first);
    const uint32_t inner = m.heads * m.vdim, gn = m.groups * m.state, channels = inner + 2 * gn;
    const uint32_t group = h / (m.heads / m.groups);
    const uint32_t pw = warp * 16;              // the warp's columns
    const bool owner = pw < width;
    pdl_wait();
    pdl_trigger();
    const uint32_t p0 = place.pos(s);
    const float a2 = -expf(m.a_log[h]) * SC_LOG2E, dt_bias = m.dt_bias[h], skip = m.d_skip[h];
    const size_t row_base = (size_t)s * place.chunk;
    const bf16* xbc = reinterpret_cast<const bf16*>(m.xbc) + row_base * channels;
    const bf16* zb = reinterpret_cast<const bf16*>(m.proj) + row_base * m.ld + h * m.vdim + p_first;
    bf16* gb = reinterpret_cast<bf16*>(m.gated) + row_base * inner + h * m.vdim + p_first;
    float* state = m.ssm + (((size_t)s * m.heads + h) * m.state) * m.vdim + p_first;

    // one operand tile: 64 rows of `w` channels from channel c0 on; rows past the chunk's end and channels past w are zero
    auto load_tile = [&](uint8_t* dst, uint32_t pitch, uint32_t padded, uint32_t c0, uint32_t w, uint32_t t0) {
        const uint32_t live = min((uint32_t)SC_Q, place.chunk - t0);
        if (vec) {
            // a thread keeps its 16-byte column and walks down the rows
            const uint32_t ch = padded / 8, step = 128 / ch, r0 = tid / ch, c = (tid % ch) * 8;
            const bf16* src = xbc + (size_t)(t0 + r0) * channels + c0 + c;
            uint8_t* to = dst + r0 * pitch + c * 2;
            const uint32_t n = c < w && live > r0 ? live - r0 : 0u;     // rows of this thread's column that exist, from r0 on
#pragma unroll 8
            for (uint32_t r = 0; r < SC_Q; r += step) {
                mx_cp16(to, r < n ? src : xbc, r < n);
                src += (size_t)step * channels;
                to += step * pitch;
            }
        } else {
            for (uint32_t i = tid; i < SC_Q * padded; i += 128) {
                const uint32_t r = i / padded, c = i % padded;
                *reinterpret_cast<bf16*>(dst + r * pitch + c * 2) =
                    r < live && c < w ? xbc[(size_t)(t0 + r) * channels + c0 + c] : __float2bfloat16_rn(0.0f);
            }
        }
    };
    auto load_c = [&](uint32_t t0) {
        if (t0 < place.chunk) load_tile(smem + S::B_BYTES, S::BP, NP, inner + gn + group * m.state, m.state, t0);
        mx_commit();
    };
    auto load_bx = [&](uint32_t t0) {
        if (t0 < place.chunk) {
            load_tile(smem, S::BP, NP, inner + group * m.state, m.state, t0);
            load_tile(smem + 2 * S::B_BYTES, S::XP, SC_P, h * m.vdim + p_first, width, t0);
        }
        mx_commit();
    };
    // warp 0: raw steps of tokens 2 lane, 2 lane + 1 of the chunk at t0; -inf (step 0) past the end
    float raw[2];
    auto fetch_steps = [&](uint32_t t0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t t = t0 + 2 * lane + i;
            raw[i] = t < place.chunk ? m.dt[(row_base + t) * m.dt_ld + h] + dt_bias : -INFINITY;
        }
    };
    auto make_decays = [&](uint32_t buf) {
        float dt[2], d2[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            dt[i] = raw[i] > 20.0f ? raw[i] : log1pf(expf(raw[i]));
            d2[i] = a2 * dt[i];
        }
        float sum = d2[0] + d2[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= (uint32_t)o) sum += up;
        }
        s_cum[buf][2 * lane + 1] = sum;
        s_cum[buf][2 * lane] = sum - d2[1];
        s_dt[buf][2 * lane] = dt[0];
        s_dt[buf][2 * lane + 1] = dt[1];
    };

    load_c(0);
    load_bx(0);
    if (warp == 0) fetch_steps(0);
    // S^T: rows p = pw + g8 (+ 8), columns n = nt * 8 + t4 * 2 (+ 1)
    float acc[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const uint32_t p = pw + g8 + (e >> 1) * 8, n = nt * 8 + t4 * 2 + (e & 1);
            acc[nt][e] = p0 > 0 && n < m.state && p < width ? state[(size_t)n * m.vdim + p] : 0.0f;
        }
    if (warp == 0) {
        make_decays(0);
        fetch_steps(SC_Q);
    }

    uint32_t buf = 0;
    for (uint32_t t0 = 0; t0 < place.chunk; t0 += SC_Q, buf ^= 1) {
        mx_wait<0>();
        __syncthreads();     // this chunk's tiles and decays are in place; everyone is done with the weights of the last one
        const uint32_t sb = mx_smem(smem), sc = sb + S::B_BYTES;
        const uint8_t* sx = smem + 2 * S::B_BYTES;
        const uint32_t sx_a = mx_smem(sx);
        const float *cum = s_cum[buf], *dts = s_dt[buf];
        const uint32_t a_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::BP + (lane >> 4) * 16;      // A operand, row-major tiles
        const uint32_t b_off = ((lane & 7) + (lane >> 4) * 8) * S::BP + ((lane >> 3) & 1) * 16;      // B operand, [n][k] tiles
        // ---- decayed weights of the warp's 16 token rows: columns up to the diagonal block ----
        {
            float gm[SC_Q / 8][4];
#pragma unroll
            for (int i = 0; i < SC_Q / 8; ++i) gm[i][0] = gm[i][1] = gm[i][2] = gm[i][3] = 0.0f;
#pragma unroll 2
            for (int kk = 0; kk < NP / 16; ++kk) {
                uint32_t ca[4], bb[4];
                mx_ldsm(sc + a_off + warp * 16 * S::BP + kk * 32, ca);
#pragma unroll
                for (int n = 0; n < SC_Q / 16; ++n) {
                    if ((uint32_t)n > warp) continue;
                    mx_ldsm(sb + b_off + n * 16 * S::BP + kk * 32, bb);
                    mx_mma(gm[2 * n], ca, bb[0], bb[1]);
                    mx_mma(gm[2 * n + 1], ca, bb[2], bb[3]);
                }
            }
            const uint32_t i0 = warp * 16 + g8, i1 = i0 + 8;
            const float cum0 = cum[i0], cum1 = cum[i1];
#pragma unroll
            for (int n = 0; n < SC_Q / 8; ++n) {
                if ((uint32_t)(n >> 1) > warp) continue;
                const uint32_t j = n * 8 + t4 * 2;
                const float2 cj = *reinterpret_cast<const float2*>(cum + j), dj = *reinterpret_cast<const float2*>(dts + j);
                const float w0 = j <= i0 ? gm[n][0] * mx_ex2(cum0 - cj.x) * dj.x : 0.0f;
                const float w1 = j + 1 <= i0 ? gm[n][1] * mx_ex2(cum0 - cj.y) * dj.y : 0.0f;
                const float w2 = j <= i1 ? gm[n][2] * mx_ex2(cum1 - cj.x) * dj.x : 0.0f;
                const float w3 = j + 1 <= i1 ? gm[n][3] * mx_ex2(cum1 - cj.y) * dj.y : 0.0f;
                uint32_t hi, lo;
                split_bf16x2(w0, w1, hi, lo);
                *reinterpret_cast<uint32_t*>(swh + i0 * S::WP + j * 2) = hi;
                *reinterpret_cast<uint32_t*>(swl + i0 * S::WP + j * 2) = lo;
                split_bf16x2(w2, w3, hi, lo);
                *reinterpret_cast<uint32_t*>(swh + i1 * S::WP + j * 2) = hi;
                *reinterpret_cast<uint32_t*>(swl + i1 * S::WP + j * 2) = lo;
            }
        }
        // ---- C . S_in, scaled by the decay since the chunk's start ----
        float y[4][2][4];
#pragma unroll
        for (int mt = 0; mt < 4; ++mt)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) y[mt][nt][0] = y[mt][nt][1] = y[mt][nt][2] = y[mt][nt][3] = 0.0f;
        if (owner) {
#pragma unroll
            for (int kk = 0; kk < NP / 16; ++kk) {
                // state rows 16 kk .. + 15: accumulator tiles 2 kk (k 0-7) and 2 kk + 1 (k 8-15); registers 0, 1 are columns
                // pw .. + 7, registers 2, 3 columns pw + 8 .. + 15
                uint32_t h00, l00, h01, l01, h10, l10, h11, l11;
                split_bf16x2(acc[2 * kk][0], acc[2 * kk][1], h00, l00);
                split_bf16x2(acc[2 * kk + 1][0], acc[2 * kk + 1][1], h01, l01);
                split_bf16x2(acc[2 * kk][2], acc[2 * kk][3], h10, l10);
                split_bf16x2(acc[2 * kk + 1][2], acc[2 * kk + 1][3], h11, l11);
                // (products of one accumulator are kept eight apart: each waits for the one before it)
                uint32_t ca[4][4];
#pragma unroll
                for (int mt = 0; mt < 4; ++mt) mx_ldsm(sc + a_off + mt * 16 * S::BP + kk * 32, ca[mt]);
#pragma unroll
                for (int mt = 0; mt < 4; ++mt) {
                    mx_mma(y[mt][0], ca[mt], h00, h01);
                    mx_mma(y[mt][1], ca[mt], h10, h11);
                }
#pragma unroll
                for (int mt = 0; mt < 4; ++mt) {
                    mx_mma(y[mt][0], ca[mt], l00, l01);
                    mx_mma(y[mt][1], ca[mt], l10, l11);
                }
            }
#pragma unroll
            for (int mt = 0; mt < 4; ++mt) {
                const float e0 = mx_ex2(cum[mt * 16 + g8]), e1 = mx_ex2(cum[mt * 16 + 8 + g8]);
#pragma unroll
                for (int nt = 0; nt < 2; ++nt) { y[mt][nt][0] *= e0; y[mt][nt][1] *= e0; y[mt][nt][2] *= e1; y[mt][nt][3] *= e1; }
            }
        }
        __syncthreads();     // the weights of all rows are in place, C has been used up
        load_c(t0 + SC_Q);
        if (owner) {
            // gate inputs of this warp's outputs: rows mt * 16 + half * 8 + g8, columns pw + nt * 8 + t4 * 2
            uint32_t z[4][2][2];
            const uint32_t c0 = pw + t4 * 2, live = place.chunk - t0 > g8 ? place.chunk - t0 - g8 : 0u;   // rows from g8 on
            {
                const bf16* src = zb + (size_t)(t0 + g8) * m.ld + c0;
                const size_t down = (size_t)8 * m.ld;
#pragma unroll
                for (int rr = 0; rr < 8; ++rr, src += down)
#pragma unroll
                    for (int nt = 0; nt < 2; ++nt) {
                        uint32_t v = 0u;
                        if ((uint32_t)rr * 8 < live && c0 + nt * 8 < width) {
                            if (vec) v = __ldg(reinterpret_cast<const uint32_t*>(src + nt * 8));
                            else v = (uint32_t)__bfloat16_as_ushort(src[nt * 8]) | (c0 + nt * 8 + 1 < width ? (uint32_t)__bfloat16_as_ushort(src[nt * 8 + 1]) << 16 : 0u);
                        }
                        z[rr >> 1][rr & 1][nt] = v;
                    }
            }
            // ---- weights . x ----
            const uint32_t w_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::WP + (lane >> 4) * 16;
            const uint32_t x_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::XP + (lane >> 4) * 16 + pw * 2;    // [token][p]: B operand, transposed
            const uint32_t swh_a = mx_smem(swh), swl_a = mx_smem(swl);
#pragma unroll 1
            for (int kk = 0; kk < SC_Q / 16; ++kk) {
                uint32_t xb[4], wa[4];
                mx_ldsm_t(sx_a + x_off + kk * 16 * S::XP, xb);
#pragma unroll
                for (int mt = 0; mt < 4; ++mt) {
                    if (mt < kk) continue;
                    mx_ldsm(swh_a + w_off + mt * 16 * S::WP + kk * 32, wa);
                    mx_mma(y[mt][0], wa, xb[0], xb[1]);
                    mx_mma(y[mt][1], wa, xb[2], xb[3]);
                }
#pragma unroll
                for (int mt = 0; mt < 4; ++mt) {
                    if (mt < kk) continue;
                    mx_ldsm(swl_a + w_off + mt * 16 * S::WP + kk * 32, wa);
                    mx_mma(y[mt][0], wa, xb[0], xb[1]);
                    mx_mma(y[mt][1], wa, xb[2], xb[3]);
                }
            }
            // ---- skip, gate, store ----
            {
                bf16* out = gb + (size_t)(t0 + g8) * inner + c0;
                const uint8_t* xr = sx + g8 * S::XP + c0 * 2;
                const size_t down = (size_t)8 * inner;
#pragma unroll
                for (int rr = 0; rr < 8; ++rr, out += down) {
                    if ((uint32_t)rr * 8 >= live) break;
#pragma unroll
                    for (int nt = 0; nt < 2; ++nt) {
                        if (c0 + nt * 8 >= width) continue;
                        const float2 x = bf16x2_to_f32(*reinterpret_cast<const uint32_t*>(xr + rr * 8 * S::XP + nt * 16));
                        const float2 zz = bf16x2_to_f32(z[rr >> 1][rr & 1][nt]);
                        const float v0 = fmaf(skip, x.x, y[rr >> 1][nt][2 * (rr & 1)]) * mx_silu(zz.x);
                        const float v1 = fmaf(skip, x.y, y[rr >> 1][nt][2 * (rr & 1) + 1]) * mx_silu(zz.y);
                        store_pair<bf16>(out + nt * 8, make_float2(v0, v1), vec, c0 + nt * 8 + 1 < width);
                    }
                }
            }
            // ---- S^T at the end of the chunk: decayed, plus (x_j weighted by what is left of it)^T . B ----
            const float last = cum[SC_Q - 1], el = mx_ex2(last);
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) { acc[nt][0] *= el; acc[nt][1] *= el; acc[nt][2] *= el; acc[nt][3] *= el; }
            const uint32_t xt_off = ((lane & 7) + (lane >> 4) * 8) * S::XP + ((lane >> 3) & 1) * 16 + pw * 2;   // x^T: A operand from [token][p]
            const uint32_t bt_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::BP + (lane >> 4) * 16;            // B: B operand from [token][n]
#pragma unroll 1
            for (int kk = 0; kk < SC_Q / 16; ++kk) {
                uint32_t xa[4], xh[4], xl[4];
                mx_ldsm_t(sx_a + xt_off + kk * 16 * S::XP, xa);
                // registers 0, 1 hold tokens t4 * 2 (+ 1), registers 2, 3 tokens 8 + t4 * 2 (+ 1)
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const uint32_t j = kk * 16 + r * 8 + t4 * 2;
                    const float2 cj = *reinterpret_cast<const float2*>(cum + j), dj = *reinterpret_cast<const float2*>(dts + j);
                    const float w0 = mx_ex2(last - cj.x) * dj.x, w1 = mx_ex2(last - cj.y) * dj.y;
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        const float2 x = bf16x2_to_f32(xa[2 * r + q]);
                        split_bf16x2(x.x * w0, x.y * w1, xh[2 * r + q], xl[2 * r + q]);
                    }
                }
#pragma unroll
                for (int n = 0; n < NT / 4; ++n) {
                    uint32_t b0[4], b1[4];
                    mx_ldsm_t(sb + bt_off + kk * 16 * S::BP + n * 64, b0);
                    mx_ldsm_t(sb + bt_off + kk * 16 * S::BP + n * 64 + 32, b1);
                    mx_mma(acc[4 * n], xh, b0[0], b0[1]);
                    mx_mma(acc[4 * n + 1], xh, b0[2], b0[3]);
                    mx_mma(acc[4 * n + 2], xh, b1[0], b1[1]);
                    mx_mma(acc[4 * n + 3], xh, b1[2], b1[3]);
                    mx_mma(acc[4 * n], xl, b0[0], b0[1]);
                    mx_mma(acc[4 * n + 1], xl, b0[2], b0[3]);
                    mx_mma(acc[4 * n + 2], xl, b1[0], b1[1]);
                    mx_mma(acc[4 * n + 3], xl, b1[2], b1[3]);
                }
            }
        }
        if (warp == 0) {     // the other buffer's decays: last read before this iteration's first barrier
            make_decays(buf ^ 1);
            fetch_steps(t0 + 2 * SC_Q);
        }
        __syncthreads();     // B and x have been used up
        load_bx(t0 + SC_Q);
    }
    mx_wait<0>();
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const uint32_t p = pw + g8 + (e >> 1) * 8, n = nt * 8 + t4 * 2 + (e & 1);
            if (n < m.state && p < width) state[(size_t)n * m.vdim + p] = acc[nt][e];
        }
}

template <int NP>
static int launch_scan(const Mamba2& m, const StepPlace& place, uint32_t vec, cudaStream_t stream) {
    static bool configured[64] = {};
    const uint32_t bytes = ScanShape<NP>::BYTES;
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64 || !configured[dev]) {
        if (cudaFuncSetAttribute(ssd_scan_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
            return check_launch("ssd_scan attribute");
        if (dev >= 0 && dev < 64) configured[dev] = true;
    }
    launch_kernel(ssd_scan_kernel<NP>, dim3(ceil_div(m.vdim, SC_P), m.heads, place.sessions), dim3(128), bytes, stream, m, place, vec);
    count_launch();
    return check_launch("ssd_scan");
}

// Rows of xbc hold the convolved x | B | C of every token of the chunk.
int launch_ssd_scan(const Mamba2& m, const StepPlace& place, cudaStream_t stream) {
    const uint32_t inner = m.heads * m.vdim;
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const uint32_t vec = m.vdim % 8 == 0 && m.state % 8 == 0 && m.ld % 2 == 0 && inner % 8 == 0 && aligned(m.xbc) && aligned(m.proj) && aligned(m.gated);
    if (m.state <= 64) return launch_scan<64>(m, place, vec, stream);
    if (m.state <= 128) return launch_scan<128>(m, place, vec, stream);
    return launch_scan<256>(m, place, vec, stream);
}

}  // namespace tb
