// Chunked scan of HGRN2 on the warp-level tensor cores.
//
// Chunks of 16 tokens.  With P_i the product of the forget gates of the chunk's tokens 0 .. i (per channel), R_j that of
// tokens j + 1 .. 15, k = 1 - f:
//     o_i   = (q_i P_i)^T S_in + sum_{j <= i} [(q_i P_i) . (k_j / P_j)] v_j
//     S_out = diag(P_15) S_in + sum_j (k_j R_j) v_j^T
// Products of gates instead of exponentials of summed logarithms: no special functions, and a factor is exact to a few ulp.
// k_j / P_j grows as the gates shrink; a chunk in which some P_15 falls below 1e-30 (sixteen gates of 0.013 on average) forms
// its inner weights gate by gate instead (`slow_weights`), so that the result never rests on how small a gate may get.
//
// A CTA owns the whole sequence of one (session, head, up to 128 columns of the state).  Each warp owns 16 columns and keeps
// its part of S transposed in accumulator registers (rows = its columns, from v^T . k): in that layout the accumulators of
// S^T are, register by register, the B operand of q . S, so the state never passes through shared memory.  Every warp forms
// the 16 x 16 inner weights itself (their accumulators are the A operand of the product with v), and all warps make the
// operands of the next chunk (gates, running products, silu), so one barrier per chunk is enough.  The RMS norm of the
// output waits in registers for the next chunk's barrier, behind which the other warps' sums of squares are in place.
//
// The state, the written k R, k / P and the inner weights enter the products as two bf16 halves (split_bf16x2), so that they
// keep 16 bits; the readout's q P is rounded to bf16 like q itself, v is bf16.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

constexpr int HS_Q = 16;
constexpr float HS_TINY = 1e-30f, HS_LOG2E = 1.4426950408889634f;

template <int NP, int WARPS>
struct HsShape {
    static constexpr uint32_t NPITCH = NP * 2 + 16, VPITCH = WARPS * 32 + 16;     // bytes; conflict-free ldmatrix
    static constexpr uint32_t OP = HS_Q * NPITCH;                                 // one operand half
    static constexpr uint32_t V_BYTES = HS_Q * VPITCH;
    static constexpr uint32_t STAGE = 5 * OP + V_BYTES + NP * 4;                  // qP, k/P and kR in two halves, v, P_15
    static constexpr uint32_t SPITCH = 18;                                        // floats: weights formed gate by gate, per warp
    static constexpr uint32_t BYTES = 2 * STAGE + WARPS * HS_Q * SPITCH * 4;
};

// f = l + (1 - l) sigmoid(z) and k = (1 - l) sigmoid(-z) from t = exp(-z): sigmoid(-z) = t sigmoid(z), so that neither end
// loses digits.  z2 = -log2(e) z; the bound keeps t finite (sigmoid(z) is zero to f32 long before).
__device__ __forceinline__ void hs_gate(float z2, float lower, float rest, float& f, float& k) {
    const float t = mx_ex2(fminf(z2, 120.0f)), s = mx_rcp(1.0f + t);
    f = fmaf(rest, s, lower);
    k = rest * (t * s);
}

// NP: channels padded to a multiple of 64; WARPS: 16 columns each.
template <int NP, int WARPS>
__global__ void __launch_bounds__(WARPS * 32, NP <= 64 ? (WARPS == 4 ? 4 : 2) : NP <= 128 ? (WARPS == 4 ? 2 : 1) : 1)
hgrn2_scan_kernel(Hgrn2 m, StepPlace place, uint32_t vec) {
    using S = HsShape<NP, WARPS>;
    constexpr int NT = NP / 8, GROUPS = NP / 16, MINE = (GROUPS + WARPS - 1) / WARPS;    // 16-channel groups, per warp
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ float s_sq[2][WARPS][HS_Q];
    __shared__ uint32_t s_tiny[4];            // by chunk modulo 4: one is set, one read and one cleared between two barriers
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t c_first = blockIdx.x * (WARPS * 16), h = blockIdx.y, s = blockIdx.z;
    const uint32_t width = min((uint32_t)(WARPS * 16), m.vdim - c_first);
    const uint32_t pw = warp * 16;              // the warp's columns
    const bool owner = pw < width, fused = m.vdim <= HGRN2_FUSED_VDIM;
    if (tid < 4) s_tiny[tid] = 0;
    pdl_wait();
    pdl_trigger();
    const uint32_t p0 = place.pos(s);
    const size_t row_base = (size_t)s * place.chunk;
    const float* fb = m.f + row_base * m.f_ld + h * m.dim;
    const bf16* qb = reinterpret_cast<const bf16*>(m.q) + row_base * m.ld + h * m.dim;
    const bf16* vb = reinterpret_cast<const bf16*>(m.v) + row_base * m.ld + h * m.vdim + c_first;
    float* state = m.state + (((size_t)s * m.heads + h) * m.dim) * m.vdim + c_first;

    // ---- operands of a chunk: a lane owns two channels of four tokens of a 16-channel group ----
    const uint32_t p8 = lane & 7, tq = lane >> 3;
    float bias2[MINE][2], lower[MINE][2];       // channels past the last one: lower 1, that is f = 1 and k = 0
#pragma unroll
    for (int i = 0; i < MINE; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const uint32_t c = (warp + i * WARPS) * 16 + p8 * 2 + e;
            bias2[i][e] = c < m.dim ? -HS_LOG2E * m.f_bias[h * m.dim + c] : 0.0f;
            lower[i][e] = c < m.dim ? m.lower[h * m.dim + c] : 1.0f;
        }
    float2 raw_f[MINE][4];
    uint32_t raw_q[MINE][4];
    auto fetch = [&](uint32_t t0) {
#pragma unroll
        for (int i = 0; i < MINE; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const uint32_t c = (warp + i * WARPS) * 16 + p8 * 2, t = t0 + tq * 4 + j;
                raw_f[i][j] = make_float2(0.0f, 0.0f);
                raw_q[i][j] = 0u;
                if (t < place.chunk && c < m.dim) {
                    const float* f = fb + (size_t)t * m.f_ld + c;
                    const bf16* q = qb + (size_t)t * m.ld + c;
                    if (vec) {
                        raw_f[i][j] = *reinterpret_cast<const float2*>(f);
                        raw_q[i][j] = *reinterpret_cast<const uint32_t*>(q);
                    } else {
                        const bool second = c + 1 < m.dim;
                        raw_f[i][j] = make_float2(f[0], second ? f[1] : 0.0f);
                        raw_q[i][j] = (uint32_t)__bfloat16_as_ushort(q[0]) | (second ? (uint32_t)__bfloat16_as_ushort(q[1]) << 16 : 0u);
                    }
                }
            }
    };
    auto load_v = [&](uint32_t t0, uint8_t* stage) {
        uint8_t* dst = stage + 5 * S::OP;
        if (t0 < place.chunk) {
            if (vec) {
                for (uint32_t i = tid; i < HS_Q * WARPS * 2; i += WARPS * 32) {
                    const uint32_t r = i / (WARPS * 2), c = (i % (WARPS * 2)) * 8;
                    const bool real = t0 + r < place.chunk && c < width;
                    mx_cp16(dst + r * S::VPITCH + c * 2, real ? vb + (size_t)(t0 + r) * m.ld + c : vb, real);
                }
            } else {
                for (uint32_t i = tid; i < HS_Q * WARPS * 16; i += WARPS * 32) {
                    const uint32_t r = i / (WARPS * 16), c = i % (WARPS * 16);
                    *reinterpret_cast<bf16*>(dst + r * S::VPITCH + c * 2) =
                        t0 + r < place.chunk && c < width ? vb[(size_t)(t0 + r) * m.ld + c] : __float2bfloat16_rn(0.0f);
                }
            }
        }
        mx_commit();
    };
    auto prepare = [&](uint32_t t0, uint8_t* stage) {
        const bool whole = t0 + HS_Q <= place.chunk;
#pragma unroll
        for (int i = 0; i < MINE; ++i) {
            const uint32_t grp = warp + i * WARPS, c = grp * 16 + p8 * 2;
            if (grp >= GROUPS) continue;       // warp-uniform
            float f[4][2], k[4][2], q[4][2], run[4][2], left[4][2], before[2], after[2], all[2];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 qv = bf16x2_to_f32(raw_q[i][j]);
                const float z[2] = {raw_f[i][j].x, raw_f[i][j].y}, qq[2] = {qv.x, qv.y};
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    hs_gate(fmaf(z[e], -HS_LOG2E, bias2[i][e]), lower[i][e], 1.0f - lower[i][e], f[j][e], k[j][e]);
                    q[j][e] = mx_silu(qq[e]);      // 0 past the end and past the last channel
                }
                if (!whole && t0 + tq * 4 + j >= place.chunk) { f[j][0] = f[j][1] = 1.0f; k[j][0] = k[j][1] = 0.0f; }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                run[0][e] = f[0][e];
                left[3][e] = 1.0f;
#pragma unroll
                for (int j = 1; j < 4; ++j) { run[j][e] = run[j - 1][e] * f[j][e]; left[3 - j][e] = left[4 - j][e] * f[4 - j][e]; }
                // products of the other quarters' four gates, before and after this one
                float x = run[3][e], y = run[3][e], u;
                u = __shfl_up_sync(0xffffffffu, x, 8);
                if (tq >= 1) x *= u;
                u = __shfl_up_sync(0xffffffffu, x, 16);
                if (tq >= 2) x *= u;
                u = __shfl_up_sync(0xffffffffu, x, 8);
                before[e] = tq >= 1 ? u : 1.0f;
                all[e] = __shfl_sync(0xffffffffu, x, 24 + p8);
                u = __shfl_down_sync(0xffffffffu, y, 8);
                if (tq <= 2) y *= u;
                u = __shfl_down_sync(0xffffffffu, y, 16);
                if (tq <= 1) y *= u;
                u = __shfl_down_sync(0xffffffffu, y, 8);
                after[e] = tq <= 2 ? u : 1.0f;
            }
            if (fminf(all[0], all[1]) < HS_TINY) s_tiny[t0 / HS_Q & 3] = 1u;        // every writer stores the same
            if (tq == 0) *reinterpret_cast<float2*>(stage + 5 * S::OP + S::V_BYTES + c * 4) = make_float2(all[0], all[1]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                uint8_t* dst = stage + (tq * 4 + j) * S::NPITCH + c * 2;
                float qp[2], kp[2], kr[2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float p = before[e] * run[j][e];
                    qp[e] = q[j][e] * p;
                    kp[e] = k[j][e] * mx_rcp(p);          // not used when the chunk is marked tiny
                    kr[e] = k[j][e] * (left[j][e] * after[e]);
                }
                uint32_t hi, lo;
                *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(qp[0], qp[1]);
                split_bf16x2(kp[0], kp[1], hi, lo);
                *reinterpret_cast<uint32_t*>(dst + S::OP) = hi;
                *reinterpret_cast<uint32_t*>(dst + 2 * S::OP) = lo;
                split_bf16x2(kr[0], kr[1], hi, lo);
                *reinterpret_cast<uint32_t*>(dst + 3 * S::OP) = hi;
                *reinterpret_cast<uint32_t*>(dst + 4 * S::OP) = lo;
            }
        }
    };
    // Inner weights of a chunk gate by gate, in the layout of the product's accumulators.
    auto slow_weights = [&](uint32_t t0, float (&gm)[2][4]) {
        float* mine = reinterpret_cast<float*>(smem + 2 * S::STAGE) + warp * HS_Q * S::SPITCH;
        for (uint32_t j = 0; j < HS_Q; ++j) {
            float g[NP / 32];
#pragma unroll
            for (int n = 0; n < NP / 32; ++n) g[n] = 0.0f;
            for (uint32_t i = j; i < HS_Q; ++i) {
                float sum = 0.0f;
#pragma unroll
                for (int n = 0; n < NP / 32; ++n) {
                    const uint32_t c = lane + 32 * n, t = t0 + i;
                    if (c >= m.dim || t >= place.chunk) continue;
                    const float lo = m.lower[h * m.dim + c];
                    float f, k;
                    hs_gate(-HS_LOG2E * (fb[(size_t)t * m.f_ld + c] + m.f_bias[h * m.dim + c]), lo, 1.0f - lo, f, k);
                    g[n] = i == j ? k : g[n] * f;
                    sum = fmaf(mx_silu(__bfloat162float(qb[(size_t)t * m.ld + c])), g[n], sum);
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
                if (lane == 0) mine[i * S::SPITCH + j] = sum;
            }
        }
        __syncwarp();
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) gm[nt][e] = mine[(g8 + (e >> 1) * 8) * S::SPITCH + nt * 8 + t4 * 2 + (e & 1)];      // above the diagonal: anything
        __syncwarp();
    };

    // S^T: rows p = pw + g8 (+ 8), columns n = nt * 8 + t4 * 2 (+ 1)
    float acc[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const uint32_t p = pw + g8 + (e >> 1) * 8, n = nt * 8 + t4 * 2 + (e & 1);
            acc[nt][e] = p0 > 0 && n < m.dim && p < width ? state[(size_t)n * m.vdim + p] : 0.0f;
        }
    float nw[4];       // norm weights of the lane's output columns pw + t4 * 2 (+ 1, + 8, + 9)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const uint32_t p = pw + (e >> 1) * 8 + t4 * 2 + (e & 1);
        nw[e] = fused && p < width ? m.norm_w[p] * m.gain : 0.0f;
    }
    fetch(0);
    load_v(0, smem);
    __syncthreads();       // s_tiny is clear
    prepare(0, smem);
    fetch(HS_Q);

    const uint32_t a_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::NPITCH + (lane >> 4) * 16;     // A operand, [token][channel]
    const uint32_t b_off = ((lane & 7) + (lane >> 4) * 8) * S::NPITCH + ((lane >> 3) & 1) * 16;     // B operand, [n = token][k = channel]
    const uint32_t bt_off = a_off;                                                                  // B operand, [k = token][n = channel], transposed
    const uint32_t v_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * S::VPITCH + (lane >> 4) * 16 + pw * 2;     // [k = token][n = column], transposed
    const uint32_t vt_off = ((lane & 7) + (lane >> 4) * 8) * S::VPITCH + ((lane >> 3) & 1) * 16 + pw * 2;    // v^T: A operand from [token][column]
    float y[2][4];         // outputs: rows g8 (+ 8), columns pw + nt * 8 + t4 * 2 (+ 1); kept until the next chunk's norm
    const float inv_vdim = 1.0f / (float)m.vdim;
    auto finish = [&](uint32_t t0) {
        const uint32_t at = t0 / HS_Q & 1;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const uint32_t t = t0 + g8 + half * 8;
            if (t >= place.chunk || !owner) continue;
            if (!fused) {
                float* raw = m.raw + (row_base + t) * ((size_t)m.heads * m.vdim) + h * m.vdim + c_first;
#pragma unroll
                for (int nt = 0; nt < 2; ++nt) {
                    const uint32_t p = pw + nt * 8 + t4 * 2;
                    if (p < width) raw[p] = y[nt][2 * half];
                    if (p + 1 < width) raw[p + 1] = y[nt][2 * half + 1];
                }
                continue;
            }
            float total = 0.0f;
#pragma unroll
            for (int w = 0; w < WARPS; ++w) total += s_sq[at][w][g8 + half * 8];
            const float inv = rsqrtf(fmaf(total, inv_vdim, m.eps));
            bf16* out = reinterpret_cast<bf16*>(m.out) + (row_base + t) * m.out_ld + h * m.vdim;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                const uint32_t p = pw + nt * 8 + t4 * 2;
                if (p < width)
                    store_pair<bf16>(out + p, make_float2(y[nt][2 * half] * inv * nw[2 * nt], y[nt][2 * half + 1] * inv * nw[2 * nt + 1]), vec, p + 1 < width);
            }
        }
    };

    uint32_t buf = 0;
    for (uint32_t t0 = 0; t0 < place.chunk; t0 += HS_Q, buf ^= 1) {
        uint8_t* stage = smem + buf * S::STAGE;
        uint8_t* next = smem + (buf ^ 1) * S::STAGE;
        const uint32_t sb = mx_smem(stage), sv = sb + 5 * S::OP;
        mx_wait<0>();
        __syncthreads();       // this chunk's operands and the last one's sums are in place, the last one's operands used up
        if (t0 > 0) finish(t0 - HS_Q);
        load_v(t0 + HS_Q, next);
        const uint32_t turn = t0 / HS_Q;
        const bool slow = s_tiny[turn & 3] != 0;
        if (tid == 0) s_tiny[(turn + 3) & 3] = 0;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[nt][e] = 0.0f;
        if (owner) {
            // ---- q P . S_in and the inner weights q P . k / P ----
            float yl[2][4] = {}, gm[2][4] = {};        // yl: a second accumulator, shorter chains of dependent products
#pragma unroll
            for (int kk = 0; kk < GROUPS; ++kk) {
                uint32_t h00, l00, h01, l01, h10, l10, h11, l11, qh[4], kh[4], kl[4];
                mx_ldsm(sb + a_off + kk * 32, qh);
                mx_ldsm(sb + S::OP + b_off + kk * 32, kh);
                mx_ldsm(sb + 2 * S::OP + b_off + kk * 32, kl);
                split_bf16x2(acc[2 * kk][0], acc[2 * kk][1], h00, l00);
                split_bf16x2(acc[2 * kk + 1][0], acc[2 * kk + 1][1], h01, l01);
                split_bf16x2(acc[2 * kk][2], acc[2 * kk][3], h10, l10);
                split_bf16x2(acc[2 * kk + 1][2], acc[2 * kk + 1][3], h11, l11);
                mx_mma(gm[0], qh, kh[0], kh[1]);
                mx_mma(gm[1], qh, kh[2], kh[3]);
                mx_mma(y[0], qh, h00, h01);
                mx_mma(y[1], qh, h10, h11);
                mx_mma(yl[0], qh, l00, l01);
                mx_mma(yl[1], qh, l10, l11);
                mx_mma(gm[0], qh, kl[0], kl[1]);
                mx_mma(gm[1], qh, kl[2], kl[3]);
            }
            if (slow) slow_weights(t0, gm);
            // ---- inner weights . v ----
            uint32_t wh[4], wl[4], vb4[4];
            mx_ldsm_t(sv + v_off, vb4);
#pragma unroll
            for (int r = 0; r < 4; ++r) {      // A operand: rows g8 (+ 8), columns t4 * 2 (+ 1, + 8, + 9)
                const uint32_t i = g8 + (r & 1) * 8, j = t4 * 2 + (r >> 1) * 8;
                const float w0 = j <= i ? gm[r >> 1][2 * (r & 1)] : 0.0f, w1 = j + 1 <= i ? gm[r >> 1][2 * (r & 1) + 1] : 0.0f;
                split_bf16x2(w0, w1, wh[r], wl[r]);
            }
            mx_mma(y[0], wh, vb4[0], vb4[1]);
            mx_mma(y[1], wh, vb4[2], vb4[3]);
            mx_mma(yl[0], wl, vb4[0], vb4[1]);
            mx_mma(yl[1], wl, vb4[2], vb4[3]);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) y[nt][e] += yl[nt][e];
            // ---- S^T: decayed, plus v^T . (k R) ----
            uint32_t va[4];
            mx_ldsm_t(sv + vt_off, va);
            const float* all = reinterpret_cast<const float*>(stage + 5 * S::OP + S::V_BYTES);
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                const float2 d = *reinterpret_cast<const float2*>(all + nt * 8 + t4 * 2);
                acc[nt][0] *= d.x; acc[nt][1] *= d.y; acc[nt][2] *= d.x; acc[nt][3] *= d.y;
            }
#pragma unroll
            for (int n = 0; n < NT / 2; ++n) {
                uint32_t kh[4], kl[4];
                mx_ldsm_t(sb + 3 * S::OP + bt_off + n * 32, kh);
                mx_ldsm_t(sb + 4 * S::OP + bt_off + n * 32, kl);
                mx_mma(acc[2 * n], va, kh[0], kh[1]);
                mx_mma(acc[2 * n + 1], va, kh[2], kh[3]);
                mx_mma(acc[2 * n], va, kl[0], kl[1]);
                mx_mma(acc[2 * n + 1], va, kl[2], kl[3]);
            }
        }
        float sq0 = 0.0f, sq1 = 0.0f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {      // columns past the width are zero: v is
            sq0 = fmaf(y[nt][0], y[nt][0], fmaf(y[nt][1], y[nt][1], sq0));
            sq1 = fmaf(y[nt][2], y[nt][2], fmaf(y[nt][3], y[nt][3], sq1));
        }
        sq0 += __shfl_xor_sync(0xffffffffu, sq0, 1);
        sq0 += __shfl_xor_sync(0xffffffffu, sq0, 2);
        sq1 += __shfl_xor_sync(0xffffffffu, sq1, 1);
        sq1 += __shfl_xor_sync(0xffffffffu, sq1, 2);
        if (t4 == 0) { s_sq[turn & 1][warp][g8] = sq0; s_sq[turn & 1][warp][g8 + 8] = sq1; }
        if (t0 + HS_Q < place.chunk) {
            prepare(t0 + HS_Q, next);
            fetch(t0 + 2 * HS_Q);       // a whole chunk ahead of its use
        }
    }
    mx_wait<0>();
    __syncthreads();
    finish((place.chunk - 1) / HS_Q * HS_Q);
    if (owner) {
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t p = pw + g8 + (e >> 1) * 8, n = nt * 8 + t4 * 2 + (e & 1);
                if (n < m.dim && p < width) state[(size_t)n * m.vdim + p] = acc[nt][e];
            }
    }
    if (fused && h + 1 == m.heads && m.out_cols > m.heads * m.vdim) {
        const uint32_t pad = m.out_cols - m.heads * m.vdim;
        for (uint64_t i = tid; i < (uint64_t)pad * place.chunk; i += WARPS * 32)
            reinterpret_cast<bf16*>(m.out)[(row_base + i / pad) * m.out_ld + m.heads * m.vdim + i % pad] = __float2bfloat16_rn(0.0f);
    }
}

template <int NP, int WARPS>
static int launch_scan(const Hgrn2& m, const StepPlace& place, uint32_t vec, cudaStream_t stream) {
    static bool configured[64] = {};
    const uint32_t bytes = HsShape<NP, WARPS>::BYTES;
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64 || !configured[dev]) {
        if (cudaFuncSetAttribute(hgrn2_scan_kernel<NP, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
            return check_launch("hgrn2_scan attribute");
        if (dev >= 0 && dev < 64) configured[dev] = true;
    }
    launch_kernel(hgrn2_scan_kernel<NP, WARPS>, dim3(ceil_div(m.vdim, WARPS * 16u), m.heads, place.sessions), dim3(WARPS * 32), bytes, stream, m, place, vec);
    count_launch();
    return check_launch("hgrn2_scan");
}

int launch_hgrn2_scan(const Hgrn2& m, const StepPlace& place, cudaStream_t stream) {
    auto aligned = [](const void* p, uint32_t to) { return reinterpret_cast<uintptr_t>(p) % to == 0; };
    const uint32_t vec = m.vdim % 8 == 0 && m.dim % 2 == 0 && m.ld % 8 == 0 && m.f_ld % 2 == 0 && m.out_ld % 2 == 0 && aligned(m.q, 4) && aligned(m.v, 16) &&
                         aligned(m.f, 8) && aligned(m.out, 4);
    if (m.vdim <= 64) {
        if (m.dim <= 64) return launch_scan<64, 4>(m, place, vec, stream);
        if (m.dim <= 128) return launch_scan<128, 4>(m, place, vec, stream);
        return launch_scan<256, 4>(m, place, vec, stream);
    }
    if (m.dim <= 64) return launch_scan<64, 8>(m, place, vec, stream);
    if (m.dim <= 128) return launch_scan<128, 8>(m, place, vec, stream);
    return launch_scan<256, 8>(m, place, vec, stream);
}

}  // namespace tb
