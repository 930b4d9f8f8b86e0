// Grouped-query attention with capped scores and a sigmoid gate per head, or with sigmoid weights (no sum to divide by),
// over all earlier keys or a window of them; bf16 caches, any widths up to 256.
//
// The query heads that share a key/value head are rows of one matrix product: row r of a (session, key/value head) is
// query token r / per and head r % per of the group (per = heads / kv_heads), so a K/V tile is loaded once for the whole
// group and the rows of a tile differ in their causal limit only.
//
//  * grouped_split_kernel   few rows (decode, short chunks): 16 rows per CTA, the keys divided over splits x 4 warps; each
//                           warp streams its own 16-key tiles through a private cp.async ring (no CTA barrier in the
//                           loop); warps merge through shared memory, splits through a workspace by whichever CTA is last,
//                           in split order, so results do not depend on timing.
//  * grouped_tile_kernel    many rows (prefill): 64 rows per CTA, all warps share double-buffered key tiles.
// Prefill with heads of 64 at a position the host knows runs on the tcgen05 kernel of prefill_tc.cu instead.
//
// Scores, softmax statistics and accumulators are f32; the weights enter the value product as two bf16 halves
// (split_bf16x2), so they keep 16 bits.  A capped score costs three special-function results instead of one:
// cap tanh(u) = cap (1 - 2 / (1 + exp(2u))).  Sigmoid weights (SIGMOID) need neither maximum nor sum: partial results of
// warps and splits are added as they are.  With a window, tiles before the first row's window are never read.
#include <algorithm>

#include "mixers.cuh"

namespace tb {

int launch_grouped_attention_rows(const GroupedAttention& a, const StepPlace& place, int dtype, cudaStream_t stream);

constexpr float GA_LOG2E = 1.4426950408889634f;
constexpr uint32_t GA_MAX_SPLITS = 32;
constexpr uint32_t GA_WARPS = 4;

struct GaScore {
    float pre, post;   // score in log2 units: capped: post * tanh(s * pre / (2 log2 e)); else s * pre
    bool capped;
};
__device__ __forceinline__ float ga_score(float s, const GaScore& f) {
    if (!f.capped) return s * f.pre;
    const float e = mx_ex2(s * f.pre);                   // exp(2u)
    return fmaf(-2.0f * f.post, mx_rcp(e + 1.0f), f.post);
}
// Weight of a key with sigmoid scores: s = q . k, pre = -scale log2(e), bias2 = -bias log2(e).
__device__ __forceinline__ float ga_sigmoid(float s, float pre, float bias2) { return mx_rcp(1.0f + mx_ex2(fmaf(s, pre, bias2))); }
// First visible key of a query at position `limit`.
__device__ __forceinline__ uint32_t ga_first(uint32_t limit, uint32_t window) { return window && limit >= window ? limit + 1 - window : 0u; }
static GaScore make_score(float scale, float softcap) {
    GaScore f;
    f.capped = softcap > 0.0f;
    f.pre = f.capped ? 2.0f * GA_LOG2E * scale / softcap : scale * GA_LOG2E;
    f.post = softcap * GA_LOG2E;
    return f;
}

struct GaParams {
    GroupedAttention a;
    StepPlace place;
    GaScore score;
    uint32_t per, rows;      // heads per key/value head; rows of a (session, key/value head) = chunk * per
    uint32_t row_tiles, splits;
    uint32_t vec;            // 16-byte copies are possible
    uint32_t* done;          // [sessions * kv_heads * row_tiles], zero between launches
    float* partial;          // [.. * splits][16][DV + 2]
};

// `n` rows of `width` bf16 (row pitch src_ld) into shared memory rows of W padded elements; rows from `live` on are zero.
template <int W>
__device__ __forceinline__ void ga_copy(uint8_t* dst, const bf16* src, size_t src_ld, uint32_t n, uint32_t live, uint32_t width,
                                        uint32_t vec, uint32_t tid, uint32_t threads) {
    constexpr uint32_t PITCH = W * 2 + 16, CH = W / 8;
    if (vec) {
        for (uint32_t i = tid; i < n * CH; i += threads) {
            const uint32_t r = i / CH, c = i % CH;
            const bool real = r < live && c * 8 < width;
            mx_cp16(dst + r * PITCH + c * 16, real ? src + (size_t)r * src_ld + c * 8 : src, real);
        }
    } else {
        for (uint32_t i = tid; i < n * W; i += threads) {
            const uint32_t r = i / W, c = i % W;
            *reinterpret_cast<bf16*>(dst + r * PITCH + c * 2) = r < live && c < width ? src[(size_t)r * src_ld + c] : __float2bfloat16_rn(0.0f);
        }
    }
}

__device__ __forceinline__ float ga_gate(const GroupedAttention& a, size_t row, uint32_t h) {
    return a.gate ? a.gain / (1.0f + __expf(-a.gate[row * a.gate_ld + h])) : a.gain;
}
// Columns of the output rows past the last head.
__device__ __forceinline__ void ga_zero_pad(const GroupedAttention& a, size_t row, uint32_t tid, uint32_t threads) {
    for (uint32_t c = a.heads * a.vdim + tid; c < a.out_cols; c += threads)
        reinterpret_cast<bf16*>(a.out)[row * a.out_ld + c] = __float2bfloat16_rn(0.0f);
}

// ---- few rows -------------------------------------------------------------------------
template <int DK, int DV, int STAGES>
struct SplitShape {
    static constexpr uint32_t KP = DK * 2 + 16, VP = DV * 2 + 16;
    static constexpr uint32_t STAGE = 16 * (KP + VP);
    static constexpr uint32_t RING = GA_WARPS * STAGES * STAGE;
    static constexpr uint32_t MERGE = GA_WARPS * 16 * (DV + 2) * 4;
    static constexpr uint32_t BYTES = RING > MERGE ? RING : MERGE;
};

// UPPER: rows 8 .. 15 of the tile are in use (more than 8 rows).
template <int DK, int DV, int STAGES, bool UPPER, bool SIGMOID>
__global__ void __launch_bounds__(GA_WARPS * 32)
grouped_split_kernel(GaParams P) {
    using S = SplitShape<DK, DV, STAGES>;
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ uint32_t s_last;
    const GroupedAttention& a = P.a;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
    const uint32_t split = blockIdx.x, tile = blockIdx.y % P.row_tiles, kvh = blockIdx.y / P.row_tiles, s = blockIdx.z;
    pdl_wait();
    pdl_trigger();
    const uint32_t p0 = P.place.pos(s), row0 = tile * 16;
    const uint32_t n_rows = min(16u, P.rows - row0);
    const uint32_t keys = min(p0 + (row0 + n_rows - 1) / P.per + 1, a.capacity);    // visible to the tile's last row
    const uint32_t tiles = (keys + 15) / 16, first_tile = ga_first(p0 + row0 / P.per, a.window) / 16;      // of the tile's first row
    const uint32_t per_split = (tiles - first_tile + P.splits - 1) / P.splits;
    const uint32_t tile0 = min(tiles, first_tile + split * per_split), tile1 = min(tiles, tile0 + per_split);

    const uint32_t lim0 = p0 + (row0 + min(g8, n_rows - 1)) / P.per, lim1 = p0 + (row0 + min(g8 + 8, n_rows - 1)) / P.per;
    const uint32_t low0 = ga_first(lim0, a.window), low1 = ga_first(lim1, a.window);
    float bias0 = 0.0f, bias1 = 0.0f;      // of the two rows' heads, SIGMOID
    if (SIGMOID && a.head_bias) {
        bias0 = -GA_LOG2E * a.head_bias[kvh * P.per + (row0 + min(g8, n_rows - 1)) % P.per];
        bias1 = -GA_LOG2E * a.head_bias[kvh * P.per + (row0 + min(g8 + 8, n_rows - 1)) % P.per];
    }

    uint8_t* ring = smem + warp * (STAGES * S::STAGE);
    const size_t k_ld = (size_t)a.kv_heads * a.dim, v_ld = (size_t)a.kv_heads * a.vdim;
    auto load = [&](uint32_t i, uint32_t stage) {     // tile i of the session; the pages of a tile's 16 keys are one page
        if (i < tile1) {
            const size_t kr = kv_row(a.paging, s, i * 16, a.capacity);
            const uint32_t live = min(16u, keys - i * 16);
            uint8_t* dst = ring + stage * S::STAGE;
            ga_copy<DK>(dst, reinterpret_cast<const bf16*>(a.k_cache) + kr * k_ld + (size_t)kvh * a.dim, k_ld, 16, live, a.dim, P.vec, lane, 32);
            ga_copy<DV>(dst + 16 * S::KP, reinterpret_cast<const bf16*>(a.v_cache) + kr * v_ld + (size_t)kvh * a.vdim, v_ld, 16, live, a.vdim,
                        P.vec, lane, 32);
        }
        mx_commit();
    };
#pragma unroll
    for (int i = 0; i < STAGES - 1; ++i) load(tile0 + warp + i * GA_WARPS, i);
    // query fragments straight from global memory: rows g8 and g8 + 8
    uint32_t qa[DK / 16][4];
    const bf16* q = reinterpret_cast<const bf16*>(a.q);
    const size_t q_ld = (size_t)a.heads * a.dim;
    auto q_pair = [&](uint32_t r, uint32_t c) -> uint32_t {
        if (r >= n_rows || c >= a.dim) return 0u;
        const uint32_t R = row0 + r;
        const bf16* src = q + ((size_t)s * P.place.chunk + R / P.per) * q_ld + (size_t)(kvh * P.per + R % P.per) * a.dim + c;
        if (P.vec) return *reinterpret_cast<const uint32_t*>(src);
        const uint32_t lo = __bfloat16_as_ushort(src[0]), hi = c + 1 < a.dim ? __bfloat16_as_ushort(src[1]) : 0u;
        return lo | (hi << 16);
    };
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
        qa[kk][0] = q_pair(g8, kk * 16 + t4 * 2);
        qa[kk][1] = UPPER ? q_pair(g8 + 8, kk * 16 + t4 * 2) : 0u;
        qa[kk][2] = q_pair(g8, kk * 16 + 8 + t4 * 2);
        qa[kk][3] = UPPER ? q_pair(g8 + 8, kk * 16 + 8 + t4 * 2) : 0u;
    }
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    uint32_t stage = 0;
    for (uint32_t i = tile0 + warp; i < tile1; i += GA_WARPS) {
        mx_wait<STAGES - 2>();
        __syncwarp();
        const uint32_t sk = mx_smem(ring + stage * S::STAGE), sv = sk + 16 * S::KP;
        float sc[2][4] = {}, odd[2][4] = {};       // even and odd k steps apart: shorter chains of dependent products
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk += 2) {
            uint32_t b[4], c[4];
            mx_ldsm(sk + ((lane & 7) + (lane >> 4) * 8) * S::KP + (kk * 16 + ((lane >> 3) & 1) * 8) * 2, b);
            mx_ldsm(sk + ((lane & 7) + (lane >> 4) * 8) * S::KP + (kk * 16 + 16 + ((lane >> 3) & 1) * 8) * 2, c);
            mx_mma(sc[0], qa[kk], b[0], b[1]);
            mx_mma(sc[1], qa[kk], b[2], b[3]);
            mx_mma(odd[0], qa[kk + 1], c[0], c[1]);
            mx_mma(odd[1], qa[kk + 1], c[2], c[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[n][e] += odd[n][e];
        uint32_t hi[4] = {0u, 0u, 0u, 0u}, lo[4] = {0u, 0u, 0u, 0u};
        if (SIGMOID) {
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float w[4];
#pragma unroll
                for (int e = 0; e < (UPPER ? 4 : 2); ++e) {
                    const uint32_t key = i * 16 + n * 8 + t4 * 2 + (e & 1);
                    const bool seen = key <= (e < 2 ? lim0 : lim1) && key >= (e < 2 ? low0 : low1);
                    w[e] = seen ? ga_sigmoid(sc[n][e], P.score.pre, e < 2 ? bias0 : bias1) : 0.0f;
                }
                split_bf16x2(w[0], w[1], hi[2 * n], lo[2 * n]);
                if (UPPER) split_bf16x2(w[2], w[3], hi[2 * n + 1], lo[2 * n + 1]);
            }
        } else {
        float mx0 = m0, mx1 = m1;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < (UPPER ? 4 : 2); ++e) {
                const uint32_t key = i * 16 + n * 8 + t4 * 2 + (e & 1);
                const bool seen = key <= (e < 2 ? lim0 : lim1) && key >= (e < 2 ? low0 : low1);
                const float v = seen ? ga_score(sc[n][e], P.score) : -INFINITY;
                sc[n][e] = v;
                if (e < 2) mx0 = fmaxf(mx0, v); else mx1 = fmaxf(mx1, v);
            }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        const float ms0 = mx0 == -INFINITY ? 0.0f : mx0, c0 = mx_ex2(m0 - ms0);
        m0 = mx0;
        float ms1 = 0.0f, c1 = 0.0f;
        if (UPPER) {
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            ms1 = mx1 == -INFINITY ? 0.0f : mx1;
            c1 = mx_ex2(m1 - ms1);
            m1 = mx1;
        }
        float r0 = 0.0f, r1 = 0.0f;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const float pa = mx_ex2(sc[n][0] - ms0), pb = mx_ex2(sc[n][1] - ms0);
            r0 += pa + pb;
            split_bf16x2(pa, pb, hi[2 * n], lo[2 * n]);
            if (UPPER) {
                const float pc = mx_ex2(sc[n][2] - ms1), pd = mx_ex2(sc[n][3] - ms1);
                r1 += pc + pd;
                split_bf16x2(pc, pd, hi[2 * n + 1], lo[2 * n + 1]);
            }
        }
        l0 = l0 * c0 + r0;
        l1 = l1 * c1 + r1;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n) { o[n][0] *= c0; o[n][1] *= c0; if (UPPER) { o[n][2] *= c1; o[n][3] *= c1; } }
        }
        // 64 columns at a time, the two halves of a weight eight products apart: one accumulator's products wait for each other
#pragma unroll
        for (int n0 = 0; n0 < DV / 16; n0 += 4) {
            uint32_t b[4][4];
#pragma unroll
            for (int n = 0; n < 4; ++n)
                mx_ldsm_t(sv + ((lane & 7) + ((lane >> 3) & 1) * 8) * S::VP + ((n0 + n) * 16 + (lane >> 4) * 8) * 2, b[n]);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                mx_mma(o[2 * (n0 + n)], hi, b[n][0], b[n][1]);
                mx_mma(o[2 * (n0 + n) + 1], hi, b[n][2], b[n][3]);
            }
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                mx_mma(o[2 * (n0 + n)], lo, b[n][0], b[n][1]);
                mx_mma(o[2 * (n0 + n) + 1], lo, b[n][2], b[n][3]);
            }
        }
        __syncwarp();    // every lane is done with the stage that the next load may overwrite
        load(i + (STAGES - 1) * GA_WARPS, (stage + STAGES - 1) % STAGES);
        stage = (stage + 1) % STAGES;
    }
    mx_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    __syncthreads();     // the ring becomes the merge buffer
    // [warp][16 rows][DV + 2]: numerators, then maximum and sum
    constexpr uint32_t RW = DV + 2;
    float* mg = reinterpret_cast<float*>(smem);
    {
        float* mine = mg + warp * 16 * RW;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n) {
            *reinterpret_cast<float2*>(mine + g8 * RW + n * 8 + t4 * 2) = make_float2(o[n][0], o[n][1]);
            if (UPPER) *reinterpret_cast<float2*>(mine + (g8 + 8) * RW + n * 8 + t4 * 2) = make_float2(o[n][2], o[n][3]);
        }
        if (t4 == 0) {
            *reinterpret_cast<float2*>(mine + g8 * RW + DV) = make_float2(m0, l0);
            if (UPPER) *reinterpret_cast<float2*>(mine + (g8 + 8) * RW + DV) = make_float2(m1, l1);
        }
    }
    __syncthreads();
    const size_t slot = ((size_t)s * a.kv_heads + kvh) * P.row_tiles + tile;
    auto finish = [&](uint32_t r, uint32_t c, float v) {
        const uint32_t R = row0 + r, h = kvh * P.per + R % P.per;
        const size_t row = (size_t)s * P.place.chunk + R / P.per;
        reinterpret_cast<bf16*>(a.out)[row * a.out_ld + (size_t)h * a.vdim + c] = __float2bfloat16_rn(v * ga_gate(a, row, h));
    };
    for (uint32_t i = threadIdx.x; i < n_rows * a.vdim; i += blockDim.x) {
        const uint32_t r = i / a.vdim, c = i % a.vdim;
        if (SIGMOID) {
            float sum = 0.0f;
#pragma unroll
            for (uint32_t w = 0; w < GA_WARPS; ++w) sum += mg[(w * 16 + r) * RW + c];
            if (P.splits == 1) finish(r, c, sum);
            else P.partial[((slot * P.splits + split) * 16 + r) * RW + c] = sum;
            continue;
        }
        float mx = -INFINITY;
#pragma unroll
        for (uint32_t w = 0; w < GA_WARPS; ++w) mx = fmaxf(mx, mg[(w * 16 + r) * RW + DV]);
        const float ms = mx == -INFINITY ? 0.0f : mx;
        float num = 0.0f, den = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < GA_WARPS; ++w) {
            const float f = mx_ex2(mg[(w * 16 + r) * RW + DV] - ms);
            num = fmaf(mg[(w * 16 + r) * RW + c], f, num);
            den = fmaf(mg[(w * 16 + r) * RW + DV + 1], f, den);
        }
        if (P.splits == 1) {
            finish(r, c, num / den);
        } else {
            float* dst = P.partial + ((slot * P.splits + split) * 16 + r) * RW;
            dst[c] = num;
            if (c == 0) { dst[DV] = mx; dst[DV + 1] = den; }
        }
    }
    if (kvh == 0 && split == 0)
        for (uint32_t t = row0 / P.per; t <= (row0 + n_rows - 1) / P.per; ++t) ga_zero_pad(a, (size_t)s * P.place.chunk + t, threadIdx.x, blockDim.x);
    if (P.splits == 1) return;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) s_last = atomicAdd(P.done + slot, 1u) + 1 == P.splits;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    for (uint32_t i = threadIdx.x; i < n_rows * a.vdim; i += blockDim.x) {
        const uint32_t r = i / a.vdim, c = i % a.vdim;
        const float* src = P.partial + (slot * P.splits * 16 + r) * RW;
        if (SIGMOID) {
            float sum = 0.0f;
            for (uint32_t w = 0; w < P.splits; ++w) sum += __ldcg(src + (size_t)w * 16 * RW + c);
            finish(r, c, sum);
            continue;
        }
        float mx = -INFINITY;
        for (uint32_t w = 0; w < P.splits; ++w) mx = fmaxf(mx, __ldcg(src + (size_t)w * 16 * RW + DV));
        float num = 0.0f, den = 0.0f;
        for (uint32_t w = 0; w < P.splits; ++w) {
            const float* pw = src + (size_t)w * 16 * RW;
            const float f = mx_ex2(__ldcg(pw + DV) - mx);      // 0 for a split without keys
            num = fmaf(__ldcg(pw + c), f, num);
            den = fmaf(__ldcg(pw + DV + 1), f, den);
        }
        finish(r, c, num / den);
    }
    if (threadIdx.x == 0) P.done[slot] = 0;
}

// ---- many rows -----------------------------------------------------------------------------
template <int DK, int DV, int BK>
struct TileShape {
    static constexpr uint32_t KP = DK * 2 + 16, VP = DV * 2 + 16;
    static constexpr uint32_t Q_BYTES = 64 * KP, K_BYTES = BK * KP, V_BYTES = BK * VP;
    static constexpr uint32_t BYTES = Q_BYTES + 2 * (K_BYTES + V_BYTES);
};

template <int DK, int DV, int BK, bool SIGMOID>
__global__ void __launch_bounds__(128)
grouped_tile_kernel(GaParams P) {
    using S = TileShape<DK, DV, BK>;
    extern __shared__ __align__(16) uint8_t smem[];
    const GroupedAttention& a = P.a;
    uint8_t* sq = smem;
    uint8_t* skv = smem + S::Q_BYTES;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
    pdl_wait();
    pdl_trigger();
    // the tiles with the most keys start first
    const uint32_t tile = P.row_tiles - 1 - blockIdx.x, kvh = blockIdx.y, s = blockIdx.z;
    const uint32_t p0 = P.place.pos(s), row0 = tile * 64, n_rows = min(64u, P.rows - row0);
    const uint32_t keys = min(p0 + (row0 + n_rows - 1) / P.per + 1, a.capacity);
    const uint32_t blocks = (keys + BK - 1) / BK, block0 = ga_first(p0 + row0 / P.per, a.window) / BK;
    const size_t k_ld = (size_t)a.kv_heads * a.dim, v_ld = (size_t)a.kv_heads * a.vdim, q_ld = (size_t)a.heads * a.dim;

    {   // query rows: row r is token r / per, head r % per of the group
        const bf16* q = reinterpret_cast<const bf16*>(a.q) + (size_t)s * P.place.chunk * q_ld + (size_t)kvh * P.per * a.dim;
        for (uint32_t i = threadIdx.x; i < 64 * (DK / 8); i += 128) {
            const uint32_t r = i / (DK / 8), c = (i % (DK / 8)) * 8, R = row0 + r;
            uint8_t* dst = sq + r * S::KP + c * 2;
            const bool row_ok = r < n_rows;
            const bf16* src = q + (size_t)(row_ok ? R / P.per : 0) * q_ld + (size_t)(row_ok ? R % P.per : 0) * a.dim + c;
            if (P.vec) {
                mx_cp16(dst, row_ok && c < a.dim ? src : q, row_ok && c < a.dim);
            } else {
                for (uint32_t j = 0; j < 8; ++j)
                    reinterpret_cast<bf16*>(dst)[j] = row_ok && c + j < a.dim ? src[j] : __float2bfloat16_rn(0.0f);
            }
        }
    }
    auto load = [&](uint32_t b, uint32_t buf) {
        uint8_t* dst = skv + buf * (S::K_BYTES + S::V_BYTES);
#pragma unroll 1
        for (uint32_t j = 0; j < BK; j += 16) {     // 16 keys never straddle pages
            const uint32_t key = b * BK + j;
            const uint32_t live = key < keys ? min(16u, keys - key) : 0u;
            const size_t kr = live ? kv_row(a.paging, s, key, a.capacity) : 0;
            ga_copy<DK>(dst + j * S::KP, reinterpret_cast<const bf16*>(a.k_cache) + kr * k_ld + (size_t)kvh * a.dim, k_ld, 16, live, a.dim,
                        P.vec, threadIdx.x, 128);
            ga_copy<DV>(dst + S::K_BYTES + j * S::VP, reinterpret_cast<const bf16*>(a.v_cache) + kr * v_ld + (size_t)kvh * a.vdim, v_ld, 16, live,
                        a.vdim, P.vec, threadIdx.x, 128);
        }
    };
    load(block0, block0 & 1);
    mx_commit();

    constexpr bool KEEP_Q = DK <= 128;
    uint32_t qa[KEEP_Q ? DK / 16 : 1][4];
    const uint32_t q_addr = mx_smem(sq) + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::KP + (lane >> 4) * 16;
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    const uint32_t r0 = warp * 16 + g8, r1 = r0 + 8;
    const uint32_t lim0 = p0 + (row0 + min(r0, n_rows - 1)) / P.per, lim1 = p0 + (row0 + min(r1, n_rows - 1)) / P.per;
    const uint32_t warp_first = p0 + (row0 + min(warp * 16, n_rows - 1)) / P.per;          // limit of the warp's first row
    const uint32_t warp_last = p0 + (row0 + min(warp * 16 + 15, n_rows - 1)) / P.per;
    const uint32_t low0 = ga_first(lim0, a.window), low1 = ga_first(lim1, a.window);
    const uint32_t warp_low = ga_first(warp_first, a.window), warp_low_last = ga_first(warp_last, a.window);
    float bias0 = 0.0f, bias1 = 0.0f;      // of the two rows' heads, SIGMOID
    if (SIGMOID && a.head_bias) {
        bias0 = -GA_LOG2E * a.head_bias[kvh * P.per + (row0 + min(r0, n_rows - 1)) % P.per];
        bias1 = -GA_LOG2E * a.head_bias[kvh * P.per + (row0 + min(r1, n_rows - 1)) % P.per];
    }

    for (uint32_t b = block0; b < blocks; ++b) {
        if (b + 1 < blocks) load(b + 1, (b + 1) & 1);
        mx_commit();
        mx_wait<1>();
        __syncthreads();
        if (KEEP_Q && b == block0) {
#pragma unroll
            for (int kk = 0; kk < (KEEP_Q ? DK / 16 : 1); ++kk) mx_ldsm(q_addr + kk * 32, qa[kk]);
        }
        const uint32_t sk = mx_smem(skv + (b & 1) * (S::K_BYTES + S::V_BYTES)), sv = sk + S::K_BYTES;
        if (b * BK <= warp_last && b * BK + BK > warp_low) {
            float sc[BK / 8][4];
#pragma unroll
            for (int i = 0; i < BK / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.0f;
#pragma unroll
            for (int kk = 0; kk < DK / 16; ++kk) {
                uint32_t qf[4];
                if (!KEEP_Q) mx_ldsm(q_addr + kk * 32, qf);
                const uint32_t* q4 = KEEP_Q ? qa[KEEP_Q ? kk : 0] : qf;
#pragma unroll
                for (int n = 0; n < BK / 16; ++n) {
                    uint32_t bb[4];
                    mx_ldsm(sk + (n * 16 + (lane & 7) + (lane >> 4) * 8) * S::KP + (kk * 16 + ((lane >> 3) & 1) * 8) * 2, bb);
                    mx_mma(sc[2 * n], q4, bb[0], bb[1]);
                    mx_mma(sc[2 * n + 1], q4, bb[2], bb[3]);
                }
            }
            const bool mask = b * BK + BK - 1 > warp_first || b * BK < warp_low_last;
            auto hidden = [&](int i, int e) {
                const uint32_t key = b * BK + i * 8 + t4 * 2 + (e & 1);
                return key > (e < 2 ? lim0 : lim1) || key < (e < 2 ? low0 : low1);
            };
            if (SIGMOID) {
#pragma unroll
                for (int i = 0; i < BK / 8; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float w = ga_sigmoid(sc[i][e], P.score.pre, e < 2 ? bias0 : bias1);
                        sc[i][e] = mask && hidden(i, e) ? 0.0f : w;
                    }
            }
            float ms0 = 0.0f, ms1 = 0.0f;
            if (!SIGMOID) {
            float mx0 = m0, mx1 = m1;
#pragma unroll
            for (int i = 0; i < BK / 8; ++i) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    float v = ga_score(sc[i][e], P.score);
                    if (mask && hidden(i, e)) v = -INFINITY;
                    sc[i][e] = v;
                }
                mx0 = fmaxf(mx0, fmaxf(sc[i][0], sc[i][1]));
                mx1 = fmaxf(mx1, fmaxf(sc[i][2], sc[i][3]));
            }
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            ms0 = mx0 == -INFINITY ? 0.0f : mx0;
            ms1 = mx1 == -INFINITY ? 0.0f : mx1;
            const float c0 = mx_ex2(m0 - ms0), c1 = mx_ex2(m1 - ms1);
            m0 = mx0;
            m1 = mx1;
            l0 *= c0;
            l1 *= c1;
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
            }
#pragma unroll
            for (int kk = 0; kk < BK / 16; ++kk) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const float* v = sc[2 * kk + n];
                    const float pa = SIGMOID ? v[0] : mx_ex2(v[0] - ms0), pb = SIGMOID ? v[1] : mx_ex2(v[1] - ms0);
                    const float pc = SIGMOID ? v[2] : mx_ex2(v[2] - ms1), pd = SIGMOID ? v[3] : mx_ex2(v[3] - ms1);
                    if (!SIGMOID) { l0 += pa + pb; l1 += pc + pd; }
                    split_bf16x2(pa, pb, hi[2 * n], lo[2 * n]);
                    split_bf16x2(pc, pd, hi[2 * n + 1], lo[2 * n + 1]);
                }
#pragma unroll
                for (int n0 = 0; n0 < DV / 16; n0 += 4) {
                    uint32_t bb[4][4];
#pragma unroll
                    for (int n = 0; n < 4; ++n)
                        mx_ldsm_t(sv + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::VP + ((n0 + n) * 16 + (lane >> 4) * 8) * 2, bb[n]);
#pragma unroll
                    for (int n = 0; n < 4; ++n) {
                        mx_mma(o[2 * (n0 + n)], hi, bb[n][0], bb[n][1]);
                        mx_mma(o[2 * (n0 + n) + 1], hi, bb[n][2], bb[n][3]);
                    }
#pragma unroll
                    for (int n = 0; n < 4; ++n) {
                        mx_mma(o[2 * (n0 + n)], lo, bb[n][0], bb[n][1]);
                        mx_mma(o[2 * (n0 + n) + 1], lo, bb[n][2], bb[n][3]);
                    }
                }
            }
        }
        __syncthreads();
    }
    mx_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    bf16* out = reinterpret_cast<bf16*>(a.out);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const uint32_t r = half ? r1 : r0;
        if (r >= n_rows) continue;
        const uint32_t R = row0 + r, h = kvh * P.per + R % P.per;
        const size_t row = (size_t)s * P.place.chunk + R / P.per;
        const float f = SIGMOID ? ga_gate(a, row, h) : ga_gate(a, row, h) / (half ? l1 : l0);
        bf16* dst = out + row * a.out_ld + (size_t)h * a.vdim;
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
            const uint32_t c = i * 8 + t4 * 2;
            const float x = o[i][2 * half] * f, y = o[i][2 * half + 1] * f;
            if (P.vec) {
                if (c < a.vdim) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(x, y);
            } else {
                if (c < a.vdim) dst[c] = __float2bfloat16_rn(x);
                if (c + 1 < a.vdim) dst[c + 1] = __float2bfloat16_rn(y);
            }
        }
    }
    if (kvh == 0)
        for (uint32_t t = row0 / P.per; t <= (row0 + n_rows - 1) / P.per; ++t) ga_zero_pad(a, (size_t)s * P.place.chunk + t, threadIdx.x, 128);
}

// ---- launch --------------------------------------------------------------------------------
namespace {

template <typename K>
int allow_smem(K kernel, uint32_t bytes, bool* configured) {
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && configured[dev]) return TNSR_B200_OK;
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess) return check_launch("grouped_attention attribute");
    if (dev >= 0 && dev < 64) configured[dev] = true;
    return TNSR_B200_OK;
}

template <int DK, int DV, int STAGES, bool UPPER, bool SIGMOID>
int launch_split_kind(const GaParams& P, cudaStream_t stream) {
    static bool configured[64] = {};
    const uint32_t bytes = SplitShape<DK, DV, STAGES>::BYTES;
    int rc = allow_smem(grouped_split_kernel<DK, DV, STAGES, UPPER, SIGMOID>, bytes, configured);
    if (rc) return rc;
    launch_kernel(grouped_split_kernel<DK, DV, STAGES, UPPER, SIGMOID>, dim3(P.splits, P.a.kv_heads * P.row_tiles, P.place.sessions), dim3(GA_WARPS * 32), bytes,
                  stream, P);
    return TNSR_B200_OK;
}

template <int DK, int DV, int STAGES, bool UPPER>
int launch_split(const GaParams& P, cudaStream_t stream) {
    return P.a.score_kind == TNSR_B200_SCORE_SIGMOID ? launch_split_kind<DK, DV, STAGES, UPPER, true>(P, stream) : launch_split_kind<DK, DV, STAGES, UPPER, false>(P, stream);
}

template <int DK, int DV, int BK, bool SIGMOID>
int launch_tile_kind(const GaParams& P, cudaStream_t stream) {
    static bool configured[64] = {};
    const uint32_t bytes = TileShape<DK, DV, BK>::BYTES;
    int rc = allow_smem(grouped_tile_kernel<DK, DV, BK, SIGMOID>, bytes, configured);
    if (rc) return rc;
    launch_kernel(grouped_tile_kernel<DK, DV, BK, SIGMOID>, dim3(P.row_tiles, P.a.kv_heads, P.place.sessions), dim3(128), bytes, stream, P);
    return TNSR_B200_OK;
}

template <int DK, int DV, int BK>
int launch_tile(const GaParams& P, cudaStream_t stream) {
    return P.a.score_kind == TNSR_B200_SCORE_SIGMOID ? launch_tile_kind<DK, DV, BK, true>(P, stream) : launch_tile_kind<DK, DV, BK, false>(P, stream);
}

uint32_t padded_width(uint32_t dim, uint32_t vdim) {
    const uint32_t w = std::max(dim, vdim);
    return w <= 64 ? 64 : w <= 128 ? 128 : 256;
}

// Splits of the keys: as many CTAs as fit the GPU at once (four, two or one per SM at padded widths 64, 128, 256) if the
// (session, key/value head, row tile) triples do not give them already.
constexpr uint64_t GA_CTAS = 592;
uint32_t splits_for(uint64_t units, uint32_t padded) {
    const uint64_t slots = padded == 64 ? GA_CTAS : padded == 128 ? 296 : 148;
    return (uint32_t)std::min<uint64_t>(GA_MAX_SPLITS, std::max<uint64_t>(1, slots / units));
}
// More than one split means at most GA_CTAS / 2 units and GA_CTAS partial tiles.
constexpr uint64_t GA_COUNTER_BYTES = 2048;
static_assert(GA_COUNTER_BYTES >= GA_CTAS / 2 * 4, "one merge counter per unit");

// Rows (chunk * heads per group) up to which the split kernel runs: one tile per 16 of them re-reads the keys.
constexpr uint32_t GA_SPLIT_ROWS = 64;

}  // namespace

uint64_t grouped_attention_workspace_bytes(uint32_t dim, uint32_t vdim) {
    return GA_COUNTER_BYTES + GA_CTAS * 16 * (padded_width(dim, vdim) + 2) * 4;
}

int launch_grouped_attention(const GroupedAttention& a, const StepPlace& place, int dtype, cudaStream_t stream) {
    if (place.sessions == 0 || place.chunk == 0) return TNSR_B200_OK;
    if (a.kv_heads == 0 || a.heads % a.kv_heads || a.dim > 256 || a.vdim > 256) {
        set_thread_error("grouped attention: kv_heads must divide heads, widths are at most 256");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    if (dtype != TNSR_B200_BF16 || a.engine == 1 || place.sessions > 65535u || a.kv_heads > 16000u)
        return launch_grouped_attention_rows(a, place, dtype, stream);
    GaParams P;
    P.a = a;
    P.place = place;
    P.score = make_score(a.scale, a.softcap);
    if (a.score_kind == TNSR_B200_SCORE_SIGMOID) P.score.pre = -GA_LOG2E * a.scale;
    P.per = a.heads / a.kv_heads;
    const uint64_t rows = (uint64_t)place.chunk * P.per;
    if (rows > 0x7fffffffull) { set_thread_error("grouped attention: too many rows"); return TNSR_B200_ERR_UNSUPPORTED; }
    P.rows = (uint32_t)rows;
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    P.vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.out_ld % 2 == 0 && aligned(a.q) && aligned(a.k_cache) && aligned(a.v_cache) && aligned(a.out);
    P.splits = 1;
    P.done = nullptr;
    P.partial = nullptr;
    const uint32_t w = padded_width(a.dim, a.vdim);
    int rc;
    if (P.rows <= GA_SPLIT_ROWS || place.chunk == 1) {
        P.row_tiles = ceil_div(P.rows, 16u);
        const uint64_t units = (uint64_t)place.sessions * a.kv_heads * P.row_tiles;
        P.splits = splits_for(units, w);
        if (a.window) P.splits = std::min(P.splits, std::max(1u, ceil_div(a.window + place.chunk, 16 * GA_WARPS)));   // a tile per warp at least
        if (!a.workspace || a.workspace_bytes < grouped_attention_workspace_bytes(a.dim, a.vdim)) P.splits = 1;
        if (P.splits > 1) {
            P.done = reinterpret_cast<uint32_t*>(a.workspace);
            P.partial = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(a.workspace) + GA_COUNTER_BYTES);
        }
        const bool upper = P.rows > 8;
        if (w == 64) rc = upper ? launch_split<64, 64, 3, true>(P, stream) : launch_split<64, 64, 3, false>(P, stream);
        else if (w == 128) rc = upper ? launch_split<128, 128, 3, true>(P, stream) : launch_split<128, 128, 3, false>(P, stream);
        else rc = upper ? launch_split<256, 256, 2, true>(P, stream) : launch_split<256, 256, 2, false>(P, stream);
    } else if (a.engine == 0 && grouped_attention_tc_eligible(a, place)) {
        return launch_grouped_attention_tc(a, place, stream);
    } else {
        P.row_tiles = ceil_div(P.rows, 64u);
        if (w == 64) rc = launch_tile<64, 64, 64>(P, stream);
        else if (w == 128) rc = launch_tile<128, 128, 64>(P, stream);
        else rc = launch_tile<256, 256, 32>(P, stream);
    }
    if (rc) return rc;
    count_launch();
    return check_launch("grouped_attention");
}

}  // namespace tb
