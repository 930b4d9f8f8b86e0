// Products of row groups with a matrix each (experts, block-diagonal gates): rows offsets[g] .. offsets[g + 1] of a [rows, k]
// times w[g] [n, k] transposed.  The group sizes live on the device, so the tile list is made there.
//
//  * gemm_grouped_tc_kernel     tcgen05, bf16.  Operands swapped as in gemm_skinny.cu: 128 WEIGHT rows are the M side (one
//                               TMEM lane per output column) and NT token rows the N side, with NT from 16 (decode: a
//                               handful of tokens per expert) to 256 (prefill), so that a group's few rows do not pay for
//                               a 128-row tile.  Persistent: every CTA walks the tiles c, c + grid, ... of a list made
//                               of the group sizes; TMA ring, one MMA thread, double-buffered accumulators, four or eight
//                               epilogue warps.  A token tile may read rows of the next group (they are in bounds of the
//                               tensor map or read as zero); their columns of the accumulator are not stored.
//  * gemm_grouped_simple_kernel CUDA cores: f32, and shapes that TMA cannot address (k not a multiple of 8).
//
// Every wait is bounded (tc_common.cuh).
#include <algorithm>

#include "feed_forward.cuh"
#include "tc_common.cuh"

namespace tb {

constexpr int GG_ROWS = 128;      // weight rows per tile
constexpr int GG_BK = 64;
constexpr uint32_t GG_W_BYTES = GG_ROWS * GG_BK * 2;
constexpr uint32_t GG_MAX_GROUPS = 1024;

template <int NT>
struct GgShape {
    static constexpr int EPI = NT >= 128 ? 8 : 4;     // epilogue warps
    static constexpr int THREADS = 64 + 32 * EPI;
    static constexpr uint32_t A_BYTES = NT * GG_BK * 2;
    static constexpr uint32_t STAGE_BYTES = GG_W_BYTES + A_BYTES;
    static constexpr int STAGES = NT >= 256 ? 4 : NT >= 128 ? 6 : NT >= 64 ? 8 : 9;
    static constexpr uint32_t ACC = NT < 32 ? 32 : NT;                  // accumulator pitch in TMEM columns
    static constexpr uint32_t TMEM_COLS = 2 * ACC;
    static constexpr uint32_t TABLE = (2 * GG_MAX_GROUPS + 2) * 4;      // row offsets and first tiles of the groups
    static constexpr uint32_t SMEM_BYTES = STAGES * STAGE_BYTES + 1024 + 256 + TABLE;
    static constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NT >> 3) << 17) | ((uint32_t)(GG_ROWS >> 4) << 24);
};

struct GgParams {
    void* out;
    const uint32_t* offsets;
    uint32_t groups, rows, n, k;
    int activation, out_dtype;
    int* d_status;
    uint64_t wait_limit_ns;
};

__device__ __forceinline__ float gg_activation(float x, int act) {
    if (act == ACT_RELU_SQUARED) { const float y = fmaxf(x, 0.0f); return y * y; }
    return apply_activation(x, act);
}

// Walks the tile list: tiles of a group are consecutive, weight tiles fastest.
struct GgWalk {
    uint32_t g = 0, row0 = 0, end = 0, n0 = 0;      // group, first token row, end of the group's rows, first weight row
    __device__ __forceinline__ void seek(uint32_t tile, const uint32_t* offs, const uint32_t* first, uint32_t tiles_n, uint32_t nt) {
        while (tile >= first[g + 1]) ++g;
        const uint32_t local = tile - first[g];
        row0 = offs[g] + local / tiles_n * nt;
        end = offs[g + 1];
        n0 = local % tiles_n * GG_ROWS;
    }
};

// Row offsets of the groups and the first tile of each, by the whole block.  A group list that does not fit the rows (it
// never comes from this library's own kernels) is cut to them, so that no index leaves the buffers.
__device__ __forceinline__ void gg_tables(const GgParams& P, uint32_t* offs, uint32_t* first, uint32_t tiles_n, uint32_t nt) {
    for (uint32_t g = threadIdx.x; g <= P.groups; g += blockDim.x)
        offs[g] = min(P.rows, P.offsets ? P.offsets[g] : (uint32_t)((uint64_t)P.rows / P.groups * g));
    __syncthreads();
    if (threadIdx.x < 32) {
        uint32_t base = 0;
        for (uint32_t g0 = 0; g0 < P.groups; g0 += 32) {
            const uint32_t g = g0 + threadIdx.x;
            const uint32_t count = g < P.groups && offs[g + 1] > offs[g] ? offs[g + 1] - offs[g] : 0u;
            uint32_t x = (count + nt - 1) / nt * tiles_n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const uint32_t y = __shfl_up_sync(0xffffffffu, x, o);
                if (threadIdx.x >= (uint32_t)o) x += y;
            }
            if (g < P.groups) first[g + 1] = base + x;
            base += __shfl_sync(0xffffffffu, x, 31);
        }
        if (threadIdx.x == 0) first[0] = 0;
    }
    __syncthreads();
}

template <int NT>
__global__ void __launch_bounds__(64 + 32 * GgShape<NT>::EPI, 1)
gemm_grouped_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_a, GgParams prm) {
    using S = GgShape<NT>;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw_addr = smem_u32(smem_raw);
    uint8_t* smem = smem_raw + ((1024u - (raw_addr & 1023u)) & 1023u);
    uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + S::STAGES * S::STAGE_BYTES);
    uint64_t* empty_bar = full_bar + S::STAGES;
    uint64_t* acc_full = empty_bar + S::STAGES;   // [2]
    uint64_t* acc_empty = acc_full + 2;           // [2]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    uint32_t* offs = reinterpret_cast<uint32_t*>(smem + S::STAGES * S::STAGE_BYTES + 256);
    uint32_t* first = offs + GG_MAX_GROUPS + 1;

    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t tiles_n = (prm.n + GG_ROWS - 1) / GG_ROWS, num_kb = (prm.k + GG_BK - 1) / GG_BK;
    if (threadIdx.x == 0) {
        for (int s = 0; s < S::STAGES; ++s) { mbar_init(full_bar + s, 1); mbar_init(empty_bar + s, 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(acc_full + s, 1); mbar_init(acc_empty + s, S::EPI); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    pdl_wait();
    pdl_trigger();
    gg_tables(prm, offs, first, tiles_n, NT);
    if (warp == 1) {
        tmem_alloc(tmem_slot, S::TMEM_COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t num_tiles = first[prm.groups];

    if (warp == 0) {
        if (lane == 0) {
            uint32_t stage = 0, phase = 0;
            bool ok = true;
            GgWalk at;
            for (uint32_t tile = blockIdx.x; ok && tile < num_tiles; tile += gridDim.x) {
                at.seek(tile, offs, first, tiles_n, NT);
                for (uint32_t kb = 0; kb < num_kb; ++kb) {
                    if (!mbar_wait(empty_bar + stage, phase ^ 1, abort_flag, prm.wait_limit_ns)) { ok = false; break; }
                    uint8_t* sw = smem + stage * S::STAGE_BYTES;
                    mbar_expect_tx(full_bar + stage, S::STAGE_BYTES);
                    tma_load_2d(sw, &map_w, (int32_t)(kb * GG_BK), (int32_t)(at.g * prm.n + at.n0), full_bar + stage);
                    tma_load_2d(sw + GG_W_BYTES, &map_a, (int32_t)(kb * GG_BK), (int32_t)at.row0, full_bar + stage);
                    if (++stage == S::STAGES) { stage = 0; phase ^= 1; }
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t stage = 0, phase = 0, it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; ok && tile < num_tiles; tile += gridDim.x, ++it) {
                const uint32_t ab = it & 1, aphase = (it >> 1) & 1;
                if (!mbar_wait(acc_empty + ab, aphase ^ 1, abort_flag, prm.wait_limit_ns)) { ok = false; break; }
                tc_fence_after();
                for (uint32_t kb = 0; kb < num_kb; ++kb) {
                    if (!mbar_wait(full_bar + stage, phase, abort_flag, prm.wait_limit_ns)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t sw = smem_u32(smem + stage * S::STAGE_BYTES);
                    const uint64_t wdesc = make_kmajor_sw128_desc(sw), adesc = make_kmajor_sw128_desc(sw + GG_W_BYTES);
#pragma unroll
                    for (uint32_t kk = 0; kk < GG_BK / 16; ++kk)
                        umma_bf16(tmem_base + ab * S::ACC, wdesc + kk * 2, adesc + kk * 2, S::IDESC, (kb | kk) != 0);
                    umma_commit(empty_bar + stage);
                    if (++stage == S::STAGES) { stage = 0; phase ^= 1; }
                }
                if (ok) umma_commit(acc_full + ab);
            }
        }
    } else {
        // ---------------- epilogue: lane = output column, registers = token rows ----------------
        const uint32_t quarter = warp & 3, half = (warp - 2) >> 2;
        constexpr uint32_t STRIDE = 32 * (S::EPI / 4);
        uint32_t it = 0;
        GgWalk at;
        for (uint32_t tile = blockIdx.x; tile < num_tiles; tile += gridDim.x, ++it) {
            const uint32_t ab = it & 1, aphase = (it >> 1) & 1;
            at.seek(tile, offs, first, tiles_n, NT);
            const uint32_t col = at.n0 + quarter * 32 + lane, live = min((uint32_t)NT, at.end - at.row0);
            if (!mbar_wait(acc_full + ab, aphase, abort_flag, prm.wait_limit_ns)) break;
            tc_fence_after();
#pragma unroll 1
            for (uint32_t j0 = half * 32; j0 < S::ACC; j0 += STRIDE) {
                if (j0 >= live) break;
                float acc[32];
                tmem_ld32(tmem_base + ((quarter * 32u) << 16) + ab * S::ACC + j0, acc);
                tmem_ld_wait();
                const uint32_t n_rows = min(32u, live - j0);
                const size_t base = (size_t)(at.row0 + j0) * prm.n;
#pragma unroll
                for (int j = 0; j < 32; ++j) acc[j] = gg_activation(acc[j], prm.activation);
                if (prm.out_dtype == TNSR_B200_F32) {
                    float* out = reinterpret_cast<float*>(prm.out) + base + col;
                    if (col < prm.n) {
#pragma unroll
                        for (int j = 0; j < 32; ++j)
                            if ((uint32_t)j < n_rows) out[(size_t)j * prm.n] = acc[j];
                    }
                } else if (prm.n % 2 == 0) {
                    // neighbouring lanes trade columns: the even one writes both columns of even rows, the odd one of odd rows
                    const bool odd = lane & 1;
                    bf16* out = reinterpret_cast<bf16*>(prm.out) + base + (col & ~1u);
                    const bool mine = (col & ~1u) < prm.n;
#pragma unroll
                    for (int j = 0; j < 32; j += 2) {
                        const float got = __shfl_xor_sync(0xffffffffu, odd ? acc[j] : acc[j + 1], 1);
                        const uint32_t row = j + (odd ? 1 : 0);
                        const uint32_t v = odd ? pack_bf16x2(got, acc[j + 1]) : pack_bf16x2(acc[j], got);
                        if (mine && row < n_rows) *reinterpret_cast<uint32_t*>(out + (size_t)row * prm.n) = v;
                    }
                } else {
                    bf16* out = reinterpret_cast<bf16*>(prm.out) + base + col;
                    if (col < prm.n) {
#pragma unroll
                        for (int j = 0; j < 32; ++j)
                            if ((uint32_t)j < n_rows) out[(size_t)j * prm.n] = __float2bfloat16_rn(acc[j]);
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(acc_empty + ab);
        }
    }

    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        // give copies that are still in flight time to land before the CTA's shared memory is released
        const uint64_t start = global_timer_ns();
        while (global_timer_ns() - start < 200000ull) __nanosleep(1000);
        if (threadIdx.x == 0 && prm.d_status) atomicCAS(prm.d_status, DEV_OK, DEV_TIMEOUT);
        __syncthreads();
    }
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, S::TMEM_COLS);
    }
}

// ---- CUDA cores: 32 x 32 tile, a thread owns 2 x 2 outputs -------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
gemm_grouped_simple_kernel(const T* __restrict__ a, const T* __restrict__ w, GgParams P) {
    constexpr uint32_t TS = 32, KS = 32;
    __shared__ float as[KS][TS + 1], ws[KS][TS + 1];
    __shared__ uint32_t offs[GG_MAX_GROUPS + 1], first[GG_MAX_GROUPS + 1];
    pdl_wait();
    pdl_trigger();
    const uint32_t tiles_n = (P.n + TS - 1) / TS, tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    gg_tables(P, offs, first, tiles_n, TS);
    const uint32_t num_tiles = first[P.groups];
    uint32_t g = 0;
    for (uint32_t tile = blockIdx.x; tile < num_tiles; tile += gridDim.x) {
        while (tile >= first[g + 1]) ++g;
        const uint32_t local = tile - first[g], row0 = offs[g] + local / tiles_n * TS, end = offs[g + 1], n0 = local % tiles_n * TS;
        const T* wg = w + (size_t)g * P.n * P.k;
        float acc[2][2] = {};
        for (uint32_t k0 = 0; k0 < P.k; k0 += KS) {
            for (uint32_t i = threadIdx.x; i < TS * KS; i += 256) {
                const uint32_t r = i / KS, kk = i % KS, gk = k0 + kk;
                as[kk][r] = gk < P.k && row0 + r < end ? to_f32(a[(size_t)(row0 + r) * P.k + gk]) : 0.0f;
                ws[kk][r] = gk < P.k && n0 + r < P.n ? to_f32(wg[(size_t)(n0 + r) * P.k + gk]) : 0.0f;
            }
            __syncthreads();
#pragma unroll 8
            for (uint32_t kk = 0; kk < KS; ++kk)
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int j = 0; j < 2; ++j) acc[i][j] = fmaf(as[kk][ty + 16 * i], ws[kk][tx + 16 * j], acc[i][j]);
            __syncthreads();
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const uint32_t row = row0 + ty + 16 * i, col = n0 + tx + 16 * j;
                if (row >= end || col >= P.n) continue;
                const float v = gg_activation(acc[i][j], P.activation);
                if (P.out_dtype == TNSR_B200_BF16) reinterpret_cast<bf16*>(P.out)[(size_t)row * P.n + col] = __float2bfloat16_rn(v);
                else reinterpret_cast<float*>(P.out)[(size_t)row * P.n + col] = v;
            }
    }
}

namespace {

int gg_sms() {
    static int n = 0;
    if (!n) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
        if (n <= 0) n = 148;
    }
    return n;
}

bool gg_map(CUtensorMap* map, const void* base, uint64_t rows, uint64_t k, uint32_t box_rows) {
    EncodeTiledFn fn = encode_fn();
    if (!fn) return false;
    cuuint64_t dims[2] = {k, rows};
    cuuint64_t strides[1] = {k * 2};
    cuuint32_t box[2] = {(cuuint32_t)GG_BK, box_rows};
    cuuint32_t estr[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int NT>
int launch_tc(const GroupedGemm& g, const GgParams& prm, cudaStream_t stream) {
    using S = GgShape<NT>;
    CUtensorMap mw, ma;
    if (!gg_map(&mw, g.w, (uint64_t)g.groups * g.n, g.k, GG_ROWS) || !gg_map(&ma, g.a, g.rows, g.k, NT)) {
        set_thread_error("grouped gemm: tensor map encoding failed");
        return TNSR_B200_ERR_CUDA;
    }
    static bool configured[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64 || !configured[dev]) {
        if (cudaFuncSetAttribute(gemm_grouped_tc_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)S::SMEM_BYTES) != cudaSuccess)
            return check_launch("gemm_grouped attribute");
        if (dev >= 0 && dev < 64) configured[dev] = true;
    }
    // at most this many tiles: every group may end in a ragged one
    const uint64_t tiles = (uint64_t)ceil_div(g.n, (uint32_t)GG_ROWS) * (g.rows / NT + std::min(g.groups, g.rows));
    const uint32_t grid = (uint32_t)std::min<uint64_t>(std::max<uint64_t>(tiles, 1), gg_sms());
    launch_kernel(gemm_grouped_tc_kernel<NT>, dim3(grid), dim3(S::THREADS), (size_t)S::SMEM_BYTES, stream, mw, ma, prm);
    count_launch();
    return check_launch("gemm_grouped");
}

}  // namespace

int launch_gemm_grouped(const GroupedGemm& g, int dtype, cudaStream_t stream) {
    if (g.groups == 0 || g.groups > GG_MAX_GROUPS || g.n == 0 || g.k == 0 || (!g.offsets && g.rows % g.groups)) {
        set_thread_error("grouped gemm: 1..1024 groups, and without offsets groups of equal size");
        return TNSR_B200_ERR_INVALID_ARGUMENT;
    }
    if (g.rows == 0) return TNSR_B200_OK;
    if (g.rows > 0x7fffffffu || (uint64_t)g.groups * g.n > 0x7fffffffull) {
        set_thread_error("grouped gemm: too many rows");
        return TNSR_B200_ERR_UNSUPPORTED;
    }
    GgParams prm;
    prm.out = g.out; prm.offsets = g.offsets; prm.groups = g.groups; prm.rows = g.rows; prm.n = g.n; prm.k = g.k;
    prm.activation = g.activation; prm.out_dtype = g.out_dtype; prm.d_status = g.d_status;
    prm.wait_limit_ns = g_wait_limit_ns.load(std::memory_order_relaxed);
    auto aligned = [](const void* p, uint32_t to) { return reinterpret_cast<uintptr_t>(p) % to == 0; };
    const bool tc = dtype == TNSR_B200_BF16 && g.engine == 0 && g_gemm_engine != 1 && g.k % 8 == 0 && aligned(g.a, 16) && aligned(g.w, 16) &&
                    aligned(g.out, 4) && encode_fn() != nullptr;
    if (tc) {
        // token rows per tile: a group's mean, less while there are fewer tiles than SMs
        const uint32_t per = ceil_div(g.rows, g.groups);
        uint32_t nt = per <= 16 ? 16 : per <= 32 ? 32 : per <= 64 ? 64 : per <= 128 ? 128 : 256;
        while (nt > 32 && (uint64_t)ceil_div(g.n, (uint32_t)GG_ROWS) * g.groups * ceil_div(per, nt) < (uint64_t)gg_sms()) nt >>= 1;
        switch (nt) {
            case 16: return launch_tc<16>(g, prm, stream);
            case 32: return launch_tc<32>(g, prm, stream);
            case 64: return launch_tc<64>(g, prm, stream);
            case 128: return launch_tc<128>(g, prm, stream);
            default: return launch_tc<256>(g, prm, stream);
        }
    }
    const uint64_t tiles = (uint64_t)ceil_div(g.n, 32u) * (g.rows / 32 + std::min(g.groups, g.rows));
    const dim3 grid((uint32_t)std::min<uint64_t>(std::max<uint64_t>(tiles, 1), 148ull * 8));
    if (dtype == TNSR_B200_BF16)
        launch_kernel(gemm_grouped_simple_kernel<bf16>, grid, dim3(256), 0, stream, (const bf16*)g.a, (const bf16*)g.w, prm);
    else
        launch_kernel(gemm_grouped_simple_kernel<float>, grid, dim3(256), 0, stream, (const float*)g.a, (const float*)g.w, prm);
    count_launch();
    return check_launch("gemm_grouped_simple");
}

}  // namespace tb
