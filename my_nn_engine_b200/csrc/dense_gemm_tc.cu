// Matrix products over unquantised 16-bit weights for many rows (prefill), dense or grouped by expert, on tcgen05 kind::f16.
//
// Persistent CTAs (one per SM).  A tile is 128 activation rows (the MMA's M, one tensor-memory lane each) times 256 weight rows (its
// N), or with gating 128 gate rows and the 128 up rows of the same outputs side by side, so that a thread of the epilogue finds
// gate and up of an output in its own lane.  Warp 0 streams both operands by TMA through a ring of four 48 KB stages (64 elements
// of the contraction each, 128-byte swizzle), warp 1 issues the MMAs into one of two 256-column accumulators, warps 2-5 drain the
// other one: tcgen05.ld, gating, rounding, 16-byte stores along the output row.
// Grouped products take their tiles from the list the router's ordering left (MoeRoute::tile_e / tile_row: 128 places that do not
// cross experts); a tile's rows past its expert's last one are computed and not stored.  Tiles run with the weight tile fastest, so
// the row tiles of one expert follow each other while its weights are in L2.
// All waits are bounded and report through the caller's status word.
#include "block_ops.cuh"
#include "common.cuh"
#include "i8_gemm.cuh"
#include "tcgen05.cuh"

#include <type_traits>

namespace mynn {

MYNN_DEFINE_WAIT_BUDGET_SETTER(dense_gemm_tc)

constexpr int kDgRows = kMoeTileRows;  // activation rows per tile (UMMA M)
static_assert(kDgRows == 128, "one tensor-memory lane per activation row");
constexpr int kDgCols = 256;           // accumulator columns per tile (UMMA N)
constexpr int kDgK = 64;               // elements per stage: 128 bytes
constexpr int kDgStages = 4;
constexpr int kDgThreads = 192;
constexpr uint32_t kDgABytes = kDgRows * kDgK * 2, kDgWBytes = kDgCols * kDgK * 2, kDgStageBytes = kDgABytes + kDgWBytes;

struct DgParams {
    void *out;
    int M, N, K;
    int n_tiles;                                  // weight tiles
    const int32_t *off, *tile_e, *tile_row, *m_tiles_dev;  // grouped: see MoeRoute; null: dense
    int row_fastest;                              // dense: walk the row tiles fastest
    int ldo, n_main, act_fn, out_block;           // see DenseGemm; out_block 0: none
    long long out_block_stride;
    float *out_f32;
    int groups, group_tiles;                      // dense: groups of rows and row tiles of each; 0: one group
    long long group_rows;                         // distance of the groups' first rows
    int *status;
};

template <typename T, typename O>
__device__ __forceinline__ void store_run(O *dst, const float (&v)[32], int n, bool vec) {  // n of 32 neighbouring outputs
    if (vec && n == 32) {
        if constexpr (sizeof(O) == 4) {
#pragma unroll
            for (int i = 0; i < 8; i++) *reinterpret_cast<float4 *>(dst + 4 * i) = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
        } else {
#pragma unroll
            for (int i = 0; i < 4; i++) {
                O o[8];
#pragma unroll
                for (int j = 0; j < 8; j++) o[j] = from_f32<O>(v[8 * i + j]);
                *reinterpret_cast<uint4 *>(dst + 8 * i) = *reinterpret_cast<const uint4 *>(o);
            }
        }
    } else {
#pragma unroll
        for (int i = 0; i < 32; i++)
            if (i < n) dst[i] = from_f32<O>(v[i]);
    }
}

template <typename T, typename O, bool GLU>
__global__ void __launch_bounds__(kDgThreads, 1)
dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, const DgParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t full_bar[kDgStages], empty_bar[kDgStages], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    constexpr int NT = GLU ? kDgCols / 2 : kDgCols;  // outputs per tile

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kblocks = (p.K + kDgK - 1) / kDgK;
    if (threadIdx.x == 0) {
        for (int s = 0; s < kDgStages; s++) {
            mbar_init(&full_bar[s], 1);
            mbar_init(&empty_bar[s], 1);
        }
        for (int b = 0; b < 2; b++) {
            mbar_init(&acc_full[b], 1);
            mbar_init(&acc_empty[b], 4);  // one arrival per epilogue warp
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(&tmem_slot, 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = tmem_slot;
    pdl_wait();  // activations and the tile list come from the preceding kernels
    const int m_tiles = p.m_tiles_dev ? *p.m_tiles_dev : p.group_tiles ? p.group_tiles * p.groups : (p.M + kDgRows - 1) / kDgRows;
    const int total = m_tiles * p.n_tiles;
    auto give_up = [&](int code) {
        atomicExch(&abort_flag, 1);
        atomicExch(p.status, code);
    };
    auto group_base = [&](int mt) { return p.group_tiles ? (int)((mt / p.group_tiles) * p.group_rows) : 0; };
    auto dense_row = [&](int mt) { return group_base(mt) + (p.group_tiles ? mt % p.group_tiles : mt) * kDgRows; };
    auto locate = [&](int tile, int &mt, int &nt) {
        if (p.row_fastest) nt = tile / m_tiles, mt = tile - nt * m_tiles;
        else mt = tile / p.n_tiles, nt = tile - mt * p.n_tiles;
    };

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            asm volatile("prefetch.tensormap [%0];" ::"l"(&map_a) : "memory");
            asm volatile("prefetch.tensormap [%0];" ::"l"(&map_w) : "memory");
            int kc = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
                int mt, nt;
                locate(tile, mt, nt);
                const int e = p.tile_e ? p.tile_e[mt] : 0, row = p.tile_row ? p.tile_row[mt] : dense_row(mt);
                const int wrow = e * (GLU ? 2 * p.N : p.N) + nt * NT;
                for (int kb = 0; kb < kblocks; kb++, kc++) {
                    const int s = kc % kDgStages, use = kc / kDgStages;
                    if (use > 0 && !mbar_wait_spin(&empty_bar[s], (use - 1) & 1, &abort_flag)) {
                        give_up(41);
                        ok = false;
                        break;
                    }
                    uint8_t *st = smem + s * kDgStageBytes;
                    mbar_expect_tx(&full_bar[s], kDgStageBytes);
                    tma_load_2d(st, &map_a, kb * 128, row, &full_bar[s]);  // byte maps: x counts bytes
                    if constexpr (GLU) {
                        tma_load_2d(st + kDgABytes, &map_w, kb * 128, wrow, &full_bar[s]);
                        tma_load_2d(st + kDgABytes + kDgWBytes / 2, &map_w, kb * 128, wrow + p.N, &full_bar[s]);
                    } else {
                        tma_load_2d(st + kDgABytes, &map_w, kb * 128, wrow, &full_bar[s]);
                    }
                }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            constexpr uint32_t ab = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;  // operand format: 0 = f16, 1 = bf16
            int kc = 0, it = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x, it++) {
                const int buf = it & 1, use = it >> 1;
                int mt, nt;
                locate(tile, mt, nt);
                // only as many columns as the tile has weight rows (gating needs both halves in place)
                const int cols = GLU ? kDgCols : min(kDgCols, ((p.N - nt * NT + 15) >> 4) << 4);
                const uint32_t idesc = (1u << 4) | (ab << 7) | (ab << 10) | ((uint32_t)(cols >> 3) << 17) | ((uint32_t)(kDgRows >> 4) << 24);
                if (use > 0 && !mbar_wait_spin(&acc_empty[buf], (use - 1) & 1, &abort_flag)) {  // the epilogue has drained it
                    give_up(42);
                    break;
                }
                tc_fence_after();
                const uint32_t d_tmem = tmem_base + (uint32_t)(buf * kDgCols);
                for (int kb = 0; kb < kblocks; kb++, kc++) {
                    const int s = kc % kDgStages;
                    if (!mbar_wait_spin(&full_bar[s], (kc / kDgStages) & 1, &abort_flag)) {
                        give_up(43);
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint32_t a_addr = smem_u32(smem + s * kDgStageBytes);
                    const uint64_t adesc = make_kmajor_sw128_desc(a_addr), bdesc = make_kmajor_sw128_desc(a_addr + kDgABytes);
#pragma unroll
                    for (int k = 0; k < kDgK / 16; k++)
                        umma_f16(d_tmem, adesc + (uint64_t)(k * 2), bdesc + (uint64_t)(k * 2), idesc, (kb | k) ? 1u : 0u);
                    umma_commit(&empty_bar[s]);
                }
                if (ok) umma_commit(&acc_full[buf]);
            }
        }
        __syncwarp();
    } else {
        // ---------------- epilogue warps 2..5: lane quadrant = warp & 3, one activation row per thread ----------------
        const int quad = warp & 3, row = quad * 32 + lane;
        constexpr int kPiece = sizeof(O) == 4 ? 4 : 8;  // elements of a 16-byte store
        const bool vec = p.ldo % kPiece == 0 && (uintptr_t)p.out % 16 == 0 && p.out_block % kPiece == 0 && p.out_block_stride % kPiece == 0;
        const bool runs = p.out_block % 32 == 0;        // 32 neighbouring columns from a multiple of 32 on lie in one block
        int it = 0;
        for (int tile = blockIdx.x; tile < total; tile += gridDim.x, it++) {
            const int buf = it & 1, use = it >> 1;
            int mt, nt;
            locate(tile, mt, nt);
            const int r0 = p.tile_row ? p.tile_row[mt] : dense_row(mt);
            const int end = p.tile_e ? p.off[p.tile_e[mt] + 1] : group_base(mt) + p.M;
            int ok = 1;
            if (lane == 0) {
                ok = mbar_wait_spin(&acc_full[buf], use & 1, &abort_flag) ? 1 : 0;
                if (!ok) give_up(44);
            }
            ok = __shfl_sync(0xffffffffu, ok, 0);
            __syncwarp();
            if (!ok) break;
            tc_fence_after();
            const uint32_t t_lane = tmem_base + ((uint32_t)(quad * 32) << 16) + (uint32_t)(buf * kDgCols);
            const int n0 = nt * NT;
            const bool mine = r0 + row < end;
            O *out = reinterpret_cast<O *>(p.out) + (size_t)(r0 + row) * p.ldo;
            float *out_f32 = p.out_f32 + (size_t)(r0 + row) * (p.N - p.n_main);  // not read without out_f32
#pragma unroll 1
            for (int c = 0; c < NT; c += 32) {
                if (n0 + c >= p.N) break;  // uniform
                float v[32];
                tmem_ld32(t_lane + c, reinterpret_cast<uint32_t *>(v));
                if constexpr (GLU) {
                    float u[32];
                    tmem_ld32(t_lane + NT + c, reinterpret_cast<uint32_t *>(u));
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; i++) v[i] = __fdividef(v[i], 1.0f + __expf(-v[i])) * u[i];
                } else {
                    tmem_ld_wait();
                }
                if (mine) {
                    const int n = n0 + c, run = min(32, p.N - n);
                    if (n + run <= p.n_main && runs) {
                        if (p.act_fn) {
#pragma unroll
                            for (int i = 0; i < 32; i++) v[i] = dense_act(v[i], p.act_fn);
                        }
                        store_run<T, O>(out + (p.out_block ? (size_t)(n / p.out_block) * p.out_block_stride + n % p.out_block : (size_t)n), v, run, vec);
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; i++) {
                            if (i >= run) continue;
                            const int j = n + i;
                            if (j >= p.n_main) out_f32[j - p.n_main] = v[i];
                            else out[p.out_block ? (size_t)(j / p.out_block) * p.out_block_stride + j % p.out_block : (size_t)j] = from_f32<O>(dense_act(v[i], p.act_fn));
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[buf]);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, 512);
}

// activation rows in expert order: one 16-byte piece per thread
__global__ void __launch_bounds__(256) gather_places_kernel(uint4 *out, const uint4 *act, const int32_t *tok_of, long long pieces, int per_row) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= pieces) return;
    const int r = (int)(i / per_row), c = (int)(i - (long long)r * per_row);
    out[i] = act[(size_t)tok_of[r] * per_row + c];
}

bool dense_gemm_tc_supported(int dtype, const DenseGemm &g) {
    if (dtype == MYNN_F32 || !g.status || !tensor_map_api_available() || g.K % 8 || g.batch > 1 || (g.lda && g.lda != g.K) || (((uintptr_t)g.act | (uintptr_t)g.w) % 16)) return false;
    const long long wrows = (long long)g.experts * g.N * (g.glu ? 2 : 1), arows = g.route ? (long long)g.M * g.top : g.M;
    if (wrows >= (1ll << 31) || arows >= (1ll << 31) || g.row_groups * g.group_rows >= (1ll << 31)) return false;
    if (!g.route) return g.M > 32;
    if (g.gather && (!g.gather_ws || (uintptr_t)g.gather_ws % 16)) return false;
    return arows >= 16ll * g.experts && g.M > 32;  // enough rows per expert for a 128-row tile to beat passes over its weights
}

template <typename T, typename O, bool GLU>
static int launch_dg(cudaStream_t st, const CUtensorMap &ma, const CUtensorMap &mw, const DgParams &p, long long tiles_bound) {
    constexpr size_t smem = (size_t)kDgStages * kDgStageBytes + 1024;
    auto kern = dense_gemm_tc_kernel<T, O, GLU>;
    static bool attr_set = false;
    if (!attr_set) {
        MYNN_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set = true;
    }
    int dev = 0, sms = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    kern<<<(unsigned)(tiles_bound < sms ? tiles_bound : sms), kDgThreads, smem, st>>>(ma, mw, p);
    MYNN_LAUNCH_OK("dense_gemm_tc_kernel");
    return MYNN_OK;
}

int launch_dense_gemm_tc(cudaStream_t st, int dtype, const DenseGemm &g) {
    const long long arows = g.route ? (long long)g.M * g.top : g.M, wrows = (long long)g.experts * g.N * (g.glu ? 2 : 1);
    const void *act = g.act;
    if (g.route && g.gather) {
        const int per_row = g.K / 8;
        const long long pieces = arows * per_row;
        gather_places_kernel<<<(unsigned)((pieces + 255) / 256), 256, 0, st>>>((uint4 *)g.gather_ws, (const uint4 *)g.act, g.route->tok_of, pieces, per_row);
        MYNN_LAUNCH_OK("gather_places_kernel");
        act = g.gather_ws;
    }
    CUtensorMap ma, mw;
    const uint64_t row_bytes = (uint64_t)g.K * 2;
    const uint64_t map_rows = g.row_groups > 1 ? (uint64_t)((g.row_groups - 1) * g.group_rows + g.M) : (uint64_t)arows;
    if (int rc = make_map(&ma, act, map_rows, row_bytes, row_bytes, kDgRows)) return rc;
    if (int rc = make_map(&mw, g.w, (uint64_t)wrows, row_bytes, row_bytes, g.glu ? kDgCols / 2 : kDgCols)) return rc;
    DgParams p = {};
    p.out = g.out;
    p.M = g.M, p.N = g.N, p.K = g.K;
    const int nt = g.glu ? kDgCols / 2 : kDgCols;
    p.n_tiles = (g.N + nt - 1) / nt;
    p.status = g.status;
    p.n_main = g.out_f32 ? g.n_main : g.N;
    p.ldo = g.ldo ? g.ldo : p.n_main;
    p.act_fn = g.act_fn;
    p.out_block = g.out_block;
    p.out_block_stride = g.out_block_stride;
    p.out_f32 = g.out_f32;
    long long m_bound = (g.M + kDgRows - 1) / kDgRows;
    if (g.row_groups > 1) {
        p.groups = g.row_groups;
        p.group_tiles = (int)m_bound;
        p.group_rows = g.group_rows;
        m_bound *= g.row_groups;
    }
    if (g.route) {
        p.off = g.route->off;
        p.tile_e = g.route->tile_e;
        p.tile_row = g.route->tile_row;
        p.m_tiles_dev = g.route->n_tiles;
        m_bound = arows / kDgRows + (g.experts < arows ? g.experts : arows);
    } else {
        p.row_fastest = 1;
    }
    const long long bound = m_bound * p.n_tiles;
    const bool f32 = g.out_dtype == MYNN_F32;
    if (dtype == MYNN_BF16) {
        using T = __nv_bfloat16;
        if (g.glu) return f32 ? launch_dg<T, float, true>(st, ma, mw, p, bound) : launch_dg<T, T, true>(st, ma, mw, p, bound);
        return f32 ? launch_dg<T, float, false>(st, ma, mw, p, bound) : launch_dg<T, T, false>(st, ma, mw, p, bound);
    }
    using T = __half;
    if (g.glu) return f32 ? launch_dg<T, float, true>(st, ma, mw, p, bound) : launch_dg<T, T, true>(st, ma, mw, p, bound);
    return f32 ? launch_dg<T, float, false>(st, ma, mw, p, bound) : launch_dg<T, T, false>(st, ma, mw, p, bound);
}

}  // namespace mynn
