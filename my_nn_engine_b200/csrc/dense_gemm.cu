// Matrix products over unquantised weights, dense or grouped by expert: out[m, n] = sum_k act[m, k] w[n, k], f32 accumulation.
//
// Three kernels behind launch_dense_gemm:
//   dense_stream_kernel   16-bit, up to a few dozen rows (decode): the weights are read once, straight from global memory into
//                         mma.m16n8k16 fragments.  The contraction index is permuted so that the 16 bytes a lane loads are two
//                         k16 fragments of its weight row (the activations use the same permutation), so nothing passes
//                         through shared memory before the reduction.  A CTA owns 16 or 32 weight rows, its eight warps deal out
//                         the contraction, and the partial sums meet in shared memory once.
//   dense_gemm_tc.cu      16-bit, many rows (prefill): tcgen05, TMA, accumulators in tensor memory.
//   dense_tile_kernel     any dtype and size: 64 x 64 tiles on the FP32 units (true 32-bit products for f32 models).
// With `glu` the gate and up rows of an output are accumulated side by side and silu(gate) * up is formed before the store.
// Grouped products walk the experts that have rows (MoeRoute::active), so a decode step touches no weight of an idle expert.
#include "attention_internal.cuh"
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

struct GemmView {  // device-side view of DenseGemm
    void *out;
    const void *act, *w;
    int M, N, K;
    const int32_t *off, *active, *n_active, *tok_of;  // null: dense
    int gather;
    int lda, ldo, n_main, act_fn, out_block, batch;
    long long act_stride, out_stride, out_block_stride;
    float *out_f32;
};

// output (row, n) of product z
template <typename O>
__device__ __forceinline__ void put_out(const GemmView &g, int z, size_t row, int n, float v) {
    if (n >= g.n_main) {
        g.out_f32[row * (g.N - g.n_main) + (n - g.n_main)] = v;
        return;
    }
    const size_t col = g.out_block ? (size_t)(n / g.out_block) * g.out_block_stride + n % g.out_block : n;
    reinterpret_cast<O *>(g.out)[z * g.out_stride + row * g.ldo + col] = from_f32<O>(dense_act(v, g.act_fn));
}

// rows [r0, r0 + cnt) of the product and the weight block of group z; false: nothing to do
__device__ __forceinline__ bool group_rows(const GemmView &g, int z, int &e, int &r0, int &cnt) {
    if (!g.off) {
        e = 0, r0 = 0, cnt = g.M;
        return true;
    }
    if (z >= *g.n_active) return false;
    e = g.active[z];
    r0 = g.off[e];
    cnt = g.off[e + 1] - r0;
    return true;
}

// ---- any dtype, any size ---------------------------------------------------------------------------------------------
// grid (ceil(N / 64), ceil(M / 64), groups), 256 threads, 4 x 4 outputs per thread
template <typename T, typename O, bool GLU>
__global__ void __launch_bounds__(256) dense_tile_kernel(const GemmView g) {
    constexpr int BK = 16;
    __shared__ float sa[BK][68], sw[BK][68], su[GLU ? BK : 1][68];
    pdl_trigger();
    pdl_wait();
    int e, r0, cnt;
    if (!group_rows(g, blockIdx.z, e, r0, cnt)) return;
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    if (m0 >= cnt) return;
    const int z = g.batch > 1 ? blockIdx.z : 0;
    const T *act = reinterpret_cast<const T *>(g.act) + z * g.act_stride, *w = reinterpret_cast<const T *>(g.w) + (size_t)(e + z) * (GLU ? 2 : 1) * g.N * g.K;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {}, accu[GLU ? 4 : 1][4] = {};
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;  // loader: row 0..63, four k
    const int am = m0 + lr;
    const T *arow = nullptr;
    if (am < cnt) arow = act + (size_t)(g.gather ? g.tok_of[r0 + am] : r0 + am) * g.lda;
    const T *wrow = n0 + lr < g.N ? w + (size_t)(n0 + lr) * g.K : nullptr;
    const T *urow = GLU && wrow ? wrow + (size_t)g.N * g.K : nullptr;
    for (int k0 = 0; k0 < g.K; k0 += BK) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int k = k0 + lk + i;
            const bool in = k < g.K;
            sa[lk + i][lr] = in && arow ? to_f32<T>(arow[k]) : 0.f;
            sw[lk + i][lr] = in && wrow ? to_f32<T>(wrow[k]) : 0.f;
            if constexpr (GLU) su[lk + i][lr] = in && urow ? to_f32<T>(urow[k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; k++) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; i++) a[i] = sa[k][ty * 4 + i], b[i] = sw[k][tx * 4 + i];
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
            if constexpr (GLU) {
#pragma unroll
                for (int j = 0; j < 4; j++) b[j] = su[k][tx * 4 + j];
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) accu[i][j] = fmaf(a[i], b[j], accu[i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int m = m0 + ty * 4 + i;
        if (m >= cnt) break;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tx * 4 + j;
            if (n >= g.N) break;
            float v = acc[i][j];
            if constexpr (GLU) v = silu_f(v) * accu[i][j];
            put_out<O>(g, z, (size_t)(r0 + m), n, v);
        }
    }
}

// ---- 16-bit weights, few rows ----------------------------------------------------------------------------------------
// grid (ceil(N / (16 RT)), groups), 256 threads.  RT: 16-row weight tiles per warp (with GLU: one gate and one up tile, RT == 1).
// MT: groups of 8 activation rows taken at a time; a group with more rows than 8 MT passes over its weights again (from L2).
constexpr int kStreamWarps = 8;
constexpr unsigned kPrefetchCtas = 3 * 148;
template <typename T, typename O, int MT, int RT, bool GLU>
__global__ void __launch_bounds__(kStreamWarps * 32, MT * RT * (GLU ? 2 : 1) <= 4 ? 2 : 1) dense_stream_kernel(const GemmView g) {
    constexpr int WT = GLU ? 2 : RT;  // weight tiles of a warp
    constexpr int U = WT == 1 ? 4 : 2;  // 32-element steps in flight
    __shared__ float red[kStreamWarps][WT * 16][MT * 8 + 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t = lane & 3;
    pdl_trigger();
    const int n0 = blockIdx.x * 16 * (GLU ? 1 : RT), z = g.batch > 1 ? blockIdx.y : 0;
    if (!g.off && gridDim.x <= kPrefetchCtas) {
        // launched as a programmatic dependent: the weights of this CTA travel to L2 while the kernel in front of it still runs
        // (a CTA of a later wave starts long after that, for it the prefetch would only be one more request)
        const size_t line = 128 / sizeof(T), total = (size_t)min(16 * (GLU ? 1 : RT), g.N - n0) * g.K;
        const T *w0 = reinterpret_cast<const T *>(g.w) + ((size_t)z * g.N + n0) * g.K;
        for (size_t i = threadIdx.x * line; i < total; i += kStreamWarps * 32 * line) {
            asm volatile("prefetch.global.L2 [%0];" ::"l"(w0 + i));
            if constexpr (GLU) asm volatile("prefetch.global.L2 [%0];" ::"l"(w0 + (size_t)g.N * g.K + i));
        }
    }
    pdl_wait();
    int e, r0, cnt;
    if (!group_rows(g, blockIdx.y, e, r0, cnt)) return;
    const T *act = reinterpret_cast<const T *>(g.act) + z * g.act_stride, *w = reinterpret_cast<const T *>(g.w) + (size_t)(e + z) * (GLU ? 2 : 1) * g.N * g.K;
    const T *wp[WT][2];  // this lane's two rows of every tile; rows past N repeat the last one and are not stored
#pragma unroll
    for (int i = 0; i < WT; i++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int n = min(n0 + (GLU ? 0 : 16 * i) + gq + 8 * h, g.N - 1);
            wp[i][h] = w + ((size_t)(GLU && i ? g.N : 0) + n) * g.K + 8 * t;
        }
    const int steps = (g.K + 31) >> 5;                                   // 32 elements of the contraction each
    const int per = (steps + kStreamWarps - 1) / kStreamWarps, s0 = warp * per, s1 = min(s0 + per, steps);
    for (int m0 = 0; m0 < cnt; m0 += 8 * MT) {
        const T *ap[MT];
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int m = min(m0 + 8 * i + gq, cnt - 1);
            ap[i] = act + (size_t)(g.gather ? g.tok_of[r0 + m] : r0 + m) * g.lda + 8 * t;
        }
        float acc[WT][MT][4];
#pragma unroll
        for (int i = 0; i < WT; i++)
#pragma unroll
            for (int j = 0; j < MT; j++) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
        for (int s = s0; s < s1; s += U) {
            uint4 wr[U][WT][2], ar[U][MT];
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int k = (s + u) << 5;
                const bool in = s + u < s1 && k + 8 * t < g.K;  // K is a multiple of 8: a lane's 8 elements are all in or all out
#pragma unroll
                for (int i = 0; i < WT; i++)
#pragma unroll
                    for (int h = 0; h < 2; h++) wr[u][i][h] = in ? ldg_16(wp[i][h] + k) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
                for (int i = 0; i < MT; i++) ar[u][i] = in ? *reinterpret_cast<const uint4 *>(ap[i] + k) : make_uint4(0u, 0u, 0u, 0u);
            }
#pragma unroll
            for (int u = 0; u < U; u++)
#pragma unroll
                for (int i = 0; i < WT; i++)
#pragma unroll
                    for (int j = 0; j < MT; j++) {
                        mma_kv<T>(acc[i][j], wr[u][i][0].x, wr[u][i][1].x, wr[u][i][0].y, wr[u][i][1].y, ar[u][j].x, ar[u][j].y);
                        mma_kv<T>(acc[i][j], wr[u][i][0].z, wr[u][i][1].z, wr[u][i][0].w, wr[u][i][1].w, ar[u][j].z, ar[u][j].w);
                    }
        }
        // accumulator registers: (row gq, cols 2t, 2t+1), (row gq + 8, same cols)
#pragma unroll
        for (int i = 0; i < WT; i++)
#pragma unroll
            for (int j = 0; j < MT; j++) {
                red[warp][16 * i + gq][8 * j + 2 * t] = acc[i][j][0];
                red[warp][16 * i + gq][8 * j + 2 * t + 1] = acc[i][j][1];
                red[warp][16 * i + gq + 8][8 * j + 2 * t] = acc[i][j][2];
                red[warp][16 * i + gq + 8][8 * j + 2 * t + 1] = acc[i][j][3];
            }
        __syncthreads();
        constexpr int NR = 16 * (GLU ? 1 : RT);
        for (int idx = threadIdx.x; idx < NR * MT * 8; idx += kStreamWarps * 32) {
            const int r = idx % NR, m = idx / NR, n = n0 + r;
            if (m0 + m < cnt && n < g.N) {
                float v = 0.f;
#pragma unroll
                for (int x = 0; x < kStreamWarps; x++) v += red[x][r][m];
                if constexpr (GLU) {
                    float up = 0.f;
#pragma unroll
                    for (int x = 0; x < kStreamWarps; x++) up += red[x][16 + r][m];
                    v = silu_f(v) * up;
                }
                put_out<O>(g, z, (size_t)(r0 + m0 + m), n, v);
            }
        }
        __syncthreads();
    }
}

template <typename T, typename O>
static int run_stream(cudaStream_t st, const GemmView &v, int rows, int groups, int glu) {
    const int mt = rows <= 8 ? 1 : rows <= 16 ? 2 : 4;
    const bool wide = !glu && (v.batch > 1 ? v.N * (long long)v.batch >= 32 * 148 * 2 : (mt > 1 || v.N >= 16 * 148 * 4) && v.N >= 32 * 100);
    const dim3 grid((v.N + (wide ? 31 : 15)) / (wide ? 32 : 16), groups);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(kStreamWarps * 32);
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;  // may start (and fetch weights) while its predecessor drains
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
#define RUN(MT)                                                                                            \
    {                                                                                                      \
        if (glu) MYNN_CUDA_OK(cudaLaunchKernelEx(&cfg, dense_stream_kernel<T, O, MT, 1, true>, v));        \
        else if (wide) MYNN_CUDA_OK(cudaLaunchKernelEx(&cfg, dense_stream_kernel<T, O, MT, 2, false>, v)); \
        else MYNN_CUDA_OK(cudaLaunchKernelEx(&cfg, dense_stream_kernel<T, O, MT, 1, false>, v));           \
    }
    if (mt == 1) RUN(1) else if (mt == 2) RUN(2) else RUN(4)
#undef RUN
    MYNN_LAUNCH_OK("dense_stream_kernel");
    return MYNN_OK;
}

template <typename T, typename O>
static int run_tile(cudaStream_t st, const GemmView &v, int groups, int glu) {
    const dim3 grid((v.N + 63) / 64, (v.M + 63) / 64, groups);
    if (glu) dense_tile_kernel<T, O, true><<<grid, 256, 0, st>>>(v);
    else dense_tile_kernel<T, O, false><<<grid, 256, 0, st>>>(v);
    MYNN_LAUNCH_OK("dense_tile_kernel");
    return MYNN_OK;
}

int launch_dense_gemm(cudaStream_t st, int dtype, const DenseGemm &g) {
    if (g.M < 0 || g.N <= 0 || g.K <= 0) return fail(MYNN_E_ARG, "dense_matmul: bad shape M=%d N=%d K=%d", g.M, g.N, g.K);
    if (!dtype_ok(dtype) || (g.out_dtype != dtype && g.out_dtype != MYNN_F32)) return fail(MYNN_E_ARG, "dense_matmul: bad dtypes %d -> %d", dtype, g.out_dtype);
    if (g.M == 0) return MYNN_OK;
    if (!g.out || !g.act || !g.w) return fail(MYNN_E_ARG, "dense_matmul: null pointer");
    if (g.row_groups > 1) {
        if (g.route || g.batch > 1 || g.out_f32 || g.group_rows < g.M) return fail(MYNN_E_ARG, "dense_matmul: %d groups of %d rows, %lld apart", g.row_groups, g.M, g.group_rows);
        if (!dense_gemm_tc_supported(dtype, g)) {  // one after the other
            for (int r = 0; r < g.row_groups; r++) {
                DenseGemm one = g;
                one.row_groups = 1;
                one.act = (const char *)g.act + (size_t)r * g.group_rows * (g.lda ? g.lda : g.K) * dtype_size(dtype);
                one.out = (char *)g.out + (size_t)r * g.group_rows * (g.ldo ? g.ldo : g.N) * dtype_size(g.out_dtype);
                if (int rc = launch_dense_gemm(st, dtype, one)) return rc;
            }
            return MYNN_OK;
        }
    }
    if (g.out_f32 ? g.n_main <= 0 || g.n_main > g.N : g.n_main != 0) return fail(MYNN_E_ARG, "dense_matmul: %d of %d columns in the main output", g.n_main, g.N);
    if (g.batch < 1 || g.batch > 65535 || (g.batch > 1 && (g.route || g.out_f32)) || (g.route && (g.out_f32 || g.out_block || g.lda || g.ldo)) ||
        (g.glu && (g.act_fn || g.out_f32)) || g.out_block < 0)
        return fail(MYNN_E_ARG, "dense_matmul: options that do not go together");
    GemmView v = {};
    v.out = g.out, v.act = g.act, v.w = g.w;
    v.M = g.M, v.N = g.N, v.K = g.K;
    v.n_main = g.out_f32 ? g.n_main : g.N;
    v.lda = g.lda ? g.lda : g.K;
    v.ldo = g.ldo ? g.ldo : v.n_main;
    v.act_fn = g.act_fn;
    v.out_block = g.out_block;
    v.out_block_stride = g.out_block_stride;
    v.batch = g.batch;
    v.act_stride = g.act_stride, v.out_stride = g.out_stride;
    v.out_f32 = g.out_f32;
    int groups = g.batch;
    long long rows = g.M;  // rows a weight block meets on average
    if (g.route) {
        v.off = g.route->off;
        v.active = g.route->active;
        v.n_active = g.route->n_active;
        v.tok_of = g.route->tok_of;
        v.gather = g.gather;
        const long long pairs = (long long)g.M * g.top;
        groups = (int)(pairs < g.experts ? pairs : g.experts);
        rows = (pairs + g.experts - 1) / g.experts * 2;  // the fuller experts of an uneven choice
        if (rows > g.M) rows = g.M;
    }
    const bool aligned = (((uintptr_t)g.act | (uintptr_t)g.w) % 16) == 0 && g.K % 8 == 0 && v.lda % 8 == 0 && g.act_stride % 8 == 0 && dtype != MYNN_F32;
    if (dense_gemm_tc_supported(dtype, g)) return launch_dense_gemm_tc(st, dtype, g);
    const bool stream = aligned && (rows <= 64 || g.batch > 1);
    const bool f32out = g.out_dtype == MYNN_F32;
    if (dtype == MYNN_F32) return run_tile<float, float>(st, v, groups, g.glu);
    if (dtype == MYNN_BF16) {
        if (stream) return f32out ? run_stream<__nv_bfloat16, float>(st, v, (int)rows, groups, g.glu) : run_stream<__nv_bfloat16, __nv_bfloat16>(st, v, (int)rows, groups, g.glu);
        return f32out ? run_tile<__nv_bfloat16, float>(st, v, groups, g.glu) : run_tile<__nv_bfloat16, __nv_bfloat16>(st, v, groups, g.glu);
    }
    if (stream) return f32out ? run_stream<__half, float>(st, v, (int)rows, groups, g.glu) : run_stream<__half, __half>(st, v, (int)rows, groups, g.glu);
    return f32out ? run_tile<__half, float>(st, v, groups, g.glu) : run_tile<__half, __half>(st, v, groups, g.glu);
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_dense_matmul(void *stream, void *out, const void *act, const void *w, int M, int N, int K, int dtype, int out_dtype, int glu,
                                      int32_t *status) {
    DenseGemm g;
    g.out = out;
    g.act = act;
    g.w = w;
    g.M = M, g.N = N, g.K = K;
    g.out_dtype = out_dtype;
    g.glu = glu;
    g.status = status;
    return launch_dense_gemm((cudaStream_t)stream, dtype, g);
}

extern "C" int mynn_b200_dense_matmul_ex(void *stream, void *out, const void *act, const void *w, int M, int N, int K, int dtype, int out_dtype, int act_fn,
                                         float *out_f32, int n_main, int out_block, long long out_block_stride, int lda, int ldo, int batch,
                                         long long act_stride, long long out_stride, int32_t *status) {
    DenseGemm g;
    g.out = out;
    g.act = act;
    g.w = w;
    g.M = M, g.N = N, g.K = K;
    g.out_dtype = out_dtype;
    g.act_fn = act_fn;
    g.out_f32 = out_f32;
    g.n_main = n_main;
    g.out_block = out_block;
    g.out_block_stride = out_block_stride;
    g.lda = lda, g.ldo = ldo;
    g.batch = batch;
    g.act_stride = act_stride, g.out_stride = out_stride;
    g.status = status;
    return launch_dense_gemm((cudaStream_t)stream, dtype, g);
}

extern "C" int mynn_b200_moe_matmul(void *stream, void *out, const void *act, const void *w, void *route_workspace, void *gather_workspace, int M, int N,
                                    int K, int experts, int top, int gather, int glu, int dtype, int out_dtype, int32_t *status) {
    if (M < 0 || experts <= 0 || top <= 0 || !route_workspace) return fail(MYNN_E_ARG, "moe_matmul: bad argument");
    if (M == 0) return MYNN_OK;
    const MoeRoute r = moe_route_bind(route_workspace, M, experts, top);
    DenseGemm g;
    g.out = out;
    g.act = act;
    g.w = w;
    g.M = M, g.N = N, g.K = K;
    g.out_dtype = out_dtype;
    g.glu = glu;
    g.route = &r;
    g.experts = experts;
    g.top = top;
    g.gather = gather;
    g.gather_ws = gather_workspace;
    g.status = status;
    return launch_dense_gemm((cudaStream_t)stream, dtype, g);
}
