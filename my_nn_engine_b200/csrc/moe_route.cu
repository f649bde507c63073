// Expert routing: softmax over the router logits, the groups with the best member, the best experts of those groups, and the
// (token, slot) pairs ordered by expert for the grouped matrix products.
//
// One warp per token makes the choice (logits in shared memory, repeated warp-wide maxima; equal scores go to the lower index).
// A step of a few tokens runs entirely in one CTA; longer ones count in global memory, order in a second kernel and scatter in a
// third.  The order of the pairs of one expert is not fixed, and nothing depends on it: every pair is a row of its own.
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

static size_t up16(size_t x) { return (x + 15) / 16 * 16; }

// The counts come first and have a fixed size: layers with different numbers of experts share one workspace, and what has to be
// zero between calls must not move over what another layer has written.
constexpr int kMaxExperts = 1024;
constexpr size_t kCountBytes = kMaxExperts * 4;

static int max_tiles(int M, int experts, int top) {
    const long long pairs = (long long)M * top;
    return (int)(pairs / kMoeTileRows + (experts < pairs ? experts : pairs) + 1);
}

size_t moe_route_bytes(int M, int experts, int top) {
    const size_t pairs = (size_t)M * top;
    return kCountBytes + 4 * up16(pairs * 4) + 2 * up16((size_t)(experts + 1) * 4) + 2 * up16((size_t)max_tiles(M, experts, top) * 4) + 32;
}

MoeRoute moe_route_bind(void *base, int M, int experts, int top) {
    const size_t pairs = (size_t)M * top;
    char *p = (char *)base;
    auto take = [&](size_t n) {
        char *r = p;
        p += up16(n);
        return r;
    };
    MoeRoute r;
    r.count = (int32_t *)take(kCountBytes);
    r.pair_w = (float *)take(pairs * 4);
    r.pair_row = (int32_t *)take(pairs * 4);
    r.pair_e = (int32_t *)take(pairs * 4);
    r.tok_of = (int32_t *)take(pairs * 4);
    r.off = (int32_t *)take((size_t)(experts + 1) * 4);
    r.active = (int32_t *)take((size_t)(experts + 1) * 4);
    r.tile_e = (int32_t *)take((size_t)max_tiles(M, experts, top) * 4);
    r.tile_row = (int32_t *)take((size_t)max_tiles(M, experts, top) * 4);
    r.n_active = (int32_t *)take(4);
    r.n_tiles = (int32_t *)take(4);
    return r;
}

// larger value first, then the lower index
__device__ __forceinline__ void warp_argmax(float &v, int &i) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float v2 = __shfl_xor_sync(0xffffffffu, v, o);
        const int i2 = __shfl_xor_sync(0xffffffffu, i, o);
        if (v2 > v || (v2 == v && i2 < i)) {
            v = v2;
            i = i2;
        }
    }
}

// The choice for one token by one warp; z holds its E logits and is overwritten.  Slot s: expert in lane s's `e`, weight in `w`.
__device__ __forceinline__ void choose(float *z, const float *src, int E, int top, int groups, int keep, int &e_out, float &w_out) {
    const int lane = threadIdx.x & 31;
    float mx = -INFINITY;
    for (int i = lane; i < E; i += 32) {
        const float v = src[i];
        z[i] = fmaxf(v, -3.0e38f);  // also for NaN: every expert stays comparable, and above the excluded ones
        mx = fmaxf(mx, z[i]);
    }
    mx = warp_max(mx);
    float sum = 0.f;
    for (int i = lane; i < E; i += 32) sum += expf(src[i] - mx);  // a NaN logit makes the weights NaN
    sum = warp_sum(sum);
    __syncwarp();
    if (keep < groups) {
        // softmax is monotonic, so group scores may be compared as logits
        const int per = E / groups;
        unsigned kept_lo = 0, kept_hi = 0;  // this lane's groups lane, lane + 32
        float gs[2];
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int g = lane + 32 * u;
            gs[u] = -INFINITY;
            if (g < groups)
                for (int i = 0; i < per; i++) gs[u] = fmaxf(gs[u], z[g * per + i]);
        }
        for (int k = 0; k < keep; k++) {
            float v = -INFINITY;
            int g = 1 << 20;
            if (lane < groups && !kept_lo) v = gs[0], g = lane;
            if (lane + 32 < groups && !kept_hi && (gs[1] > v || g == 1 << 20)) v = gs[1], g = lane + 32;
            warp_argmax(v, g);
            if (g == lane) kept_lo = 1;
            if (g == lane + 32) kept_hi = 1;
        }
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int g = lane + 32 * u;
            if (g < groups && !(u ? kept_hi : kept_lo))
                for (int i = 0; i < per; i++) z[g * per + i] = -INFINITY;
        }
        __syncwarp();
    }
    e_out = 0;
    w_out = 0.f;
    for (int s = 0; s < top; s++) {
        float v = -INFINITY;
        int e = 1 << 20;
        for (int i = lane; i < E; i += 32)
            if (z[i] > v || e == 1 << 20) v = z[i], e = i;
        warp_argmax(v, e);
        if (lane == s) {
            e_out = e;
            w_out = expf(v - mx) / sum;
        }
        __syncwarp();
        if (lane == 0) z[e] = -INFINITY;
        __syncwarp();
    }
}

// counts -> offsets, list of used experts, tiles; one warp.  Counts are cleared on the way.
__device__ __forceinline__ void order_experts(const MoeRoute &r, int32_t *count, int E) {
    const int lane = threadIdx.x & 31;
    int off = 0, act = 0, tiles = 0;
    for (int base = 0; base < E; base += 32) {
        const int e = base + lane, c = e < E ? count[e] : 0;
        const int nt = (c + kMoeTileRows - 1) / kMoeTileRows, used = c > 0;
        int so = c, st = nt, su = used;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int a = __shfl_up_sync(0xffffffffu, so, o), b = __shfl_up_sync(0xffffffffu, st, o), d = __shfl_up_sync(0xffffffffu, su, o);
            if (lane >= o) so += a, st += b, su += d;
        }
        const int my_off = off + so - c, my_tile = tiles + st - nt;
        if (e < E) {
            r.off[e] = my_off;
            if (used) r.active[act + su - 1] = e;
            for (int t = 0; t < nt; t++) {
                r.tile_e[my_tile + t] = e;
                r.tile_row[my_tile + t] = my_off + t * kMoeTileRows;
            }
            count[e] = 0;
        }
        off += __shfl_sync(0xffffffffu, so, 31);
        tiles += __shfl_sync(0xffffffffu, st, 31);
        act += __shfl_sync(0xffffffffu, su, 31);
    }
    if (lane == 0) {
        r.off[E] = off;
        *r.n_active = act;
        *r.n_tiles = tiles;
    }
}

// everything for a few tokens: one CTA; dynamic shared memory: E logits per warp, then E counts
__global__ void __launch_bounds__(1024) moe_route_small_kernel(const MoeRoute r, const float *logits, int M, int E, int top, int groups, int keep) {
    extern __shared__ float sm[];
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    float *z = sm + (size_t)warp * E;
    int32_t *count = reinterpret_cast<int32_t *>(sm + (size_t)warps * E);
    for (int i = threadIdx.x; i < E; i += blockDim.x) count[i] = 0;
    __syncthreads();
    for (int t = warp; t < M; t += warps) {
        int e;
        float w;
        choose(z, logits + (size_t)t * E, E, top, groups, keep, e, w);
        if (lane < top) {
            const size_t pair = (size_t)t * top + lane;
            r.pair_w[pair] = w;
            r.pair_e[pair] = e;
            r.pair_row[pair] = atomicAdd(&count[e], 1);  // place inside the expert for now
        }
    }
    __syncthreads();
    if (warp == 0) order_experts(r, count, E);
    __syncthreads();  // global writes of this CTA are visible to it
    for (int i = threadIdx.x; i < M * top; i += blockDim.x) {
        const int row = r.off[r.pair_e[i]] + r.pair_row[i];
        r.pair_row[i] = row;
        r.tok_of[row] = i / top;
    }
}

__global__ void __launch_bounds__(256) moe_choose_kernel(const MoeRoute r, const float *logits, int M, int E, int top, int groups, int keep) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * (blockDim.x >> 5) + warp;
    if (t >= M) return;
    int e;
    float w;
    choose(sm + (size_t)warp * E, logits + (size_t)t * E, E, top, groups, keep, e, w);
    if (lane < top) {
        const size_t pair = (size_t)t * top + lane;
        r.pair_w[pair] = w;
        r.pair_e[pair] = e;
        r.pair_row[pair] = atomicAdd(&r.count[e], 1);
    }
}
__global__ void moe_order_kernel(const MoeRoute r, int E) { order_experts(r, r.count, E); }
__global__ void __launch_bounds__(256) moe_scatter_kernel(const MoeRoute r, int pairs, int top) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= pairs) return;
    const int row = r.off[r.pair_e[i]] + r.pair_row[i];
    r.pair_row[i] = row;
    r.tok_of[row] = i / top;
}

int launch_moe_route(cudaStream_t st, const MoeRoute &r, const float *logits, int M, int E, int top, int groups, int keep) {
    if (M <= 0 || E <= 0 || top <= 0 || top > 32 || top > E || groups <= 0 || groups > 64 || E % groups || keep <= 0 || keep > groups || E > kMaxExperts ||
        (long long)top > (long long)keep * (E / groups))
        return fail(MYNN_E_ARG, "moe_route: bad routing (%d experts, top %d, %d of %d groups)", E, top, keep, groups);
    if ((long long)M * top > (1ll << 30)) return fail(MYNN_E_UNSUPPORTED, "moe_route: too many tokens");
    if (M <= 64) {
        const int warps = M < 32 ? M : 32;
        const size_t smem = (size_t)(warps + 1) * E * 4;
        if (smem > 48 * 1024) MYNN_CUDA_OK(cudaFuncSetAttribute(moe_route_small_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        moe_route_small_kernel<<<1, warps * 32, smem, st>>>(r, logits, M, E, top, groups, keep);
        MYNN_LAUNCH_OK("moe_route_small_kernel");
        return MYNN_OK;
    }
    moe_choose_kernel<<<(M + 7) / 8, 256, (size_t)8 * E * 4, st>>>(r, logits, M, E, top, groups, keep);
    MYNN_LAUNCH_OK("moe_choose_kernel");
    moe_order_kernel<<<1, 32, 0, st>>>(r, E);
    MYNN_LAUNCH_OK("moe_order_kernel");
    moe_scatter_kernel<<<(M * top + 255) / 256, 256, 0, st>>>(r, M * top, top);
    MYNN_LAUNCH_OK("moe_scatter_kernel");
    return MYNN_OK;
}

}  // namespace mynn

using namespace mynn;

extern "C" size_t mynn_b200_moe_workspace_bytes(int M, int experts, int top) {
    if (M <= 0 || experts <= 0 || top <= 0) return 0;
    return moe_route_bytes(M, experts, top);
}

extern "C" int mynn_b200_moe_route(void *stream, void *workspace, size_t workspace_bytes, float *weights_out, int32_t *experts_out, const float *logits,
                                   int M, int experts, int top, int groups, int groups_keep) {
    if (M < 0 || experts <= 0 || top <= 0) return fail(MYNN_E_ARG, "moe_route: bad shape");
    if (M == 0) return MYNN_OK;
    if (!workspace || !logits) return fail(MYNN_E_ARG, "moe_route: null pointer");
    if (workspace_bytes < moe_route_bytes(M, experts, top) || (uintptr_t)workspace % 16)
        return fail(MYNN_E_ARG, "moe_route: a 16-byte aligned workspace of %zu bytes is needed, %zu given", moe_route_bytes(M, experts, top), workspace_bytes);
    const MoeRoute r = moe_route_bind(workspace, M, experts, top);
    cudaStream_t st = (cudaStream_t)stream;
    if (int rc = launch_moe_route(st, r, logits, M, experts, top, groups, groups_keep)) return rc;
    const size_t n = (size_t)M * top * 4;
    if (weights_out) MYNN_CUDA_OK(cudaMemcpyAsync(weights_out, r.pair_w, n, cudaMemcpyDeviceToDevice, st));
    if (experts_out) MYNN_CUDA_OK(cudaMemcpyAsync(experts_out, r.pair_e, n, cudaMemcpyDeviceToDevice, st));
    return MYNN_OK;
}
