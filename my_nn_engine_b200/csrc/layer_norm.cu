// Layer norms (and norms by root mean square) of the block decoder, fused with the residual step in front of them.
//
// A sandwich-normed layer does x += mult * LN(sublayer output) and then feeds LN(x) to the next sublayer.  Both norms, the
// residual sum, the combination of routed experts and the addition of the embedding output at the start of a repeated pass
// are row operations, so one kernel does them with one read of the sublayer output and one read and write of x.
// Mean and squared deviations are gathered per thread around the thread's own mean and merged pairwise (the update of Chan, Golub
// and LeVeque), which needs one block reduction per norm and stays accurate when the mean is large against the deviations.
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

struct Moments {
    float n, mean, m2;
};
__device__ __forceinline__ Moments merge(const Moments &a, const Moments &b) {
    Moments r;
    r.n = a.n + b.n;
    const float d = b.mean - a.mean, f = r.n > 0.f ? b.n / r.n : 0.f;
    r.mean = a.mean + d * f;
    r.m2 = a.m2 + b.m2 + d * d * a.n * f;
    return r;
}

// every thread gets the moments of the whole row; sm holds one entry per warp
__device__ __forceinline__ Moments block_moments(Moments v, Moments *sm) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        Moments u;
        u.n = __shfl_xor_sync(0xffffffffu, v.n, o);
        u.mean = __shfl_xor_sync(0xffffffffu, v.mean, o);
        u.m2 = __shfl_xor_sync(0xffffffffu, v.m2, o);
        v = merge(v, u);
    }
    const int warps = blockDim.x >> 5;
    __syncthreads();  // sm may still be read from the previous call
    if ((threadIdx.x & 31) == 0) sm[threadIdx.x >> 5] = v;
    __syncthreads();
    Moments t = sm[0];
    for (int w = 1; w < warps; w++) t = merge(t, sm[w]);
    return t;
}

template <typename T, int V>
__device__ __forceinline__ void load_vec(const T *p, float (&v)[V]) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 r = *reinterpret_cast<const uint2 *>(p);
        const T *e = reinterpret_cast<const T *>(&r);
#pragma unroll
        for (int i = 0; i < 4; i++) v[i] = to_f32<T>(e[i]);
    } else if constexpr (V == 4) {
        const float4 r = *reinterpret_cast<const float4 *>(p);
        v[0] = r.x, v[1] = r.y, v[2] = r.z, v[3] = r.w;
    } else {
#pragma unroll
        for (int i = 0; i < V; i++) v[i] = to_f32<T>(p[i]);
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_vec(T *p, const float (&v)[V]) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        uint2 r;
        T *e = reinterpret_cast<T *>(&r);
#pragma unroll
        for (int i = 0; i < 4; i++) e[i] = from_f32<T>(v[i]);
        *reinterpret_cast<uint2 *>(p) = r;
    } else if constexpr (V == 4) {
        *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
#pragma unroll
        for (int i = 0; i < V; i++) p[i] = from_f32<T>(v[i]);
    }
}

// grid = rows.  NV groups of V elements per thread live in registers between the passes (NV * V * blockDim.x >= W).
template <typename T, int V, int NV>
__global__ void __launch_bounds__(NV == 1 ? 256 : 1024) norm_step_kernel(const NormStep p) {
    __shared__ Moments sm[32];
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x, W = p.W;
    const int src = p.row_map ? p.row_map[row] : row;
    float xv[NV][V];
    const int step = blockDim.x * V, i0 = threadIdx.x * V;
    auto moments = [&](const float (&v)[NV][V]) {
        Moments m = {0.f, 0.f, 0.f};
        float s = 0.f;
        int n = 0;
#pragma unroll
        for (int j = 0; j < NV; j++)
            if (i0 + j * step < W) {
#pragma unroll
                for (int e = 0; e < V; e++) s += v[j][e];
                n += V;
            }
        m.n = (float)n;
        m.mean = n ? s / (float)n : 0.f;
#pragma unroll
        for (int j = 0; j < NV; j++)
            if (i0 + j * step < W) {
#pragma unroll
                for (int e = 0; e < V; e++) {
                    const float d = v[j][e] - m.mean;
                    m.m2 += d * d;
                }
            }
        return block_moments(m, sm);
    };
    // reciprocal deviation; for a norm by root mean square nothing is taken off, and mean(v^2) = var + mean^2
    auto scale_of = [&](Moments &m) {
        float v = m.m2 / (float)W;
        if (p.rms) {
            v += m.mean * m.mean;
            m.mean = 0.f;
        }
        return 1.0f / sqrtf(v + p.eps);
    };
    if (p.embed) {
        const long long id = min(max((long long)p.ids[row], 0ll), (long long)p.vocab - 1);
        const T *e = reinterpret_cast<const T *>(p.embed) + (size_t)id * W;
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int i = i0 + j * step;
            if (i < W) {
                load_vec<T, V>(e + i, xv[j]);
#pragma unroll
                for (int k = 0; k < V; k++) xv[j][k] *= p.embed_scale;
                store_vec<float, V>(p.x + (size_t)row * W + i, xv[j]);
                if (p.x0) store_vec<float, V>(p.x0 + (size_t)row * W + i, xv[j]);
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int i = i0 + j * step;
            if (i < W) load_vec<float, V>(p.x + (size_t)src * W + i, xv[j]);
        }
        if (p.sub) {
            float sv[NV][V];
            const T *sub = reinterpret_cast<const T *>(p.sub);
            if (p.pair_row) {
#pragma unroll
                for (int j = 0; j < NV; j++)
#pragma unroll
                    for (int k = 0; k < V; k++) sv[j][k] = 0.f;
                for (int s = 0; s < p.top; s++) {
                    const T *r = sub + (size_t)p.pair_row[(size_t)row * p.top + s] * W;
                    const float g = p.pair_w[(size_t)row * p.top + s];
#pragma unroll
                    for (int j = 0; j < NV; j++) {
                        const int i = i0 + j * step;
                        if (i < W) {
                            float t[V];
                            load_vec<T, V>(r + i, t);
#pragma unroll
                            for (int k = 0; k < V; k++) sv[j][k] += g * t[k];
                        }
                    }
                }
            } else {
#pragma unroll
                for (int j = 0; j < NV; j++) {
                    const int i = i0 + j * step;
                    if (i < W) load_vec<T, V>(sub + (size_t)row * W + i, sv[j]);
                }
            }
            Moments m = {0.f, 0.f, 0.f};
            float inv = 1.f;
            if (p.w1) {
                m = moments(sv);
                inv = scale_of(m);
            }
#pragma unroll
            for (int j = 0; j < NV; j++) {
                const int i = i0 + j * step;
                if (i < W) {
                    float w[V], b[V], z[V];
#pragma unroll
                    for (int k = 0; k < V; k++) w[k] = 1.f, b[k] = 0.f;
                    if (p.w1) load_vec<float, V>(p.w1 + i, w);
                    if (p.w1 && !p.rms) load_vec<float, V>(p.b1 + i, b);
                    if (p.add_x0) load_vec<float, V>(p.x0 + (size_t)row * W + i, z);
#pragma unroll
                    for (int k = 0; k < V; k++) {
                        xv[j][k] += p.mult * ((sv[j][k] - m.mean) * inv * w[k] + b[k]);
                        if (p.add_x0) xv[j][k] += z[k];
                    }
                    store_vec<float, V>(p.x + (size_t)row * W + i, xv[j]);
                }
            }
        }
    }
    if (!p.out) return;
    Moments m = moments(xv);
    const float inv = scale_of(m);
    T *out = reinterpret_cast<T *>(p.out) + (size_t)row * W;
#pragma unroll
    for (int j = 0; j < NV; j++) {
        const int i = i0 + j * step;
        if (i < W) {
            float w[V], b[V], y[V];
            load_vec<float, V>(p.w2 + i, w);
#pragma unroll
            for (int k = 0; k < V; k++) b[k] = 0.f;
            if (!p.rms) load_vec<float, V>(p.b2 + i, b);
#pragma unroll
            for (int k = 0; k < V; k++) y[k] = (xv[j][k] - m.mean) * inv * w[k] + b[k];
            store_vec<T, V>(out + i, y);
        }
    }
}

template <typename T, int V>
static int run_norm(cudaStream_t st, const NormStep &p, int rows) {
    const int groups = (p.W + V - 1) / V;
    const int nv = groups <= 256 ? 1 : groups <= 2048 ? 2 : groups <= 4096 ? 4 : groups <= 8192 ? 8 : V == 1 && groups <= 32768 ? 32 : 0;
    if (!nv) return fail(MYNN_E_UNSUPPORTED, "layer_norm: rows of %d elements", p.W);
    const int threads = ((groups + nv - 1) / nv + 31) / 32 * 32;
    switch (nv) {
        case 1: norm_step_kernel<T, V, 1><<<rows, threads, 0, st>>>(p); break;
        case 2: norm_step_kernel<T, V, 2><<<rows, threads, 0, st>>>(p); break;
        case 4: norm_step_kernel<T, V, 4><<<rows, threads, 0, st>>>(p); break;
        case 8: norm_step_kernel<T, V, 8><<<rows, threads, 0, st>>>(p); break;
        default:
            if constexpr (V == 1) norm_step_kernel<T, V, 32><<<rows, threads, 0, st>>>(p);
            break;
    }
    MYNN_LAUNCH_OK("norm_step_kernel");
    return MYNN_OK;
}

int launch_norm_step(cudaStream_t st, int dtype, const NormStep &p, int rows) {
    if (rows < 0 || p.W <= 0 || !p.x) return fail(MYNN_E_ARG, "layer_norm: bad shape rows=%d W=%d", rows, p.W);
    if (rows == 0) return MYNN_OK;
    uintptr_t a = (uintptr_t)p.embed | (uintptr_t)p.x | (uintptr_t)p.x0 | (uintptr_t)p.sub | (uintptr_t)p.out | (uintptr_t)p.w1 | (uintptr_t)p.b1 |
                  (uintptr_t)p.w2 | (uintptr_t)p.b2;
    const bool vec = p.W % 4 == 0 && a % 16 == 0;
    MYNN_DISPATCH_DTYPE(dtype, T, { return vec ? run_norm<T, 4>(st, p, rows) : run_norm<T, 1>(st, p, rows); });
    return MYNN_OK;
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_layer_norm(void *stream, void *out, const float *x, const float *weight, const float *bias, float eps, int rows,
                                    int W, int out_dtype) {
    if (rows < 0 || W <= 0) return fail(MYNN_E_ARG, "layer_norm: bad shape rows=%d W=%d", rows, W);
    if (!dtype_ok(out_dtype)) return fail(MYNN_E_ARG, "layer_norm: bad dtype %d", out_dtype);
    if (rows == 0) return MYNN_OK;
    if (!out || !x || !weight || !bias) return fail(MYNN_E_ARG, "layer_norm: null pointer");
    NormStep p;
    p.x = const_cast<float *>(x);  // without a sublayer output the kernel only reads it
    p.w2 = weight;
    p.b2 = bias;
    p.eps = eps;
    p.out = out;
    p.W = W;
    return launch_norm_step((cudaStream_t)stream, out_dtype, p, rows);
}

extern "C" int mynn_b200_residual_layer_norm(void *stream, float *x, const void *sub, const float *post_weight, const float *post_bias, float mult,
                                             const float *extra, const float *weight, const float *bias, void *out, float eps, int rows, int W,
                                             int dtype) {
    if (rows < 0 || W <= 0) return fail(MYNN_E_ARG, "residual_layer_norm: bad shape rows=%d W=%d", rows, W);
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "residual_layer_norm: bad dtype %d", dtype);
    if (rows == 0) return MYNN_OK;
    if (!x || !sub || !post_weight || !post_bias || (out && (!weight || !bias))) return fail(MYNN_E_ARG, "residual_layer_norm: null pointer");
    NormStep p;
    p.x = x;
    p.x0 = const_cast<float *>(extra);
    p.add_x0 = extra != nullptr;
    p.sub = sub;
    p.w1 = post_weight;
    p.b1 = post_bias;
    p.w2 = weight;
    p.b2 = bias;
    p.mult = mult;
    p.eps = eps;
    p.out = out;
    p.W = W;
    return launch_norm_step((cudaStream_t)stream, dtype, p, rows);
}

extern "C" int mynn_b200_residual_rms_norm(void *stream, float *x, const void *sub, const float *weight, void *out, float eps, int rows, int W, int dtype) {
    if (rows < 0 || W <= 0) return fail(MYNN_E_ARG, "residual_rms_norm: bad shape rows=%d W=%d", rows, W);
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "residual_rms_norm: bad dtype %d", dtype);
    if (rows == 0) return MYNN_OK;
    if (!x || (out && !weight)) return fail(MYNN_E_ARG, "residual_rms_norm: null pointer");
    NormStep p;
    p.x = x;
    p.sub = sub;
    p.w2 = weight;
    p.eps = eps;
    p.rms = 1;
    p.out = out;
    p.W = W;
    return launch_norm_step((cudaStream_t)stream, dtype, p, rows);
}
