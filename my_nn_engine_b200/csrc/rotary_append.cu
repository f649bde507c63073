// The step between the q/k/v projection and attention in a layer without convolutions: rotation of q and k, their division by the
// root mean square per head, and the append to the ring caches, in one launch.
//
// One warp takes one head of one token.  The head is staged as f32 in shared memory, because a rotated dimension's partner can sit
// in any lane (half a rotated range away, or next door); angles, rotation and norm are f32, the result is rounded once.
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

constexpr int kRotWarps = 8;

template <typename T, int V>
__device__ __forceinline__ void load_piece(const T *p, float (&v)[V]) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 r = *reinterpret_cast<const uint2 *>(p);
        const T *e = reinterpret_cast<const T *>(&r);
#pragma unroll
        for (int i = 0; i < 4; i++) v[i] = to_f32<T>(e[i]);
    } else if constexpr (V == 4) {
        const float4 r = *reinterpret_cast<const float4 *>(p);
        v[0] = r.x, v[1] = r.y, v[2] = r.z, v[3] = r.w;
    } else {
        v[0] = to_f32<T>(p[0]);
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_piece(T *p, const float (&v)[V]) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        uint2 r;
        T *e = reinterpret_cast<T *>(&r);
#pragma unroll
        for (int i = 0; i < 4; i++) e[i] = from_f32<T>(v[i]);
        *reinterpret_cast<uint2 *>(p) = r;
    } else if constexpr (V == 4) {
        *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        p[0] = from_f32<T>(v[0]);
    }
}

// grid (ceil((Hq + 2 G) / kRotWarps), B * S); dynamic shared memory: kRotWarps heads of D floats.  V: elements a lane moves at a time
// (4 needs D, E and, with halves, rot_dims / 2 to be multiples of 4).
template <typename T, int V>
__global__ void __launch_bounds__(kRotWarps * 32) rotary_append_kernel(const RotaryAppend p) {
    extern __shared__ float sm[];
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, job = blockIdx.x * kRotWarps + warp;
    if (job >= p.Hq + 2 * p.G) return;
    const int b = blockIdx.y / p.S, s = blockIdx.y - b * p.S, pos = *p.past + s, slot = pos % p.cache_rows;
    const int C = (p.Hq + p.G) * p.D + p.G * p.E;
    const T *row = reinterpret_cast<const T *>(p.proj) + (size_t)blockIdx.y * C;
    if (job >= p.Hq + p.G) {  // a value head: copied
        const int g = job - p.Hq - p.G;
        const T *src = row + (size_t)(p.Hq + p.G) * p.D + (size_t)g * p.E;
        T *dst = reinterpret_cast<T *>(p.v_cache) + ((size_t)(b * p.G + g) * p.cache_rows + slot) * p.E;
        for (int d = lane * V; d < p.E; d += 32 * V) {
            float v[V];
            load_piece<T, V>(src + d, v);
            store_piece<T, V>(dst + d, v);
        }
        return;
    }
    float *x = sm + (size_t)warp * p.D;
    const T *src = row + (size_t)job * p.D;
    for (int d = lane * V; d < p.D; d += 32 * V) {
        float v[V];
        load_piece<T, V>(src + d, v);
        store_piece<float, V>(x + d, v);
    }
    __syncwarp();
    const int half = p.rot_dims >> 1;
    const float *cs = p.cos_t + (size_t)pos * half, *sn = p.sin_t + (size_t)pos * half;
    auto rotated = [&](int d, float (&v)[V]) {
        load_piece<float, V>(x + d, v);
        if (d >= p.rot_dims) return;
        if (p.halves) {
            const bool low = d < half;
            const int i = low ? d : d - half;
            float u[V], c[V], a[V];
            load_piece<float, V>(x + (low ? d + half : i), u);
            load_piece<float, V>(cs + i, c);
            load_piece<float, V>(sn + i, a);
#pragma unroll
            for (int k = 0; k < V; k++) v[k] = low ? rope_low(v[k], u[k], c[k], a[k]) : rope_high(u[k], v[k], c[k], a[k]);
        } else {
#pragma unroll
            for (int k = 0; k < V; k++) {
                const int e = d + k;
                if (e >= p.rot_dims) break;
                const float c = cs[e >> 1], a = sn[e >> 1], w = x[e], u = x[e ^ 1];
                v[k] = e & 1 ? rope_high(u, w, c, a) : rope_low(w, u, c, a);
            }
        }
    };
    float inv = 1.f;
    if (p.qk_norm) {
        float ss = 0.f;
        for (int d = lane * V; d < p.D; d += 32 * V) {
            float v[V];
            rotated(d, v);
#pragma unroll
            for (int k = 0; k < V; k++) ss += v[k] * v[k];
        }
        inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.D + p.eps);
    }
    T *dst = job < p.Hq ? reinterpret_cast<T *>(p.q_out) + ((size_t)(b * p.Hq + job) * p.S + s) * p.D
                        : reinterpret_cast<T *>(p.k_cache) + ((size_t)(b * p.G + job - p.Hq) * p.cache_rows + slot) * p.D;
    for (int d = lane * V; d < p.D; d += 32 * V) {
        float v[V];
        rotated(d, v);
#pragma unroll
        for (int k = 0; k < V; k++) v[k] *= inv;
        store_piece<T, V>(dst + d, v);
    }
}

int launch_rotary_append(cudaStream_t st, int dtype, const RotaryAppend &p) {
    if (p.B <= 0 || p.S <= 0 || p.Hq <= 0 || p.G <= 0 || p.D <= 0 || p.E <= 0 || p.cache_rows <= 0 || p.rot_dims < 0 || p.rot_dims > p.D || p.rot_dims % 2)
        return fail(MYNN_E_ARG, "rotary_append: bad shape");
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "rotary_append: bad dtype %d", dtype);
    if (p.S > p.cache_rows) return fail(MYNN_E_ARG, "rotary_append: %d new positions in a ring of %d rows", p.S, p.cache_rows);
    if (!p.proj || !p.q_out || !p.k_cache || !p.v_cache || !p.past || (p.rot_dims && (!p.cos_t || !p.sin_t))) return fail(MYNN_E_ARG, "rotary_append: null pointer");
    if ((long long)p.B * p.S > 65535 || p.D > 1024) return fail(MYNN_E_UNSUPPORTED, "rotary_append: %d x %d tokens with heads of %d in one step", p.B, p.S, p.D);
    const uintptr_t a = (uintptr_t)p.proj | (uintptr_t)p.q_out | (uintptr_t)p.k_cache | (uintptr_t)p.v_cache | (uintptr_t)p.cos_t | (uintptr_t)p.sin_t;
    const bool vec = p.D % 4 == 0 && p.E % 4 == 0 && a % 16 == 0 && (!p.halves || (p.rot_dims / 2) % 4 == 0);
    const dim3 grid((p.Hq + 2 * p.G + kRotWarps - 1) / kRotWarps, p.B * p.S);
    const size_t smem = (size_t)kRotWarps * p.D * sizeof(float);
    MYNN_DISPATCH_DTYPE(dtype, T, {
        if (vec) rotary_append_kernel<T, 4><<<grid, kRotWarps * 32, smem, st>>>(p);
        else rotary_append_kernel<T, 1><<<grid, kRotWarps * 32, smem, st>>>(p);
    });
    MYNN_LAUNCH_OK("rotary_append_kernel");
    return MYNN_OK;
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_rotary_append(void *stream, void *q_out, void *k_cache, void *v_cache, const void *proj, const float *cos_table,
                                       const float *sin_table, int B, int S, int Hq, int Hkv, int D, int E, int rot_dims, int halves, int qk_norm,
                                       float eps, int cache_rows, const int32_t *past_dev, int dtype) {
    RotaryAppend p;
    p.proj = proj;
    p.cos_t = cos_table, p.sin_t = sin_table;
    p.rot_dims = rot_dims;
    p.halves = halves;
    p.qk_norm = qk_norm;
    p.eps = eps;
    p.q_out = q_out;
    p.k_cache = k_cache, p.v_cache = v_cache;
    p.cache_rows = cache_rows;
    p.B = B, p.S = S, p.Hq = Hq, p.G = Hkv, p.D = D, p.E = E;
    p.past = past_dev;
    return launch_rotary_append((cudaStream_t)stream, dtype, p);
}
