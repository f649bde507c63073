// The step between the q/k/v projection and attention in a layer with short convolutions: causal convolution over time on every
// projected channel, rotation of q and k, and the append to the ring caches, in one launch.
//
// A thread owns 8 neighbouring channels of one token (16-byte accesses; a scalar form covers sizes that are not multiples
// of 8) and reads the taps of the earlier tokens from the projection of the same step or, for the first taps - 1 tokens, from the
// ring that keeps the projections of the last hist_rows positions.  The rotation pairs dimensions 2i and 2i + 1, so a pair never
// leaves its thread.  New projections enter the ring in the same launch when the step is short enough that no slot read here can
// be one written here (always for a decode step); longer steps append their tail with a second small kernel.
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

// one channel of token s at step-relative time: projection, history, or zero before the sequence
template <typename T>
__device__ __forceinline__ const T *conv_source(const ConvStep &p, int b, int s, int lag, int past, int C, bool &zero) {
    const int t = s - lag;
    zero = false;
    if (t >= 0) return reinterpret_cast<const T *>(p.proj) + ((size_t)b * p.S + t) * C;
    const int pos = past + t;
    if (pos < 0) {
        zero = true;
        return reinterpret_cast<const T *>(p.proj);
    }
    return reinterpret_cast<const T *>(p.hist) + ((size_t)b * p.hist_rows + pos % p.hist_rows) * C;
}

template <typename T>
__global__ void __launch_bounds__(256) conv_step_vec_kernel(const ConvStep p, int write_hist) {
    pdl_trigger();
    pdl_wait();
    const int Cq = p.Hq * p.D, Ck = p.G * p.D, Cv = p.G * p.E, C = Cq + Ck + Cv;
    const int per = C >> 3;
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)p.B * p.S * per) return;
    const int row = (int)(idx / per), c = (int)(idx - (long long)row * per) << 3;
    const int b = row / p.S, s = row - b * p.S;
    const int past = *p.past, pos = past + s;
    float y[8] = {};
    const uint4 own = *reinterpret_cast<const uint4 *>(reinterpret_cast<const T *>(p.proj) + (size_t)row * C + c);
    auto add = [&](const uint4 &r, const float *w) {
        const T *e = reinterpret_cast<const T *>(&r);
        const float4 w0 = *reinterpret_cast<const float4 *>(w), w1 = *reinterpret_cast<const float4 *>(w + 4);
        y[0] += w0.x * to_f32<T>(e[0]), y[1] += w0.y * to_f32<T>(e[1]), y[2] += w0.z * to_f32<T>(e[2]), y[3] += w0.w * to_f32<T>(e[3]);
        y[4] += w1.x * to_f32<T>(e[4]), y[5] += w1.y * to_f32<T>(e[5]), y[6] += w1.z * to_f32<T>(e[6]), y[7] += w1.w * to_f32<T>(e[7]);
    };
    if (p.taps) {
        for (int j = 0; j + 1 < p.taps; j++) {
            bool zero;
            const T *src = conv_source<T>(p, b, s, p.taps - 1 - j, past, C, zero);
            if (!zero) add(*reinterpret_cast<const uint4 *>(src + c), p.w + (size_t)j * C + c);
        }
        add(own, p.w + (size_t)(p.taps - 1) * C + c);
        if (write_hist && s >= p.S - p.hist_rows)
            *reinterpret_cast<uint4 *>(reinterpret_cast<T *>(p.hist) + ((size_t)b * p.hist_rows + pos % p.hist_rows) * C + c) = own;
    } else {
        const T *e = reinterpret_cast<const T *>(&own);
#pragma unroll
        for (int i = 0; i < 8; i++) y[i] = to_f32<T>(e[i]);
    }
    T *dst;
    int d;
    if (c < Cq) {
        const int h = c / p.D;
        d = c - h * p.D;
        dst = reinterpret_cast<T *>(p.q_out) + (((size_t)b * p.Hq + h) * p.S + s) * p.D + d;
    } else if (c < Cq + Ck) {
        const int h = (c - Cq) / p.D;
        d = c - Cq - h * p.D;
        dst = reinterpret_cast<T *>(p.k_cache) + (((size_t)b * p.G + h) * p.cache_rows + pos % p.cache_rows) * p.D + d;
    } else {
        const int h = (c - Cq - Ck) / p.E;
        d = c - Cq - Ck - h * p.E;
        dst = reinterpret_cast<T *>(p.v_cache) + (((size_t)b * p.G + h) * p.cache_rows + pos % p.cache_rows) * p.E + d;
        d = 1 << 30;  // values are not rotated
    }
    if (d < p.rot_dims) {
        const size_t tab = (size_t)pos * (p.rot_dims >> 1) + (d >> 1);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            if (d + 2 * i >= p.rot_dims) break;
            const float cs = p.cos_t[tab + i], sn = p.sin_t[tab + i], u = y[2 * i], v = y[2 * i + 1];
            y[2 * i] = rope_low(u, v, cs, sn);
            y[2 * i + 1] = rope_high(u, v, cs, sn);
        }
    }
    T o[8];
#pragma unroll
    for (int i = 0; i < 8; i++) o[i] = from_f32<T>(y[i]);
    *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(o);
}

// any sizes and dtypes: one channel per thread; a rotated channel computes its partner's convolution as well
template <typename T>
__global__ void __launch_bounds__(256) conv_step_kernel(const ConvStep p, int write_hist) {
    pdl_trigger();
    pdl_wait();
    const int Cq = p.Hq * p.D, Ck = p.G * p.D, Cv = p.G * p.E, C = Cq + Ck + Cv;
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)p.B * p.S * C) return;
    const int row = (int)(idx / C), c = (int)(idx - (long long)row * C);
    const int b = row / p.S, s = row - b * p.S;
    const int past = *p.past, pos = past + s;
    const T *proj = reinterpret_cast<const T *>(p.proj) + (size_t)row * C;
    auto conv = [&](int ch) {
        if (!p.taps) return to_f32<T>(proj[ch]);
        float acc = 0.f;
        for (int j = 0; j < p.taps; j++) {
            bool zero;
            const T *src = conv_source<T>(p, b, s, p.taps - 1 - j, past, C, zero);
            if (!zero) acc += p.w[(size_t)j * C + ch] * to_f32<T>(src[ch]);
        }
        return acc;
    };
    float y = conv(c);
    if (p.taps && write_hist && s >= p.S - p.hist_rows)
        reinterpret_cast<T *>(p.hist)[((size_t)b * p.hist_rows + pos % p.hist_rows) * C + c] = proj[c];
    T *dst;
    int d;
    if (c < Cq) {
        const int h = c / p.D;
        d = c - h * p.D;
        dst = reinterpret_cast<T *>(p.q_out) + (((size_t)b * p.Hq + h) * p.S + s) * p.D + d;
    } else if (c < Cq + Ck) {
        const int h = (c - Cq) / p.D;
        d = c - Cq - h * p.D;
        dst = reinterpret_cast<T *>(p.k_cache) + (((size_t)b * p.G + h) * p.cache_rows + pos % p.cache_rows) * p.D + d;
    } else {
        const int h = (c - Cq - Ck) / p.E;
        d = c - Cq - Ck - h * p.E;
        dst = reinterpret_cast<T *>(p.v_cache) + (((size_t)b * p.G + h) * p.cache_rows + pos % p.cache_rows) * p.E + d;
        d = 1 << 30;
    }
    if (d < p.rot_dims) {
        const size_t tab = (size_t)pos * (p.rot_dims >> 1) + (d >> 1);
        const float cs = p.cos_t[tab], sn = p.sin_t[tab], other = conv(d & 1 ? c - 1 : c + 1);
        y = d & 1 ? rope_high(other, y, cs, sn) : rope_low(y, other, cs, sn);
    }
    *dst = from_f32<T>(y);
}

// the last min(S, hist_rows) projections of a long step -> ring
template <typename T>
__global__ void __launch_bounds__(256) conv_history_kernel(const ConvStep p, int keep, int C) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)p.B * keep * C) return;
    const int c = (int)(idx % C), r = (int)((idx / C) % keep), b = (int)(idx / C / keep);
    const int s = p.S - keep + r, pos = *p.past + s;
    reinterpret_cast<T *>(p.hist)[((size_t)b * p.hist_rows + pos % p.hist_rows) * C + c] =
        reinterpret_cast<const T *>(p.proj)[((size_t)b * p.S + s) * C + c];
}

int launch_conv_step(cudaStream_t st, int dtype, const ConvStep &p) {
    if (p.B <= 0 || p.S <= 0 || p.Hq <= 0 || p.G <= 0 || p.D <= 0 || p.E <= 0 || p.cache_rows <= 0 || p.taps < 0 || p.rot_dims < 0 || p.rot_dims > p.D ||
        p.rot_dims % 2)
        return fail(MYNN_E_ARG, "conv_step: bad shape");
    if (p.S > p.cache_rows) return fail(MYNN_E_ARG, "conv_step: %d new positions in a ring of %d rows", p.S, p.cache_rows);
    if (p.taps && (!p.w || !p.hist || p.hist_rows < p.taps)) return fail(MYNN_E_ARG, "conv_step: %d taps need a history of as many rows (%d given)", p.taps, p.hist_rows);
    if (!p.proj || !p.q_out || !p.k_cache || !p.v_cache || !p.past || (p.rot_dims && (!p.cos_t || !p.sin_t))) return fail(MYNN_E_ARG, "conv_step: null pointer");
    const int C = p.Hq * p.D + p.G * (p.D + p.E);
    const uintptr_t a = (uintptr_t)p.proj | (uintptr_t)p.hist | (uintptr_t)p.w | (uintptr_t)p.q_out | (uintptr_t)p.k_cache | (uintptr_t)p.v_cache;
    const bool vec = dtype != MYNN_F32 && p.D % 8 == 0 && p.E % 8 == 0 && a % 16 == 0;
    const int fused = p.S + p.taps - 1 <= p.hist_rows;  // no ring slot is both read and written by this step
    const long long n = (long long)p.B * p.S * (vec ? C / 8 : C);
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (vec) {
        if (dtype == MYNN_BF16) conv_step_vec_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>(p, fused);
        else conv_step_vec_kernel<__half><<<blocks, 256, 0, st>>>(p, fused);
        MYNN_LAUNCH_OK("conv_step_vec_kernel");
    } else {
        MYNN_DISPATCH_DTYPE(dtype, T, { conv_step_kernel<T><<<blocks, 256, 0, st>>>(p, fused); });
        MYNN_LAUNCH_OK("conv_step_kernel");
    }
    if (p.taps && !fused) {
        const int keep = p.S < p.hist_rows ? p.S : p.hist_rows;
        const unsigned hb = (unsigned)(((long long)p.B * keep * C + 255) / 256);
        MYNN_DISPATCH_DTYPE(dtype, T, { conv_history_kernel<T><<<hb, 256, 0, st>>>(p, keep, C); });
        MYNN_LAUNCH_OK("conv_history_kernel");
    }
    return MYNN_OK;
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_short_conv_append(void *stream, void *q_out, void *k_cache, void *v_cache, void *history, const void *proj,
                                           const float *conv, const float *cos_table, const float *sin_table, int B, int S, int Hq, int Hkv, int D,
                                           int E, int taps, int rot_dims, int cache_rows, int history_rows, const int32_t *past_dev, int dtype) {
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "short_conv_append: bad dtype %d", dtype);
    ConvStep p;
    p.proj = proj;
    p.hist = history;
    p.hist_rows = history_rows;
    p.w = conv;
    p.taps = taps;
    p.cos_t = cos_table;
    p.sin_t = sin_table;
    p.rot_dims = rot_dims;
    p.q_out = q_out;
    p.k_cache = k_cache;
    p.v_cache = v_cache;
    p.cache_rows = cache_rows;
    p.B = B, p.S = S, p.Hq = Hq, p.G = Hkv, p.D = D, p.E = E;
    p.past = past_dev;
    return launch_conv_step((cudaStream_t)stream, dtype, p);
}
