// The step between the q/k/v projection and attention in a layer with short convolutions: causal convolution over time on every
// projected channel, rotation of q and k, and the append to the ring caches, in one launch.
//
// A thread owns 8 neighbouring channels of one or four tokens (16-byte accesses; a scalar form covers sizes that are not multiples
// of 8 and more than four taps) and reads the taps of the earlier tokens from the projection of the same step or, for the first taps - 1 tokens, from the
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

// grid (channel groups of 8 / 128, B * ceil(S / TPT)), 128 threads.  A thread takes TPT tokens in a row: its weights stay in registers
// and every projection row is read once for all the taps it takes part in.
template <typename T, int TAPS, int TPT>
__global__ void __launch_bounds__(128) conv_step_vec_kernel(const ConvStep p, int write_hist) {
    pdl_trigger();
    pdl_wait();
    const int Cq = p.Hq * p.D, Ck = p.G * p.D, C = Cq + Ck + p.G * p.E;
    const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
    if (c >= C) return;
    const int groups = (p.S + TPT - 1) / TPT, b = blockIdx.y / groups, s0 = (blockIdx.y - b * groups) * TPT;
    const int past = *p.past;
    constexpr int LAG = TAPS > 0 ? TAPS - 1 : 0;
    uint4 raw[TPT + LAG];  // rows s0 - LAG .. s0 + TPT - 1
#pragma unroll
    for (int i = 0; i < TPT + LAG; i++) {
        raw[i] = make_uint4(0u, 0u, 0u, 0u);
        const int s = s0 + i - LAG;
        if (s < p.S) {
            bool zero;
            const T *src = conv_source<T>(p, b, s, 0, past, C, zero);
            if (!zero) raw[i] = *reinterpret_cast<const uint4 *>(src + c);
        }
    }
    float w[TAPS > 0 ? TAPS : 1][8];
#pragma unroll
    for (int j = 0; j < TAPS; j++) {
        const float4 a = *reinterpret_cast<const float4 *>(p.w + (size_t)j * C + c), d = *reinterpret_cast<const float4 *>(p.w + (size_t)j * C + c + 4);
        w[j][0] = a.x, w[j][1] = a.y, w[j][2] = a.z, w[j][3] = a.w, w[j][4] = d.x, w[j][5] = d.y, w[j][6] = d.z, w[j][7] = d.w;
    }
    // where token 0 of the sequence's step goes, and how far apart tokens are
    int d, rows = 0;
    T *dst;
    if (c < Cq) {
        const int h = c / p.D;
        d = c - h * p.D;
        dst = reinterpret_cast<T *>(p.q_out) + ((size_t)b * p.Hq + h) * p.S * p.D + d;
    } else if (c < Cq + Ck) {
        const int h = (c - Cq) / p.D;
        d = c - Cq - h * p.D;
        rows = p.cache_rows;
        dst = reinterpret_cast<T *>(p.k_cache) + ((size_t)b * p.G + h) * rows * p.D + d;
    } else {
        const int h = (c - Cq - Ck) / p.E;
        rows = p.cache_rows;
        dst = reinterpret_cast<T *>(p.v_cache) + ((size_t)b * p.G + h) * rows * p.E + (c - Cq - Ck - h * p.E);
        d = 1 << 30;  // values are not rotated
    }
    const int width = c < Cq + Ck ? p.D : p.E;
#pragma unroll
    for (int t = 0; t < TPT; t++) {
        const int s = s0 + t, pos = past + s;
        if (s >= p.S) break;
        float y[8] = {};
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS; j++) {
                const T *e = reinterpret_cast<const T *>(&raw[t + j]);
#pragma unroll
                for (int i = 0; i < 8; i++) y[i] += w[j][i] * to_f32<T>(e[i]);
            }
            if (write_hist && s >= p.S - p.hist_rows)
                *reinterpret_cast<uint4 *>(reinterpret_cast<T *>(p.hist) + ((size_t)b * p.hist_rows + pos % p.hist_rows) * C + c) = raw[t + LAG];
        } else {
            const T *e = reinterpret_cast<const T *>(&raw[t]);
#pragma unroll
            for (int i = 0; i < 8; i++) y[i] = to_f32<T>(e[i]);
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
        *reinterpret_cast<uint4 *>(dst + (size_t)(rows ? pos % rows : s) * width) = *reinterpret_cast<const uint4 *>(o);
    }
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

template <typename T>
static int launch_history(cudaStream_t st, const ConvStep &p, int C, int fused) {
    if (!p.taps || fused) return MYNN_OK;
    const int keep = p.S < p.hist_rows ? p.S : p.hist_rows;
    conv_history_kernel<T><<<(unsigned)(((long long)p.B * keep * C + 255) / 256), 256, 0, st>>>(p, keep, C);
    MYNN_LAUNCH_OK("conv_history_kernel");
    return MYNN_OK;
}

template <typename T, int TPT>
static int run_conv_vec(cudaStream_t st, const ConvStep &p, int C, int fused) {
    const dim3 grid((C / 8 + 127) / 128, p.B * ((p.S + TPT - 1) / TPT));
    switch (p.taps) {
        case 0: conv_step_vec_kernel<T, 0, TPT><<<grid, 128, 0, st>>>(p, fused); break;
        case 1: conv_step_vec_kernel<T, 1, TPT><<<grid, 128, 0, st>>>(p, fused); break;
        case 2: conv_step_vec_kernel<T, 2, TPT><<<grid, 128, 0, st>>>(p, fused); break;
        case 3: conv_step_vec_kernel<T, 3, TPT><<<grid, 128, 0, st>>>(p, fused); break;
        default: conv_step_vec_kernel<T, 4, TPT><<<grid, 128, 0, st>>>(p, fused); break;
    }
    MYNN_LAUNCH_OK("conv_step_vec_kernel");
    return launch_history<T>(st, p, C, fused);
}

template <typename T>
static int launch_conv_vec(cudaStream_t st, const ConvStep &p, int C, int fused) {
    // the grid's second dimension holds 65535 token groups
    if (p.S >= 8 || (long long)p.B * p.S > 65535) {
        if ((long long)p.B * ((p.S + 3) / 4) > 65535) return fail(MYNN_E_UNSUPPORTED, "conv_step: %d x %d tokens in one step", p.B, p.S);
        return run_conv_vec<T, 4>(st, p, C, fused);
    }
    return run_conv_vec<T, 1>(st, p, C, fused);
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
    const bool vec = dtype != MYNN_F32 && p.D % 8 == 0 && p.E % 8 == 0 && a % 16 == 0 && p.taps <= 4;
    const int fused = p.S + p.taps - 1 <= p.hist_rows;  // no ring slot is both read and written by this step
    if (vec) return dtype == MYNN_BF16 ? launch_conv_vec<__nv_bfloat16>(st, p, C, fused) : launch_conv_vec<__half>(st, p, C, fused);
    const unsigned blocks = (unsigned)(((long long)p.B * p.S * C + 255) / 256);
    {
        MYNN_DISPATCH_DTYPE(dtype, T, { conv_step_kernel<T><<<blocks, 256, 0, st>>>(p, fused); });
        MYNN_LAUNCH_OK("conv_step_kernel");
    }
    MYNN_DISPATCH_DTYPE(dtype, T, { return launch_history<T>(st, p, C, fused); });
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
