// Causal attention with a sliding window or chunks and a score soft cap over ring caches (position p lives in cache row p % cache_rows).
//
// launch_window_attention picks the kernel: the TMA-ring decode kernel (attention.cu) and the tcgen05 prefill kernels
// (attention_prefill_tc.cu) take 16-bit tensors with equal key and value sizes of 64 or 128; this file's own kernel takes any
// sizes and dtypes.  It gives one CTA to a query row: its warps deal out tiles of 32 keys, one key per lane for the scores (whole
// rows in f32 against the query in shared memory), value columns across the lanes for the weighted sum, running maximum and sum
// per warp, and one merge of the warps at the end.
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

constexpr int kWinWarps = 4;

// x -> cap * tanh(x / cap) in f32
__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

// dynamic shared memory: q [D], then per warp the output row [E]
template <typename T, int NE>
__global__ void __launch_bounds__(kWinWarps * 32) window_attention_kernel(const WindowAttention p) {
    extern __shared__ float sm[];
    __shared__ float sm_m[kWinWarps], sm_l[kWinWarps];
    pdl_trigger();
    pdl_wait();
    float *sq = sm, *so = sm + p.D;
    const int sq_i = blockIdx.x % p.Sq, bh = blockIdx.x / p.Sq, h = bh % p.Hq, b = bh / p.Hq, kvh = h / (p.Hq / p.Hkv);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int active = p.active ? *p.active : p.active_host;
    const int pos = active - p.Sq + sq_i, end = pos + 1;
    const int lo = max(max(0, active - p.cache_rows), first_visible(pos, p.window, p.chunk));
    const size_t q_row = p.layout == kByBatch ? blockIdx.x : p.layout == kByHead ? ((size_t)h * p.B + b) * p.Sq + sq_i : ((size_t)b * p.Sq + sq_i) * p.Hq + h;
    const T *q = reinterpret_cast<const T *>(p.q) + q_row * p.D;
    for (int d = threadIdx.x; d < p.D; d += blockDim.x) sq[d] = to_f32<T>(q[d]);
    __syncthreads();
    const size_t pair = p.layout == kByHead ? (size_t)kvh * p.B + b : (size_t)b * p.Hkv + kvh;
    const T *kb = reinterpret_cast<const T *>(p.k) + pair * p.cache_rows * p.D;
    const T *vb = reinterpret_cast<const T *>(p.v) + pair * p.cache_rows * p.E;
    float o[NE], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int e = 0; e < NE; e++) o[e] = 0.f;
    for (int base = lo + 32 * warp; base < end; base += 32 * kWinWarps) {
        const int key = base + lane;
        float s = -INFINITY;
        if (key < end) {
            const T *kr = kb + (size_t)(key % p.cache_rows) * p.D;
            float dot = 0.f;
            constexpr int V = 16 / sizeof(T);
            if (p.D % V == 0 && (uintptr_t)kb % 16 == 0) {
                for (int d = 0; d < p.D; d += V) {
                    const uint4 r = *reinterpret_cast<const uint4 *>(kr + d);
                    const T *e = reinterpret_cast<const T *>(&r);
#pragma unroll
                    for (int i = 0; i < V; i++) dot += sq[d + i] * to_f32<T>(e[i]);
                }
            } else {
                for (int d = 0; d < p.D; d++) dot += sq[d] * to_f32<T>(kr[d]);
            }
            s = dot * p.scale;
            if (p.softcap > 0.f) s = soft_cap(s, p.softcap);
        }
        const float m_new = fmaxf(m, warp_max(s));
        const float f = expf(m - m_new), w = expf(s - m_new);
        l = l * f + warp_sum(w);
        m = m_new;
#pragma unroll
        for (int e = 0; e < NE; e++) o[e] *= f;
        const int n = min(32, end - base);
        for (int i = 0; i < n; i++) {
            const float wi = __shfl_sync(0xffffffffu, w, i);
            const T *vr = vb + (size_t)((base + i) % p.cache_rows) * p.E;
#pragma unroll
            for (int e = 0; e < NE; e++) {
                const int d = lane + 32 * e;
                if (d < p.E) o[e] += wi * to_f32<T>(vr[d]);
            }
        }
    }
    if (lane == 0) {
        sm_m[warp] = m;
        sm_l[warp] = l;
    }
#pragma unroll
    for (int e = 0; e < NE; e++) {
        const int d = lane + 32 * e;
        if (d < p.E) so[warp * p.E + d] = o[e];
    }
    __syncthreads();
    float mx = sm_m[0];
#pragma unroll
    for (int w = 1; w < kWinWarps; w++) mx = fmaxf(mx, sm_m[w]);
    float L = 0.f, f[kWinWarps];
#pragma unroll
    for (int w = 0; w < kWinWarps; w++) {
        f[w] = sm_m[w] == -INFINITY ? 0.f : expf(sm_m[w] - mx);
        L += sm_l[w] * f[w];
    }
    T *out = reinterpret_cast<T *>(p.out) + (((size_t)b * p.Sq + sq_i) * p.Hq + h) * p.E;
    for (int d = threadIdx.x; d < p.E; d += blockDim.x) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWinWarps; w++) v += so[w * p.E + d] * f[w];
        out[d] = from_f32<T>(L > 0.f ? v / L : 0.f);
    }
}

template <typename T>
static int run_window(cudaStream_t st, const WindowAttention &p) {
    const unsigned rows = (unsigned)((long long)p.B * p.Hq * p.Sq);
    const size_t smem = (size_t)(p.D + kWinWarps * p.E) * sizeof(float);
    if (p.E <= 32) window_attention_kernel<T, 1><<<rows, kWinWarps * 32, smem, st>>>(p);
    else if (p.E <= 64) window_attention_kernel<T, 2><<<rows, kWinWarps * 32, smem, st>>>(p);
    else if (p.E <= 128) window_attention_kernel<T, 4><<<rows, kWinWarps * 32, smem, st>>>(p);
    else if (p.E <= 256) window_attention_kernel<T, 8><<<rows, kWinWarps * 32, smem, st>>>(p);
    else if (p.E <= 512) window_attention_kernel<T, 16><<<rows, kWinWarps * 32, smem, st>>>(p);
    else window_attention_kernel<T, 32><<<rows, kWinWarps * 32, smem, st>>>(p);
    MYNN_LAUNCH_OK("window_attention_kernel");
    return MYNN_OK;
}

static int check(int dtype, const WindowAttention &p) {
    if (p.B <= 0 || p.Hq <= 0 || p.Hkv <= 0 || p.Sq <= 0 || p.D <= 0 || p.E <= 0 || p.cache_rows <= 0 || p.Hq % p.Hkv) return fail(MYNN_E_ARG, "window_attention: bad shape");
    if (p.D > 1024 || p.E > 1024 || p.window < 0 || p.chunk < 0) return fail(MYNN_E_UNSUPPORTED, "window_attention: head sizes %d / %d", p.D, p.E);
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "window_attention: bad dtype %d", dtype);
    if (p.Sq > p.cache_rows) return fail(MYNN_E_ARG, "window_attention: %d query rows over a ring of %d rows", p.Sq, p.cache_rows);
    if (!p.out || !p.q || !p.k || !p.v) return fail(MYNN_E_ARG, "window_attention: null pointer");
    return MYNN_OK;
}

int launch_window_attention_plain(cudaStream_t st, int dtype, const WindowAttention &p) {
    if (int rc = check(dtype, p)) return rc;
    MYNN_DISPATCH_DTYPE(dtype, T, { return run_window<T>(st, p); });
    return MYNN_OK;
}

int launch_window_attention(cudaStream_t st, int dtype, const WindowAttention &p) {
    if (int rc = check(dtype, p)) return rc;
    if (window_attention_decode_supported(dtype, p)) return launch_window_attention_decode(st, dtype, p);
    if (window_attention_prefill_supported(dtype, p)) return launch_window_attention_prefill(st, dtype, p);
    return launch_window_attention_plain(st, dtype, p);
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_chunk_attention(void *stream, void *out, const void *q, const void *k, const void *v, float scale, float softcap,
                                         int window, int chunk, int head_major, int B, int Hq, int Hkv, int Sq, int D, int E, int cache_rows, int active,
                                          const int32_t *active_dev, int dtype, void *workspace, size_t workspace_bytes, int plain) {
    WindowAttention p;
    p.out = out;
    p.q = q, p.k = k, p.v = v;
    p.scale = scale;
    p.softcap = softcap;
    p.window = window > 0 ? window : 0;
    p.chunk = chunk > 0 ? chunk : 0;
    p.layout = head_major ? kByHead : kByBatch;
    p.B = B, p.Hq = Hq, p.Hkv = Hkv, p.Sq = Sq, p.D = D, p.E = E;
    p.cache_rows = cache_rows;
    p.active_host = active;
    p.active = active_dev;
    p.workspace = workspace;
    p.workspace_bytes = workspace_bytes;
    if (!active_dev && (active < Sq || active < 0)) return fail(MYNN_E_ARG, "window_attention: %d positions for %d query rows", active, Sq);
    return plain ? launch_window_attention_plain((cudaStream_t)stream, dtype, p) : launch_window_attention((cudaStream_t)stream, dtype, p);
}

extern "C" int mynn_b200_window_attention(void *stream, void *out, const void *q, const void *k, const void *v, float scale, float softcap,
                                          int window, int B, int Hq, int Hkv, int Sq, int D, int E, int cache_rows, int active,
                                          const int32_t *active_dev, int dtype, void *workspace, size_t workspace_bytes, int plain) {
    return mynn_b200_chunk_attention(stream, out, q, k, v, scale, softcap, window, 0, 0, B, Hq, Hkv, Sq, D, E, cache_rows, active, active_dev, dtype, workspace,
                                     workspace_bytes, plain);
}
