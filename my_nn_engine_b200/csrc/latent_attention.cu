// Attention over a cache of latents: one row of R numbers per position serves all heads as key and as value, once the queries have
// been brought into latent space (q W_uk) and with the value projection applied to the weighted mean of latents afterwards.
//
// latent_append_kernel      norms the two latents of a new token (queries', and the one that is cached) and appends the second.
// latent_attention_kernel   16-bit, R = 128, 256 or 512: few queries per sequence (decode, short portions).  A CTA takes 16 or 32 heads of
//                           one query and a range of positions, in tiles of 64 that cp.async keeps two of in shared memory.  The
//                           tile is the B operand of both products: scores (warps deal out heads and keys) and weighted sum (warps
//                           deal out the R columns).  Weights enter the second product as a high part and its remainder.
// latent_merge_kernel       combines the ranges of a query.
// Everything else (32-bit, other R) goes to the window attention kernel for any sizes, keys and values being the same rows.
#include <algorithm>

#include "attention_internal.cuh"
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

// grid (2, B * S): the queries' latent, the cached latent
template <typename T>
__global__ void __launch_bounds__(128) latent_append_kernel(const LatentAppend p) {
    __shared__ float red[4];
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.y, second = blockIdx.x, W = second ? p.R : p.Q;
    const T *x = reinterpret_cast<const T *>(p.proj) + (size_t)row * (p.Q + p.R) + (second ? p.Q : 0);
    const float *w = second ? p.wc : p.wq;
    T *out;
    if (second) {
        const int b = row / p.S, pos = *p.past + row - b * p.S;
        out = reinterpret_cast<T *>(p.cache) + ((size_t)b * p.cache_rows + pos % p.cache_rows) * p.R;
    } else {
        out = reinterpret_cast<T *>(p.q_out) + (size_t)row * p.Q;
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < W; i += 128) {
        const float v = to_f32<T>(x[i]);
        ss += v * v;
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    const float inv = 1.0f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)W + p.eps);
    for (int i = threadIdx.x; i < W; i += 128) out[i] = from_f32<T>(to_f32<T>(x[i]) * inv * w[i]);
}

int launch_latent_append(cudaStream_t st, int dtype, const LatentAppend &p) {
    if (p.B <= 0 || p.S <= 0 || p.Q <= 0 || p.R <= 0 || p.cache_rows < p.S) return fail(MYNN_E_ARG, "latent_append: bad shape");
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "latent_append: bad dtype %d", dtype);
    if (!p.proj || !p.wq || !p.wc || !p.q_out || !p.cache || !p.past) return fail(MYNN_E_ARG, "latent_append: null pointer");
    if ((long long)p.B * p.S > 65535) return fail(MYNN_E_UNSUPPORTED, "latent_append: %d x %d tokens in one step", p.B, p.S);
    MYNN_DISPATCH_DTYPE(dtype, T, { latent_append_kernel<T><<<dim3(2, p.B * p.S), 128, 0, st>>>(p); });
    MYNN_LAUNCH_OK("latent_append_kernel");
    return MYNN_OK;
}

// ---- attention -------------------------------------------------------------------------------------------------------
constexpr int kLatKeys = 64, kLatThreads = 256, kLatMaxSplits = 64;

struct LatParams {
    void *out;
    const void *q, *c;
    float scale_log2;  // scale * log2(e)
    int Sq, H, cache_rows, active_host, splits, groups;  // groups: CTAs that share the heads of a query
    const int32_t *active;
    float *ws_o, *ws_ml;  // [query][head][split][R], [query][head][split][2]
};

template <typename T, int R, int MT>
struct LatSmem {
    static constexpr int LD = R + 8, LP = kLatKeys + 8;
    T c[2][kLatKeys][LD];
    T q[16 * MT][LD];
    T p_hi[16 * MT][LP], p_lo[16 * MT][LP];
    float s[16 * MT][kLatKeys + 4];
    float alpha[16 * MT], m[16 * MT], l[16 * MT];
};

// grid (splits, B * Sq, head groups)
template <typename T, int R, int MT>
__global__ void __launch_bounds__(kLatThreads, 1) latent_attention_kernel(const LatParams p) {
    extern __shared__ __align__(16) uint8_t lat_smem[];
    using Sm = LatSmem<T, R, MT>;
    Sm &sm = *reinterpret_cast<Sm *>(lat_smem);
    constexpr int HB = 16 * MT, PIECES = R / 8, NT = R / 64;  // heads of the CTA, 16-byte pieces of a row, column tiles per warp
    pdl_trigger();
    pdl_wait();
    const int split = blockIdx.x, query = blockIdx.y, b = query / p.Sq, s_i = query - b * p.Sq, h0 = blockIdx.z * HB;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t4 = lane & 3;
    const int active = p.active ? *p.active : p.active_host;
    const int seen = active - p.Sq + s_i + 1;  // positions 0 .. seen - 1
    const int per = ((seen + p.splits - 1) / p.splits + kLatKeys - 1) / kLatKeys * kLatKeys;
    const int beg = min(split * per, seen), end = min(beg + per, seen), tiles = (end - beg + kLatKeys - 1) / kLatKeys;
    const T *cache = reinterpret_cast<const T *>(p.c) + (size_t)b * p.cache_rows * R;
    const int heads = min(HB, p.H - h0);
    const size_t slot0 = (size_t)query * p.H + h0;

    auto fetch = [&](int j) {
        for (int i = threadIdx.x; i < kLatKeys * PIECES; i += kLatThreads) {
            const int r = i / PIECES, d = (i % PIECES) * 8, pos = beg + j * kLatKeys + r;
            const bool in = pos < end;
            copy16(&sm.c[j & 1][r][d], cache + (size_t)(in ? pos : 0) * R + d, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (tiles > 0) fetch(0);
    {
        const T *q = reinterpret_cast<const T *>(p.q) + slot0 * R;
        for (int i = threadIdx.x; i < HB * PIECES; i += kLatThreads) {
            const int r = i / PIECES, d = (i % PIECES) * 8;
            *reinterpret_cast<uint4 *>(&sm.q[r][d]) = r < heads ? *reinterpret_cast<const uint4 *>(q + (size_t)r * R + d) : make_uint4(0u, 0u, 0u, 0u);
        }
        if (threadIdx.x < HB) sm.m[threadIdx.x] = -INFINITY, sm.l[threadIdx.x] = 0.f;
    }
    float o[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < NT; j++) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;

    for (int j = 0; j < tiles; j++) {
        const int buf = j & 1, key0 = beg + j * kLatKeys;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // tile j is there, tile j - 1 has been read by all
        if (j + 1 < tiles) fetch(j + 1);
        // ---- scores ----
        if constexpr (MT == 2) {  // 16 heads x 16 keys per warp
            const int mt = warp & 1, k0 = (warp >> 1) * 16;
            float sc[2][2][4] = {};
#pragma unroll 4
            for (int kk = 0; kk < R; kk += 32) {
#pragma unroll
                for (int u = 0; u < 2; u++) {  // two chains
                    uint32_t qa[4], kb[4];
                    ldsm4(qa, &sm.q[16 * mt + (lane & 15)][kk + 16 * u + 8 * (lane >> 4)]);
                    ldsm4(kb, &sm.c[buf][k0 + (lane & 7) + 8 * (lane >> 4)][kk + 16 * u + 8 * ((lane >> 3) & 1)]);
                    mma_kv<T>(sc[u][0], qa[0], qa[1], qa[2], qa[3], kb[0], kb[1]);
                    mma_kv<T>(sc[u][1], qa[0], qa[1], qa[2], qa[3], kb[2], kb[3]);
                }
            }
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int x = 0; x < 4; x++) sm.s[16 * mt + gq + 8 * (x >> 1)][k0 + 8 * n + 2 * t4 + (x & 1)] = sc[0][n][x] + sc[1][n][x];
        } else {  // 16 heads x 8 keys per warp
            const int k0 = warp * 8;
            float sc[2][4] = {};
#pragma unroll 4
            for (int kk = 0; kk < R; kk += 32) {
                uint32_t qa[4], qb[4], kb[4];
                ldsm4(qa, &sm.q[lane & 15][kk + 8 * (lane >> 4)]);
                ldsm4(qb, &sm.q[lane & 15][kk + 16 + 8 * (lane >> 4)]);
                ldsm4(kb, &sm.c[buf][k0 + (lane & 7)][kk + 8 * (lane >> 3)]);
                mma_kv<T>(sc[0], qa[0], qa[1], qa[2], qa[3], kb[0], kb[1]);
                mma_kv<T>(sc[1], qb[0], qb[1], qb[2], qb[3], kb[2], kb[3]);
            }
#pragma unroll
            for (int x = 0; x < 4; x++) sm.s[gq + 8 * (x >> 1)][k0 + 2 * t4 + (x & 1)] = sc[0][x] + sc[1][x];
        }
        __syncthreads();
        // ---- softmax: a warp takes 2 MT heads, two keys per lane ----
#pragma unroll
        for (int i = 0; i < 2 * MT; i++) {
            const int r = warp * 2 * MT + i, k = 2 * lane;
            const float2 raw = *reinterpret_cast<const float2 *>(&sm.s[r][k]);
            const float x0 = key0 + k < end ? raw.x * p.scale_log2 : -INFINITY, x1 = key0 + k + 1 < end ? raw.y * p.scale_log2 : -INFINITY;
            const float m_old = sm.m[r], m_new = fmaxf(m_old, warp_max(fmaxf(x0, x1)));  // finite: the tile has a key
            const float w0 = exp2f(x0 - m_new), w1 = exp2f(x1 - m_new), al = exp2f(m_old - m_new), sum = warp_sum(w0 + w1);
            uint32_t hi, lo;
            split_pack<T>(w0, w1, hi, lo);
            *reinterpret_cast<uint32_t *>(&sm.p_hi[r][k]) = hi;
            *reinterpret_cast<uint32_t *>(&sm.p_lo[r][k]) = lo;
            __syncwarp();
            if (lane == 0) {
                sm.m[r] = m_new;
                sm.l[r] = sm.l[r] * al + sum;
                sm.alpha[r] = al;
            }
        }
        __syncthreads();
        // ---- weighted sum: R / 8 columns per warp ----
        const int c0 = warp * (R / 8);
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const float a0 = sm.alpha[16 * i + gq], a1 = sm.alpha[16 * i + gq + 8];
#pragma unroll
            for (int n = 0; n < NT; n++) o[i][n][0] *= a0, o[i][n][1] *= a0, o[i][n][2] *= a1, o[i][n][3] *= a1;
        }
#pragma unroll
        for (int kk = 0; kk < kLatKeys; kk += 16) {
            uint32_t vb[NT / 2][4];
#pragma unroll
            for (int n = 0; n < NT / 2; n++) ldsm4t(vb[n], &sm.c[buf][kk + (lane & 15)][c0 + 16 * n + 8 * (lane >> 4)]);
#pragma unroll
            for (int i = 0; i < MT; i++) {
                uint32_t ph[4], pl[4];
                ldsm4(ph, &sm.p_hi[16 * i + (lane & 15)][kk + 8 * (lane >> 4)]);
                ldsm4(pl, &sm.p_lo[16 * i + (lane & 15)][kk + 8 * (lane >> 4)]);
#pragma unroll
                for (int n = 0; n < NT; n++) mma_kv<T>(o[i][n], ph[0], ph[1], ph[2], ph[3], vb[n >> 1][2 * (n & 1)], vb[n >> 1][2 * (n & 1) + 1]);
#pragma unroll
                for (int n = 0; n < NT; n++) mma_kv<T>(o[i][n], pl[0], pl[1], pl[2], pl[3], vb[n >> 1][2 * (n & 1)], vb[n >> 1][2 * (n & 1) + 1]);
            }
        }
    }
    __syncthreads();  // also orders the first writes of m and l when there was no tile
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int x = 0; x < 2; x++) {
            const int r = 16 * i + gq + 8 * x;
            if (r >= heads) continue;
            const float l = sm.l[r];
            if (p.splits == 1) {
                const float inv = l > 0.f ? 1.0f / l : 0.f;
                T *out = reinterpret_cast<T *>(p.out) + (slot0 + r) * R + warp * (R / 8) + 2 * t4;
#pragma unroll
                for (int n = 0; n < NT; n++) {
                    T two[2] = {from_f32<T>(o[i][n][2 * x] * inv), from_f32<T>(o[i][n][2 * x + 1] * inv)};
                    *reinterpret_cast<uint32_t *>(out + 8 * n) = *reinterpret_cast<const uint32_t *>(two);
                }
            } else if (tiles > 0) {
                float *out = p.ws_o + ((slot0 + r) * p.splits + split) * R + warp * (R / 8) + 2 * t4;
#pragma unroll
                for (int n = 0; n < NT; n++) *reinterpret_cast<float2 *>(out + 8 * n) = make_float2(o[i][n][2 * x], o[i][n][2 * x + 1]);
            }
        }
    if (p.splits > 1 && (int)threadIdx.x < heads) {
        float *ml = p.ws_ml + ((slot0 + threadIdx.x) * p.splits + split) * 2;
        ml[0] = sm.m[threadIdx.x];
        ml[1] = sm.l[threadIdx.x];
    }
}

// one CTA per (query, head), two neighbouring columns per thread (R / 2 threads)
template <typename T>
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatParams p, int R) {
    pdl_trigger();
    pdl_wait();
    const size_t slot = blockIdx.x;
    const float *ml = p.ws_ml + slot * p.splits * 2, *o = p.ws_o + slot * p.splits * R + 2 * threadIdx.x;
    float mx = -INFINITY;
    for (int s = 0; s < p.splits; s++) mx = fmaxf(mx, ml[2 * s]);
    float L = 0.f;
    float2 acc = make_float2(0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < p.splits; s++) {
        if (ml[2 * s] == -INFINITY) continue;
        const float f = exp2f(ml[2 * s] - mx);
        const float2 v = *reinterpret_cast<const float2 *>(o + (size_t)s * R);
        L += f * ml[2 * s + 1];
        acc.x += f * v.x, acc.y += f * v.y;
    }
    const float inv = L > 0.f ? 1.0f / L : 0.f;
    T two[2] = {from_f32<T>(acc.x * inv), from_f32<T>(acc.y * inv)};
    *reinterpret_cast<uint32_t *>(reinterpret_cast<T *>(p.out) + slot * R + 2 * threadIdx.x) = *reinterpret_cast<const uint32_t *>(two);
}

static int lat_splits(int queries, int groups, int rows_bound) {
    int s = 148 / (queries * groups);
    s = std::min(s, rows_bound / (2 * kLatKeys));  // at least two tiles each
    return std::max(1, std::min(s, kLatMaxSplits));
}
// 16 heads per CTA while that still leaves SMs idle, else 32 (the latents are then read half as often)
static int lat_head_tiles(int queries, int H, int rows_bound) {
    if (H <= 16) return 1;
    const int g = (H + 31) / 32;
    return queries * g * lat_splits(queries, g, rows_bound) < 74 ? 1 : 2;
}

size_t latent_attention_workspace_bytes(int B, int Sq, int H, int R, int cache_rows) {
    const long long queries = (long long)B * Sq;
    if (queries <= 0 || queries > 148) return 0;
    const int s = std::max(lat_splits((int)queries, (H + 15) / 16, cache_rows), lat_splits((int)queries, (H + 31) / 32, cache_rows));
    return s == 1 ? 0 : (size_t)queries * H * s * (R + 2) * sizeof(float) + 256;
}

static bool latent_tc_supported(int dtype, const LatentAttention &p) {
    return dtype != MYNN_F32 && (p.R == 128 || p.R == 256 || p.R == 512) && (((uintptr_t)p.q | (uintptr_t)p.c | (uintptr_t)p.out) % 16) == 0 &&
           (long long)p.B * p.Sq <= 65535 && p.H <= 65535 * 16;
}

template <typename T, int R, int MT>
static int run_latent(cudaStream_t st, const LatParams &l, int queries) {
    constexpr size_t smem = sizeof(LatSmem<T, R, MT>);
    static_assert(smem <= 227 * 1024, "shared memory of a CTA");
    auto kern = latent_attention_kernel<T, R, MT>;
    static bool attr_set = false;
    if (!attr_set) {
        MYNN_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set = true;
    }
    kern<<<dim3(l.splits, queries, l.groups), kLatThreads, smem, st>>>(l);
    MYNN_LAUNCH_OK("latent_attention_kernel");
    if (l.splits > 1) {
        latent_merge_kernel<T><<<(unsigned)((long long)queries * l.H), R / 2, 0, st>>>(l, R);
        MYNN_LAUNCH_OK("latent_merge_kernel");
    }
    return MYNN_OK;
}

template <typename T>
static int run_latent_any(cudaStream_t st, const LatParams &l, int queries, int R, int mt) {
    if (R == 128) return mt == 1 ? run_latent<T, 128, 1>(st, l, queries) : run_latent<T, 128, 2>(st, l, queries);
    if (R == 256) return mt == 1 ? run_latent<T, 256, 1>(st, l, queries) : run_latent<T, 256, 2>(st, l, queries);
    return mt == 1 ? run_latent<T, 512, 1>(st, l, queries) : run_latent<T, 512, 2>(st, l, queries);
}

int launch_latent_attention(cudaStream_t st, int dtype, const LatentAttention &p, bool plain) {
    if (p.B <= 0 || p.Sq <= 0 || p.H <= 0 || p.R <= 0 || p.cache_rows < p.Sq) return fail(MYNN_E_ARG, "latent_attention: bad shape");
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "latent_attention: bad dtype %d", dtype);
    if (!p.out || !p.q || !p.c) return fail(MYNN_E_ARG, "latent_attention: null pointer");
    if (plain || !latent_tc_supported(dtype, p)) {
        WindowAttention w;
        w.out = p.out;
        w.q = p.q, w.k = p.c, w.v = p.c;
        w.scale = p.scale;
        w.layout = kByToken;
        w.B = p.B, w.Hq = p.H, w.Hkv = 1, w.Sq = p.Sq, w.D = p.R, w.E = p.R;
        w.cache_rows = p.cache_rows;
        w.active_host = p.active_host;
        w.active = p.active;
        return launch_window_attention_plain(st, dtype, w);
    }
    const int queries = p.B * p.Sq, bound = p.active ? p.cache_rows : std::min(p.active_host, p.cache_rows);
    LatParams l = {};
    l.out = p.out;
    l.q = p.q, l.c = p.c;
    l.scale_log2 = p.scale * 1.4426950408889634f;
    l.Sq = p.Sq, l.H = p.H;
    l.cache_rows = p.cache_rows;
    l.active_host = p.active_host;
    l.active = p.active;
    const int mt = lat_head_tiles(queries, p.H, bound);
    l.groups = (p.H + 16 * mt - 1) / (16 * mt);
    l.splits = lat_splits(queries, l.groups, bound);
    if (l.splits > 1) {
        const size_t ml = (size_t)queries * p.H * l.splits * 2 * sizeof(float), head = (ml + 255) / 256 * 256;
        if (!p.workspace || p.workspace_bytes < head + (size_t)queries * p.H * l.splits * p.R * sizeof(float)) l.splits = 1;  // one CTA walks all positions
        l.ws_ml = (float *)p.workspace;
        l.ws_o = (float *)((char *)p.workspace + head);
    }
    return dtype == MYNN_BF16 ? run_latent_any<__nv_bfloat16>(st, l, queries, p.R, mt) : run_latent_any<__half>(st, l, queries, p.R, mt);
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_latent_append(void *stream, void *q_out, void *cache, const void *proj, const float *q_weight, const float *c_weight, float eps,
                                       int B, int S, int Q, int R, int cache_rows, const int32_t *past_dev, int dtype) {
    LatentAppend p;
    p.proj = proj;
    p.wq = q_weight, p.wc = c_weight;
    p.eps = eps;
    p.q_out = q_out, p.cache = cache;
    p.B = B, p.S = S, p.Q = Q, p.R = R;
    p.cache_rows = cache_rows;
    p.past = past_dev;
    return launch_latent_append((cudaStream_t)stream, dtype, p);
}

extern "C" size_t mynn_b200_latent_attention_workspace_bytes(int B, int Sq, int H, int R, int cache_rows) {
    return latent_attention_workspace_bytes(B, Sq, H, R, cache_rows);
}

extern "C" int mynn_b200_latent_attention(void *stream, void *out, const void *q, const void *cache, float scale, int B, int Sq, int H, int R, int cache_rows,
                                          int active, const int32_t *active_dev, int dtype, void *workspace, size_t workspace_bytes, int plain) {
    if (!active_dev && (active < Sq || active > cache_rows)) return fail(MYNN_E_ARG, "latent_attention: %d positions for %d query rows over %d rows", active, Sq, cache_rows);
    LatentAttention p;
    p.out = out;
    p.q = q, p.c = cache;
    p.scale = scale;
    p.B = B, p.Sq = Sq, p.H = H, p.R = R;
    p.cache_rows = cache_rows;
    p.active_host = active;
    p.active = active_dev;
    p.workspace = workspace;
    p.workspace_bytes = workspace_bytes;
    return launch_latent_attention((cudaStream_t)stream, dtype, p, plain != 0);
}
