// Attention over a cache of latents: one row of R numbers per position serves all heads as key and as value, once the queries have
// been brought into latent space (q W_uk) and with the value projection applied to the weighted mean of latents afterwards.
//
// latent_append_kernel      norms the two latents of a new token (queries', and the one that is cached) and appends the second.
// latent_attention_kernel   16-bit, R = 128, 256 or 512: few queries per sequence (decode, short portions).  A CTA takes 16 or 32 heads of
//                           one query and a range of positions, in tiles of 64 that cp.async keeps two of in shared memory.  The
//                           tile is the B operand of both products.  For the scores a warp takes 16 heads and a part of the R columns, so
//                           that its queries stay in registers; the parts meet in shared memory.  For the weighted sum the warps deal
//                           out the R columns; weights are rounded to 16 bits there, as in the prefill kernels (mma.sync sets the
//                           pace with 32 heads: a second product for the remainders costs 20 % of the kernel).
// latent_merge_kernel       combines the ranges of a query.
// Everything else (32-bit, other R) goes to the window attention kernel for any sizes, keys and values being the same rows.
#include <algorithm>

#include "attention_internal.cuh"
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

// grid (2, B * S): the queries' latent, the cached latent.  V: elements a thread moves at a time (8 needs 16-bit rows of 16-byte pieces); up
// to 2 V elements per thread stay in registers between the sum and the store, longer rows are read again.
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_append_kernel(const LatentAppend p) {
    __shared__ float red[8];
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
    auto load = [&](int i, float (&v)[V]) {
        if constexpr (V == 8) {
            const uint4 r = *reinterpret_cast<const uint4 *>(x + i);
            const T *e = reinterpret_cast<const T *>(&r);
#pragma unroll
            for (int k = 0; k < 8; k++) v[k] = to_f32<T>(e[k]);
        } else {
            v[0] = to_f32<T>(x[i]);
        }
    };
    float v[2][V], ss = 0.f;
    const int step = 256 * V, i0 = threadIdx.x * V;
#pragma unroll
    for (int j = 0; j < 2; j++)
        if (i0 + j * step < W) {
            load(i0 + j * step, v[j]);
#pragma unroll
            for (int k = 0; k < V; k++) ss += v[j][k] * v[j][k];
        }
    for (int i = i0 + 2 * step; i < W; i += step) {
        float u[V];
        load(i, u);
#pragma unroll
        for (int k = 0; k < V; k++) ss += u[k] * u[k];
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int k = 0; k < 8; k++) total += red[k];
    const float inv = 1.0f / sqrtf(total / (float)W + p.eps);
    auto store = [&](int i, const float (&u)[V]) {
        if constexpr (V == 8) {
            const float4 a = *reinterpret_cast<const float4 *>(w + i), b = *reinterpret_cast<const float4 *>(w + i + 4);
            const float g[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
            uint4 r;
            T *e = reinterpret_cast<T *>(&r);
#pragma unroll
            for (int k = 0; k < 8; k++) e[k] = from_f32<T>(u[k] * inv * g[k]);
            *reinterpret_cast<uint4 *>(out + i) = r;
        } else {
            out[i] = from_f32<T>(u[0] * inv * w[i]);
        }
    };
#pragma unroll
    for (int j = 0; j < 2; j++)
        if (i0 + j * step < W) store(i0 + j * step, v[j]);
    for (int i = i0 + 2 * step; i < W; i += step) {
        float u[V];
        load(i, u);
        store(i, u);
    }
}

int launch_latent_append(cudaStream_t st, int dtype, const LatentAppend &p) {
    if (p.B <= 0 || p.S <= 0 || p.Q <= 0 || p.R <= 0 || p.cache_rows < p.S) return fail(MYNN_E_ARG, "latent_append: bad shape");
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "latent_append: bad dtype %d", dtype);
    if (!p.proj || !p.wq || !p.wc || !p.q_out || !p.cache || !p.past) return fail(MYNN_E_ARG, "latent_append: null pointer");
    if ((long long)p.B * p.S > 65535) return fail(MYNN_E_UNSUPPORTED, "latent_append: %d x %d tokens in one step", p.B, p.S);
    const dim3 grid(2, p.B * p.S);
    const uintptr_t a = (uintptr_t)p.proj | (uintptr_t)p.q_out | (uintptr_t)p.cache | (uintptr_t)p.wq | (uintptr_t)p.wc;
    if (dtype != MYNN_F32 && p.Q % 8 == 0 && p.R % 8 == 0 && a % 16 == 0) {
        if (dtype == MYNN_BF16) latent_append_kernel<__nv_bfloat16, 8><<<grid, 256, 0, st>>>(p);
        else latent_append_kernel<__half, 8><<<grid, 256, 0, st>>>(p);
    } else {
        MYNN_DISPATCH_DTYPE(dtype, T, { latent_append_kernel<T, 1><<<grid, 256, 0, st>>>(p); });
    }
    MYNN_LAUNCH_OK("latent_append_kernel");
    return MYNN_OK;
}

// ---- attention -------------------------------------------------------------------------------------------------------
constexpr int kLatKeys = 64, kLatMaxSplits = 64;
constexpr int lat_warps(int R) { return R == 128 ? 8 : 16; }  // a warp takes at least 16 columns of the weighted sum

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
    static constexpr int LD = R + 8, LP = kLatKeys + 8, LS = kLatKeys + 8, WARPS = lat_warps(R), PARTS = WARPS / MT;
    T c[2][kLatKeys][LD];
    T p[16 * MT][LP];
    float s[PARTS][16 * MT][LS];  // partial scores
    float alpha[16 * MT], m[16 * MT], l[16 * MT];
};

__device__ __forceinline__ float lat_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// grid (splits, B * Sq, head groups)
template <typename T, int R, int MT>
__global__ void __launch_bounds__(lat_warps(R) * 32, R == 128 ? 2 : 1) latent_attention_kernel(const LatParams p) {
    extern __shared__ __align__(16) uint8_t lat_smem[];
    using Sm = LatSmem<T, R, MT>;
    Sm &sm = *reinterpret_cast<Sm *>(lat_smem);
    constexpr int WARPS = Sm::WARPS, HB = 16 * MT, PIECES = R / 8, NT = R / (8 * WARPS);  // heads of the CTA, 16-byte pieces of a row, column tiles per warp
    constexpr int PARTS = Sm::PARTS, RP = R / PARTS, KS = RP / 16;  // the scores' contraction is cut into parts
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

    // a thread copies one 16-byte column of every RC-th row
    constexpr int RC = WARPS * 32 / PIECES;
    const int c_row = threadIdx.x / PIECES, c_col = (threadIdx.x % PIECES) * 8;
    const uint32_t c_dst = (uint32_t)__cvta_generic_to_shared(&sm.c[0][c_row][c_col]);
    auto fetch = [&](int j) {
        const T *src = cache + (size_t)(beg + j * kLatKeys + c_row) * R + c_col;
        const uint32_t dst = c_dst + (j & 1) * (uint32_t)sizeof(sm.c[0]);
        const int left = end - beg - j * kLatKeys - c_row;
#pragma unroll
        for (int i = 0; i < kLatKeys / RC; i++) {
            const bool in = i * RC < left;
            copy16_at(dst + i * RC * Sm::LD * (uint32_t)sizeof(T), in ? src + (size_t)i * RC * R : cache, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (tiles > 0) fetch(0);
    const int mt = warp % MT, part = warp / MT;
    uint32_t qa[KS][4];  // queries of 16 heads, RP columns
    {
        const int r0 = 16 * mt + gq;
        const T *q = reinterpret_cast<const T *>(p.q) + slot0 * R + part * RP + 2 * t4;
#pragma unroll
        for (int ks = 0; ks < KS; ks++)
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const int r = r0 + 8 * (x & 1);
                qa[ks][x] = r < heads ? *reinterpret_cast<const uint32_t *>(q + (size_t)r * R + 16 * ks + 8 * (x >> 1)) : 0u;
            }
        if (threadIdx.x < HB) sm.m[threadIdx.x] = -INFINITY, sm.l[threadIdx.x] = 0.f;
    }
    float o[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < NT; j++) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
    const int c0 = warp * (R / WARPS);
    const uint32_t k_addr = (uint32_t)__cvta_generic_to_shared(&sm.c[0][(lane & 7) + 8 * (lane >> 4)][part * RP + 8 * ((lane >> 3) & 1)]);
    const uint32_t v_addr = (uint32_t)__cvta_generic_to_shared(&sm.c[0][lane & 15][c0 + 8 * (lane >> 4)]);
    const uint32_t p_addr = (uint32_t)__cvta_generic_to_shared(&sm.p[lane & 15][8 * (lane >> 4)]);
    constexpr uint32_t kRow = Sm::LD * sizeof(T), kPRow = Sm::LP * sizeof(T);

    for (int j = 0; j < tiles; j++) {
        const int key0 = beg + j * kLatKeys;
        const uint32_t buf = (j & 1) * (uint32_t)sizeof(sm.c[0]);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // tile j is there, tile j - 1 has been read by all
        if (j + 1 < tiles) fetch(j + 1);
        // ---- scores: 16 heads x 64 keys over RP columns ----
        {
            float sc[kLatKeys / 8][4];
#pragma unroll
            for (int n = 0; n < kLatKeys / 8; n++) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ks++)
#pragma unroll
                for (int n = 0; n < kLatKeys / 16; n++) {
                    uint32_t kb[4];  // 16 keys: (first 8, k low), (first 8, k high), (last 8, ..)
                    ldsm4_at(kb, k_addr + buf + n * 16 * kRow + ks * 32);
                    mma_kv<T>(sc[2 * n], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[0], kb[1]);
                    mma_kv<T>(sc[2 * n + 1], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], kb[2], kb[3]);
                }
#pragma unroll
            for (int n = 0; n < kLatKeys / 8; n++) {
                *reinterpret_cast<float2 *>(&sm.s[part][16 * mt + gq][8 * n + 2 * t4]) = make_float2(sc[n][0], sc[n][1]);
                *reinterpret_cast<float2 *>(&sm.s[part][16 * mt + gq + 8][8 * n + 2 * t4]) = make_float2(sc[n][2], sc[n][3]);
            }
        }
        __syncthreads();
        // ---- softmax: a warp takes RW heads, two keys per lane ----
        {
            constexpr int RW = HB / WARPS;
            float w0[RW], w1[RW], top[RW], sum[RW], al[RW];
            const int k = 2 * lane;
#pragma unroll
            for (int i = 0; i < RW; i++) {
                const int r = warp * RW + i;
                float x0 = 0.f, x1 = 0.f;
#pragma unroll
                for (int q = 0; q < PARTS; q++) {
                    const float2 v = *reinterpret_cast<const float2 *>(&sm.s[q][r][k]);
                    x0 += v.x, x1 += v.y;
                }
                w0[i] = key0 + k < end ? x0 * p.scale_log2 : -INFINITY, w1[i] = key0 + k + 1 < end ? x1 * p.scale_log2 : -INFINITY;
                top[i] = fmaxf(w0[i], w1[i]);
            }
#pragma unroll
            for (int s = 16; s > 0; s >>= 1)
#pragma unroll
                for (int i = 0; i < RW; i++) top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], s));
#pragma unroll
            for (int i = 0; i < RW; i++) {
                const int r = warp * RW + i;
                const float m_old = sm.m[r], m_new = fmaxf(m_old, top[i]);  // finite: the tile has a key
                w0[i] = lat_exp2(w0[i] - m_new), w1[i] = lat_exp2(w1[i] - m_new), al[i] = lat_exp2(m_old - m_new);
                top[i] = m_new;
                sum[i] = w0[i] + w1[i];
                T two[2] = {from_f32<T>(w0[i]), from_f32<T>(w1[i])};
                *reinterpret_cast<uint32_t *>(&sm.p[r][k]) = *reinterpret_cast<const uint32_t *>(two);
            }
#pragma unroll
            for (int s = 16; s > 0; s >>= 1)
#pragma unroll
                for (int i = 0; i < RW; i++) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], s);
            if (lane == 0) {
#pragma unroll
                for (int i = 0; i < RW; i++) {
                    const int r = warp * RW + i;
                    sm.m[r] = top[i];
                    sm.l[r] = sm.l[r] * al[i] + sum[i];
                    sm.alpha[r] = al[i];
                }
            }
        }
        __syncthreads();
        // ---- weighted sum: R / WARPS columns per warp ----
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
            for (int n = 0; n < NT / 2; n++) ldsm4t_at(vb[n], v_addr + buf + kk * kRow + n * 32);
#pragma unroll
            for (int i = 0; i < MT; i++) {
                uint32_t ph[4];
                ldsm4_at(ph, p_addr + 16 * i * kPRow + kk * 2);
#pragma unroll
                for (int n = 0; n < NT; n++) mma_kv<T>(o[i][n], ph[0], ph[1], ph[2], ph[3], vb[n >> 1][2 * (n & 1)], vb[n >> 1][2 * (n & 1) + 1]);
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
                T *out = reinterpret_cast<T *>(p.out) + (slot0 + r) * R + warp * (R / WARPS) + 2 * t4;
#pragma unroll
                for (int n = 0; n < NT; n++) {
                    T two[2] = {from_f32<T>(o[i][n][2 * x] * inv), from_f32<T>(o[i][n][2 * x + 1] * inv)};
                    *reinterpret_cast<uint32_t *>(out + 8 * n) = *reinterpret_cast<const uint32_t *>(two);
                }
            } else if (tiles > 0) {
                float *out = p.ws_o + ((slot0 + r) * p.splits + split) * R + warp * (R / WARPS) + 2 * t4;
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

// one CTA per (query, head), two neighbouring columns per thread (R / 2 threads); eight splits in flight
template <typename T>
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatParams p, int R) {
    __shared__ float f[kLatMaxSplits];
    __shared__ float total;
    pdl_trigger();
    pdl_wait();
    const size_t slot = blockIdx.x;
    const float *ml = p.ws_ml + slot * p.splits * 2, *o = p.ws_o + slot * p.splits * R + 2 * threadIdx.x;
    float2 v[8];
    auto load = [&](int s0) {
#pragma unroll
        for (int j = 0; j < 8; j++) v[j] = s0 + j < p.splits ? *reinterpret_cast<const float2 *>(o + (size_t)(s0 + j) * R) : make_float2(0.f, 0.f);
    };
    load(0);  // travels while the factors are formed; a split without positions left stale numbers, which meet a factor of 0
    if (threadIdx.x < 32) {
        float m[kLatMaxSplits / 32], mx = -INFINITY, L = 0.f;
#pragma unroll
        for (int j = 0; j < kLatMaxSplits / 32; j++) {
            const int s = threadIdx.x + 32 * j;
            m[j] = s < p.splits ? ml[2 * s] : -INFINITY;
            mx = fmaxf(mx, m[j]);
        }
        mx = warp_max(mx);
#pragma unroll
        for (int j = 0; j < kLatMaxSplits / 32; j++) {
            const int s = threadIdx.x + 32 * j;
            const float w = m[j] == -INFINITY ? 0.f : lat_exp2(m[j] - mx);
            if (s < p.splits) L += w * ml[2 * s + 1];
            f[s] = w;
        }
        L = warp_sum(L);
        if (threadIdx.x == 0) total = L;
    }
    __syncthreads();
    float2 acc = make_float2(0.f, 0.f);
    for (int s0 = 0; s0 < p.splits; s0 += 8) {
        if (s0) load(s0);
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (s0 + j < p.splits && f[s0 + j] != 0.f) acc.x += f[s0 + j] * v[j].x, acc.y += f[s0 + j] * v[j].y;
    }
    const float inv = total > 0.f ? 1.0f / total : 0.f;
    T two[2] = {from_f32<T>(acc.x * inv), from_f32<T>(acc.y * inv)};
    *reinterpret_cast<uint32_t *>(reinterpret_cast<T *>(p.out) + slot * R + 2 * threadIdx.x) = *reinterpret_cast<const uint32_t *>(two);
}

static int lat_splits(int queries, int groups, int rows_bound) {
    int s = 148 / (queries * groups);
    s = std::min(s, rows_bound / (2 * kLatKeys));  // at least four tiles each
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
    kern<<<dim3(l.splits, queries, l.groups), lat_warps(R) * 32, smem, st>>>(l);
    MYNN_LAUNCH_OK("latent_attention_kernel");
    if (l.splits > 1) {
        MYNN_CUDA_OK(launch_dependent(latent_merge_kernel<T>, dim3((unsigned)((long long)queries * l.H)), dim3(R / 2), 0, st, l, R));
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
