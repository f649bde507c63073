// Matrix memory with exponential gates (see MlstmStep in block_ops.cuh): a state of D x E floats per head, decayed and added to at
// every token.
//
// Two forms of one computation:
//   mlstm_scan_kernel    token by token, any sizes and dtypes, also the decode step.  A CTA owns 32 columns of one head's memory, eight
//                        warps deal out its rows, and the tile stays in registers over all the tokens of the call.  The sum vector n, the
//                        running maximum and the denominators are small, so every CTA of a head follows them by itself.
//   mlstm_chunk_kernel   16-bit prompts, 64 tokens at a time on the tensor cores.  With b_t the running sum of the log forget gates
//                        inside the chunk and a_s = i_s - b_s, the recurrence's maximum is m_t = b_t + max(m_0, max_{s <= t} a_s), and
//                        o_t needs  e^(b_t + m_0 - m_t) q_t S_0  +  sum_{s <= t} e^(b_t + a_s - m_t) (q_t.k_s) v_s:  two products of
//                        chunk matrices, and a third one brings S to the chunk's end.  All exponents are at most 0.  The state is carried in
//                        f32 accumulators; S, the weighted scores and the weighted values enter their products as a high 16-bit
//                        part and its rounding remainder (two MMAs), q, k and v as they come from the projection.
// Both write o in f32; it is normed per head, weighted and gated by the last CTA of a head (one token) or by mlstm_out_kernel.
// The state of a head is replaced only by CTAs that own it: the memory by tiles, n and m by the head's last CTA to finish.
#include "attention_internal.cuh"
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

constexpr float kMlstmFloor = 1e-6f;  // added to the denominator
constexpr int kScanWarps = 8, kScanCols = 32, kMlstmMaxDim = 512;

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// the finished row of one head: o over its root mean square, weighted, gated; called by whole warps, `lanes` threads from `id` on
template <typename T>
__device__ __forceinline__ void gated_row(const MlstmStep &p, int row, int h, float inv, int id, int lanes) {
    const float *o = p.o + ((size_t)row * p.H + h) * p.E, *w = p.norm_w + (size_t)h * p.E;
    const T *z = reinterpret_cast<const T *>(p.proj) + (size_t)row * 2 * p.H * (p.D + p.E) + (size_t)p.H * (2 * p.D + p.E) + (size_t)h * p.E;
    T *out = reinterpret_cast<T *>(p.out) + ((size_t)row * p.H + h) * p.E;
    for (int e = id; e < p.E; e += lanes) out[e] = from_f32<T>(__ldcg(o + e) * inv * w[e] * sigmoid_f(to_f32<T>(z[e])));
}

// one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) mlstm_out_kernel(const MlstmStep p) {
    pdl_trigger();
    pdl_wait();
    const int job = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (job >= p.B * p.S * p.H) return;
    const int row = job / p.H, h = job - row * p.H;
    const float *o = p.o + ((size_t)row * p.H + h) * p.E;
    const T *z = reinterpret_cast<const T *>(p.proj) + (size_t)row * 2 * p.H * (p.D + p.E) + (size_t)p.H * (2 * p.D + p.E) + (size_t)h * p.E;
    const bool vec = p.E % 4 == 0 && p.D % 2 == 0 && (((uintptr_t)p.proj | (uintptr_t)p.out) % 8) == 0 && sizeof(T) == 2;
    float ss = 0.f;
    if (vec) {
        for (int e = lane * 4; e < p.E; e += 128) {
            const float4 r = *reinterpret_cast<const float4 *>(o + e);
            ss += r.x * r.x + r.y * r.y + r.z * r.z + r.w * r.w;
        }
    } else {
        for (int e = lane; e < p.E; e += 32) ss += o[e] * o[e];
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.E + p.eps);
    if (!vec) {
        gated_row<T>(p, row, h, inv, lane, 32);
        return;
    }
    const float *w = p.norm_w + (size_t)h * p.E;
    T *out = reinterpret_cast<T *>(p.out) + ((size_t)row * p.H + h) * p.E;
    for (int e = lane * 4; e < p.E; e += 128) {
        const float4 r = *reinterpret_cast<const float4 *>(o + e), g = *reinterpret_cast<const float4 *>(w + e);
        const uint2 zr = *reinterpret_cast<const uint2 *>(z + e);
        const T *ze = reinterpret_cast<const T *>(&zr);
        uint2 res;
        T *re = reinterpret_cast<T *>(&res);
        re[0] = from_f32<T>(r.x * inv * g.x * sigmoid_f(to_f32<T>(ze[0])));
        re[1] = from_f32<T>(r.y * inv * g.y * sigmoid_f(to_f32<T>(ze[1])));
        re[2] = from_f32<T>(r.z * inv * g.z * sigmoid_f(to_f32<T>(ze[2])));
        re[3] = from_f32<T>(r.w * inv * g.w * sigmoid_f(to_f32<T>(ze[3])));
        *reinterpret_cast<uint2 *>(out + e) = res;
    }
}

// Arrival of a CTA of head (b, h) that has read all it needs of the head's n and m and stored its part of o: true in the last one.
__device__ __forceinline__ bool last_of_head(const MlstmStep &p, int pair, int tiles, unsigned *flag) {
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        *flag = atomicAdd(&p.ticket[pair], 1u) == (unsigned)(tiles - 1) ? 1u : 0u;
        if (*flag) p.ticket[pair] = 0u;
    }
    __syncthreads();
    if (!*flag) return false;
    __threadfence();
    return true;
}

// grid (ceil(E / 32), H, B), 256 threads.  Warp w holds rows [w NR, (w + 1) NR) of the memory tile, lane l column l.
template <typename T, int NR>
__global__ void __launch_bounds__(kScanWarps * 32) mlstm_scan_kernel(const MlstmStep p) {
    constexpr int DP = kScanWarps * NR;  // rows with padding
    __shared__ __align__(16) float sm_q[2][DP], sm_k[2][DP];
    __shared__ float sm_num[2][kScanWarps][kScanCols], sm_den[2][kScanWarps];
    __shared__ float sm_ss[kScanWarps];
    __shared__ unsigned flag;
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, b = blockIdx.z, pair = b * p.H + h, tiles = gridDim.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, col = blockIdx.x * kScanCols + lane;
    const bool fresh = *p.past == 0, in = col < p.E;
    const int C = 2 * p.H * (p.D + p.E);
    float *mem = p.mem + (size_t)pair * p.D * p.E + col;
    float S[NR];
    constexpr int NN = (NR + 31) / 32;  // elements of n a lane keeps: rows warp * NR + lane + 32 j
    float n[NN];
#pragma unroll
    for (int r = 0; r < NR; r++) {
        const int d = warp * NR + r;
        S[r] = !fresh && in && d < p.D ? mem[(size_t)d * p.E] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < NN; j++) {
        const int r = lane + 32 * j, d = warp * NR + r;
        n[j] = !fresh && r < NR && d < p.D ? p.sum[(size_t)pair * p.D + d] : 0.f;
    }
    float m = fresh ? 0.f : p.top[pair];
    const float q_scale = 1.0f / sqrtf((float)p.D), bias_i = p.gate_bias[h], bias_f = p.gate_bias[p.H + h];
    constexpr int PT = (DP + 255) / 256;  // elements of q and of k a thread stages
    auto stage = [&](int t) {
        const T *row = reinterpret_cast<const T *>(p.proj) + (size_t)(b * p.S + t) * C + (size_t)h * p.D;
#pragma unroll
        for (int j = 0; j < PT; j++) {
            const int d = threadIdx.x + 256 * j;
            if (d < DP) {
                sm_q[t & 1][d] = d < p.D ? to_f32<T>(row[d]) * q_scale : 0.f;
                sm_k[t & 1][d] = d < p.D ? to_f32<T>(row[(size_t)p.H * p.D + d]) : 0.f;
            }
        }
    };
    stage(0);
    __syncthreads();
    for (int t = 0; t < p.S; t++) {
        const size_t row = (size_t)b * p.S + t;
        const float v = in ? to_f32<T>(reinterpret_cast<const T *>(p.proj)[row * C + (size_t)2 * p.H * p.D + (size_t)h * p.E + col]) : 0.f;
        const float gi = capped(p.gates[row * 2 * p.H + h] + bias_i, p.cap), gf = log_sigmoid(capped(p.gates[row * 2 * p.H + p.H + h] + bias_f, p.cap));
        const float m_new = fmaxf(gf + m, gi), keep = expf(gf + m - m_new), take = expf(gi - m_new);
        m = m_new;
        const float *q = sm_q[t & 1] + warp * NR, *k = sm_k[t & 1] + warp * NR;
        float num = 0.f, den = 0.f;
        const float tv = take * v;
#pragma unroll
        for (int r = 0; r < NR; r += 4) {
            const float4 kk = *reinterpret_cast<const float4 *>(k + r), qq = *reinterpret_cast<const float4 *>(q + r);
            S[r] = keep * S[r] + kk.x * tv, num += S[r] * qq.x;
            S[r + 1] = keep * S[r + 1] + kk.y * tv, num += S[r + 1] * qq.y;
            S[r + 2] = keep * S[r + 2] + kk.z * tv, num += S[r + 2] * qq.z;
            S[r + 3] = keep * S[r + 3] + kk.w * tv, num += S[r + 3] * qq.w;
        }
#pragma unroll
        for (int j = 0; j < NN; j++) {
            const int r = lane + 32 * j;
            if (r < NR) {
                n[j] = keep * n[j] + take * k[r];
                den += n[j] * q[r];
            }
        }
        den = warp_sum(den);
        sm_num[t & 1][warp][lane] = num;
        if (lane == 0) sm_den[t & 1][warp] = den;
        if (t + 1 < p.S) stage(t + 1);
        __syncthreads();
        if (warp == 0 && in) {
            float a = 0.f, d = 0.f;
#pragma unroll
            for (int w = 0; w < kScanWarps; w++) a += sm_num[t & 1][w][lane], d += sm_den[t & 1][w];
            p.o[(row * p.H + h) * p.E + col] = a / (fmaxf(fabsf(d), expf(-m)) + kMlstmFloor);
        }
    }
#pragma unroll
    for (int r = 0; r < NR; r++) {
        const int d = warp * NR + r;
        if (in && d < p.D) mem[(size_t)d * p.E] = S[r];
    }
    if (!last_of_head(p, pair, tiles, &flag)) return;
#pragma unroll
    for (int j = 0; j < NN; j++) {
        const int r = lane + 32 * j, d = warp * NR + r;
        if (r < NR && d < p.D) p.sum[(size_t)pair * p.D + d] = n[j];
    }
    if (threadIdx.x == 0) p.top[pair] = m;
    if (p.S == 1) {
        const float *o = p.o + (size_t)pair * p.E;
        float ss = 0.f;
        for (int e = threadIdx.x; e < p.E; e += blockDim.x) {
            const float x = __ldcg(o + e);
            ss += x * x;
        }
        ss = warp_sum(ss);
        if (lane == 0) sm_ss[warp] = ss;
        __syncthreads();
        float total = 0.f;
#pragma unroll
        for (int w = 0; w < kScanWarps; w++) total += sm_ss[w];
        gated_row<T>(p, b, h, 1.0f / sqrtf(total / (float)p.E + p.eps), threadIdx.x, blockDim.x);
    }
}

// ---- chunkwise -------------------------------------------------------------------------------------------------------
constexpr int kChunk = 64, kChunkCols = 32, kChunkThreads = 256;

template <typename T>
__device__ __forceinline__ void split_one(float x, T &hi, T &lo) {
    hi = from_f32<T>(x);
    lo = from_f32<T>(x - to_f32<T>(hi));
}

template <typename T, int KD>
struct ChunkSmem {
    static constexpr int LD = KD + 8, LV = kChunkCols + 8, LP = kChunk + 8;  // row lengths: 16 bytes past a multiple of 128 (of 64)
    T q[2][kChunk][LD], k[2][kChunk][LD], v[2][kChunk][LV];
    T s_hi[KD][LV], s_lo[KD][LV];
    T p_hi[kChunk][LP], p_lo[kChunk][LP];
    T w_hi[kChunk][LV], w_lo[kChunk][LV];  // values times their weight at the chunk's end
    float n[KD];
    float r[2][kChunk], a[2][kChunk], m[2][kChunk], end[2][kChunk];  // b_t - m_t, a_s, m_t, weight of token s at the chunk's end
    float carry[2][2];                                              // factor of the old state at the chunk's end; m_0
    float qn[kChunk], part[2][kChunk];                              // q.n_0; row sums of the weighted scores by column half
    unsigned flag;
};

// grid (ceil(E / 32), H, B).  KD: D padded to 64, 128 or 256.
template <typename T, int KD>
__global__ void __launch_bounds__(kChunkThreads, 1) mlstm_chunk_kernel(const MlstmStep p) {
    extern __shared__ __align__(16) uint8_t chunk_smem[];
    using Sm = ChunkSmem<T, KD>;
    Sm &sm = *reinterpret_cast<Sm *>(chunk_smem);
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, b = blockIdx.z, pair = b * p.H + h, e0 = blockIdx.x * kChunkCols;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t4 = lane & 3;
    const bool fresh = *p.past == 0;
    const size_t C = (size_t)2 * p.H * (p.D + p.E);
    const T *base = reinterpret_cast<const T *>(p.proj) + (size_t)b * p.S * C;
    const float q_scale = 1.0f / sqrtf((float)p.D);
    const int n_chunks = (p.S + kChunk - 1) / kChunk;

    auto fetch = [&](int c) {
        const int buf = c & 1, t0 = c * kChunk;
        constexpr int PQ = KD / 8;
        for (int i = threadIdx.x; i < kChunk * PQ; i += kChunkThreads) {
            const int t = i / PQ, d = (i - t * PQ) * 8;
            const bool in = t0 + t < p.S && d < p.D;
            const T *src = base + (size_t)(in ? t0 + t : 0) * C + (size_t)h * p.D + (in ? d : 0);
            copy16(&sm.q[buf][t][d], src, in);
            copy16(&sm.k[buf][t][d], src + (size_t)p.H * p.D, in);
        }
        for (int i = threadIdx.x; i < kChunk * (kChunkCols / 8); i += kChunkThreads) {
            const int t = i / (kChunkCols / 8), e = (i % (kChunkCols / 8)) * 8;
            const bool in = t0 + t < p.S && e0 + e < p.E;
            copy16(&sm.v[buf][t][e], base + (size_t)(in ? t0 + t : 0) * C + (size_t)2 * p.H * p.D + (size_t)h * p.E + (in ? e0 + e : 0), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // gates of chunk c by one warp, two neighbouring tokens per lane; m0: the maximum at the chunk's start.  Returns m at its end.
    auto gates = [&](int c, float m0) {
        const int buf = c & 1;
        float gi[2], gf[2];
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int t = c * kChunk + 2 * lane + j;
            gi[j] = -INFINITY, gf[j] = 0.f;
            if (t < p.S) {
                const float *g = p.gates + ((size_t)b * p.S + t) * 2 * p.H + h;
                gi[j] = capped(g[0] + p.gate_bias[h], p.cap);
                gf[j] = log_sigmoid(capped(g[p.H] + p.gate_bias[p.H + h], p.cap));
            }
        }
        float sum = gf[0] + gf[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += u;
        }
        const float b1 = sum, b0 = sum - gf[1], total = __shfl_sync(0xffffffffu, sum, 31);
        const float a0 = gi[0] - b0, a1 = gi[1] - b1;
        float mx = fmaxf(a0, a1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, mx, o);
            if (lane >= o) mx = fmaxf(mx, u);
        }
        float before = __shfl_up_sync(0xffffffffu, mx, 1);
        if (lane == 0) before = -INFINITY;
        const float top0 = fmaxf(m0, fmaxf(before, a0)), top1 = fmaxf(m0, mx);  // m_t - b_t
        const float end_top = __shfl_sync(0xffffffffu, top1, 31);
        sm.r[buf][2 * lane] = -top0, sm.r[buf][2 * lane + 1] = -top1;
        sm.a[buf][2 * lane] = a0, sm.a[buf][2 * lane + 1] = a1;
        sm.m[buf][2 * lane] = b0 + top0, sm.m[buf][2 * lane + 1] = b1 + top1;
        sm.end[buf][2 * lane] = expf(a0 - end_top), sm.end[buf][2 * lane + 1] = expf(a1 - end_top);
        if (lane == 0) sm.carry[buf][0] = expf(m0 - end_top), sm.carry[buf][1] = m0;
        return total + end_top;
    };

    // the memory tile [KD, 32] in accumulators: warp w holds ST row tiles of 16 by SN column tiles of 8
    constexpr int ST = KD >= 128 ? KD / 128 : 1, SN = KD >= 128 ? 4 : 2;
    const int s_row = KD >= 128 ? warp * 16 * ST : (warp & 3) * 16, s_col = KD >= 128 ? 0 : (warp >> 2) * 16;
    float S[ST][SN][4];
    float *mem = p.mem + (size_t)pair * p.D * p.E;
#pragma unroll
    for (int i = 0; i < ST; i++)
#pragma unroll
        for (int j = 0; j < SN; j++)
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const int d = s_row + 16 * i + gq + 8 * (x >> 1), e = e0 + s_col + 8 * j + 2 * t4 + (x & 1);
                S[i][j][x] = !fresh && d < p.D && e < p.E ? mem[(size_t)d * p.E + e] : 0.f;
            }
    auto publish = [&]() {  // the tile as high part and remainder
#pragma unroll
        for (int i = 0; i < ST; i++)
#pragma unroll
            for (int j = 0; j < SN; j++)
#pragma unroll
                for (int x = 0; x < 2; x++) {
                    uint32_t hi, lo;
                    split_pack<T>(S[i][j][2 * x], S[i][j][2 * x + 1], hi, lo);
                    const int d = s_row + 16 * i + gq + 8 * x, e = s_col + 8 * j + 2 * t4;
                    *reinterpret_cast<uint32_t *>(&sm.s_hi[d][e]) = hi;
                    *reinterpret_cast<uint32_t *>(&sm.s_lo[d][e]) = lo;
                }
    };
    fetch(0);
    float m_carry = fresh ? 0.f : p.top[pair];
    if (warp == 0) m_carry = gates(0, m_carry);  // warp 0 follows the maximum from here on
    for (int d = threadIdx.x; d < KD; d += kChunkThreads) sm.n[d] = !fresh && d < p.D ? p.sum[(size_t)pair * p.D + d] : 0.f;
    publish();

    const int mt = warp & 3, nh = warp >> 2;  // 16 query tokens; a half of the key tokens, then of the value columns
    for (int c = 0; c < n_chunks; c++) {
        const int buf = c & 1, t0 = c * kChunk;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // chunk c, its gates, S and n are in shared memory; chunk c - 1 has been read by all
        if (c + 1 < n_chunks) fetch(c + 1);

        // ---- scores of 16 x 32 tokens, and q S_0 for 16 tokens x 16 columns ----
        float sc[4][4], acc[2][4];
#pragma unroll
        for (int j = 0; j < 4; j++) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
        for (int j = 0; j < 2; j++) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        const bool scores = 16 * mt + 15 >= 32 * nh;  // some pair s <= t
#pragma unroll 4
        for (int kk = 0; kk < KD; kk += 16) {
            uint32_t qa[4], bh[4], bl[4];
            ldsm4(qa, &sm.q[buf][16 * mt + (lane & 15)][kk + 8 * (lane >> 4)]);
            // [d][e] rows read transposed: two k halves of two column tiles
            ldsm4t(bh, &sm.s_hi[kk + (lane & 15)][16 * nh + 8 * (lane >> 4)]);
            ldsm4t(bl, &sm.s_lo[kk + (lane & 15)][16 * nh + 8 * (lane >> 4)]);
#pragma unroll
            for (int j = 0; j < 2; j++) {
                mma_kv<T>(acc[j], qa[0], qa[1], qa[2], qa[3], bh[2 * j], bh[2 * j + 1]);
                mma_kv<T>(acc[j], qa[0], qa[1], qa[2], qa[3], bl[2 * j], bl[2 * j + 1]);
            }
            if (scores) {
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    uint32_t kb[4];  // key tokens 32 nh + 16 j .. + 15: (first 8, k low), (first 8, k high), (last 8, ..)
                    ldsm4(kb, &sm.k[buf][32 * nh + 16 * j + (lane & 7) + 8 * (lane >> 4)][kk + 8 * ((lane >> 3) & 1)]);
                    mma_kv<T>(sc[2 * j], qa[0], qa[1], qa[2], qa[3], kb[0], kb[1]);
                    mma_kv<T>(sc[2 * j + 1], qa[0], qa[1], qa[2], qa[3], kb[2], kb[3]);
                }
            }
        }
        // ---- weights, row sums, high and low parts ----
        const int tr[2] = {16 * mt + gq, 16 * mt + gq + 8};
        const float rr[2] = {sm.r[buf][tr[0]], sm.r[buf][tr[1]]};
        float rs[2] = {0.f, 0.f};
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int s = 32 * nh + 8 * j + 2 * t4;
            const float a0 = sm.a[buf][s], a1 = sm.a[buf][s + 1];
#pragma unroll
            for (int x = 0; x < 2; x++) {
                const float w0 = s <= tr[x] ? sc[j][2 * x] * q_scale * __expf(rr[x] + a0) : 0.f;
                const float w1 = s + 1 <= tr[x] ? sc[j][2 * x + 1] * q_scale * __expf(rr[x] + a1) : 0.f;
                rs[x] += w0 + w1;
                uint32_t hi, lo;
                split_pack<T>(w0, w1, hi, lo);
                *reinterpret_cast<uint32_t *>(&sm.p_hi[tr[x]][s]) = hi;
                *reinterpret_cast<uint32_t *>(&sm.p_lo[tr[x]][s]) = lo;
            }
        }
#pragma unroll
        for (int x = 0; x < 2; x++) {
            rs[x] += __shfl_xor_sync(0xffffffffu, rs[x], 1);
            rs[x] += __shfl_xor_sync(0xffffffffu, rs[x], 2);
            if (t4 == 0) sm.part[nh][tr[x]] = rs[x];
        }
        // ---- q.n_0 of eight tokens per warp; values times their weight at the chunk's end ----
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int t = 8 * warp + i;
            float dot = 0.f;
#pragma unroll
            for (int d = 2 * lane; d < KD; d += 64) {
                const uint32_t two = *reinterpret_cast<const uint32_t *>(&sm.q[buf][t][d]);
                const T *e = reinterpret_cast<const T *>(&two);
                dot += to_f32<T>(e[0]) * sm.n[d] + to_f32<T>(e[1]) * sm.n[d + 1];
            }
            dot = warp_sum(dot);
            if (lane == 0) sm.qn[t] = dot;
        }
        for (int i = threadIdx.x; i < kChunk * kChunkCols; i += kChunkThreads) {
            const int t = i / kChunkCols, e = i % kChunkCols;
            split_one<T>(to_f32<T>(sm.v[buf][t][e]) * sm.end[buf][t], sm.w_hi[t][e], sm.w_lo[t][e]);
        }
        const float m0 = sm.carry[buf][1], keep = sm.carry[buf][0];
        // what the old state contributes to these tokens' rows
        const float f0 = __expf(rr[0] + m0) * q_scale, f1 = __expf(rr[1] + m0) * q_scale;
#pragma unroll
        for (int j = 0; j < 2; j++) acc[j][0] *= f0, acc[j][1] *= f0, acc[j][2] *= f1, acc[j][3] *= f1;
        __syncthreads();  // scores, weighted values and q.n_0 are there; S and n have been read

        // ---- + weighted scores times values ----
        for (int kk = 0; kk <= 16 * mt; kk += 16) {  // later key tokens weigh nothing
            uint32_t ph[4], pl[4], vb[4];
            ldsm4(ph, &sm.p_hi[16 * mt + (lane & 15)][kk + 8 * (lane >> 4)]);
            ldsm4(pl, &sm.p_lo[16 * mt + (lane & 15)][kk + 8 * (lane >> 4)]);
            ldsm4t(vb, &sm.v[buf][kk + (lane & 15)][16 * nh + 8 * (lane >> 4)]);
#pragma unroll
            for (int j = 0; j < 2; j++) {
                mma_kv<T>(acc[j], ph[0], ph[1], ph[2], ph[3], vb[2 * j], vb[2 * j + 1]);
                mma_kv<T>(acc[j], pl[0], pl[1], pl[2], pl[3], vb[2 * j], vb[2 * j + 1]);
            }
        }
#pragma unroll
        for (int x = 0; x < 2; x++) {
            const int t = t0 + tr[x];
            if (t >= p.S) continue;
            const float den = (x ? f1 : f0) * sm.qn[tr[x]] + sm.part[0][tr[x]] + sm.part[1][tr[x]];
            const float inv = 1.0f / (fmaxf(fabsf(den), expf(-sm.m[buf][tr[x]])) + kMlstmFloor);
            float *o = p.o + (((size_t)b * p.S + t) * p.H + h) * p.E;
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int e = e0 + 16 * nh + 8 * j + 2 * t4;  // E is a multiple of 8: both or none
                if (e < p.E) *reinterpret_cast<float2 *>(o + e) = make_float2(acc[j][2 * x] * inv, acc[j][2 * x + 1] * inv);
            }
        }
        // ---- state at the chunk's end ----
#pragma unroll
        for (int i = 0; i < ST; i++)
#pragma unroll
            for (int j = 0; j < SN; j++)
#pragma unroll
                for (int x = 0; x < 4; x++) S[i][j][x] *= keep;
#pragma unroll
        for (int kk = 0; kk < kChunk; kk += 16) {
            uint32_t wh[SN / 2][4], wl[SN / 2][4];
#pragma unroll
            for (int j = 0; j < SN / 2; j++) {
                ldsm4t(wh[j], &sm.w_hi[kk + (lane & 15)][s_col + 16 * j + 8 * (lane >> 4)]);
                ldsm4t(wl[j], &sm.w_lo[kk + (lane & 15)][s_col + 16 * j + 8 * (lane >> 4)]);
            }
#pragma unroll
            for (int i = 0; i < ST; i++) {
                uint32_t ka[4];  // k transposed: (rows 0-7, tokens 0-7), (rows 8-15, tokens 0-7), (rows 0-7, tokens 8-15), ..
                ldsm4t(ka, &sm.k[buf][kk + (lane & 7) + 8 * (lane >> 4)][s_row + 16 * i + 8 * ((lane >> 3) & 1)]);
#pragma unroll
                for (int j = 0; j < SN / 2; j++)
#pragma unroll
                    for (int x = 0; x < 2; x++) {
                        mma_kv<T>(S[i][2 * j + x], ka[0], ka[1], ka[2], ka[3], wh[j][2 * x], wh[j][2 * x + 1]);
                        mma_kv<T>(S[i][2 * j + x], ka[0], ka[1], ka[2], ka[3], wl[j][2 * x], wl[j][2 * x + 1]);
                    }
            }
        }
        publish();
        for (int d = threadIdx.x; d < KD; d += kChunkThreads) {
            float x = keep * sm.n[d];
#pragma unroll 8
            for (int t = 0; t < kChunk; t++) x += sm.end[buf][t] * to_f32<T>(sm.k[buf][t][d]);
            sm.n[d] = x;
        }
        if (warp == 0 && c + 1 < n_chunks) m_carry = gates(c + 1, m_carry);
    }
#pragma unroll
    for (int i = 0; i < ST; i++)
#pragma unroll
        for (int j = 0; j < SN; j++)
#pragma unroll
            for (int x = 0; x < 2; x++) {
                const int d = s_row + 16 * i + gq + 8 * x, e = e0 + s_col + 8 * j + 2 * t4;
                if (d < p.D && e < p.E) *reinterpret_cast<float2 *>(mem + (size_t)d * p.E + e) = make_float2(S[i][j][2 * x], S[i][j][2 * x + 1]);
            }
    if (!last_of_head(p, pair, gridDim.x, &sm.flag)) return;
    for (int d = threadIdx.x; d < p.D; d += kChunkThreads) p.sum[(size_t)pair * p.D + d] = sm.n[d];
    if (threadIdx.x == 0) p.top[pair] = m_carry;
}

bool mlstm_chunkwise_supported(int dtype, const MlstmStep &p) {
    const uintptr_t a = (uintptr_t)p.proj | (uintptr_t)p.o | (uintptr_t)p.mem;
    return dtype != MYNN_F32 && p.D <= 256 && p.D % 8 == 0 && p.E % 8 == 0 && a % 16 == 0;
}

template <typename T>
static int run_out(cudaStream_t st, const MlstmStep &p) {
    mlstm_out_kernel<T><<<(unsigned)(((long long)p.B * p.S * p.H + 7) / 8), 256, 0, st>>>(p);
    MYNN_LAUNCH_OK("mlstm_out_kernel");
    return MYNN_OK;
}

template <typename T>
static int run_scan(cudaStream_t st, const MlstmStep &p) {
    const dim3 grid((p.E + kScanCols - 1) / kScanCols, p.H, p.B);
    if (p.D <= 64) mlstm_scan_kernel<T, 8><<<grid, 256, 0, st>>>(p);
    else if (p.D <= 128) mlstm_scan_kernel<T, 16><<<grid, 256, 0, st>>>(p);
    else if (p.D <= 256) mlstm_scan_kernel<T, 32><<<grid, 256, 0, st>>>(p);
    else mlstm_scan_kernel<T, 64><<<grid, 256, 0, st>>>(p);
    MYNN_LAUNCH_OK("mlstm_scan_kernel");
    return p.S == 1 ? MYNN_OK : run_out<T>(st, p);
}

template <typename T, int KD>
static int run_chunk(cudaStream_t st, const MlstmStep &p) {
    constexpr size_t smem = sizeof(ChunkSmem<T, KD>);
    static_assert(smem <= 227 * 1024, "shared memory of a CTA");
    auto kern = mlstm_chunk_kernel<T, KD>;
    static bool attr_set = false;
    if (!attr_set) {
        MYNN_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set = true;
    }
    kern<<<dim3((p.E + kChunkCols - 1) / kChunkCols, p.H, p.B), kChunkThreads, smem, st>>>(p);
    MYNN_LAUNCH_OK("mlstm_chunk_kernel");
    return run_out<T>(st, p);
}

template <typename T>
static int run_chunk_any(cudaStream_t st, const MlstmStep &p) {
    if (p.D <= 64) return run_chunk<T, 64>(st, p);
    if (p.D <= 128) return run_chunk<T, 128>(st, p);
    return run_chunk<T, 256>(st, p);
}

int launch_mlstm(cudaStream_t st, int dtype, const MlstmStep &p) {
    if (p.B <= 0 || p.S <= 0 || p.H <= 0 || p.D <= 0 || p.E <= 0 || !(p.cap > 0.f)) return fail(MYNN_E_ARG, "mlstm: bad shape");
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "mlstm: bad dtype %d", dtype);
    if (p.D > kMlstmMaxDim || p.H > 65535 || p.B > 65535) return fail(MYNN_E_UNSUPPORTED, "mlstm: %d heads of %d", p.H, p.D);
    if (!p.proj || !p.gates || !p.gate_bias || !p.norm_w || !p.mem || !p.sum || !p.top || !p.o || !p.ticket || !p.out || !p.past) return fail(MYNN_E_ARG, "mlstm: null pointer");
    const bool can = mlstm_chunkwise_supported(dtype, p);
    if (p.form == 2 && !can) return fail(MYNN_E_UNSUPPORTED, "mlstm: not a shape of the chunkwise kernel");
    if (p.form == 2 || (p.form == 0 && can && p.S > 16)) return dtype == MYNN_BF16 ? run_chunk_any<__nv_bfloat16>(st, p) : run_chunk_any<__half>(st, p);
    MYNN_DISPATCH_DTYPE(dtype, T, { return run_scan<T>(st, p); });
    return MYNN_OK;
}

}  // namespace mynn

using namespace mynn;

extern "C" int mynn_b200_mlstm(void *stream, void *out, float *mem, float *sum, float *top, const void *proj, const float *gates, const float *gate_bias,
                               const float *norm_weight, float cap, float eps, int B, int S, int H, int D, int E, const int32_t *past_dev, float *scratch,
                               uint32_t *tickets, int dtype, int form) {
    MlstmStep p;
    p.proj = proj;
    p.gates = gates;
    p.gate_bias = gate_bias;
    p.norm_w = norm_weight;
    p.cap = cap, p.eps = eps;
    p.mem = mem, p.sum = sum, p.top = top;
    p.o = scratch;
    p.ticket = tickets;
    p.out = out;
    p.B = B, p.S = S, p.H = H, p.D = D, p.E = E;
    p.past = past_dev;
    p.form = form;
    return launch_mlstm((cudaStream_t)stream, dtype, p);
}
