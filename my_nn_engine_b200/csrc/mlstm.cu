// Matrix memory with exponential gates (see MlstmStep in block_ops.cuh): a state of D x E floats per head, decayed and added to at
// every token.
//
// Two forms of one computation:
//   mlstm_scan_kernel    token by token, any sizes and dtypes, also the decode step.  A CTA owns 32 columns of one head's memory, eight
//                        warps deal out its rows, and the tile stays in registers over all the tokens of the call.  The sum vector n, the
//                        running maximum and the denominators are small, so every CTA of a head follows them by itself.
//   mlstm_chunk_kernel   16-bit prompts (mlstm_tc.cu has it with its large products on tcgen05, for large heads), 64 tokens at a time on the tensor cores.  With b_t the running sum of the log forget gates
//                        inside the chunk, a_s = i_s - b_s and c_t = max_{s <= t} a_s, the recurrence's maximum is m_t = b_t + max(m_0, c_t),
//                        and o_t needs  e^(b_t + m_0 - m_t) q_t S_0  +  sum_{s <= t} e^(b_t + a_s - m_t) (q_t.k_s) v_s:  two products of
//                        chunk matrices, and a third one brings S to the chunk's end.  All exponents are at most 0.  A warp carries 16
//                        columns of S, transposed, in f32 accumulators, whose layout is that of the first operand of q S_0: the
//                        state never passes through shared memory.  S, the weighted scores and the weighted values enter their products
//                        as a high 16-bit part and its rounding remainder (two MMAs), q, k and v as they come from the projection.
// Few heads leave SMs idle, so a prompt is then cut into segments that run side by side: the kernel without its output half leaves what
// every segment adds to the memory, and the second pass starts every segment from the sum of what came before it.
// Both forms write o in f32; it is normed per head, weighted and gated by the last CTA of a head (one token) or by mlstm_out_kernel.
// The state of a head is replaced only by CTAs that own it: the memory by tiles, n and m by the head's last CTA to finish.
#include "mlstm_internal.cuh"

namespace mynn {

constexpr int kScanWarps = 8, kScanCols = 32, kMlstmMaxDim = 512;

// the finished row of one head: o over its root mean square, weighted, gated; called by whole warps, `lanes` threads from `id` on
template <typename T>
__device__ __forceinline__ void gated_row(const MlstmStep &p, int row, int h, float inv, int id, int lanes) {
    const float *o = p.workspace + ((size_t)row * p.H + h) * p.E, *w = p.norm_w + (size_t)h * p.E;
    const T *z = reinterpret_cast<const T *>(p.proj) + (size_t)row * 2 * p.H * (p.D + p.E) + (size_t)p.H * (2 * p.D + p.E) + (size_t)h * p.E;
    T *out = reinterpret_cast<T *>(p.out) + ((size_t)row * p.H + h) * p.E;
    for (int e = id; e < p.E; e += lanes) out[e] = from_f32<T>(__ldcg(o + e) * inv * w[e] * sigmoid_f(to_f32<T>(z[e])));
}

constexpr int kChunkWarps = 8, kChunkThreads = kChunkWarps * 32;
static_assert(kChunkCols == 16 * kChunkWarps, "16 columns of the memory per warp");
constexpr int kMaxSegments = 16;  // a segment reads what all before it left

// one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) mlstm_out_kernel(const MlstmStep p) {
    pdl_trigger();
    pdl_wait();
    const int job = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (job >= p.B * p.S * p.H) return;
    const int row = job / p.H, h = job - row * p.H;
    const float *o = p.workspace + ((size_t)row * p.H + h) * p.E;
    const T *z = reinterpret_cast<const T *>(p.proj) + (size_t)row * 2 * p.H * (p.D + p.E) + (size_t)p.H * (2 * p.D + p.E) + (size_t)h * p.E;
    if (p.E % 4 == 0 && p.E <= 512 && p.D % 2 == 0 && (((uintptr_t)p.proj | (uintptr_t)p.out) % 8) == 0 && sizeof(T) == 2) {
        // every load is on its way before the first sum
        float4 r[4], g[4];
        uint2 zr[4];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int e = 4 * lane + 128 * j;
            r[j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (e < p.E) {
                r[j] = *reinterpret_cast<const float4 *>(o + e);
                zr[j] = *reinterpret_cast<const uint2 *>(z + e);
                g[j] = *reinterpret_cast<const float4 *>(p.norm_w + (size_t)h * p.E + e);
            }
        }
#pragma unroll
        for (int j = 0; j < 4; j++) ss += r[j].x * r[j].x + r[j].y * r[j].y + r[j].z * r[j].z + r[j].w * r[j].w;
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.E + p.eps);
        T *out = reinterpret_cast<T *>(p.out) + ((size_t)row * p.H + h) * p.E;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int e = 4 * lane + 128 * j;
            if (e < p.E) {
                const T *ze = reinterpret_cast<const T *>(&zr[j]);
                uint2 res;
                T *re = reinterpret_cast<T *>(&res);
                re[0] = from_f32<T>(r[j].x * inv * g[j].x * fast_sigmoid(to_f32<T>(ze[0])));
                re[1] = from_f32<T>(r[j].y * inv * g[j].y * fast_sigmoid(to_f32<T>(ze[1])));
                re[2] = from_f32<T>(r[j].z * inv * g[j].z * fast_sigmoid(to_f32<T>(ze[2])));
                re[3] = from_f32<T>(r[j].w * inv * g[j].w * fast_sigmoid(to_f32<T>(ze[3])));
                *reinterpret_cast<uint2 *>(out + e) = res;
            }
        }
        return;
    }
    float ss = 0.f;
    for (int e = lane; e < p.E; e += 32) ss += o[e] * o[e];
    gated_row<T>(p, row, h, 1.0f / sqrtf(warp_sum(ss) / (float)p.E + p.eps), lane, 32);
}

// grid (ceil(E / 32), H, B), 256 threads.  Warp w holds rows [w NR, (w + 1) NR) of the memory tile, lane l column l.  ONE: a single token, which
// is all about reading and writing the memory: four CTAs per SM keep enough of it on its way.
template <typename T, int NR, bool ONE>
__global__ void __launch_bounds__(kScanWarps * 32, ONE && NR <= 32 ? 4 : 1) mlstm_scan_kernel(const MlstmStep p) {
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
    for (int t = 0; t < p.S; t++) {  // also with ONE a loop: all of the memory's reads are then on their way in front of it
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
        if (!ONE && t + 1 < p.S) stage(t + 1);
        __syncthreads();
        if (warp == 0 && in) {
            float a = 0.f, d = 0.f;
#pragma unroll
            for (int w = 0; w < kScanWarps; w++) a += sm_num[t & 1][w][lane], d += sm_den[t & 1][w];
            p.workspace[(row * p.H + h) * p.E + col] = a / (fmaxf(fabsf(d), expf(-m)) + kMlstmFloor);
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
    if constexpr (ONE) {
        const float *o = p.workspace + (size_t)pair * p.E;
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
static void bind_chunk_ws(ChunkWs &w, const MlstmStep &p, float *base, size_t *bytes) {
    w.chunks = (p.S + kChunk - 1) / kChunk;
    const int tiles = (p.E + kChunkCols - 1) / kChunkCols;
    const long long ctas = (long long)p.B * p.H * tiles;
    int g = (int)(148 / ctas);
    g = g < 1 ? 1 : g > kMaxSegments ? kMaxSegments : g;
    w.per = (w.chunks + g - 1) / g;
    if (w.per < 2) w.per = 2;  // a segment of one chunk costs more to bring together than it saves
    w.segments = (w.chunks + w.per - 1) / w.per;
    size_t off = 0;
    auto area = [&](size_t n) {
        float *at = base ? base + off : nullptr;
        off += (n + 63) / 64 * 64;
        return at;
    };
    const size_t pairs = (size_t)p.B * p.H, g_n = w.segments > 1 ? w.segments : 0;
    w.o = area((size_t)p.B * p.S * p.H * p.E);
    w.gate = area(pairs * w.chunks * (4 * kChunk + p.D));
    w.scores = area(p.D >= 128 ? pairs * w.chunks * kChunk * kChunk : 0);
    w.seg_s = area(pairs * g_n * p.D * p.E);
    w.seg_n = area(pairs * g_n * p.D);
    w.seg_m = area(pairs * g_n * 2);
    if (bytes) *bytes = off * sizeof(float);
}

// a, b, c of one chunk per warp, two neighbouring tokens per lane
__global__ void __launch_bounds__(256) mlstm_gates_kernel(const MlstmStep p, const ChunkWs w) {
    pdl_trigger();
    pdl_wait();
    const int job = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (job >= p.B * p.H * w.chunks) return;
    const int pair = job / w.chunks, c = job - pair * w.chunks, b = pair / p.H, h = pair - b * p.H;
    float ga[2], gb[2], gc[2];
    chunk_gates(p, b, h, c, lane, ga, gb, gc);
    float *out = w.gate + (size_t)job * 3 * kChunk + 2 * lane;
    *reinterpret_cast<float2 *>(out) = make_float2(ga[0], ga[1]);
    *reinterpret_cast<float2 *>(out + kChunk) = make_float2(gb[0], gb[1]);
    *reinterpret_cast<float2 *>(out + 2 * kChunk) = make_float2(gc[0], gc[1]);
}

template <typename T, int KD, bool OUT>
struct ChunkSmem {
    static constexpr int LD = KD + 8, LV = kChunkCols + 8, LP = kChunk + 8;  // row lengths: an odd number of 16-byte pieces
    T k[2][kChunk][LD], v[2][kChunk][LV];
    T q[OUT ? 2 : 1][OUT ? kChunk : 1][LD];
    T p_hi[OUT ? kChunk : 1][LP], p_lo[OUT ? kChunk : 1][LP];
    T n_part[OUT ? 8 : 1][LD];  // n_0 as high part and remainder (rows 0 and 1; the others are zero)
    float gate[2][3][kChunk];
    float n[KD];
    float qn[kChunk], part[2][kChunk], inv[kChunk];  // q.n_0; row sums of the weighted scores by column half; 1 / denominator
    unsigned flag;
};

// grid (ceil(E / 128), H, B * segments), 256 threads.  KD: D padded to 64, 128 or 256.  OUT: outputs, from the state in front of the
// segment, and the state behind the last one; else the first pass over all segments but the last (see add_segment).
template <typename T, int KD, bool OUT>
__global__ void __launch_bounds__(kChunkThreads, 1) mlstm_chunk_kernel(const MlstmStep p, const ChunkWs w) {
    extern __shared__ __align__(16) uint8_t chunk_smem[];
    using Sm = ChunkSmem<T, KD, OUT>;
    Sm &sm = *reinterpret_cast<Sm *>(chunk_smem);
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, b = blockIdx.z / (OUT ? w.segments : w.segments - 1), seg = blockIdx.z - b * (OUT ? w.segments : w.segments - 1), pair = b * p.H + h;
    const bool single = w.segments == 1, final_state = OUT && seg == w.segments - 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t4 = lane & 3;
    const int e0 = blockIdx.x * kChunkCols, ew = e0 + 16 * warp;  // the CTA's and the warp's first column
    const bool work = ew < p.E;                                   // warps past the last column only help with the scores
    const size_t C = (size_t)2 * p.H * (p.D + p.E);
    const T *base = reinterpret_cast<const T *>(p.proj) + (size_t)b * p.S * C;
    const float q_scale = 1.0f / sqrtf((float)p.D);
    const int c_beg = seg * w.per, c_end = min(c_beg + w.per, w.chunks);

    auto fetch = [&](int c) {
        const int buf = c & 1, t0 = c * kChunk;
        constexpr int PQ = KD / 8, PV = kChunkCols / 8;
        for (int i = threadIdx.x; i < kChunk * PQ; i += kChunkThreads) {
            const int t = i / PQ, d = (i - t * PQ) * 8;
            const bool in = t0 + t < p.S && d < p.D;
            const T *src = base + (size_t)(in ? t0 + t : 0) * C + (size_t)h * p.D + (in ? d : 0);
            if constexpr (OUT) copy16(&sm.q[buf][t][d], src, in);
            copy16(&sm.k[buf][t][d], src + (size_t)p.H * p.D, in);
        }
        for (int i = threadIdx.x; i < kChunk * PV; i += kChunkThreads) {
            const int t = i / PV, e = (i - t * PV) * 8;
            const bool in = t0 + t < p.S && e0 + e < p.E;
            copy16(&sm.v[buf][t][e], base + (size_t)(in ? t0 + t : 0) * C + (size_t)2 * p.H * p.D + (size_t)h * p.E + (in ? e0 + e : 0), in);
        }
        if (threadIdx.x < 3 * kChunk / 4) copy16(&sm.gate[buf][0][0] + 4 * threadIdx.x, w.gate + ((size_t)pair * w.chunks + c) * 3 * kChunk + 4 * threadIdx.x, true);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(c_beg);

    // S transposed: row tile = the warp's 16 columns e, column tile j = rows d 8 j .. 8 j + 7.  Register x: e = ew + gq + 8 (x >> 1),
    // d = 8 j + 2 t4 + (x & 1)
    constexpr int NS = KD / 8;
    float S[NS][4];
    const size_t DE = (size_t)p.D * p.E, slot0 = (size_t)pair * w.segments;
    const bool fresh = *p.past == 0, first = single || (!OUT && seg == 0);  // starts from the state in front of the call
    // memory and sum vector to start from, and the running maximum, which every thread follows
    const float *from_s = first ? p.mem + pair * DE : w.seg_s + (slot0 + (seg == 0 ? w.segments - 1 : 0)) * DE;
    const float *from_n = first ? p.sum + (size_t)pair * p.D : w.seg_n + (slot0 + (seg == 0 ? w.segments - 1 : 0)) * p.D;
    const bool empty = first ? fresh : !OUT;
    float m0 = first ? (fresh ? 0.f : p.top[pair]) : !OUT ? -INFINITY : w.seg_m[(slot0 + (seg == 0 ? w.segments - 1 : 0)) * 2 + 1];
#pragma unroll
    for (int j = 0; j < NS; j++)
#pragma unroll
        for (int x = 0; x < 4; x++) {
            const int e = ew + gq + 8 * (x >> 1), d = 8 * j + 2 * t4 + (x & 1);
            const bool in = e < p.E && d < p.D;
            S[j][x] = !empty && in ? from_s[(size_t)d * p.E + e] : 0.f;
            if (!OUT && seg == 0 && in) w.seg_s[(slot0 + w.segments - 1) * DE + (size_t)d * p.E + e] = S[j][x];
        }
    const float m_front = m0;
    if (OUT && !single)
        for (int g = 1; g < seg; g++) {
            float keep, take;
            add_segment(w, pair, g, m0, keep, take);
            const float *more = w.seg_s + (slot0 + g) * DE;
#pragma unroll
            for (int j = 0; j < NS; j++)
#pragma unroll
                for (int x = 0; x < 4; x++) {
                    const int e = ew + gq + 8 * (x >> 1), d = 8 * j + 2 * t4 + (x & 1);
                    S[j][x] = keep * S[j][x] + take * (e < p.E && d < p.D ? more[(size_t)d * p.E + e] : 0.f);
                }
        }
    auto n_front = [&](int d) {  // n in front of the segment
        float n = !empty && d < p.D ? from_n[d] : 0.f;
        if (!OUT && seg == 0 && blockIdx.x == 0 && d < p.D) w.seg_n[(slot0 + w.segments - 1) * p.D + d] = n;
        if (OUT && !single && d < p.D) {
            float m = m_front, keep, take;
            for (int g = 1; g < seg; g++) {
                add_segment(w, pair, g, m, keep, take);
                n = keep * n + take * w.seg_n[(slot0 + g) * p.D + d];
            }
        }
        return n;
    };
    if (!OUT && seg == 0 && blockIdx.x == 0 && threadIdx.x == 0) w.seg_m[(slot0 + w.segments - 1) * 2 + 1] = m0;
    float forgotten = 0.f;
    auto set_n = [&](int d, float x) {
        sm.n[d] = x;
        if constexpr (OUT) split_one<T>(x, sm.n_part[0][d], sm.n_part[1][d]);
    };
    if constexpr (OUT)
        for (int i = threadIdx.x; i < 6 * Sm::LD; i += kChunkThreads) (&sm.n_part[2][0])[i] = from_f32<T>(0.f);
    for (int d = threadIdx.x; d < KD; d += kChunkThreads) set_n(d, n_front(d));

    const int mt = warp & 3, nh = warp >> 2;  // scores: 16 query tokens, a half of the key tokens
    for (int c = c_beg; c < c_end; c++) {
        const int buf = c & 1, t0 = c * kChunk;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // chunk c and n are in shared memory; chunk c - 1 has been read by all
        if (c + 1 < c_end) fetch(c + 1);
        const float *ga = sm.gate[buf][0], *gb = sm.gate[buf][1], *gc = sm.gate[buf][2];
        const float end_top = fmaxf(m0, gc[kChunk - 1]), keep = __expf(m0 - end_top);
        float acc[8][4];  // o transposed: the warp's 16 columns e x 64 tokens
        if constexpr (OUT) {
            // ---- scores of 16 x 32 tokens and q.n_0 ----
            {
                float sc[4][4], qn[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int j = 0; j < 4; j++) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
                const bool some = 16 * mt + 15 >= 32 * nh;  // some pair s <= t
#pragma unroll 4
                for (int kk = 0; kk < KD; kk += 16) {
                    uint32_t qa[4];
                    ldsm4(qa, &sm.q[buf][16 * mt + (lane & 15)][kk + 8 * (lane >> 4)]);
                    if (nh) {
                        const uint32_t n0 = *reinterpret_cast<const uint32_t *>(&sm.n_part[gq][kk + 2 * t4]), n1 = *reinterpret_cast<const uint32_t *>(&sm.n_part[gq][kk + 8 + 2 * t4]);
                        mma_kv<T>(qn, qa[0], qa[1], qa[2], qa[3], n0, n1);
                    }
                    if (some) {
#pragma unroll
                        for (int j = 0; j < 2; j++) {
                            uint32_t kb[4];  // key tokens 32 nh + 16 j .. + 15: (first 8, k low), (first 8, k high), (last 8, ..)
                            ldsm4(kb, &sm.k[buf][32 * nh + 16 * j + (lane & 7) + 8 * (lane >> 4)][kk + 8 * ((lane >> 3) & 1)]);
                            mma_kv<T>(sc[2 * j], qa[0], qa[1], qa[2], qa[3], kb[0], kb[1]);
                            mma_kv<T>(sc[2 * j + 1], qa[0], qa[1], qa[2], qa[3], kb[2], kb[3]);
                        }
                    }
                }
                const int tr[2] = {16 * mt + gq, 16 * mt + gq + 8};
                const float rr[2] = {-fmaxf(m0, gc[tr[0]]), -fmaxf(m0, gc[tr[1]])};  // b_t - m_t
                float rs[2] = {0.f, 0.f};
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int s = 32 * nh + 8 * j + 2 * t4;
                    const float a0 = ga[s], a1 = ga[s + 1];
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
                    if (t4 == 0) {
                        sm.part[nh][tr[x]] = rs[x];
                        if (nh) sm.qn[tr[x]] = qn[2 * x] + qn[2 * x + 1];  // columns 0 and 1: high part and remainder
                    }
                }
            }
            // ---- what the old state contributes: S_0^T q^T ----
#pragma unroll
            for (int j = 0; j < 8; j++) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
            if (work) {
#pragma unroll
                for (int kk = 0; kk < NS; kk += 2) {  // 16 rows d
                    uint32_t ah[4], al[4];
                    split_pack<T>(S[kk][0], S[kk][1], ah[0], al[0]);
                    split_pack<T>(S[kk][2], S[kk][3], ah[1], al[1]);
                    split_pack<T>(S[kk + 1][0], S[kk + 1][1], ah[2], al[2]);
                    split_pack<T>(S[kk + 1][2], S[kk + 1][3], ah[3], al[3]);
#pragma unroll
                    for (int j = 0; j < 4; j++) {
                        uint32_t qb[4];  // tokens 16 j .. + 15
                        ldsm4(qb, &sm.q[buf][16 * j + (lane & 7) + 8 * (lane >> 4)][8 * kk + 8 * ((lane >> 3) & 1)]);
                        mma_kv<T>(acc[2 * j], ah[0], ah[1], ah[2], ah[3], qb[0], qb[1]);
                        mma_kv<T>(acc[2 * j + 1], ah[0], ah[1], ah[2], ah[3], qb[2], qb[3]);
                        mma_kv<T>(acc[2 * j], al[0], al[1], al[2], al[3], qb[0], qb[1]);
                        mma_kv<T>(acc[2 * j + 1], al[0], al[1], al[2], al[3], qb[2], qb[3]);
                    }
                }
#pragma unroll
                for (int j = 0; j < 8; j++) {
                    const int t = 8 * j + 2 * t4;
                    const float f0 = __expf(m0 - fmaxf(m0, gc[t])) * q_scale, f1 = __expf(m0 - fmaxf(m0, gc[t + 1])) * q_scale;
                    acc[j][0] *= f0, acc[j][1] *= f1, acc[j][2] *= f0, acc[j][3] *= f1;
                }
            }
            __syncthreads();  // weighted scores, their sums and q.n_0 are there; n has been read
            if (threadIdx.x < kChunk) {
                const int t = threadIdx.x;
                const float top = fmaxf(m0, gc[t]), den = __expf(m0 - top) * q_scale * sm.qn[t] + sm.part[0][t] + sm.part[1][t];
                sm.inv[t] = 1.0f / (fmaxf(fabsf(den), expf(-(gb[t] + top))) + kMlstmFloor);
            }
        }
        // ---- values: + weighted scores (V^T P^T), and into the state at the chunk's end (V'^T K) ----
        if (work) {
            const bool grow = !OUT || final_state || c + 1 < c_end;  // else the next segment knows it from the first pass
            if (grow) {
#pragma unroll
                for (int j = 0; j < NS; j++)
#pragma unroll
                    for (int x = 0; x < 4; x++) S[j][x] *= keep;
            }
#pragma unroll
            for (int kk = 0; kk < kChunk; kk += 16) {  // 16 key tokens
                uint32_t va[4];  // v transposed: (e 0-7, s 0-7), (e 8-15, s 0-7), (e 0-7, s 8-15), ..
                ldsm4t(va, &sm.v[buf][kk + (lane & 7) + 8 * (lane >> 4)][16 * warp + 8 * ((lane >> 3) & 1)]);
                if constexpr (OUT) {
#pragma unroll
                    for (int j = kk / 16; j < 4; j++) {  // earlier query tokens do not see them
                        uint32_t ph[4], pl[4];
                        ldsm4(ph, &sm.p_hi[16 * j + (lane & 7) + 8 * (lane >> 4)][kk + 8 * ((lane >> 3) & 1)]);
                        ldsm4(pl, &sm.p_lo[16 * j + (lane & 7) + 8 * (lane >> 4)][kk + 8 * ((lane >> 3) & 1)]);
                        mma_kv<T>(acc[2 * j], va[0], va[1], va[2], va[3], ph[0], ph[1]);
                        mma_kv<T>(acc[2 * j + 1], va[0], va[1], va[2], va[3], ph[2], ph[3]);
                        mma_kv<T>(acc[2 * j], va[0], va[1], va[2], va[3], pl[0], pl[1]);
                        mma_kv<T>(acc[2 * j + 1], va[0], va[1], va[2], va[3], pl[2], pl[3]);
                    }
                }
                if (grow) {
                    uint32_t wh[4], wl[4];
#pragma unroll
                    for (int x = 0; x < 4; x++) {
                        const int s = kk + 2 * t4 + 8 * (x >> 1);
                        const T *two = reinterpret_cast<const T *>(&va[x]);
                        split_pack<T>(to_f32<T>(two[0]) * __expf(ga[s] - end_top), to_f32<T>(two[1]) * __expf(ga[s + 1] - end_top), wh[x], wl[x]);
                    }
#pragma unroll
                    for (int j = 0; j < NS; j += 2) {
                        uint32_t kb[4];  // k [s][d] read transposed: (s 0-7, d 0-7), (s 8-15, d 0-7), (s 0-7, d 8-15), ..
                        ldsm4t(kb, &sm.k[buf][kk + (lane & 15)][8 * j + 8 * (lane >> 4)]);
                        mma_kv<T>(S[j], wh[0], wh[1], wh[2], wh[3], kb[0], kb[1]);
                        mma_kv<T>(S[j + 1], wh[0], wh[1], wh[2], wh[3], kb[2], kb[3]);
                        mma_kv<T>(S[j], wl[0], wl[1], wl[2], wl[3], kb[0], kb[1]);
                        mma_kv<T>(S[j + 1], wl[0], wl[1], wl[2], wl[3], kb[2], kb[3]);
                    }
                }
            }
        }
        // ---- n, two rows per thread ----
        for (int d = 2 * threadIdx.x; d < KD; d += 2 * kChunkThreads) {
            float x0 = keep * sm.n[d], x1 = keep * sm.n[d + 1];
#pragma unroll 8
            for (int t = 0; t < kChunk; t++) {
                const uint32_t two = *reinterpret_cast<const uint32_t *>(&sm.k[buf][t][d]);
                const T *e = reinterpret_cast<const T *>(&two);
                const float f = __expf(ga[t] - end_top);
                x0 += f * to_f32<T>(e[0]), x1 += f * to_f32<T>(e[1]);
            }
            set_n(d, x0), set_n(d + 1, x1);
        }
        if constexpr (OUT) {
            __syncthreads();  // 1 / denominator
            if (work) {
#pragma unroll
                for (int j = 0; j < 8; j++)
#pragma unroll
                    for (int x = 0; x < 4; x++) {
                        const int t = 8 * j + 2 * t4 + (x & 1), e = ew + gq + 8 * (x >> 1);
                        if (t0 + t < p.S && e < p.E) w.o[(((size_t)b * p.S + t0 + t) * p.H + h) * p.E + e] = acc[j][x] * sm.inv[t];
                    }
            }
        }
        forgotten += gb[kChunk - 1];
        m0 = gb[kChunk - 1] + end_top;
    }
    if (OUT && !final_state) return;
    float *to_s = OUT ? p.mem + pair * DE : w.seg_s + (slot0 + seg) * DE;
#pragma unroll
    for (int j = 0; j < NS; j++)
#pragma unroll
        for (int x = 0; x < 4; x++) {
            const int e = ew + gq + 8 * (x >> 1), d = 8 * j + 2 * t4 + (x & 1);
            if (e < p.E && d < p.D) to_s[(size_t)d * p.E + e] = S[j][x];
        }
    if constexpr (OUT) {
        if (single ? !last_of_head(p, pair, gridDim.x, &sm.flag) : blockIdx.x != 0) return;
    } else if (blockIdx.x != 0) {
        return;
    }
    __syncthreads();
    float *to_n = OUT ? p.sum + (size_t)pair * p.D : w.seg_n + (slot0 + seg) * p.D;
    for (int d = threadIdx.x; d < p.D; d += kChunkThreads) to_n[d] = sm.n[d];
    if (threadIdx.x == 0) {
        if (OUT) p.top[pair] = m0;
        else w.seg_m[(slot0 + seg) * 2] = forgotten, w.seg_m[(slot0 + seg) * 2 + 1] = m0;
    }
}

bool mlstm_chunkwise_supported(int dtype, const MlstmStep &p) {
    const uintptr_t a = (uintptr_t)p.proj | (uintptr_t)p.workspace | (uintptr_t)p.mem;
    return dtype != MYNN_F32 && p.D <= 256 && p.D % 8 == 0 && p.E % 8 == 0 && a % 16 == 0;
}

size_t mlstm_workspace_bytes(int dtype, int B, int S, int H, int D, int E) {
    MlstmStep p;
    p.B = B, p.S = S, p.H = H, p.D = D, p.E = E;
    ChunkWs w;
    size_t chunkwise = 0;
    const size_t plain = (size_t)B * S * H * E * sizeof(float);
    if (!mlstm_chunkwise_supported(dtype, p)) return plain;
    bind_chunk_ws(w, p, nullptr, &chunkwise);
    return chunkwise > plain ? chunkwise : plain;
}

template <typename T>
static int run_out(cudaStream_t st, const MlstmStep &p) {
    mlstm_out_kernel<T><<<(unsigned)(((long long)p.B * p.S * p.H + 7) / 8), 256, 0, st>>>(p);
    MYNN_LAUNCH_OK("mlstm_out_kernel");
    return MYNN_OK;
}

template <typename T, bool ONE>
static int run_scan(cudaStream_t st, const MlstmStep &p) {
    const dim3 grid((p.E + kScanCols - 1) / kScanCols, p.H, p.B);
    if (p.D <= 64) mlstm_scan_kernel<T, 8, ONE><<<grid, 256, 0, st>>>(p);
    else if (p.D <= 128) mlstm_scan_kernel<T, 16, ONE><<<grid, 256, 0, st>>>(p);
    else if (p.D <= 256) mlstm_scan_kernel<T, 32, ONE><<<grid, 256, 0, st>>>(p);
    else mlstm_scan_kernel<T, 64, ONE><<<grid, 256, 0, st>>>(p);
    MYNN_LAUNCH_OK("mlstm_scan_kernel");
    return ONE ? MYNN_OK : run_out<T>(st, p);
}

template <typename T, int KD, bool OUT>
static int run_chunk_pass(cudaStream_t st, const MlstmStep &p, const ChunkWs &w) {
    constexpr size_t smem = sizeof(ChunkSmem<T, KD, OUT>);
    static_assert(smem <= 227 * 1024, "shared memory of a CTA");
    auto kern = mlstm_chunk_kernel<T, KD, OUT>;
    static bool attr_set = false;
    if (!attr_set) {
        MYNN_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set = true;
    }
    kern<<<dim3((p.E + kChunkCols - 1) / kChunkCols, p.H, p.B * (OUT ? w.segments : w.segments - 1)), kChunkThreads, smem, st>>>(p, w);
    MYNN_LAUNCH_OK("mlstm_chunk_kernel");
    return MYNN_OK;
}

template <typename T, int KD>
static int run_chunk(cudaStream_t st, int dtype, const MlstmStep &p) {
    ChunkWs w;
    size_t need = 0;
    bind_chunk_ws(w, p, p.workspace, &need);
    if (p.workspace_bytes < need) return fail(MYNN_E_ARG, "mlstm: workspace of %zu bytes, %zu are needed", p.workspace_bytes, need);
    const bool tc = p.form == 3 || (p.form == 0 && mlstm_tc_supported(dtype, p));
    if (tc) {
        if (int rc = launch_mlstm_prepare(st, dtype, p, w)) return rc;
    } else {
        mlstm_gates_kernel<<<(unsigned)(((long long)p.B * p.H * w.chunks + 7) / 8), 256, 0, st>>>(p, w);
        MYNN_LAUNCH_OK("mlstm_gates_kernel");
    }
    if (w.segments > 1)
        if (int rc = tc ? launch_mlstm_tc(st, dtype, p, w, false) : run_chunk_pass<T, KD, false>(st, p, w)) return rc;
    if (int rc = tc ? launch_mlstm_tc(st, dtype, p, w, true) : run_chunk_pass<T, KD, true>(st, p, w)) return rc;
    return run_out<T>(st, p);
}

template <typename T>
static int run_chunk_any(cudaStream_t st, int dtype, const MlstmStep &p) {
    if (p.D <= 64) return run_chunk<T, 64>(st, dtype, p);
    if (p.D <= 128) return run_chunk<T, 128>(st, dtype, p);
    return run_chunk<T, 256>(st, dtype, p);
}

int launch_mlstm(cudaStream_t st, int dtype, const MlstmStep &p) {
    if (p.B <= 0 || p.S <= 0 || p.H <= 0 || p.D <= 0 || p.E <= 0 || !(p.cap > 0.f)) return fail(MYNN_E_ARG, "mlstm: bad shape");
    if (!dtype_ok(dtype)) return fail(MYNN_E_ARG, "mlstm: bad dtype %d", dtype);
    if (p.D > kMlstmMaxDim || p.H > 65535 || p.B > 65535) return fail(MYNN_E_UNSUPPORTED, "mlstm: %d heads of %d", p.H, p.D);
    if (!p.proj || !p.gates || !p.gate_bias || !p.norm_w || !p.mem || !p.sum || !p.top || !p.workspace || !p.ticket || !p.out || !p.past) return fail(MYNN_E_ARG, "mlstm: null pointer");
    if (p.workspace_bytes < (size_t)p.B * p.S * p.H * p.E * sizeof(float)) return fail(MYNN_E_ARG, "mlstm: workspace of %zu bytes", p.workspace_bytes);
    const bool can = mlstm_chunkwise_supported(dtype, p);
    if ((p.form == 2 && !can) || (p.form == 3 && !(can && mlstm_tc_supported(dtype, p)))) return fail(MYNN_E_UNSUPPORTED, "mlstm: not a shape of the chunkwise kernel");
    if (p.form >= 2 || (p.form == 0 && can && p.S > 12)) return dtype == MYNN_BF16 ? run_chunk_any<__nv_bfloat16>(st, dtype, p) : run_chunk_any<__half>(st, dtype, p);
    MYNN_DISPATCH_DTYPE(dtype, T, { return p.S == 1 ? run_scan<T, true>(st, p) : run_scan<T, false>(st, p); });
    return MYNN_OK;
}

}  // namespace mynn

using namespace mynn;

extern "C" size_t mynn_b200_mlstm_workspace_bytes(int B, int S, int H, int D, int E, int dtype) {
    return B <= 0 || S <= 0 || H <= 0 || D <= 0 || E <= 0 ? 0 : mlstm_workspace_bytes(dtype, B, S, H, D, E);
}

extern "C" int mynn_b200_mlstm(void *stream, void *out, float *mem, float *sum, float *top, const void *proj, const float *gates, const float *gate_bias,
                               const float *norm_weight, float cap, float eps, int B, int S, int H, int D, int E, const int32_t *past_dev, void *workspace,
                               size_t workspace_bytes, uint32_t *tickets, int dtype, int form, int32_t *status) {
    MlstmStep p;
    p.proj = proj;
    p.gates = gates;
    p.gate_bias = gate_bias;
    p.norm_w = norm_weight;
    p.cap = cap, p.eps = eps;
    p.mem = mem, p.sum = sum, p.top = top;
    p.workspace = (float *)workspace;
    p.workspace_bytes = workspace_bytes;
    p.ticket = tickets;
    p.out = out;
    p.B = B, p.S = S, p.H = H, p.D = D, p.E = E;
    p.past = past_dev;
    p.form = form;
    p.status = status;
    return launch_mlstm((cudaStream_t)stream, dtype, p);
}
