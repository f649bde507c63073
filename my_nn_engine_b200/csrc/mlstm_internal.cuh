// Pieces shared by the kernels of the matrix memory: mlstm.cu (token by token, chunkwise on mma.sync) and mlstm_tc.cu (chunkwise on tcgen05).
#pragma once
#include "attention_internal.cuh"
#include "block_ops.cuh"
#include "common.cuh"

namespace mynn {

constexpr float kMlstmFloor = 1e-6f;  // added to the denominator
constexpr int kChunk = 64;            // tokens the chunkwise forms take at a time
constexpr int kChunkCols = 128;       // columns of the memory per CTA

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
// for results that are rounded to 16 bits
__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// scratch of the chunkwise form
struct ChunkWs {
    float *o;      // [B S, H E]
    float *gate;   // [B H][chunk][3][64]: a, b, c of every token; on tcgen05 a record per chunk (mlstm_tc.cu)
    void *scores;  // on tcgen05 [B H][chunk][2][64][64] 16-bit: the weighted scores
    float *seg_s;  // [B H][segment][D, E]: what a segment leaves
    float *seg_n;  // [B H][segment][D]
    float *seg_m;  // [B H][segment][2]: sum of its log forget gates, maximum of what it adds
    int chunks = 0, segments = 0, per = 0;  // chunks per segment
};

// Segments (w.segments > 1).  The first pass runs segments 0 .. G - 2: segment 0 from the state in front of the call, of which it leaves a copy
// in place G - 1, the others from nothing.  The state in front of segment g is then that copy (g == 0) or segment 0's result with what
// the segments up to g - 1 add.  The factors of one more segment j, and the maximum behind it:
__device__ __forceinline__ void add_segment(const ChunkWs &w, int pair, int j, float &m, float &keep, float &take) {
    const float *sm = w.seg_m + ((size_t)pair * w.segments + j) * 2;
    const float kept = sm[0] + m, added = sm[1];
    m = fmaxf(kept, added);
    keep = expf(kept - m), take = expf(added - m);
}

template <typename T>
__device__ __forceinline__ void split_one(float x, T &hi, T &lo) {
    hi = from_f32<T>(x);
    lo = from_f32<T>(x - to_f32<T>(hi));
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

// a, b, c of chunk c by one warp, tokens 2 lane and 2 lane + 1
__device__ __forceinline__ void chunk_gates(const MlstmStep &p, int b, int h, int c, int lane, float (&a)[2], float (&bb)[2], float (&cc)[2]) {
    float gi[2], gf[2];
#pragma unroll
    for (int j = 0; j < 2; j++) {
        const int t = c * kChunk + 2 * lane + j;
        gi[j] = -INFINITY, gf[j] = 0.f;  // past the end: nothing added, nothing forgotten
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
    bb[0] = sum - gf[1], bb[1] = sum;
    a[0] = gi[0] - bb[0], a[1] = gi[1] - bb[1];
    float mx = fmaxf(a[0], a[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, u);
    }
    float before = __shfl_up_sync(0xffffffffu, mx, 1);
    if (lane == 0) before = -INFINITY;
    cc[0] = fmaxf(before, a[0]), cc[1] = mx;
}

// The chunkwise kernels on tcgen05; OUT and no OUT as for mlstm_chunk_kernel.
int launch_mlstm_prepare(cudaStream_t st, int dtype, const MlstmStep &p, const ChunkWs &w);
bool mlstm_tc_supported(int dtype, const MlstmStep &p);
int launch_mlstm_tc(cudaStream_t st, int dtype, const MlstmStep &p, const ChunkWs &w, bool out);

}  // namespace mynn
