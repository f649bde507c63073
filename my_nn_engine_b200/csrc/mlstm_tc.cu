// The chunkwise matrix memory (see mlstm.cu) with its products on tcgen05, for heads of 128 or 256 rows.
//
// mlstm_prepare_kernel   what a chunk of 64 tokens needs and the state does not enter: with a, b, c as in mlstm.cu, the scores weighted with
//                        e^(a_s - c_t) (in two 16-bit parts) and their sums over s, and the sum of the keys weighted with e^(a_s - c_63).  The
//                        recurrence's maximum then only multiplies whole rows, by e^(c_t - m_t + b_t).  Once per head and chunk.
// mlstm_tc_kernel        A CTA carries 128 columns e of one head's memory, transposed: thread = tensor-memory lane e, a quarter of the rows d
//                        in 32-bit registers.  q, k and v of a chunk come by TMA, two chunks in flight, and stay in shared memory as they are.
//                        One thread issues all products of a chunk, which run in the order they are issued:
//   1. V^T P^T, the weighted scores in two parts
//   2. S_0^T q^T, the memory as high 16-bit part and remainder from tensor memory
//   3. V'^T K, the values weighted with e^(a_s - c_63) in two parts; the increment of the memory overwrites the columns in which product 2
//      found the memory's parts
// While they run the warps form q.n_0 and the denominators and store the outputs of the chunk before, 128 neighbouring bytes per warp.  Waits are bounded and report through the
// caller's word.
#include <type_traits>

#include "i8_gemm.cuh"
#include "mlstm_internal.cuh"
#include "tcgen05.cuh"

namespace mynn {

MYNN_DEFINE_WAIT_BUDGET_SETTER(mlstm_tc)

constexpr int kMtThreads = 512;
constexpr uint32_t kMtSlab = kChunk * 128;  // 64 rows of 64 elements

// Tiles [64][.] stand in slabs of 64 columns with the 128-byte swizzle: the 16-byte piece c of row r of a slab is at r * 128 + ((c ^ r) & 7) * 16.
// Byte offset of element (row, col) for slabs of `slab` bytes:
__device__ __forceinline__ uint32_t slab_off(int row, int col, uint32_t slab = kMtSlab) {
    return (uint32_t)(col >> 6) * slab + (uint32_t)row * 128u + (uint32_t)((((col >> 3) & 7) ^ (row & 7)) << 4) + (uint32_t)(col & 7) * 2u;
}

// One chunk of one head, left by mlstm_prepare_kernel: f32 a, b, c, sum of the weighted scores (64 each), weighted key sum (KD); and the
// weighted scores [64][64] in the swizzled layout, high parts, then remainders.
constexpr int kMtRecord = 4 * kChunk;
constexpr uint32_t kMtScoreBytes = 2 * kMtSlab;

// grid (chunks, H, B), 256 threads; dynamic shared memory: q and k of the chunk
template <typename T, int KD>
__global__ void __launch_bounds__(256) mlstm_prepare_kernel(const MlstmStep p, const ChunkWs w) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    constexpr int SLABS = KD / 64, PQ = KD / 8, RQ = 256 / PQ;
    constexpr uint32_t kKeys = SLABS * kMtSlab;
    __shared__ float ga[kChunk], gc[kChunk], w_end[kChunk], part[2][kChunk], n_red[2][KD];
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, pair = b * p.H + h, t0 = c * kChunk;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t4 = lane & 3;
    const size_t C = (size_t)2 * p.H * (p.D + p.E), job = (size_t)pair * w.chunks + c;
    float *rec = w.gate + job * (kMtRecord + KD);
    uint8_t *scores = reinterpret_cast<uint8_t *>(w.scores) + job * kMtScoreBytes;
    const float q_scale = 1.0f / sqrtf((float)p.D);
    {
        const int row = threadIdx.x / PQ, col = (threadIdx.x % PQ) * 8;
        const T *src = reinterpret_cast<const T *>(p.proj) + (size_t)b * p.S * C + (size_t)h * p.D + col;
        const uint32_t dst = smem_u32(smem) + slab_off(row, col);
#pragma unroll
        for (int j = 0; j < kChunk / RQ; j++) {
            const int t = t0 + row + j * RQ;
            const T *at = src + (size_t)(t < p.S ? t : 0) * C;
            copy16_at(dst + j * RQ * 128, at, t < p.S);
            copy16_at(dst + kKeys + j * RQ * 128, at + (size_t)p.H * p.D, t < p.S);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    if (warp == 0) {
        float a[2], bb[2], cc[2];
        chunk_gates(p, b, h, c, lane, a, bb, cc);
        const float last = __shfl_sync(0xffffffffu, cc[1], 31);
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int t = 2 * lane + j;
            ga[t] = a[j], gc[t] = cc[j], w_end[t] = __expf(a[j] - last);
            rec[t] = a[j], rec[kChunk + t] = bb[j], rec[2 * kChunk + t] = cc[j];
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // ---- scores: a warp takes 16 query and 32 key tokens ----
    const int mt = warp & 3, nh = warp >> 2;
    float sc[4][4];
#pragma unroll
    for (int j = 0; j < 4; j++) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
    if (16 * mt + 15 >= 32 * nh) {  // some pair s <= t
        const uint32_t base = smem_u32(smem), aa = base + slab_off(16 * mt + (lane & 15), 8 * (lane >> 4)),
                       bb = base + kKeys + slab_off(32 * nh + (lane & 7) + 8 * (lane >> 4), 8 * ((lane >> 3) & 1));
#pragma unroll
        for (int x = 0; x < 4; x++)  // the swizzle turns a step of 16 columns inside a slab into an exclusive or
#pragma unroll
            for (int sl = 0; sl < SLABS; sl++) {
                uint32_t qa[4], kb[4], kc[4];
                ldsm4_at(qa, (aa ^ (x << 5)) + sl * kMtSlab);
                ldsm4_at(kb, (bb ^ (x << 5)) + sl * kMtSlab);
                ldsm4_at(kc, (bb ^ (x << 5)) + sl * kMtSlab + 16 * 128);
                mma_kv<T>(sc[0], qa[0], qa[1], qa[2], qa[3], kb[0], kb[1]);
                mma_kv<T>(sc[1], qa[0], qa[1], qa[2], qa[3], kb[2], kb[3]);
                mma_kv<T>(sc[2], qa[0], qa[1], qa[2], qa[3], kc[0], kc[1]);
                mma_kv<T>(sc[3], qa[0], qa[1], qa[2], qa[3], kc[2], kc[3]);
            }
    }
#pragma unroll
    for (int x = 0; x < 2; x++) {
        const int t = 16 * mt + gq + 8 * x;
        float rs = 0.f;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int s = 32 * nh + 8 * j + 2 * t4;
            const float w0 = s <= t ? sc[j][2 * x] * q_scale * __expf(ga[s] - gc[t]) : 0.f;
            const float w1 = s + 1 <= t ? sc[j][2 * x + 1] * q_scale * __expf(ga[s + 1] - gc[t]) : 0.f;
            rs += w0 + w1;
            uint32_t hi, lo;
            split_pack<T>(w0, w1, hi, lo);
            const uint32_t off = slab_off(t, s);
            *reinterpret_cast<uint32_t *>(scores + off) = hi;
            *reinterpret_cast<uint32_t *>(scores + kMtSlab + off) = lo;
        }
        rs += __shfl_xor_sync(0xffffffffu, rs, 1);
        rs += __shfl_xor_sync(0xffffffffu, rs, 2);
        if (t4 == 0) part[nh][t] = rs;
    }
    // ---- weighted key sum: two rows and half of the tokens per thread ----
    if (threadIdx.x < KD) {
        const int d = 2 * (threadIdx.x % (KD / 2)), g = threadIdx.x / (KD / 2);
        float x0 = 0.f, x1 = 0.f;
#pragma unroll 8
        for (int i = 0; i < kChunk / 2; i++) {
            const int t = g * (kChunk / 2) + i;
            const uint32_t two = *reinterpret_cast<const uint32_t *>(smem + kKeys + slab_off(t, d));
            const T *x = reinterpret_cast<const T *>(&two);
            x0 += w_end[t] * to_f32<T>(x[0]), x1 += w_end[t] * to_f32<T>(x[1]);
        }
        n_red[g][d] = x0, n_red[g][d + 1] = x1;
    }
    __syncthreads();
    if (threadIdx.x < kChunk) rec[3 * kChunk + threadIdx.x] = part[0][threadIdx.x] + part[1][threadIdx.x];
    for (int d = threadIdx.x; d < KD; d += 256) rec[kMtRecord + d] = n_red[0][d] + n_red[1][d];
}

template <int KD, bool OUT>
struct MtLayout {
    static constexpr int kSlabs = KD / 64, kStages = OUT ? 2 : 3;  // chunks in flight
    static constexpr uint32_t kQ = 0, kK = kQ + (OUT ? kStages * kSlabs * kMtSlab : 0), kV = kK + kStages * kSlabs * kMtSlab, kVw = kV + kStages * 2 * kMtSlab,
                              kP = kVw + 4 * kMtSlab, kBytes = kP + (OUT ? 2 * kMtSlab : 0);
    static constexpr uint32_t kTmemCols = OUT ? 512 : KD;
    static constexpr uint32_t kColInter = KD, kColPv = KD + 64;  // the memory's parts and the increment: columns 0 .. KD - 1
    static constexpr uint32_t kRecordBytes = (kMtRecord + KD) * 4, kChunkBytes = ((OUT ? 2 : 1) * kSlabs + 2) * kMtSlab + kRecordBytes;
};

// grid (ceil(E / 128), H, B * segments)
template <typename T, int KD, bool OUT>
__global__ void __launch_bounds__(kMtThreads, 1) mlstm_tc_kernel(const __grid_constant__ CUtensorMap map, const MlstmStep p, const ChunkWs w) {
    using L = MtLayout<KD, OUT>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    constexpr int DQ = KD / 4, SLABS = L::kSlabs;
    __shared__ __align__(16) float record[L::kStages][kMtRecord + KD], sn[KD];
    __shared__ float f_old[kChunk], f_new[kChunk];  // what the old state's and the chunk's own part of an output are multiplied with
    __shared__ uint64_t full[L::kStages], p_full, bar_s;
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    __shared__ unsigned last_flag;

    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, b = blockIdx.z / (OUT ? w.segments : w.segments - 1), seg = blockIdx.z - b * (OUT ? w.segments : w.segments - 1), pair = b * p.H + h;
    const bool single = w.segments == 1, final_state = OUT && seg == w.segments - 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int quad = warp & 3, quarter = warp >> 2, e0 = blockIdx.x * kChunkCols, e = e0 + quad * 32 + lane, d0 = quarter * DQ;
    const float q_scale = 1.0f / sqrtf((float)p.D);
    const int c_beg = seg * w.per, c_end = min(c_beg + w.per, w.chunks);
    const uint32_t smem_base = smem_u32(smem);

    if (threadIdx.x == 0) {
        for (int i = 0; i < L::kStages; i++) mbar_init(&full[i], 1);
        mbar_init(&p_full, 1);
        mbar_init(&bar_s, 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(&tmem_slot, L::kTmemCols);
    // one thread; rows past the sequence bring its neighbour's tokens or zeros, whose weights are zero
    auto fetch = [&](int c) {
        const int buf = (c - c_beg) % L::kStages, y = b * p.S + c * kChunk, x = 2 * h * p.D;
        mbar_expect_tx(&full[buf], L::kChunkBytes);
#pragma unroll
        for (int sl = 0; sl < 2; sl++) tma_load_2d(smem + L::kV + (buf * 2 + sl) * kMtSlab, &map, 4 * p.H * p.D + 2 * (h * p.E + e0) + 128 * sl, y, &full[buf]);
        bulk_load_1d(record[buf], w.gate + ((size_t)pair * w.chunks + c) * (kMtRecord + KD), L::kRecordBytes, &full[buf]);
#pragma unroll
        for (int sl = 0; sl < SLABS; sl++) {
            if constexpr (OUT) tma_load_2d(smem + L::kQ + (buf * SLABS + sl) * kMtSlab, &map, x + 128 * sl, y, &full[buf]);  // byte map: x counts bytes
            tma_load_2d(smem + L::kK + (buf * SLABS + sl) * kMtSlab, &map, 2 * p.H * p.D + x + 128 * sl, y, &full[buf]);
        }
    };
    auto fetch_scores = [&](int c) {
        mbar_expect_tx(&p_full, kMtScoreBytes);
        bulk_load_1d(smem + L::kP, reinterpret_cast<const uint8_t *>(w.scores) + ((size_t)pair * w.chunks + c) * kMtScoreBytes, kMtScoreBytes, &p_full);
    };

    tc_fence_before();
    __syncthreads();  // barriers and the tensor memory's address are there
    tc_fence_after();
    const uint32_t tm = tmem_slot, t_lane = tm + ((uint32_t)(quad * 32) << 16);
    if (threadIdx.x == 0) {
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map) : "memory");
        for (int i = 0; i < L::kStages && c_beg + i < c_end; i++) fetch(c_beg + i);
        if constexpr (OUT) fetch_scores(c_beg);
    }
    __syncwarp();

    const size_t DE = (size_t)p.D * p.E, slot0 = (size_t)pair * w.segments;
    const bool fresh = *p.past == 0, first = single || (!OUT && seg == 0);  // starts from the state in front of the call
    // memory and sum vector to start from, and the running maximum, which every thread follows
    const float *from_s = first ? p.mem + pair * DE : w.seg_s + (slot0 + (seg == 0 ? w.segments - 1 : 0)) * DE;
    const float *from_n = first ? p.sum + (size_t)pair * p.D : w.seg_n + (slot0 + (seg == 0 ? w.segments - 1 : 0)) * p.D;
    const bool empty = first ? fresh : !OUT;
    float m0 = first ? (fresh ? 0.f : p.top[pair]) : !OUT ? -INFINITY : w.seg_m[(slot0 + (seg == 0 ? w.segments - 1 : 0)) * 2 + 1], forgotten = 0.f;
    float S[DQ];  // S[i] = memory[d0 + i][e]
    const bool in = e < p.E;
#pragma unroll
    for (int i = 0; i < DQ; i++) S[i] = !empty && in ? from_s[(size_t)(d0 + i) * p.E + e] : 0.f;
    float n = threadIdx.x < KD && !empty ? from_n[threadIdx.x] : 0.f;
    if (!OUT && seg == 0) {  // the copy for the second pass
#pragma unroll
        for (int i = 0; i < DQ; i++)
            if (in) w.seg_s[(slot0 + w.segments - 1) * DE + (size_t)(d0 + i) * p.E + e] = S[i];
        if (blockIdx.x == 0 && threadIdx.x < KD) w.seg_n[(slot0 + w.segments - 1) * p.D + threadIdx.x] = n;
        if (blockIdx.x == 0 && threadIdx.x == 0) w.seg_m[(slot0 + w.segments - 1) * 2 + 1] = m0;
    }
    if (OUT && !single)
        for (int g = 1; g < seg; g++) {
            float keep, take;
            add_segment(w, pair, g, m0, keep, take);
            const float *more = w.seg_s + (slot0 + g) * DE + (size_t)d0 * p.E + (in ? e : 0);
#pragma unroll
            for (int i = 0; i < DQ; i++) S[i] = keep * S[i] + take * more[(size_t)i * p.E];
            if (threadIdx.x < KD) n = keep * n + take * w.seg_n[(slot0 + g) * p.D + threadIdx.x];
        }
    if (threadIdx.x < KD) sn[threadIdx.x] = n;

    constexpr uint32_t ab = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;  // operand format: 0 = f16, 1 = bf16
    constexpr uint32_t kIdesc = (1u << 4) | (ab << 7) | (ab << 10) | ((uint32_t)(kChunkCols >> 4) << 24), kAmn = 1u << 15, kBmn = 1u << 16;
    auto wait = [&](uint64_t *bar, uint32_t parity) {  // whole warps
        int done = 1;
        if (lane == 0) done = mbar_wait_spin(bar, parity, &abort_flag) ? 1 : 0;
        done = __shfl_sync(0xffffffffu, done, 0);
        __syncwarp();
        return done != 0;
    };
    const int v_row = threadIdx.x >> 4, v_col = (threadIdx.x & 15) * 8;  // this thread's pieces of the value tile: rows v_row and v_row + 32
    const uint32_t v_off = slab_off(v_row, v_col);
    float o[16];  // outputs of the chunk before: this thread's column, tokens 16 quarter ..
    auto store_outputs = [&](int c) {
        const size_t step = (size_t)p.H * p.E;
        float *at = w.o + ((size_t)b * p.S + c * kChunk + 16 * quarter) * step + (size_t)h * p.E + e;
        const int n = min(16, p.S - c * kChunk - 16 * quarter);
        if (e < p.E) {
#pragma unroll
            for (int i = 0; i < 16; i++) {
                if (i < n) *at = o[i];
                at += step;
            }
        }
        __syncwarp();
    };
    bool ok = true;
    for (int c = c_beg; c < c_end; c++) {
        const int n_done = c - c_beg, buf = n_done % L::kStages;
        if (OUT && threadIdx.x == 32 && c > c_beg && c + 1 < c_end) fetch(c + 1);  // over chunk c - 1, which nothing reads any more
        __syncwarp();
        const uint32_t parity = n_done & 1, off_k = buf * SLABS * kMtSlab, off_v = buf * 2 * kMtSlab;
        // ---- operands: the memory's two parts, the weighted values' two parts ----
        if constexpr (OUT) {
#pragma unroll
            for (int g = 0; g < DQ / 32; g++) {
                uint32_t hi[16], lo[16];
#pragma unroll
                for (int i = 0; i < 16; i++) split_pack<T>(S[32 * g + 2 * i], S[32 * g + 2 * i + 1], hi[i], lo[i]);
                tmem_st16(t_lane + quarter * DQ + 16 * g, hi);
                tmem_st16(t_lane + quarter * DQ + DQ / 2 + 16 * g, lo);
            }
        }
        ok = wait(&full[buf], (n_done / L::kStages) & 1);
        const float *ga = record[buf], *gb = ga + kChunk, *gc = gb + kChunk, *gp = gc + kChunk, *gn = gp + kChunk;
        const float last = gc[kChunk - 1], b_last = gb[kChunk - 1], end_top = fmaxf(m0, last), keep = __expf(m0 - end_top), add = __expf(last - end_top);
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int s = v_row + 32 * j;
            const uint32_t off = v_off + 32 * 128 * j;
            const uint4 raw = *reinterpret_cast<const uint4 *>(smem + L::kV + off_v + off);
            const T *x = reinterpret_cast<const T *>(&raw);
            const float f = __expf(ga[s] - last);
            uint4 hi, lo;
            split_pack<T>(to_f32<T>(x[0]) * f, to_f32<T>(x[1]) * f, hi.x, lo.x);
            split_pack<T>(to_f32<T>(x[2]) * f, to_f32<T>(x[3]) * f, hi.y, lo.y);
            split_pack<T>(to_f32<T>(x[4]) * f, to_f32<T>(x[5]) * f, hi.z, lo.z);
            split_pack<T>(to_f32<T>(x[6]) * f, to_f32<T>(x[7]) * f, hi.w, lo.w);
            *reinterpret_cast<uint4 *>(smem + L::kVw + off) = hi;
            *reinterpret_cast<uint4 *>(smem + L::kVw + 2 * kMtSlab + off) = lo;
        }
        if constexpr (OUT) tmem_st_wait();
        fence_proxy_async_smem();
        tc_fence_before();
        if (__syncthreads_or(!ok)) {  // operands and n are in place; chunk c - 1 has been read by all
            ok = false;
            break;
        }
        if (threadIdx.x == 0) {
            tc_fence_after();
            if constexpr (OUT) {
                ok = mbar_wait_spin(&p_full, parity, &abort_flag);
                constexpr uint32_t idesc = kIdesc | ((uint32_t)(kChunk >> 3) << 17);
                const uint64_t dq = make_kmajor_sw128_desc(smem_base + L::kQ + off_k);
                const uint64_t dv = make_sw128_desc(smem_base + L::kV + off_v, kMtSlab, 1024), dp = make_kmajor_sw128_desc(smem_base + L::kP);
#pragma unroll
                for (int i = 0; i < 2 * (kChunk / 16); i++) {
                    const int hp = i / (kChunk / 16), ks = i % (kChunk / 16);
                    umma_f16(tm + L::kColPv, dv + (uint64_t)((ks * 2048) >> 4), dp + (uint64_t)((hp * kMtSlab + ks * 32) >> 4), idesc | kAmn, i ? 1u : 0u);
                }
#pragma unroll
                for (int i = 0; i < 2 * (KD / 16); i++) {
                    const int hp = i / (KD / 16), ks = i % (KD / 16);
                    umma_f16_ta(tm + L::kColInter, tm + (ks / (DQ / 16)) * DQ + hp * (DQ / 2) + (ks % (DQ / 16)) * 8,
                                dq + (uint64_t)(((ks >> 2) * kMtSlab + (ks & 3) * 32) >> 4), idesc, i ? 1u : 0u);
                }
            }
            constexpr uint32_t idesc = kIdesc | kAmn | kBmn | ((uint32_t)(KD >> 3) << 17);
            const uint64_t da = make_sw128_desc(smem_base + L::kVw, kMtSlab, 1024), db = make_sw128_desc(smem_base + L::kK + off_k, kMtSlab, 1024);
#pragma unroll
            for (int i = 0; i < 2 * (kChunk / 16); i++) {
                const int hp = i / (kChunk / 16), ks = i % (kChunk / 16);
                umma_f16(tm, da + (uint64_t)((hp * 2 * kMtSlab + ks * 2048) >> 4), db + (uint64_t)((ks * 2048) >> 4), idesc, i ? 1u : 0u);
            }
            umma_commit(&bar_s);
        } else if (!OUT && threadIdx.x == 32 && c > c_beg && c + 2 < c_end) {
            fetch(c + 2);  // over chunk c - 1
        }
        ok = __all_sync(0xffffffffu, ok);  // whole warps go on together
        if constexpr (OUT) {
            // q.n_0 of four tokens per warp, eight lanes each; the factors of a token's outputs
            const int t = 4 * warp + (lane >> 3), part = lane & 7;
            float qn = 0.f;
#pragma unroll
            for (int sl = 0; sl < SLABS; sl++) {
                const uint4 raw = *reinterpret_cast<const uint4 *>(smem + L::kQ + off_k + slab_off(t, 64 * sl + 8 * part));
                const T *x = reinterpret_cast<const T *>(&raw);
                const float4 n0 = *reinterpret_cast<const float4 *>(&sn[64 * sl + 8 * part]), n1 = *reinterpret_cast<const float4 *>(&sn[64 * sl + 8 * part + 4]);
                qn += to_f32<T>(x[0]) * n0.x + to_f32<T>(x[1]) * n0.y + to_f32<T>(x[2]) * n0.z + to_f32<T>(x[3]) * n0.w;
                qn += to_f32<T>(x[4]) * n1.x + to_f32<T>(x[5]) * n1.y + to_f32<T>(x[6]) * n1.z + to_f32<T>(x[7]) * n1.w;
            }
#pragma unroll
            for (int s = 1; s < 8; s <<= 1) qn += __shfl_xor_sync(0xffffffffu, qn, s);
            if (part == 0) {
                const float top = fmaxf(m0, gc[t]), fo = __expf(m0 - top) * q_scale, fn = __expf(gc[t] - top), den = fo * qn + fn * gp[t];
                const float inv = 1.0f / (fmaxf(fabsf(den), expf(-(gb[t] + top))) + kMlstmFloor);
                f_old[t] = fo * inv;
                f_new[t] = fn * inv;
            }
            __syncwarp();
            if (c > c_beg) store_outputs(c - 1);
        }
        // ---- state at the chunk's end ----
        ok = wait(&bar_s, parity) && ok;
        tc_fence_after();
        if (ok) {
#pragma unroll
            for (int g = 0; g < DQ / 32; g++) {
                float u[32];
                tmem_ld32(t_lane + quarter * DQ + 32 * g, reinterpret_cast<uint32_t *>(u));
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; i++) S[32 * g + i] = keep * S[32 * g + i] + add * u[i];
            }
        }
        const float n_add = threadIdx.x < KD ? gn[threadIdx.x] : 0.f;
        if constexpr (OUT) {
            if (threadIdx.x == 0 && c + 1 < c_end && ok) fetch_scores(c + 1);
            __syncwarp();
            uint32_t x[16], y[16];
            tmem_ld16(t_lane + L::kColInter + 16 * quarter, x);
            tmem_ld16(t_lane + L::kColPv + 16 * quarter, y);
            tmem_ld_wait();
            tc_fence_before();
            if (__syncthreads_or(!ok)) {
                ok = false;
                break;
            }
#pragma unroll
            for (int i = 0; i < 16; i++) o[i] = f_old[16 * quarter + i] * __uint_as_float(x[i]) + f_new[16 * quarter + i] * __uint_as_float(y[i]);
        }
        if (threadIdx.x < KD) sn[threadIdx.x] = keep * sn[threadIdx.x] + add * n_add;
        forgotten += b_last;
        m0 = b_last + end_top;
    }
    if (!ok && threadIdx.x == 0) {
        atomicExch(&abort_flag, 1);
        atomicExch(p.status, OUT ? 51 : 52);
    }
    if (OUT && ok) store_outputs(c_end - 1);
    if (!OUT || final_state) {
        float *to_s = OUT ? p.mem + pair * DE : w.seg_s + (slot0 + seg) * DE;
#pragma unroll
        for (int i = 0; i < DQ; i++)
            if (in) to_s[(size_t)(d0 + i) * p.E + e] = S[i];
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tm, L::kTmemCols);
    if (OUT && !final_state) return;
    if (OUT && single) {
        if (!last_of_head(p, pair, gridDim.x, &last_flag)) return;
    } else if (blockIdx.x != 0) {
        return;
    }
    float *to_n = OUT ? p.sum + (size_t)pair * p.D : w.seg_n + (slot0 + seg) * p.D;
    if (threadIdx.x < KD) to_n[threadIdx.x] = sn[threadIdx.x];
    if (threadIdx.x == 0) {
        if (OUT) p.top[pair] = m0;
        else w.seg_m[(slot0 + seg) * 2] = forgotten, w.seg_m[(slot0 + seg) * 2 + 1] = m0;
    }
}

bool mlstm_tc_supported(int dtype, const MlstmStep &p) {
    return dtype != MYNN_F32 && p.status && (p.D == 128 || p.D == 256) && p.E >= 64 && p.E % 8 == 0 && (uintptr_t)p.proj % 16 == 0 && tensor_map_api_available() &&
           (long long)p.B * p.S < (1ll << 31);
}

template <typename T, int KD, bool OUT>
static int run_mt(cudaStream_t st, const MlstmStep &p, const ChunkWs &w) {
    constexpr size_t smem = MtLayout<KD, OUT>::kBytes + 1024;
    static_assert(smem + 10 * 1024 <= 227 * 1024, "shared memory of a CTA");
    auto kern = mlstm_tc_kernel<T, KD, OUT>;
    static bool attr_set = false;
    if (!attr_set) {
        MYNN_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set = true;
    }
    CUtensorMap map;
    const uint64_t row = (uint64_t)2 * p.H * (p.D + p.E) * 2;
    if (int rc = make_map(&map, p.proj, (uint64_t)p.B * p.S, row, row, kChunk)) return rc;
    kern<<<dim3((p.E + kChunkCols - 1) / kChunkCols, p.H, p.B * (OUT ? w.segments : w.segments - 1)), kMtThreads, smem, st>>>(map, p, w);
    MYNN_LAUNCH_OK("mlstm_tc_kernel");
    return MYNN_OK;
}

template <typename T, int KD>
static int run_prepare(cudaStream_t st, const MlstmStep &p, const ChunkWs &w) {
    constexpr size_t smem = 2 * (KD / 64) * kMtSlab + 1024;
    auto kern = mlstm_prepare_kernel<T, KD>;
    static bool attr_set = false;
    if (!attr_set) {
        MYNN_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set = true;
    }
    kern<<<dim3(w.chunks, p.H, p.B), 256, smem, st>>>(p, w);
    MYNN_LAUNCH_OK("mlstm_prepare_kernel");
    return MYNN_OK;
}

int launch_mlstm_prepare(cudaStream_t st, int dtype, const MlstmStep &p, const ChunkWs &w) {
    if (!mlstm_tc_supported(dtype, p)) return fail(MYNN_E_UNSUPPORTED, "mlstm: not a shape of the tcgen05 kernel");
    if (dtype == MYNN_BF16) return p.D == 128 ? run_prepare<__nv_bfloat16, 128>(st, p, w) : run_prepare<__nv_bfloat16, 256>(st, p, w);
    return p.D == 128 ? run_prepare<__half, 128>(st, p, w) : run_prepare<__half, 256>(st, p, w);
}

int launch_mlstm_tc(cudaStream_t st, int dtype, const MlstmStep &p, const ChunkWs &w, bool out) {
    if (!mlstm_tc_supported(dtype, p)) return fail(MYNN_E_UNSUPPORTED, "mlstm: not a shape of the tcgen05 kernel");
    if (dtype == MYNN_BF16) {
        using T = __nv_bfloat16;
        if (p.D == 128) return out ? run_mt<T, 128, true>(st, p, w) : run_mt<T, 128, false>(st, p, w);
        return out ? run_mt<T, 256, true>(st, p, w) : run_mt<T, 256, false>(st, p, w);
    }
    using T = __half;
    if (p.D == 128) return out ? run_mt<T, 128, true>(st, p, w) : run_mt<T, 128, false>(st, p, w);
    return out ? run_mt<T, 256, true>(st, p, w) : run_mt<T, 256, false>(st, p, w);
}

}  // namespace mynn
