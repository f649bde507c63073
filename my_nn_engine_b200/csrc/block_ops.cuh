// Operators of the block decoder (block_model.cu): norms with their residual step, the short causal convolution or the rotation with
// the append to the caches, windowed and chunked attention, attention over latents, matrix memory, expert routing, and dense / grouped
// matrix products over unquantised weights.  Every size and constant is a parameter; nothing here knows a particular model.
#pragma once
#include <cuda_runtime.h>
#include <stddef.h>
#include <stdint.h>

#include "../../include/mynn_b200.h"

namespace mynn {

// ---- layer_norm.cu ---------------------------------------------------------------------------------------------------
// One step of the residual stream x (f32 [rows, W]), in this order, every part optional:
//   x  = embed[ids] * embed_scale                         (embed != null; also copied to x0 when that is given)
//   x += mult * LN(sub; w1, b1)                           (sub != null: one row of dtype per row of x)
//        with pair_row: sub := sum_s pair_w[row, s] * sub[pair_row[row, s]]   (combination of routed experts)
//   x += x0                                               (add_x0)
//   out = LN(x; w2, b2) in dtype                          (out != null)
// row_map: rows of `out` are taken from rows row_map[i] of x and x is left alone (head of the model).
// LN(v; w, b) = (v - mean) / sqrt(var + eps) * w + b in f32, var = mean of the squared deviations; w, b f32 [W].
// rms: the norms are v / sqrt(mean(v^2) + eps) * w instead (b is not read).  w1 == null: the sublayer output is added as it is.
struct NormStep {
    const void *embed = nullptr;
    const int64_t *ids = nullptr;
    float embed_scale = 1.f;
    int vocab = 0;
    float *x = nullptr, *x0 = nullptr;
    const void *sub = nullptr;
    const int32_t *pair_row = nullptr;
    const float *pair_w = nullptr;
    int top = 0;
    const float *w1 = nullptr, *b1 = nullptr, *w2 = nullptr, *b2 = nullptr;
    float mult = 1.f, eps = 0.f;
    int add_x0 = 0;
    int rms = 0;
    void *out = nullptr;
    const int32_t *row_map = nullptr;
    int W = 0;
};
int launch_norm_step(cudaStream_t st, int dtype, const NormStep &p, int rows);

// ---- short_conv.cu ---------------------------------------------------------------------------------------------------
// The projection rows of S new tokens of B sequences, proj [B * S, C] with C = Hq*D + G*D + G*E (q, k, v), go through the
// causal convolution y_t[c] = sum_j w[j, c] u_{t-taps+1+j}[c] (f32 [taps, C]; taps == 0: none), q and k through the interleaved
// rotation of the first rot_dims dimensions of each head (cos / sin f32 [positions, rot_dims / 2]), and on to
//   q_out [B, Hq, S, D],  k_cache [B, G, cache_rows, D],  v_cache [B, G, cache_rows, E]  (position p in row p % cache_rows).
// hist [B, hist_rows, C] keeps the unconvolved projection of the last hist_rows positions (position p in row p % hist_rows,
// hist_rows >= taps).  The new tokens sit at positions *past .. *past + S - 1; positions before 0 count as zero.
struct ConvStep {
    const void *proj = nullptr;
    void *hist = nullptr;
    int hist_rows = 0;
    const float *w = nullptr;
    int taps = 0;
    const float *cos_t = nullptr, *sin_t = nullptr;
    int rot_dims = 0;
    void *q_out = nullptr, *k_cache = nullptr, *v_cache = nullptr;
    int cache_rows = 0;
    int B = 0, S = 0, Hq = 0, G = 0, D = 0, E = 0;
    const int32_t *past = nullptr;
};
int launch_conv_step(cudaStream_t st, int dtype, const ConvStep &p);

// ---- attention_window.cu ---------------------------------------------------------------------------------------------
// Causal attention over ring caches: query row s of a sequence sits at position *active - Sq + s and sees the `window` positions
// up to and including its own (window <= 0: all of them); position p is read from cache row p % cache_rows.  Scores are
// scale * q.k, then softcap * tanh(score / softcap) when softcap > 0.  q [B, Hq, Sq, D]; out [B, Sq, Hq, E].
// chunk > 0: positions are cut into chunks of that many from position 0 on, and a query sees no key before its own chunk.
// layout: 0 q [B, Hq, Sq, D] and caches [B, Hkv, rows, .]; 1 head-major q [Hq, B, Sq, D] and caches [Hkv, B, rows, .]; 2 token-major
// q [B, Sq, Hq, D] (caches as in 0; the kernel for any sizes only).
enum { kByBatch = 0, kByHead = 1, kByToken = 2 };
struct WindowAttention {
    void *out = nullptr;
    const void *q = nullptr, *k = nullptr, *v = nullptr;
    float scale = 1.f, softcap = 0.f;
    int window = 0, chunk = 0;
    int layout = kByBatch;
    int B = 0, Hq = 0, Hkv = 0, Sq = 0, D = 0, E = 0, cache_rows = 0;
    int active_host = 0;               // used when active == null
    const int32_t *active = nullptr;   // device: positions written so far, the new rows included
    void *workspace = nullptr;
    size_t workspace_bytes = 0;
    int *status_word = nullptr;
};
int launch_window_attention(cudaStream_t st, int dtype, const WindowAttention &p);
// The kernel for any sizes and dtypes, whatever the tuned ones would take.
int launch_window_attention_plain(cudaStream_t st, int dtype, const WindowAttention &p);
// Tensor-core forms (attention.cu, attention_prefill_tc.cu); they return MYNN_E_UNSUPPORTED for shapes they do not take.
bool window_attention_decode_supported(int dtype, const WindowAttention &p);
int launch_window_attention_decode(cudaStream_t st, int dtype, const WindowAttention &p);
bool window_attention_prefill_supported(int dtype, const WindowAttention &p);
int launch_window_attention_prefill(cudaStream_t st, int dtype, const WindowAttention &p);
// First position that the query at position `pos` sees.
__host__ __device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
    int lo = window > 0 && pos >= window ? pos - window + 1 : 0;
    if (chunk > 0) {
        const int c = pos - pos % chunk;
        lo = lo > c ? lo : c;
    }
    return lo;
}

// ---- rotary_append.cu ------------------------------------------------------------------------------------------------
// The same step without a convolution, one head per warp: the projection rows of S new tokens of B sequences, proj
// [B * S, Hq*D + G*D + G*E], through the rotation of the first rot_dims dimensions of every q and k head (halves: dimension i pairs
// with i + rot_dims / 2, else 2i with 2i + 1), then, with qk_norm, each q and k head over its root mean square
// (v / sqrt(mean(v^2) + eps), no weight), and on to q_out [B, Hq, S, D] and the ring caches.
struct RotaryAppend {
    const void *proj = nullptr;
    const float *cos_t = nullptr, *sin_t = nullptr;  // f32 [positions, rot_dims / 2]
    int rot_dims = 0, halves = 0, qk_norm = 0;
    float eps = 0.f;
    void *q_out = nullptr, *k_cache = nullptr, *v_cache = nullptr;
    int cache_rows = 0;
    int B = 0, S = 0, Hq = 0, G = 0, D = 0, E = 0;
    const int32_t *past = nullptr;
};
int launch_rotary_append(cudaStream_t st, int dtype, const RotaryAppend &p);

// ---- latent_attention.cu ---------------------------------------------------------------------------------------------
// proj [B * S, Q + R] of S new tokens: the first Q columns RMS-normed with weight wq into q_out [B * S, Q], the other R with weight wc
// into the ring of latents cache [B, cache_rows, R] (position p in row p % cache_rows).
struct LatentAppend {
    const void *proj = nullptr;
    const float *wq = nullptr, *wc = nullptr;
    float eps = 0.f;
    void *q_out = nullptr, *cache = nullptr;
    int B = 0, S = 0, Q = 0, R = 0, cache_rows = 0;
    const int32_t *past = nullptr;
};
int launch_latent_append(cudaStream_t st, int dtype, const LatentAppend &p);
// Attention of H heads over one shared latent row per position: q [B, Sq, H, R] (queries brought into latent space), keys and values
// are both the cached rows [B, cache_rows, R]; out [B, Sq, H, R] is the weighted mean of latents.  Causal, positions as for
// WindowAttention.  The tensor-core kernel takes 16-bit latents of 128, 256 or 512; everything else goes to the window kernel for any sizes.
struct LatentAttention {
    void *out = nullptr;
    const void *q = nullptr, *c = nullptr;
    float scale = 1.f;
    int B = 0, Sq = 0, H = 0, R = 0, cache_rows = 0;
    int active_host = 0;
    const int32_t *active = nullptr;
    void *workspace = nullptr;  // latent_attention_workspace_bytes; without it one CTA walks all positions of a query
    size_t workspace_bytes = 0;
};
size_t latent_attention_workspace_bytes(int B, int Sq, int H, int R, int cache_rows);
int launch_latent_attention(cudaStream_t st, int dtype, const LatentAttention &p, bool plain = false);

// ---- mlstm.cu --------------------------------------------------------------------------------------------------------
// Matrix memory with exponential gates (mLSTM).  proj [B * S, 2 H D + 2 H E] holds q, k, v and the output gate's logits z, gates f32
// [B * S, 2 H] the input and forget gates' products, gate_bias f32 [2 H] what is added to them.  Per head, from zero state:
//   i = cap tanh((gates_i + bias_i) / cap),  f = log sigmoid(cap tanh((gates_f + bias_f) / cap)),  m' = max(f + m, i),
//   S' = e^(f + m - m') S + e^(i - m') k v^T,  n' = e^(f + m - m') n + e^(i - m') k,
//   o = S'^T q~ / (max(|n'.q~|, e^-m') + 1e-6),  q~ = q / sqrt(D)
//   out = o / sqrt(mean(o^2) + eps) * norm_w * sigmoid(z)                                  (norm_w f32 [H E])
// State f32, read and written in place: mem [B, H, D, E], sum [B, H, D], top [B, H] (m, from 0).  A step at position 0 (*past == 0)
// starts from zero whatever the buffers hold.
struct MlstmStep {
    const void *proj = nullptr;
    const float *gates = nullptr, *gate_bias = nullptr, *norm_w = nullptr;
    float cap = 1.f, eps = 0.f;
    float *mem = nullptr, *sum = nullptr, *top = nullptr;
    float *workspace = nullptr;  // mlstm_workspace_bytes; begins with o, f32 [B * S, H E]
    size_t workspace_bytes = 0;
    unsigned *ticket = nullptr;  // scratch [B * H], zero between calls
    void *out = nullptr;         // [B * S, H E]
    int B = 0, S = 0, H = 0, D = 0, E = 0;
    const int32_t *past = nullptr;
    int form = 0;                // 0: by size, 1: token by token, 2: chunkwise on mma.sync, 3: chunkwise on tcgen05 (both 16-bit)
    int *status = nullptr;       // status word of the bounded waits (tcgen05 form only)
};
int launch_mlstm(cudaStream_t st, int dtype, const MlstmStep &p);
bool mlstm_chunkwise_supported(int dtype, const MlstmStep &p);
size_t mlstm_workspace_bytes(int dtype, int B, int S, int H, int D, int E);

// ---- moe_route.cu ----------------------------------------------------------------------------------------------------
// Expert choice of M tokens from f32 logits [M, E]: s = softmax(z); of `groups` equal groups of neighbouring experts the `keep`
// with the largest member stay; the `top` largest s among their experts are chosen, weight s (not renormalised).  The
// (token, slot) pairs are then ordered by expert.
struct MoeRoute {
    float *pair_w;      // [M, top] weights
    int32_t *pair_row;  // [M, top] place of the pair in the expert order
    int32_t *pair_e;    // [M, top] chosen expert
    int32_t *tok_of;    // [M * top] token of the pair at that place
    int32_t *off;       // [E + 1] first place of every expert
    int32_t *active;    // [E] experts with at least one pair
    int32_t *n_active;  // [1]
    int32_t *count;     // [E] scratch, zero between calls
    int32_t *tile_e, *tile_row, *n_tiles;  // tiles of kMoeTileRows places that do not cross experts (tensor-core kernel)
};
constexpr int kMoeTileRows = 128;
size_t moe_route_bytes(int M, int experts, int top);
MoeRoute moe_route_bind(void *base, int M, int experts, int top);
int launch_moe_route(cudaStream_t st, const MoeRoute &r, const float *logits, int M, int experts, int top, int groups, int keep);

// ---- dense_gemm.cu / dense_gemm_tc.cu --------------------------------------------------------------------------------
// out[m, n] = sum_k act[m, k] w[n, k], f32 accumulation, weights in `dtype`, out in out_dtype.
//   glu:      w holds 2 N rows (N gate rows, then N up rows); out[m, n] = silu(gate) * up
//   experts:  w holds `experts` such blocks; the rows are the (token, slot) places of `route`, place r of expert e is multiplied
//             with block e; gather: its activation row is tok_of[r], else r.  M is then the number of TOKENS and out has
//             M * top rows.
//   act_fn:   applied to the f32 sum before the store
//   out_f32:  columns from n_main on go to out_f32 [M, N - n_main] in f32 instead (no act_fn)
//   out_block: column n of row m is stored at (n / out_block) * out_block_stride + m * ldo + n % out_block (one block per head, say)
//   batch:    independent products side by side (rows of act lda apart, product z at act + z * act_stride, w + z * N * K,
//             out + z * out_stride); not on the tensor-memory kernel
//   row_groups: the rows come in that many groups of M, group r at rows r * group_rows .. of act and out (the live rows of every sequence's
//             cache, say)
enum { kActNone = MYNN_ACT_NONE, kActSquareRelu = MYNN_ACT_SQUARE_RELU };
struct DenseGemm {
    void *out = nullptr;
    const void *act = nullptr, *w = nullptr;
    int M = 0, N = 0, K = 0;
    int out_dtype = 0;
    int glu = 0;
    const MoeRoute *route = nullptr;
    int experts = 1, top = 1, gather = 0;
    void *gather_ws = nullptr;  // [M * top, K] of dtype: sorted copy of the gathered rows (tensor-core kernel only)
    int *status = nullptr;      // status word of the bounded waits (tensor-core kernel only)
    int act_fn = kActNone;
    float *out_f32 = nullptr;
    int n_main = 0;             // used with out_f32
    int out_block = 0;
    long long out_block_stride = 0;
    int lda = 0, ldo = 0;       // row strides in elements, 0: K and N (n_main with out_f32)
    int batch = 1;
    long long act_stride = 0, out_stride = 0;
    int row_groups = 1;
    long long group_rows = 0;
};
__device__ __forceinline__ float dense_act(float v, int fn) {
    if (fn == kActSquareRelu) {
        v = fmaxf(v, 0.f);
        v *= v;
    }
    return v;
}
int launch_dense_gemm(cudaStream_t st, int dtype, const DenseGemm &g);
bool dense_gemm_tc_supported(int dtype, const DenseGemm &g);
int launch_dense_gemm_tc(cudaStream_t st, int dtype, const DenseGemm &g);

}  // namespace mynn
