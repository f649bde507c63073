// State of a model behind the model_init / model / model_destroy entry points, shared by the graphs that step it: the Llama-family
// int8 graph (model.cu) and the block decoder (block_model.cu).
#pragma once
#include <cuda_runtime.h>

#include <vector>

#include "common.cuh"
#include "tp_fused.cuh"

namespace mynn {

struct BlockModel;  // block_model.cu

struct LayerW {
    const void *ln1, *ln2;
    const int8_t *wq, *wk, *wv, *wo, *wg, *wu, *wd;
    const void *sq, *sk, *sv, *so, *sg, *su, *sd;
    void *kc, *vc;
    void *ksc, *vsc;  // per-token scales of an int8 cache
    bool qkv_fused, gu_fused;
};

struct Model {
    mynn_b200_model_config c;
    BlockModel *blocks = nullptr;  // not null: the step runs the block decoder's graph
    int logits_dtype = 0;          // dtype of the logits handed out (the storage dtype, f32 for the block decoder)
    int head_capacity = 0;         // rows of the logits buffer
    int32_t *rows_dev = nullptr;   // rows of x whose logits are wanted (several per prefill chunk)
    int Hq, Hkv, ffn, vocab_l;  // per-rank sizes
    int max_rows;               // batch * max(1, max_prefill)
    std::vector<LayerW> layers;
    const int8_t *embed;
    const void *embed_scale, *final_norm, *lm_scale, *cos_t, *sin_t;
    const int8_t *lm_w;
    // device buffers
    char *arena = nullptr;
    // step inputs, contiguous so that one host-to-device copy delivers them: {past, active, pos0, ids[rows]}
    int32_t *past_dev, *active_dev;
    int64_t *pos0_dev, *ids_dev;
    int64_t *pos_dev;  // positions of a prefill chunk
    int32_t *tok_dev;
    char *h_in = nullptr;  // pinned mirror of the input block
    int *h_status = nullptr;  // pinned: status words of the GEMM workspace and of the tensor-parallel block, fetched with the result
    void *x, *n, *qkv, *q_rot, *attn, *gu, *h, *last_x, *logits, *logits_full;
    float *part, *pairs, *pairs_all;  // part = f32 partial sums of a row-parallel product (tp_world > 1, ncclAllReduce path)
    char *tp_block = nullptr;         // cudaMalloc'd block shared with the peers (fused reduction of decode steps, tp_fused.cuh)
    size_t tp_block_bytes = 0;
    TpPeers tp = {};
    bool tp_attached = false;
    bool weights_aligned = false;  // every projection weight is 16-byte aligned (the TMA-fed kernels can take all of them)
    void *attn_ws, *gemm_ws;
    size_t attn_ws_bytes, gemm_ws_bytes;
    // streaming (sink + ring) cache: per-slot key positions and the scratch that holds one layer's rotated keys
    int64_t *kvpos_dev = nullptr;
    void *k_rot = nullptr;
    void *k_deq = nullptr, *v_deq = nullptr;  // int8 cache: 16-bit copy of one layer's live rows for the tensor-core prefill attention
    cudaGraphExec_t stream_graph_exec = nullptr;
    bool tc_attention_ran = false;  // the step just enqueued went through the tcgen05 prefill attention (its status word is checked)
    cudaStream_t stream = nullptr;
    cudaGraphExec_t graph_exec = nullptr;
};

inline size_t up256(size_t x) { return (x + 255) / 256 * 256; }

#define RC(expr)            \
    do {                    \
        int rc__ = (expr);  \
        if (rc__) return rc__; \
    } while (0)

// The block decoder as a graph of Model: validation of its configuration, building, one forward pass, and what a caller may do
// with positions.
int block_configure(const mynn_b200_block_model_config *cfg);   // keeps a copy of cfg for the next block_create
int block_create(Model &m, void **initializer, void **session_state);
void block_destroy(Model &m);
int block_forward(Model &m, cudaStream_t st, int S, int head_rows);
// past_len of the next step of T tokens against the rows the ring caches still hold; records the step
int block_admit(Model &m, int past_len, int T);

}  // namespace mynn
