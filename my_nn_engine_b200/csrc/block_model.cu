// The block decoder: a model described layer by layer (mynn_b200_block_model_config), stepped through the entry points of model.cu.
//
// A layer run is nine launches:
//     q/k/v product -> convolution + rotation + append -> attention -> output product -> [post norm, residual, norm]
//     -> router product -> expert choice -> gate/up products with SiLU gating -> down products
//     -> [combination of the experts, post norm, residual, (embedding output of a repeated pass), norm of the next layer]
// (the norm kernel closes one sublayer and opens the next).  The residual stream is f32.  Every run has ring caches of its own; a
// position's row depends on the position alone, so a chunk may be cut anywhere, and a new sequence simply starts at position 0
// again.  The decode step is captured in the CUDA graph that model.cu replays; past length and row count are device scalars.
#include <algorithm>
#include <climits>

#include "block_ops.cuh"
#include "i8_gemm.cuh"
#include "model_internal.cuh"
#include "ops_internal.cuh"

namespace mynn {

struct BlockLayer {
    mynn_b200_block c;
    const float *n1w, *n1b, *p1w, *p1b, *n2w, *n2b, *p2w, *p2b;
    const void *qkv, *o, *router, *gate_up, *down;
    const float *conv, *cos_t, *sin_t;
};
struct BlockRun {
    int layer;
    bool add_embed;  // the embedding output is added to x in front of it
    void *kc, *vc, *hist;
};
struct BlockModel {
    mynn_b200_block_model_config c;
    std::vector<BlockLayer> layers;
    std::vector<BlockRun> runs;
    const void *embed, *head;
    const float *fnw, *fnb;
    // activations
    float *x, *x0, *z;  // residual stream, embedding output (with a loop), router logits
    void *h, *proj, *q, *attn, *sub, *hidden, *gathered, *route;
    int32_t *last_rows;  // row of every sequence's last token in a chunk
    // what the rings hold: positions stored since the sequence began, and the most that were ever stored in it
    int stored = 0, high = 0, slack = INT_MAX;
};

static mynn_b200_block_model_config g_blocks_cfg;
static std::vector<mynn_b200_block> g_blocks_layers;

static int columns(const mynn_b200_block &b) { return b.heads * b.dim + b.kv_heads * (b.dim + b.vdim); }

int block_configure(const mynn_b200_block_model_config *cfg) {
    if (!cfg || !cfg->layers) return fail(MYNN_E_ARG, "model_configure_blocks: null config");
    const mynn_b200_block_model_config &c = *cfg;
    if (c.n_layers <= 0 || c.hidden <= 0 || c.vocab <= 0 || c.max_seq_len <= 0 || c.batch <= 0 || c.max_prefill < 0 || c.max_rewind < 0)
        return fail(MYNN_E_ARG, "model_configure_blocks: non-positive dimension");
    if (!dtype_ok(c.dtype)) return fail(MYNN_E_ARG, "model_configure_blocks: bad dtype %d", c.dtype);
    if (c.output_mode != 0 && c.output_mode != 1) return fail(MYNN_E_ARG, "model_configure_blocks: bad output mode %d", c.output_mode);
    if (c.loop_times > 1 && (c.loop_start < 0 || c.loop_stop <= c.loop_start || c.loop_stop > c.n_layers))
        return fail(MYNN_E_ARG, "model_configure_blocks: loop over layers [%d, %d) of %d", c.loop_start, c.loop_stop, c.n_layers);
    const int chunk = std::max(c.max_prefill, 1);
    for (int l = 0; l < c.n_layers; l++) {
        const mynn_b200_block &b = c.layers[l];
        if (b.heads <= 0 || b.kv_heads <= 0 || b.dim <= 0 || b.vdim <= 0 || b.heads % b.kv_heads)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d has %d heads of %d over %d kv heads of %d", l, b.heads, b.dim, b.kv_heads, b.vdim);
        if (b.conv_taps < 0 || b.rot_dims < 0 || b.rot_dims % 2 || b.rot_dims > b.dim || b.window < 0 || b.softcap < 0.f)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: taps %d, rotated dims %d, window %d, soft cap %g", l, b.conv_taps, b.rot_dims, b.window, b.softcap);
        const long long need = b.window > 0 ? std::min<long long>(c.max_seq_len, (long long)b.window - 1 + chunk + c.max_rewind) : c.max_seq_len;
        if (b.cache_rows < need || b.cache_rows % 128)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: %d cache rows, a multiple of 128 of at least %lld is needed", l, b.cache_rows, need);
        if (b.conv_taps && b.history_rows < b.conv_taps + c.max_rewind)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: %d history rows, %d are needed", l, b.history_rows, b.conv_taps + c.max_rewind);
        if (b.experts < 0 || (b.experts > 0 && (b.expert_ff <= 0 || b.top <= 0 || b.top > 32 || b.groups <= 0 || b.groups > 64 || b.experts % b.groups ||
                                                b.experts > 1024 || b.groups_keep <= 0 || b.groups_keep > b.groups || b.top > b.groups_keep * (b.experts / b.groups))))
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: %d experts of %d, top %d, %d of %d groups", l, b.experts, b.expert_ff, b.top, b.groups_keep, b.groups);
    }
    g_blocks_layers.assign(c.layers, c.layers + c.n_layers);
    g_blocks_cfg = c;
    g_blocks_cfg.layers = nullptr;
    return MYNN_OK;
}

int block_create(Model &m, void **initializer, void **session_state) {
    m.blocks = new BlockModel();
    BlockModel &b = *m.blocks;
    b.c = g_blocks_cfg;
    const mynn_b200_block_model_config &c = b.c;
    m.logits_dtype = MYNN_F32;
    m.vocab_l = c.vocab;
    int i = 0;
    bool missing = false;
    auto take = [&](bool wanted = true) -> const void * {
        const void *p = initializer[i++];
        if (wanted && !p) missing = true;
        return wanted ? p : nullptr;
    };
    b.embed = take();
    for (const mynn_b200_block &lc : g_blocks_layers) {
        BlockLayer L;
        L.c = lc;
        const bool ff = lc.experts > 0;
        L.n1w = (const float *)take(), L.n1b = (const float *)take(), L.p1w = (const float *)take(), L.p1b = (const float *)take();
        L.qkv = take();
        L.conv = (const float *)take(lc.conv_taps > 0);
        L.o = take();
        L.cos_t = (const float *)take(lc.rot_dims > 0), L.sin_t = (const float *)take(lc.rot_dims > 0);
        L.n2w = (const float *)take(ff), L.n2b = (const float *)take(ff), L.p2w = (const float *)take(ff), L.p2b = (const float *)take(ff);
        L.router = take(ff), L.gate_up = take(ff), L.down = take(ff);
        b.layers.push_back(L);
    }
    b.fnw = (const float *)take(), b.fnb = (const float *)take();
    b.head = take();
    if (missing) return fail(MYNN_E_ARG, "model_init: an initializer is null");
    const int times = c.loop_times > 1 ? c.loop_times : 1;
    auto add_run = [&](int l, bool add) { b.runs.push_back({l, add, nullptr, nullptr, nullptr}); };
    if (times == 1) {
        for (int l = 0; l < c.n_layers; l++) add_run(l, false);
    } else {
        for (int l = 0; l < c.loop_start; l++) add_run(l, false);
        for (int t = 0; t < times; t++)
            for (int l = c.loop_start; l < c.loop_stop; l++) add_run(l, t > 0 && l == c.loop_start);
        for (int l = c.loop_stop; l < c.n_layers; l++) add_run(l, false);
    }
    for (size_t r = 0; r < b.runs.size(); r++) {
        BlockRun &run = b.runs[r];
        const mynn_b200_block &lc = b.layers[run.layer].c;
        run.kc = session_state[3 * r];
        run.vc = session_state[3 * r + 1];
        run.hist = session_state[3 * r + 2];
        if (!run.kc || !run.vc || (lc.conv_taps && !run.hist)) return fail(MYNN_E_ARG, "model_init: a state buffer of layer run %zu is null", r);
        // how far past_len may fall behind the most positions ever stored before a ring has dropped what a step needs
        if (lc.window > 0 && lc.cache_rows < c.max_seq_len) b.slack = std::min(b.slack, lc.cache_rows - lc.window + 1);
        if (lc.conv_taps && lc.history_rows < c.max_seq_len) b.slack = std::min(b.slack, lc.history_rows - lc.conv_taps + 1);
    }
    // ---- arena ----
    const int chunk = std::max(c.max_prefill, 1);
    const size_t R = m.max_rows, esz = dtype_size(c.dtype), H = c.hidden;
    m.head_capacity = std::max(c.batch, std::min(64, m.max_rows));
    size_t col = 0, qn = 0, an = 0, pairs_ff = 0, pairs_h = 0, gat = 0, route = 0, zn = 0, aws = 0;
    for (const BlockLayer &L : b.layers) {
        const mynn_b200_block &l = L.c;
        col = std::max(col, (size_t)columns(l));
        qn = std::max(qn, (size_t)l.heads * l.dim);
        an = std::max(an, (size_t)l.heads * l.vdim);
        aws = std::max(aws, mynn_b200_attention_workspace_bytes(c.batch, l.heads, l.kv_heads, l.dim, l.cache_rows));
        if (l.experts) {
            pairs_ff = std::max(pairs_ff, R * l.top * (size_t)l.expert_ff);
            pairs_h = std::max(pairs_h, R * l.top * H);
            route = std::max(route, moe_route_bytes(m.max_rows, l.experts, l.top));
            zn = std::max(zn, R * (size_t)l.experts);
            if (c.dtype != MYNN_F32 && m.max_rows > 64) gat = pairs_h;
        }
    }
    size_t off = 0;
    auto area = [&](size_t bytes) {
        const size_t o = off;
        off += up256(bytes);
        return o;
    };
    const size_t o_in = area(16 + R * 8), o_pos = area((size_t)chunk * 8), o_tok = area((size_t)c.batch * 4), o_x = area(R * H * 4),
                 o_x0 = area(times > 1 ? R * H * 4 : 0), o_h = area(std::max(R, (size_t)m.head_capacity) * H * esz), o_proj = area(R * col * esz),
                 o_q = area(R * qn * esz), o_attn = area(R * an * esz), o_sub = area(std::max(R * H, pairs_h) * esz), o_hid = area(pairs_ff * esz),
                 o_gat = area(gat * esz), o_route = area(route), o_z = area(zn * 4), o_log = area((size_t)m.head_capacity * c.vocab * 4),
                 o_rows = area((size_t)m.head_capacity * 4), o_last = area((size_t)c.batch * 4), o_pairs = area((size_t)c.batch * 8 * 16), o_aws = area(aws),
                 o_stat = area(512);
    cudaError_t e = cudaMalloc(&m.arena, off);
    if (e != cudaSuccess) return fail(MYNN_E_CUDA, "model_init: cudaMalloc(%zu) failed: %s", off, cudaGetErrorString(e));
    MYNN_CUDA_OK(cudaMemset(m.arena, 0, off));
    char *a = m.arena;
    m.past_dev = (int32_t *)(a + o_in);
    m.active_dev = (int32_t *)(a + o_in + 4);
    m.pos0_dev = (int64_t *)(a + o_in + 8);
    m.ids_dev = (int64_t *)(a + o_in + 16);
    m.pos_dev = (int64_t *)(a + o_pos);
    m.tok_dev = (int32_t *)(a + o_tok);
    m.logits = a + o_log;
    m.rows_dev = (int32_t *)(a + o_rows);
    m.pairs_all = (float *)(a + o_pairs);
    m.attn_ws = a + o_aws;
    m.attn_ws_bytes = aws;
    m.gemm_ws = a + o_stat;  // only its status word is used; the step's end reads it
    m.gemm_ws_bytes = 512;
    b.x = (float *)(a + o_x);
    b.x0 = times > 1 ? (float *)(a + o_x0) : nullptr;
    b.h = a + o_h;
    b.proj = a + o_proj;
    b.q = a + o_q;
    b.attn = a + o_attn;
    b.sub = a + o_sub;
    b.hidden = a + o_hid;
    b.gathered = gat ? a + o_gat : nullptr;
    b.route = a + o_route;
    b.z = (float *)(a + o_z);
    b.last_rows = (int32_t *)(a + o_last);
    return MYNN_OK;
}

void block_destroy(Model &m) {
    delete m.blocks;
    m.blocks = nullptr;
}

int block_admit(Model &m, int past_len, int T) {
    BlockModel &b = *m.blocks;
    if (past_len == 0) b.stored = b.high = 0;
    if (past_len > b.stored) return fail(MYNN_E_STATE, "step at position %d, but only %d positions are stored", past_len, b.stored);
    if ((long long)past_len < (long long)b.high - b.slack) return fail(MYNN_E_STATE, "step at position %d: the rings have moved on to %d (rewind at most %d)", past_len, b.high, b.slack);
    b.stored = past_len + T;
    b.high = std::max(b.high, b.stored);
    return MYNN_OK;
}

__global__ void last_rows_kernel(int32_t *rows, int B, int S) {
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b < B) rows[b] = b * S + S - 1;
}

int block_forward(Model &m, cudaStream_t st, int S, int head_rows) {
    BlockModel &b = *m.blocks;
    const mynn_b200_block_model_config &c = b.c;
    const int B = c.batch, M = B * S, H = c.hidden, dt = c.dtype;
    int *status = (int *)m.gemm_ws;
    if (S > 1) m.tc_attention_ran = true;

    auto product = [&](void *out, int out_dtype, const void *act, const void *w, int rows, int N, int K) {
        DenseGemm g;
        g.out = out;
        g.act = act;
        g.w = w;
        g.M = rows, g.N = N, g.K = K;
        g.out_dtype = out_dtype;
        g.status = status;
        return launch_dense_gemm(st, dt, g);
    };
    // the row kernel between two sublayers: closes the one in `p` and norms x with (w2, b2) for the next
    auto step = [&](NormStep p, const float *w2, const float *b2) {
        p.x = b.x;
        p.x0 = p.embed || p.add_x0 ? b.x0 : nullptr;
        p.mult = c.residual_mult;
        p.eps = c.norm_eps;
        p.W = H;
        p.w2 = w2;
        p.b2 = b2;
        p.out = w2 ? b.h : nullptr;
        return launch_norm_step(st, dt, p, M);
    };
    {
        NormStep p;
        p.embed = b.embed;
        p.ids = m.ids_dev;
        p.embed_scale = c.embed_scale;
        p.vocab = c.vocab;
        RC(step(p, b.layers[b.runs[0].layer].n1w, b.layers[b.runs[0].layer].n1b));
    }
    for (size_t r = 0; r < b.runs.size(); r++) {
        const BlockRun &run = b.runs[r];
        const BlockLayer &L = b.layers[run.layer];
        const mynn_b200_block &l = L.c;
        const bool last = r + 1 == b.runs.size();
        const BlockLayer *next = last ? nullptr : &b.layers[b.runs[r + 1].layer];
        const int add_x0 = !last && b.runs[r + 1].add_embed;
        // ---- mixer ----
        RC(product(b.proj, dt, b.h, L.qkv, M, columns(l), H));
        ConvStep cv;
        cv.proj = b.proj;
        cv.hist = run.hist;
        cv.hist_rows = l.history_rows;
        cv.w = L.conv;
        cv.taps = l.conv_taps;
        cv.cos_t = L.cos_t, cv.sin_t = L.sin_t;
        cv.rot_dims = l.rot_dims;
        cv.q_out = b.q;
        cv.k_cache = run.kc, cv.v_cache = run.vc;
        cv.cache_rows = l.cache_rows;
        cv.B = B, cv.S = S, cv.Hq = l.heads, cv.G = l.kv_heads, cv.D = l.dim, cv.E = l.vdim;
        cv.past = m.past_dev;
        RC(launch_conv_step(st, dt, cv));
        WindowAttention at;
        at.out = b.attn;
        at.q = b.q;
        at.k = run.kc, at.v = run.vc;
        at.scale = l.attn_scale;
        at.softcap = l.softcap;
        at.window = l.window;
        at.B = B, at.Hq = l.heads, at.Hkv = l.kv_heads, at.Sq = S, at.D = l.dim, at.E = l.vdim;
        at.cache_rows = l.cache_rows;
        at.active = m.active_dev;
        at.workspace = m.attn_ws;
        at.workspace_bytes = m.attn_ws_bytes;
        at.status_word = status;
        RC(launch_window_attention(st, dt, at));
        RC(product(b.sub, dt, b.attn, L.o, M, H, l.heads * l.vdim));
        NormStep p;
        p.sub = b.sub;
        p.w1 = L.p1w, p.b1 = L.p1b;
        if (l.experts == 0) {
            p.add_x0 = add_x0;
            RC(step(p, next ? next->n1w : nullptr, next ? next->n1b : nullptr));
            continue;
        }
        RC(step(p, L.n2w, L.n2b));
        // ---- routed experts ----
        const MoeRoute rt = moe_route_bind(b.route, m.max_rows, l.experts, l.top);
        RC(product(b.z, MYNN_F32, b.h, L.router, M, l.experts, H));
        RC(launch_moe_route(st, rt, b.z, M, l.experts, l.top, l.groups, l.groups_keep));
        DenseGemm g;
        g.route = &rt;
        g.experts = l.experts;
        g.top = l.top;
        g.M = M;
        g.out_dtype = dt;
        g.status = status;
        g.act = b.h;
        g.w = L.gate_up;
        g.out = b.hidden;
        g.N = l.expert_ff, g.K = H;
        g.glu = 1;
        g.gather = 1;
        g.gather_ws = b.gathered;
        RC(launch_dense_gemm(st, dt, g));
        g.act = b.hidden;
        g.w = L.down;
        g.out = b.sub;
        g.N = H, g.K = l.expert_ff;
        g.glu = g.gather = 0;
        RC(launch_dense_gemm(st, dt, g));
        NormStep f;
        f.sub = b.sub;
        f.pair_row = rt.pair_row;
        f.pair_w = rt.pair_w;
        f.top = l.top;
        f.w1 = L.p2w, f.b1 = L.p2b;
        f.add_x0 = add_x0;
        RC(step(f, next ? next->n1w : nullptr, next ? next->n1b : nullptr));
    }
    if (head_rows < 0) return MYNN_OK;
    // ---- head: every sequence's last token, or the rows asked for ----
    const int rows = head_rows > 0 ? head_rows : B;
    NormStep f;
    f.x = b.x;
    f.w2 = b.fnw, f.b2 = b.fnb;
    f.eps = c.norm_eps;
    f.W = H;
    f.out = b.h;
    f.row_map = nullptr;
    if (head_rows > 0) {
        f.row_map = m.rows_dev;
    } else if (S > 1) {
        last_rows_kernel<<<(B + 255) / 256, 256, 0, st>>>(b.last_rows, B, S);
        MYNN_LAUNCH_OK("last_rows_kernel");
        f.row_map = b.last_rows;
    }
    RC(launch_norm_step(st, dt, f, rows));
    RC(product(m.logits, MYNN_F32, b.h, b.head, rows, c.vocab, H));
    if (c.output_mode == 1) {
        if (c.vocab >= 16384) RC(launch_argmax_two_stage(st, MYNN_F32, m.tok_dev, m.pairs_all, m.logits, B, c.vocab, 16));
        else RC(mynn_b200_argmax_last(st, m.tok_dev, m.logits, B, c.vocab, MYNN_F32));
        if (S == 1) RC(launch_tok_feedback(st, m.ids_dev, m.tok_dev, B));
    }
    return MYNN_OK;
}

}  // namespace mynn
