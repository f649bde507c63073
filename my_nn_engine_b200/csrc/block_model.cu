// The block decoder: a model described layer by layer (mynn_b200_block_model_config), stepped through the entry points of model.cu.
//
// A layer run is a mixer, closed by the norm kernel, and perhaps a feed-forward, closed by it again (the norm kernel closes one sublayer
// and opens the next):
//     attention: q/k/v product -> convolution + rotation + append, or rotation + head norms + append -> attention -> output product
//     latents:   product of both latents -> norms + append -> query product -> (few tokens) queries into latent space -> attention over the
//                latents -> value product per head, or (prompts) keys and values of all positions -> attention -> output product
//     mlstm:     one product for q, k, v and all gates -> state update with head norm and output gate -> output product
//     experts:   router product -> expert choice -> gate/up products with SiLU gating -> down products
//     dense:     up product with the activation -> down product
//     [combination of the experts, post norm, residual, (embedding output of a repeated pass), norm of the next sublayer]
// The residual stream is f32.  Every run has state of its own.  A cached position's row depends on the position alone and a recurrent
// state starts from zero at position 0, so a chunk may be cut anywhere, and a new sequence simply starts at position 0 again.  The
// decode step is captured in the CUDA graph that model.cu replays; past length and row count are device scalars.
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
    const float *vec0, *vec1;            // latent: weights of the two latents' norms; mlstm: head norm weight, gate biases
    const void *uq, *uk, *uk_t, *uv;     // latent
};
struct BlockRun {
    int layer;
    bool add_embed;  // the embedding output is added to x in front of it
    void *kc, *vc, *hist;  // the three state buffers: see session_state in mynn_b200.h
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
    void *lat_q, *lat_o, *lat_k, *lat_v, *lat_c;  // latent attention: queries and results in latent space, or keys and values; normed queries' latent
    void *lat_ws;
    size_t lat_ws_bytes;
    float *gates, *mem_ws;  // mlstm: gate products, workspace
    size_t mem_ws_bytes;
    unsigned *tickets;
    int32_t *last_rows;  // row of every sequence's last token in a chunk
    // what the rings hold: positions stored since the sequence began, and the most that were ever stored in it
    int stored = 0, high = 0, slack = INT_MAX;
    bool recurrent = false;  // some layer's state cannot go back
};

constexpr int kLatentTokens = 16;  // up to so many new tokens per sequence latent attention runs in latent space

static mynn_b200_block_model_config g_blocks_cfg;
static std::vector<mynn_b200_block> g_blocks_layers;

static int columns(const mynn_b200_block &b) {  // rows of the first product of the mixer
    if (b.mixer == MYNN_MIX_LATENT) return b.q_rank + b.kv_rank;
    if (b.mixer == MYNN_MIX_MLSTM) return b.heads * (2 * (b.dim + b.vdim) + 2);
    return b.heads * b.dim + b.kv_heads * (b.dim + b.vdim);
}
// how many positions up to its own a query sees at most, 0: all of them
static int reach(const mynn_b200_block &b) { return b.window > 0 && b.chunk > 0 ? std::min(b.window, b.chunk) : std::max(b.window, b.chunk); }

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
        if (b.mixer != MYNN_MIX_ATTENTION && b.mixer != MYNN_MIX_LATENT && b.mixer != MYNN_MIX_MLSTM)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d has mixer %d", l, b.mixer);
        if (b.mixer != MYNN_MIX_ATTENTION && (b.conv_taps || b.rot_dims || b.rot_halves || b.qk_norm || b.window || b.chunk || b.softcap != 0.f))
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: an option of another mixer", l);
        if (b.mixer == MYNN_MIX_LATENT && (b.q_rank <= 0 || b.kv_rank <= 0 || b.kv_rank > 1024 || b.dim > 1024 || b.vdim > 1024 || b.heads <= 0))
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: latents of %d and %d, %d heads of %d / %d", l, b.q_rank, b.kv_rank, b.heads, b.dim, b.vdim);
        if (b.mixer == MYNN_MIX_MLSTM && (!(b.gate_cap > 0.f) || b.dim > 512))
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: gate cap %g, memory of %d rows", l, b.gate_cap, b.dim);
        if (b.chunk < 0 || b.dense_ff < 0 || (b.dense_ff > 0 && b.experts > 0) || (b.ff_act != MYNN_ACT_NONE && b.ff_act != MYNN_ACT_SQUARE_RELU) ||
            (b.conv_taps > 0 && (b.rot_halves || b.qk_norm)))
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: chunk %d, feed-forward %d beside %d experts, activation %d, %d taps", l, b.chunk, b.dense_ff, b.experts, b.ff_act, b.conv_taps);
        if (b.heads <= 0 || b.kv_heads <= 0 || b.dim <= 0 || b.vdim <= 0 || b.heads % b.kv_heads)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d has %d heads of %d over %d kv heads of %d", l, b.heads, b.dim, b.kv_heads, b.vdim);
        if (b.conv_taps < 0 || b.rot_dims < 0 || b.rot_dims % 2 || b.rot_dims > b.dim || b.window < 0 || b.softcap < 0.f)
            return fail(MYNN_E_ARG, "model_configure_blocks: layer %d: taps %d, rotated dims %d, window %d, soft cap %g", l, b.conv_taps, b.rot_dims, b.window, b.softcap);
        const long long need = reach(b) ? std::min<long long>(c.max_seq_len, (long long)reach(b) - 1 + chunk + c.max_rewind) : c.max_seq_len;
        if (b.mixer != MYNN_MIX_MLSTM && (b.cache_rows < need || b.cache_rows % 128))
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
        const bool ff = lc.experts > 0 || lc.dense_ff > 0, bias = !c.rms_norm, post = c.post_norm, latent = lc.mixer == MYNN_MIX_LATENT;
        L.n1w = (const float *)take(), L.n1b = (const float *)take(bias), L.p1w = (const float *)take(post), L.p1b = (const float *)take(post && bias);
        L.qkv = take();
        L.conv = (const float *)take(lc.conv_taps > 0);
        L.o = take();
        L.cos_t = (const float *)take(lc.rot_dims > 0), L.sin_t = (const float *)take(lc.rot_dims > 0);
        L.n2w = (const float *)take(ff), L.n2b = (const float *)take(ff && bias), L.p2w = (const float *)take(ff && post), L.p2b = (const float *)take(ff && post && bias);
        L.router = take(lc.experts > 0), L.gate_up = take(ff), L.down = take(ff);
        L.vec0 = (const float *)take(lc.mixer != MYNN_MIX_ATTENTION), L.vec1 = (const float *)take(lc.mixer != MYNN_MIX_ATTENTION);
        L.uq = take(latent), L.uk = take(latent), L.uk_t = take(latent), L.uv = take(latent);
        b.layers.push_back(L);
    }
    b.fnw = (const float *)take(), b.fnb = (const float *)take(!c.rms_norm);
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
        if (!run.kc || (lc.mixer != MYNN_MIX_LATENT && !run.vc) || ((lc.conv_taps || lc.mixer == MYNN_MIX_MLSTM) && !run.hist)) return fail(MYNN_E_ARG, "model_init: a state buffer of layer run %zu is null", r);
        // how far past_len may fall behind the most positions ever stored before a ring has dropped what a step needs
        if (reach(lc) && lc.cache_rows < c.max_seq_len) b.slack = std::min(b.slack, lc.cache_rows - reach(lc) + 1);
        if (lc.mixer == MYNN_MIX_MLSTM) b.recurrent = true;
        if (lc.conv_taps && lc.history_rows < c.max_seq_len) b.slack = std::min(b.slack, lc.history_rows - lc.conv_taps + 1);
    }
    // ---- arena ----
    const int chunk = std::max(c.max_prefill, 1);
    const size_t R = m.max_rows, esz = dtype_size(c.dtype), H = c.hidden;
    m.head_capacity = std::max(c.batch, std::min(64, m.max_rows));
    size_t col = 0, qn = 0, an = 0, pairs_ff = 0, pairs_h = 0, gat = 0, route = 0, zn = 0, aws = 0;
    size_t lq = 0, lk = 0, lv = 0, lc_n = 0, lws = 0, gn = 0, mo = 0, tk = 0;
    const size_t few = (size_t)c.batch * std::min(chunk, kLatentTokens);
    for (const BlockLayer &L : b.layers) {
        const mynn_b200_block &l = L.c;
        col = std::max(col, (size_t)columns(l));
        qn = std::max(qn, (size_t)l.heads * l.dim);
        an = std::max(an, (size_t)l.heads * l.vdim);
        if (l.mixer == MYNN_MIX_ATTENTION) aws = std::max(aws, mynn_b200_attention_workspace_bytes(c.batch, l.heads, l.kv_heads, l.dim, l.cache_rows));
        if (l.mixer == MYNN_MIX_LATENT) {
            lc_n = std::max(lc_n, R * (size_t)l.q_rank);
            lq = std::max(lq, few * l.heads * (size_t)l.kv_rank);
            for (int s = 1; s <= std::min(chunk, kLatentTokens); s++) lws = std::max(lws, latent_attention_workspace_bytes(c.batch, s, l.heads, l.kv_rank, l.cache_rows));
            if (chunk > kLatentTokens) {
                lk = std::max(lk, (size_t)c.batch * l.heads * l.cache_rows * l.dim);
                lv = std::max(lv, (size_t)c.batch * l.heads * l.cache_rows * l.vdim);
            }
        }
        if (l.mixer == MYNN_MIX_MLSTM) {
            gn = std::max(gn, R * 2 * (size_t)l.heads);
            // not monotonic in the number of tokens: fewer tokens may be cut into more segments
            for (int s = 1; s <= chunk; s++) mo = std::max(mo, mlstm_workspace_bytes(c.dtype, c.batch, s, l.heads, l.dim, l.vdim));
            tk = std::max(tk, (size_t)c.batch * l.heads);
        }
        if (l.dense_ff) pairs_ff = std::max(pairs_ff, R * (size_t)l.dense_ff);
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
                 o_stat = area(512), o_lq = area(lq * esz), o_lo = area(lq * esz), o_lk = area(lk * esz), o_lv = area(lv * esz), o_lc = area(lc_n * esz),
                 o_lws = area(lws), o_gates = area(gn * 4), o_mo = area(mo), o_tk = area(tk * 4);
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
    b.lat_q = a + o_lq, b.lat_o = a + o_lo, b.lat_k = a + o_lk, b.lat_v = a + o_lv, b.lat_c = a + o_lc;
    b.lat_ws = a + o_lws;
    b.lat_ws_bytes = lws;
    b.gates = (float *)(a + o_gates);
    b.mem_ws = (float *)(a + o_mo);
    b.mem_ws_bytes = mo;
    b.tickets = (unsigned *)(a + o_tk);
    return MYNN_OK;
}

void block_destroy(Model &m) {
    delete m.blocks;
    m.blocks = nullptr;
}

int block_admit(Model &m, int past_len, int T) {
    BlockModel &b = *m.blocks;
    if (past_len == 0) b.stored = b.high = 0;
    if (b.recurrent && past_len != b.stored) return fail(MYNN_E_STATE, "step at position %d: the recurrent state is at position %d", past_len, b.stored);
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

static DenseGemm plain_product(Model &m, void *out, int out_dtype, const void *act, const void *w, int rows, int N, int K) {
    DenseGemm g;
    g.out = out;
    g.act = act;
    g.w = w;
    g.M = rows, g.N = N, g.K = K;
    g.out_dtype = out_dtype;
    g.status = (int *)m.gemm_ws;
    return g;
}

// The mixers: normed rows b.h -> heads side by side in b.attn.
static int mix_attention(Model &m, cudaStream_t st, const BlockLayer &L, const BlockRun &run, int S) {
    BlockModel &b = *m.blocks;
    const mynn_b200_block &l = L.c;
    const int B = b.c.batch, M = B * S, H = b.c.hidden, dt = b.c.dtype;
    RC(launch_dense_gemm(st, dt, plain_product(m, b.proj, dt, b.h, L.qkv, M, columns(l), H)));
    if (l.rot_halves || l.qk_norm) {
        RotaryAppend ra;
        ra.proj = b.proj;
        ra.cos_t = L.cos_t, ra.sin_t = L.sin_t;
        ra.rot_dims = l.rot_dims;
        ra.halves = l.rot_halves;
        ra.qk_norm = l.qk_norm;
        ra.eps = b.c.norm_eps;
        ra.q_out = b.q;
        ra.k_cache = run.kc, ra.v_cache = run.vc;
        ra.cache_rows = l.cache_rows;
        ra.B = B, ra.S = S, ra.Hq = l.heads, ra.G = l.kv_heads, ra.D = l.dim, ra.E = l.vdim;
        ra.past = m.past_dev;
        RC(launch_rotary_append(st, dt, ra));
    } else {
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
    }
    WindowAttention at;
    at.out = b.attn;
    at.q = b.q;
    at.k = run.kc, at.v = run.vc;
    at.scale = l.attn_scale;
    at.softcap = l.softcap;
    at.window = l.window;
    at.chunk = l.chunk;
    at.B = B, at.Hq = l.heads, at.Hkv = l.kv_heads, at.Sq = S, at.D = l.dim, at.E = l.vdim;
    at.cache_rows = l.cache_rows;
    at.active = m.active_dev;
    at.workspace = m.attn_ws;
    at.workspace_bytes = m.attn_ws_bytes;
    at.status_word = (int *)m.gemm_ws;
    return launch_window_attention(st, dt, at);
}

static int mix_latent(Model &m, cudaStream_t st, const BlockLayer &L, const BlockRun &run, int S) {
    BlockModel &b = *m.blocks;
    const mynn_b200_block &l = L.c;
    const int B = b.c.batch, M = B * S, H = b.c.hidden, dt = b.c.dtype, R = l.kv_rank;
    RC(launch_dense_gemm(st, dt, plain_product(m, b.proj, dt, b.h, L.qkv, M, columns(l), H)));
    LatentAppend la;
    la.proj = b.proj;
    la.wq = L.vec0, la.wc = L.vec1;
    la.eps = b.c.norm_eps;
    la.q_out = b.lat_c;
    la.cache = run.kc;
    la.B = B, la.S = S, la.Q = l.q_rank, la.R = R;
    la.cache_rows = l.cache_rows;
    la.past = m.past_dev;
    RC(launch_latent_append(st, dt, la));
    DenseGemm q = plain_product(m, b.q, dt, b.lat_c, L.uq, M, l.heads * l.dim, l.q_rank);
    if (S <= kLatentTokens) {
        RC(launch_dense_gemm(st, dt, q));
        DenseGemm in = plain_product(m, b.lat_q, dt, b.q, L.uk_t, M, R, l.dim);  // per head: q W_uk
        in.batch = l.heads;
        in.act_stride = l.dim, in.lda = l.heads * l.dim;
        in.out_stride = R, in.ldo = l.heads * R;
        RC(launch_dense_gemm(st, dt, in));
        LatentAttention at;
        at.out = b.lat_o;
        at.q = b.lat_q, at.c = run.kc;
        at.scale = l.attn_scale;
        at.B = B, at.Sq = S, at.H = l.heads, at.R = R;
        at.cache_rows = l.cache_rows;
        at.active = m.active_dev;
        at.workspace = b.lat_ws;
        at.workspace_bytes = b.lat_ws_bytes;
        RC(launch_latent_attention(st, dt, at));
        DenseGemm out = plain_product(m, b.attn, dt, b.lat_o, L.uv, M, l.vdim, R);
        out.batch = l.heads;
        out.act_stride = R, out.lda = l.heads * R;
        out.out_stride = l.vdim, out.ldo = l.heads * l.vdim;
        return launch_dense_gemm(st, dt, out);
    }
    // a prompt: keys and values of all stored positions, head-major
    q.out_block = l.dim, q.out_block_stride = (long long)M * l.dim, q.ldo = l.dim;
    RC(launch_dense_gemm(st, dt, q));
    const long long rows = (long long)B * l.cache_rows;
    DenseGemm k = plain_product(m, b.lat_k, dt, run.kc, L.uk, b.stored, l.heads * l.dim, R);
    k.out_block = l.dim, k.out_block_stride = rows * l.dim, k.ldo = l.dim;
    k.row_groups = B, k.group_rows = l.cache_rows;
    RC(launch_dense_gemm(st, dt, k));
    DenseGemm v = plain_product(m, b.lat_v, dt, run.kc, L.uv, b.stored, l.heads * l.vdim, R);
    v.out_block = l.vdim, v.out_block_stride = rows * l.vdim, v.ldo = l.vdim;
    v.row_groups = B, v.group_rows = l.cache_rows;
    RC(launch_dense_gemm(st, dt, v));
    WindowAttention at;
    at.out = b.attn;
    at.q = b.q;
    at.k = b.lat_k, at.v = b.lat_v;
    at.scale = l.attn_scale;
    at.layout = kByHead;
    at.B = B, at.Hq = l.heads, at.Hkv = l.heads, at.Sq = S, at.D = l.dim, at.E = l.vdim;
    at.cache_rows = l.cache_rows;
    at.active = m.active_dev;
    at.status_word = (int *)m.gemm_ws;
    return launch_window_attention(st, dt, at);
}

static int mix_mlstm(Model &m, cudaStream_t st, const BlockLayer &L, const BlockRun &run, int S) {
    BlockModel &b = *m.blocks;
    const mynn_b200_block &l = L.c;
    const int M = b.c.batch * S, dt = b.c.dtype;
    DenseGemm g = plain_product(m, b.proj, dt, b.h, L.qkv, M, columns(l), b.c.hidden);
    g.out_f32 = b.gates;  // the input and forget gates' rows come last
    g.n_main = columns(l) - 2 * l.heads;
    RC(launch_dense_gemm(st, dt, g));
    MlstmStep p;
    p.proj = b.proj;
    p.gates = b.gates;
    p.norm_w = L.vec0;
    p.gate_bias = L.vec1;
    p.cap = l.gate_cap;
    p.eps = b.c.norm_eps;
    p.mem = (float *)run.kc, p.sum = (float *)run.vc, p.top = (float *)run.hist;
    p.workspace = b.mem_ws;
    p.workspace_bytes = b.mem_ws_bytes;
    p.ticket = b.tickets;
    p.out = b.attn;
    p.B = b.c.batch, p.S = S, p.H = l.heads, p.D = l.dim, p.E = l.vdim;
    p.past = m.past_dev;
    p.status = (int *)m.gemm_ws;
    return launch_mlstm(st, dt, p);
}

int block_forward(Model &m, cudaStream_t st, int S, int head_rows) {
    BlockModel &b = *m.blocks;
    const mynn_b200_block_model_config &c = b.c;
    const int B = c.batch, M = B * S, H = c.hidden, dt = c.dtype;
    int *status = (int *)m.gemm_ws;
    if (S > 1) m.tc_attention_ran = true;

    auto product = [&](void *out, int out_dtype, const void *act, const void *w, int rows, int N, int K) {
        return launch_dense_gemm(st, dt, plain_product(m, out, out_dtype, act, w, rows, N, K));
    };
    // the row kernel between two sublayers: closes the one in `p` and norms x with (w2, b2) for the next
    auto step = [&](NormStep p, const float *w2, const float *b2) {
        p.x = b.x;
        p.x0 = p.embed || p.add_x0 ? b.x0 : nullptr;
        p.mult = c.residual_mult;
        p.eps = c.norm_eps;
        p.rms = c.rms_norm;
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
        if (l.mixer == MYNN_MIX_LATENT) RC(mix_latent(m, st, L, run, S));
        else if (l.mixer == MYNN_MIX_MLSTM) RC(mix_mlstm(m, st, L, run, S));
        else RC(mix_attention(m, st, L, run, S));
        RC(product(b.sub, dt, b.attn, L.o, M, H, l.heads * l.vdim));
        NormStep p;
        p.sub = b.sub;
        p.w1 = L.p1w, p.b1 = L.p1b;
        if (l.experts == 0 && l.dense_ff == 0) {
            p.add_x0 = add_x0;
            RC(step(p, next ? next->n1w : nullptr, next ? next->n1b : nullptr));
            continue;
        }
        RC(step(p, L.n2w, L.n2b));
        if (l.dense_ff) {
            DenseGemm up = plain_product(m, b.hidden, dt, b.h, L.gate_up, M, l.dense_ff, H);
            up.act_fn = l.ff_act;
            RC(launch_dense_gemm(st, dt, up));
            RC(product(b.sub, dt, b.hidden, L.down, M, H, l.dense_ff));
            NormStep f;
            f.sub = b.sub;
            f.w1 = L.p2w, f.b1 = L.p2b;
            f.add_x0 = add_x0;
            RC(step(f, next ? next->n1w : nullptr, next ? next->n1b : nullptr));
            continue;
        }
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
    f.rms = c.rms_norm;
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
