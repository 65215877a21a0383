// Layer-described models: construction from descriptions, weights by name, the layer loop, and the mixers with norms on their outputs.
#include "stack.cuh"
#include "elem.cuh"

#include <algorithm>
#include <cmath>

namespace b200 {

// ---- construction ---------------------------------------------------------------------------------------------------------
static int make_mlstm(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, MlstmOp& op) {
    B2_CHECK_ARG(d.heads > 0 && d.dim > 0 && d.vdim > 0 && d.gate_cap > 0, "mLSTM layer: bad sizes");
    op.elem = elem;
    op.width = c.width;
    MlstmShape& sh = op.sh;
    sh.heads = d.heads; sh.dim = d.dim; sh.vdim = d.vdim;
    sh.gate_cap = (float)d.gate_cap; sh.eps = (float)c.norm_eps;
    sh.n_vt = ceil_div(d.vdim, kMlstmTile);
    sh.vt = sh.n_vt == 1 ? round_up(d.vdim, 4) : kMlstmTile;
    // Tensor-core prefill wants whole 64-column blocks per head; the other path only 16-byte rows.
    sh.dp = round_up(d.dim, 64); sh.vp = round_up(d.vdim, 64);
    op.chunk = elem == ELEM_BF16 && mlstm_chunk_fits(sh);
    if (!op.chunk) { sh.dp = round_up(d.dim, 8); sh.vp = round_up(d.vdim, 8); }
    const size_t e = elem_bytes(elem);
    B2_TRY(op.w_in.alloc((size_t)sh.pitch() * c.width * e));
    B2_TRY(op.w_out.alloc((size_t)c.width * sh.heads * sh.vp * e));
    B2_TRY(op.bias.alloc((size_t)2 * sh.heads * 4));
    return op.norm_w.alloc((size_t)sh.heads * sh.vp * 4);
}

static int make_latent(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, LatentOp& op) {
    B2_CHECK_ARG(d.heads > 0 && d.dim > 0 && d.vdim > 0 && d.kv_rank > 0 && d.rot_dim >= 0 && d.rot_dim % 2 == 0 && d.window >= 0,
                 "latent-attention layer: bad sizes");
    if (d.kv_rank > 1024) B2_FAIL(B200ATTN_ERR_UNSUPPORTED, "latent-attention layer: kv_rank %d above 1024", d.kv_rank);
    op.elem = elem;
    op.width = c.width;
    LatentShape& sh = op.sh;
    sh.heads = d.heads; sh.dim = d.dim; sh.rot = d.rot_dim; sh.vdim = d.vdim; sh.rank = d.kv_rank; sh.window = d.window;
    sh.scale = (float)d.scale; sh.eps = (float)c.norm_eps;
    sh.own = d.kv_from < 0;
    sh.dp = round_up(d.dim, 64); sh.rp = round_up(d.rot_dim, 64); sh.vp = round_up(d.vdim, 64);
    op.tc_prefill = elem == ELEM_BF16 && latent_prefill_fits(sh);
    if (!op.tc_prefill) { sh.dp = round_up(d.dim, 8); sh.rp = round_up(d.rot_dim, 8); sh.vp = round_up(d.vdim, 8); }
    op.tc_decode = elem == ELEM_BF16 && latent_decode_fits(sh, c.max_seqs);
    const size_t e = elem_bytes(elem);
    B2_TRY(op.w_in.alloc((size_t)sh.pitch() * c.width * e));
    B2_TRY(op.w_uk.alloc((size_t)sh.heads * sh.dp * sh.rank * e));
    B2_TRY(op.w_uv.alloc((size_t)sh.heads * sh.vp * sh.rank * e));
    B2_TRY(op.w_out.alloc((size_t)c.width * sh.heads * sh.vp * e));
    B2_TRY(op.c_norm.alloc((size_t)sh.rank * 4));
    return 0;
}

// Index of a rotation's table, added where no layer before has it.
static int rot_table(BlockModel& m, double base, int half) {
    for (size_t k = 0; k < m.rot.size(); ++k)
        if (m.rot[k].base == base && m.rot[k].half == half) return (int)k;
    m.rot.emplace_back();
    m.rot.back().base = base;
    m.rot.back().half = half;
    return (int)m.rot.size() - 1;
}

int block_model_create(const b200attn_model_config* cfg, const b200attn_layer_desc* layers, int num_layers, b200attn_stack st) {
    B2_CHECK_ARG(cfg->dtype == B200ATTN_DTYPE_BF16 || cfg->dtype == B200ATTN_DTYPE_F32, "model: bad dtype");
    st->blocks.reset(new (std::nothrow) BlockModel());
    if (!st->blocks) B2_FAIL(B200ATTN_ERR_NOMEM, "model: host allocation failed");
    BlockModel& m = *st->blocks;
    m.cfg = *cfg;
    m.elem = cfg->dtype == B200ATTN_DTYPE_F32 ? ELEM_F32 : ELEM_BF16;
    const size_t e = elem_bytes(m.elem), W = cfg->width;
    const long long all = (long long)cfg->max_seqs * cfg->max_seq_len;
    m.max_rows = std::max(cfg->max_seqs, cfg->max_pass_rows > 0 ? cfg->max_pass_rows : (int)std::min(all, 8192ll));
    st->max_rows = m.max_rows;

    m.layers.resize(num_layers);
    m.missing = {"embed", "final.norm"};
    if (cfg->own_head) m.missing.push_back("head");
    BlockSizes z;
    for (int i = 0; i < num_layers; ++i) {
        const b200attn_layer_desc& d = layers[i];
        BlockLayer& L = m.layers[i];
        auto need = [&](const char* n) { L.missing.push_back(n); };
        need("norm1");
        if (d.mixer == B200ATTN_MIXER_MLSTM) {
            L.mlstm.reset(new MlstmOp());
            B2_TRY(make_mlstm(d, *cfg, m.elem, *L.mlstm));
            const MlstmShape& sh = L.mlstm->sh;
            z.proj = std::max(z.proj, (size_t)sh.pitch());
            z.mixed = std::max(z.mixed, (size_t)sh.heads * sh.vp);
            if (L.mlstm->chunk || sh.n_vt > 1) z.core = std::max(z.core, (size_t)sh.heads * sh.vp);
            if (L.mlstm->chunk) z.gates = std::max(z.gates, (size_t)2 * sh.heads);
            for (const char* n : {"mix.q", "mix.k", "mix.v", "mix.g", "mix.o", "mix.norm", "mix.i", "mix.i.b", "mix.f", "mix.f.b"}) need(n);
        } else if (d.mixer == B200ATTN_MIXER_LATENT) {
            L.latent.reset(new LatentOp());
            LatentOp& op = *L.latent;
            B2_TRY(make_latent(d, *cfg, m.elem, op));
            const LatentShape& sh = op.sh;
            op.kv_from = d.kv_from;
            if (sh.own) {
                for (const char* n : {"mix.dkv", "mix.dkv.norm"}) need(n);
            } else {
                B2_CHECK_ARG(d.kv_from < i && m.layers[d.kv_from].latent && m.layers[d.kv_from].latent->sh.own,
                             "layer %d: kv_from %d is not an earlier layer with latents of its own", i, d.kv_from);
                const LatentShape& src = m.layers[d.kv_from].latent->sh;
                B2_CHECK_ARG(src.rank == sh.rank && src.rot == sh.rot, "layer %d: kv_rank and rot_dim differ from those of layer %d", i, d.kv_from);
            }
            for (const char* n : {"mix.q", "mix.uk", "mix.uv", "mix.o"}) need(n);
            op.rot_table = rot_table(m, d.rot_base, sh.rot / 2);
            z.proj = std::max(z.proj, (size_t)sh.pitch());
            z.mixed = std::max(z.mixed, (size_t)sh.heads * sh.vp);
            z.q = std::max(z.q, (size_t)sh.q_cols());
            z.qa = std::max(z.qa, (size_t)sh.heads * sh.row_pitch());
            z.olat = std::max(z.olat, (size_t)sh.heads * sh.rank);
            if (op.tc_prefill) {
                z.cst = std::max(z.cst, (size_t)sh.rank); z.rst = std::max(z.rst, (size_t)sh.rp);
                z.kup = std::max(z.kup, (size_t)sh.heads * sh.dp); z.vup = std::max(z.vup, (size_t)sh.heads * sh.vp);
                z.max_window = std::max(z.max_window, sh.window > 0 ? std::min(sh.window, cfg->max_seq_len) : cfg->max_seq_len);
            }
            if (op.tc_decode) {
                z.part = std::max(z.part, latent_decode_scratch_floats(sh, cfg->max_seqs));
                z.counters = std::max(z.counters, (size_t)cfg->max_seqs * ceil_div(sh.heads, 16));
            }
        } else if (d.mixer == B200ATTN_MIXER_LIGHTNING) {
            L.mlstm.reset(new MlstmOp());
            B2_TRY(make_lightning(d, *cfg, m.elem, *L.mlstm, z));
            for (const char* n : {"mix.q", "mix.k", "mix.v", "mix.g", "mix.o", "mix.norm"}) need(n);
        } else if (d.mixer == B200ATTN_MIXER_CHANNEL_DELTA) {
            L.delta.reset(new DeltaOp());
            B2_TRY(make_delta(d, *cfg, m.elem, *L.delta, z));
            for (const char* n : {"mix.q", "mix.q.conv", "mix.k", "mix.k.conv", "mix.v", "mix.v.conv", "mix.b", "mix.A_log", "mix.norm", "mix.a1", "mix.a2",
                                  "mix.dt_bias", "mix.g1", "mix.g2", "mix.o"}) need(n);
        } else if (d.mixer == B200ATTN_MIXER_DIFF) {
            L.diff.reset(new DiffOp());
            B2_TRY(make_diff(d, *cfg, m.elem, *L.diff, z));
            L.diff->rot_table = rot_table(m, d.rot_base, d.rot_dim / 2);
            for (const char* n : {"mix.q", "mix.k", "mix.v", "mix.q.norm", "mix.k.norm", "mix.lq1", "mix.lk1", "mix.lq2", "mix.lk2", "mix.o"}) need(n);
        } else {
            B2_FAIL(B200ATTN_ERR_INVALID, "layer %d: unknown mixer %d", i, d.mixer);
        }
        B2_TRY(L.norm1.alloc(W * 4));
        B2_CHECK_ARG(d.act == B200ATTN_ACT_GELU_TANH || d.act == B200ATTN_ACT_SILU, "layer %d: unknown activation %d", i, d.act);
        L.ff = d.ff;
        L.act = d.act;
        if (d.ff > 0) {
            B2_TRY(L.norm2.alloc(W * 4));
            B2_TRY(L.w_gu.alloc((size_t)2 * d.ff * W * e));
            B2_TRY(L.w_down.alloc((size_t)d.ff * W * e));
            z.ff = std::max(z.ff, (size_t)d.ff);
            for (const char* n : {"norm2", "mlp.gate", "mlp.up", "mlp.down"}) need(n);
        }
    }

    // The layers in the order they run; every run has its own state and cache.
    const int times = std::max(1, cfg->loop_times), start = times > 1 ? cfg->loop_start : 0, stop = times > 1 ? cfg->loop_stop : 0;
    B2_CHECK_ARG(times == 1 || (0 <= start && start < stop && stop <= num_layers), "model: loop over layers [%d, %d) of %d", start, stop, num_layers);
    if (times > 1 && !cfg->pre_norm) B2_FAIL(B200ATTN_ERR_UNSUPPORTED, "model: loops need norms on the sublayers' inputs");
    auto run = [&](int i, bool again) { m.runs.emplace_back(); m.runs.back().layer = i; m.runs.back().add_embedding = again; };
    for (int i = 0; i < start; ++i) run(i, false);
    for (int t = 0; t < times; ++t)
        for (int i = start; i < stop; ++i) run(i, t > 0 && i == start);
    for (int i = stop; i < num_layers; ++i) run(i, false);
    std::vector<size_t> state_floats;
    std::vector<int> row_pitch, last_pool_layer(num_layers, -1);
    for (LayerRun& r : m.runs) {
        BlockLayer& L = m.layers[r.layer];
        auto state = [&](size_t n) { r.state_layer = (int)state_floats.size(); state_floats.push_back(n); };
        auto cache = [&](int pitch) { r.pool_layer = last_pool_layer[r.layer] = (int)row_pitch.size(); row_pitch.push_back(pitch); };
        if (L.mlstm) state(L.mlstm->sh.state_floats());
        if (L.delta) state(L.delta->sh.state_floats());
        if (L.diff) cache(L.diff->sh.row_pitch());
        if (L.latent && L.latent->sh.own) cache(L.latent->sh.row_pitch());
        if (L.latent && !L.latent->sh.own) r.pool_layer = last_pool_layer[L.latent->kv_from];     // its source's latest run
    }
    B2_TRY(m.embed.alloc((size_t)cfg->vocab_size * W * e));
    B2_TRY(m.final_norm.alloc(W * 4));
    if (cfg->own_head) B2_TRY(m.head.alloc((size_t)cfg->vocab_size * W * e));

    if (!state_floats.empty()) B2_TRY(state_pool_create_blocks(state_floats, cfg->max_seqs, &st->state));
    if (!row_pitch.empty()) {
        const int per_seq = ceil_div(cfg->max_seq_len, kPageTokens);
        B2_TRY(kv_pool_create_latent(row_pitch, m.elem, cfg->num_pages > 0 ? cfg->num_pages : per_seq * cfg->max_seqs, cfg->max_seqs, per_seq, &st->pool));
        for (int i = 0; i < cfg->max_seqs; ++i) {
            int slot = -1;
            B2_TRY(b200attn_kv_seq_alloc(st->pool, cfg->num_pages > 0 ? 0 : cfg->max_seq_len, &slot));
        }
    }
    m.pool = st->pool;
    m.state = st->state;

    const size_t R = m.max_rows;
    m.abs_rows = (int)std::min<size_t>(R, std::max(4096, cfg->max_seqs));
    m.ctx_rows = (int)R + z.max_window;
    m.max_spans = (int)std::max<size_t>(cfg->max_seqs, 1);
    for (RotTable& t : m.rot) {
        std::vector<double> f(std::max(1, t.half));
        for (int i = 0; i < t.half; ++i) f[i] = std::pow(t.base, -(double)i / t.half);
        B2_TRY(t.freq.alloc(f.size() * 8));
        B2_CUDA(cudaMemcpy(t.freq.p, f.data(), f.size() * 8, cudaMemcpyHostToDevice));
        B2_TRY(t.cs.alloc(R * f.size() * sizeof(float2)));
    }
    B2_TRY(m.x.alloc(R * W * 4));
    if (times > 1) B2_TRY(m.x0.alloc(R * W * 4));
    B2_TRY(m.xt.alloc(R * W * e));
    if (!cfg->pre_norm) B2_TRY(m.y.alloc(R * W * 4));
    B2_TRY(m.proj.alloc(R * z.proj * 4));
    B2_TRY(m.gates.alloc(R * z.gates * 4));
    B2_TRY(m.low.alloc(R * z.low * e));
    B2_TRY(m.core.alloc(R * z.core * 4));
    B2_TRY(m.mixed.alloc(R * z.mixed * e));
    B2_TRY(m.gu.alloc(R * 2 * z.ff * e));
    B2_TRY(m.act.alloc(R * z.ff * e));
    B2_TRY(m.q.alloc(R * z.q * e));
    B2_TRY(m.qa.alloc((size_t)m.abs_rows * z.qa * e));
    B2_TRY(m.olat.alloc((size_t)m.abs_rows * z.olat * e));
    B2_TRY(m.c_stage.alloc((size_t)m.ctx_rows * z.cst * e));
    B2_TRY(m.r_stage.alloc((size_t)m.ctx_rows * z.rst * e));
    B2_TRY(m.k_up.alloc((size_t)m.ctx_rows * z.kup * e));
    B2_TRY(m.v_up.alloc((size_t)m.ctx_rows * z.vup * e));
    B2_TRY(m.chunk.alloc((R / 64 + m.max_spans + 1) * z.chunk));
    B2_TRY(m.part.alloc(z.part * 4));
    B2_TRY(m.counters.alloc(z.counters * 4));
    const size_t tiles = R / 128 + m.max_spans + 1;
    B2_TRY(m.meta.alloc((2 * R + 7 * (size_t)m.max_spans + 5 * tiles) * 4));
    return m.error.alloc(4);
}

int block_model_ready(const BlockModel& m) {
    if (!m.missing.empty()) B2_FAIL(B200ATTN_ERR_NOT_READY, "model: tensor '%s' not set", m.missing[0].c_str());
    for (size_t i = 0; i < m.layers.size(); ++i)
        if (!m.layers[i].missing.empty()) B2_FAIL(B200ATTN_ERR_NOT_READY, "model: tensor 'l%zu.%s' not set", i, m.layers[i].missing[0].c_str());
    return 0;
}

int block_model_status(BlockModel& m, int* code) {
    B2_CUDA(cudaDeviceSynchronize());
    B2_CUDA(cudaMemcpy(code, m.error.p, sizeof(int), cudaMemcpyDeviceToHost));
    if (*code) B2_CUDA(cudaMemset(m.error.p, 0, sizeof(int)));
    return 0;
}

// ---- weights by name ---------------------------------------------------------------------------------------------------------
int check_shape(const Source& t, const char* name, long long rows, long long cols) {
    B2_CHECK_ARG(t.rows == rows && t.cols == cols, "tensor '%s': shape [%lld, %lld], expected [%lld, %lld]", name, t.rows, t.cols, rows, cols);
    return 0;
}

int put(DevBuf& dst, ElemType elem, size_t ld, size_t row0, size_t col0, const Source& t, size_t src_row, size_t src_col, size_t rows, size_t cols) {
    const size_t e = elem_bytes(elem);
    std::vector<char> h(rows * cols * e);
    for (size_t r = 0; r < rows; ++r)
        for (size_t c = 0; c < cols; ++c) {
            const size_t i = (src_row + r) * t.cols + src_col + c;
            if (elem == ELEM_F32) {
                reinterpret_cast<float*>(h.data())[r * cols + c] = t.at(i);
            } else if (!t.f32) {
                reinterpret_cast<uint16_t*>(h.data())[r * cols + c] = static_cast<const uint16_t*>(t.data)[i];
            } else {
                reinterpret_cast<__nv_bfloat16*>(h.data())[r * cols + c] = __float2bfloat16_rn(t.at(i));
            }
        }
    B2_CUDA(cudaMemcpy2D(static_cast<char*>(dst.p) + (row0 * ld + col0) * e, ld * e, h.data(), cols * e, cols * e, rows, cudaMemcpyHostToDevice));
    return 0;
}

int put_vector(DevBuf& dst, const char* name, const Source& t, size_t at, long long n) {
    B2_TRY(check_shape(t, name, n, 1));
    return put(dst, ELEM_F32, 1, at, 0, t, 0, 0, n, 1);
}

int put_heads(DevBuf& dst, ElemType elem, size_t row0, int stride, const Source& t, int heads, int size, int in, int src_stride, int src_off) {
    for (int h = 0; h < heads; ++h) B2_TRY(put(dst, elem, in, row0 + (size_t)h * stride, 0, t, (size_t)h * src_stride + src_off, 0, size, in));
    return 0;
}

int put_out(DevBuf& dst, ElemType elem, const char* name, const Source& t, int width, int heads, int vdim, int vp) {
    B2_TRY(check_shape(t, name, width, (long long)heads * vdim));
    for (int h = 0; h < heads; ++h) B2_TRY(put(dst, elem, (size_t)heads * vp, 0, (size_t)h * vp, t, 0, (size_t)h * vdim, width, vdim));
    return 0;
}

namespace {
int set_mlstm(MlstmOp& op, const std::string& n, const char* name, const Source& t) {
    const MlstmShape& sh = op.sh;
    const int W = op.width, H = sh.heads;
    auto heads = [&](int row0, int stride, int size) -> int {
        B2_TRY(check_shape(t, name, (long long)H * size, W));
        return put_heads(op.w_in, op.elem, row0, stride, t, H, size, W, size, 0);
    };
    if (n == "q") return heads(sh.off_q(), sh.dp, sh.dim);
    if (n == "k") return heads(sh.off_k(), sh.dp, sh.dim);
    if (n == "v") return heads(sh.off_v(), sh.vp, sh.vdim);
    if (n == "g") return heads(sh.off_g(), sh.vp, sh.vdim);
    if (n == "i") return heads(sh.off_i(), 1, 1);
    if (n == "f") return heads(sh.off_f(), 1, 1);
    if (n == "i.b") return put_vector(op.bias, name, t, 0, H);
    if (n == "f.b") return put_vector(op.bias, name, t, H, H);
    if (n == "o") return put_out(op.w_out, op.elem, name, t, W, H, sh.vdim, sh.vp);
    if (n == "norm") {
        B2_TRY(check_shape(t, name, (long long)H * sh.vdim, 1));
        for (int h = 0; h < H; ++h) B2_TRY(put(op.norm_w, ELEM_F32, 1, (size_t)h * sh.vp, 0, t, (size_t)h * sh.vdim, 0, sh.vdim, 1));
        return 0;
    }
    B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': an mLSTM layer has no such tensor", name);
}

int set_latent(LatentOp& op, const std::string& n, const char* name, const Source& t) {
    const LatentShape& sh = op.sh;
    const int W = op.width, H = sh.heads;
    if (n == "q") {
        B2_TRY(check_shape(t, name, (long long)H * (sh.dim + sh.rot), W));
        B2_TRY(put_heads(op.w_in, op.elem, 0, sh.dp + sh.rp, t, H, sh.dim, W, sh.dim + sh.rot, 0));
        return put_heads(op.w_in, op.elem, sh.dp, sh.dp + sh.rp, t, H, sh.rot, W, sh.dim + sh.rot, sh.dim);
    }
    if (n == "dkv" && sh.own) {
        B2_TRY(check_shape(t, name, sh.rank + sh.rot, W));
        return put(op.w_in, op.elem, W, sh.q_cols(), 0, t, 0, 0, sh.rank + sh.rot, W);
    }
    if (n == "dkv.norm" && sh.own) return put_vector(op.c_norm, name, t, 0, sh.rank);
    if (n == "uk") {
        B2_TRY(check_shape(t, name, (long long)H * sh.dim, sh.rank));
        return put_heads(op.w_uk, op.elem, 0, sh.dp, t, H, sh.dim, sh.rank, sh.dim, 0);
    }
    if (n == "uv") {
        B2_TRY(check_shape(t, name, (long long)H * sh.vdim, sh.rank));
        return put_heads(op.w_uv, op.elem, 0, sh.vp, t, H, sh.vdim, sh.rank, sh.vdim, 0);
    }
    if (n == "o") return put_out(op.w_out, op.elem, name, t, W, H, sh.vdim, sh.vp);
    B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': this latent-attention layer has no such tensor", name);
}

int set_tensor(BlockModel& m, const char* name, const Source& t) {
    const int W = m.cfg.width;
    auto given = [](std::vector<std::string>& missing, const std::string& n) { missing.erase(std::remove(missing.begin(), missing.end(), n), missing.end()); };
    const std::string full = name;
    if (full == "embed" || (full == "head" && m.cfg.own_head)) {
        B2_TRY(check_shape(t, name, m.cfg.vocab_size, W));
        B2_TRY(put(full == "head" ? m.head : m.embed, m.elem, W, 0, 0, t, 0, 0, t.rows, W));
        given(m.missing, full);
        return 0;
    }
    if (full == "final.norm") {
        B2_TRY(put_vector(m.final_norm, name, t, 0, W));
        given(m.missing, full);
        return 0;
    }
    int layer = -1, used = 0;
    if (std::sscanf(name, "l%d.%n", &layer, &used) != 1 || used == 0 || layer < 0 || layer >= (int)m.layers.size())
        B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': unknown name", name);
    BlockLayer& L = m.layers[layer];
    const std::string n = name + used;
    if (n == "norm1") B2_TRY(put_vector(L.norm1, name, t, 0, W));
    else if (n == "norm2" && L.ff > 0) B2_TRY(put_vector(L.norm2, name, t, 0, W));
    else if ((n == "mlp.gate" || n == "mlp.up") && L.ff > 0) {
        B2_TRY(check_shape(t, name, L.ff, W));
        B2_TRY(put(L.w_gu, m.elem, W, n == "mlp.up" ? L.ff : 0, 0, t, 0, 0, L.ff, W));
    } else if (n == "mlp.down" && L.ff > 0) {
        B2_TRY(check_shape(t, name, W, L.ff));
        B2_TRY(put(L.w_down, m.elem, L.ff, 0, 0, t, 0, 0, W, L.ff));
    } else if (n.rfind("mix.", 0) == 0) {
        const std::string w = n.substr(4);
        if (L.mlstm) B2_TRY(L.mlstm->sh.gated ? set_mlstm(*L.mlstm, w, name, t) : set_lightning(*L.mlstm, w, name, t));
        else if (L.delta) B2_TRY(set_delta(*L.delta, w, name, t));
        else if (L.diff) B2_TRY(set_diff(*L.diff, w, name, t));
        else B2_TRY(set_latent(*L.latent, w, name, t));
    } else {
        B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': unknown name", name);
    }
    given(L.missing, n);
    return 0;
}
}  // namespace

// ---- layer loop ---------------------------------------------------------------------------------------------------------------
static int mlstm_forward(BlockModel& m, MlstmOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s) {
    const MlstmShape& sh = op.sh;
    const int W = m.cfg.width;
    float* state = m.state->d_recurrent + m.state->block_offset[run.state_layer];
    if (!p.decode && op.chunk && p.max_count >= 16) {
        // q | k | v | g in bf16 for the tensor cores, the gate pre-activations in fp32
        B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.cols(), op.elem, ELEM_BF16, p.rows, sh.cols(), W));
        B2_TRY(gemm_typed(s, m.xt.p, W, (const char*)op.w_in.p + (size_t)sh.off_i() * W * elem_bytes(op.elem), m.gates.p, 2 * sh.heads, op.elem, ELEM_F32,
                          p.rows, 2 * sh.heads, W));
        {
            ProfScope prof(PROF_LA_PREFILL, s);
            B2_TRY(launch_mlstm_chunk(sh, m.proj.p, p.rows, m.gates.f(), 2 * sh.heads, op.bias.f(), p.d_seqs, p.n_seqs, m.cfg.max_seqs, state,
                                      m.core.f(), m.error.i(), s));
        }
        B2_TRY(launch_mlstm_head_norm(op.elem, sh, m.core.f(), m.proj.p, false, sh.cols(), op.norm_w.f(), p.rows, m.mixed.p, s));
    } else {
        B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.pitch(), op.elem, ELEM_F32, p.rows, sh.pitch(), W));
        MlstmStepArgs a{sh, m.proj.f(), op.bias.f(), op.norm_w.f(), state, p.decode ? p.d_slots : nullptr, p.decode ? nullptr : p.d_seqs,
                        m.cfg.max_seqs, m.core.f(), m.mixed.p};
        B2_TRY(launch_mlstm_step(op.elem, a, p.n_seqs, s));
        if (sh.n_vt > 1)
            B2_TRY(launch_mlstm_head_norm(op.elem, sh, m.core.f(), m.proj.p, true, sh.pitch(), op.norm_w.f(), p.rows, m.mixed.p, s));
    }
    return 0;
}

// Attention with the up-projections absorbed into the queries and outputs: decode, and prefill in blocks of rows.
static int latent_absorbed(BlockModel& m, LatentOp& op, const PassRows& p, const LatentView& cache, cudaStream_t s) {
    const LatentShape& sh = op.sh;
    const size_t e = elem_bytes(op.elem);
    const int hw = sh.dp + sh.rp, vcols = sh.heads * sh.vp;
    for (int r0 = 0; r0 < p.rows; r0 += m.abs_rows) {
        const int n = std::min(m.abs_rows, p.rows - r0);
        void* q = (char*)m.q.p + (size_t)r0 * sh.q_cols() * e;
        const int *slot = p.row_slot + r0, *pos = p.row_pos + r0;
        LatentPreArgs a{sh, m.proj.f() + (size_t)r0 * sh.pitch(), (const float2*)m.rot[op.rot_table].cs.p + (size_t)r0 * (sh.rot / 2), op.c_norm.f(), slot, pos, cache, q, m.qa.p};
        B2_TRY(launch_latent_pre(op.elem, a, n, s));
        B2_TRY(gemm_heads(s, q, sh.q_cols(), hw, op.w_uk.p, true, m.qa.p, sh.heads * sh.row_pitch(), sh.row_pitch(), op.elem, op.elem, n, sh.rank, sh.dp,
                          sh.heads));
        if (p.decode && op.tc_decode) {
            B2_TRY(launch_latent_decode(sh, m.qa.p, cache, slot, pos, n, m.part.f(), m.counters.i(), m.olat.p, s));
        } else {
            B2_TRY(launch_latent_attn_rows(op.elem, sh, m.qa.p, cache, slot, pos, n, m.olat.p, s));
        }
        B2_TRY(gemm_heads(s, m.olat.p, sh.heads * sh.rank, sh.rank, op.w_uv.p, false, (char*)m.mixed.p + (size_t)r0 * vcols * e, vcols, sh.vp, op.elem,
                          op.elem, n, sh.vp, sh.rank, sh.heads));
    }
    return 0;
}

// The context a prefill pass needs of one sequence: its own rows and the window before them.
static LatentSpan context_span(const LatentShape& sh, int slot, int base, int count, int ctx0) {
    const int first = sh.window > 0 ? std::max(0, base - sh.window + 1) : 0;
    return LatentSpan{slot, ctx0, first, base + count - first};
}

// Prefill on the tensor cores: the context's latents are staged and up-projected to keys and values once per pass.
static int latent_expanded(BlockModel& m, LatentOp& op, const LayerRun& run, const PassRows& p, const LatentView& cache, cudaStream_t s) {
    const LatentShape& sh = op.sh;
    LatentPreArgs a{sh, m.proj.f(), (const float2*)m.rot[op.rot_table].cs.p, op.c_norm.f(), p.row_slot, p.row_pos, cache, m.q.p, nullptr};
    B2_TRY(launch_latent_pre(op.elem, a, p.rows, s));
    std::vector<LatentSpan> spans;
    std::vector<LatentTile> tiles;
    int ctx = 0, longest = 0, row = 0;
    for (int i = 0; i < p.n_seqs; ++i) {
        const LatentSpan sp = context_span(sh, p.h_slots[i], p.h_base[i], p.h_counts[i], ctx);
        for (int r = 0; r < p.h_counts[i]; r += 128)
            tiles.push_back(LatentTile{row + r, p.h_base[i] + r, std::min(128, p.h_counts[i] - r), sp.ctx0, sp.pos0});
        spans.push_back(sp);
        ctx += sp.count;
        row += p.h_counts[i];
        longest = std::max(longest, sp.count);
    }
    B2_CHECK_ARG(ctx <= m.ctx_rows, "latent attention: %d context rows exceed the staging buffer (%d)", ctx, m.ctx_rows);
    const int W = sh.window > 0 ? sh.window : 1 << 30;
    std::stable_sort(tiles.begin(), tiles.end(), [&](const LatentTile& x, const LatentTile& y) {     // most keys first
        return std::min(x.q_pos0 + 1, W) + x.n_rows > std::min(y.q_pos0 + 1, W) + y.n_rows;
    });
    auto same = [&] {
        if (m.staged_layer != run.pool_layer || m.staged.size() != spans.size()) return false;
        for (size_t i = 0; i < spans.size(); ++i)
            if (std::memcmp(&m.staged[i], &spans[i], sizeof(LatentSpan)) != 0) return false;
        return true;
    };
    if (!same()) {
        B2_CUDA(cudaMemcpyAsync(m.spans(), spans.data(), spans.size() * sizeof(LatentSpan), cudaMemcpyHostToDevice, s));
        B2_TRY(launch_latent_stage(sh, cache, m.spans(), (int)spans.size(), longest, m.c_stage.p, m.r_stage.p, s));
        m.staged_layer = run.pool_layer;
        m.staged = spans;
    }
    B2_CUDA(cudaMemcpyAsync(m.tiles(), tiles.data(), tiles.size() * sizeof(LatentTile), cudaMemcpyHostToDevice, s));
    const int kcols = sh.heads * sh.dp, vcols = sh.heads * sh.vp;
    B2_TRY(gemm_typed(s, m.c_stage.p, sh.rank, op.w_uk.p, m.k_up.p, kcols, op.elem, op.elem, ctx, kcols, sh.rank));
    B2_TRY(gemm_typed(s, m.c_stage.p, sh.rank, op.w_uv.p, m.v_up.p, vcols, op.elem, op.elem, ctx, vcols, sh.rank));
    ProfScope prof(PROF_FA_PREFILL, s);
    return launch_latent_prefill(sh, m.q.p, p.rows, m.k_up.p, m.r_stage.p, m.v_up.p, ctx, m.tiles(), (int)tiles.size(), m.mixed.p, m.error.i(), s);
}

static int latent_forward(BlockModel& m, LatentOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s) {
    const LatentShape& sh = op.sh;
    const int W = m.cfg.width;
    const LatentView cache = m.pool->latent_view(run.pool_layer);
    B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.pitch(), op.elem, ELEM_F32, p.rows, sh.pitch(), W));
    return !p.decode && op.tc_prefill ? latent_expanded(m, op, run, p, cache, s) : latent_absorbed(m, op, p, cache, s);
}

static int run_layers(BlockModel& m, const PassRows& p, cudaStream_t s) {
    const int W = m.cfg.width, R = p.rows;
    const float eps = (float)m.cfg.norm_eps;
    const bool pre = m.cfg.pre_norm != 0;
    m.staged_layer = -1;
    for (RotTable& t : m.rot)
        if (t.half > 0) B2_TRY(launch_rot_table(p.row_pos, (const double*)t.freq.p, t.half, R, (float2*)t.cs.p, s));
    if (m.x0.bytes) B2_CUDA(cudaMemcpyAsync(m.x0.p, m.x.p, (size_t)R * W * 4, cudaMemcpyDeviceToDevice, s));
    // A sublayer's last product: into y, whose norm is added to x, or straight onto x.
    auto out = [&](const void* in, int cols, const DevBuf& w, const DevBuf& norm) -> int {
        if (pre) return gemm_typed(s, in, cols, w.p, m.x.p, W, m.elem, ELEM_F32, R, W, cols, 1.0f);
        B2_TRY(gemm_typed(s, in, cols, w.p, m.y.p, W, m.elem, ELEM_F32, R, W, cols));
        return launch_post_norm_residual(m.elem, m.y.f(), norm.f(), eps, R, W, m.x.f(), m.xt.p, s);
    };
    for (size_t i = 0; i < m.runs.size(); ++i) {
        if (m.stop_after >= 0 && (int)i >= m.stop_after) break;
        const LayerRun& run = m.runs[i];
        BlockLayer& L = m.layers[run.layer];
        if (pre) B2_TRY(launch_pre_norm(m.elem, m.x.f(), run.add_embedding ? m.x0.f() : nullptr, L.norm1.f(), eps, R, W, m.xt.p, s));
        if (L.mlstm) {
            const MlstmShape& sh = L.mlstm->sh;
            B2_TRY(sh.gated ? mlstm_forward(m, *L.mlstm, run, p, s) : lightning_forward(m, *L.mlstm, run, p, s));
            B2_TRY(out(m.mixed.p, sh.heads * sh.vp, L.mlstm->w_out, L.norm1));
        } else if (L.latent) {
            B2_TRY(latent_forward(m, *L.latent, run, p, s));
            B2_TRY(out(m.mixed.p, L.latent->sh.heads * L.latent->sh.vp, L.latent->w_out, L.norm1));
        } else if (L.delta) {
            B2_TRY(delta_forward(m, *L.delta, run, p, s));
            B2_TRY(out(m.mixed.p, L.delta->sh.heads * L.delta->sh.vp, L.delta->w_out, L.norm1));
        } else {
            B2_TRY(diff_forward(m, *L.diff, run, p, s));
            B2_TRY(out(m.mixed.p, L.diff->sh.heads * L.diff->sh.vp, L.diff->w_out, L.norm1));
        }
        if (L.ff == 0) continue;
        if (pre) B2_TRY(launch_pre_norm(m.elem, m.x.f(), nullptr, L.norm2.f(), eps, R, W, m.xt.p, s));
        B2_TRY(gemm_typed(s, m.xt.p, W, L.w_gu.p, m.gu.p, 2 * L.ff, m.elem, m.elem, R, 2 * L.ff, W));
        B2_TRY(launch_act_mul(m.elem, L.act, m.gu.p, R, L.ff, m.act.p, s));
        B2_TRY(out(m.act.p, L.ff, L.w_down, L.norm2));
    }
    if (m.pool)
        B2_TRY(launch_lens_advance(m.pool->d_lens, m.pool->cfg.num_layers, m.cfg.max_seqs, p.d_slots, p.decode ? nullptr : p.d_seqs, p.n_seqs, s));
    return 0;
}

int block_decode_rows(BlockModel& m, int n, const int* d_tokens, const int* d_slots, cudaStream_t s) {
    PassRows p;
    p.decode = true;
    p.rows = p.n_seqs = n;
    p.max_count = 1;
    p.d_slots = d_slots;
    p.row_slot = m.row_slot();
    p.row_pos = m.row_pos();
    B2_TRY(launch_embed_scaled(m.elem, d_tokens, m.embed.p, m.cfg.vocab_size, m.cfg.width, (float)m.cfg.embed_scale, n, d_slots,
                               m.pool ? m.pool->d_lens : nullptr, m.cfg.max_seqs, m.row_slot(), m.row_pos(), m.x.f(), m.xt.p, s));
    return run_layers(m, p, s);
}

int block_pass_sequences(BlockModel& m, int n_seqs, const int* h_slots, const int* h_counts, int* n_out) {
    std::vector<int> base(n_seqs, 0);
    if (m.pool) {
        B2_TRY(m.pool->sync_lens());
        for (int i = 0; i < n_seqs; ++i) base[i] = m.pool->h_lens[h_slots[i]];
    }
    long long rows = 0;
    std::vector<long long> ctx(m.layers.size(), 0);
    int n = 0;
    for (; n < n_seqs && n < m.max_spans; ++n) {
        rows += h_counts[n];
        bool fits = rows <= m.max_rows;
        for (size_t l = 0; l < m.layers.size(); ++l)
            if (m.layers[l].latent && m.layers[l].latent->tc_prefill) {
                ctx[l] += context_span(m.layers[l].latent->sh, 0, base[n], h_counts[n], 0).count;
                fits = fits && ctx[l] <= m.ctx_rows;
            }
        if (!fits) break;
    }
    if (n == 0) B2_FAIL(B200ATTN_ERR_INVALID, "a prompt portion of %d tokens exceeds a pass of %d rows", h_counts[0], m.max_rows);
    *n_out = n;
    return 0;
}

int block_prefill_rows(BlockModel& m, int n_seqs, const int* h_slots, const int* h_counts, const int* d_tokens, cudaStream_t s) {
    PassRows p;
    std::vector<LaSeqMeta> seqs(n_seqs);
    std::vector<int> base(n_seqs, 0);
    if (m.pool) B2_TRY(m.pool->sync_lens());
    B2_CHECK_ARG(n_seqs > 0 && n_seqs <= m.max_spans, "prefill: %d sequences in one pass, at most %d", n_seqs, m.max_spans);
    for (int i = 0; i < n_seqs; ++i) {
        B2_CHECK_ARG(h_counts[i] > 0 && h_slots[i] >= 0 && h_slots[i] < m.cfg.max_seqs, "prefill: bad slot or count");
        if (m.pool) {
            base[i] = m.pool->h_lens[h_slots[i]];
            B2_CHECK_ARG(base[i] + h_counts[i] <= m.pool->h_capacity[h_slots[i]], "prefill: %d + %d tokens exceed the pages of slot %d", base[i],
                         h_counts[i], h_slots[i]);
        }
        seqs[i] = LaSeqMeta{h_slots[i], p.rows, h_counts[i]};
        p.rows += h_counts[i];
        p.max_count = std::max(p.max_count, h_counts[i]);
    }
    B2_CHECK_ARG(p.rows <= m.max_rows, "prefill: %d rows exceed a pass of %d", p.rows, m.max_rows);
    B2_CUDA(cudaMemcpyAsync(m.seqs(), seqs.data(), seqs.size() * sizeof(LaSeqMeta), cudaMemcpyHostToDevice, s));
    p.n_seqs = n_seqs;
    p.d_seqs = m.seqs();
    p.h_slots = h_slots;
    p.h_counts = h_counts;
    p.h_base = base.data();
    p.row_slot = m.row_slot();
    p.row_pos = m.row_pos();
    B2_TRY(launch_row_map(p.d_seqs, n_seqs, p.max_count, m.pool ? m.pool->d_lens : nullptr, m.row_slot(), m.row_pos(), s));
    B2_TRY(launch_embed_scaled(m.elem, d_tokens, m.embed.p, m.cfg.vocab_size, m.cfg.width, (float)m.cfg.embed_scale, p.rows, nullptr, nullptr,
                               m.cfg.max_seqs, nullptr, nullptr, m.x.f(), m.xt.p, s));
    B2_TRY(run_layers(m, p, s));
    if (m.pool)
        for (int l = 0; l < m.pool->cfg.num_layers; ++l)
            for (int i = 0; i < n_seqs; ++i) m.pool->h_lens[(size_t)l * m.cfg.max_seqs + h_slots[i]] += h_counts[i];
    return 0;
}

int block_logits(BlockModel& m, int n, const int* d_row_index, float* d_logits, cudaStream_t s) {
    const int W = m.cfg.width;
    B2_TRY(launch_rms_norm_rows(m.elem, m.x.f(), d_row_index, m.final_norm.f(), (float)m.cfg.norm_eps, n, W, m.xt.p, s));
    B2_TRY(gemm_typed(s, m.xt.p, W, m.cfg.own_head ? m.head.p : m.embed.p, d_logits, m.cfg.vocab_size, m.elem, ELEM_F32, n, m.cfg.vocab_size, W, 0.f,
                      (float)m.cfg.logit_scale));
    return m.cfg.logit_softcap > 0 ? launch_softcap(d_logits, (size_t)n * m.cfg.vocab_size, (float)m.cfg.logit_softcap, s) : 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200attn_stack_set_tensor(b200attn_stack st, const char* name, const void* h_data, int dtype, long long rows, long long cols) {
    B2_CHECK_ARG(st && name && h_data && rows > 0 && cols > 0, "stack_set_tensor: bad argument");
    B2_CHECK_ARG(st->blocks, "stack_set_tensor: not a layer-described stack");
    B2_CHECK_ARG(dtype == B200ATTN_DTYPE_BF16 || dtype == B200ATTN_DTYPE_F32, "stack_set_tensor: bad dtype");
    return set_tensor(*st->blocks, name, Source{h_data, dtype == B200ATTN_DTYPE_F32, rows, cols});
}

extern "C" int b200attn_stack_residual(b200attn_stack st, int rows, float* d_out, int stop_after, b200attn_stream stream) {
    B2_CHECK_ARG(st && st->blocks, "stack_residual: not a layer-described stack");
    BlockModel& m = *st->blocks;
    B2_CHECK_ARG(rows >= 0 && rows <= m.max_rows && (rows == 0 || d_out), "stack_residual: bad argument");
    if (rows > 0) B2_CUDA(cudaMemcpyAsync(d_out, m.x.p, (size_t)rows * m.cfg.width * 4, cudaMemcpyDeviceToDevice, as_stream(stream)));
    if (stop_after >= -1) m.stop_after = stop_after;
    return 0;
}
