// Mixers of layers with norms on their inputs: construction, weights by name, and the launches of a pass.
#include "stack.cuh"
#include "elem.cuh"

#include <algorithm>
#include <cmath>

namespace b200 {

// ---- lightning attention: the matrix memory of mlstm.cu with one constant decay per head -----------------------------------------
int make_lightning(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, MlstmOp& op, BlockSizes& z) {
    B2_CHECK_ARG(d.heads > 0 && d.dim > 0 && d.vdim > 0 && d.decay, "lightning layer: bad sizes");
    op.elem = elem;
    op.width = c.width;
    MlstmShape& sh = op.sh;
    sh.heads = d.heads; sh.dim = d.dim; sh.vdim = d.vdim;
    sh.eps = (float)c.norm_eps;
    sh.gated = false;
    sh.n_vt = ceil_div(d.vdim, kMlstmTile);
    sh.vt = sh.n_vt == 1 ? round_up(d.vdim, 4) : kMlstmTile;
    sh.dp = round_up(d.dim, 64); sh.vp = round_up(d.vdim, 64);
    op.chunk = elem == ELEM_BF16 && mlstm_chunk_fits(sh);
    if (!op.chunk) { sh.dp = round_up(d.dim, 8); sh.vp = round_up(d.vdim, 8); }
    const size_t e = elem_bytes(elem);
    std::vector<float> dec(2 * (size_t)d.heads);
    for (int h = 0; h < d.heads; ++h) {
        B2_CHECK_ARG(d.decay[h] >= 0.0 && d.decay[h] <= 1.0, "lightning layer: decay %g outside [0, 1]", d.decay[h]);
        dec[h] = (float)d.decay[h];
        dec[d.heads + h] = (float)std::max(std::log(d.decay[h]), -200.0);    // a decay of zero: nothing survives one token either way
    }
    B2_TRY(op.w_in.alloc((size_t)sh.pitch() * c.width * e));
    B2_TRY(op.w_out.alloc((size_t)c.width * sh.heads * sh.vp * e));
    B2_TRY(op.bias.alloc(dec.size() * 4));
    B2_CUDA(cudaMemcpy(op.bias.p, dec.data(), dec.size() * 4, cudaMemcpyHostToDevice));
    z.proj = std::max(z.proj, (size_t)sh.pitch());
    z.mixed = std::max(z.mixed, (size_t)sh.heads * sh.vp);
    z.core = std::max(z.core, (size_t)sh.heads * sh.vp);
    return op.norm_w.alloc((size_t)sh.heads * sh.vp * 4);
}

int set_lightning(MlstmOp& op, const std::string& n, const char* name, const Source& t) {
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
    if (n == "o") return put_out(op.w_out, op.elem, name, t, W, H, sh.vdim, sh.vp);
    if (n == "norm") {
        B2_TRY(check_shape(t, name, (long long)H * sh.vdim, 1));
        return put(op.norm_w, ELEM_F32, sh.vp, 0, 0, Source{t.data, t.f32, H, sh.vdim}, 0, 0, H, sh.vdim);
    }
    B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': a lightning layer has no such tensor", name);
}

int lightning_forward(BlockModel& m, MlstmOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s) {
    const MlstmShape& sh = op.sh;
    const int W = m.cfg.width;
    float* state = m.state->d_recurrent + m.state->block_offset[run.state_layer];
    if (!p.decode && op.chunk && p.max_count >= 16) {
        B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.cols(), op.elem, ELEM_BF16, p.rows, sh.cols(), W));
        B2_TRY(launch_silu_cols(op.elem, m.proj.p, p.rows, sh.off_g(), sh.cols(), s));
        {
            ProfScope prof(PROF_LA_PREFILL, s);
            B2_TRY(launch_mlstm_chunk(sh, m.proj.p, p.rows, nullptr, 0, op.bias.f(), p.d_seqs, p.n_seqs, m.cfg.max_seqs, state, m.core.f(), m.error.i(), s));
        }
        return launch_row_norm_gate(op.elem, sh, m.core.f(), m.proj.p, false, sh.cols(), op.norm_w.f(), p.rows, m.mixed.p, s);
    }
    B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.pitch(), op.elem, ELEM_F32, p.rows, sh.pitch(), W));
    MlstmStepArgs a{sh, m.proj.f(), op.bias.f(), op.norm_w.f(), state, p.decode ? p.d_slots : nullptr, p.decode ? nullptr : p.d_seqs, m.cfg.max_seqs,
                    m.core.f(), m.mixed.p};
    B2_TRY(launch_mlstm_step(op.elem, a, p.n_seqs, s));
    return launch_row_norm_gate(op.elem, sh, m.core.f(), m.proj.p, true, sh.pitch(), op.norm_w.f(), p.rows, m.mixed.p, s);
}

// ---- gated delta rule with a decay per key channel ------------------------------------------------------------------------------
int make_delta(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, DeltaOp& op, BlockSizes& z) {
    B2_CHECK_ARG(d.heads > 0 && d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.dim > 0 && d.vdim > 0 && d.conv_taps > 0 && d.a_rank > 0 && d.g_rank > 0,
                 "channel-delta layer: bad sizes");
    op.elem = elem;
    op.width = c.width;
    DeltaShape& sh = op.sh;
    sh.heads = d.heads; sh.kv_heads = d.kv_heads; sh.dim = d.dim; sh.vdim = d.vdim; sh.taps = d.conv_taps; sh.a_rank = d.a_rank; sh.g_rank = d.g_rank;
    sh.eps = (float)c.norm_eps;
    sh.dp = round_up(d.dim, 8); sh.vp = round_up(d.vdim, 8); sh.ap = round_up(d.a_rank, 8); sh.gp = round_up(d.g_rank, 8);
    sh.n_vt = ceil_div(d.vdim, kMlstmTile);
    sh.vt = sh.n_vt == 1 ? round_up(d.vdim, 4) : kMlstmTile;
    if ((3 * (size_t)round_up(d.dim, 4) + 17 * kMlstmTile + 32 + sh.hist_floats()) * 4 > 200 * 1024)
        B2_FAIL(B200ATTN_ERR_UNSUPPORTED, "channel-delta layer: %d taps of %d key channels exceed shared memory", d.conv_taps, d.dim);
    const size_t e = elem_bytes(elem);
    B2_TRY(op.w_in.alloc((size_t)sh.pitch() * c.width * e));
    B2_TRY(op.w_low.alloc((size_t)sh.low() * c.width * e));
    B2_TRY(op.w_gate.alloc((size_t)sh.gate_cols() * sh.low() * e));      // block diagonal: decay gates from the first inner columns, output gates from the others
    B2_TRY(op.w_out.alloc((size_t)c.width * sh.heads * sh.vp * e));
    B2_TRY(op.conv.alloc((size_t)sh.off_b() * sh.taps * 4));
    if (sh.taps <= 4) B2_TRY(op.conv4.alloc((size_t)4 * sh.off_b() * 4));
    B2_TRY(op.a_log.alloc((size_t)sh.heads * 4));
    B2_TRY(op.dt_bias.alloc((size_t)sh.heads * sh.dp * 4));
    z.proj = std::max(z.proj, (size_t)sh.pitch());
    z.low = std::max(z.low, (size_t)sh.low());
    z.gates = std::max(z.gates, (size_t)sh.gate_cols());
    z.mixed = std::max(z.mixed, (size_t)sh.heads * sh.vp);
    op.chunk = elem == ELEM_BF16 && delta_chunk_fits(sh);
    if (op.chunk) {
        z.gates = std::max(z.gates, (size_t)sh.gate_cols() + sh.heads);
        z.chunk = std::max(z.chunk, delta_chunk_bytes(sh));
    }
    if (op.chunk || sh.n_vt > 1) z.core = std::max(z.core, (size_t)sh.heads * sh.vp);
    return op.norm_w.alloc((size_t)sh.vp * 4);
}

int set_delta(DeltaOp& op, const std::string& n, const char* name, const Source& t) {
    const DeltaShape& sh = op.sh;
    const int W = op.width, H = sh.heads, G = sh.kv_heads;
    struct Part { const char* n; int row0, heads, size, stride; };
    for (const Part& p : {Part{"q", 0, G, sh.dim, sh.dp}, Part{"k", sh.off_k(), G, sh.dim, sh.dp}, Part{"v", sh.off_v(), H, sh.vdim, sh.vp},
                          Part{"b", sh.off_b(), H, 1, 1}}) {
        if (n == p.n) {
            B2_TRY(check_shape(t, name, (long long)p.heads * p.size, W));
            return put_heads(op.w_in, op.elem, p.row0, p.stride, t, p.heads, p.size, W, p.size, 0);
        }
        if (n == std::string(p.n) + ".conv" && n != "b.conv") {
            B2_TRY(check_shape(t, name, (long long)p.heads * p.size, sh.taps));
            for (int j = 0; j < sh.taps && sh.taps <= 4; ++j)
                for (int h = 0; h < p.heads; ++h)
                    B2_TRY(put(op.conv4, ELEM_F32, 1, (size_t)(4 - sh.taps + j) * sh.off_b() + p.row0 + (size_t)h * p.stride, 0, t, (size_t)h * p.size, j, p.size, 1));
            return put_heads(op.conv, ELEM_F32, p.row0, p.stride, t, p.heads, p.size, sh.taps, p.size, 0);
        }
    }
    if (n == "a1" || n == "g1") {
        const int rank = n == "a1" ? sh.a_rank : sh.g_rank;
        B2_TRY(check_shape(t, name, rank, W));
        return put(op.w_low, op.elem, W, n == "a1" ? 0 : sh.ap, 0, t, 0, 0, rank, W);
    }
    if (n == "a2" || n == "g2") {
        const bool a = n == "a2";
        const int size = a ? sh.dim : sh.vdim, stride = a ? sh.dp : sh.vp, rank = a ? sh.a_rank : sh.g_rank;
        B2_TRY(check_shape(t, name, (long long)H * size, rank));
        for (int h = 0; h < H; ++h)
            B2_TRY(put(op.w_gate, op.elem, sh.low(), (a ? 0 : H * sh.dp) + (size_t)h * stride, a ? 0 : sh.ap, t, (size_t)h * size, 0, size, rank));
        return 0;
    }
    if (n == "A_log") return put_vector(op.a_log, name, t, 0, H);
    if (n == "dt_bias") {
        B2_TRY(check_shape(t, name, (long long)H * sh.dim, 1));
        return put(op.dt_bias, ELEM_F32, sh.dp, 0, 0, Source{t.data, t.f32, H, sh.dim}, 0, 0, H, sh.dim);
    }
    if (n == "norm") return put_vector(op.norm_w, name, t, 0, sh.vdim);
    if (n == "o") return put_out(op.w_out, op.elem, name, t, W, H, sh.vdim, sh.vp);
    B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': a channel-delta layer has no such tensor", name);
}

int delta_forward(BlockModel& m, DeltaOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s) {
    const DeltaShape& sh = op.sh;
    const int W = m.cfg.width;
    float* state = m.state->d_recurrent + m.state->block_offset[run.state_layer];
    B2_TRY(gemm_typed(s, m.xt.p, W, op.w_low.p, m.low.p, sh.low(), op.elem, op.elem, p.rows, sh.low(), W));
    if (!p.decode && op.chunk && p.max_count >= 16) {
        // q | k | v in bf16; decay and beta pre-activations in fp32, those of the output gate in bf16 behind them
        const int acols = sh.heads * sh.dp, gcols = sh.heads * sh.vp, qkv = sh.off_b();
        float *a = m.gates.f(), *b = a + (size_t)p.rows * acols;
        void* g = b + ((size_t)p.rows * sh.heads + 3) / 4 * 4;
        const size_t e = elem_bytes(op.elem);
        B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, qkv, op.elem, op.elem, p.rows, qkv, W));
        B2_TRY(gemm_typed(s, m.xt.p, W, (const char*)op.w_in.p + (size_t)qkv * W * e, b, sh.heads, op.elem, ELEM_F32, p.rows, sh.heads, W));
        B2_TRY(gemm_typed(s, m.low.p, sh.low(), op.w_gate.p, a, acols, op.elem, ELEM_F32, p.rows, acols, sh.low()));
        B2_TRY(gemm_typed(s, m.low.p, sh.low(), (const char*)op.w_gate.p + (size_t)acols * sh.low() * e, g, gcols, op.elem, op.elem, p.rows, gcols, sh.low()));
        {
            ProfScope prof(PROF_DELTA_PREFILL, s);
            B2_TRY(launch_delta_chunk(sh, m.proj.p, a, b, sh.taps <= 4 ? op.conv4.f() : op.conv.f(), op.a_log.f(), op.dt_bias.f(), p.d_seqs, p.n_seqs, p.max_count, p.rows, m.cfg.max_seqs, state,
                                      m.chunk.p, m.core.f(), m.error.i(), s));
        }
        return launch_delta_head_norm(op.elem, sh, m.core.f(), g, false, gcols, op.norm_w.f(), p.rows, m.mixed.p, s);
    }
    B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.pitch(), op.elem, ELEM_F32, p.rows, sh.pitch(), W));
    B2_TRY(gemm_typed(s, m.low.p, sh.low(), op.w_gate.p, m.gates.p, sh.gate_cols(), op.elem, ELEM_F32, p.rows, sh.gate_cols(), sh.low()));
    DeltaStepArgs a{sh, m.proj.f(), m.gates.f(), op.conv.f(), sh.taps <= 4 ? op.conv4.f() : nullptr, op.a_log.f(), op.dt_bias.f(), op.norm_w.f(), state, p.decode ? p.d_slots : nullptr,
                    p.decode ? nullptr : p.d_seqs, m.cfg.max_seqs, m.core.f(), m.mixed.p};
    B2_TRY(launch_delta_step(op.elem, a, p.n_seqs, s));
    if (sh.n_vt > 1)
        B2_TRY(launch_delta_head_norm(op.elem, sh, m.core.f(), m.gates.f() + sh.heads * sh.dp, true, sh.gate_cols(), op.norm_w.f(), p.rows, m.mixed.p, s));
    return 0;
}

// ---- differential attention -------------------------------------------------------------------------------------------------------
int make_diff(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, DiffOp& op, BlockSizes& z) {
    B2_CHECK_ARG(d.heads > 0 && d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.dim > 0 && d.vdim > 0 && d.rot_dim >= 0 && d.rot_dim % 2 == 0 &&
                     d.rot_dim <= d.dim && d.window >= 0 && d.keep_first >= 0, "differential-attention layer: bad sizes");
    if (d.vdim > 1024) B2_FAIL(B200ATTN_ERR_UNSUPPORTED, "differential-attention layer: vdim %d above 1024", d.vdim);
    op.elem = elem;
    op.width = c.width;
    DiffShape& sh = op.sh;
    sh.heads = d.heads; sh.kv_heads = d.kv_heads; sh.dim = d.dim; sh.vdim = d.vdim; sh.rot = d.rot_dim; sh.window = d.window; sh.keep = d.keep_first;
    sh.scale = (float)d.scale; sh.eps = (float)c.norm_eps; sh.diff = (float)d.diff;
    sh.dp = round_up(d.dim, 64); sh.vp = round_up(d.vdim, 64);
    op.tc_prefill = elem == ELEM_BF16 && diff_prefill_fits(sh);
    if (!op.tc_prefill) { sh.dp = round_up(d.dim, 8); sh.vp = round_up(d.vdim, 8); }
    op.tc_decode = elem == ELEM_BF16 && diff_decode_fits(sh, c.max_seqs);
    const size_t e = elem_bytes(elem);
    B2_TRY(op.w_in.alloc((size_t)sh.pitch() * c.width * e));
    B2_TRY(op.w_out.alloc((size_t)c.width * sh.heads * sh.vp * e));
    B2_TRY(op.q_norm.alloc((size_t)sh.dp * 4));
    z.proj = std::max(z.proj, (size_t)sh.pitch());
    z.mixed = std::max(z.mixed, (size_t)sh.heads * sh.vp);
    z.q = std::max(z.q, (size_t)sh.q_cols());
    if (op.tc_decode) {
        z.qa = std::max(z.qa, (size_t)sh.kv_heads * 16 * sh.qp());
        z.part = std::max(z.part, diff_decode_scratch_floats(sh, c.max_seqs));
        z.counters = std::max(z.counters, (size_t)c.max_seqs * sh.kv_heads);
    }
    return op.k_norm.alloc((size_t)sh.dp * 4);
}

int set_diff(DiffOp& op, const std::string& n, const char* name, const Source& t) {
    const DiffShape& sh = op.sh;
    const int W = op.width;
    struct Part { const char* n; int row0, heads, size, stride; };
    for (const Part& p : {Part{"q", 0, 2 * sh.heads, sh.dim, sh.dp}, Part{"k", sh.off_k(), 2 * sh.kv_heads, sh.dim, sh.dp},
                          Part{"v", sh.off_v(), sh.kv_heads, sh.vdim, sh.vp}})
        if (n == p.n) {
            B2_TRY(check_shape(t, name, (long long)p.heads * p.size, W));
            return put_heads(op.w_in, op.elem, p.row0, p.stride, t, p.heads, p.size, W, p.size, 0);
        }
    if (n == "q.norm") return put_vector(op.q_norm, name, t, 0, sh.dim);
    if (n == "k.norm") return put_vector(op.k_norm, name, t, 0, sh.dim);
    if (n == "o") return put_out(op.w_out, op.elem, name, t, W, sh.heads, sh.vdim, sh.vp);
    const char* lam[4] = {"lq1", "lk1", "lq2", "lk2"};
    for (int i = 0; i < 4; ++i)
        if (n == lam[i]) {
            B2_TRY(check_shape(t, name, sh.dim, 1));
            op.lam[i].resize(sh.dim);
            for (int c = 0; c < sh.dim; ++c) op.lam[i][c] = t.at(c);
            double dot[2] = {0.0, 0.0};
            for (int k = 0; k < 2; ++k)
                for (size_t c = 0; c < std::min(op.lam[2 * k].size(), op.lam[2 * k + 1].size()); ++c) dot[k] += (double)op.lam[2 * k][c] * op.lam[2 * k + 1][c];
            op.lambda = (float)(std::exp(dot[0]) - std::exp(dot[1]) + sh.diff);      // complete once all four are there
            return 0;
        }
    B2_FAIL(B200ATTN_ERR_INVALID, "tensor '%s': a differential-attention layer has no such tensor", name);
}

int diff_forward(BlockModel& m, DiffOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s) {
    const DiffShape& sh = op.sh;
    const int W = m.cfg.width;
    const LatentView cache = m.pool->latent_view(run.pool_layer);
    B2_TRY(gemm_typed(s, m.xt.p, W, op.w_in.p, m.proj.p, sh.pitch(), op.elem, ELEM_F32, p.rows, sh.pitch(), W));
    const bool split = p.decode && op.tc_decode;
    DiffPreArgs a{sh, m.proj.f(), (const float2*)m.rot[op.rot_table].cs.p, op.q_norm.f(), op.k_norm.f(), p.row_slot, p.row_pos, cache, m.q.p,
                  split ? m.qa.p : nullptr};
    B2_TRY(launch_diff_pre(op.elem, a, p.rows, s));
    if (split) return launch_diff_decode(sh, op.lambda, m.qa.p, cache, p.row_slot, p.row_pos, p.rows, m.part.f(), m.counters.i(), m.mixed.p, s);
    if (!p.decode && op.tc_prefill) {
        std::vector<DiffTile> tiles;
        for (int i = 0, row = 0; i < p.n_seqs; row += p.h_counts[i++])
            for (int r = 0; r < p.h_counts[i]; r += 128) tiles.push_back(DiffTile{row + r, p.h_base[i] + r, std::min(128, p.h_counts[i] - r), p.h_slots[i]});
        const int most = sh.window > 0 ? sh.window : 1 << 30;
        std::stable_sort(tiles.begin(), tiles.end(), [&](const DiffTile& x, const DiffTile& y) {      // most keys first
            return std::min(x.q_pos0 + 1, most) + x.n_rows > std::min(y.q_pos0 + 1, most) + y.n_rows;
        });
        B2_CUDA(cudaMemcpyAsync(m.tiles(), tiles.data(), tiles.size() * sizeof(DiffTile), cudaMemcpyHostToDevice, s));
        ProfScope prof(PROF_FA_PREFILL, s);
        return launch_diff_prefill(sh, op.lambda, m.q.p, p.rows, cache, reinterpret_cast<const DiffTile*>(m.tiles()), (int)tiles.size(), m.mixed.p, m.error.i(), s);
    }
    return launch_diff_attn_rows(op.elem, sh, op.lambda, m.q.p, cache, p.row_slot, p.row_pos, p.rows, m.mixed.p, s);
}

}  // namespace b200
