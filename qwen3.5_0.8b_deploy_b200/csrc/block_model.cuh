// Models given by a list of layer descriptions: the operators, the working buffers and the layer loop behind
// b200attn_stack_create_layers.  A layer is a mixer and a feed-forward, with RMS norms on the sublayers' outputs
// (x += norm1(mixer(x)): the sublayers read the residual stream itself) or on their inputs (x += mixer(norm1(x)): the last
// product of a sublayer adds to the residual stream).  Sizes and constants come from the description; element types are
// bf16 (serving) or fp32; the residual stream, norms, positions, scores and recurrent state are fp32 in both.
#pragma once

#include "kernels.cuh"

#include <memory>
#include <string>
#include <vector>

namespace b200 {

constexpr int round_up(int v, int a) { return (v + a - 1) / a * a; }

// Device buffer freed with its owner.
struct DevBuf {
    void* p = nullptr;
    size_t bytes = 0;
    DevBuf() = default;
    DevBuf(const DevBuf&) = delete;
    DevBuf& operator=(const DevBuf&) = delete;
    DevBuf(DevBuf&& o) noexcept : p(o.p), bytes(o.bytes) { o.p = nullptr; o.bytes = 0; }
    ~DevBuf() { cudaFree(p); }
    int alloc(size_t n) {            // zeroed
        cudaFree(p);
        p = nullptr;
        bytes = n;
        B2_CUDA(cudaMalloc(&p, n ? n : 16));
        B2_CUDA(cudaMemset(p, 0, n ? n : 16));
        return 0;
    }
    float* f() const { return static_cast<float*>(p); }
    int* i() const { return static_cast<int*>(p); }
};

// The rows of one pass.  Prefill: h_* describe the sequences, d_seqs is their device copy.  Decode: one row per entry of
// d_slots (-1 = inactive).  row_slot / row_pos hold every row's slot and position in both.
struct PassRows {
    bool decode = false;
    int rows = 0, n_seqs = 0;
    const int* d_slots = nullptr;
    const LaSeqMeta* d_seqs = nullptr;
    const int* h_slots = nullptr;
    const int* h_counts = nullptr;
    const int* h_base = nullptr;       // tokens each sequence held before the pass
    const int* row_slot = nullptr;
    const int* row_pos = nullptr;
    int max_count = 0;
};

// ---- block_kernels.cu: element-wise steps around the mixers -----------------------------------------------------------
int launch_row_map(const LaSeqMeta* d_seqs, int n_seqs, int max_count, const int* lens, int* row_slot, int* row_pos, cudaStream_t s);
// table[row][i] = (cos, sin) of row_pos[row] * freq[i].
int launch_rot_table(const int* row_pos, const double* freq, int half, int rows, float2* table, cudaStream_t s);
// x = embed[token] * scale, with a copy in the element type; decode also fills row_slot / row_pos from d_slots and lens.
int launch_embed_scaled(ElemType t, const int* tokens, const void* embed, int vocab, int width, float scale, int rows, const int* d_slots,
                        const int* lens, int max_seqs, int* row_slot, int* row_pos, float* x, void* xt, cudaStream_t s);
// x += y / rms(y) * w, with a copy in the element type.
int launch_post_norm_residual(ElemType t, const float* y, const float* w, float eps, int rows, int width, float* x, void* xt, cudaStream_t s);
// out = x[row_index] / rms * w in the element type (row_index may be null).
int launch_rms_norm_rows(ElemType t, const float* x, const int* row_index, const float* w, float eps, int rows, int width, void* out,
                         cudaStream_t s);
// x += add (may be null), out = x / rms * w in the element type.
int launch_pre_norm(ElemType t, float* x, const float* add, const float* w, float eps, int rows, int width, void* out, cudaStream_t s);
// act = f(gate) * up over rows of [gate | up], f a b200attn_act.
int launch_act_mul(ElemType t, int f, const void* gu, int rows, int ff, void* act, cudaStream_t s);
// logits = cap * tanh(logits / cap)
int launch_softcap(float* logits, size_t n, float cap, cudaStream_t s);
// lens[layer][slot] += count for every layer of a pool.
int launch_lens_advance(int* lens, int n_layers, int max_seqs, const int* d_slots, const LaSeqMeta* d_seqs, int n, cudaStream_t s);
int launch_argmax_rows(const float* logits, int rows, int vocab, int* out, cudaStream_t s);   // stack.cu

// ---- mlstm.cu, mlstm_chunk.cu: matrix memory with exponential gating, or with a constant decay per head -----------------------
constexpr int kMlstmTile = 128;        // value columns of one state tile
struct MlstmShape {
    int heads = 0, dim = 0, vdim = 0;
    float gate_cap = 0.f, eps = 0.f;
    bool gated = true;                 // exponential gates, normaliser and head norm; else constant decays and silu on q, k, v
    int dp = 0, vp = 0;                // head sizes in the projections, padded with zero weights
    int vt = 0, n_vt = 0;              // state tile width and tiles per head
    constexpr int off_q() const { return 0; }
    constexpr int off_k() const { return heads * dp; }
    constexpr int off_v() const { return 2 * heads * dp; }
    constexpr int off_g() const { return 2 * heads * dp + heads * vp; }
    constexpr int off_i() const { return 2 * heads * (dp + vp); }
    constexpr int off_f() const { return off_i() + heads; }
    constexpr int cols() const { return off_i(); }                             // q | k | v | g
    constexpr int pitch() const { return round_up(off_i() + (gated ? 2 * heads : 0), 4); }   // fp32 rows with the gate columns behind
    constexpr size_t tile_floats() const { return (size_t)dim * vt + round_up(dim, 4) + 4; }   // S [dim][vt], n [dim], m
    constexpr size_t state_floats() const { return tile_floats() * n_vt * heads; }
};
struct MlstmStepArgs {                 // the token-serial kernel: decode (one token a row) and plain prefill
    MlstmShape sh;
    const float* proj;                 // [rows][pitch]
    const float* bias;                 // [2 * heads]: i then f; not gated: decays, then their logarithms
    const float* norm_w;               // [heads * vp]
    float* state;
    const int* d_slots;
    const LaSeqMeta* seqs;             // prefill, else null
    int max_seqs;
    float* core;                       // [rows][heads * vp]: outputs before the head norm (several tiles per head)
    void* gated;                       // [rows][heads * vp] in the element type: after norm and gate (one tile per head)
};
int launch_mlstm_step(ElemType t, const MlstmStepArgs& a, int n, cudaStream_t s);
// gated = core / rms(head) * w * sigmoid(g); g in fp32 rows (pitch) or in the element type.
int launch_mlstm_head_norm(ElemType t, const MlstmShape& sh, const float* core, const void* g, bool g_f32, int g_pitch, const float* norm_w,
                           int rows, void* gated, cudaStream_t s);
bool mlstm_chunk_fits(const MlstmShape& sh);
int launch_mlstm_chunk(const MlstmShape& sh, const void* qkvg, int rows, const float* gates, int gate_pitch, const float* bias,
                       const LaSeqMeta* d_seqs, int n_seqs, int max_seqs, float* state, float* core, int* d_error, cudaStream_t s);

// gated = core / rms(all heads) * w * sigmoid(g): the norm of a memory that is not gated.
int launch_row_norm_gate(ElemType t, const MlstmShape& sh, const float* core, const void* g, bool g_f32, int g_pitch, const float* norm_w, int rows,
                         void* gated, cudaStream_t s);
// silu in place on the first `cols` columns (a multiple of four) of rows of `pitch` values.
int launch_silu_cols(ElemType t, void* p, int rows, int cols, int pitch, cudaStream_t s);

struct MlstmOp {
    MlstmShape sh;
    ElemType elem = ELEM_BF16;
    int width = 0;
    bool chunk = false;                // prefill through the chunked tensor-core kernel
    DevBuf w_in, w_out, bias, norm_w;
};

// ---- latent.cu, page_decode.cu, latent_prefill.cu: attention over cached latents -----------------------------------------
struct LatentShape {
    int heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0, window = 0;     // window <= 0: every earlier position
    float scale = 0.f, eps = 0.f;
    int dp = 0, rp = 0, vp = 0;        // padded head sizes of the projections
    bool own = true;                   // has latents of its own (else it reads another layer's)
    constexpr int q_cols() const { return heads * (dp + rp); }
    constexpr int pitch() const { return round_up(q_cols() + (own ? rank + rot : 0), 4); }
    constexpr int row_pitch() const { return round_up(rank + rot, 16) + 8; }       // cache rows and absorbed queries: an odd number of 16-byte units
};
struct LatentPreArgs {                 // behind the input projection: rotate q, norm and rotate the new latents, append them
    LatentShape sh;
    const float* proj;
    const float2* cs;                  // [rows][rot / 2] cos and sin of the rows' angles
    const float* c_norm;               // [rank]
    const int* row_slot;
    const int* row_pos;
    LatentView cache;
    void* q;                           // [rows][heads][dp + rp]
    void* qa;                          // [rows][heads][row_pitch]: rotated part and zero tail of the absorbed query (may be null)
};
int launch_latent_pre(ElemType t, const LatentPreArgs& a, int rows, cudaStream_t s);
// Absorbed attention, one (row, head) at a time, any size: out [rows][heads][rank].
int launch_latent_attn_rows(ElemType t, const LatentShape& sh, const void* qa, const LatentView& cache, const int* row_slot,
                            const int* row_pos, int rows, void* out, cudaStream_t s);
bool latent_decode_fits(const LatentShape& sh, int max_rows);
size_t latent_decode_scratch_floats(const LatentShape& sh, int max_rows);
int launch_latent_decode(const LatentShape& sh, const void* qa, const LatentView& cache, const int* row_slot, const int* row_pos, int rows,
                         float* part, int* counters, void* out, cudaStream_t s);
struct LatentSpan {                    // one sequence of a prefill pass: its staged context rows
    int slot, ctx0, pos0, count;       // first staging row, its position, rows
};
int launch_latent_stage(const LatentShape& sh, const LatentView& cache, const LatentSpan* d_spans, int n_spans, int max_count, void* c_stage,
                        void* r_stage, cudaStream_t s);
struct LatentTile {                    // 128 query rows of one sequence
    int q_row0, q_pos0, n_rows;
    int ctx_row0, ctx_pos0;            // staging row of context position ctx_pos0
};
bool latent_prefill_fits(const LatentShape& sh);
int launch_latent_prefill(const LatentShape& sh, const void* q, int rows, const void* k, const void* k_rot, const void* v, int ctx_rows,
                          const LatentTile* d_tiles, int n_tiles, void* out, int* d_error, cudaStream_t s);

struct LatentOp {
    LatentShape sh;
    ElemType elem = ELEM_BF16;
    int width = 0, kv_from = -1;
    bool tc_prefill = false, tc_decode = false;
    int rot_table = 0;                 // index of its rotation's table
    DevBuf w_in, w_uk, w_uv, w_out, c_norm;
};

// ---- channel_delta.cu: gated delta rule with a decay per key channel ------------------------------------------------------------
struct DeltaShape {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1, a_rank = 0, g_rank = 0;
    float eps = 0.f;
    int dp = 0, vp = 0, ap = 0, gp = 0;      // head and rank sizes padded with zero weights
    int vt = 0, n_vt = 0;                    // state tile width and tiles per head
    // fp32 rows of the input projection: q | k | v | b; the short convolutions' weights and inputs follow the first three
    constexpr int off_k() const { return kv_heads * dp; }
    constexpr int off_v() const { return 2 * kv_heads * dp; }
    constexpr int off_b() const { return off_v() + heads * vp; }
    constexpr int pitch() const { return round_up(off_b() + heads, 4); }
    constexpr int low() const { return ap + gp; }                            // inner columns of the two low-rank gates
    constexpr int gate_cols() const { return heads * (dp + vp); }            // decay | output gate pre-activations
    // a state tile: S [dim][vt], then the convolutions' last taps - 1 inputs: q [..][dim], k [..][dim], v [..][vt]
    constexpr size_t hist_floats() const { return (size_t)(taps - 1) * (2 * round_up(dim, 4) + vt); }
    constexpr size_t tile_floats() const { return (size_t)dim * vt + hist_floats(); }
    constexpr size_t state_floats() const { return tile_floats() * n_vt * heads; }
};
struct DeltaStepArgs {                 // the token-serial kernel: decode (one token a row) and plain prefill
    DeltaShape sh;
    const float* proj;                 // [rows][pitch]
    const float* gates;                // [rows][gate_cols]
    const float* conv;                 // [off_b][taps]
    const float* conv4;                // [4][off_b] with leading zeros; null with more than four taps
    const float* a_log;                // [heads]
    const float* dt_bias;              // [heads * dp]
    const float* norm_w;               // [vdim]
    float* state;
    const int* d_slots;
    const LaSeqMeta* seqs;             // prefill, else null
    int max_seqs;
    float* core;                       // [rows][heads * vp]: outputs before the head norm (several tiles per head)
    void* gated;                       // [rows][heads * vp] in the element type: after norm and gate (one tile per head)
};
int launch_delta_step(ElemType t, const DeltaStepArgs& a, int n, cudaStream_t s);
// gated = core / rms(head) * w * sigmoid(g), g in fp32 rows or in the element type.
int launch_delta_head_norm(ElemType t, const DeltaShape& sh, const float* core, const void* g, bool g_f32, int g_pitch, const float* norm_w, int rows,
                           void* gated, cudaStream_t s);

// channel_delta_chunk.cu: prefill in chunks of 64 tokens.
bool delta_chunk_fits(const DeltaShape& sh);
size_t delta_chunk_bytes(const DeltaShape& sh);        // scratch per 64 rows of a pass (and one more such piece per sequence)
// qkv: bf16 [rows][off_b]; conv: conv4 with up to four taps; a: fp32 [rows][heads * dp], b: fp32 [rows][heads], the gates' pre-activations.
int launch_delta_chunk(const DeltaShape& sh, const void* qkv, const float* a, const float* b, const float* conv, const float* a_log, const float* dt_bias,
                       const LaSeqMeta* d_seqs, int n_seqs, int max_count, int rows, int max_seqs, float* state, void* scratch, float* core, int* d_error,
                       cudaStream_t s);

struct DeltaOp {
    DeltaShape sh;
    ElemType elem = ELEM_BF16;
    int width = 0;
    bool chunk = false;                // prefill through the chunked tensor-core kernels
    DevBuf w_in, w_low, w_gate, w_out, conv, conv4, a_log, dt_bias, norm_w;     // conv4: [4][off_b], up to four taps behind leading zeros
};

// ---- diff_attn.cu, diff_prefill.cu: differential attention ----------------------------------------------------------------------
struct DiffShape {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, rot = 0, window = 0, keep = 0;    // window <= 0: every earlier position
    float scale = 0.f, eps = 0.f, diff = 0.f;
    int dp = 0, vp = 0;                // padded head sizes
    constexpr int q_cols() const { return heads * 2 * dp; }                  // projections: q | k | v, q and k [head][map][dp]
    constexpr int off_k() const { return q_cols(); }
    constexpr int off_v() const { return off_k() + kv_heads * 2 * dp; }
    constexpr int pitch() const { return round_up(off_v() + kv_heads * vp, 4); }
    constexpr int hp() const { return 2 * dp + vp + 8; }                     // cache row of a key / value head: k of both maps, v
    constexpr int row_pitch() const { return kv_heads * hp(); }              // a page holds head after head, 64 rows each
    constexpr int qp() const { return 2 * dp + 8; }                          // decode query rows, 16 per key / value head
};
struct DiffPreArgs {                   // behind the input projection: norm and rotate q and k, append keys and values
    DiffShape sh;
    const float* proj;
    const float2* cs;                  // [rows][rot / 2]
    const float *q_norm, *k_norm;      // [dim]
    const int* row_slot;
    const int* row_pos;
    LatentView cache;
    void* q;                           // [rows][heads][2][dp], or
    void* qd;                          // [rows][kv_heads][16][qp]: a group's map 1 in rows 0 .. 7, columns 0 .. dp, map 2 in the others
};
int launch_diff_pre(ElemType t, const DiffPreArgs& a, int rows, cudaStream_t s);
// Any size, one (row, head) at a time: out [rows][heads][vp].
int launch_diff_attn_rows(ElemType t, const DiffShape& sh, float lambda, const void* q, const LatentView& cache, const int* row_slot,
                          const int* row_pos, int rows, void* out, cudaStream_t s);

bool diff_decode_fits(const DiffShape& sh, int max_rows);
size_t diff_decode_scratch_floats(const DiffShape& sh, int max_rows);
int launch_diff_decode(const DiffShape& sh, float lambda, const void* qd, const LatentView& cache, const int* row_slot, const int* row_pos, int rows,
                       float* part, int* counters, void* out, cudaStream_t s);       // page_decode.cu
struct DiffTile { int q_row0, q_pos0, n_rows, slot; };      // up to 128 query rows of one sequence
bool diff_prefill_fits(const DiffShape& sh);
int launch_diff_prefill(const DiffShape& sh, float lambda, const void* q, int rows, const LatentView& cache, const DiffTile* d_tiles, int n_tiles,
                        void* out, int* d_error, cudaStream_t s);

struct DiffOp {
    DiffShape sh;
    ElemType elem = ELEM_BF16;
    int width = 0;
    bool tc_prefill = false, tc_decode = false;
    int rot_table = 0;
    float lambda = 0.f;
    std::vector<float> lam[4];         // lq1, lk1, lq2, lk2
    DevBuf w_in, w_out, q_norm, k_norm;
};

struct RotTable {                      // one rotation (base and size) of a model: filled once per pass, shared by the layers that use it
    double base = 0;
    int half = 0;
    DevBuf freq, cs;
};

// ---- block_model.cu ---------------------------------------------------------------------------------------------------------
struct BlockLayer {
    std::unique_ptr<MlstmOp> mlstm;
    std::unique_ptr<LatentOp> latent;
    std::unique_ptr<DeltaOp> delta;
    std::unique_ptr<DiffOp> diff;
    int ff = 0, act = 0;               // ff 0: no feed-forward
    DevBuf norm1, norm2, w_gu, w_down;
    std::vector<std::string> missing;  // tensors not given yet
};

struct LayerRun {                      // one run of a layer in a pass over the model
    int layer = 0;
    int state_layer = -1, pool_layer = -1;   // its block of the state pool, its layer of the cache
    bool add_embedding = false;        // first layer of a repeated pass of the loop
};

// What the mixers of a model need of the working buffers (per row unless said otherwise), gathered while its layers are made.
struct BlockSizes {
    size_t proj = 0, mixed = 0, core = 0, gates = 0, low = 0, ff = 0, q = 0, qa = 0, olat = 0, cst = 0, rst = 0, kup = 0, vup = 0;
    size_t chunk = 0;                  // bytes per 64 rows
    size_t part = 0, counters = 0;     // whole buffers
    int max_window = 0;
};

struct BlockModel {
    b200attn_model_config cfg{};
    ElemType elem = ELEM_BF16;
    std::vector<BlockLayer> layers;
    std::vector<LayerRun> runs;
    std::vector<RotTable> rot;
    std::vector<std::string> missing;
    DevBuf embed, final_norm, head;
    int stop_after = -1;               // >= 0: passes end behind that many layer runs
    int max_rows = 0, abs_rows = 0, ctx_rows = 0, max_spans = 0;
    b200attn_kv_pool pool = nullptr;   // owned by the stack
    b200attn_la_state state = nullptr;
    DevBuf x, x0, xt, low, proj, gates, core, mixed, y, gu, act, q, qa, olat, c_stage, r_stage, k_up, v_up, part, counters, chunk, meta, error;
    int* row_slot() const { return meta.i(); }
    int* row_pos() const { return meta.i() + max_rows; }
    LaSeqMeta* seqs() const { return reinterpret_cast<LaSeqMeta*>(meta.i() + 2 * (size_t)max_rows); }
    LatentSpan* spans() const { return reinterpret_cast<LatentSpan*>(meta.i() + 2 * (size_t)max_rows + 3 * (size_t)max_spans); }
    LatentTile* tiles() const { return reinterpret_cast<LatentTile*>(meta.i() + 2 * (size_t)max_rows + 7 * (size_t)max_spans); }
    // what the staging buffers hold (layers that share latents share the staged rows of a pass)
    int staged_layer = -1;
    std::vector<LatentSpan> staged;
};

// block_mixers.cu: the mixers of layers with norms on their inputs.
int make_lightning(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, MlstmOp& op, BlockSizes& z);
int make_delta(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, DeltaOp& op, BlockSizes& z);
int make_diff(const b200attn_layer_desc& d, const b200attn_model_config& c, ElemType elem, DiffOp& op, BlockSizes& z);
int set_lightning(MlstmOp& op, const std::string& n, const char* name, const struct Source& t);
int set_delta(DeltaOp& op, const std::string& n, const char* name, const struct Source& t);
int set_diff(DiffOp& op, const std::string& n, const char* name, const struct Source& t);
// A mixer reads m.xt and leaves its heads' outputs, one row of `cols` values each, in m.mixed.
int lightning_forward(BlockModel& m, MlstmOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s);
int delta_forward(BlockModel& m, DeltaOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s);
int diff_forward(BlockModel& m, DiffOp& op, const LayerRun& run, const PassRows& p, cudaStream_t s);

// ---- weights by name: host data of a tensor and the helpers that put it into device matrices ----
struct Source {
    const void* data;
    bool f32;
    long long rows, cols;
    float at(size_t i) const {
        if (f32) return static_cast<const float*>(data)[i];
        const uint32_t u = (uint32_t)static_cast<const uint16_t*>(data)[i] << 16;
        float v;
        std::memcpy(&v, &u, 4);
        return v;
    }
};
int check_shape(const Source& t, const char* name, long long rows, long long cols);
// Copies a [rows, cols] block of the source to (row0, col0) of a device matrix with row pitch ld.
int put(DevBuf& dst, ElemType elem, size_t ld, size_t row0, size_t col0, const Source& t, size_t src_row, size_t src_col, size_t rows, size_t cols);
int put_vector(DevBuf& dst, const char* name, const Source& t, size_t at, long long n);
// [heads * size, in] rows into rows of padded heads.
int put_heads(DevBuf& dst, ElemType elem, size_t row0, int stride, const Source& t, int heads, int size, int in, int src_stride, int src_off);
int put_out(DevBuf& dst, ElemType elem, const char* name, const Source& t, int width, int heads, int vdim, int vp);

int block_model_create(const b200attn_model_config* cfg, const b200attn_layer_desc* layers, int num_layers, b200attn_stack st);
int block_model_ready(const BlockModel& m);
int block_model_status(BlockModel& m, int* code);
// One decode step over n rows: d_x of the rows' final residual stream is left in m.x.
int block_decode_rows(BlockModel& m, int n, const int* d_tokens, const int* d_slots, cudaStream_t s);
// A prefill pass over sequences continuing from their caches; rows must fit one pass (block_pass_sequences).
int block_prefill_rows(BlockModel& m, int n_seqs, const int* h_slots, const int* h_counts, const int* d_tokens, cudaStream_t s);
// How many of the given sequences the next pass can take (0: the first one alone does not fit).
int block_pass_sequences(BlockModel& m, int n_seqs, const int* h_slots, const int* h_counts, int* n_out);
// Logits of n selected rows (row_index null: rows 0 .. n-1).
int block_logits(BlockModel& m, int n, const int* d_row_index, float* d_logits, cudaStream_t s);

}  // namespace b200
