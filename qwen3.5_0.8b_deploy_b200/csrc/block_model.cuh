// Models given by a list of layer descriptions: the operators, the working buffers and the layer loop behind
// b200attn_stack_create_layers.  A layer is x += norm1(mixer(x)), then x += norm2(ff(x)): the sublayers read the residual
// stream itself and RMS norms sit on their outputs.  Sizes and constants come from the description; element types are
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
// act = gelu_tanh(gate) * up over rows of [gate | up].
int launch_gelu_mul(ElemType t, const void* gu, int rows, int ff, void* act, cudaStream_t s);
// lens[layer][slot] += count for every layer of a pool.
int launch_lens_advance(int* lens, int n_layers, int max_seqs, const int* d_slots, const LaSeqMeta* d_seqs, int n, cudaStream_t s);
int launch_argmax_rows(const float* logits, int rows, int vocab, int* out, cudaStream_t s);   // stack.cu

// ---- mlstm.cu, mlstm_chunk.cu: matrix memory with exponential gating -----------------------------------------------------
constexpr int kMlstmTile = 128;        // value columns of one state tile
struct MlstmShape {
    int heads = 0, dim = 0, vdim = 0;
    float gate_cap = 0.f, eps = 0.f;
    int dp = 0, vp = 0;                // head sizes in the projections, padded with zero weights
    int vt = 0, n_vt = 0;              // state tile width and tiles per head
    constexpr int off_q() const { return 0; }
    constexpr int off_k() const { return heads * dp; }
    constexpr int off_v() const { return 2 * heads * dp; }
    constexpr int off_g() const { return 2 * heads * dp + heads * vp; }
    constexpr int off_i() const { return 2 * heads * (dp + vp); }
    constexpr int off_f() const { return off_i() + heads; }
    constexpr int cols() const { return off_i(); }                             // q | k | v | g
    constexpr int pitch() const { return round_up(off_i() + 2 * heads, 4); }   // fp32 rows with the gate columns behind
    constexpr size_t tile_floats() const { return (size_t)dim * vt + round_up(dim, 4) + 4; }   // S [dim][vt], n [dim], m
    constexpr size_t state_floats() const { return tile_floats() * n_vt * heads; }
};
struct MlstmStepArgs {                 // the token-serial kernel: decode (one token a row) and plain prefill
    MlstmShape sh;
    const float* proj;                 // [rows][pitch]
    const float* bias;                 // [2 * heads]: i then f
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

struct MlstmOp {
    MlstmShape sh;
    ElemType elem = ELEM_BF16;
    int width = 0, state_layer = 0;
    bool chunk = false;                // prefill through the chunked tensor-core kernel
    DevBuf w_in, w_out, bias, norm_w;
};

// ---- latent.cu, latent_decode.cu, latent_prefill.cu: attention over cached latents -----------------------------------------
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
    int width = 0, pool_layer = 0;     // the pool layer it reads (its own or its source's)
    bool tc_prefill = false, tc_decode = false;
    int rot_table = 0;                 // index of its rotation's table
    DevBuf w_in, w_uk, w_uv, w_out, c_norm;
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
    int ff = 0;                        // 0: no feed-forward
    DevBuf norm1, norm2, w_gu, w_down;
    std::vector<std::string> missing;  // tensors not given yet
};

struct BlockModel {
    b200attn_model_config cfg{};
    ElemType elem = ELEM_BF16;
    std::vector<BlockLayer> layers;
    std::vector<RotTable> rot;
    std::vector<std::string> missing;
    DevBuf embed, final_norm;
    int stop_after = -1;               // >= 0: passes end behind that many layers
    int max_rows = 0, abs_rows = 0, ctx_rows = 0, max_spans = 0;
    b200attn_kv_pool pool = nullptr;   // owned by the stack
    b200attn_la_state state = nullptr;
    DevBuf x, xt, proj, gates, core, mixed, y, gu, act, q, qa, olat, c_stage, r_stage, k_up, v_up, part, counters, meta, error;
    int* row_slot() const { return meta.i(); }
    int* row_pos() const { return meta.i() + max_rows; }
    LaSeqMeta* seqs() const { return reinterpret_cast<LaSeqMeta*>(meta.i() + 2 * (size_t)max_rows); }
    LatentSpan* spans() const { return reinterpret_cast<LatentSpan*>(meta.i() + 2 * (size_t)max_rows + 3 * (size_t)max_spans); }
    LatentTile* tiles() const { return reinterpret_cast<LatentTile*>(meta.i() + 2 * (size_t)max_rows + 7 * (size_t)max_spans); }
    // what the staging buffers hold (layers that share latents share the staged rows of a pass)
    int staged_layer = -1;
    std::vector<LatentSpan> staged;
};

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
