// The stack handle, shared by the hybrid stack (stack.cu) and the layer-described one (block_model.cu).
#pragma once

#include "block_model.cuh"
#include "kernels.cuh"

#include <memory>
#include <vector>

struct b200attn_stack_s {
    std::unique_ptr<b200::BlockModel> blocks;   // set for a stack built from layer descriptions (block_model.cu); the hybrid stack leaves it empty
    b200attn_stack_config cfg{};
    int n_fa = 0, n_la = 0;
    std::vector<int> layer_kind;      // 1 = full attention, 0 = DeltaNet
    std::vector<int> layer_sub;       // index inside the kv pool / state pool
    std::vector<b200attn_fa> fa;
    std::vector<b200attn_la> la;
    std::vector<float*> d_in_norm, d_post_norm;
    std::vector<__half*> d_wgu, d_wdown;   // [2*inter, hidden], [hidden, inter]
    std::vector<char> layer_ready;
    __half* d_embed = nullptr;  // [vocab, hidden]
    float* d_final_norm = nullptr;
    bool embed_ready = false;
    b200attn_kv_pool pool = nullptr;
    b200attn_la_state state = nullptr;
    b200::Scratch op_scratch;
    int max_rows = 0;
    float* d_h = nullptr;              // [max_rows, hidden] residual stream
    __half* d_xb = nullptr;     // [max_rows, hidden]
    __half* d_gu = nullptr;     // [max_rows, 2*inter]
    __half* d_act = nullptr;    // [max_rows, inter]
    float* d_last = nullptr;           // [max_seqs, hidden]
    float* d_logits = nullptr;         // [max_seqs, vocab]
    int* d_tokens = nullptr;           // [max_seqs] decode token buffer (in place)
    int* d_slots = nullptr;            // [max_seqs] identity slots
    __half* d_xh = nullptr;            // [128, hidden] fp16 copy of the residual stream in the fused decode step
    float* d_rowsq = nullptr;          // [128][kRowsqParts] partial sums of squares of the residual rows
    unsigned long long* d_packed = nullptr;   // [128] running argmax words of the LM head
    int* d_error = nullptr;            // device status word of the stack's own tcgen05 GEMMs
    int* d_last_idx = nullptr;         // [max_seqs] row of every sequence's last prompt token inside a prefill pass
    int* d_want = nullptr;             // row indices of the logits a b200attn_stack_extend call asks for
    int want_cap = 0;
    // Continuous batching: row r of a decode step is bound to slot row_slot[r] (its KV pages and DeltaNet state), -1 =
    // inactive.  Empty in the plain mode, where row r is slot r.
    bool batching = false;
    std::vector<int> row_slot;
    std::vector<int> free_slots;
    int n_active = 0;
    cudaGraph_t graph = nullptr;
    cudaGraphExec_t graph_exec = nullptr;
    int graph_nseqs = 0;
    long long graph_nodes = 0;
};
