// Models described layer by layer (ctox_stack_config + ctox_layer_config), run by the decode executor.
//
// The session, the paged cache with its page tables, prefill, decode, selection and evidence calls are
// the executor's (exec.cu); this part holds the weights of such a model and runs a pass over it.
#pragma once
#include <vector>

#include "dense.cuh"
#include "exec.cuh"

namespace ctox {

struct StackLayer {
    ctox_layer_config c{};
    uint32_t owner = 0;  // the layer whose cache this one reads (itself, or its kv_from)
    uint32_t dim_pad = 0, rot_pad = 0, vdim_pad = 0, kv_pad = 0, head_w = 0;  // head sizes rounded up to 16
    // What the mixer projects from the stream, x hidden. Latent attention: [query down | key/value down]; grouped
    // attention: [q | k | v]; matrix memory: [q | k | v | output gate] with padded heads, then from gate_row on the
    // gates' rows [input | forget].
    DenseMat fan;
    uint32_t gate_row = 0;
    DenseMat q_up;       // heads x [dim_pad | rot_pad] rows
    DenseMat k_up;       // heads x dim_pad rows, columns kv_pad (long passes)
    DenseMat k_up_t;     // heads x kv_pad rows, columns dim_pad (short passes)
    DenseMat v_up;       // heads x vdim_pad rows, columns kv_pad
    DenseMat o;          // columns heads x vdim_pad
    DenseMat up, down;   // up of a gated feed-forward: rows 2i and 2i + 1 are gate and up of unit i
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *q_norm = nullptr,
          *kv_norm = nullptr;
    float *k_norm = nullptr, *fan_bias = nullptr, *o_bias = nullptr, *sink = nullptr, *v_mix = nullptr;  // grouped attention
    float *in_bias = nullptr, *forget_bias = nullptr, *head_norm = nullptr;  // matrix memory
    bool mixes_values = false;  // v_mix is applied: not in the first layer that has it
    float *state = nullptr, *top = nullptr;  // matrix memory of the session (parts of StackModel::memory)
    float *freq = nullptr;     // [rot_dim / 2]
    float2 *table = nullptr;   // [position of the pass][rot_dim / 2] (cos, sin), shared by layers that rotate alike
    uint64_t loaded = 0;    // bit per tensor id
    // cache of an owner: ring of pages through the page table. Rows of slot_cols values: latent attention [kv_pad |
    // rot_pad], grouped attention kv_heads x [dim_pad | vdim_pad]
    uint32_t slot_cols = 0;
    void *cache = nullptr;
    uint32_t *page_table = nullptr;
    uint32_t slots = 0;
};

struct StackModel {
    ctox_stack_config c{};
    std::vector<StackLayer> layers;
    DenseMat embed, head;
    float *final_norm = nullptr;
    uint64_t loaded = 0;
    uint32_t pass_cap = 0;  // most positions of one pass
    // pass buffers (rows = positions of the pass)
    float *x[2] = {nullptr, nullptr}, *y = nullptr, *fan = nullptr;
    float *q = nullptr, *q_abs = nullptr, *att = nullptr, *u = nullptr, *ws_o = nullptr, *ws_ml = nullptr;
    __nv_bfloat16 *h_b = nullptr, *cq_b = nullptr, *q_b = nullptr, *k_b = nullptr, *vt_b = nullptr, *att_b = nullptr,
                  *u_b = nullptr, *head_b = nullptr;
    uint32_t span_cap = 0;  // key rows of k_b, columns of vt_b
    std::vector<uint32_t> table_layers;  // one layer of every distinct rotation
    float *head_in = nullptr;
    uint32_t *rows_dev = nullptr;
    uint32_t head_rows = 0;  // rows of e->logits
    float *v_first = nullptr;     // values of the first layer that mixes them, of the pass
    uint32_t *arrived = nullptr;  // counters of the split merge
    float *memory = nullptr;      // states of all matrix memories, cleared with the session
    uint64_t memory_floats = 0;
    __nv_bfloat16 *fan_b = nullptr, *mem_start = nullptr;
    float *gates = nullptr, *mem_scan = nullptr, *mem_delta = nullptr, *mem_raw = nullptr;
    // the stream at the end of the last pass: x[cur], plus y when it is pending (its norm y_norm applied, if any)
    int cur = 0;
    bool pending = false;
    const float *y_norm = nullptr;
    float *streams = nullptr;  // [layer][max_context_tokens][hidden] when kept (evidence)
};

ctox_status stack_create(ctox_ctx *ctx, const ctox_stack_config *c, const ctox_layer_config *layers, ctox_exec **out);
void stack_destroy(ctox_exec *e);
ctox_status stack_load_matrix(ctox_exec *e, uint32_t layer, uint32_t tensor, const ctox_fused_matvec_op *op);
// Where a vector goes: `n` values from `offset` on of an array of `total` (allocated with its first part).
struct VectorSlot {
    float **base = nullptr;
    uint64_t n = 0, total = 0, offset = 0;
    uint64_t *loaded = nullptr;
};
bool stack_vector_slot(ctox_exec *e, uint32_t layer, uint32_t tensor, VectorSlot *slot);
// A new session: recurrent states start at zero.
ctox_status stack_reset(ctox_exec *e);
ctox_status stack_fill_synthetic(ctox_exec *e, uint64_t seed);
ctox_status stack_warmup(ctox_exec *e);
ctox_status stack_prefill_synthetic(ctox_exec *e, uint64_t n, uint64_t seed);
// The m tokens in e->tokens_dev at positions pos0 ...: appends to the cache, leaves the final hidden
// state of the last one in e->hist_hidden.
ctox_status stack_pass(ctox_exec *e, uint32_t m, uint64_t pos0);
// Logits of the last position of the pass into row 0 of e->logits.
ctox_status stack_head_last(ctox_exec *e);
// Logits of n <= head_rows positions of the pass (host list of places) into e->logits.
ctox_status stack_head_rows(ctox_exec *e, const uint32_t *rows, uint32_t n);
ctox_status stack_keep_streams(ctox_exec *e);

}  // namespace ctox
