// The decode executor's state, shared by the entry points (exec.cu) and the layer-stack models (stack.cu).
#pragma once
#include <cstdint>
#include <vector>

#include "common.cuh"
#include "layers.cuh"
#include "matvec.cuh"

namespace ctox {
constexpr uint32_t kMaxPass = 8;  // positions per pass (verify rows / prefill chunk)

struct LayerW {
    bool full = false;
    float *in_ln = nullptr, *post_ln = nullptr;
    ctox_matvec *in_fan = nullptr, *out = nullptr, *gate_up = nullptr, *down = nullptr;
    float *conv_w = nullptr, *a_log = nullptr, *dt_bias = nullptr, *lin_norm = nullptr;
    float *q_norm = nullptr, *k_norm = nullptr;
};

struct LayerS {
    float *conv_state = nullptr;                  // [channels][kernel], committed
    float *delta[2] = {nullptr, nullptr};         // [heads][128][128]; delta[cur] is committed
    int cur = 0;
    float *conv_in = nullptr;                     // [kMaxPass][channels] inputs of the last pass
    float *q = nullptr, *k = nullptr, *v = nullptr, *g = nullptr, *beta = nullptr;  // last pass
    void *k_cache = nullptr, *v_cache = nullptr;  // [slots][kv_heads][head_dim]
};

struct StackModel;  // a layer stack described layer by layer (stack.cuh)
}  // namespace ctox

using ctox::kMaxPass;
using ctox::LayerS;
using ctox::LayerW;
using ctox::CommitLayer;
using ctox::kAttnMaxSplits;

struct ctox_exec {
    ctox_ctx *ctx = nullptr;
    ctox_model_config cfg{};  // this rank's shard: heads and FFN width divided by the group size
    uint32_t tp_world = 1, tp_rank = 0;
    uint32_t vocab_l = 0, vocab_off = 0;      // rows of lm_head on this rank
    uint32_t kv_heads_global = 0;             // KV heads of the unsharded model
    uint32_t draft_lo = 0, draft_n = 0;       // this rank's range of the draft id table
    std::vector<uint32_t> draft_ids_host;
    float *tp_buf = nullptr;                  // [kMaxPass][hidden] vector being summed over the group
    uint32_t n_layers = 0;  // target layers; index n_layers is the MTP layer when present
    uint32_t key_width = 0, value_width = 0, channels = 0, q_width = 0, kv_width = 0;
    std::vector<LayerW> w;
    std::vector<LayerS> s;
    ctox_matvec *embed = nullptr, *lm_head = nullptr, *mtp_fc = nullptr, *draft_head = nullptr;
    float *final_norm = nullptr, *mtp_norm_e = nullptr, *mtp_norm_h = nullptr, *mtp_norm = nullptr;
    uint32_t *draft_ids = nullptr;  // device, [draft_vocab]
    CommitLayer *commit_table = nullptr;  // device, one entry per linear-attention layer
    uint32_t n_linear = 0;
    bool lm_head_is_embed = false;
    // session
    uint64_t position = 0;     // tokens consumed by the target so far
    bool have_hidden = false;  // hist_hidden[0 .. hist_n) holds the final hidden of the last hist_n positions
    uint32_t hist_n = 0;       // committed positions of the last block (1..kMaxPass)
    uint32_t hist_tokens[kMaxPass] = {0};  // tokens at positions position-hist_n+1 .. position-1 (drafts accepted)
    uint64_t step_counter = 0;
    bool warmed = false, keep_logits = false;
    // Speculative transaction (engine.rs:322-362): an MTP decode resolves and commits its accepted
    // prefix on the device and leaves the count here until commit_speculative confirms it.
    int32_t pending = -1;
    double last_enqueue_us = 0.0;  // host time the last decode spent enqueuing before it waited for the device
    // Optional device times of the phases of a decode call (events at the phase boundaries):
    // drafting, target pass, head + acceptance, commit.
    bool phase_timing = false;
    cudaEvent_t phase_ev[6] = {};
    float phase_ms[4] = {0.f, 0.f, 0.f, 0.f};
    bool commit_timed = false;
    // A device error or a failed call after work was enqueued leaves the session state undefined:
    // every call fails until reset_session (engine.rs:594-611 invalidates the session the same way).
    bool poisoned = false;
    // evidence of the last decode call (with keep_logits): the MTP layer's final hidden of every
    // (token, hidden) pair it ran, in order, and the logits of every draft
    float *mtp_trace = nullptr, *draft_trace = nullptr;
    uint32_t mtp_trace_n = 0, draft_trace_n = 0, draft_rows = 0;
    // buffers ([kMaxPass] rows each)
    float *h = nullptr, *final_hidden = nullptr, *hist_hidden = nullptr, *embed_rows = nullptr;
    float *mtp_h = nullptr, *mtp_hidden = nullptr;
    float *aq = nullptr, *agate = nullptr, *attn_ws = nullptr;
    float *lz = nullptr, *lcore = nullptr, *norm_scratch = nullptr;
    float *draft_logits = nullptr, *logits = nullptr;
    uint32_t *tokens_dev = nullptr;  // [kMaxPass + 1]: verify inputs = [token, drafts...]
    uint32_t *mtp_tokens_dev = nullptr;
    uint32_t *page_table = nullptr, *mtp_page_table = nullptr;
    uint32_t attn_splits_max = kAttnMaxSplits;
    uint64_t model_bytes = 0, session_bytes = 0;
    ctox::StackModel *stack = nullptr;  // set: a layer-stack model; the fields of the hybrid model above stay empty
    std::vector<std::pair<void *, size_t>> owned;  // tracked raw allocations (vectors, buffers, states)
};

namespace ctox {

// Tracked allocation owned by the executor (freed by ctox_exec_destroy), zeroed unless told otherwise.
inline ctox_status xalloc(ctox_exec *e, void **p, size_t bytes, bool session, bool zero = true) {
    ctox_status rc = dev_alloc(e->ctx, p, bytes);
    if (rc) return rc;
    e->owned.emplace_back(*p, bytes);
    (session ? e->session_bytes : e->model_bytes) += bytes;
    if (zero) CTOX_CUDA(e->ctx, cudaMemsetAsync(*p, 0, bytes, e->ctx->stream));
    return CTOX_OK;
}

}  // namespace ctox
