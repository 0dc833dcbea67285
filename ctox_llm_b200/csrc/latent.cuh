// Attention over a compressed cache: every cached token is one latent row [kv_pad | rot_pad] that all
// heads share (latent.cu).
#pragma once
#include "dense.cuh"

namespace ctox {

// Short passes: queries are carried into the latent space (q_abs = W_uk^T q), scores and weighted sums run
// on the cache rows themselves, split over the context; the merge of the splits is the prologue of the
// value product (VecIn::ws_o). Row = position * heads + head.
struct LatentAttn {
    const float *q_abs;  // [row][kv_pad]
    const float *q_rot;  // [row][q_stride], the rotated part of the query
    uint32_t q_stride;
    const void *cache;
    int bf16;
    const uint32_t *page_table;
    uint32_t page_tokens, heads, kv_pad, rot_pad;
    uint32_t pos0, m, window;  // window 0: every earlier token
    float scale;
    float *ws_o, *ws_ml;  // [split][row][kv_pad], [split][row]{max, sum}
};
// Context splits of a pass, and the floats its workspace needs.
uint32_t latent_attn_splits(const ctox_ctx *ctx, const LatentAttn &a);
ctox_status launch_latent_attention(ctox_ctx *ctx, const LatentAttn &a, uint32_t splits);

}  // namespace ctox
