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

// Long passes (latent_prefill.cu): keys and values of the visible span are expanded per head first, then
// tiled attention on the tensor cores. q [m][heads * head_w] with head_w = dim_pad + rot_pad; k [span][heads *
// dim_pad]; vt [heads * vdim_pad][vt_ld], the values transposed; the rotated key part comes from the cache.
// Span row r holds position row0 + r (row0 a multiple of 128).
struct LatentPrefill {
    const __nv_bfloat16 *q, *k, *vt, *cache;
    __nv_bfloat16 *out;  // [m][heads * vdim_pad]
    const uint32_t *page_table;
    uint32_t page_tokens, slots, heads, dim_pad, rot_pad, vdim_pad, kv_pad;
    uint32_t pos0, m, window, row0, span, vt_ld;
    float scale;
};
bool latent_prefill_fits(const ctox_ctx *ctx, uint32_t dim_pad, uint32_t rot_pad, uint32_t vdim_pad);
ctox_status launch_latent_prefill(ctox_ctx *ctx, const LatentPrefill &a);

}  // namespace ctox
