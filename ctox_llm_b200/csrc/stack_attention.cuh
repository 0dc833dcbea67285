// Attention of layer stacks over a paged cache. A cached token is one row of slot_cols values, cut into
// kv_heads parts that hold a key and a value each.
#pragma once
#include "dense.cuh"

namespace ctox {

// Short passes (stack_attention.cu): scores and weighted sums over the cached rows, split over the context. A
// query row is (position, head), row = position * heads + head; head h reads part h / (heads / kv_heads). In a
// part, the first key_cols values meet the query, val_cols values from val_off on are summed up.
//
// Latent attention: one part, [latent | rotated key]; queries are carried into the latent space (W_uk^T q), the
// values are the latent itself, and the merge of the splits is the prologue of the value product
// (VecIn::ws_o). Grouped attention: parts [key | value]; the CTA that finishes last merges the splits into out.
struct CacheAttn {
    const float *q;       // [row][q_stride], values 0 .. q_cols of the query
    const float *q_tail;  // [row][tail_stride], values q_cols .. key_cols
    uint32_t q_stride, q_cols, tail_stride;
    const void *cache;
    int bf16;
    const uint32_t *page_table;
    uint32_t page_tokens, heads, kv_heads, slot_cols, head_cols, key_cols, val_off, val_cols;
    uint32_t pos0, m, window;  // window 0: every earlier token
    float scale;
    float *ws_o, *ws_ml;   // [split][row][val_cols], [split][row]{max, sum}
    float *out;            // [row][val_cols]; null: the splits stay as they are (one part only)
    const float *sink;     // [heads], may be null (with out only)
    uint32_t *arrived;     // zero on entry and on return, one per tile of query rows (cache_attn_tiles)
};
// Context splits of a pass, and tiles of query rows.
uint32_t cache_attn_splits(const ctox_ctx *ctx, const CacheAttn &a);
uint32_t cache_attn_tiles(const ctox_ctx *ctx, const CacheAttn &a);
ctox_status launch_cache_attention(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits);

// Long passes (stack_prefill.cu): tiled attention on the tensor cores. q [m][heads * head_w] with head_w =
// dim_pad + rot_pad, out [m][heads * vdim_pad]. row0 is a multiple of 128, at or before the first visible key.
//
// Latent attention (kv_heads 0): keys and values of the visible span are expanded per head first: k [span][heads *
// dim_pad]; vt [heads * vdim_pad][vt_ld], the values transposed; the rotated key part comes from the cache. Span
// row r holds position row0 + r. Grouped attention: keys and values come from the cache (rot_pad 0).
struct PrefillAttn {
    const __nv_bfloat16 *q, *k, *vt, *cache;
    __nv_bfloat16 *out;
    const uint32_t *page_table;
    uint32_t page_tokens, slots, heads, kv_heads, dim_pad, rot_pad, vdim_pad;
    uint32_t slot_cols, rot_off;  // values of a cached token; where its rotated part starts (latent)
    uint32_t pos0, m, window, row0, span, vt_ld;
    float scale;
    const float *sink;  // [heads], may be null
};
bool prefill_attention_fits(const ctox_ctx *ctx, uint32_t dim_pad, uint32_t rot_pad, uint32_t vdim_pad);
ctox_status launch_prefill_attention(ctox_ctx *ctx, const PrefillAttn &a);

// Between the projection of queries, keys and values and grouped attention (qkv.cu): norms over the whole
// query and the whole key projection, rotation of the first rot_dim dimensions of every head (i with i + rot_dim /
// 2), mixing of the values, the queries padded per head, keys and values into the cache.
struct QkvPrep {
    const float *fan;  // [position][fan_stride], [q: heads * dim | k: kv_heads * dim | v: kv_heads * vdim]
    uint32_t fan_stride, heads, kv_heads, dim, vdim, dim_pad, vdim_pad, rot_dim;
    const float *q_norm, *k_norm;  // null: no norm
    float eps;
    const float *freq;  // [rot_dim / 2]
    const float *v_mix;  // the weight (device), null: nothing is mixed
    float *v_first;      // [position][kv_heads * vdim]: read with v_mix, written without (null: neither)
    float *q_f32;        // [position][heads * dim_pad], one of the two
    __nv_bfloat16 *q_b16;
    void *cache;
    int bf16;
    const uint32_t *page_table;
    uint32_t page_tokens, pos0;
};
ctox_status launch_qkv_prep(ctox_ctx *ctx, const QkvPrep &a, uint32_t m);

}  // namespace ctox
