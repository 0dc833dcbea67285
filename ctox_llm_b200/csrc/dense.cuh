// Products with dense bf16 weights, and the norms around them (dense.cu).
//
// Two forms. A pass of up to kDensePass positions is a matrix-vector product: weights are streamed
// once, activations stay fp32, and the kernel's prologue forms its own input (residual add, norm,
// merge of attention splits), its epilogue the activation or rotation. A longer pass is a tiled
// tensor-core product over bf16 activations (gemm.cu).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cstdint>

#include "common.cuh"

namespace ctox {

constexpr uint32_t kDensePass = 8;       // positions per pass of the matrix-vector form
constexpr uint32_t kAttnSplitsDense = 64;  // most context splits a merge prologue takes

// Row-major [rows][ld] bf16, ld = columns rounded up to 8 (16-byte rows), padding zero.
struct DenseMat {
    __nv_bfloat16 *w = nullptr;
    uint32_t rows = 0, cols = 0, ld = 0;
};

enum NormKind : int { NORM_NONE = 0, NORM_LAYER = 1, NORM_RMS = 2 };

// Input vector of a matrix-vector product, [position][x_stride] (a grouped product adds
// group * x_group). With a norm, `cols` values are normalised and weighted by w. With y set the input is
// first x + y (layer norm with wb set: x + layer_norm(y; wb)), which the first CTA stores to x_out. With
// ws_o set the input is the merge of `splits` partial attention results of row position * groups +
// group instead.
struct VecIn {
    const float *x;
    uint32_t x_stride, x_group, cols;
    int norm;
    const float *w;
    float eps;
    const float *y;
    uint32_t y_stride;
    const float *wb;
    float *x_out;
    const float *ws_o, *ws_ml;
    uint32_t splits, ws_rows, groups;
};

enum OutKind : int { OUT_PLAIN = 0, OUT_RELU2 = 1, OUT_SOFTCAP = 2, OUT_ROPE = 3, OUT_CLAMPED_GLU = 4 };

// Output vector [position][y_stride], the row's bias (may be null) added first. OUT_ROPE: rows come in heads
// of head_width, of which the rows rope0 .. rope0 + rope_dims are turned in interleaved pairs by (pos0 +
// position) * freq[pair]. OUT_CLAMPED_GLU: rows 2i and 2i + 1 are gate and up of output i (cap: the limit).
struct VecOut {
    float *y;
    uint32_t y_stride;
    int kind;
    const float *bias;
    float cap, slope;
    uint32_t head_width, rope0, rope_dims, pos0;
    const float *freq;
};

// Latent cache append of one position: RMS norm of the latent part of a down projection, rotation of
// its last rot_dim values, both into the cache row of the position (row = [kv_pad | rot_pad]).
struct LatentAppend {
    const float *fan;  // [position][fan_stride]; the latent starts at fan_off
    uint32_t fan_stride, fan_off, kv_rank, rot_dim, kv_pad, rot_pad;
    const float *norm_w;
    float eps;
    void *cache;
    int bf16;
    const uint32_t *page_table;
    uint32_t page_tokens, pos0;
    const float *freq;
};

// y = W x for m <= kDensePass positions; groups > 1: rows and inputs come in `groups` equal parts. With
// `append`, extra CTAs of the same launch append the m positions to the latent cache.
ctox_status launch_dense_matvec(ctox_ctx *ctx, const DenseMat &w, uint32_t groups, uint32_t m, const VecIn &in,
                                const VecOut &out, const LatentAppend *append);

// x <- x + layer_norm(y; wb), or x + y without wb (y may be null; x_out may equal x), then the norm (w) of
// the result as fp32 and / or bf16. One CTA per row; `rows` (device, may be null) picks input rows.
struct StreamNorm {
    int norm;  // NORM_LAYER or NORM_RMS
    const float *x;
    const float *y, *wb, *w;
    float eps;
    uint32_t width;
    float *x_out;             // may be null
    float *f32_out;           // [row][width], may be null
    __nv_bfloat16 *bf16_out;  // [row][bf16_ld], may be null
    uint32_t bf16_ld;
    const uint32_t *rows;
};
ctox_status launch_stream_norm(ctox_ctx *ctx, const StreamNorm &a, uint32_t m);

// RMS norm of the first q_rank values of every fan row as bf16, and the latent append (append may be null).
ctox_status launch_latent_split(ctox_ctx *ctx, const float *fan, uint32_t fan_stride, uint32_t q_rank,
                                const float *q_norm, float eps, __nv_bfloat16 *cq, uint32_t cq_ld,
                                const LatentAppend *append, uint32_t m);

ctox_status launch_embed_dense(ctox_ctx *ctx, const __nv_bfloat16 *embed, uint32_t ld, const uint32_t *tokens,
                               uint32_t width, uint32_t m, float scale, float *x);

// Index map of one axis when a matrix is laid out anew: groups of `group` indices become groups of
// group_pad, the indices of a group from `split` on start at split_pad.
struct PadAxis {
    uint32_t group, split, split_pad, group_pad;
};
// dst[map(row)][map(col)] = src[row][col] (dst zeroed by the caller); transpose_group > 0: the padded
// rows come in groups of transpose_group that are transposed, dst[group][col][row in group].
ctox_status launch_relayout(ctox_ctx *ctx, const __nv_bfloat16 *src, uint32_t rows, uint32_t cols, PadAxis ra,
                            PadAxis ca, __nv_bfloat16 *dst, uint32_t dst_ld, uint32_t transpose_group,
                            uint32_t transpose_cols);

ctox_status launch_fill_normal_bf16(ctox_ctx *ctx, __nv_bfloat16 *out, uint64_t n, float std, uint64_t seed);
ctox_status launch_fill_normal_f32(ctox_ctx *ctx, float *out, uint64_t n, float std, uint64_t seed);

}  // namespace ctox

#ifdef __CUDACC__
namespace ctox {
__device__ __forceinline__ void rope_pair(float &u, float &v, float angle) {
    float s, c;
    sincosf(angle, &s, &c);
    const float a = u * c - v * s, b = v * c + u * s;
    u = a;
    v = b;
}
// Gated feed-forward with clamped inputs: g = min(gate, limit), u = clamp(up, +-limit); g sigmoid(slope g) (u + 1).
__device__ __forceinline__ float clamped_glu(float gate, float up, float limit, float slope) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g / (1.0f + expf(-slope * g)) * (u + 1.0f);
}
// Cache slot of position t.
__device__ __forceinline__ size_t paged_slot(const uint32_t *page_table, uint32_t page_tokens, uint32_t t) {
    return (size_t)page_table[t / page_tokens] * page_tokens + t % page_tokens;
}
}  // namespace ctox
#endif
