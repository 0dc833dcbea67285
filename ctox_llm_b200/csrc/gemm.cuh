// Tensor-core products of long passes (gemm.cu): D[m][n] = sum_k A[m][k] B[n][k], bf16 operands, fp32
// accumulation in tensor memory.
#pragma once
#include "dense.cuh"

namespace ctox {

// Rows of `ld` bf16 values, `cols` of them live. With a page table, rows live in a paged cache: row
// r of the operand is the cache row of position row0 + r (row0 a multiple of the 128-row tile, pages a
// multiple of 128 tokens).
struct GemmOperand {
    const __nv_bfloat16 *p;
    uint32_t rows, cols, ld;
    const uint32_t *page_table;
    uint32_t page_tokens, row0, store_rows;  // store_rows: rows of the whole cache
};

struct GemmOut {
    void *d;
    uint32_t ld;
    int bf16;
    int kind;  // OutKind
    const float *bias;  // per column, may be null
    float cap, slope;   // OUT_CLAMPED_GLU: columns 2i and 2i + 1 are gate and up of output column i
    // columns from `split` (a multiple of 32; 0: none) on go to d2 as fp32, counted from there
    uint32_t split;
    float *d2;
    uint32_t ld2;
    // OUT_ROPE: columns come in heads of head_width; columns rope0 .. rope0 + rope_dims of a head are turned in
    // pairs by table[row][pair] = (cos, sin)
    uint32_t head_width, rope0, rope_dims;
    const float2 *table;
};

ctox_status launch_gemm(ctox_ctx *ctx, const GemmOperand &a, const GemmOperand &b, const GemmOut &out);

// table[row][pair] = (cos, sin) of (pos0 + row) * freq[pair].
ctox_status launch_rope_table(ctox_ctx *ctx, const float *freq, uint32_t pairs, uint32_t pos0, uint32_t rows,
                              float2 *table);

}  // namespace ctox
