// Matrix memory (mLSTM): per head a state S [vdim][dim] with a normaliser n [dim] and a running maximum m of
// the log gates. With log input gate i and log forget gate f of a token:
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') v k^T;  n' likewise with 1 for v;
//   o = S' q / (max(|n' q|, e^-m') + 1e-6)
// then an RMS norm per head, a weight and an output gate.
#pragma once
#include "dense.cuh"

namespace ctox {

constexpr uint32_t kMemRows = 16;    // rows of the state behind vdim_pad; the first is the normaliser
constexpr uint32_t kMemChunk = 128;  // tokens that a long pass takes at once

struct MatrixMemory {
    uint32_t heads, dim, vdim, dim_pad, vdim_pad;
    float gate_cap, eps;
    const float *i_bias, *f_bias;  // [heads]
    const float *norm_w;           // [heads * vdim]
    float *state;                  // [head][vdim_pad + kMemRows][dim_pad]
    float *top;                    // [head] running maximum
};
inline uint64_t memory_rows(const MatrixMemory &a) { return a.vdim_pad + kMemRows; }

// Short passes. fan [position][fan_stride]: [q: heads * dim_pad | k: heads * dim_pad | v: heads * vdim_pad | gate: heads *
// vdim_pad], the gates' preactivations [i: heads | f: heads] at gate_off. out [position][heads * vdim_pad].
ctox_status launch_matrix_memory(ctox_ctx *ctx, const MatrixMemory &a, const float *fan, uint32_t fan_stride,
                                 uint32_t gate_off, uint32_t m, float *out);

// Long passes, by chunks of kMemChunk tokens: the projections as bf16 rows of fan_ld, the gates' preactivations as
// fp32 [position][2 * heads]. Work buffers are sized by memory_long_sizes for the longest pass.
struct MemoryLong {
    const __nv_bfloat16 *fan;
    uint32_t fan_ld;
    const float *gates;
    __nv_bfloat16 *out;       // [position][heads * vdim_pad]
    float *scan;              // [head][3][position], then [head][chunk] x 2
    float *delta;             // [chunk][head][vdim_pad + kMemRows][dim_pad] what a chunk adds
    __nv_bfloat16 *start;     // [hi, lo][chunk][head][vdim_pad + kMemRows][dim_pad] the state before a chunk
    float *raw;               // [position][heads * vdim_pad] outputs before their norm
};
struct MemoryLongSizes {
    uint64_t scan, delta, start, raw;  // elements
};
MemoryLongSizes memory_long_sizes(const MatrixMemory &a, uint32_t pass_tokens);
bool memory_long_fits(const ctox_ctx *ctx, const MatrixMemory &a);
ctox_status launch_matrix_memory_long(ctox_ctx *ctx, const MatrixMemory &a, const MemoryLong &w, uint32_t m);

}  // namespace ctox

#ifdef __CUDACC__
namespace ctox {
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
}  // namespace ctox
#endif
