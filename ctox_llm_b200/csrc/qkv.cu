// Between the projection of queries, keys and values and grouped attention (QkvPrep).
#include "stack_attention.cuh"

namespace ctox {

constexpr int kQkvThreads = 512;

// One CTA per (position, share of the outputs). Every CTA of a position forms the norms over the whole query
// and key projection itself; each writes its share of the padded queries, keys and values.
__global__ void __launch_bounds__(kQkvThreads) k_qkv_prep(QkvPrep a) {
    pdl_launch();
    extern __shared__ __align__(16) float2 cs_s[];  // [rot_dim / 2] (cos, sin)
    __shared__ float red[2][kQkvThreads / 32];
    const uint32_t m = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pos = a.pos0 + m;
    const uint32_t half = a.rot_dim / 2, nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    for (uint32_t i = tid; i < half; i += kQkvThreads) {
        float s, c;
        sincosf((float)pos * a.freq[i], &s, &c);
        cs_s[i] = make_float2(c, s);
    }
    pdl_wait();
    const float *q = a.fan + (size_t)m * a.fan_stride, *k = q + nq, *v = k + nk;
    float sq = 0.f, sk = 0.f;
    if (a.q_norm)
        for (uint32_t c = tid; c < nq; c += kQkvThreads) sq = fmaf(q[c], q[c], sq);
    if (a.k_norm)
        for (uint32_t c = tid; c < nk; c += kQkvThreads) sk = fmaf(k[c], k[c], sk);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if (lane == 0) {
        red[0][warp] = sq;
        red[1][warp] = sk;
    }
    __syncthreads();
    float q_inv = 0.f, k_inv = 0.f;
#pragma unroll
    for (int w = 0; w < kQkvThreads / 32; ++w) {
        q_inv += red[0][w];
        k_inv += red[1][w];
    }
    q_inv = a.q_norm ? 1.0f / sqrtf(q_inv / (float)nq + a.eps) : 1.f;
    k_inv = a.k_norm ? 1.0f / sqrtf(k_inv / (float)nk + a.eps) : 1.f;
    // value d of a head of x after norm and rotation
    auto turned = [&](const float *x, const float *w, float inv, uint32_t head, uint32_t d) {
        const uint32_t at = head * a.dim + d;
        const float u = x[at] * inv * (w ? w[at] : 1.f);
        if (d >= a.rot_dim) return u;
        const bool low = d < half;
        const uint32_t pair = low ? at + half : at - half;
        const float p = x[pair] * inv * (w ? w[pair] : 1.f);
        const float2 cs = cs_s[low ? d : d - half];
        return low ? u * cs.x - p * cs.y : u * cs.x + p * cs.y;
    };
    const uint32_t step = gridDim.x * kQkvThreads, first = blockIdx.x * kQkvThreads + tid;
    const uint32_t q_cols = a.heads * a.dim_pad;
    for (uint32_t c = first; c < q_cols; c += step) {
        const uint32_t d = c % a.dim_pad;
        const float r = d < a.dim ? turned(q, a.q_norm, q_inv, c / a.dim_pad, d) : 0.f;
        if (a.q_b16)
            a.q_b16[(size_t)m * q_cols + c] = __float2bfloat16_rn(r);
        else
            a.q_f32[(size_t)m * q_cols + c] = r;
    }
    const uint32_t part = a.dim_pad + a.vdim_pad, slot_cols = a.kv_heads * part;
    const size_t base = paged_slot(a.page_table, a.page_tokens, pos) * slot_cols;
    const float mix = a.v_mix ? *a.v_mix : 0.f;
    for (uint32_t c = first; c < slot_cols; c += step) {
        const uint32_t head = c / part, d = c % part;
        float r = 0.f;
        if (d < a.dim) {
            r = turned(k, a.k_norm, k_inv, head, d);
        } else if (d >= a.dim_pad && d - a.dim_pad < a.vdim) {
            const uint32_t at = head * a.vdim + d - a.dim_pad;
            r = v[at];
            if (a.v_mix)
                r = (1.f - mix) * r + mix * a.v_first[(size_t)m * nv + at];
            else if (a.v_first)
                a.v_first[(size_t)m * nv + at] = r;
        }
        if (a.bf16)
            ((__nv_bfloat16 *)a.cache)[base + c] = __float2bfloat16_rn(r);
        else
            ((float *)a.cache)[base + c] = r;
    }
}

ctox_status launch_qkv_prep(ctox_ctx *ctx, const QkvPrep &a, uint32_t m) {
    const uint32_t outs = a.heads * a.dim_pad + a.kv_heads * (a.dim_pad + a.vdim_pad);
    uint32_t parts = m <= kDensePass ? (outs + kQkvThreads - 1) / kQkvThreads : 1;
    if (parts > 16) parts = 16;
    const size_t smem = (size_t)(a.rot_dim / 2) * sizeof(float2);
    if (smem > 40 * 1024) return fail(ctx, CTOX_SHAPE, "a rotation over %u dimensions", a.rot_dim);
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_qkv_prep, dim3(parts, m), dim3(kQkvThreads), smem, ctx->stream, a));
    timing_end(ctx, KC_QKV, (double)m * ((a.heads + a.kv_heads) * a.dim * 4.0 + a.kv_heads * a.vdim * 4.0 +
                                         a.heads * a.dim_pad * (a.q_b16 ? 2.0 : 4.0) +
                                         a.kv_heads * (a.dim_pad + a.vdim_pad) * (a.bf16 ? 2.0 : 4.0)), 0);
    return CTOX_OK;
}

}  // namespace ctox
