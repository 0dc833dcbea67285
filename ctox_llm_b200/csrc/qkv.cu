// Between the projection of queries, keys and values and grouped attention (QkvPrep).
#include "stack_attention.cuh"

namespace ctox {

constexpr int kQkvThreads = 512;

// One CTA per (position, share of the outputs). Every CTA of a position brings the projections into shared memory and
// forms the norms over the whole query and key projection itself; a thread then makes groups of four outputs.
__global__ void __launch_bounds__(kQkvThreads) k_qkv_prep(QkvPrep a) {
    pdl_launch();
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[2][kQkvThreads / 32];
    const uint32_t m = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pos = a.pos0 + m;
    const uint32_t half = a.rot_dim / 2, nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, all = nq + nk + nv;
    float *x = sm;                                                     // [q | k | v]
    float2 *cs_s = reinterpret_cast<float2 *>(sm + (all + 3) / 4 * 4);  // [half] (cos, sin)
    for (uint32_t i = tid; i < half; i += kQkvThreads) {
        float s, c;
        sincosf((float)pos * a.freq[i], &s, &c);
        cs_s[i] = make_float2(c, s);
    }
    // the norms' weights are constants: bring their lines in before the wait
    for (uint32_t c = tid * 32; c < nq + nk; c += kQkvThreads * 32) {
        const float *w = c < nq ? a.q_norm : a.k_norm;
        if (w) asm volatile("prefetch.global.L1 [%0];" ::"l"(w + (c < nq ? c : c - nq)));
    }
    pdl_wait();
    const float *row = a.fan + (size_t)m * a.fan_stride;
    float sq = 0.f, sk = 0.f;
    auto add = [&](uint32_t c, float v) {
        if (c < nq)
            sq = fmaf(v, v, sq);
        else if (c < nq + nk)
            sk = fmaf(v, v, sk);
    };
    if (a.fan_stride % 4 == 0 && ((uintptr_t)a.fan & 15) == 0) {
#pragma unroll 4
        for (uint32_t c = tid * 4; c < all; c += kQkvThreads * 4) {  // a row is padded to whole vectors by its stride
            const float4 v = *reinterpret_cast<const float4 *>(row + c);
            *reinterpret_cast<float4 *>(x + c) = v;
            add(c, v.x);
            add(c + 1, v.y);
            add(c + 2, v.z);
            add(c + 3, v.w);
        }
    } else {
        for (uint32_t c = tid; c < all; c += kQkvThreads) {
            x[c] = row[c];
            add(c, row[c]);
        }
    }
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
    if (a.q_norm) {
        q_inv = 1.0f / sqrtf(q_inv / (float)nq + a.eps);
        for (uint32_t c = tid; c < nq; c += kQkvThreads) x[c] *= q_inv * a.q_norm[c];
    }
    if (a.k_norm) {
        k_inv = 1.0f / sqrtf(k_inv / (float)nk + a.eps);
        for (uint32_t c = tid; c < nk; c += kQkvThreads) x[nq + c] *= k_inv * a.k_norm[c];
    }
    __syncthreads();
    // values d .. d + 4 of the head at h, rotated
    const bool vec = a.dim % 4 == 0 && half % 4 == 0;  // then a group lies in one half, and so does its pair
    auto turned = [&](const float *h, uint32_t d, float *r) {
        if (vec && d < a.dim) {
            *reinterpret_cast<float4 *>(r) = *reinterpret_cast<const float4 *>(h + d);
            if (d < a.rot_dim) {
                const bool low = d < half;
                const float4 p = *reinterpret_cast<const float4 *>(low ? h + d + half : h + d - half);
                const float pv[4] = {p.x, p.y, p.z, p.w};
                const float2 *cs = cs_s + (low ? d : d - half);
#pragma unroll
                for (int j = 0; j < 4; ++j) r[j] = low ? r[j] * cs[j].x - pv[j] * cs[j].y : r[j] * cs[j].x + pv[j] * cs[j].y;
            }
            return;
        }
#pragma unroll
        for (uint32_t j = 0; j < 4; ++j) {
            const uint32_t i = d + j;
            r[j] = i < a.dim ? h[i] : 0.f;
            if (i < half) {
                const float2 cs = cs_s[i];
                r[j] = r[j] * cs.x - h[i + half] * cs.y;
            } else if (i < a.rot_dim) {
                const float2 cs = cs_s[i - half];
                r[j] = r[j] * cs.x + h[i - half] * cs.y;
            }
        }
    };
    auto store = [&](__nv_bfloat16 *b16, float *f32, size_t at, const float *r) {
        if (b16) {
            const __nv_bfloat162 h[2] = {__floats2bfloat162_rn(r[0], r[1]), __floats2bfloat162_rn(r[2], r[3])};
            *reinterpret_cast<uint2 *>(b16 + at) = *reinterpret_cast<const uint2 *>(h);
        } else {
            *reinterpret_cast<float4 *>(f32 + at) = make_float4(r[0], r[1], r[2], r[3]);
        }
    };
    const uint32_t q_groups = a.heads * a.dim_pad / 4, part = a.dim_pad + a.vdim_pad, slot_cols = a.kv_heads * part;
    const size_t base = paged_slot(a.page_table, a.page_tokens, pos) * slot_cols;
    const float mix = a.v_mix ? *a.v_mix : 0.f;
    for (uint32_t g = blockIdx.x * kQkvThreads + tid; g < q_groups + slot_cols / 4; g += gridDim.x * kQkvThreads) {
        __align__(16) float r[4];
        if (g < q_groups) {
            const uint32_t c = g * 4;
            turned(x + c / a.dim_pad * a.dim, c % a.dim_pad, r);
            store(a.q_b16, a.q_f32, (size_t)m * a.heads * a.dim_pad + c, r);
            continue;
        }
        const uint32_t c = (g - q_groups) * 4, head = c / part, d = c % part;
        if (d < a.dim_pad) {
            turned(x + nq + head * a.dim, d, r);
        } else {
#pragma unroll
            for (uint32_t j = 0; j < 4; ++j) {
                const uint32_t i = d - a.dim_pad + j, at = head * a.vdim + i;
                r[j] = i < a.vdim ? x[nq + nk + at] : 0.f;
                if (i < a.vdim && a.v_mix)
                    r[j] = (1.f - mix) * r[j] + mix * a.v_first[(size_t)m * nv + at];
                else if (i < a.vdim && a.v_first)
                    a.v_first[(size_t)m * nv + at] = r[j];
            }
        }
        store(a.bf16 ? (__nv_bfloat16 *)a.cache : nullptr, (float *)a.cache, base + c, r);
    }
}

ctox_status launch_qkv_prep(ctox_ctx *ctx, const QkvPrep &a, uint32_t m) {
    const uint32_t outs = (a.heads * a.dim_pad + a.kv_heads * (a.dim_pad + a.vdim_pad)) / 4;
    uint32_t parts = m <= kDensePass ? (outs + kQkvThreads - 1) / kQkvThreads : 1;
    if (parts > 16) parts = 16;
    const size_t all = (size_t)(a.heads + a.kv_heads) * a.dim + (size_t)a.kv_heads * a.vdim;
    const size_t smem = (all + 3) / 4 * 16 + (size_t)(a.rot_dim / 2) * sizeof(float2);
    if (smem + 1024 > (size_t)ctx->max_smem_optin)
        return fail(ctx, CTOX_MEMORY_BUDGET, "queries, keys and values of %zu values do not fit shared memory", all);
    if (smem > 40 * 1024)
        CTOX_CUDA(ctx, cudaFuncSetAttribute(k_qkv_prep, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_qkv_prep, dim3(parts, m), dim3(kQkvThreads), smem, ctx->stream, a));
    timing_end(ctx, KC_QKV, (double)m * ((a.heads + a.kv_heads) * a.dim * 4.0 + a.kv_heads * a.vdim * 4.0 +
                                         a.heads * a.dim_pad * (a.q_b16 ? 2.0 : 4.0) +
                                         a.kv_heads * (a.dim_pad + a.vdim_pad) * (a.bf16 ? 2.0 : 4.0)), 0);
    return CTOX_OK;
}

}  // namespace ctox
