// Attention of layer stacks in long passes: 128 queries of one head per CTA against 64-token key tiles.
//
// Scores and the weighted sum run on tcgen05.mma with operands staged by TMA; scores (double-buffered) and
// the output accumulate in tensor memory. One warp loads, one issues the products, four hold one query
// row per thread for the softmax: they read the scores from tensor memory, write the weights over them as
// the next product's operand, and rescale the output only when a row's maximum has grown by more than 2^8
// since its last reference (the final division makes up for it). Two CTAs share an SM when their buffers
// fit, so one's softmax overlaps the other's products.
#include "stack_attention.cuh"
#include "umma.cuh"

#include <cmath>

namespace ctox {

constexpr int kSpThreads = 192;
constexpr uint32_t kSpQ = 128, kSpK = 64;

// CACHED: keys and values are tiles of the cache itself, the values as an operand whose rows run along the
// keys; otherwise both come expanded per head (values transposed) with a rotated key part from the cache.
template <bool CACHED>
__global__ void __launch_bounds__(kSpThreads)
    k_prefill_attention(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_qr,
                     const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_kr,
                     const __grid_constant__ CUtensorMap map_v, PrefillAttn a, uint32_t k_stages, uint32_t v_stages, uint32_t tmem_cols,
                     int32_t *error_word) {
    using namespace umma;
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t bars[16];
    __shared__ uint32_t tmem_slot;
    __shared__ volatile int dead;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t D = a.dim_pad + a.rot_pad;
    const HeadBox bd = head_box(a.dim_pad), br = head_box(a.rot_pad);
    const uint32_t v_boxes = (a.vdim_pad + 63) / 64;  // CACHED: boxes of 64 values x 64 keys
    const uint32_t q_bytes = kSpQ * D * 2, k_bytes = kSpK * D * 2, v_bytes = (CACHED ? v_boxes * 64 : a.vdim_pad) * kSpK * 2;
    const uint32_t base = (smem_addr(raw) + 1023) & ~1023u;
    const uint32_t q_s = base, k_s = q_s + q_bytes, v_s = k_s + k_stages * k_bytes;
    const uint32_t b0 = smem_addr(bars), q_full = b0, k_full = b0 + 8, k_empty = b0 + 24, v_full = b0 + 40,
                   v_empty = b0 + 56, s_full = b0 + 72, p_full = b0 + 88, o_done = b0 + 104, drained = b0 + 120;
    if (tid == 0) {
        dead = 0;
        bar_init(q_full, 1);
        for (uint32_t i = 0; i < 2; ++i) {
            bar_init(k_full + i * 8, 1);
            bar_init(k_empty + i * 8, 1);
            bar_init(v_full + i * 8, 1);
            bar_init(v_empty + i * 8, 1);
            bar_init(s_full + i * 8, 1);
            bar_init(p_full + i * 8, 4);
            bar_init(o_done + i * 8, 1);
        }
        bar_init(drained, 1);
        bar_init_fence();
    }
    if (warp == 1) tmem_alloc(smem_addr(&tmem_slot), tmem_cols);
    fence_before();
    __syncthreads();
    fence_after();
    pdl_launch();
    const uint32_t tmem = tmem_slot, tmem_o = tmem + 2 * kSpK;
    const uint32_t q_tiles = (a.m + kSpQ - 1) / kSpQ;
    const uint32_t i0 = (q_tiles - 1 - blockIdx.x % q_tiles) * kSpQ, head = blockIdx.x / q_tiles;
    const uint32_t part = CACHED ? head / (a.heads / a.kv_heads) * (a.dim_pad + a.vdim_pad) : 0;  // of a cached token
    const uint32_t p_first = a.pos0 + i0, p_last = a.pos0 + min(i0 + kSpQ, a.m) - 1;
    const uint32_t key_lo = a.window && p_first + 1 > a.window ? p_first + 1 - a.window : 0;
    const uint32_t t_lo = (key_lo - a.row0) / kSpK, n = (p_last - a.row0) / kSpK - t_lo + 1;
    pdl_wait();
    if (warp == 0) {
        if (lane == 0) {
            bar_expect(q_full, q_bytes);
            for (uint32_t i = 0; i < bd.n; ++i)
                tma_load(q_s + i * kSpQ * bd.width * 2, &map_q, q_full, (int)(head * D + i * bd.width), (int)i0);
            for (uint32_t i = 0; i < br.n; ++i)
                tma_load(q_s + kSpQ * a.dim_pad * 2 + i * kSpQ * br.width * 2, &map_qr, q_full,
                         (int)(head * D + a.dim_pad + i * br.width), (int)i0);
            uint32_t k_issued = 0, v_issued = 0;
            bool ok = true;
            for (uint32_t j = 0; j < n; ++j) {
                const uint32_t row = (t_lo + j) * kSpK, s = j % k_stages, round = j / k_stages, vs = j % v_stages,
                               v_round = j / v_stages;
                if (round > 0 && !(ok = bar_wait(k_empty + s * 8, (round - 1) & 1, &dead))) break;
                const uint32_t pos = a.row0 + row;
                const int slot = (int)(a.page_table[pos / a.page_tokens] * a.page_tokens + pos % a.page_tokens);
                const uint32_t kd = k_s + s * k_bytes;
                bar_expect(k_full + s * 8, k_bytes);
                for (uint32_t i = 0; i < bd.n; ++i)
                    tma_load(kd + i * kSpK * bd.width * 2, &map_k, k_full + s * 8,
                             (int)((CACHED ? part : head * a.dim_pad) + i * bd.width), CACHED ? slot : (int)row);
                for (uint32_t i = 0; i < br.n; ++i)
                    tma_load(kd + kSpK * a.dim_pad * 2 + i * kSpK * br.width * 2, &map_kr, k_full + s * 8,
                             (int)(a.rot_off + i * br.width), slot);
                ++k_issued;
                if (v_round > 0 && !(ok = bar_wait(v_empty + vs * 8, (v_round - 1) & 1, &dead))) break;
                bar_expect(v_full + vs * 8, v_bytes);
                if (CACHED)
                    for (uint32_t i = 0; i < v_boxes; ++i)
                        tma_load(v_s + vs * v_bytes + i * 64 * kSpK * 2, &map_v, v_full + vs * 8, (int)(part + a.dim_pad + i * 64), slot);
                else
                    tma_load(v_s + vs * v_bytes, &map_v, v_full + vs * 8, (int)row, (int)(head * a.vdim_pad));
                ++v_issued;
            }
            if (!ok) {  // leave no copy in flight behind
                bar_drain(q_full, 0);
                for (uint32_t s = 0; s < k_stages && s < k_issued; ++s) bar_drain(k_full + s * 8, ((k_issued - 1 - s) / k_stages) & 1);
                for (uint32_t s = 0; s < v_stages && s < v_issued; ++s) bar_drain(v_full + s * 8, ((v_issued - 1 - s) / v_stages) & 1);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = idesc_bf16(kSpQ, kSpK), idesc_o = idesc_bf16_mn(kSpQ, a.vdim_pad, false, CACHED);
            auto scores = [&](uint32_t j) -> bool {
                const uint32_t s = j % k_stages;
                if (!bar_wait(k_full + s * 8, (j / k_stages) & 1, &dead)) return false;
                fence_after();
                const uint32_t d = tmem + (j & 1) * kSpK, kd = k_s + s * k_bytes;
                bool acc = false;
                for (uint32_t i = 0; i < bd.n; ++i)
                    for (uint32_t k = 0; k < bd.width; k += 16, acc = true)
                        mma_f16(d, smem_desc(q_s + i * kSpQ * bd.width * 2 + k * 2, bd.width * 2),
                                smem_desc(kd + i * kSpK * bd.width * 2 + k * 2, bd.width * 2), idesc_s, acc);
                for (uint32_t i = 0; i < br.n; ++i)
                    for (uint32_t k = 0; k < br.width; k += 16, acc = true)
                        mma_f16(d, smem_desc(q_s + kSpQ * a.dim_pad * 2 + i * kSpQ * br.width * 2 + k * 2, br.width * 2),
                                smem_desc(kd + kSpK * a.dim_pad * 2 + i * kSpK * br.width * 2 + k * 2, br.width * 2), idesc_s,
                                acc);
                commit(k_empty + s * 8);
                commit(s_full + (j & 1) * 8);
                return true;
            };
            bool ok = bar_wait(q_full, 0, &dead) && scores(0);
            for (uint32_t j = 0; j < n && ok; ++j) {
                if (j + 1 < n && !(ok = scores(j + 1))) break;
                const uint32_t s = j % v_stages;
                if (!(ok = bar_wait(p_full + (j & 1) * 8, (j >> 1) & 1, &dead) && bar_wait(v_full + s * 8, (j / v_stages) & 1, &dead))) break;
                fence_after();
                const uint32_t p = tmem + (j & 1) * kSpK;  // the weights, where the scores were
                const uint64_t dv = CACHED ? smem_desc_mn(v_s + s * v_bytes, 128, 64 * kSpK * 2) : smem_desc(v_s + s * v_bytes, 128);
#pragma unroll
                for (uint32_t k = 0; k < kSpK / 16; ++k)
                    mma_f16_ts(tmem_o, p + k * 8, dv + k * (CACHED ? 16 * 128 / 16 : 2), idesc_o, j > 0 || k > 0);
                commit(v_empty + s * 8);
                commit(o_done + (j & 1) * 8);
            }
            if (!ok) {
                commit(drained);
                bar_drain(drained, 0);
            }
        }
    } else {
        const uint32_t quarter = warp & 3, row = quarter * 32 + lane;
        const uint32_t lanes = (quarter * 32) << 16;
        const uint32_t pos = a.pos0 + i0 + row;
        const float c = a.scale * 1.4426950408889634f;
        float ref = -INFINITY, sum[4] = {0.f, 0.f, 0.f, 0.f};
        if (a.sink) {  // a first key whose score is the sink and whose value is zero
            ref = a.sink[head] * 1.4426950408889634f;
            sum[0] = 1.f;
        }
        bool ok = true;
        for (uint32_t j = 0; j < n; ++j) {
            if (!(ok = __all_sync(0xffffffffu, bar_wait(s_full + (j & 1) * 8, (j >> 1) & 1, &dead)))) break;
            fence_after();
            float s[kSpK];
            tmem_ld32(tmem + (j & 1) * kSpK + lanes, s);
            tmem_ld32(tmem + (j & 1) * kSpK + 32 + lanes, s + 32);
            tmem_ld_wait();
            const uint32_t t0 = a.row0 + (t_lo + j) * kSpK;
            const bool all = t0 + kSpK - 1 <= p_first && (!a.window || p_last < t0 + a.window);
            if (!all) {
#pragma unroll
                for (uint32_t k = 0; k < kSpK; ++k) {
                    const uint32_t t = t0 + k;
                    if (t > pos || (a.window && pos - t >= a.window)) s[k] = -INFINITY;
                }
            }
            float m4[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
            for (uint32_t k = 4; k < kSpK; ++k) m4[k & 3] = fmaxf(m4[k & 3], s[k]);
            const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * c;
            const bool grow = mx > ref + 8.f || (ref == -INFINITY && mx > ref);
            if (__any_sync(0xffffffffu, grow)) {
                const float f = grow ? ex2(ref - mx) : 1.f;  // ref = -inf: 0, and nothing but zeros was added
                if (grow) {
                    ref = mx;
#pragma unroll
                    for (int i = 0; i < 4; ++i) sum[i] *= f;
                }
                if (j > 0) {  // the output belongs to the product of the tile before until that has finished
                    if (!(ok = __all_sync(0xffffffffu, bar_wait(o_done + ((j - 1) & 1) * 8, ((j - 1) >> 1) & 1, &dead)))) break;
                    fence_after();
                    for (uint32_t d = 0; d < a.vdim_pad; d += 16) {
                        float o[16];
                        tmem_ld16(tmem_o + d + lanes, o);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 16; ++i) o[i] *= f;
                        tmem_st16(tmem_o + d + lanes, o);
                    }
                }
            }
            const float r = ref == -INFINITY ? 0.f : ref;
            uint32_t p[kSpK / 2];
#pragma unroll
            for (uint32_t k = 0; k < kSpK; k += 2) {
                const float a0 = ex2(fmaf(s[k], c, -r)), a1 = ex2(fmaf(s[k + 1], c, -r));
                sum[k & 2] += a0;
                sum[(k & 2) + 1] += a1;
                const __nv_bfloat162 b = __floats2bfloat162_rn(a0, a1);
                p[k / 2] = *reinterpret_cast<const uint32_t *>(&b);
            }
            tmem_st32(tmem + (j & 1) * kSpK + lanes, p);
            tmem_st_wait();
            fence_before();
            __syncwarp();
            // A warp may be one tile ahead of another (the next scores are already there), but not two: those
            // are issued once all four have arrived here. Hence a barrier each for even and odd tiles.
            if (lane == 0) bar_arrive(p_full + (j & 1) * 8);
        }
        // Most tiles skip the wait for the product before them, and a wait tells a phase from its neighbours
        // only. Hence one barrier for even and one for odd tiles: having seen the scores of tile j, the
        // products up to j - 2 are complete and the one of tile j + 1 cannot be, so either wait (here and at a
        // rescale) meets its barrier in the phase it asks for or the one right before.
        if (ok && (ok = __all_sync(0xffffffffu, bar_wait(o_done + ((n - 1) & 1) * 8, ((n - 1) >> 1) & 1, &dead)))) {
            fence_after();
            const float inv = 1.0f / ((sum[0] + sum[1]) + (sum[2] + sum[3]));
            __nv_bfloat16 *out = a.out + ((size_t)(i0 + row) * a.heads + head) * a.vdim_pad;
            for (uint32_t d = 0; d < a.vdim_pad; d += 16) {
                float o[16];
                tmem_ld16(tmem_o + d + lanes, o);
                tmem_ld_wait();
                uint32_t h[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const __nv_bfloat162 b = __floats2bfloat162_rn(o[2 * i] * inv, o[2 * i + 1] * inv);
                    h[i] = *reinterpret_cast<const uint32_t *>(&b);
                }
                if (i0 + row < a.m) {
                    *reinterpret_cast<uint4 *>(out + d) = make_uint4(h[0], h[1], h[2], h[3]);
                    *reinterpret_cast<uint4 *>(out + d + 8) = make_uint4(h[4], h[5], h[6], h[7]);
                }
            }
            fence_before();
        }
    }
    __syncwarp();
    __syncthreads();
    if (warp == 1) {
        fence_after();
        tmem_free(tmem, tmem_cols);
    }
    if (tid == 0 && dead) *error_word = DEV_ERR_WAIT_TIMEOUT;
}

namespace {

size_t sp_smem(uint32_t dim_pad, uint32_t rot_pad, uint32_t vdim_pad, uint32_t k_stages, uint32_t v_stages) {
    const size_t D = dim_pad + rot_pad;
    return 1024 + kSpQ * D * 2 + k_stages * kSpK * D * 2 + (size_t)v_stages * ((vdim_pad + 63) / 64 * 64) * kSpK * 2;
}

}  // namespace

bool prefill_attention_fits(const ctox_ctx *ctx, uint32_t dim_pad, uint32_t rot_pad, uint32_t vdim_pad) {
    return vdim_pad <= 256 && sp_smem(dim_pad, rot_pad, vdim_pad, 1, 1) + 1024 <= (size_t)ctx->max_smem_optin;
}

template <bool CACHED>
static ctox_status prefill_attention_launch(ctox_ctx *ctx, const PrefillAttn &a) {
    if (!prefill_attention_fits(ctx, a.dim_pad, a.rot_pad, a.vdim_pad) || a.page_tokens % kSpQ || a.row0 % kSpQ ||
        (!CACHED && a.vt_ld % 8) || (CACHED && (a.rot_pad || a.heads % a.kv_heads)))
        return fail(ctx, CTOX_SHAPE, "prefill attention: unsupported sizes");
    const size_t half = ((size_t)ctx->max_smem_optin - 2048) / 2 - 1024;  // two CTAs on an SM
    // the deepest buffering that lets two CTAs share an SM; else the deepest that fits one
    uint32_t ks = 0, vs = 0;
    for (size_t limit : {half, (size_t)ctx->max_smem_optin - 1024}) {
        for (uint32_t i = 0; i < 4 && !ks; ++i) {
            const uint32_t k = i < 2 ? 2 : 1, v = i == 0 || i == 2 ? 2 : 1;
            if (sp_smem(a.dim_pad, a.rot_pad, a.vdim_pad, k, v) <= limit) {
                ks = k;
                vs = v;
            }
        }
    }
    const size_t smem = sp_smem(a.dim_pad, a.rot_pad, a.vdim_pad, ks, vs);
    uint32_t cols = 256;  // scores 2 x 64 and the output
    if (2 * kSpK + a.vdim_pad > 256) cols = 512;
    const HeadBox bd = head_box(a.dim_pad), br = a.rot_pad ? head_box(a.rot_pad) : HeadBox{16, 0};
    const uint64_t qw = (uint64_t)a.heads * (a.dim_pad + a.rot_pad), kw = (uint64_t)a.heads * a.dim_pad, cw = a.slot_cols;
    CUtensorMap mq, mqr, mk, mkr, mv;
    EX(tensor_map_bf16(ctx, &mq, a.q, a.m, qw, qw, kSpQ, bd.width));
    EX(tensor_map_bf16(ctx, &mqr, a.q, a.m, qw, qw, kSpQ, br.width));
    if (CACHED) {
        EX(tensor_map_bf16(ctx, &mk, a.cache, a.slots, cw, cw, kSpK, bd.width));
        EX(tensor_map_bf16(ctx, &mv, a.cache, a.slots, cw, cw, kSpK, 64));
    } else {
        EX(tensor_map_bf16(ctx, &mk, a.k, a.span, kw, kw, kSpK, bd.width));
        EX(tensor_map_bf16(ctx, &mv, a.vt, (uint64_t)a.heads * a.vdim_pad, a.span, a.vt_ld, a.vdim_pad, kSpK));
    }
    EX(tensor_map_bf16(ctx, &mkr, a.cache, a.slots, cw, cw, kSpK, br.width));
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_prefill_attention<CACHED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const uint32_t grid = (a.m + kSpQ - 1) / kSpQ * a.heads;
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_prefill_attention<CACHED>, dim3(grid), dim3(kSpThreads), smem, ctx->stream, mq, mqr, mk, mkr, mv,
                              a, ks, vs, cols, ctx->dev_error));
    double pairs = 0;  // visible (query, key) pairs
    if (ctx->timing)
        for (uint32_t i = 0; i < a.m; ++i) {
            const uint32_t seen = a.pos0 + i + 1;
            pairs += a.window && seen > a.window ? a.window : seen;
        }
    const double keys = CACHED ? (double)a.span * cw : a.span * (kw + (double)a.heads * a.vdim_pad);
    timing_end(ctx, KC_STACK_PREFILL, 2.0 * (a.m * (qw + (double)a.heads * a.vdim_pad) + keys),
               2.0 * pairs * a.heads * (a.dim_pad + a.rot_pad + a.vdim_pad));
    return CTOX_OK;
}

ctox_status launch_prefill_attention(ctox_ctx *ctx, const PrefillAttn &a) {
    return a.kv_heads ? prefill_attention_launch<true>(ctx, a) : prefill_attention_launch<false>(ctx, a);
}

}  // namespace ctox
