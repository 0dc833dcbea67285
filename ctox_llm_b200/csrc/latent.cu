// Attention over the latent cache for short passes (decode and small portions of a prompt).
#include "latent.cuh"

#include <cmath>

namespace ctox {

constexpr int kLaThreads = 256, kLaWarps = 8;
constexpr int kLaRowsMma = 16, kLaTileMma = 64;  // query rows per CTA, tokens per tile (tensor cores)
constexpr int kLaRowsFma = 8, kLaTileFma = 32;   // the same on CUDA cores

struct KeyRange {
    uint32_t lo, hi;
};
__host__ __device__ inline KeyRange key_range(uint32_t pos0, uint32_t m, uint32_t window) {
    KeyRange r;
    r.hi = pos0 + m;
    r.lo = window && pos0 + 1 > window ? pos0 + 1 - window : 0;
    return r;
}
__device__ __forceinline__ bool key_visible(uint32_t key, uint32_t pos, uint32_t window) {
    return key <= pos && (!window || pos - key < window);
}

template <typename T>
__device__ __forceinline__ float cache_value(const T *p);
template <>
__device__ __forceinline__ float cache_value<float>(const float *p) { return *p; }
template <>
__device__ __forceinline__ float cache_value<__nv_bfloat16>(const __nv_bfloat16 *p) { return __bfloat162float(*p); }

// CUDA cores, fp32 throughout: eight query rows against 32-token tiles; a warp scores one row (lane =
// token), then every thread owns J latent columns of all eight rows.
template <typename T, int J>
__global__ void __launch_bounds__(kLaThreads) k_latent_attention(LatentAttn a, uint32_t splits) {
    pdl_launch();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const uint32_t D = a.kv_pad + a.rot_pad, ldk = D + 1, rows = a.m * a.heads;
    float *q_s = sm;                           // [8][D]
    float *k_s = q_s + kLaRowsFma * D;          // [32][D + 1]
    float *p_s = k_s + kLaTileFma * ldk;        // [8][32]
    float *al_s = p_s + kLaRowsFma * kLaTileFma;  // [8]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t row0 = blockIdx.x * kLaRowsFma, sp = blockIdx.y, row = row0 + warp;
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const uint32_t tiles = (kr.hi - kr.lo + kLaTileFma - 1) / kLaTileFma;
    const uint32_t t_beg = (uint32_t)((uint64_t)tiles * sp / splits), t_end = (uint32_t)((uint64_t)tiles * (sp + 1) / splits);
    for (uint32_t i = tid; i < kLaRowsFma * D; i += kLaThreads) {
        const uint32_t r = row0 + i / D, c = i % D;
        q_s[i] = r >= rows ? 0.f
                           : (c < a.kv_pad ? a.q_abs[(size_t)r * a.kv_pad + c] : a.q_rot[(size_t)r * a.q_stride + c - a.kv_pad]);
    }
    float o[kLaRowsFma][J];
#pragma unroll
    for (int r = 0; r < kLaRowsFma; ++r)
#pragma unroll
        for (int j = 0; j < J; ++j) o[r][j] = 0.f;
    float mx = -INFINITY, sum = 0.f;
    const uint32_t pos = a.pos0 + row / a.heads;
    for (uint32_t tile = t_beg; tile < t_end; ++tile) {
        const uint32_t t0 = kr.lo + tile * kLaTileFma;
        __syncthreads();
        for (uint32_t r = warp; r < kLaTileFma; r += kLaWarps) {
            const uint32_t t = t0 + r;
            const T *src = t < kr.hi ? (const T *)a.cache + paged_slot(a.page_table, a.page_tokens, t) * D : nullptr;
            for (uint32_t c = lane; c < D; c += 32) k_s[r * ldk + c] = src ? cache_value(src + c) : 0.f;
        }
        __syncthreads();
        const uint32_t t = t0 + lane;
        float s = -INFINITY;
        if (row < rows && t < kr.hi && key_visible(t, pos, a.window)) {
            float s0 = 0.f, s1 = 0.f;
            const float *q = q_s + warp * D, *k = k_s + lane * ldk;
            for (uint32_t c = 0; c < D; c += 2) {
                s0 = fmaf(q[c], k[c], s0);
                s1 = fmaf(q[c + 1], k[c + 1], s1);
            }
            s = (s0 + s1) * a.scale;
        }
        float tm = s;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, off));
        const float nm = fmaxf(mx, tm);
        const float alpha = nm == -INFINITY ? 1.f : expf(mx - nm);
        const float p = s == -INFINITY ? 0.f : expf(s - nm);
        float ps = p;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, off);
        sum = sum * alpha + ps;
        mx = nm;
        p_s[warp * kLaTileFma + lane] = p;
        if (lane == 0) al_s[warp] = alpha;
        __syncthreads();
#pragma unroll
        for (int r = 0; r < kLaRowsFma; ++r) {
            const float al = al_s[r];
#pragma unroll
            for (int j = 0; j < J; ++j) o[r][j] *= al;
        }
        for (uint32_t k = 0; k < kLaTileFma; ++k) {
            float v[J];
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const uint32_t c = tid + j * kLaThreads;
                v[j] = c < a.kv_pad ? k_s[k * ldk + c] : 0.f;
            }
#pragma unroll
            for (int r = 0; r < kLaRowsFma; ++r) {
                const float pr = p_s[r * kLaTileFma + k];
#pragma unroll
                for (int j = 0; j < J; ++j) o[r][j] = fmaf(pr, v[j], o[r][j]);
            }
        }
    }
    if (lane == 0 && row < rows) {
        a.ws_ml[((size_t)sp * rows + row) * 2] = mx;
        a.ws_ml[((size_t)sp * rows + row) * 2 + 1] = sum;
    }
#pragma unroll
    for (int r = 0; r < kLaRowsFma; ++r)
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const uint32_t c = tid + j * kLaThreads;
            if (c < a.kv_pad && row0 + r < rows) a.ws_o[((size_t)sp * rows + row0 + r) * a.kv_pad + c] = o[r][j];
        }
}

// ------------------------------------------------------------------ tensor cores, bf16 cache
__device__ __forceinline__ uint32_t smem_u32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm_x4(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
__device__ __forceinline__ void mma_bf16(float *c, const uint32_t *a, const uint32_t *b) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void split_bf16(float v, __nv_bfloat16 &hi, __nv_bfloat16 &lo) {
    hi = __float2bfloat16_rn(v);
    lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}

// Sixteen query rows against 64-token tiles of cache rows. The row dimension is dealt to the warps in steps
// of 16 values, so a warp keeps its part of the queries in registers and reads its part of a tile once;
// the partial scores meet in shared memory, where sixteen threads hold a query row for the softmax.
// Weighted sum: each warp every eighth group of eight latent columns, the same tile read as the
// transposed operand. Queries and weights are split into two bf16 parts (about 16 bits), so the only bf16
// rounding is the cache's. NT: groups of eight latent columns per warp.
__host__ __device__ constexpr int la_steps(int nt) { return nt <= 2 ? 2 : nt / 2 + 1; }  // 16-value steps of a row per warp
constexpr uint32_t kLaLdP = kLaTileMma + 8, kLaLdS = kLaTileMma + 4;

template <int NT>
__global__ void __launch_bounds__(kLaThreads, 1) k_latent_attention_mma(LatentAttn a, uint32_t splits, uint32_t stages) {
    constexpr int NK = la_steps(NT), JG = NT < 4 ? NT : 4;
    pdl_launch();
    extern __shared__ __align__(16) uint8_t smraw[];
    const uint32_t D = a.kv_pad + a.rot_pad, ld = D + 8, rows = a.m * a.heads;
    __nv_bfloat16 *k_s = reinterpret_cast<__nv_bfloat16 *>(smraw);           // [stages][64][ld]
    float *s_s = reinterpret_cast<float *>(k_s + (size_t)stages * kLaTileMma * ld);  // [8 warps][16][kLaLdS]
    __nv_bfloat16 *p_s = reinterpret_cast<__nv_bfloat16 *>(s_s + kLaWarps * kLaRowsMma * kLaLdS);  // [hi, lo][16][kLaLdP]
    float *al_s = reinterpret_cast<float *>(p_s + 2 * kLaRowsMma * kLaLdP);  // [16]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t row0 = blockIdx.x * kLaRowsMma, sp = blockIdx.y;
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const uint32_t tiles = (kr.hi - kr.lo + kLaTileMma - 1) / kLaTileMma;
    const uint32_t t_beg = (uint32_t)((uint64_t)tiles * sp / splits), t_end = (uint32_t)((uint64_t)tiles * (sp + 1) / splits);
    const uint32_t chunks = D / 8;
    pdl_wait();
    auto load_tile = [&](uint32_t tile, uint32_t stage) {
        // lane i < 8 looks the slot of this warp's row i up, for all lanes
        const uint32_t mine = kr.lo + tile * kLaTileMma + warp + (lane & 7) * kLaWarps;
        const uint32_t slot = mine < kr.hi ? (uint32_t)paged_slot(a.page_table, a.page_tokens, mine) : 0xffffffffu;
#pragma unroll
        for (uint32_t i = 0; i < kLaTileMma / kLaWarps; ++i) {
            const uint32_t r = warp + i * kLaWarps, from = __shfl_sync(0xffffffffu, slot, i);
            const bool in = from != 0xffffffffu;
            const __nv_bfloat16 *src = (const __nv_bfloat16 *)a.cache + (in ? (size_t)from * D : 0);
            __nv_bfloat16 *dst = k_s + ((size_t)stage * kLaTileMma + r) * ld;
            for (uint32_t c = lane; c < chunks; c += 32)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + c * 8)), "l"(src + c * 8),
                             "r"(in ? 16 : 0)
                             : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (t_beg < t_end) load_tile(t_beg, 0);
    if (stages == 2 && t_beg + 1 < t_end) load_tile(t_beg + 1, 1);
    // ---- this warp's part of the queries: steps warp, warp + 8, ... as operand fragments
    const float qscale = a.scale * 1.4426950408889634f;  // scores in units of log 2
    uint32_t qh[NK][4], ql[NK][4];
    {
        float2 v[NK][4];
#pragma unroll
        for (int i = 0; i < NK; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {  // rows g, g + 8; values 2 t4 and 2 t4 + 8
                const uint32_t row = row0 + g + (j & 1) * 8, c = (warp + i * kLaWarps) * 16 + t4 * 2 + (j >> 1) * 8;
                v[i][j] = make_float2(0.f, 0.f);
                if (row < rows && c < D)
                    v[i][j] = *reinterpret_cast<const float2 *>(c < a.kv_pad ? a.q_abs + (size_t)row * a.kv_pad + c
                                                                             : a.q_rot + (size_t)row * a.q_stride + (c - a.kv_pad));
            }
#pragma unroll
        for (int i = 0; i < NK; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                __nv_bfloat162 hi, lo;
                split_bf16(v[i][j].x * qscale, hi.x, lo.x);
                split_bf16(v[i][j].y * qscale, hi.y, lo.y);
                qh[i][j] = *reinterpret_cast<uint32_t *>(&hi);
                ql[i][j] = *reinterpret_cast<uint32_t *>(&lo);
            }
    }
    float o[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    // softmax: thread = (query row, four tokens of a tile)
    const uint32_t srow = tid >> 4, stok = (tid & 15) * 4, qrow = row0 + srow, qpos = a.pos0 + qrow / a.heads;
    float mx = -INFINITY, sum = 0.f;
    const uint32_t p_addr = smem_u32(p_s + (lane & 15) * kLaLdP + (lane >> 4) * 8);
    for (uint32_t tile = t_beg; tile < t_end; ++tile) {
        const uint32_t st = stages == 2 ? (tile - t_beg) & 1 : 0;
        if (stages == 2 && tile + 1 < t_end)  // the next tile may still be on its way
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        else
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const __nv_bfloat16 *kt = k_s + (size_t)st * kLaTileMma * ld;
        // ---- partial scores over this warp's steps
        float s[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
        const uint32_t k_addr = smem_u32(kt + ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int i = 0; i < NK; ++i) {
            const uint32_t c = (warp + i * kLaWarps) * 16;
            if (c < D) {
#pragma unroll
                for (int n = 0; n < 8; n += 4) {  // two groups of eight tokens per load
                    uint32_t b[8];
                    ldsm_x4(b, k_addr + (n * 8 * ld + c) * 2);
                    ldsm_x4(b + 4, k_addr + ((n + 2) * 8 * ld + c) * 2);
#pragma unroll
                    for (int k = 0; k < 4; ++k) mma_bf16(s[n + k], qh[i], b + 2 * k);
#pragma unroll
                    for (int k = 0; k < 4; ++k) mma_bf16(s[n + k], ql[i], b + 2 * k);
                }
            }
        }
        float *sw = s_s + warp * kLaRowsMma * kLaLdS;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            *reinterpret_cast<float2 *>(sw + g * kLaLdS + n * 8 + t4 * 2) = make_float2(s[n][0], s[n][1]);
            *reinterpret_cast<float2 *>(sw + (g + 8) * kLaLdS + n * 8 + t4 * 2) = make_float2(s[n][2], s[n][3]);
        }
        __syncthreads();
        // ---- scores of one row's four tokens, softmax
        float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int w = 0; w < kLaWarps; ++w) {
            const float4 q = *reinterpret_cast<const float4 *>(s_s + (w * kLaRowsMma + srow) * kLaLdS + stok);
            v[0] += q.x;
            v[1] += q.y;
            v[2] += q.z;
            v[3] += q.w;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const uint32_t t = kr.lo + tile * kLaTileMma + stok + j;
            if (qrow >= rows || t >= kr.hi || !key_visible(t, qpos, a.window)) v[j] = -INFINITY;
        }
        float nm = fmaxf(fmaxf(v[0], v[1]), fmaxf(v[2], v[3]));
#pragma unroll
        for (int off = 8; off > 0; off >>= 1) nm = fmaxf(nm, __shfl_xor_sync(0xffffffffu, nm, off));
        nm = fmaxf(nm, mx);
        const float alpha = nm == -INFINITY ? 1.f : exp2f(mx - nm);
        mx = nm;
        __nv_bfloat16 hi[4], lo[4];
        float ps = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float p = v[j] == -INFINITY ? 0.f : exp2f(v[j] - nm);
            ps += p;
            split_bf16(p, hi[j], lo[j]);
        }
        sum = sum * alpha + ps;  // this thread's tokens; the row is added up at the end
        *reinterpret_cast<uint2 *>(p_s + srow * kLaLdP + stok) = *reinterpret_cast<uint2 *>(hi);
        *reinterpret_cast<uint2 *>(p_s + (kLaRowsMma + srow) * kLaLdP + stok) = *reinterpret_cast<uint2 *>(lo);
        if ((tid & 15) == 0) al_s[srow] = alpha;
        __syncthreads();
        // ---- weighted sum of the cache rows
        const float al0 = al_s[g], al1 = al_s[g + 8];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            o[j][0] *= al0;
            o[j][1] *= al0;
            o[j][2] *= al1;
            o[j][3] *= al1;
        }
#pragma unroll
        for (uint32_t k = 0; k < kLaTileMma; k += 32) {
            uint32_t ph[2][4], pl[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                ldsm_x4(ph[i], p_addr + (k + i * 16) * 2);
                ldsm_x4(pl[i], p_addr + kLaRowsMma * kLaLdP * 2 + (k + i * 16) * 2);
            }
            const uint32_t v_addr = smem_u32(kt + (k + lane) * ld);
#pragma unroll
            for (int j0 = 0; j0 < NT; j0 += JG) {  // JG independent accumulators between dependent products
                uint32_t b[JG][4];
#pragma unroll
                for (int j = 0; j < JG; ++j) {  // groups past the latent repeat the first (never stored)
                    const uint32_t n = (warp + (j0 + j) * kLaWarps) * 8;
                    ldsm_x4_t(b[j], v_addr + (n < a.kv_pad ? n : 0) * 2);
                }
#pragma unroll
                for (int j = 0; j < JG; ++j) mma_bf16(o[j0 + j], ph[0], b[j]);
#pragma unroll
                for (int j = 0; j < JG; ++j) mma_bf16(o[j0 + j], pl[0], b[j]);
#pragma unroll
                for (int j = 0; j < JG; ++j) mma_bf16(o[j0 + j], ph[1], b[j] + 2);
#pragma unroll
                for (int j = 0; j < JG; ++j) mma_bf16(o[j0 + j], pl[1], b[j] + 2);
            }
        }
        __syncthreads();
        if (tile + stages < t_end) load_tile(tile + stages, st);  // into the buffer just read
    }
#pragma unroll
    for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    if ((tid & 15) == 0 && qrow < rows) {
        a.ws_ml[((size_t)sp * rows + qrow) * 2] = mx * 0.6931471805599453f;
        a.ws_ml[((size_t)sp * rows + qrow) * 2 + 1] = sum;
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        const uint32_t n = (warp + j * kLaWarps) * 8;
        if (n >= a.kv_pad) continue;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t row = row0 + g + i * 8;
            if (row < rows)
                *reinterpret_cast<float2 *>(a.ws_o + ((size_t)sp * rows + row) * a.kv_pad + n + t4 * 2) =
                    make_float2(o[j][i * 2], o[j][i * 2 + 1]);
        }
    }
}

namespace {

size_t mma_smem(const LatentAttn &a, uint32_t stages) {
    return (size_t)stages * kLaTileMma * (a.kv_pad + a.rot_pad + 8) * 2 + kLaWarps * kLaRowsMma * kLaLdS * 4 +
           2 * kLaRowsMma * kLaLdP * 2 + kLaRowsMma * 4;
}
// Smallest form (NT) of the tensor-core kernel that takes these rows; 0: none does.
int mma_form(const LatentAttn &a) {
    for (int nt : {1, 2, 4, 8, 16})
        if (a.kv_pad <= 64u * nt && a.kv_pad + a.rot_pad <= 128u * la_steps(nt)) return nt;
    return 0;
}
// Tile stages of the tensor-core form (0: it does not apply).
uint32_t mma_stages(const ctox_ctx *ctx, const LatentAttn &a) {
    if (!a.bf16 || !mma_form(a)) return 0;
    for (uint32_t st = 2; st > 0; --st)
        if (mma_smem(a, st) <= (size_t)ctx->max_smem_optin) return st;
    return 0;
}
size_t fma_smem(const LatentAttn &a) {
    const size_t D = a.kv_pad + a.rot_pad;
    return (kLaRowsFma * D + kLaTileFma * (D + 1) + kLaRowsFma * kLaTileFma + kLaRowsFma) * 4;
}

template <typename T, int J>
ctox_status fma_launch(ctox_ctx *ctx, const LatentAttn &a, uint32_t splits, uint32_t row_tiles, size_t smem) {
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_latent_attention<T, J>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CTOX_CUDA(ctx, launch_pdl(k_latent_attention<T, J>, dim3(row_tiles, splits), dim3(kLaThreads), smem, ctx->stream, a, splits));
    return CTOX_OK;
}
template <int NT>
ctox_status mma_launch(ctox_ctx *ctx, const LatentAttn &a, uint32_t splits, uint32_t row_tiles, size_t smem, uint32_t stages) {
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_latent_attention_mma<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CTOX_CUDA(ctx, launch_pdl(k_latent_attention_mma<NT>, dim3(row_tiles, splits), dim3(kLaThreads), smem, ctx->stream, a,
                              splits, stages));
    return CTOX_OK;
}

}  // namespace

uint32_t latent_attn_splits(const ctox_ctx *ctx, const LatentAttn &a) {
    const bool mma = mma_stages(ctx, a) > 0;
    const uint32_t rows = a.m * a.heads, per = mma ? kLaRowsMma : kLaRowsFma, tile = mma ? kLaTileMma : kLaTileFma;
    const uint32_t row_tiles = (rows + per - 1) / per;
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const uint32_t tiles = (kr.hi - kr.lo + tile - 1) / tile;
    uint32_t s = (uint32_t)ctx->sm_count / row_tiles;
    // every product that merges the splits reads them all: many only where they shorten a long chain of tiles
    const uint32_t most = tiles >= 256 ? kAttnSplitsDense : kAttnSplitsDense / 2;
    if (s > most) s = most;
    if (s > tiles) s = tiles;
    return s ? s : 1;
}

static ctox_status latent_attention_any(ctox_ctx *ctx, const LatentAttn &a, uint32_t splits) {
    const uint32_t rows = a.m * a.heads, stages = mma_stages(ctx, a);
    if (stages) {
        const uint32_t row_tiles = (rows + kLaRowsMma - 1) / kLaRowsMma;
        const size_t smem = mma_smem(a, stages);
        switch (mma_form(a)) {
            case 1: return mma_launch<1>(ctx, a, splits, row_tiles, smem, stages);
            case 2: return mma_launch<2>(ctx, a, splits, row_tiles, smem, stages);
            case 4: return mma_launch<4>(ctx, a, splits, row_tiles, smem, stages);
            case 8: return mma_launch<8>(ctx, a, splits, row_tiles, smem, stages);
            default: return mma_launch<16>(ctx, a, splits, row_tiles, smem, stages);
        }
    }
    const size_t smem = fma_smem(a);
    const uint32_t row_tiles = (rows + kLaRowsFma - 1) / kLaRowsFma, j = (a.kv_pad + kLaThreads - 1) / kLaThreads;
    if (smem > (size_t)ctx->max_smem_optin || j > 8)
        return fail(ctx, CTOX_MEMORY_BUDGET, "latent attention: a latent of %u + %u values does not fit shared memory",
                    a.kv_pad, a.rot_pad);
#define FMA(T)                                                             \
    (j <= 1 ? fma_launch<T, 1>(ctx, a, splits, row_tiles, smem)            \
     : j <= 2 ? fma_launch<T, 2>(ctx, a, splits, row_tiles, smem)          \
     : j <= 4 ? fma_launch<T, 4>(ctx, a, splits, row_tiles, smem)          \
              : fma_launch<T, 8>(ctx, a, splits, row_tiles, smem))
    return a.bf16 ? FMA(__nv_bfloat16) : FMA(float);
#undef FMA
}

ctox_status launch_latent_attention(ctox_ctx *ctx, const LatentAttn &a, uint32_t splits) {
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const double keys = kr.hi - kr.lo;
    timing_begin(ctx);
    EX(latent_attention_any(ctx, a, splits));
    timing_end(ctx, KC_LATENT_ATTENTION, keys * (a.kv_pad + a.rot_pad) * (a.bf16 ? 2 : 4),
               2.0 * keys * a.m * a.heads * (2 * a.kv_pad + a.rot_pad));
    return CTOX_OK;
}

}  // namespace ctox
