// Attention of layer stacks over the paged cache, short passes (decode and small portions of a prompt).
#include "stack_attention.cuh"

#include <cmath>

namespace ctox {

constexpr int kCaThreads = 256, kCaWarps = 8;
constexpr int kCaRowsMma = 16, kCaTileMma = 64;  // query rows per CTA, tokens per tile (tensor cores)
constexpr int kCaRowsFma = 8, kCaTileFma = 32;   // the same on CUDA cores
constexpr int kSplitLanes = (kAttnSplitsDense + 31) / 32;  // splits per lane of a merging warp

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

// Query rows of one part of the cache: r = position * (heads per part) + head within the part.
// Without GROUPED there is one part, and r is the row.
template <bool GROUPED>
struct PartRows {
    uint32_t share, part, heads, n;
    __device__ __forceinline__ PartRows(const CacheAttn &a)
        : share(GROUPED ? a.heads / a.kv_heads : a.heads), part(GROUPED ? blockIdx.z : 0), heads(a.heads), n(a.m * share) {}
    __device__ __forceinline__ uint32_t position(uint32_t r) const { return r / share; }
    __device__ __forceinline__ uint32_t row(uint32_t r) const {
        return GROUPED ? r / share * heads + part * share + r % share : r;
    }
};

// The CTA that delivers the last split of a tile of query rows merges the tile: a warp per row, the splits in
// their order, the sink as one more term of the denominator.
__device__ void merge_splits(const CacheAttn &a, const PartRows<true> &pr, uint32_t splits, uint32_t row0, uint32_t tile_rows) {
    __shared__ uint32_t last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        uint32_t *word = a.arrived + blockIdx.z * gridDim.x + blockIdx.x;
        last = atomicAdd(word, 1u) == splits - 1;
        if (last) *word = 0;
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rows = a.m * a.heads;
    for (uint32_t r = row0 + warp; r < row0 + tile_rows && r < pr.n; r += blockDim.x >> 5) {
        const uint32_t row = pr.row(r);
        const float sink = a.sink ? a.sink[row % a.heads] : -INFINITY;
        float mv[kSplitLanes], mx = sink, den = 0.f;
#pragma unroll
        for (int i = 0; i < kSplitLanes; ++i) {
            const uint32_t sp = lane + i * 32;
            const float2 ml = sp < splits ? __ldcg(reinterpret_cast<const float2 *>(a.ws_ml + ((size_t)sp * rows + row) * 2))
                                          : make_float2(-INFINITY, 0.f);
            mv[i] = ml.x;
            mx = fmaxf(mx, ml.x);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
        for (int i = 0; i < kSplitLanes; ++i) {
            const uint32_t sp = lane + i * 32;
            mv[i] = mv[i] == -INFINITY ? 0.f : expf(mv[i] - mx);
            if (sp < splits) den += __ldcg(a.ws_ml + ((size_t)sp * rows + row) * 2 + 1) * mv[i];
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
        if (a.sink) den += expf(sink - mx);
        const float inv = 1.0f / den;
        for (uint32_t c0 = 0; c0 < a.val_cols; c0 += 128) {
            const uint32_t c = c0 + lane * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            for (uint32_t s0 = 0; s0 < splits; s0 += 8) {
                float4 o[8];
#pragma unroll
                for (uint32_t i = 0; i < 8; ++i)
                    o[i] = s0 + i < splits && c < a.val_cols
                               ? __ldcg(reinterpret_cast<const float4 *>(a.ws_o + ((size_t)(s0 + i) * rows + row) * a.val_cols + c))
                               : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (uint32_t i = 0; i < 8; ++i) {
                    const uint32_t sp = s0 + i;
                    float w = 0.f;
#pragma unroll
                    for (int j = 0; j < kSplitLanes; ++j) {
                        const float t = __shfl_sync(0xffffffffu, mv[j], sp & 31);
                        if (sp >> 5 == (uint32_t)j) w = t;
                    }
                    v.x = fmaf(w, o[i].x, v.x);
                    v.y = fmaf(w, o[i].y, v.y);
                    v.z = fmaf(w, o[i].z, v.z);
                    v.w = fmaf(w, o[i].w, v.w);
                }
            }
            if (c < a.val_cols)
                *reinterpret_cast<float4 *>(a.out + (size_t)row * a.val_cols + c) =
                    make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv);
        }
    }
}

template <typename T>
__device__ __forceinline__ float cache_value(const T *p);
template <>
__device__ __forceinline__ float cache_value<float>(const float *p) { return *p; }
template <>
__device__ __forceinline__ float cache_value<__nv_bfloat16>(const __nv_bfloat16 *p) { return __bfloat162float(*p); }

// CUDA cores, fp32 throughout: eight query rows against 32-token tiles; a warp scores one row (lane =
// token), then every thread owns J value columns of all eight rows.
template <typename T, int J, bool GROUPED>
__global__ void __launch_bounds__(kCaThreads) k_cache_attention(CacheAttn a, uint32_t splits) {
    pdl_launch();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const PartRows<GROUPED> pr(a);
    const uint32_t D = a.key_cols, ldk = a.head_cols + 1, rows = a.m * a.heads;
    float *q_s = sm;                           // [8][D]
    float *k_s = q_s + kCaRowsFma * D;          // [32][head_cols + 1]
    float *p_s = k_s + kCaTileFma * ldk;        // [8][32]
    float *al_s = p_s + kCaRowsFma * kCaTileFma;  // [8]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t row0 = blockIdx.x * kCaRowsFma, sp = blockIdx.y, row = row0 + warp;
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const uint32_t tiles = (kr.hi - kr.lo + kCaTileFma - 1) / kCaTileFma;
    const uint32_t t_beg = (uint32_t)((uint64_t)tiles * sp / splits), t_end = (uint32_t)((uint64_t)tiles * (sp + 1) / splits);
    for (uint32_t i = tid; i < kCaRowsFma * D; i += kCaThreads) {
        const uint32_t r = row0 + i / D, c = i % D, qr = pr.row(r);
        q_s[i] = r >= pr.n ? 0.f
                           : (c < a.q_cols ? a.q[(size_t)qr * a.q_stride + c] : a.q_tail[(size_t)qr * a.tail_stride + c - a.q_cols]);
    }
    float o[kCaRowsFma][J];
#pragma unroll
    for (int r = 0; r < kCaRowsFma; ++r)
#pragma unroll
        for (int j = 0; j < J; ++j) o[r][j] = 0.f;
    float mx = -INFINITY, sum = 0.f;
    const uint32_t pos = a.pos0 + pr.position(row);
    for (uint32_t tile = t_beg; tile < t_end; ++tile) {
        const uint32_t t0 = kr.lo + tile * kCaTileFma;
        __syncthreads();
        for (uint32_t r = warp; r < kCaTileFma; r += kCaWarps) {
            const uint32_t t = t0 + r;
            const T *src = t < kr.hi ? (const T *)a.cache + paged_slot(a.page_table, a.page_tokens, t) * a.slot_cols +
                                           (size_t)pr.part * a.head_cols
                                     : nullptr;
            for (uint32_t c = lane; c < a.head_cols; c += 32) k_s[r * ldk + c] = src ? cache_value(src + c) : 0.f;
        }
        __syncthreads();
        const uint32_t t = t0 + lane;
        float s = -INFINITY;
        if (row < pr.n && t < kr.hi && key_visible(t, pos, a.window)) {
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
        p_s[warp * kCaTileFma + lane] = p;
        if (lane == 0) al_s[warp] = alpha;
        __syncthreads();
#pragma unroll
        for (int r = 0; r < kCaRowsFma; ++r) {
            const float al = al_s[r];
#pragma unroll
            for (int j = 0; j < J; ++j) o[r][j] *= al;
        }
        for (uint32_t k = 0; k < kCaTileFma; ++k) {
            float v[J];
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const uint32_t c = tid + j * kCaThreads;
                v[j] = c < a.val_cols ? k_s[k * ldk + a.val_off + c] : 0.f;
            }
#pragma unroll
            for (int r = 0; r < kCaRowsFma; ++r) {
                const float pr = p_s[r * kCaTileFma + k];
#pragma unroll
                for (int j = 0; j < J; ++j) o[r][j] = fmaf(pr, v[j], o[r][j]);
            }
        }
    }
    if (lane == 0 && row < pr.n) {
        a.ws_ml[((size_t)sp * rows + pr.row(row)) * 2] = mx;
        a.ws_ml[((size_t)sp * rows + pr.row(row)) * 2 + 1] = sum;
    }
#pragma unroll
    for (int r = 0; r < kCaRowsFma; ++r)
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const uint32_t c = tid + j * kCaThreads;
            if (c < a.val_cols && row0 + r < pr.n) a.ws_o[((size_t)sp * rows + pr.row(row0 + r)) * a.val_cols + c] = o[r][j];
        }
    if constexpr (GROUPED) merge_splits(a, pr, splits, row0, kCaRowsFma);
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
// Weighted sum: each warp every eighth group of eight value columns, read as the transposed operand.
// Queries and weights are split into two bf16 parts (about 16 bits), so the only bf16 rounding is the
// cache's. NT: groups of eight value columns per warp.
__host__ __device__ constexpr int ca_steps(int nt) { return nt <= 2 ? 2 : nt / 2 + 1; }  // 16-value steps of a row per warp
constexpr uint32_t kCaLdP = kCaTileMma + 8, kCaLdS = kCaTileMma + 4;

template <int NT, bool GROUPED>
__global__ void __launch_bounds__(kCaThreads, NT <= 2 ? 2 : 1) k_cache_attention_mma(CacheAttn a, uint32_t splits, uint32_t stages) {
    constexpr int NK = ca_steps(NT), JG = NT < 4 ? NT : 4;
    pdl_launch();
    extern __shared__ __align__(16) uint8_t smraw[];
    const PartRows<GROUPED> pr(a);
    const uint32_t D = a.key_cols, ld = a.head_cols + 8, rows = a.m * a.heads;
    __nv_bfloat16 *k_s = reinterpret_cast<__nv_bfloat16 *>(smraw);           // [stages][64][ld]
    float *s_s = reinterpret_cast<float *>(k_s + (size_t)stages * kCaTileMma * ld);  // [8 warps][16][kCaLdS]
    __nv_bfloat16 *p_s = reinterpret_cast<__nv_bfloat16 *>(s_s + kCaWarps * kCaRowsMma * kCaLdS);  // [hi, lo][16][kCaLdP]
    float *al_s = reinterpret_cast<float *>(p_s + 2 * kCaRowsMma * kCaLdP);  // [16]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t row0 = blockIdx.x * kCaRowsMma, sp = blockIdx.y;
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const uint32_t tiles = (kr.hi - kr.lo + kCaTileMma - 1) / kCaTileMma;
    const uint32_t t_beg = (uint32_t)((uint64_t)tiles * sp / splits), t_end = (uint32_t)((uint64_t)tiles * (sp + 1) / splits);
    const uint32_t chunks = a.head_cols / 8;
    pdl_wait();
    auto load_tile = [&](uint32_t tile, uint32_t stage) {
        // lane i < 8 looks the slot of this warp's row i up, for all lanes
        const uint32_t mine = kr.lo + tile * kCaTileMma + warp + (lane & 7) * kCaWarps;
        const uint32_t slot = mine < kr.hi ? (uint32_t)paged_slot(a.page_table, a.page_tokens, mine) : 0xffffffffu;
#pragma unroll
        for (uint32_t i = 0; i < kCaTileMma / kCaWarps; ++i) {
            const uint32_t r = warp + i * kCaWarps, from = __shfl_sync(0xffffffffu, slot, i);
            const bool in = from != 0xffffffffu;
            const __nv_bfloat16 *src = (const __nv_bfloat16 *)a.cache + (in ? (size_t)from * a.slot_cols : 0) + pr.part * a.head_cols;
            __nv_bfloat16 *dst = k_s + ((size_t)stage * kCaTileMma + r) * ld;
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
                const uint32_t r = row0 + g + (j & 1) * 8, c = (warp + i * kCaWarps) * 16 + t4 * 2 + (j >> 1) * 8;
                v[i][j] = make_float2(0.f, 0.f);
                if (r < pr.n && c < D)
                    v[i][j] = *reinterpret_cast<const float2 *>(c < a.q_cols ? a.q + (size_t)pr.row(r) * a.q_stride + c
                                                                             : a.q_tail + (size_t)pr.row(r) * a.tail_stride + (c - a.q_cols));
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
    const uint32_t srow = tid >> 4, stok = (tid & 15) * 4, qrow = row0 + srow, qpos = a.pos0 + pr.position(qrow);
    float mx = -INFINITY, sum = 0.f;
    const uint32_t p_addr = smem_u32(p_s + (lane & 15) * kCaLdP + (lane >> 4) * 8);
    for (uint32_t tile = t_beg; tile < t_end; ++tile) {
        const uint32_t st = stages == 2 ? (tile - t_beg) & 1 : 0;
        if (stages == 2 && tile + 1 < t_end)  // the next tile may still be on its way
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        else
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const __nv_bfloat16 *kt = k_s + (size_t)st * kCaTileMma * ld;
        // ---- partial scores over this warp's steps
        float s[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
        const uint32_t k_addr = smem_u32(kt + ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int i = 0; i < NK; ++i) {
            const uint32_t c = (warp + i * kCaWarps) * 16;
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
        float *sw = s_s + warp * kCaRowsMma * kCaLdS;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            *reinterpret_cast<float2 *>(sw + g * kCaLdS + n * 8 + t4 * 2) = make_float2(s[n][0], s[n][1]);
            *reinterpret_cast<float2 *>(sw + (g + 8) * kCaLdS + n * 8 + t4 * 2) = make_float2(s[n][2], s[n][3]);
        }
        __syncthreads();
        // ---- scores of one row's four tokens, softmax
        float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int w = 0; w < kCaWarps; ++w) {
            const float4 q = *reinterpret_cast<const float4 *>(s_s + (w * kCaRowsMma + srow) * kCaLdS + stok);
            v[0] += q.x;
            v[1] += q.y;
            v[2] += q.z;
            v[3] += q.w;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const uint32_t t = kr.lo + tile * kCaTileMma + stok + j;
            if (qrow >= pr.n || t >= kr.hi || !key_visible(t, qpos, a.window)) v[j] = -INFINITY;
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
        *reinterpret_cast<uint2 *>(p_s + srow * kCaLdP + stok) = *reinterpret_cast<uint2 *>(hi);
        *reinterpret_cast<uint2 *>(p_s + (kCaRowsMma + srow) * kCaLdP + stok) = *reinterpret_cast<uint2 *>(lo);
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
        for (uint32_t k = 0; k < kCaTileMma; k += 32) {
            uint32_t ph[2][4], pl[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                ldsm_x4(ph[i], p_addr + (k + i * 16) * 2);
                ldsm_x4(pl[i], p_addr + kCaRowsMma * kCaLdP * 2 + (k + i * 16) * 2);
            }
            const uint32_t v_addr = smem_u32(kt + (k + lane) * ld + a.val_off);
#pragma unroll
            for (int j0 = 0; j0 < NT; j0 += JG) {  // JG independent accumulators between dependent products
                uint32_t b[JG][4];
#pragma unroll
                for (int j = 0; j < JG; ++j) {  // groups past the last one repeat the first (never stored)
                    const uint32_t n = (warp + (j0 + j) * kCaWarps) * 8;
                    ldsm_x4_t(b[j], v_addr + (n < a.val_cols ? n : 0) * 2);
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
    if ((tid & 15) == 0 && qrow < pr.n) {
        a.ws_ml[((size_t)sp * rows + pr.row(qrow)) * 2] = mx * 0.6931471805599453f;
        a.ws_ml[((size_t)sp * rows + pr.row(qrow)) * 2 + 1] = sum;
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        const uint32_t n = (warp + j * kCaWarps) * 8;
        if (n >= a.val_cols) continue;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t r = row0 + g + i * 8;
            if (r < pr.n)
                *reinterpret_cast<float2 *>(a.ws_o + ((size_t)sp * rows + pr.row(r)) * a.val_cols + n + t4 * 2) =
                    make_float2(o[j][i * 2], o[j][i * 2 + 1]);
        }
    }
    if constexpr (GROUPED) merge_splits(a, pr, splits, row0, kCaRowsMma);
}

namespace {

size_t mma_smem(const CacheAttn &a, uint32_t stages) {
    return (size_t)stages * kCaTileMma * (a.head_cols + 8) * 2 + kCaWarps * kCaRowsMma * kCaLdS * 4 +
           2 * kCaRowsMma * kCaLdP * 2 + kCaRowsMma * 4;
}
// Smallest form (NT) of the tensor-core kernel that takes these rows; 0: none does.
int mma_form(const CacheAttn &a) {
    for (int nt : {1, 2, 4, 8, 16})
        if (a.val_cols <= 64u * nt && a.key_cols <= 128u * ca_steps(nt)) return nt;
    return 0;
}
// Tile stages of the tensor-core form (0: it does not apply).
uint32_t mma_stages(const ctox_ctx *ctx, const CacheAttn &a) {
    if (!a.bf16 || !mma_form(a)) return 0;
    for (uint32_t st = 2; st > 0; --st)
        if (mma_smem(a, st) + 256 <= (size_t)ctx->max_smem_optin) return st;
    return 0;
}
size_t fma_smem(const CacheAttn &a) {
    return ((size_t)kCaRowsFma * a.key_cols + kCaTileFma * (a.head_cols + 1) + kCaRowsFma * kCaTileFma + kCaRowsFma) * 4;
}

template <typename T, int J, bool GROUPED>
ctox_status fma_kernel(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits, uint32_t row_tiles, size_t smem) {
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_cache_attention<T, J, GROUPED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CTOX_CUDA(ctx, launch_pdl(k_cache_attention<T, J, GROUPED>, dim3(row_tiles, splits, a.kv_heads), dim3(kCaThreads), smem, ctx->stream, a, splits));
    return CTOX_OK;
}
template <int NT, bool GROUPED>
ctox_status mma_kernel(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits, uint32_t row_tiles, size_t smem, uint32_t stages) {
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_cache_attention_mma<NT, GROUPED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CTOX_CUDA(ctx, launch_pdl(k_cache_attention_mma<NT, GROUPED>, dim3(row_tiles, splits, a.kv_heads), dim3(kCaThreads), smem, ctx->stream, a,
                              splits, stages));
    return CTOX_OK;
}

// A grouped cache is the one whose splits are merged here (out).
template <typename T, int J>
ctox_status fma_launch(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits, uint32_t row_tiles, size_t smem) {
    return a.out ? fma_kernel<T, J, true>(ctx, a, splits, row_tiles, smem) : fma_kernel<T, J, false>(ctx, a, splits, row_tiles, smem);
}
template <int NT>
ctox_status mma_launch(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits, uint32_t row_tiles, size_t smem, uint32_t stages) {
    return a.out ? mma_kernel<NT, true>(ctx, a, splits, row_tiles, smem, stages)
                 : mma_kernel<NT, false>(ctx, a, splits, row_tiles, smem, stages);
}

}  // namespace

static uint32_t row_tiles_of(const CacheAttn &a, bool mma) {
    const uint32_t rows = a.m * (a.heads / a.kv_heads), per = mma ? kCaRowsMma : kCaRowsFma;
    return (rows + per - 1) / per;
}

uint32_t cache_attn_tiles(const ctox_ctx *ctx, const CacheAttn &a) {
    return row_tiles_of(a, mma_stages(ctx, a) > 0) * a.kv_heads;
}

uint32_t cache_attn_splits(const ctox_ctx *ctx, const CacheAttn &a) {
    const bool mma = mma_stages(ctx, a) > 0;
    const uint32_t tile = mma ? kCaTileMma : kCaTileFma, row_tiles = row_tiles_of(a, mma) * a.kv_heads;
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const uint32_t tiles = (kr.hi - kr.lo + tile - 1) / tile;
    // a CTA waits at several barriers per tile: two of them on an SM where their buffers fit
    const bool two = mma && mma_form(a) <= 2 && 2 * (mma_smem(a, mma_stages(ctx, a)) + 1280) <= (size_t)ctx->max_smem_optin + 1024;
    uint32_t s = (uint32_t)ctx->sm_count * (two ? 2 : 1) / row_tiles;
    // whoever merges the splits reads them all: many only where they shorten a long chain of tiles
    const uint32_t most = tiles >= 256 ? kAttnSplitsDense : kAttnSplitsDense / 2;
    if (s > most) s = most;
    if (s > tiles) s = tiles;
    return s ? s : 1;
}

static ctox_status cache_attention_any(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits) {
    const uint32_t stages = mma_stages(ctx, a), row_tiles = row_tiles_of(a, stages > 0);
    if (stages) {
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
    const uint32_t j = (a.val_cols + kCaThreads - 1) / kCaThreads;
    if (smem + 256 > (size_t)ctx->max_smem_optin || j > 8)
        return fail(ctx, CTOX_MEMORY_BUDGET, "cache attention: rows of %u values (%u of them summed) do not fit shared memory", a.head_cols, a.val_cols);
#define FMA(T)                                                             \
    (j <= 1 ? fma_launch<T, 1>(ctx, a, splits, row_tiles, smem)            \
     : j <= 2 ? fma_launch<T, 2>(ctx, a, splits, row_tiles, smem)          \
     : j <= 4 ? fma_launch<T, 4>(ctx, a, splits, row_tiles, smem)          \
              : fma_launch<T, 8>(ctx, a, splits, row_tiles, smem))
    return a.bf16 ? FMA(__nv_bfloat16) : FMA(float);
#undef FMA
}

ctox_status launch_cache_attention(ctox_ctx *ctx, const CacheAttn &a, uint32_t splits) {
    const KeyRange kr = key_range(a.pos0, a.m, a.window);
    const double keys = kr.hi - kr.lo;
    timing_begin(ctx);
    EX(cache_attention_any(ctx, a, splits));
    timing_end(ctx, KC_STACK_ATTENTION, keys * a.slot_cols * (a.bf16 ? 2 : 4),
               2.0 * keys * a.m * a.heads * (a.key_cols + a.val_cols));
    return CTOX_OK;
}

}  // namespace ctox
