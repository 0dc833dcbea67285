// Matrix memory, long passes: chunks of kMemChunk tokens. With F the sum of the log forget gates since the start
// of a chunk, a_s = i_s - F_s and M_t = m_t - F_t, token s counts e^(a_s - M_t) at token t of the same chunk and
// the state before the chunk e^(m_0 - M_t). Four kernels:
//   gates   the scalars of every token, for a head at a time
//   delta   what each chunk adds to the state, sum_s e^(a_s - M_L) v_s k_s^T (all chunks at once)
//   scan    the state before every chunk, and after the last
//   output  q k^T, weighted and multiplied by the values, plus the state's share; norm and output gate
// The products run on tcgen05.mma. What enters the recurrence beside the projections (the weighted values, the
// state) is an operand in two bf16 parts, about 16 bits; sums are fp32.
#include "matrix_memory.cuh"
#include "umma.cuh"

#include <algorithm>
#include <cmath>

namespace ctox {

constexpr float kLog2e = 1.4426950408889634f;

// Scalars of a pass: rows a, M, e^-m of every head [head][3][tokens], then m_0 and M_L of every chunk.
struct MemScan {
    float *a, *M, *floor, *chunk;  // of one head; chunk [n][2]
};
__host__ __device__ inline MemScan mem_scan(float *base, uint32_t heads, uint32_t chunks, uint32_t head) {
    const size_t P = (size_t)chunks * kMemChunk;
    MemScan s;
    s.a = base + head * 3 * P;
    s.M = s.a + P;
    s.floor = s.M + P;
    s.chunk = base + heads * 3 * P + (size_t)head * chunks * 2;
    return s;
}

// ------------------------------------------------------------------ gates
constexpr int kMgThreads = 256, kMgTokens = 8;  // tokens per thread; sixteen threads hold a chunk
static_assert(kMgTokens * 16 == (int)kMemChunk, "a half warp holds a chunk");

__global__ void __launch_bounds__(kMgThreads) k_memory_gates(MatrixMemory a, const float *__restrict__ gates, uint32_t m,
                                                             uint32_t chunks, float *__restrict__ scan) {
    pdl_launch();
    pdl_wait();
    __shared__ float warp_f[kMgThreads / 32], warp_i[kMgThreads / 32], carry;
    const uint32_t head = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const MemScan out = mem_scan(scan, a.heads, chunks, head);
    const float ib = a.i_bias[head], fb = a.f_bias[head];
    float top = a.top[head];
    for (uint32_t base = 0; base < chunks * kMemChunk; base += kMgThreads * kMgTokens) {
        const uint32_t t0 = base + tid * kMgTokens;
        float i[kMgTokens], f[kMgTokens], F = 0.f, I = -INFINITY;
#pragma unroll
        for (int u = 0; u < kMgTokens; ++u) {
            i[u] = -INFINITY;
            f[u] = 0.f;
            if (t0 + u < m) {
                const float *g = gates + (size_t)(t0 + u) * 2 * a.heads + head;
                i[u] = soft_cap(g[0] + ib, a.gate_cap);
                f[u] = log_sigmoid(soft_cap(g[a.heads] + fb, a.gate_cap));
            }
            I = fmaxf(I + f[u], i[u]);
            F += f[u];
        }
        // m -> max(F + m, I) composes: an inclusive scan of the pairs over the threads
        float Fs = F, Is = I;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fl = __shfl_up_sync(0xffffffffu, Fs, o), Il = __shfl_up_sync(0xffffffffu, Is, o);
            if ((int)lane >= o) {
                Is = fmaxf(Il + Fs, Is);
                Fs += Fl;
            }
        }
        if (lane == 31) {
            warp_f[warp] = Fs;
            warp_i[warp] = Is;
        }
        __syncthreads();
        float m_in = top;  // the running maximum before this warp, then before this thread
        for (uint32_t w = 0; w < warp; ++w) m_in = fmaxf(warp_f[w] + m_in, warp_i[w]);
        const float Fx = __shfl_up_sync(0xffffffffu, Fs, 1), Ix = __shfl_up_sync(0xffffffffu, Is, 1);
        if (lane > 0) m_in = fmaxf(Fx + m_in, Ix);
        const float m0 = __shfl_sync(0xffffffffu, m_in, 0, 16);  // before the chunk
        float Fc = F;                                            // since the start of the chunk
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) {
            const float l = __shfl_up_sync(0xffffffffu, Fc, o, 16);
            if ((int)(lane & 15) >= o) Fc += l;
        }
        Fc = __shfl_up_sync(0xffffffffu, Fc, 1, 16);
        if ((lane & 15) == 0) Fc = 0.f;
        float mt = m_in;
        const bool in = t0 < chunks * kMemChunk;
#pragma unroll
        for (int u = 0; u < kMgTokens; ++u) {
            Fc += f[u];
            mt = fmaxf(f[u] + mt, i[u]);
            if (in) {
                out.a[t0 + u] = i[u] - Fc;
                out.M[t0 + u] = mt - Fc;
                out.floor[t0 + u] = expf(-mt);
            }
        }
        if (in && (lane & 15) == 15) {
            out.chunk[t0 / kMemChunk * 2] = m0;
            out.chunk[t0 / kMemChunk * 2 + 1] = mt - Fc;
        }
        if (tid == kMgThreads - 1) carry = mt;
        __syncthreads();
        top = carry;
        __syncthreads();
    }
    if (tid == 0) a.top[head] = top;
}

// ------------------------------------------------------------------ what a chunk adds
constexpr int kMdThreads = 256;
constexpr uint32_t kMdRows = 128;  // value rows per CTA

__host__ __device__ constexpr uint32_t tmem_width(uint32_t cols) {
    return cols <= 32 ? 32 : cols <= 64 ? 64 : cols <= 128 ? 128 : cols <= 256 ? 256 : 512;
}

// delta[v][d] = sum_s (e^(a_s - M_L) v_s)[v] k_s[d]: both operands are tiles whose rows run along the tokens.
__global__ void __launch_bounds__(kMdThreads) k_memory_delta(const __grid_constant__ CUtensorMap map_k,
                                                             const __grid_constant__ CUtensorMap map_v, MatrixMemory a,
                                                             float *__restrict__ scan, float *__restrict__ delta, uint32_t chunks,
                                                             int32_t *error_word) {
    using namespace umma;
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t bars[2];
    __shared__ uint32_t tmem_slot;
    __shared__ volatile int dead;
    __shared__ float w_s[kMemChunk], norm_s[kMdThreads / 32][256];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t v0 = blockIdx.x * kMdRows, chunk = blockIdx.y, head = blockIdx.z;
    const HeadBox bd = head_box(a.dim_pad);
    const uint32_t base = (smem_addr(raw) + 1023) & ~1023u;
    uint8_t *base_p = raw + (base - smem_addr(raw));
    constexpr uint32_t kBox = kMemChunk * 128;  // bytes of a box of 64 value columns
    const uint32_t lo_off = 2 * kBox, k_off = 4 * kBox, k_box = kMemChunk * bd.width * 2;
    const uint32_t cols = tmem_width(a.dim_pad);
    const uint32_t loaded = smem_addr(bars), done = loaded + 8;
    if (tid == 0) {
        dead = 0;
        bar_init(loaded, 1);
        bar_init(done, 1);
        bar_init_fence();
    }
    if (warp == 0) tmem_alloc(smem_addr(&tmem_slot), cols);
    fence_before();
    __syncthreads();
    fence_after();
    pdl_launch();
    const uint32_t tmem = tmem_slot;
    pdl_wait();
    const int row = (int)(chunk * kMemChunk);
    if (tid == 0) {
        bar_expect(loaded, 2 * kBox + bd.n * k_box);
        for (uint32_t i = 0; i < 2; ++i)
            tma_load(base + i * kBox, &map_v, loaded, (int)(2 * a.heads * a.dim_pad + head * a.vdim_pad + v0 + i * 64), row);
        for (uint32_t i = 0; i < bd.n; ++i)
            tma_load(base + k_off + i * k_box, &map_k, loaded, (int)((a.heads + head) * a.dim_pad + i * bd.width), row);
    }
    const MemScan sc = mem_scan(scan, a.heads, chunks, head);
    if (tid < kMemChunk) w_s[tid] = expf(sc.a[chunk * kMemChunk + tid] - sc.chunk[chunk * 2 + 1]);
    __syncthreads();
    const bool ok = bar_wait(loaded, 0, &dead);
    if (!ok) bar_drain(loaded, 0);
    // the weights into the values, in two parts (a 16-byte piece keeps its place, whatever the swizzle)
#pragma unroll 4
    for (uint32_t u = tid; u < 2 * kBox / 16; u += kMdThreads) {
        const float w = w_s[u * 16 % kBox / 128];
        uint4 *hp = reinterpret_cast<uint4 *>(base_p + u * 16);
        const uint4 in = *hp;
        const uint32_t x[4] = {in.x, in.y, in.z, in.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float p = w * __uint_as_float(x[j] << 16), q = w * __uint_as_float(x[j] & 0xffff0000u);
            const __nv_bfloat162 h = __floats2bfloat162_rn(p, q);
            const __nv_bfloat162 l = __floats2bfloat162_rn(p - __bfloat162float(h.x), q - __bfloat162float(h.y));
            hi[j] = *reinterpret_cast<const uint32_t *>(&h);
            lo[j] = *reinterpret_cast<const uint32_t *>(&l);
        }
        *hp = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4 *>(base_p + lo_off + u * 16) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    fence_before();
    __syncthreads();
    fence_after();
    if (tid == 0) {
        const uint32_t idesc = idesc_bf16_mn(kMdRows, a.dim_pad, true, true);
        for (uint32_t h = 0; h < 2; ++h) {
            const uint64_t da = smem_desc_mn(base + h * lo_off, 128, kBox), db = smem_desc_mn(base + k_off, bd.width * 2, k_box);
#pragma unroll
            for (uint32_t k = 0; k < kMemChunk / 16; ++k)
                mma_f16(tmem, da + k * (16 * 128 / 16), db + k * (16 * bd.width * 2 / 16), idesc, h > 0 || k > 0);
        }
        commit(done);
    }
    float *dst = delta + ((size_t)chunk * a.heads + head) * (a.vdim_pad + kMemRows) * a.dim_pad;
    if (blockIdx.x == 0) {  // the normaliser: the weighted sum of the keys; a warp takes every eighth token
        const uint32_t mask = bd.width / 8 - 1, shift = bd.width == 64 ? 0 : bd.width == 32 ? 1 : 2;
        for (uint32_t d = lane * 8; d < a.dim_pad; d += 256) {
            const uint8_t *box = base_p + k_off + d / bd.width * k_box;
            float n[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
            for (uint32_t t = warp; t < kMemChunk; t += kMdThreads / 32) {
                const uint4 k = *reinterpret_cast<const uint4 *>(box + t * bd.width * 2 + ((d % bd.width / 8) ^ ((t >> shift) & mask)) * 16);
                const uint32_t x[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    n[2 * j] = fmaf(w_s[t], __uint_as_float(x[j] << 16), n[2 * j]);
                    n[2 * j + 1] = fmaf(w_s[t], __uint_as_float(x[j] & 0xffff0000u), n[2 * j + 1]);
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) norm_s[warp][d + j] = n[j];
        }
        __syncthreads();
        for (uint32_t d = tid; d < a.dim_pad; d += kMdThreads)
            dst[(size_t)a.vdim_pad * a.dim_pad + d] = ((norm_s[0][d] + norm_s[1][d]) + (norm_s[2][d] + norm_s[3][d])) +
                                                      ((norm_s[4][d] + norm_s[5][d]) + (norm_s[6][d] + norm_s[7][d]));
    }
    const bool finished = bar_wait(done, 0, &dead);
    if (!finished) bar_drain(done, 0);
    __syncthreads();  // the operands' buffers are free
    fence_after();
    {   // a row of the product goes to its own padded line (two warps share the columns), and from there as one copy
        const uint32_t quarter = warp & 3, row_bytes = a.dim_pad * 4 + 16, line = (quarter * 32 + lane) * row_bytes;
        for (uint32_t d = (warp >> 2) * 16; d < a.dim_pad; d += 32) {
            float x[16];
            tmem_ld16(tmem + d + ((quarter * 32) << 16), x);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 4; ++j)
                *reinterpret_cast<float4 *>(base_p + line + d * 4 + j * 16) = make_float4(x[4 * j], x[4 * j + 1], x[4 * j + 2], x[4 * j + 3]);
        }
        fence_before();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        __syncthreads();
        if (tid < kMdRows && v0 + tid < a.vdim_pad) {
            asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst + (size_t)(v0 + tid) * a.dim_pad),
                         "r"(base + tid * row_bytes), "r"(a.dim_pad * 4)
                         : "memory");
            asm volatile("cp.async.bulk.commit_group;\n\tcp.async.bulk.wait_group 0;" ::: "memory");
        }
    }
    __syncthreads();
    if (warp == 0) {
        fence_after();
        tmem_free(tmem, cols);
    }
    if (tid == 0 && dead) *error_word = DEV_ERR_WAIT_TIMEOUT;
}

// ------------------------------------------------------------------ the state before every chunk
constexpr int kMcThreads = 256, kMcBatch = 4;

__global__ void __launch_bounds__(kMcThreads) k_memory_scan(MatrixMemory a, float *__restrict__ scan, const float *__restrict__ delta,
                                                            __nv_bfloat16 *__restrict__ start, uint32_t chunks) {
    pdl_launch();
    const uint32_t head = blockIdx.y, n = (a.vdim_pad + 1) * a.dim_pad / 4, i = blockIdx.x * kMcThreads + threadIdx.x;
    const size_t block = (size_t)(a.vdim_pad + kMemRows) * a.dim_pad, step = block * a.heads;
    pdl_wait();
    if (i >= n) return;
    const MemScan sc = mem_scan(scan, a.heads, chunks, head);
    float4 *state = reinterpret_cast<float4 *>(a.state + head * block) + i;
    const float4 *add = reinterpret_cast<const float4 *>(delta + head * block) + i;
    uint2 *hi = reinterpret_cast<uint2 *>(start + head * block) + i, *lo = reinterpret_cast<uint2 *>(start + chunks * step + head * block) + i;
    float4 s = *state;
    for (uint32_t c0 = 0; c0 < chunks; c0 += kMcBatch) {
        float4 d[kMcBatch];
        float keep[kMcBatch];
#pragma unroll
        for (int j = 0; j < kMcBatch; ++j)
            if (c0 + j < chunks) {
                d[j] = add[(size_t)(c0 + j) * step / 4];
                keep[j] = expf(sc.chunk[(c0 + j) * 2] - sc.chunk[(c0 + j) * 2 + 1]);
            }
#pragma unroll
        for (int j = 0; j < kMcBatch; ++j)
            if (c0 + j < chunks) {
                const __nv_bfloat162 h0 = __floats2bfloat162_rn(s.x, s.y), h1 = __floats2bfloat162_rn(s.z, s.w);
                const __nv_bfloat162 l0 = __floats2bfloat162_rn(s.x - __bfloat162float(h0.x), s.y - __bfloat162float(h0.y)),
                                     l1 = __floats2bfloat162_rn(s.z - __bfloat162float(h1.x), s.w - __bfloat162float(h1.y));
                hi[(size_t)(c0 + j) * step / 4] = make_uint2(*reinterpret_cast<const uint32_t *>(&h0), *reinterpret_cast<const uint32_t *>(&h1));
                lo[(size_t)(c0 + j) * step / 4] = make_uint2(*reinterpret_cast<const uint32_t *>(&l0), *reinterpret_cast<const uint32_t *>(&l1));
                s.x = fmaf(keep[j], s.x, d[j].x);
                s.y = fmaf(keep[j], s.y, d[j].y);
                s.z = fmaf(keep[j], s.z, d[j].z);
                s.w = fmaf(keep[j], s.w, d[j].w);
            }
    }
    *state = s;
}

// ------------------------------------------------------------------ outputs
constexpr int kMoThreads = 320;      // warp 0: TMA, warp 1: MMA, warps 2-9: two threads per token, half of the columns each
constexpr uint32_t kMoSlice = 64;    // value columns at once
constexpr uint32_t kMoBatch = 4;     // rows whose loads are in flight together

// Tensor memory: scores, two buffers each of the state's share and of the chunk's own, n . q, the weighted scores.
constexpr uint32_t kMoState = 128, kMoOwn = 256, kMoNorm = 384, kMoWeights = 416, kMoCols = 512;

// One whole 32-byte sector.
__device__ __forceinline__ void store8(float *p, const float *v) {
    asm volatile("st.global.v8.f32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"l"(p), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]),
                 "f"(v[5]), "f"(v[6]), "f"(v[7])
                 : "memory");
}

__global__ void __launch_bounds__(kMoThreads) k_memory_output(const __grid_constant__ CUtensorMap map_qk,
                                                              const __grid_constant__ CUtensorMap map_v,
                                                              const __grid_constant__ CUtensorMap map_s,
                                                              const __grid_constant__ CUtensorMap map_n, MatrixMemory a, MemoryLong w,
                                                              uint32_t m, uint32_t chunks, int32_t *error_word) {
    using namespace umma;
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t bars[14];
    __shared__ uint32_t tmem_slot;
    __shared__ volatile int dead;
    __shared__ float red_s[3][kMemChunk];  // a, then sums of squares in the first two; n . q of the chunk's own in the last two
    float *a_s = red_s[0];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t chunk = blockIdx.x % chunks, head = blockIdx.x / chunks;
    const HeadBox bd = head_box(a.dim_pad);
    // Two stages of a slice: state [hi | lo] and values. The second one's state takes the place of the keys and its values
    // that of the normaliser, once those have been used.
    const uint32_t qk_bytes = kMemChunk * a.dim_pad * 2, s_bytes = kMoSlice * a.dim_pad * 2, v_bytes = kMemChunk * kMoSlice * 2,
                   n_bytes = kMemRows * a.dim_pad * 2;
    static_assert(2 * kMoSlice == kMemChunk && 2 * kMemRows * 256 <= kMemChunk * kMoSlice, "what the second stage replaces");
    const uint32_t base = (smem_addr(raw) + 1023) & ~1023u;
    const uint32_t q_s = base, k_s = q_s + qk_bytes, v_s = k_s + 2 * qk_bytes, n_s = v_s + v_bytes;
    auto state_of = [&](uint32_t s) { return s ? k_s : k_s + qk_bytes; };
    const uint32_t b0 = smem_addr(bars), qk_full = b0, n_full = b0 + 8, s_full = b0 + 16, p_full = b0 + 24, nq_full = b0 + 32,
                   st_full = b0 + 40, st_empty = b0 + 56, o_full = b0 + 72, o_empty = b0 + 88, drained = b0 + 104;
    if (tid == 0) {
        dead = 0;
        for (uint32_t bar : {qk_full, n_full, s_full, nq_full, drained}) bar_init(bar, 1);
        bar_init(p_full, 8);
        for (uint32_t i = 0; i < 2; ++i) {
            bar_init(st_full + i * 8, 1);
            bar_init(st_empty + i * 8, 1);
            bar_init(o_full + i * 8, 1);
            bar_init(o_empty + i * 8, 8);
        }
        bar_init_fence();
    }
    if (warp == 1) tmem_alloc(smem_addr(&tmem_slot), kMoCols);
    fence_before();
    __syncthreads();
    fence_after();
    pdl_launch();
    const uint32_t tmem = tmem_slot, slices = (a.vdim_pad + kMoSlice - 1) / kMoSlice;
    const uint32_t state_rows = a.vdim_pad + kMemRows, row0 = (chunk * a.heads + head) * state_rows, lo_rows = chunks * a.heads * state_rows;
    pdl_wait();
    if (warp == 0) {
        if (lane == 0) {
            const int tok = (int)(chunk * kMemChunk);
            bar_expect(qk_full, 2 * qk_bytes);
            for (uint32_t i = 0; i < bd.n; ++i) {
                tma_load(q_s + i * kMemChunk * bd.width * 2, &map_qk, qk_full, (int)(head * a.dim_pad + i * bd.width), tok);
                tma_load(k_s + i * kMemChunk * bd.width * 2, &map_qk, qk_full, (int)((a.heads + head) * a.dim_pad + i * bd.width), tok);
            }
            bar_expect(n_full, 2 * n_bytes);
            for (uint32_t h = 0; h < 2; ++h)
                for (uint32_t i = 0; i < bd.n; ++i)
                    tma_load(n_s + h * n_bytes + i * kMemRows * bd.width * 2, &map_n, n_full, (int)(i * bd.width),
                             (int)(row0 + a.vdim_pad + h * lo_rows));
            uint32_t issued = 0;
            bool ok = true;
            for (uint32_t j = 0; j < slices; ++j) {
                const uint32_t s = j & 1, dst = state_of(s), bar = st_full + s * 8;
                if (j == 1 && !(ok = bar_wait(nq_full, 0, &dead))) break;
                if (j >= 2 && !(ok = bar_wait(st_empty + s * 8, ((j >> 1) - 1) & 1, &dead))) break;
                bar_expect(bar, 2 * s_bytes + v_bytes);
                for (uint32_t h = 0; h < 2; ++h)
                    for (uint32_t i = 0; i < bd.n; ++i)
                        tma_load(dst + h * s_bytes + i * kMoSlice * bd.width * 2, &map_s, bar, (int)(i * bd.width),
                                 (int)(row0 + j * kMoSlice + h * lo_rows));
                tma_load(v_s + s * v_bytes, &map_v, bar, (int)(2 * a.heads * a.dim_pad + head * a.vdim_pad + j * kMoSlice), tok);
                ++issued;
            }
            if (!ok) {  // leave no copy in flight behind
                bar_drain(qk_full, 0);
                bar_drain(n_full, 0);
                for (uint32_t s = 0; s < 2 && s < issued; ++s) bar_drain(st_full + s * 8, ((issued - 1 - s) >> 1) & 1);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // D [128][n] (+)= Q B^T over the head's dimensions, B of box_rows rows per box
            auto over_dims = [&](uint32_t d, uint32_t b, uint32_t box_rows, uint32_t n, bool acc) {
                const uint32_t idesc = idesc_bf16(kMemChunk, n), rb = bd.width * 2;
                for (uint32_t i = 0; i < bd.n; ++i)
                    for (uint32_t k = 0; k < bd.width; k += 16, acc = true)
                        mma_f16(d, smem_desc(q_s + i * kMemChunk * rb + k * 2, rb), smem_desc(b + i * box_rows * rb + k * 2, rb), idesc, acc);
            };
            bool ok = bar_wait(qk_full, 0, &dead);
            if (ok) {
                fence_after();
                over_dims(tmem, k_s, kMemChunk, kMemChunk, false);
                commit(s_full);
                ok = bar_wait(n_full, 0, &dead);
            }
            if (ok) {
                fence_after();
                over_dims(tmem + kMoNorm, n_s, kMemRows, kMemRows, false);
                over_dims(tmem + kMoNorm, n_s + n_bytes, kMemRows, kMemRows, true);
                commit(nq_full);
            }
            const uint32_t idesc_v = idesc_bf16_mn(kMemChunk, kMoSlice, false, true);
            for (uint32_t j = 0; j < slices && ok; ++j) {
                const uint32_t o = j & 1, src = state_of(o);  // the slice's stage, and its buffers in tensor memory
                if (!(ok = bar_wait(st_full + o * 8, (j >> 1) & 1, &dead))) break;
                if (j >= 2 && !(ok = bar_wait(o_empty + o * 8, ((j >> 1) - 1) & 1, &dead))) break;
                fence_after();
                over_dims(tmem + kMoState + o * kMoSlice, src, kMoSlice, kMoSlice, false);
                over_dims(tmem + kMoState + o * kMoSlice, src + s_bytes, kMoSlice, kMoSlice, true);
                if (j == 0) {
                    if (!(ok = bar_wait(p_full, 0, &dead))) break;
                    fence_after();
                }
                const uint64_t dv = smem_desc_mn(v_s + o * v_bytes, 128, v_bytes);
#pragma unroll
                for (uint32_t k = 0; k < kMemChunk / 16; ++k)
                    mma_f16_ts(tmem + kMoOwn + o * kMoSlice, tmem + kMoWeights + k * 8, dv + k * (16 * 128 / 16), idesc_v, k > 0);
                commit(st_empty + o * 8);
                commit(o_full + o * 8);
            }
            if (!ok) {
                commit(drained);
                bar_drain(drained, 0);
            }
        }
    } else {
        const uint32_t quarter = warp & 3, part = (warp - 2) >> 2, row = quarter * 32 + lane, lanes = (quarter * 32) << 16,
                       tok = chunk * kMemChunk + row;
        const MemScan sc = mem_scan(w.scan, a.heads, chunks, head);
        if (part == 0) a_s[row] = sc.a[tok] * kLog2e;
        const float M = sc.M[tok], Ml = M * kLog2e, floor = sc.floor[tok];
        const float scale = 1.0f / sqrtf((float)a.dim), from_state = expf(sc.chunk[chunk * 2] - M) * scale;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        // `ok` may differ between warps: the barriers below are passed by all of them
        bool ok = __all_sync(0xffffffffu, bar_wait(s_full, 0, &dead));
        if (ok) {
            float nq = 0.f;
            fence_after();
#pragma unroll 1
            for (uint32_t b = part * 2; b < part * 2 + 2; ++b) {
                float s[32];
                tmem_ld32(tmem + b * 32 + lanes, s);
                tmem_ld_wait();
                float p[16];
#pragma unroll
                for (uint32_t j = 0; j < 32; j += 2) {
                    const uint32_t k = b * 32 + j;
                    const float x = k <= row ? s[j] * scale * ex2(a_s[k] - Ml) : 0.f;
                    const float y = k + 1 <= row ? s[j + 1] * scale * ex2(a_s[k + 1] - Ml) : 0.f;
                    nq += x + y;
                    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
                    p[j / 2] = *reinterpret_cast<const float *>(&h);
                }
                tmem_st16(tmem + kMoWeights + b * 16 + lanes, p);
            }
            red_s[1 + part][row] = nq;
            tmem_st_wait();
            fence_before();
            __syncwarp();
            if (lane == 0) bar_arrive(p_full);
            ok = __all_sync(0xffffffffu, bar_wait(nq_full, 0, &dead));
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        float inv = 0.f, sq = 0.f;
        if (ok) {
            fence_after();
            float n[16];
            tmem_ld16(tmem + kMoNorm + lanes, n);
            tmem_ld_wait();
            const float nq = fmaf(from_state, n[0], red_s[1][row] + red_s[2][row]);
            inv = 1.0f / (fmaxf(fabsf(nq), floor) + 1e-6f);
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        float *raw_row = w.raw + ((size_t)tok * a.heads + head) * a.vdim_pad;
        for (uint32_t j = 0; j < slices && ok; ++j) {
            const uint32_t o = j & 1, c = part * 32, v = j * kMoSlice + c;  // vdim_pad is a multiple of 16
            if (!(ok = __all_sync(0xffffffffu, bar_wait(o_full + o * 8, (j >> 1) & 1, &dead)))) break;
            fence_after();
            float x[32], y[32];
            tmem_ld32(tmem + kMoState + o * kMoSlice + c + lanes, x);
            tmem_ld32(tmem + kMoOwn + o * kMoSlice + c + lanes, y);
            tmem_ld_wait();
            fence_before();
            __syncwarp();
            if (lane == 0) bar_arrive(o_empty + o * 8);
#pragma unroll
            for (int i = 0; i < 32; ++i) x[i] = fmaf(from_state, x[i], y[i]) * inv;
#pragma unroll
            for (int i = 0; i < 32; i += 8)
                if (v + i < a.vdim_pad && tok < m) {
#pragma unroll
                    for (int e = 0; e < 8; e += 2) sq += x[i + e] * x[i + e] + x[i + e + 1] * x[i + e + 1];
                    store8(raw_row + v + i, x + i);
                }
        }
        red_s[part][row] = sq;
        __threadfence_block();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (ok) {  // norm and output gate: a warp goes through sixteen rows, a lane holds eight values
            const uint32_t r0 = (warp - 2) * 16, t0 = chunk * kMemChunk + r0, n = t0 < m ? min(16u, m - t0) : 0;
            const size_t ld = (size_t)a.heads * a.vdim_pad;
            for (uint32_t v = lane * 8; v < a.vdim_pad; v += 256) {
                float nw[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) nw[i] = v + i < a.vdim ? a.norm_w[head * a.vdim + v + i] : 0.f;
                const float *rp = w.raw + t0 * ld + head * a.vdim_pad + v;
                const __nv_bfloat16 *gp = w.fan + (size_t)t0 * w.fan_ld + a.heads * (2 * a.dim_pad + a.vdim_pad) + head * a.vdim_pad + v;
                __nv_bfloat16 *op = w.out + t0 * ld + head * a.vdim_pad + v;
                for (uint32_t k0 = 0; k0 < n; k0 += kMoBatch) {
                    float x[kMoBatch][8];
                    uint4 g[kMoBatch];
#pragma unroll
                    for (uint32_t k = 0; k < kMoBatch; ++k)
                        if (k0 + k < n) {
                            *reinterpret_cast<float4 *>(x[k]) = *reinterpret_cast<const float4 *>(rp + (k0 + k) * ld);
                            *reinterpret_cast<float4 *>(x[k] + 4) = *reinterpret_cast<const float4 *>(rp + (k0 + k) * ld + 4);
                            g[k] = *reinterpret_cast<const uint4 *>(gp + (size_t)(k0 + k) * w.fan_ld);
                        }
#pragma unroll
                    for (uint32_t k = 0; k < kMoBatch; ++k)
                        if (k0 + k < n) {
                            const uint32_t gw[4] = {g[k].x, g[k].y, g[k].z, g[k].w};
                            const float r = 1.0f / sqrtf((red_s[0][r0 + k0 + k] + red_s[1][r0 + k0 + k]) / (float)a.vdim + a.eps);
                            __nv_bfloat162 h[4];
#pragma unroll
                            for (int i = 0; i < 4; ++i) {
                                const float g0 = __uint_as_float(gw[i] << 16), g1 = __uint_as_float(gw[i] & 0xffff0000u);
                                h[i] = __floats2bfloat162_rn(__fdividef(x[k][2 * i] * r * nw[2 * i], 1.0f + __expf(-g0)),
                                                             __fdividef(x[k][2 * i + 1] * r * nw[2 * i + 1], 1.0f + __expf(-g1)));
                            }
                            *reinterpret_cast<uint4 *>(op + (k0 + k) * ld) = *reinterpret_cast<const uint4 *>(h);
                        }
                }
            }
        }
    }
    __syncwarp();
    __syncthreads();
    if (warp == 1) {
        fence_after();
        tmem_free(tmem, kMoCols);
    }
    if (tid == 0 && dead) *error_word = DEV_ERR_WAIT_TIMEOUT;
}

namespace {

size_t output_smem(const MatrixMemory &a) { return 1024 + 3 * (size_t)kMemChunk * a.dim_pad * 2 + 2 * (size_t)kMemChunk * kMoSlice * 2; }
size_t delta_smem(const MatrixMemory &a) {
    return 1024 + std::max(4 * (size_t)kMemChunk * 128 + (size_t)kMemChunk * a.dim_pad * 2, (size_t)kMdRows * (a.dim_pad * 4 + 16));
}

}  // namespace

MemoryLongSizes memory_long_sizes(const MatrixMemory &a, uint32_t pass_tokens) {
    const uint64_t chunks = (pass_tokens + kMemChunk - 1) / kMemChunk, block = memory_rows(a) * a.dim_pad;
    return MemoryLongSizes{chunks * a.heads * (3 * kMemChunk + 2), chunks * a.heads * block, 2 * chunks * a.heads * block,
                           (uint64_t)pass_tokens * a.heads * a.vdim_pad};
}

bool memory_long_fits(const ctox_ctx *ctx, const MatrixMemory &a) {
    return a.dim_pad <= 256 && std::max(output_smem(a), delta_smem(a) + 4096) + 2048 <= (size_t)ctx->max_smem_optin;
}

ctox_status launch_matrix_memory_long(ctox_ctx *ctx, const MatrixMemory &a, const MemoryLong &w, uint32_t m) {
    if (!memory_long_fits(ctx, a)) return fail(ctx, CTOX_SHAPE, "matrix memory: %u dimensions per head in a long pass", a.dim);
    const uint32_t chunks = (m + kMemChunk - 1) / kMemChunk;
    const HeadBox bd = head_box(a.dim_pad);
    const uint64_t fan_cols = 2ull * a.heads * (a.dim_pad + a.vdim_pad), rows = memory_rows(a);
    CUtensorMap qk, v, s, n;
    EX(tensor_map_bf16(ctx, &qk, w.fan, m, fan_cols, w.fan_ld, kMemChunk, bd.width));
    EX(tensor_map_bf16(ctx, &v, w.fan, m, fan_cols, w.fan_ld, kMemChunk, 64));
    EX(tensor_map_bf16(ctx, &s, w.start, 2ull * chunks * a.heads * rows, a.dim_pad, a.dim_pad, kMoSlice, bd.width));
    EX(tensor_map_bf16(ctx, &n, w.start, 2ull * chunks * a.heads * rows, a.dim_pad, a.dim_pad, kMemRows, bd.width));
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_memory_delta, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)delta_smem(a)));
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_memory_output, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)output_smem(a)));
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_memory_gates, dim3(a.heads), dim3(kMgThreads), 0, ctx->stream, a, w.gates, m, chunks, w.scan));
    CTOX_CUDA(ctx, launch_pdl(k_memory_delta, dim3((a.vdim_pad + kMdRows - 1) / kMdRows, chunks, a.heads), dim3(kMdThreads),
                              delta_smem(a), ctx->stream, qk, v, a, w.scan, w.delta, chunks, ctx->dev_error));
    const uint32_t items = (a.vdim_pad + 1) * a.dim_pad / 4;
    CTOX_CUDA(ctx, launch_pdl(k_memory_scan, dim3((items + kMcThreads - 1) / kMcThreads, a.heads), dim3(kMcThreads), 0, ctx->stream, a,
                              w.scan, (const float *)w.delta, w.start, chunks));
    CTOX_CUDA(ctx, launch_pdl(k_memory_output, dim3(chunks * a.heads), dim3(kMoThreads), output_smem(a), ctx->stream, qk, v, s, n,
                              a, w, m, chunks, ctx->dev_error));
    // algorithmic work: projections in, result out, the state once each way; per token the chunk's triangle and the state's share
    timing_end(ctx, KC_MEMORY_PREFILL, m * (fan_cols * 2.0 + a.heads * a.vdim_pad * 2.0) + 8.0 * a.heads * a.vdim * a.dim,
               2.0 * m * a.heads * ((a.dim + a.vdim) * (kMemChunk / 2.0) + 2.0 * a.dim * a.vdim));
    return CTOX_OK;
}

}  // namespace ctox
