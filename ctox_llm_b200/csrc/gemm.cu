// Persistent tensor-core product for long passes: one CTA per SM, 128 x BN tiles, operands staged by TMA
// (one thread), multiplied by tcgen05.mma (one thread), accumulators double-buffered in tensor memory so
// that four epilogue warps drain a tile while the next one is computed.
#include "gemm.cuh"
#include "umma.cuh"

namespace ctox {

constexpr int kGmThreads = 192;  // warp 0: TMA, warp 1: MMA, warps 2-5: epilogue
constexpr uint32_t kGmM = 128, kGmK = 64, kGmStageMax = 8;

ctox_status tensor_map_bf16(ctox_ctx *ctx, CUtensorMap *map, const void *base, uint64_t rows, uint64_t cols, uint64_t ld,
                            uint32_t box_rows, uint32_t box_cols) {
    using Encode = CUresult (*)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static Encode encode = nullptr;
    if (!encode) {
        void *fn = nullptr;
        cudaDriverEntryPointQueryResult q;
        CTOX_CUDA(ctx, cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &fn, 12000, cudaEnableDefault, &q));
        if (!fn || q != cudaDriverEntryPointSuccess)
            return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "cuTensorMapEncodeTiled is not available");
        encode = (Encode)fn;
    }
    const cuuint64_t dims[2] = {cols, rows}, strides[1] = {ld * 2};
    const cuuint32_t box[2] = {box_cols, box_rows}, step[2] = {1, 1};
    const CUtensorMapSwizzle sw = box_cols * 2 == 128  ? CU_TENSOR_MAP_SWIZZLE_128B
                                  : box_cols * 2 == 64 ? CU_TENSOR_MAP_SWIZZLE_64B
                                                       : CU_TENSOR_MAP_SWIZZLE_32B;
    const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, step,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, sw, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS)
        return fail(ctx, CTOX_SHAPE, "tensor map of %llu x %llu (ld %llu): error %d", (unsigned long long)rows,
                    (unsigned long long)cols, (unsigned long long)ld, (int)r);
    return CTOX_OK;
}

struct GemmPages {  // cache rows behind an operand (table null: rows as they are)
    const uint32_t *table;
    uint32_t page_tokens, row0;
};
__device__ __forceinline__ int operand_row(const GemmPages &p, uint32_t row) {
    if (!p.table) return (int)row;
    const uint32_t pos = p.row0 + row;
    return (int)(p.table[pos / p.page_tokens] * p.page_tokens + pos % p.page_tokens);
}

// 32 columns n0 .. n0 + 32 of one output row.
__device__ __forceinline__ void gemm_store(const GemmOut &o, float *v, uint32_t m, uint32_t n0, uint32_t N) {
    if (o.bias) {
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (n0 + j < N) v[j] += __ldg(o.bias + n0 + j);
    }
    if (o.kind == OUT_CLAMPED_GLU) {
        __nv_bfloat16 *d = (__nv_bfloat16 *)o.d + (size_t)m * o.ld + n0 / 2;
        __nv_bfloat162 h[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            h[j] = __floats2bfloat162_rn(clamped_glu(v[4 * j], v[4 * j + 1], o.cap, o.slope),
                                         clamped_glu(v[4 * j + 2], v[4 * j + 3], o.cap, o.slope));
        if (n0 + 32 <= N && o.ld % 8 == 0) {
            *reinterpret_cast<uint4 *>(d) = *reinterpret_cast<uint4 *>(h);
            *reinterpret_cast<uint4 *>(d + 8) = *reinterpret_cast<uint4 *>(h + 4);
        } else {
#pragma unroll
            for (int j = 0; j < 16; ++j)
                if (n0 + 2 * j < N) d[j] = j & 1 ? h[j / 2].y : h[j / 2].x;
        }
        return;
    }
    if (o.kind == OUT_RELU2) {
#pragma unroll
        for (int j = 0; j < 32; ++j) v[j] = v[j] > 0.f ? v[j] * v[j] : 0.f;
    } else if (o.kind == OUT_SOFTCAP) {
#pragma unroll
        for (int j = 0; j < 32; ++j) v[j] = o.cap * tanhf(v[j] / o.cap);
    } else if (o.kind == OUT_ROPE) {
        uint32_t w = n0 % o.head_width;  // heads are a multiple of 16 wide: w is even, a pair never straddles two
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
            if (w >= o.rope0 && w < o.rope0 + o.rope_dims) {
                const float2 cs = o.table[(size_t)m * (o.rope_dims / 2) + ((w - o.rope0) >> 1)];
                const float a = v[j] * cs.x - v[j + 1] * cs.y, b = v[j + 1] * cs.x + v[j] * cs.y;
                v[j] = a;
                v[j + 1] = b;
            }
            w += 2;
            if (w >= o.head_width) w -= o.head_width;
        }
    }
    const bool full = n0 + 32 <= N;
    if (o.split && n0 >= o.split) {
        float *d = o.d2 + (size_t)m * o.ld2 + (n0 - o.split);
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (n0 + j < N) d[j] = v[j];
    } else if (o.bf16) {
        __nv_bfloat16 *d = (__nv_bfloat16 *)o.d + (size_t)m * o.ld + n0;
        if (full && o.ld % 8 == 0) {
#pragma unroll
            for (int j = 0; j < 32; j += 8) {
                __nv_bfloat162 h[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[j + 2 * i], v[j + 2 * i + 1]);
                *reinterpret_cast<uint4 *>(d + j) = *reinterpret_cast<uint4 *>(h);
            }
        } else {
#pragma unroll
            for (int j = 0; j < 32; ++j)
                if (n0 + j < N) d[j] = __float2bfloat16_rn(v[j]);
        }
    } else {
        float *d = (float *)o.d + (size_t)m * o.ld + n0;
        if (full && o.ld % 4 == 0) {
#pragma unroll
            for (int j = 0; j < 32; j += 4) *reinterpret_cast<float4 *>(d + j) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
        } else {
#pragma unroll
            for (int j = 0; j < 32; ++j)
                if (n0 + j < N) d[j] = v[j];
        }
    }
}

template <uint32_t BN>
__global__ void __launch_bounds__(kGmThreads, 1)
    k_gemm(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b, GemmPages pa, GemmPages pb,
           uint32_t M, uint32_t N, uint32_t K, uint32_t stages, GemmOut out, int32_t *error_word) {
    using namespace umma;
    constexpr uint32_t kABytes = kGmM * kGmK * 2, kBBytes = BN * kGmK * 2, kBBox = BN < 128 ? BN : 128;
    constexpr uint32_t kCols = 2 * BN < 32 ? 32 : 2 * BN;
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t bars[2 * kGmStageMax + 5];
    __shared__ uint32_t tmem_slot;
    __shared__ volatile int dead;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t base = (smem_addr(raw) + 1023) & ~1023u;
    const uint32_t full = smem_addr(bars), empty = full + kGmStageMax * 8, acc_full = empty + kGmStageMax * 8,
                   acc_empty = acc_full + 16, drained = acc_empty + 16;
    if (tid == 0) {
        dead = 0;
        for (uint32_t i = 0; i < stages; ++i) {
            bar_init(full + i * 8, 1);
            bar_init(empty + i * 8, 1);
        }
        for (uint32_t i = 0; i < 2; ++i) {
            bar_init(acc_full + i * 8, 1);
            bar_init(acc_empty + i * 8, 4);
        }
        bar_init(drained, 1);
        bar_init_fence();
        tma_prefetch_map(&map_a);
        tma_prefetch_map(&map_b);
    }
    if (warp == 1) tmem_alloc(smem_addr(&tmem_slot), kCols);
    fence_before();
    __syncthreads();
    fence_after();
    pdl_launch();  // a later kernel's allocation must not come before this one's (see umma.cuh)
    const uint32_t tmem = tmem_slot;
    const uint32_t tiles_m = (M + kGmM - 1) / kGmM, tiles_n = (N + BN - 1) / BN, tiles = tiles_m * tiles_n;
    const uint32_t ksteps = (K + kGmK - 1) / kGmK;
    pdl_wait();
    if (warp == 0) {
        if (lane == 0) {
            uint32_t issued = 0;
            bool ok = true;
            for (uint32_t t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const uint32_t m0 = t % tiles_m * kGmM, n0 = t / tiles_m * BN;
                const int ra = operand_row(pa, m0);
                int rb[(BN + 127) / 128];
#pragma unroll
                for (uint32_t i = 0; i < (BN + 127) / 128; ++i) rb[i] = n0 + i * 128 < N ? operand_row(pb, n0 + i * 128) : (int)(n0 + i * 128);
                for (uint32_t k = 0; k < ksteps; ++k, ++issued) {
                    const uint32_t s = issued % stages, round = issued / stages;
                    if (round > 0 && !(ok = bar_wait(empty + s * 8, (round - 1) & 1, &dead))) break;
                    const uint32_t bar = full + s * 8, dst = base + s * (kABytes + kBBytes);
                    bar_expect(bar, kABytes + kBBytes);
                    tma_load(dst, &map_a, bar, (int)(k * kGmK), ra);
#pragma unroll
                    for (uint32_t i = 0; i < (BN + 127) / 128; ++i)
                        tma_load(dst + kABytes + i * kBBox * kGmK * 2, &map_b, bar, (int)(k * kGmK), rb[i]);
                }
            }
            if (!ok) {  // leave no copy in flight behind
                for (uint32_t s = 0; s < stages && s < issued; ++s) bar_drain(full + s * 8, ((issued - 1 - s) / stages) & 1);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t used = 0, n_tile = 0;
            bool ok = true;
            const uint32_t idesc = idesc_bf16(kGmM, BN);
            for (uint32_t t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++n_tile) {
                const uint32_t acc = n_tile & 1, d = tmem + acc * BN;
                if (n_tile >= 2 && !(ok = bar_wait(acc_empty + acc * 8, ((n_tile >> 1) - 1) & 1, &dead))) break;
                fence_after();
                for (uint32_t k = 0; k < ksteps; ++k, ++used) {
                    const uint32_t s = used % stages;
                    if (!(ok = bar_wait(full + s * 8, (used / stages) & 1, &dead))) break;
                    fence_after();
                    const uint32_t src = base + s * (kABytes + kBBytes);
                    const uint64_t da = smem_desc(src, 128), db = smem_desc(src + kABytes, 128);
#pragma unroll
                    for (uint32_t i = 0; i < kGmK / 16; ++i) mma_f16(d, da + i * 2, db + i * 2, idesc, k > 0 || i > 0);
                    commit(empty + s * 8);
                }
                if (ok) commit(acc_full + acc * 8);
            }
            if (!ok) {
                commit(drained);
                bar_drain(drained, 0);
            }
        }
    } else {
        const uint32_t quarter = warp & 3;  // the lanes of tensor memory this warp may read
        uint32_t n_tile = 0;
        for (uint32_t t = blockIdx.x; t < tiles; t += gridDim.x, ++n_tile) {
            const uint32_t acc = n_tile & 1, m = t % tiles_m * kGmM + quarter * 32 + lane, n0 = t / tiles_m * BN;
            if (!__all_sync(0xffffffffu, bar_wait(acc_full + acc * 8, (n_tile >> 1) & 1, &dead))) break;
            fence_after();
            const uint32_t src = tmem + acc * BN + ((quarter * 32) << 16);
#pragma unroll 1
            for (uint32_t c = 0; c < BN; c += 32) {
                float v[32];
                tmem_ld32(src + c, v);
                tmem_ld_wait();
                if (m < M && n0 + c < N) gemm_store(out, v, m, n0 + c, N);
            }
            fence_before();
            __syncwarp();
            if (lane == 0) bar_arrive(acc_empty + acc * 8);
        }
    }
    __syncwarp();
    __syncthreads();
    if (warp == 1) {
        fence_after();
        tmem_free(tmem, kCols);
    }
    if (tid == 0 && dead) *error_word = DEV_ERR_WAIT_TIMEOUT;
}

namespace {

template <uint32_t BN>
ctox_status gemm_launch(ctox_ctx *ctx, const GemmOperand &a, const GemmOperand &b, const GemmOut &out) {
    const uint32_t stage_bytes = kGmM * kGmK * 2 + BN * kGmK * 2;
    uint32_t stages = ((uint32_t)ctx->max_smem_optin - 2048) / stage_bytes;
    if (stages > kGmStageMax) stages = kGmStageMax;
    const size_t smem = (size_t)stages * stage_bytes + 1024;
    CUtensorMap ma, mb;
    auto encode = [&](CUtensorMap *m, const GemmOperand &o, uint32_t box) {
        return tensor_map_bf16(ctx, m, o.p, o.page_table ? o.store_rows : o.rows, o.cols, o.ld, box, kGmK);
    };
    ctox_status rc = encode(&ma, a, kGmM);
    if (!rc) rc = encode(&mb, b, BN < 128 ? BN : 128);
    if (rc) return rc;
    CTOX_CUDA(ctx, cudaFuncSetAttribute(k_gemm<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const uint32_t tiles = ((a.rows + kGmM - 1) / kGmM) * ((b.rows + BN - 1) / BN);
    const uint32_t grid = tiles < (uint32_t)ctx->sm_count ? tiles : (uint32_t)ctx->sm_count;
    CTOX_CUDA(ctx, launch_pdl(k_gemm<BN>, dim3(grid), dim3(kGmThreads), smem, ctx->stream, ma, mb,
                              GemmPages{a.page_table, a.page_tokens, a.row0}, GemmPages{b.page_table, b.page_tokens, b.row0},
                              a.rows, b.rows, a.cols, stages, out, ctx->dev_error));
    return CTOX_OK;
}

}  // namespace

ctox_status launch_gemm(ctox_ctx *ctx, const GemmOperand &a, const GemmOperand &b, const GemmOut &out) {
    if (!a.rows || !b.rows) return CTOX_OK;
    if (a.cols != b.cols || a.ld % 8 || b.ld % 8) return fail(ctx, CTOX_SHAPE, "gemm: operand layouts");
    for (const GemmOperand *o : {&a, &b})
        if (o->page_table && (o->page_tokens % 128 || o->row0 % 128))
            return fail(ctx, CTOX_SHAPE, "gemm: pages of %u tokens are not whole tiles", o->page_tokens);
    // tile width by rounds over the SMs; a narrower tile has less reuse, hence the constant
    uint32_t best = 0, best_cost = 0xffffffffu;
    for (uint32_t bn : {256u, 128u, 64u}) {
        const uint32_t tiles = ((a.rows + kGmM - 1) / kGmM) * ((b.rows + bn - 1) / bn);
        const uint32_t cost = ((tiles + ctx->sm_count - 1) / ctx->sm_count) * (bn + 64);
        if (cost < best_cost) {
            best_cost = cost;
            best = bn;
        }
    }
    timing_begin(ctx);
    EX(best == 256 ? gemm_launch<256>(ctx, a, b, out) : best == 128 ? gemm_launch<128>(ctx, a, b, out)
                                                                   : gemm_launch<64>(ctx, a, b, out));
    timing_end(ctx, KC_GEMM, 2.0 * ((double)a.rows + b.rows) * a.cols + (out.bf16 ? 2.0 : 4.0) * a.rows * b.rows,
               2.0 * a.rows * b.rows * a.cols);
    return CTOX_OK;
}

__global__ void k_rope_table(const float *__restrict__ freq, uint32_t pairs, uint32_t pos0, uint32_t rows,
                             float2 *__restrict__ table) {
    pdl_launch();
    pdl_wait();
    const uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * pairs) return;
    float s, c;
    sincosf((float)(pos0 + i / pairs) * freq[i % pairs], &s, &c);
    table[i] = make_float2(c, s);
}

ctox_status launch_rope_table(ctox_ctx *ctx, const float *freq, uint32_t pairs, uint32_t pos0, uint32_t rows,
                              float2 *table) {
    CTOX_CUDA(ctx, launch_pdl(k_rope_table, dim3((rows * pairs + 255) / 256), dim3(256), 0, ctx->stream, freq, pairs, pos0,
                              rows, table));
    return CTOX_OK;
}

}  // namespace ctox
