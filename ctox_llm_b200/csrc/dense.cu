// Matrix-vector products with dense bf16 weights for short passes, the norms of longer passes, and
// the small kernels that go with them (embedding rows, weight layout).
#include "dense.cuh"

#include <map>
#include <mutex>
#include <tuple>

namespace ctox {

constexpr int kDvThreads = 256, kDvWarps = kDvThreads / 32;
constexpr uint64_t kUnitCost = 20000;                        // of a unit of rows, in columns
constexpr uint32_t kBatch = 4;                               // vectors a thread requests at once
constexpr int kSplitLanes = (kAttnSplitsDense + 31) / 32;  // splits per lane of a merging warp

// Columns c .. c + 3 of p, zero from `end` on.
__device__ __forceinline__ float4 load4(const float *p, uint32_t c, uint32_t end, bool vec) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c + 4 <= end && vec) return *reinterpret_cast<const float4 *>(p + c);
    if (c < end) v.x = p[c];
    if (c + 1 < end) v.y = p[c + 1];
    if (c + 2 < end) v.z = p[c + 2];
    if (c + 3 < end) v.w = p[c + 3];
    return v;
}
__device__ __forceinline__ void store4(float *p, uint32_t c, uint32_t end, const float4 &v) {
    if (c + 4 <= end && ((uintptr_t)p & 15) == 0) {
        *reinterpret_cast<float4 *>(p + c) = v;
        return;
    }
    if (c < end) p[c] = v.x;
    if (c + 1 < end) p[c + 1] = v.y;
    if (c + 2 < end) p[c + 2] = v.z;
    if (c + 3 < end) p[c + 3] = v.w;
}
__device__ __forceinline__ void prefetch_l1(const void *p) { asm volatile("prefetch.global.L1 [%0];" ::"l"(p)); }

// Sum over the kDvThreads / M threads of a position (whole warps); every thread of the CTA calls it.
template <int M>
__device__ __forceinline__ float position_sum(float v, float *red) {
    constexpr int W = kDvWarps / M;  // warps per position
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if (W == 1) return v;
    const int warp = threadIdx.x >> 5;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[warp] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < W; ++i) s += red[warp / W * W + i];
    return s;
}

__device__ void latent_append_row(const LatentAppend &a, uint32_t m, uint32_t tid, uint32_t nthreads, float *red) {
    const float *row = a.fan + (size_t)m * a.fan_stride + a.fan_off;
    float sq = 0.f;
    for (uint32_t c = tid; c < a.kv_rank; c += nthreads) sq += row[c] * row[c];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    __syncthreads();
    if ((tid & 31) == 0) red[tid >> 5] = sq;
    __syncthreads();
    float total = 0.f;
    for (uint32_t w = 0; w < nthreads / 32; ++w) total += red[w];
    const float inv = 1.0f / sqrtf(total / (float)a.kv_rank + a.eps);
    const uint32_t pos = a.pos0 + m;
    const size_t base = paged_slot(a.page_table, a.page_tokens, pos) * (a.kv_pad + a.rot_pad);
    auto store = [&](uint32_t c, float v) {
        if (a.bf16)
            ((__nv_bfloat16 *)a.cache)[base + c] = __float2bfloat16_rn(v);
        else
            ((float *)a.cache)[base + c] = v;
    };
    for (uint32_t c = tid; c < a.kv_pad; c += nthreads) store(c, c < a.kv_rank ? row[c] * inv * a.norm_w[c] : 0.f);
    for (uint32_t i = tid; i < a.rot_pad / 2; i += nthreads) {
        float u = 0.f, v = 0.f;
        if (2 * i < a.rot_dim) {
            u = row[a.kv_rank + 2 * i];
            v = row[a.kv_rank + 2 * i + 1];
            rope_pair(u, v, (float)pos * a.freq[i]);
        }
        store(a.kv_pad + 2 * i, u);
        store(a.kv_pad + 2 * i + 1, v);
    }
}

// One warp group of 2^lpr_log2 lanes per R rows, `ks` warps side by side on the columns of the same
// rows. The activations sit in shared memory in the order the lanes read them: blocks of LPR * 8
// columns as [half][lane][4]. The first weights of every warp are requested before the dependency
// wait (they are constants), so they arrive while the prologue forms the input.
// Weights are read once: their lines stay out of L1. Volatile, so that requests made ahead of the dependency wait stay
// ahead of it.
__device__ __forceinline__ uint4 load_weights(const __nv_bfloat16 *p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// IN: how the prologue forms the input (InKind); one kernel each, since every launch reads its code anew.
enum InKind : int { IN_PLAIN, IN_RMS, IN_LAYER, IN_MERGE };

template <int M, int R, int IN>
__global__ void __launch_bounds__(kDvThreads, 2)
    k_dense_matvec(const __nv_bfloat16 *__restrict__ W, uint32_t ld, uint32_t rows_per_group, uint32_t units_per_group,
                   uint32_t units, uint32_t ks, uint32_t lpr_log2, uint32_t npos, VecIn in, VecOut out,
                   LatentAppend ap, uint32_t append_positions) {
    pdl_launch();
    extern __shared__ __align__(16) float xs[];  // [M][ldx]
    __shared__ float red[kDvWarps];
    __shared__ float part[kDvWarps][32 * 4];  // partial sums of the column parts: [warp][subgroup rows x positions]
    __shared__ float mw[IN == IN_MERGE ? M : 1][kAttnSplitsDense];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t grid = gridDim.x - append_positions;
    if (blockIdx.x >= grid) {
        pdl_wait();
        latent_append_row(ap, blockIdx.x - grid, tid, kDvThreads, red);
        return;
    }
    const uint32_t lpr = 1u << lpr_log2, sub = lane >> lpr_log2, l = lane & (lpr - 1), nsub = 32u >> lpr_log2;
    const uint32_t span = lpr * 8;                       // columns per step
    const uint32_t nsteps = (ld + span - 1) / span, ldx = nsteps * span;
    const uint32_t kp = warp % ks, rg = warp / ks;       // column part, row group of this warp
    const uint32_t unit_rows = kDvWarps / ks * nsub * R;
    const uint32_t cnt = kp < nsteps ? (nsteps - kp + ks - 1) / ks : 0;
    constexpr int D = 8 / R;  // steps in flight
    uint4 buf[D][R];
    auto row_of = [&](uint32_t unit) { return (unit % units_per_group) * unit_rows + (rg * nsub + sub) * R; };
    auto fetch = [&](const __nv_bfloat16 *base, uint32_t row0, uint32_t i, uint4 *dst) {
        const uint32_t c = (kp + i * ks) * span + l * 8;
#pragma unroll
        for (int r = 0; r < R; ++r) {
            dst[r] = make_uint4(0, 0, 0, 0);
            if (i < cnt && c < ld && row0 + r < rows_per_group)
                dst[r] = load_weights(base + (size_t)(row0 + r) * ld + c);
        }
    };
    // ---- the input of `group`, normalised, into xs. Loads are issued in batches of kBatch vectors before
    // anything is stored, so that a thread waits for one round trip per batch.
    constexpr uint32_t T = kDvThreads / M;
    const uint32_t pm = tid / T, pt = tid % T;  // position and thread within it
    float *xm = xs + pm * ldx;
    const uint32_t cols = in.cols;
    auto at = [&](uint32_t c) { return c / span * span + ((c >> 2) & 1) * (lpr * 4) + (c % span) / 8 * 4; };  // c % 4 == 0
    auto slot4 = [&](uint32_t c) -> float4 & { return *reinterpret_cast<float4 *>(xm + at(c)); };
    auto each = [&](uint32_t end, auto &&f) {
        for (uint32_t c = pt * 4; c < end; c += T * 4) f(c);
    };
    auto stage = [&](uint32_t group) {
        const bool live = pm < npos;
        const uint32_t end = live ? cols : 0;
        if constexpr (IN == IN_MERGE) {
            const size_t row = (size_t)pm * in.groups + group;
            if (live) {  // every warp forms the weights of the splits: lane = split and split + 32
                float mv[kSplitLanes], sv[kSplitLanes], mx = -INFINITY, den = 0.f;
#pragma unroll
                for (int i = 0; i < kSplitLanes; ++i) {
                    const uint32_t sp = lane + i * 32;
                    const float2 ml = sp < in.splits ? *reinterpret_cast<const float2 *>(in.ws_ml + ((size_t)sp * in.ws_rows + row) * 2)
                                                     : make_float2(-INFINITY, 0.f);
                    mv[i] = ml.x;
                    sv[i] = ml.y;
                    mx = fmaxf(mx, ml.x);
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
                for (int i = 0; i < kSplitLanes; ++i) {
                    mv[i] = mv[i] == -INFINITY ? 0.f : expf(mv[i] - mx);
                    den += sv[i] * mv[i];
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
                if (pt < 32)
#pragma unroll
                    for (int i = 0; i < kSplitLanes; ++i) mw[pm][lane + i * 32] = mv[i] / den;
            }
            __syncthreads();
            each(ldx, [&](uint32_t c) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < end)
                    for (uint32_t s0 = 0; s0 < in.splits; s0 += kBatch * 2) {
                        float4 o[kBatch * 2];
#pragma unroll
                        for (uint32_t i = 0; i < kBatch * 2; ++i)
                            o[i] = s0 + i < in.splits ? *reinterpret_cast<const float4 *>(in.ws_o + ((size_t)(s0 + i) * in.ws_rows + row) * cols + c)
                                                      : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                        for (uint32_t i = 0; i < kBatch * 2; ++i) {
                            const float w = s0 + i < in.splits ? mw[pm][s0 + i] : 0.f;
                            v.x = fmaf(w, o[i].x, v.x);
                            v.y = fmaf(w, o[i].y, v.y);
                            v.z = fmaf(w, o[i].z, v.z);
                            v.w = fmaf(w, o[i].w, v.w);
                        }
                    }
                slot4(c) = v;
            });
            return;
        }
        const float *x = in.x + (size_t)pm * in.x_stride + (size_t)group * in.x_group;
        // f(c, values of p at c .. c + 3, values of q) for this thread's columns below `until`; zero from `end` on
        auto stream = [&](const float *p, const float *q, uint32_t until, auto &&f) {
            const bool vec_p = ((uintptr_t)p & 15) == 0, vec_q = ((uintptr_t)q & 15) == 0;
            for (uint32_t c0 = pt * 4; c0 < until; c0 += T * 4 * kBatch) {
                float4 a[kBatch], b[kBatch];
#pragma unroll
                for (uint32_t i = 0; i < kBatch; ++i) {
                    const uint32_t c = c0 + i * T * 4;
                    a[i] = load4(p, c, end, vec_p);
                    if (q) b[i] = load4(q, c, end, vec_q);
                }
#pragma unroll
                for (uint32_t i = 0; i < kBatch; ++i) {
                    const uint32_t c = c0 + i * T * 4;
                    if (c < until) f(c, a[i], b[i]);
                }
            }
        };
        if constexpr (IN == IN_PLAIN) {
            stream(x, nullptr, ldx, [&](uint32_t c, const float4 &v, const float4 &) { slot4(c) = v; });
            return;
        }
        auto sum4 = [](const float4 &v) { return (v.x + v.y) + (v.z + v.w); };
        auto sq4 = [](const float4 &v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); };
        const float n = (float)cols;
        float s = 0.f;
        if constexpr (IN == IN_RMS) {
            stream(x, in.y ? in.y + (size_t)pm * in.y_stride : nullptr, ldx, [&](uint32_t c, const float4 &xv, const float4 &yv) {
                float4 v = xv;
                if (in.y) {
                    v = make_float4(v.x + yv.x, v.y + yv.y, v.z + yv.z, v.w + yv.w);
                    if (blockIdx.x == 0 && c < end) store4(in.x_out + (size_t)pm * in.x_stride, c, cols, v);
                }
                slot4(c) = v;
                s += sq4(v);
            });
            const float inv = 1.0f / sqrtf(position_sum<M>(s, red) / n + in.eps);
            stream(in.w, nullptr, end, [&](uint32_t c, const float4 &w, const float4 &) {
                float4 v = slot4(c);
                slot4(c) = make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w);
            });
            return;
        }
        // sum of squared deviations of what xs holds (columns past the last one do not count)
        auto deviations = [&](float mean) {
            float q = 0.f;
            each(end, [&](uint32_t c) {
                float4 v = slot4(c);
                v = make_float4(v.x - mean, c + 1 < cols ? v.y - mean : 0.f, c + 2 < cols ? v.z - mean : 0.f,
                                c + 3 < cols ? v.w - mean : 0.f);
                q += sq4(v);
            });
            return q;
        };
        float mean = 0.f, inv = 0.f;
        const bool post = in.y && in.wb;
        if (in.y && !in.wb) {
            stream(in.y + (size_t)pm * in.y_stride, nullptr, end, [&](uint32_t c, const float4 &v, const float4 &) { slot4(c) = v; });
        } else if (in.y) {
            stream(in.y + (size_t)pm * in.y_stride, nullptr, end, [&](uint32_t c, const float4 &v, const float4 &) {
                slot4(c) = v;
                s += sum4(v);
            });
            mean = position_sum<M>(s, red) / n;
            inv = 1.0f / sqrtf(position_sum<M>(deviations(mean), red) / n + in.eps);
            s = 0.f;
        }
        stream(x, post ? in.wb : nullptr, ldx, [&](uint32_t c, const float4 &xv, const float4 &wb) {
            float4 v = xv;
            if (in.y && c < end) {
                const float4 y = slot4(c);
                v.x += post ? (y.x - mean) * inv * wb.x : y.x;
                v.y += post ? (y.y - mean) * inv * wb.y : y.y;  // the weight is zero past the last column
                v.z += post ? (y.z - mean) * inv * wb.z : y.z;
                v.w += post ? (y.w - mean) * inv * wb.w : y.w;
                if (blockIdx.x == 0) store4(in.x_out + (size_t)pm * in.x_stride, c, cols, v);
            }
            slot4(c) = v;
            s += sum4(v);
        });
        mean = position_sum<M>(s, red) / n;
        inv = 1.0f / sqrtf(position_sum<M>(deviations(mean), red) / n + in.eps);
        stream(in.w, nullptr, end, [&](uint32_t c, const float4 &w, const float4 &) {
            const float4 v = slot4(c);
            slot4(c) = make_float4((v.x - mean) * inv * w.x, (v.y - mean) * inv * w.y, (v.z - mean) * inv * w.z,
                                   (v.w - mean) * inv * w.w);
        });
    };
    // norm weights are constants: bring their lines in before the wait
    if constexpr (IN == IN_RMS || IN == IN_LAYER)
        each(cols, [&](uint32_t c) {
            prefetch_l1(in.w + c);
            if (IN == IN_LAYER && in.y && in.wb) prefetch_l1(in.wb + c);
        });

    uint32_t staged = 0xffffffffu;
    for (uint32_t unit = blockIdx.x; unit < units; unit += grid) {
        const uint32_t group = unit / units_per_group, row0 = row_of(unit);
        const __nv_bfloat16 *base = W + (size_t)group * rows_per_group * ld;
#pragma unroll
        for (int d = 0; d < D; ++d) fetch(base, row0, d, buf[d]);
        if (group != staged) {
            if (staged == 0xffffffffu)
                pdl_wait();
            else
                __syncthreads();
            stage(group);
            __syncthreads();
            staged = group;
        }
        float acc[M][R];
#pragma unroll
        for (int m = 0; m < M; ++m)
#pragma unroll
            for (int r = 0; r < R; ++r) acc[m][r] = 0.f;
        for (uint32_t i0 = 0; i0 < cnt; i0 += D) {
#pragma unroll
            for (int d = 0; d < D; ++d) {
                uint4 w[R];
#pragma unroll
                for (int r = 0; r < R; ++r) w[r] = buf[d][r];
                fetch(base, row0, i0 + d + D, buf[d]);
                if (i0 + d < cnt) {
                    const float *xp = xs + (kp + (i0 + d) * ks) * span + l * 4;
#pragma unroll
                    for (int m = 0; m < M; ++m) {
                        const float4 a = *reinterpret_cast<const float4 *>(xp + m * ldx);
                        const float4 b = *reinterpret_cast<const float4 *>(xp + m * ldx + lpr * 4);
#pragma unroll
                        for (int r = 0; r < R; ++r) {
                            float s = acc[m][r];
                            s = fmaf(__uint_as_float(w[r].x << 16), a.x, s);
                            s = fmaf(__uint_as_float(w[r].x & 0xffff0000u), a.y, s);
                            s = fmaf(__uint_as_float(w[r].y << 16), a.z, s);
                            s = fmaf(__uint_as_float(w[r].y & 0xffff0000u), a.w, s);
                            s = fmaf(__uint_as_float(w[r].z << 16), b.x, s);
                            s = fmaf(__uint_as_float(w[r].z & 0xffff0000u), b.y, s);
                            s = fmaf(__uint_as_float(w[r].w << 16), b.z, s);
                            s = fmaf(__uint_as_float(w[r].w & 0xffff0000u), b.w, s);
                            acc[m][r] = s;
                        }
                    }
                }
            }
        }
#pragma unroll
        for (int m = 0; m < M; ++m)
#pragma unroll
            for (int r = 0; r < R; ++r)
                for (uint32_t o = lpr >> 1; o > 0; o >>= 1) acc[m][r] += __shfl_xor_sync(0xffffffffu, acc[m][r], o);
        if (ks > 1) {  // add the column parts of the rows up (part order), in the first of their warps
            __syncthreads();
            if (l == 0)
#pragma unroll
                for (int m = 0; m < M; ++m)
#pragma unroll
                    for (int r = 0; r < R; ++r) part[warp][sub * (M * R) + m * R + r] = acc[m][r];
            __syncthreads();
            if (kp == 0) {
                for (uint32_t q = 1; q < ks; ++q)
#pragma unroll
                    for (int m = 0; m < M; ++m)
#pragma unroll
                        for (int r = 0; r < R; ++r) acc[m][r] += part[warp + q][sub * (M * R) + m * R + r];
            }
        }
        if (kp == 0) {
            for (uint32_t k = l; k < (uint32_t)(M * R); k += lpr) {
                float v = 0.f, pair = 0.f;
#pragma unroll
                for (int m = 0; m < M; ++m)
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        if (k == (uint32_t)(m * R + r)) v = acc[m][r];
                        if ((k ^ 1u) == (uint32_t)(m * R + r)) pair = acc[m][r];
                    }
                const uint32_t m = k / R, row = row0 + k % R;
                if (m >= npos || row >= rows_per_group) continue;
                if (out.bias) {
                    v += out.bias[(size_t)group * rows_per_group + row];
                    if ((row ^ 1u) < rows_per_group) pair += out.bias[(size_t)group * rows_per_group + (row ^ 1u)];
                }
                if (out.kind == OUT_CLAMPED_GLU) {
                    if (!(row & 1)) out.y[(size_t)m * out.y_stride + (row >> 1)] = clamped_glu(v, pair, out.cap, out.slope);
                    continue;
                }
                if (out.kind == OUT_RELU2) {
                    v = v > 0.f ? v * v : 0.f;
                } else if (out.kind == OUT_SOFTCAP) {
                    v = out.cap * tanhf(v / out.cap);
                } else if (out.kind == OUT_ROPE) {
                    const uint32_t w = row % out.head_width;
                    if (w >= out.rope0 && w < out.rope0 + out.rope_dims) {
                        const float angle = (float)(out.pos0 + m) * out.freq[(w - out.rope0) >> 1];
                        float a = (w & 1) ? pair : v, b = (w & 1) ? v : pair;
                        rope_pair(a, b, angle);
                        v = (w & 1) ? b : a;
                    }
                }
                out.y[(size_t)m * out.y_stride + (size_t)group * rows_per_group + row] = v;
            }
        }
    }
}

namespace {

template <int M, int R, int IN>
ctox_status matvec_kernel(ctox_ctx *ctx, const DenseMat &w, uint32_t groups, uint32_t m, const VecIn &in,
                          const VecOut &out, const LatentAppend *append, uint32_t append_positions, size_t smem,
                          uint32_t ks, uint32_t lpr_log2) {
    static std::mutex mu;
    static std::map<std::tuple<int, size_t>, int> resident;  // CTAs per SM by (device, shared memory)
    int per_sm = 0;
    {
        std::lock_guard<std::mutex> lock(mu);
        auto it = resident.find({ctx->device, smem});
        if (it == resident.end()) {
            CTOX_CUDA(ctx, cudaFuncSetAttribute(k_dense_matvec<M, R, IN>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                ctx->max_smem_optin - 8192));
            // One split of the SM's memory into L1 and shared for all of them: kernels that ask for different ones
            // do not overlap on an SM.
            CTOX_CUDA(ctx, cudaFuncSetAttribute(k_dense_matvec<M, R, IN>, cudaFuncAttributePreferredSharedMemoryCarveout, 75));
            CTOX_CUDA(ctx, cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, k_dense_matvec<M, R, IN>, kDvThreads, smem));
            if (per_sm < 1) return fail(ctx, CTOX_MEMORY_BUDGET, "dense matvec: %zu bytes of shared memory", smem);
            resident[{ctx->device, smem}] = per_sm;
        } else {
            per_sm = it->second;
        }
    }
    const uint32_t rows_per_group = w.rows / groups, unit_rows = kDvWarps / ks * (32u >> lpr_log2) * R;
    const uint32_t units_per_group = (rows_per_group + unit_rows - 1) / unit_rows, units = units_per_group * groups;
    const uint32_t fit = (uint32_t)(per_sm * ctx->sm_count), waves = (units + fit - 1) / fit;
    const uint32_t grid = (units + waves - 1) / waves;
    const LatentAppend ap = append ? *append : LatentAppend{};
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_dense_matvec<M, R, IN>, dim3(grid + append_positions), dim3(kDvThreads), smem, ctx->stream,
                              (const __nv_bfloat16 *)w.w, w.ld, rows_per_group, units_per_group, units, ks, lpr_log2, m,
                              in, out, ap, append_positions));
    timing_end(ctx, KC_DENSE_MATVEC, 2.0 * w.rows * w.ld, 2.0 * w.rows * w.ld * m);
    return CTOX_OK;
}

template <int M, int R, typename... Args>
ctox_status matvec_launch(ctox_ctx *ctx, const DenseMat &w, uint32_t groups, uint32_t m, const VecIn &in, Args... args) {
    if (in.ws_o) return matvec_kernel<M, R, IN_MERGE>(ctx, w, groups, m, in, args...);
    if (in.norm == NORM_NONE) return matvec_kernel<M, R, IN_PLAIN>(ctx, w, groups, m, in, args...);
    if (in.norm == NORM_RMS) return matvec_kernel<M, R, IN_RMS>(ctx, w, groups, m, in, args...);
    return matvec_kernel<M, R, IN_LAYER>(ctx, w, groups, m, in, args...);
}

}  // namespace

ctox_status launch_dense_matvec(ctox_ctx *ctx, const DenseMat &w, uint32_t groups, uint32_t m, const VecIn &in,
                                const VecOut &out, const LatentAppend *append) {
    uint32_t lpr_log2 = 5;  // lanes per row: fewer for narrow matrices
    while (lpr_log2 > 3 && w.ld <= (8u << (lpr_log2 - 1))) --lpr_log2;
    const uint32_t span = 8u << lpr_log2, nsteps = (w.ld + span - 1) / span;
    const size_t row_bytes = (size_t)nsteps * span * 4;
    uint32_t M = m <= 1 ? 1 : m <= 2 ? 2 : m <= 4 ? 4 : 8;
    while (M > 1 && M * row_bytes + 8192 > (size_t)ctx->max_smem_optin) M /= 2;
    if (M * row_bytes + 8192 > (size_t)ctx->max_smem_optin)
        return fail(ctx, CTOX_MEMORY_BUDGET, "dense matvec: %u columns do not fit shared memory", w.ld);
    for (uint32_t p = 0; p < m; p += M) {
        const uint32_t n = m - p < M ? m - p : M;
        VecIn i = in;
        VecOut o = out;
        if (i.x) i.x += (size_t)p * i.x_stride;
        if (i.y) i.y += (size_t)p * i.y_stride;
        if (i.x_out) i.x_out += (size_t)p * i.x_stride;
        if (i.ws_o) {
            i.ws_o += (size_t)p * i.groups * i.cols;
            i.ws_ml += (size_t)p * i.groups * 2;
        }
        o.y += (size_t)p * o.y_stride;
        o.pos0 += p;
        // Rows per warp (R) and warps per row (ks): the least work of the busiest CTA with two CTAs per SM,
        // a unit's fixed cost counted as some columns.
        const uint32_t rows = w.rows / groups, nsub = 32u >> lpr_log2, fit = 2 * (uint32_t)ctx->sm_count;
        uint32_t R = 2, ks = 1;
        uint64_t best = ~0ull;
        for (uint32_t r = 2; r <= (M <= 2 ? 4u : 2u); r *= 2)
            for (uint32_t k = 1; k <= kDvWarps && k <= nsteps; k *= 2) {
                const uint32_t unit = kDvWarps / k * nsub * r, units = (rows + unit - 1) / unit * groups;
                const uint64_t cols = (uint64_t)((nsteps + k - 1) / k) * k * span;
                const uint64_t cost = (uint64_t)((units + fit - 1) / fit) * (unit * cols + kUnitCost);
                if (cost < best) {
                    best = cost;
                    R = r;
                    ks = k;
                }
            }
        const uint32_t na = append && p == 0 ? m : 0;
        const size_t smem = M * row_bytes;
        ctox_status rc;
#define DV(MM, RR) matvec_launch<MM, RR>(ctx, w, groups, n, i, o, append, na, smem, ks, lpr_log2)
        if (M == 1)
            rc = R == 4 ? DV(1, 4) : DV(1, 2);
        else if (M == 2)
            rc = R == 4 ? DV(2, 4) : DV(2, 2);
        else if (M == 4)
            rc = DV(4, 2);
        else
            rc = DV(8, 2);
#undef DV
        if (rc) return rc;
    }
    return CTOX_OK;
}

// ------------------------------------------------------------------ norms of the residual stream
constexpr int kSnThreads = 256;

__global__ void __launch_bounds__(kSnThreads) k_stream_norm(StreamNorm a) {
    pdl_launch();
    pdl_wait();
    extern __shared__ __align__(16) float v_s[];  // [width rounded up to 4]
    __shared__ float red[kDvWarps];
    const uint32_t row = a.rows ? a.rows[blockIdx.x] : blockIdx.x, tid = threadIdx.x, W = a.width;
    const float n = (float)W;
    const float *x = a.x + (size_t)row * W, *y = a.y ? a.y + (size_t)row * W : nullptr;
    auto slot4 = [&](uint32_t c) -> float4 & { return *reinterpret_cast<float4 *>(v_s + c); };
    auto stream = [&](const float *p, const float *q, auto &&f) {  // batches of loads, then the work on them
        const bool vec_p = ((uintptr_t)p & 15) == 0, vec_q = ((uintptr_t)q & 15) == 0;
        for (uint32_t c0 = tid * 4; c0 < W; c0 += kSnThreads * 4 * kBatch) {
            float4 u[kBatch], v[kBatch];
#pragma unroll
            for (uint32_t i = 0; i < kBatch; ++i) {
                u[i] = load4(p, c0 + i * kSnThreads * 4, W, vec_p);
                if (q) v[i] = load4(q, c0 + i * kSnThreads * 4, W, vec_q);
            }
#pragma unroll
            for (uint32_t i = 0; i < kBatch; ++i)
                if (c0 + i * kSnThreads * 4 < W) f(c0 + i * kSnThreads * 4, u[i], v[i]);
        }
    };
    auto deviations = [&](float mean) {
        float q = 0.f;
        for (uint32_t c = tid * 4; c < W; c += kSnThreads * 4) {
            const float4 v = slot4(c);
            const float d0 = v.x - mean, d1 = c + 1 < W ? v.y - mean : 0.f, d2 = c + 2 < W ? v.z - mean : 0.f,
                        d3 = c + 3 < W ? v.w - mean : 0.f;
            q += (d0 * d0 + d1 * d1) + (d2 * d2 + d3 * d3);
        }
        return q;
    };
    float s = 0.f, mean = 0.f, inv = 0.f;
    const bool post = y && a.wb, rms = a.norm == NORM_RMS;
    if (post) {
        stream(y, nullptr, [&](uint32_t c, const float4 &v, const float4 &) {
            slot4(c) = v;
            s += (v.x + v.y) + (v.z + v.w);
        });
        mean = position_sum<1>(s, red) / n;
        inv = 1.0f / sqrtf(position_sum<1>(deviations(mean), red) / n + a.eps);
        s = 0.f;
    }
    stream(x, post ? a.wb : y, [&](uint32_t c, const float4 &xv, const float4 &wb) {
        float4 v = xv;
        if (y && !post) {
            v = make_float4(v.x + wb.x, v.y + wb.y, v.z + wb.z, v.w + wb.w);
        } else if (y) {
            const float4 u = slot4(c);
            v.x += (u.x - mean) * inv * wb.x;
            v.y += (u.y - mean) * inv * wb.y;  // the weight is zero past the last column
            v.z += (u.z - mean) * inv * wb.z;
            v.w += (u.w - mean) * inv * wb.w;
        }
        if (a.x_out) store4(a.x_out + (size_t)row * W, c, W, v);
        slot4(c) = v;
        s += rms ? (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w) : (v.x + v.y) + (v.z + v.w);
    });
    if (!a.w) return;
    s = position_sum<1>(s, red) / n;
    mean = rms ? 0.f : s;
    inv = 1.0f / sqrtf((rms ? s : position_sum<1>(deviations(mean), red) / n) + a.eps);
    stream(a.w, nullptr, [&](uint32_t c, const float4 &w, const float4 &) {
        const float4 u = slot4(c);
        const float4 v = make_float4((u.x - mean) * inv * w.x, (u.y - mean) * inv * w.y, (u.z - mean) * inv * w.z,
                                     (u.w - mean) * inv * w.w);
        if (a.f32_out) store4(a.f32_out + (size_t)blockIdx.x * W, c, W, v);
        if (a.bf16_out) {  // rows are padded to whole vectors of eight
            const __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
            *reinterpret_cast<uint2 *>(a.bf16_out + (size_t)blockIdx.x * a.bf16_ld + c) = *reinterpret_cast<const uint2 *>(h);
        }
    });
}

ctox_status launch_stream_norm(ctox_ctx *ctx, const StreamNorm &a, uint32_t m) {
    const size_t smem = ((size_t)a.width + 3) / 4 * 16;
    if (smem + 1024 > (size_t)ctx->max_smem_optin)
        return fail(ctx, CTOX_MEMORY_BUDGET, "stream norm: width %u does not fit shared memory", a.width);
    if (smem > 40 * 1024)
        CTOX_CUDA(ctx, cudaFuncSetAttribute(k_stream_norm, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_stream_norm, dim3(m), dim3(kSnThreads), smem, ctx->stream, a));
    timing_end(ctx, KC_NORM,
               (double)m * a.width * (4 + (a.y ? 4 : 0) + (a.x_out ? 4 : 0) + (a.f32_out ? 4 : 0) + (a.bf16_out ? 2 : 0)), 0);
    return CTOX_OK;
}

__global__ void __launch_bounds__(kSnThreads) k_latent_split(const float *__restrict__ fan, uint32_t fan_stride,
                                                             uint32_t q_rank, const float *__restrict__ q_norm,
                                                             float eps, __nv_bfloat16 *__restrict__ cq, uint32_t cq_ld,
                                                             LatentAppend ap, int has_append) {
    pdl_launch();
    pdl_wait();
    __shared__ float red[kDvWarps];
    const uint32_t m = blockIdx.x, tid = threadIdx.x;
    const float *row = fan + (size_t)m * fan_stride;
    float s = 0.f;
    for (uint32_t c = tid; c < q_rank; c += kSnThreads) s += row[c] * row[c];
    const float inv = 1.0f / sqrtf(position_sum<1>(s, red) / (float)q_rank + eps);
    for (uint32_t c = tid; c < q_rank; c += kSnThreads)
        cq[(size_t)m * cq_ld + c] = __float2bfloat16_rn(row[c] * inv * q_norm[c]);
    if (has_append) latent_append_row(ap, m, tid, kSnThreads, red);
}

ctox_status launch_latent_split(ctox_ctx *ctx, const float *fan, uint32_t fan_stride, uint32_t q_rank,
                                const float *q_norm, float eps, __nv_bfloat16 *cq, uint32_t cq_ld,
                                const LatentAppend *append, uint32_t m) {
    const LatentAppend ap = append ? *append : LatentAppend{};
    timing_begin(ctx);
    CTOX_CUDA(ctx, launch_pdl(k_latent_split, dim3(m), dim3(kSnThreads), 0, ctx->stream, fan, fan_stride, q_rank, q_norm,
                              eps, cq, cq_ld, ap, (int)(append != nullptr)));
    timing_end(ctx, KC_QKV, (double)m * (fan_stride * 4.0 + q_rank * 2.0 + (ap.kv_pad + ap.rot_pad) * 2.0), 0);
    return CTOX_OK;
}

// ------------------------------------------------------------------ embedding rows, weight layout
__global__ void __launch_bounds__(256) k_embed_dense(const __nv_bfloat16 *__restrict__ embed, uint32_t ld,
                                                     const uint32_t *__restrict__ tokens, uint32_t width,
                                                     float scale, float *__restrict__ x) {
    pdl_launch();
    pdl_wait();
    const __nv_bfloat16 *row = embed + (size_t)tokens[blockIdx.x] * ld;
    for (uint32_t c = threadIdx.x; c < width; c += 256) x[(size_t)blockIdx.x * width + c] = __bfloat162float(row[c]) * scale;
}

ctox_status launch_embed_dense(ctox_ctx *ctx, const __nv_bfloat16 *embed, uint32_t ld, const uint32_t *tokens,
                               uint32_t width, uint32_t m, float scale, float *x) {
    CTOX_CUDA(ctx, launch_pdl(k_embed_dense, dim3(m), dim3(256), 0, ctx->stream, embed, ld, tokens, width, scale, x));
    return CTOX_OK;
}

__device__ __forceinline__ uint32_t pad_index(const PadAxis &a, uint32_t i) {
    const uint32_t g = i / a.group, w = i % a.group;
    return g * a.group_pad + (w < a.split ? w : w - a.split + a.split_pad);
}

__global__ void k_relayout(const __nv_bfloat16 *__restrict__ src, uint32_t rows, uint32_t cols, PadAxis ra, PadAxis ca,
                           __nv_bfloat16 *__restrict__ dst, uint32_t dst_ld, uint32_t transpose_group,
                           uint32_t transpose_cols) {
    const uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (uint64_t)rows * cols) return;
    const uint32_t r = pad_index(ra, (uint32_t)(i / cols)), c = pad_index(ca, (uint32_t)(i % cols));
    if (transpose_group)
        dst[((size_t)(r / transpose_group) * transpose_cols + c) * dst_ld + r % transpose_group] = src[i];
    else
        dst[(size_t)r * dst_ld + c] = src[i];
}

ctox_status launch_relayout(ctox_ctx *ctx, const __nv_bfloat16 *src, uint32_t rows, uint32_t cols, PadAxis ra,
                            PadAxis ca, __nv_bfloat16 *dst, uint32_t dst_ld, uint32_t transpose_group,
                            uint32_t transpose_cols) {
    const uint64_t n = (uint64_t)rows * cols;
    k_relayout<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(src, rows, cols, ra, ca, dst, dst_ld,
                                                                     transpose_group, transpose_cols);
    CTOX_CUDA(ctx, cudaGetLastError());
    return CTOX_OK;
}

template <typename T>
__global__ void k_fill_normal_dense(T *__restrict__ out, uint64_t n, float std, uint64_t seed) {
    const uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    uint64_t x = seed + (i + 1) * 0x9E3779B97F4A7C15ull;  // splitmix64
    x = (x ^ (x >> 30)) * 0xBF58476D1CE4E5B9ull;
    x = (x ^ (x >> 27)) * 0x94D049BB133111EBull;
    x ^= x >> 31;
    const float u1 = ((float)(x >> 40) + 0.5f) * (1.0f / 16777216.0f);
    const float u2 = (float)((x >> 16) & 0xffffff) * (1.0f / 16777216.0f);
    out[i] = (T)(std * sqrtf(-2.0f * logf(u1)) * cosf(6.28318530718f * u2));
}

ctox_status launch_fill_normal_bf16(ctox_ctx *ctx, __nv_bfloat16 *out, uint64_t n, float std, uint64_t seed) {
    k_fill_normal_dense<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(out, n, std, seed);
    CTOX_CUDA(ctx, cudaGetLastError());
    return CTOX_OK;
}
ctox_status launch_fill_normal_f32(ctox_ctx *ctx, float *out, uint64_t n, float std, uint64_t seed) {
    k_fill_normal_dense<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(out, n, std, seed);
    CTOX_CUDA(ctx, cudaGetLastError());
    return CTOX_OK;
}

}  // namespace ctox
