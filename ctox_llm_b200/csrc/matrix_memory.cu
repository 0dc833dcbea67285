// Matrix memory, short passes: one pass over the state for up to kDensePass positions.
#include <cooperative_groups.h>

#include "matrix_memory.cuh"

namespace ctox {

namespace cg = cooperative_groups;
constexpr int kMmThreads = 256, kMmWarps = kMmThreads / 32, kMmRows = 4;  // state rows a warp works on at once

// A cluster per head, its CTAs share the state's rows (value dimensions, the normaliser behind them). A row stays
// in registers for all M positions: the gates' scales of every position are known before the state is touched.
// The head's norm needs the outputs of all CTAs: they meet through distributed shared memory.
template <int M>
__global__ void __launch_bounds__(kMmThreads) k_matrix_memory(MatrixMemory a, const float *__restrict__ fan, uint32_t fan_stride,
                                                              uint32_t gate_off, uint32_t npos, uint32_t rows_per, float *__restrict__ out) {
    pdl_launch();
    extern __shared__ __align__(16) float sm[];
    __shared__ float keep[M], take[M], floor_s[M], part[kMmWarps][M];
    __shared__ float xch[M][2];  // for the cluster: sum of squares of this CTA's rows, n . q (from its owner)
    cg::cluster_group cluster = cg::this_cluster();
    const uint32_t ctas = cluster.num_blocks(), rank = cluster.block_rank(), head = blockIdx.x / ctas;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *q_s = sm;                       // [M][dim_pad]
    float *k_s = q_s + M * a.dim_pad;      // [M][dim_pad]
    float *v_s = k_s + M * a.dim_pad;      // [M][rows_per]
    float *num = v_s + M * rows_per;       // [M][rows_per]
    const uint32_t row_beg = rank * rows_per, all = a.vdim + 1;  // row vdim stands for the normaliser
    const uint32_t rows = row_beg < all ? min(rows_per, all - row_beg) : 0;
    float *state = a.state + (size_t)head * (a.vdim_pad + kMemRows) * a.dim_pad;
    auto state_row = [&](uint32_t r) { return state + (size_t)(r < a.vdim ? r : a.vdim_pad) * a.dim_pad; };
    pdl_wait();
    const uint32_t k_off = a.heads * a.dim_pad, v_off = 2 * k_off, g_off = v_off + a.heads * a.vdim_pad;
    if (warp == 0) {  // lane = position; the running maximum goes from lane to lane
        float i = 0.f, f = 0.f, top = a.top[head], before = 0.f, after = 0.f;
        if (lane < npos) {
            const float *g = fan + (size_t)lane * fan_stride + gate_off + head;
            i = soft_cap(g[0] + a.i_bias[head], a.gate_cap);
            f = log_sigmoid(soft_cap(g[a.heads] + a.f_bias[head], a.gate_cap));
        }
        for (uint32_t t = 0; t < npos; ++t) {
            const float next = fmaxf(__shfl_sync(0xffffffffu, f, t) + top, __shfl_sync(0xffffffffu, i, t));
            if (lane == t) {
                before = top;
                after = next;
            }
            top = next;
        }
        if (lane < npos) {
            keep[lane] = expf(f + before - after);
            take[lane] = expf(i - after);
            floor_s[lane] = expf(-after);
        }
        if (lane == 0) xch[0][0] = top;  // parked until every CTA has read the old one
    }
    const float scale = 1.0f / sqrtf((float)a.dim);
    for (uint32_t i = tid; i < M * a.dim_pad; i += kMmThreads) {
        const uint32_t t = i / a.dim_pad, d = i % a.dim_pad;
        const float *row = fan + (size_t)t * fan_stride + head * a.dim_pad + d;
        q_s[i] = t < npos ? row[0] * scale : 0.f;
        k_s[i] = t < npos ? row[k_off] : 0.f;
    }
    for (uint32_t i = tid; i < M * rows; i += kMmThreads) {
        const uint32_t t = i / rows, r = i % rows;
        v_s[t * rows_per + r] = t >= npos               ? 0.f
                                : row_beg + r < a.vdim ? fan[(size_t)t * fan_stride + v_off + head * a.vdim_pad + row_beg + r]
                                                       : 1.f;
    }
    __syncthreads();
    const float top_new = xch[0][0];
    for (uint32_t r0 = warp * kMmRows; r0 < rows; r0 += kMmWarps * kMmRows) {
        float acc[kMmRows][M];
        float *sp[kMmRows];
#pragma unroll
        for (int r = 0; r < kMmRows; ++r) {
            sp[r] = state_row(row_beg + min(r0 + r, rows - 1));
#pragma unroll
            for (int t = 0; t < M; ++t) acc[r][t] = 0.f;
        }
        for (uint32_t d = lane * 4; d < a.dim_pad; d += 128) {
            float4 s[kMmRows];
#pragma unroll
            for (int r = 0; r < kMmRows; ++r) s[r] = *reinterpret_cast<const float4 *>(sp[r] + d);
#pragma unroll
            for (int t = 0; t < M; ++t) {
                if (t >= (int)npos) break;
                const float4 k = *reinterpret_cast<const float4 *>(k_s + t * a.dim_pad + d);
                const float4 q = *reinterpret_cast<const float4 *>(q_s + t * a.dim_pad + d);
                const float kp = keep[t], tk = take[t];
#pragma unroll
                for (int r = 0; r < kMmRows; ++r) {
                    const float v = tk * v_s[t * rows_per + min(r0 + r, rows - 1)];
                    s[r].x = fmaf(kp, s[r].x, v * k.x);
                    s[r].y = fmaf(kp, s[r].y, v * k.y);
                    s[r].z = fmaf(kp, s[r].z, v * k.z);
                    s[r].w = fmaf(kp, s[r].w, v * k.w);
                    acc[r][t] += (s[r].x * q.x + s[r].y * q.y) + (s[r].z * q.z + s[r].w * q.w);
                }
            }
#pragma unroll
            for (int r = 0; r < kMmRows; ++r)
                if (r0 + r < rows) *reinterpret_cast<float4 *>(sp[r] + d) = s[r];
        }
#pragma unroll
        for (int r = 0; r < kMmRows; ++r)
#pragma unroll
            for (int t = 0; t < M; ++t) {
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) acc[r][t] += __shfl_xor_sync(0xffffffffu, acc[r][t], o);
                if (lane == 0 && r0 + r < rows) num[t * rows_per + r0 + r] = acc[r][t];
            }
    }
    __syncthreads();
    // ---- sums of squares of the numerators, over this CTA's value rows
    float sq[M];
#pragma unroll
    for (int t = 0; t < M; ++t) sq[t] = 0.f;
    for (uint32_t r = tid; r < rows; r += kMmThreads)
        if (row_beg + r < a.vdim)
#pragma unroll
            for (int t = 0; t < M; ++t) sq[t] += num[t * rows_per + r] * num[t * rows_per + r];
#pragma unroll
    for (int t = 0; t < M; ++t) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sq[t] += __shfl_xor_sync(0xffffffffu, sq[t], o);
        if (lane == 0) part[warp][t] = sq[t];
    }
    __syncthreads();
    if (tid < M) {
        float s = 0.f;
        for (int w = 0; w < kMmWarps; ++w) s += part[w][tid];
        xch[tid][0] = s;
        if (a.vdim >= row_beg && a.vdim < row_beg + rows) xch[tid][1] = num[tid * rows_per + a.vdim - row_beg];
    }
    cluster.sync();
    if (rank == 0 && tid == 0) a.top[head] = top_new;
    const uint32_t owner = a.vdim / rows_per;
    if (tid < M) {  // part[0]: 1 / denominator, part[1]: 1 / root mean square
        const float nq = *cluster.map_shared_rank(&xch[tid][1], owner);
        float s = 0.f;
        for (uint32_t c = 0; c < ctas; ++c) s += *cluster.map_shared_rank(&xch[tid][0], c);
        const float inv = 1.0f / (fmaxf(fabsf(nq), floor_s[tid]) + 1e-6f);
        part[0][tid] = inv;
        part[1][tid] = 1.0f / sqrtf(s * inv * inv / (float)a.vdim + a.eps);
    }
    cluster.sync();  // nobody leaves while its shared memory is read
    for (uint32_t i = tid; i < npos * rows; i += kMmThreads) {
        const uint32_t t = i / rows, r = i % rows, v = row_beg + r;
        if (v >= a.vdim) continue;
        const float g = fan[(size_t)t * fan_stride + g_off + head * a.vdim_pad + v];
        out[(size_t)t * a.heads * a.vdim_pad + head * a.vdim_pad + v] =
            num[t * rows_per + r] * part[0][t] * part[1][t] * a.norm_w[head * a.vdim + v] * sigmoid(g);
    }
    if (rank == 0)
        for (uint32_t i = tid; i < npos * (a.vdim_pad - a.vdim); i += kMmThreads)
            out[(size_t)(i / (a.vdim_pad - a.vdim)) * a.heads * a.vdim_pad + head * a.vdim_pad + a.vdim + i % (a.vdim_pad - a.vdim)] = 0.f;
}

namespace {

template <int M>
ctox_status memory_launch(ctox_ctx *ctx, const MatrixMemory &a, const float *fan, uint32_t fan_stride, uint32_t gate_off,
                          uint32_t m, float *out) {
    uint32_t ctas = 8;
    while (ctas > 1 && a.vdim < ctas * 16) ctas /= 2;
    const uint32_t rows_per = (a.vdim + 1 + ctas - 1) / ctas;
    const size_t smem = (size_t)2 * M * (a.dim_pad + rows_per) * 4;
    if (smem + 2048 > (size_t)ctx->max_smem_optin)
        return fail(ctx, CTOX_MEMORY_BUDGET, "matrix memory: %u x %u per head does not fit shared memory", a.dim, a.vdim);
    if (smem > 40 * 1024)
        CTOX_CUDA(ctx, cudaFuncSetAttribute(k_matrix_memory<M>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CTOX_CUDA(ctx, launch_pdl_cluster(k_matrix_memory<M>, dim3(a.heads * ctas), dim3(kMmThreads), smem, ctx->stream, ctas, a, fan,
                                      fan_stride, gate_off, m, rows_per, out));
    return CTOX_OK;
}

}  // namespace

ctox_status launch_matrix_memory(ctox_ctx *ctx, const MatrixMemory &a, const float *fan, uint32_t fan_stride,
                                 uint32_t gate_off, uint32_t m, float *out) {
    const double state = 4.0 * a.heads * (a.vdim + 1) * a.dim_pad;
    timing_begin(ctx);
    EX(m <= 1   ? memory_launch<1>(ctx, a, fan, fan_stride, gate_off, m, out)
       : m <= 2 ? memory_launch<2>(ctx, a, fan, fan_stride, gate_off, m, out)
       : m <= 4 ? memory_launch<4>(ctx, a, fan, fan_stride, gate_off, m, out)
                : memory_launch<8>(ctx, a, fan, fan_stride, gate_off, m, out));
    timing_end(ctx, KC_MEMORY, 2 * state, 6.0 * m * a.heads * a.vdim * a.dim);
    return CTOX_OK;
}

}  // namespace ctox
