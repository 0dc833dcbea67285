// Fifth-generation tensor cores, tensor memory, TMA and mbarriers: thin wrappers over the PTX
// instructions, with bounded waits.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include <cstdint>

#include "common.cuh"

namespace ctox {

// Row-major bf16 matrix, box_cols x box_rows boxes with the matching shared-memory swizzle
// (box_cols * 2 = 32, 64 or 128 bytes). Out-of-range elements read as zero.
ctox_status tensor_map_bf16(ctox_ctx *ctx, CUtensorMap *map, const void *base, uint64_t rows, uint64_t cols, uint64_t ld,
                            uint32_t box_rows, uint32_t box_cols);

// A segment of a head's dimensions (a multiple of 16), cut into boxes one swizzle atom wide.
struct HeadBox {
    uint32_t width, n;
};
__host__ __device__ inline HeadBox head_box(uint32_t dims) {
    const uint32_t w = dims % 64 == 0 ? 64 : dims % 32 == 0 ? 32 : 16;
    return HeadBox{w, dims / w};
}

#ifdef __CUDACC__
namespace umma {

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void bar_init(uint32_t bar, uint32_t count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory");
}
__device__ __forceinline__ void bar_init_fence() { asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory"); }
__device__ __forceinline__ void bar_expect(uint32_t bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void bar_arrive(uint32_t bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ bool bar_try(uint32_t bar, uint32_t parity) {
    uint32_t ok;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(ok)
        : "r"(bar), "r"(parity)
        : "memory");
    return ok != 0;
}
// Waits for a phase of a barrier, for about a second at most. On a time-out, or when another role of the
// CTA has given up (*dead), returns false: the caller leaves its loop.
constexpr long long kWaitCycles = 2000000000ll;
__device__ __forceinline__ bool bar_wait(uint32_t bar, uint32_t parity, volatile int *dead) {
    if (bar_try(bar, parity)) return true;
    const long long t0 = clock64();
    while (!bar_try(bar, parity)) {
        if (*dead) return false;
        if (clock64() - t0 > kWaitCycles) {
            *dead = 1;
            return false;
        }
    }
    return true;
}
// The same when the kernel is giving up: nothing may stay in flight when it returns.
__device__ __forceinline__ void bar_drain(uint32_t bar, uint32_t parity) {
    const long long t0 = clock64();
    while (!bar_try(bar, parity) && clock64() - t0 < kWaitCycles) {
    }
}
__device__ __forceinline__ void tma_load(uint32_t dst, const CUtensorMap *map, uint32_t bar, int x, int y) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cta.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(dst),
        "l"(map), "r"(bar), "r"(x), "r"(y)
        : "memory");
}
__device__ __forceinline__ void tma_prefetch_map(const CUtensorMap *map) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(map) : "memory");
}
// An allocation waits until the SM has the columns. A kernel that is launched early (pdl_launch) holds what it
// allocates until the kernels before it have finished, so those must have allocated by then: a kernel calls
// pdl_launch after its allocation, on every CTA.
__device__ __forceinline__ void tmem_alloc(uint32_t smem_result, uint32_t cols) {  // one warp
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_result), "r"(cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_free(uint32_t tmem, uint32_t cols) {  // the same warp
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}
__device__ __forceinline__ void fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
// D (tensor memory) (+)= A B^T, both operands in shared memory, 16 values of k.
__device__ __forceinline__ void mma_f16(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, bool accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.u32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d),
        "l"(a), "l"(b), "r"(idesc), "r"((uint32_t)accumulate)
        : "memory");
}
// The same with A in tensor memory: lane = row, two values of k per column.
__device__ __forceinline__ void mma_f16_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, bool accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.u32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(d),
        "r"(a), "l"(b), "r"(idesc), "r"((uint32_t)accumulate)
        : "memory");
}
// Instruction descriptor: bf16 x bf16 -> fp32, both operands k-major.
__host__ __device__ constexpr uint32_t idesc_bf16(uint32_t m, uint32_t n) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((n >> 3) << 17) | ((m >> 4) << 24);
}
// Shared-memory descriptor of a k-major tile whose rows are one swizzle atom wide (row_bytes = 32, 64 or
// 128): groups of eight rows follow one another. Adding k * 32 bytes to the address moves along k.
__device__ __forceinline__ uint64_t smem_desc(uint32_t addr, uint32_t row_bytes) {
    const uint64_t swizzle = row_bytes == 128 ? 2 : row_bytes == 64 ? 4 : 6;
    return (uint64_t)((addr & 0x3ffff) >> 4) | (1ull << 16) | ((uint64_t)(row_bytes * 8 >> 4) << 32) | (1ull << 46) |
           (swizzle << 61);
}
// The same for an operand whose rows run along k (MN-major): rows of one swizzle atom of m or n values, all k
// rows of an atom in a row, `atom_stride` bytes from one atom to the next. Sixteen values of k are 16 *
// row_bytes apart. The instruction descriptor names such operands (a_mn, b_mn).
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr, uint32_t row_bytes, uint32_t atom_stride) {
    const uint64_t swizzle = row_bytes == 128 ? 2 : row_bytes == 64 ? 4 : 6;
    return (uint64_t)((addr & 0x3ffff) >> 4) | ((uint64_t)(atom_stride >> 4) << 16) | ((uint64_t)(row_bytes * 8 >> 4) << 32) |
           (1ull << 46) | (swizzle << 61);
}
__host__ __device__ constexpr uint32_t idesc_bf16_mn(uint32_t m, uint32_t n, bool a_mn, bool b_mn) {
    return idesc_bf16(m, n) | ((uint32_t)a_mn << 15) | ((uint32_t)b_mn << 16);
}
// 32 lanes x 32 columns of tensor memory, one register per column.
__device__ __forceinline__ void tmem_ld32(uint32_t tmem, float *v) {
    uint32_t *r = reinterpret_cast<uint32_t *>(v);
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, "
        "[%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]),
          "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]),
          "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(tmem));
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_st16(uint32_t tmem, const float *v) {
    const uint32_t *r = reinterpret_cast<const uint32_t *>(v);
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(tmem),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
        "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
}
__device__ __forceinline__ void tmem_st32(uint32_t tmem, const uint32_t *r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};" ::"r"(
            tmem),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
        "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]),
        "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]),
        "r"(r[30]), "r"(r[31])
        : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_ld16(uint32_t tmem, float *v) {
    uint32_t *r = reinterpret_cast<uint32_t *>(v);
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(tmem));
}

}  // namespace umma
#endif
}  // namespace ctox
