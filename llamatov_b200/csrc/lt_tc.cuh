// Plumbing of the tensor-core kernels (tcgen05 + tensor memory + TMA): mbarriers with bounded waits, tiled loads,
// shared-memory operand descriptors, tensor-memory loads, the tensor-map encoder.
#pragma once
#include <cuda.h>

#include "lt_common.cuh"

namespace lt {
namespace tc {

constexpr long long WAIT_LIMIT = 3000000000LL;  // SM clocks (> 1 s) before a wait gives up

__device__ __forceinline__ unsigned smem_u32(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void mbar_init(unsigned long long* bar, unsigned count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(unsigned long long* bar, unsigned bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(unsigned long long* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(unsigned long long* bar, unsigned parity) {
    unsigned ok;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
    return ok != 0;
}

// Bounded wait.  *abort_flag (shared) is set by the first wait of the CTA that runs out of time;
// from then on every wait returns immediately so that all roles run to the end of their loops.
template <int SLEEP_NS = 0>
__device__ __forceinline__ void mbar_wait(unsigned long long* bar, unsigned parity, volatile int* abort_flag,
                                          int* status) {
    if (mbar_try_wait(bar, parity)) return;
    const long long t0 = clock64();
    while (!mbar_try_wait(bar, parity)) {
        if (SLEEP_NS > 0) __nanosleep(SLEEP_NS);
        if (*abort_flag) return;
        if (clock64() - t0 > WAIT_LIMIT) {
            *abort_flag = 1;
            atomicOr(status, LT_STATUS_WAIT_TIMEOUT);
            return;
        }
    }
}

__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, int x, int y, unsigned long long* bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(
            smem_u32(dst)),
        "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
        : "memory");
}

__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }

__device__ __forceinline__ void mma_commit(unsigned long long* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar))
                 : "memory");
}

// K-major shared-memory operand descriptor.  Rows are `row_bytes` apart inside an 8-row swizzle
// atom, atoms follow each other every 8*row_bytes (the stride byte offset); the leading byte
// offset is unused for swizzled K-major operands whose K extent fits the swizzle width.
template <int CB>
__device__ __forceinline__ unsigned long long smem_desc(unsigned addr) {
    constexpr unsigned long long layout = CB == 4 ? 2ull : (CB == 2 ? 4ull : 6ull);  // 128B / 64B / 32B swizzle
    constexpr unsigned long long sbo = (8ull * CB * 32ull) >> 4;
    return (unsigned long long)((addr >> 4) & 0x3FFFu) | (1ull << 16) | (sbo << 32) | (1ull << 46) | (layout << 61);
}

template <int CW>
__device__ __forceinline__ void tmem_ld(unsigned taddr, int (&v)[CW]);
template <>
__device__ __forceinline__ void tmem_ld<4>(unsigned taddr, int (&v)[4]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0,%1,%2,%3}, [%4];"
                 : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3])
                 : "r"(taddr));
}
template <>
__device__ __forceinline__ void tmem_ld<8>(unsigned taddr, int (&v)[8]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7])
                 : "r"(taddr));
}
template <>
__device__ __forceinline__ void tmem_ld<16>(unsigned taddr, int (&v)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]),
          "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
        : "r"(taddr));
}
// Completes the TMEM loads of this thread.  The loaded registers are passed through the
// statement (eight at a time) so that no use of them can be scheduled above the wait.
__device__ __forceinline__ void reg_fence4(int* v) {
    asm volatile("" : "+r"(v[0]), "+r"(v[1]), "+r"(v[2]), "+r"(v[3])::"memory");
}

// ---------------------------------------------------------------------------- host side

typedef CUresult (*encode_fn_t)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline encode_fn_t encode_fn() {
    static encode_fn_t fn = nullptr;
    if (fn == nullptr) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult qr;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &qr) == cudaSuccess &&
            qr == cudaDriverEntryPointSuccess)
            fn = (encode_fn_t)p;
    }
    return fn;
}

}  // namespace tc
}  // namespace lt
