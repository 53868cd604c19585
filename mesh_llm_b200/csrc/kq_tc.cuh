// tcgen05 building blocks of the 16-bit kernels: shared-memory descriptors under the 128-byte swizzle, MMAs of
// kind::f16 with f32 accumulators in TMEM, and TMEM loads and stores.
#pragma once
#include "kq_common.cuh"

#include <cuda.h> // CUtensorMap

b200_status kq_tmap_encode(void *map128, int elem_bytes, int rank, const void *base, const uint64_t *dims,
                           const uint64_t *strides_bytes, const uint32_t *box, int swizzle128);

#ifdef __CUDACC__
__device__ __forceinline__ uint32_t smem_u32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ uint64_t tc_desc(uint32_t saddr, uint32_t lbo, uint32_t sbo) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr & 0x3FFFF) >> 4);
    d |= (uint64_t)(lbo >> 4) << 16;
    d |= (uint64_t)(sbo >> 4) << 32;
    d |= (uint64_t)1 << 46; // descriptor version of this architecture
    d |= (uint64_t)2 << 61; // SWIZZLE_128B
    return d;
}
// Waits of a pipeline.  The common case is a few tries; only a wait that lasts looks at the clock (reading %globaltimer
// costs more than a usual wait) and at the CTA's give-up word, and after limit_ns sets that word and the error word.
__device__ __forceinline__ bool tc_wait(uint32_t bar, uint32_t parity, volatile int *give_up, int *error_word, int code, uint64_t limit_ns) {
#pragma unroll 1
    for (int i = 0; i < 32; i++)
        if (kq_mbar_try(bar, parity)) return true;
    const uint64_t t0 = kq_globaltimer_ns();
    while (!kq_mbar_try(bar, parity)) {
        if (*give_up) return false;
        if (kq_globaltimer_ns() - t0 > limit_ns) {
            *give_up = 1;
            atomicExch(error_word, code);
            return false;
        }
    }
    return true;
}
// one lane of a converged warp
__device__ __forceinline__ bool tc_elect() {
    uint32_t ok;
    asm volatile("{\n\t.reg .pred p;\n\telect.sync _|p, 0xffffffff;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(ok));
    return ok != 0;
}
// K-major operand: rows of 128 bytes (64 elements), 8-row groups 1024 bytes apart; K step s of 16 elements
__device__ __forceinline__ uint64_t tc_desc_k(uint32_t tile, int s) { return tc_desc(tile + s * 32, 16, 1024); }
// MN-major operand: 64-element atoms `atom_bytes` apart, groups of 8 K rows 1024 bytes apart; K step s of 16 rows
__device__ __forceinline__ uint64_t tc_desc_mn(uint32_t tile, uint32_t atom_bytes, int s) { return tc_desc(tile + s * 2048, atom_bytes, 1024); }
// kind::f16 with f32 accumulation; bf16: both operands bf16 (else f16); b_mn: B is MN-major
__device__ __forceinline__ constexpr uint32_t tc_idesc(int m, int n, bool bf16, bool b_mn) {
    return (1u << 4) | (bf16 ? (1u << 7) | (1u << 10) : 0u) | ((b_mn ? 1u : 0u) << 16) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}
__device__ __forceinline__ void tc_mma_ss(uint32_t d_tmem, uint64_t a, uint64_t b, uint32_t id, uint32_t acc) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
                 :
                 : "r"(d_tmem), "l"(a), "l"(b), "r"(id), "r"(acc)
                 : "memory");
}
__device__ __forceinline__ void tc_mma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b, uint32_t id, uint32_t acc) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
                 :
                 : "r"(d_tmem), "r"(a_tmem), "l"(b), "r"(id), "r"(acc)
                 : "memory");
}
__device__ __forceinline__ void tc_commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}

#define TMEM_LD16(taddr, r)                                                                                             \
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];" \
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),      \
                   "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]) \
                 : "r"(taddr)                                                                                           \
                 : "memory")
#define TMEM_LD32(taddr, r)                                                                                             \
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"        \
                 "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"                              \
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),      \
                   "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), \
                   "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]),            \
                   "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]),            \
                   "=r"(r[30]), "=r"(r[31])                                                                             \
                 : "r"(taddr)                                                                                           \
                 : "memory")
#define TMEM_ST32(taddr, r)                                                                                             \
    asm volatile("tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"  \
                 "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"                                     \
                 :                                                                                                      \
                 : "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),  \
                   "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),         \
                   "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),       \
                   "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])        \
                 : "memory")
#define TMEM_ST16(taddr, r)                                                                                             \
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" \
                 :                                                                                                      \
                 : "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),  \
                   "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])          \
                 : "memory")
#endif
