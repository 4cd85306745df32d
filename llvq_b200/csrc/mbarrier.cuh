// Shared-memory barriers and the bulk copies that complete on them. Every wait is bounded: a caller that sees `false`
// records it and leaves.
#pragma once

namespace llvq {

constexpr unsigned int kPipeSpinLimit = 1u << 22;

__device__ __forceinline__ unsigned int pipe_smem_addr(const void* p) {
    return (unsigned int)__cvta_generic_to_shared(p);
}

// Bounded wait for the phase of the given parity of an mbarrier; false when the spin limit ran out.
__device__ __forceinline__ bool pipe_mbar_wait(unsigned int bar, unsigned int parity = 0) {
    unsigned int done = 0;
    for (unsigned int spin = 0; spin < kPipeSpinLimit && !done; ++spin) {
        asm volatile(
            "{\n\t.reg .pred p;\n\t"
            "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
            "selp.u32 %0, 1, 0, p;\n\t}"
            : "=r"(done)
            : "r"(bar), "r"(parity)
            : "memory");
    }
    return done != 0;
}

__device__ __forceinline__ void pipe_expect_tx(unsigned int bar, unsigned int bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void pipe_bulk_copy(unsigned int dst, const void* src, unsigned int bytes, unsigned int bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst),
                 "l"(src), "r"(bytes), "r"(bar)
                 : "memory");
}

__device__ __forceinline__ void mbar_init(unsigned int bar, unsigned int arrivals) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(arrivals));
}
__device__ __forceinline__ void mbar_init_fence() { asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory"); }

}  // namespace llvq
