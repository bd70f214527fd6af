// Pieces the tcgen05 kernels of attention and the mLSTM share.
#pragma once

#include "../gemm_stream.cuh"
#include "decoder_common.cuh"

namespace b200
{

// (A descriptor's address field counts sixteen bytes: adding n >> 4 to a descriptor moves it on by n bytes.)
// An MN-major operand [k][64 elements] with the 128-byte swizzle: 8-k groups 1024 bytes apart, 64-element blocks of 64 rows (8192
// bytes) one behind the other.
__device__ __forceinline__ uint64_t umma_desc_mnmajor_sw128(uint32_t smem_addr)
{
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
    d |= (uint64_t)(8192 >> 4) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// Has the phase of this parity completed?  Does not wait (a try_wait may, for a while).
__device__ __forceinline__ bool mbar_test(uint64_t* bar, uint32_t parity)
{
    uint32_t ok;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.test_wait.parity.acquire.cta.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(ok)
        : "r"(smem_u32(bar)), "r"(parity)
        : "memory");
    return ok != 0;
}
__device__ __forceinline__ float exp2_f32(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

}    // namespace b200
