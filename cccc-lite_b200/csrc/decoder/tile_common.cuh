// Pieces the tcgen05 kernels of attention and the mLSTM share.
#pragma once

#include "../gemm_stream.cuh"
#include "decoder_common.cuh"

namespace b200
{

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
__device__ __forceinline__ float exp2_f32(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

}    // namespace b200
