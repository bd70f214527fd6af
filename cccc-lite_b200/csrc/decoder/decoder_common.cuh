// Shared pieces of the decoder-layer kernels: element type traits, launch helper, the epilogue of the linears.
#pragma once

#include "../../../include/cccc_b200_decoder.h"
#include "../common.cuh"

#include <cstring>

namespace b200
{

// The status word of this library's bounded waits (device memory, allocated once per device); nullptr on failure.
unsigned int* decoder_status_word();
struct DecoderDevice
{
    int sm_count = 0, max_smem = 0;
};
const DecoderDevice* decoder_device();

template <class T>
struct Elem;
template <>
struct Elem<float>
{
    static constexpr int type = DT_FLOAT;
    static __device__ __forceinline__ float get(float v) { return v; }
    static __device__ __forceinline__ float put(float v) { return v; }
};
template <>
struct Elem<__nv_bfloat16>
{
    static constexpr int type = DT_BF16;
    static __device__ __forceinline__ float get(__nv_bfloat16 v) { return __bfloat162float(v); }
    static __device__ __forceinline__ __nv_bfloat16 put(float v) { return __float2bfloat16_rn(v); }
};

__device__ __forceinline__ void grid_dependency_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void grid_dependency_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p)
{
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v)
{
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a);
    u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }

__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) { v += __shfl_xor_sync(0xFFFFFFFFu, v, o); }
    return v;
}

// The part of a linear's epilogue that does not depend on where the result goes.
__device__ __forceinline__ float linear_activation(int activation, float a, float up)
{
    if (activation == B200_ACT_RELU2)
    {
        a = fmaxf(a, 0.f);
        return a * a;
    }
    if (activation == B200_ACT_SILU_GATE) { return a * sigmoid_f32(a) * up; }
    return a;
}

template <class K, class... Args>
static int launch_kernel(const char* label, K kernel, dim3 grid, dim3 block, size_t smem, void* stream, bool pdl, Args... args)
{
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    {
        report_launch(label);
        return 1;
    }
    cudaLaunchConfig_t cfg;
    memset(&cfg, 0, sizeof(cfg));
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = (cudaStream_t)stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl ? 1 : 0;
    count_launch();
    if (cudaLaunchKernelEx(&cfg, kernel, args...) != cudaSuccess)
    {
        report_launch(label);
        return 1;
    }
    return 0;
}

}    // namespace b200
