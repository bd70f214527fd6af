// Shared pieces of the decoder-layer kernels: element type traits, launch helper, the epilogue of the linears.
#pragma once

#include "../../../include/cccc_b200_decoder.h"
#include "../common.cuh"

#include <atomic>
#include <cstring>

namespace b200
{

// The status word of this library's bounded waits (device memory, allocated once per device); nullptr on failure.
unsigned int* decoder_status_word();
// What the status word says of the first wait that ran out: which kernel, which of its roles, at which of the role's steps.
enum : unsigned int
{
    WAIT_LINEAR_TILE = 1,
    WAIT_ATTENTION_TILE = 2,
    WAIT_MLSTM_STATES = 3,
    WAIT_MLSTM_OUTPUTS = 4,
    WAIT_ATTENTION_LATENT = 5
};
__device__ __forceinline__ void note_timeout(unsigned int* status, unsigned int kernel, unsigned int role, unsigned int step)
{
    atomicCAS(status, 0u, kernel << 28 | role << 24 | (step & 0xFFFFFFu));
}

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

__host__ __device__ __forceinline__ bool activation_gated(int activation) { return activation == B200_ACT_SILU_GATE || activation == B200_ACT_GELU_GATE; }

// sigmoid by the hardware's exponential and reciprocal (a few units in the last place), for results that become BF16
__device__ __forceinline__ float sigmoid_fast(float z)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(-1.44269504088896341f * z));
    return __fdividef(1.0f, 1.0f + y);
}

// The part of a linear's epilogue that does not depend on where the result goes.  GELU in its tanh form: (1 + tanh u) / 2 is the sigmoid
// of 2u.
template <int ACT, bool FAST>
__device__ __forceinline__ float activate(float a, float up, float cap)
{
    if constexpr (ACT == B200_ACT_RELU2)
    {
        a = fmaxf(a, 0.f);
        return a * a;
    }
    else if constexpr (ACT == B200_ACT_SILU_GATE) { return a * (FAST ? sigmoid_fast(a) : sigmoid_f32(a)) * up; }
    else if constexpr (ACT == B200_ACT_GELU_GATE)
    {
        const float u = 0.7978845608028654f * (a + 0.044715f * a * a * a);
        return FAST ? a * sigmoid_fast(2.0f * u) * up : 0.5f * a * (1.0f + tanhf(u)) * up;
    }
    else if constexpr (ACT == B200_ACT_SOFTCAP) { return cap * tanhf(a / cap); }
    else { return a; }
}
template <bool FAST>
__device__ __forceinline__ float linear_activation(int activation, float a, float up, float cap)
{
    switch (activation)
    {
    case B200_ACT_RELU2: return activate<B200_ACT_RELU2, FAST>(a, up, cap);
    case B200_ACT_SILU_GATE: return activate<B200_ACT_SILU_GATE, FAST>(a, up, cap);
    case B200_ACT_GELU_GATE: return activate<B200_ACT_GELU_GATE, FAST>(a, up, cap);
    case B200_ACT_SOFTCAP: return activate<B200_ACT_SOFTCAP, FAST>(a, up, cap);
    default: return a;
    }
}

// Element d of a head after its first `dims` elements have been turned pair by pair (element i goes with i + dims / 2, or,
// interleaved, 2i with 2i + 1); rot: (cos, sin) of the position's angles.
__device__ __forceinline__ float rotated(const float* head, unsigned int d, unsigned int dims, bool interleaved, const float2* rot)
{
    if (d >= dims) { return head[d]; }
    const unsigned int half = dims / 2, i = interleaved ? d / 2 : d % half;
    const bool second = interleaved ? (d & 1u) != 0 : d >= half;
    const float2 cs = rot[i];
    const float u = head[interleaved ? 2 * i : i], v = head[interleaved ? 2 * i + 1 : i + half];
    return second ? v * cs.x + u * cs.y : u * cs.x - v * cs.y;
}

// Once per kernel (its own `done`) and device: of an SM's memory, a quarter as shared memory is enough.
template <class K>
static void prefer_l1(K kernel, std::atomic<unsigned long long>& done)
{
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64 || (done.load(std::memory_order_relaxed) >> dev & 1ull)) { return; }
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, 25) != cudaSuccess) { cudaGetLastError(); }
    done.fetch_or(1ull << dev, std::memory_order_relaxed);
}

// A launch in clusters of `cluster` CTAs along x (1: none).
template <class K, class... Args>
static int launch_cluster(const char* label, K kernel, dim3 grid, dim3 block, size_t smem, unsigned int cluster, void* stream, bool pdl, Args... args)
{
    if (smem > 24 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
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
    cudaLaunchAttribute attr[2];
    cfg.attrs = attr;
    if (pdl)
    {
        attr[cfg.numAttrs].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[cfg.numAttrs++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 8 && cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) != cudaSuccess)
    {
        report_launch(label);
        return 1;
    }
    if (cluster > 1)
    {
        attr[cfg.numAttrs].id = cudaLaunchAttributeClusterDimension;
        attr[cfg.numAttrs].val.clusterDim.x = cluster;
        attr[cfg.numAttrs].val.clusterDim.y = 1;
        attr[cfg.numAttrs++].val.clusterDim.z = 1;
    }
    count_launch();
    if (cudaLaunchKernelEx(&cfg, kernel, args...) != cudaSuccess)
    {
        report_launch(label);
        return 1;
    }
    return 0;
}

template <class K, class... Args>
static int launch_kernel(const char* label, K kernel, dim3 grid, dim3 block, size_t smem, void* stream, bool pdl, Args... args)
{
    return launch_cluster(label, kernel, grid, block, smem, 1, stream, pdl, args...);
}

}    // namespace b200
