// The mLSTM recurrence: parameters and pieces shared by its kernels.
#pragma once

#include "decoder_common.cuh"

namespace b200
{

// State of a (slot, head): S [dim][v_ld], n [n_ld], m.
__host__ __device__ __forceinline__ unsigned int mlstm_v_ld(unsigned int vdim) { return (vdim + 3) / 4 * 4; }
__host__ __device__ __forceinline__ unsigned int mlstm_n_ld(unsigned int dim) { return (dim + 3) / 4 * 4; }
__host__ __device__ __forceinline__ size_t mlstm_state_floats(unsigned int dim, unsigned int vdim)
{
    return (size_t)dim * mlstm_v_ld(vdim) + mlstm_n_ld(dim) + 4;
}

struct MlstmParams
{
    const void* qkvg;
    const float *gates, *bias, *norm;
    void* out;
    float *state, *work;
    const int *slot, *pos, *start, *n, *token_entry;
    unsigned int ld, ld_gates, ldo, k_off, v_off, g_off, f_off;
    unsigned int heads, dim, vdim;
    unsigned int e0, t0, entries, tokens, max_n;
    float cap, eps, q_scale;
};

// mlstm_step.cu, mlstm_chunk.cu (BF16): -1 where the sizes are not taken
int launch_mlstm_step(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl);
int launch_mlstm_chunk(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl);
bool mlstm_chunk_takes(unsigned int dim, unsigned int vdim);
unsigned long long mlstm_chunk_floats(unsigned int tokens, unsigned int entries, unsigned int heads, unsigned int dim, unsigned int vdim);

__device__ __forceinline__ float log_sigmoid_f32(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// Logarithms of the input and the forget gate of a token's head.
__device__ __forceinline__ void mlstm_gates(const MlstmParams& p, unsigned int token, unsigned int head, float& in, float& forget)
{
    const float* g = p.gates + (size_t)token * p.ld_gates;
    in = p.cap * tanhf((g[head] + p.bias[head]) / p.cap);
    forget = log_sigmoid_f32(p.cap * tanhf((g[p.f_off + head] + p.bias[p.heads + head]) / p.cap));
}

__device__ __forceinline__ float* mlstm_state_of(const MlstmParams& p, unsigned int e, unsigned int head)
{
    return p.state + ((size_t)p.slot[e] * p.heads + head) * mlstm_state_floats(p.dim, p.vdim);
}

}    // namespace b200
