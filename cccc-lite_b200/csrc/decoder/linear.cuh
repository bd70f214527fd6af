// One linear of a launch as the kernels see it, and where its results go.
#pragma once

#include "decoder_common.cuh"

namespace b200
{

constexpr unsigned int LINEAR_MAX_MEMBERS = 3;

struct LinearMember
{
    const void *W, *X;
    void* Y;
    const float* row_scale;
    const int *group_offset, *x_row, *active;
    const void* head_gate;           // of the launch's dtype
    float* Y_tail;
    unsigned int rows, N, K, ldw, ldx, ldy;
    unsigned int groups, group_rows, up_row;
    unsigned int blocks, x_step, y_step, ld_gate;    // block-diagonal: 1 or more
    unsigned int tail, ld_tail;      // first feature of the float tail (none: past all features)
    unsigned int slots;              // groups the launch walks: 1, the blocks, the groups, or the active list's length
    unsigned int block0, fblocks;    // streaming kernel: first CTA, CTAs per group
    int out_type, activation, accumulate;
    float alpha, cap;
};

// What a row of block `block` is multiplied by.
template <class T>
__device__ __forceinline__ float linear_row_factor(const LinearMember& m, unsigned int row, unsigned int block)
{
    float s = m.row_scale != nullptr ? m.row_scale[row] : 1.f;
    if (m.head_gate != nullptr) { s *= sigmoid_f32(Elem<T>::get(((const T*)m.head_gate)[(size_t)row * m.ld_gate + block])); }
    return s;
}

// f: column of Y (the block's first column included)
__device__ __forceinline__ void linear_store(const LinearMember& m, unsigned int row, unsigned int f, float v)
{
    if (f >= m.tail)
    {
        m.Y_tail[(size_t)row * m.ld_tail + f - m.tail] = v;
        return;
    }
    const size_t i = (size_t)row * m.ldy + f;
    if (m.out_type == DT_BF16) { ((__nv_bfloat16*)m.Y)[i] = __float2bfloat16_rn(v); }
    else if (m.accumulate) { ((float*)m.Y)[i] += v; }
    else { ((float*)m.Y)[i] = v; }
}

// linear_tile.cu: more than a few rows, tcgen05
int launch_linear_tile(const LinearMember& m, cudaStream_t stream, bool pdl);

}    // namespace b200
