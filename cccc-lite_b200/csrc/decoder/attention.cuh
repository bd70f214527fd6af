// Attention over a KV cache with separate key and value sizes: parameters shared by its kernels.
#pragma once

#include "decoder_common.cuh"

namespace b200
{

struct AttnParams
{
    void *qkvg, *out, *k_cache, *v_cache, *v_first;
    float* partial;    // [slots][16 * (vdim_pad + 2)]
    int* counter;      // [kAttnCounters], zero between launches
    const int *slot, *pos, *start, *n, *token_entry, *floor;
    const float *q_norm, *k_norm, *sink;
    const void* head_gate;
    const float2* rotary;    // (cos, sin) [T_max][rot_dims / 2]
    unsigned int ld, ldo, k_off, v_off, g_off, v_first_ld;
    unsigned int H, Hkv, G, dim, vdim, k_ld, v_ld, T_max;
    unsigned int splits, row_tiles;
    unsigned int e0, t0;        // first entry, first token of the launch
    unsigned int q_ld;          // elements from a query head to the next
    unsigned int rot_dims, window, ld_gate;
    int rot_interleaved;
    int v_mix, qk_norm, gate;
    int fused;    // the attention kernel itself brings q and k to unit RMS, mixes v and appends (one token per sequence)
    float lambda, eps, scale;
};

// The first key a row of entry e sees that sees none from `lim` on.
__device__ __forceinline__ unsigned int first_key(const AttnParams& p, unsigned int e, unsigned int lim)
{
    const unsigned int low = p.window != 0 && lim > p.window ? lim - p.window : 0u;
    return p.floor != nullptr ? max(low, (unsigned int)p.floor[e]) : low;
}

// What a head's output is multiplied by.
template <class T>
__device__ __forceinline__ float head_factor(const AttnParams& p, size_t token, unsigned int head)
{
    return p.head_gate != nullptr ? sigmoid_f32(Elem<T>::get(((const T*)p.head_gate)[token * p.ld_gate + head])) : 1.f;
}

constexpr unsigned int kAttnCounters = 4096, kAttnPartials = 2048;

bool plan_splits(AttnParams& p, unsigned int entries, unsigned int max_n, unsigned int max_len, unsigned int ctas_per_sm);
// attention_direct.cu, attention_mma.cu: -1 where the sizes are not taken
int launch_attention_direct(const AttnParams& p, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl);
// attention_latent.cu: k_cache is v_cache, one kv head
int launch_attention_latent(const AttnParams& p, unsigned int slots, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl);
// attention_tile.cu
int launch_attention_tile(const AttnParams& p, unsigned int slots, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl);
int launch_attention_split(const AttnParams& p, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl);
int launch_attention_tiled(const AttnParams& p, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl);

}    // namespace b200
