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
    const int *slot, *pos, *start, *n, *token_entry;
    unsigned int ld, ldo, k_off, v_off, g_off, v_first_ld;
    unsigned int H, Hkv, G, dim, vdim, k_ld, v_ld, T_max;
    unsigned int splits, row_tiles;
    int v_mix, qk_norm, gate;
    int fused;    // the attention kernel itself brings q and k to unit RMS, mixes v and appends (one token per sequence)
    float lambda, eps, scale;
};

constexpr unsigned int kAttnCounters = 4096, kAttnPartials = 2048;

bool plan_splits(AttnParams& p, unsigned int entries, unsigned int max_len, unsigned int ctas_per_sm);
// attention_direct.cu, attention_mma.cu: -1 where the sizes are not taken
int launch_attention_direct(const AttnParams& p, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl);
// attention_tile.cu
int launch_attention_tile(const AttnParams& p, unsigned int slots, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl);
int launch_attention_split(const AttnParams& p, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl);
int launch_attention_tiled(const AttnParams& p, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl);

}    // namespace b200
