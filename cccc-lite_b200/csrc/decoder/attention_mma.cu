// Which instance of the mma.sync attention kernels a launch takes, and how far the sequences are split.
#include "attention_mma.cuh"

namespace b200
{

template <>
int attention_split_dk<64>(const AttnParams&, unsigned int, cudaStream_t, bool);
template <>
int attention_split_dk<128>(const AttnParams&, unsigned int, cudaStream_t, bool);
template <>
int attention_split_dk<256>(const AttnParams&, unsigned int, cudaStream_t, bool);
template <>
int attention_tiled_dk<64>(const AttnParams&, unsigned int, unsigned int, cudaStream_t, bool);
template <>
int attention_tiled_dk<128>(const AttnParams&, unsigned int, unsigned int, cudaStream_t, bool);
template <>
int attention_tiled_dk<256>(const AttnParams&, unsigned int, unsigned int, cudaStream_t, bool);

int launch_attention_split(const AttnParams& p0, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl)
{
    AttnParams p = p0;
    if (p.dim > 256 || p.vdim > 256 || entries > 65535u) { return -1; }
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return 1; }
    p.row_tiles = (max_n * p.G + 15) / 16;
    const unsigned long long units = (unsigned long long)entries * p.Hkv * p.row_tiles;
    if ((unsigned long long)p.Hkv * p.row_tiles > 65535ull) { return -1; }
    // two CTAs per SM, at least 64 keys (a tile per warp) in a split
    unsigned int s = 1;
    if (units <= kAttnCounters)
    {
        const unsigned long long want = (2ull * dev->sm_count + units - 1) / units, most = ((unsigned long long)max_len + 63) / 64;
        s = (unsigned int)(want < most ? want : most);
        if (s > 64) { s = 64; }
        while (s > 1 && units * s > kAttnPartials) { s--; }
        if (s == 0) { s = 1; }
    }
    p.splits = s;
    if (p.dim <= 64) { return attention_split_dk<64>(p, entries, stream, pdl); }
    if (p.dim <= 128) { return attention_split_dk<128>(p, entries, stream, pdl); }
    return attention_split_dk<256>(p, entries, stream, pdl);
}

int launch_attention_tiled(const AttnParams& p, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl)
{
    if (p.dim > 256 || p.vdim > 256 || entries > 65535u || p.Hkv > 65535u) { return -1; }
    if (p.dim <= 64) { return attention_tiled_dk<64>(p, entries, max_n, stream, pdl); }
    if (p.dim <= 128) { return attention_tiled_dk<128>(p, entries, max_n, stream, pdl); }
    return attention_tiled_dk<256>(p, entries, max_n, stream, pdl);
}

}    // namespace b200
