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

// How many splits a (sequence, kv head, row tile) is cut into: the least estimated time, a wave of CTAs taking a fixed part
// and a part that goes with the keys of a split.
bool plan_splits(AttnParams& p, unsigned int entries, unsigned int max_n, unsigned int max_len, unsigned int ctas_per_sm)
{
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return false; }
    if (p.window != 0 && max_len > p.window + max_n) { max_len = p.window + max_n; }
    p.splits = 1;
    const unsigned long long units = (unsigned long long)entries * p.Hkv * p.row_tiles, slots = (unsigned long long)dev->sm_count * ctas_per_sm;
    if (units > kAttnCounters) { return true; }
    double best = 1e30;
    for (unsigned int s = 1; s <= kMaxSplits && units * s <= kAttnPartials && (s == 1 || max_len / s >= 64); s++)
    {
        const unsigned long long waves = (units * s + slots - 1) / slots;
        const double t = (double)waves * (3.0 + (double)((max_len + s - 1) / s) * 0.012 * ctas_per_sm) + (s > 1 ? 1.5 + 0.06 * s : 0.0);
        if (t < best)
        {
            best = t;
            p.splits = s;
        }
    }
    return true;
}

int launch_attention_split(const AttnParams& p0, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl)
{
    AttnParams p = p0;
    if (p.dim > 256 || p.vdim > 256 || entries > 65535u) { return -1; }
    p.row_tiles = (max_n * p.G + 15) / 16;
    if ((unsigned long long)p.Hkv * p.row_tiles > 65535ull) { return -1; }
    if (!plan_splits(p, entries, max_n, max_len, 1)) { return 1; }
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
