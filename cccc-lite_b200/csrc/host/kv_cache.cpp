#include "kv_cache.h"

namespace cccc
{

KvCache::~KvCache()
{
    for (auto& l : layers_)
    {
        gpu_->free(l.k);
        gpu_->free(l.v);
        gpu_->free(l.state);
    }
}

bool KvCache::init(GpuControl* gpu, const std::vector<KvLayerShape>& layers, int elem_bytes, int slots, int rows, std::string* err)
{
    gpu_ = gpu;
    rows_ = rows;
    length_.assign((size_t)slots, 0);
    open_.assign((size_t)slots, false);
    for (const auto& s : layers)
    {
        Layer l;
        l.k_ld = (s.k_dim + 15) / 16 * 16;
        l.v_ld = (s.v_dim + 15) / 16 * 16;
        const size_t per = (size_t)slots * s.kv_heads * rows * elem_bytes;
        l.k_bytes = per * l.k_ld;
        l.v_bytes = per * l.v_ld;
        l.state_bytes = (size_t)slots * s.state_floats * 4;
        if (l.k_bytes) { l.k = gpu->malloc(l.k_bytes); }
        if (l.v_bytes) { l.v = gpu->malloc(l.v_bytes); }
        if (l.state_bytes) { l.state = (float*)gpu->malloc(l.state_bytes); }
        layers_.push_back(l);
        if ((l.k_bytes && !l.k) || (l.v_bytes && !l.v) || (l.state_bytes && !l.state))
        {
            if (err) { *err = "no device memory for the KV cache"; }
            return false;
        }
        bytes_ += l.k_bytes + l.v_bytes + l.state_bytes;
    }
    clear();
    return true;
}

int KvCache::open()
{
    for (int s = 0; s < slots(); s++)
    {
        if (!open_[s])
        {
            open_[s] = true;
            length_[s] = 0;
            return s;
        }
    }
    return -1;
}

void KvCache::close(int slot)
{
    if (!isOpen(slot)) { return; }
    open_[slot] = false;
    length_[slot] = 0;
}

void KvCache::clear()
{
    gpu_->setAsCurrent();
    for (auto& l : layers_)
    {
        if (l.k) { cudaMemsetAsync(l.k, 0, l.k_bytes, gpu_->stream()); }
        if (l.v) { cudaMemsetAsync(l.v, 0, l.v_bytes, gpu_->stream()); }
        if (l.state) { cudaMemsetAsync(l.state, 0, l.state_bytes, gpu_->stream()); }
    }
    for (auto& n : length_) { n = 0; }
    gpu_->synchronize();
}

}    // namespace cccc
