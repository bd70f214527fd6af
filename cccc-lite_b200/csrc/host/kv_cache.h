// What a decoder keeps of its live sequences, one slot each: per layer a key and a value array [slot][kv head][row][elements]
// (or one array, where values are read from the key rows), or a recurrent state of fixed size, in floats.  Slots are handed out
// and taken back here; their lengths say how many rows count.  A sequence of length 0 starts from an empty state, whatever its
// slot's state memory holds.
#pragma once

#include "cccc_host.h"

#include <string>
#include <vector>

namespace cccc
{

struct KvLayerShape
{
    int kv_heads = 0, k_dim = 0, v_dim = 0;    // v_dim 0: no value array
    size_t state_floats = 0;                   // per slot
};

class KvCache
{
public:
    KvCache() = default;
    ~KvCache();
    KvCache(const KvCache&) = delete;
    KvCache& operator=(const KvCache&) = delete;
    // elem_bytes 2 or 4.  Rows are padded to sixteen elements; the padding is zero and stays so.
    bool init(GpuControl* gpu, const std::vector<KvLayerShape>& layers, int elem_bytes, int slots, int rows, std::string* err);
    void* k(int layer) const { return layers_[layer].k; }
    void* v(int layer) const { return layers_[layer].v; }
    float* state(int layer) const { return layers_[layer].state; }
    int kLd(int layer) const { return layers_[layer].k_ld; }
    int vLd(int layer) const { return layers_[layer].v_ld; }
    int slots() const { return (int)length_.size(); }
    int rows() const { return rows_; }
    size_t bytes() const { return bytes_; }
    int open();              // a free slot of length 0, or -1
    void close(int slot);    // gives the slot back
    bool isOpen(int slot) const { return slot >= 0 && slot < slots() && open_[slot]; }
    int length(int slot) const { return length_[slot]; }
    void setLength(int slot, int n) { length_[slot] = n; }
    void clear();            // zeroes the memory (on the device's stream) and every length

private:
    struct Layer
    {
        void *k = nullptr, *v = nullptr;
        float* state = nullptr;
        int k_ld = 0, v_ld = 0;
        size_t k_bytes = 0, v_bytes = 0, state_bytes = 0;
    };
    GpuControl* gpu_ = nullptr;
    std::vector<Layer> layers_;
    std::vector<int> length_;
    std::vector<bool> open_;
    int rows_ = 0;
    size_t bytes_ = 0;
};

}    // namespace cccc
