// A decoder given as a list of layers: each a mixer (attention with separate key and value sizes) and a feed-forward
// (dense, or a mixture of experts with an optional shared one), over a residual stream in float.  Weights are BF16 (or, in
// the float mode, floats).  What a design fixes or configures is data here - a DecoderSpec that the design's own file
// builds from its config.json; the kernels are those of include/cccc_b200_decoder.h.
//
// Launches per layer of a decode step: norm (which first adds the experts' outputs of the layer before), q+k+v+gate,
// append, attention (which applies the output gate), o (added to the stream), norm, then up and down, or router, choice,
// gate+up of the chosen experts and the shared one, down of both.
#pragma once

#include "language_model.h"
#include "tensor_source.h"

#include "../../../include/cccc_b200_decoder.h"

#include <map>

namespace cccc
{

struct AttentionSpec
{
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1.0f;
    bool qk_norm = false;    // q and k heads to unit RMS
    bool v_mix = false;      // mix in the values of the first layer that has this set
    std::string q, k, v, o;    // tensor names
    std::string gate, vmix;    // empty: no output gate; no mixing factor
};

struct ExpertSpec
{
    int ff = 0;
    std::string gate, up, down;
};

struct MlpSpec
{
    enum Kind
    {
        NONE,
        DENSE,    // down(act(up x))
        MOE       // gated experts: down(silu(gate x) * up x)
    } kind = NONE;
    int activation = B200_ACT_RELU2;    // of the dense form
    ExpertSpec dense;
    int top = 0;
    std::string router;
    std::vector<ExpertSpec> experts;    // one size
    ExpertSpec shared;                  // ff 0: none
    std::string shared_gate;
};

struct LayerSpec
{
    std::string norm1, norm2;    // weights; with ".b" added, the biases of a layer norm
    AttentionSpec mixer;
    MlpSpec mlp;
};

struct DecoderSpec
{
    int vocab = 0, width = 0;
    float embed_scale = 1.0f, logit_scale = 1.0f, eps = 1e-5f;
    int norm_kind = B200_NORM_LAYER;
    std::string embed, head, final_norm;    // head: the embedding's name where the table is shared
    std::vector<LayerSpec> layers;
};

class LayeredDecoder : public LanguageModel
{
public:
    LayeredDecoder() = default;
    ~LayeredDecoder() override;
    bool load(const ModelOptions& o, const DecoderSpec& spec, TensorSource& source, std::string* err);

    int vocab() const override { return spec_.vocab; }
    KvCache& cache() override { return cache_; }
    int step(const std::vector<StepEntry>& entries, float* logits, int* choice) override;
    int launchesLastStep() const override { return last_launches_; }
    size_t weightBytes() const override { return weight_bytes_; }
    float timeStep(int entries, int tokens, int context, int inner, int repeat) override;

private:
    struct Weight
    {
        void* w = nullptr;
        int rows = 0, k = 0, ld = 0;
    };
    struct Norm
    {
        float *w = nullptr, *b = nullptr;
    };
    struct Layer
    {
        Norm norm1, norm2;
        Weight qkvg, o;
        int k_off = 0, v_off = 0, g_off = 0, n_qkvg = 0;
        int v_mix = 0;    // 1: the first mixing layer, 2: a later one
        float lambda = 0.f;
        Weight up, down;                                 // dense
        Weight router, experts_in, experts_out;          // experts one below the other: gate rows, then up rows
        Weight shared_in, shared_out;
    };
    // One pass: a ragged batch in the device's step arrays, laid out one behind the other.
    struct Pass
    {
        int tokens = 0, entries = 0, wants = 0, max_n = 0, max_len = 0;
        bool decode = false;    // one wanted token per entry
        std::vector<int> host;
    };
    const int* devIds(const Pass&) const { return d_meta_; }
    const int* devTokenEntry(const Pass& p) const { return d_meta_ + p.tokens; }
    const int* devEntries(const Pass& p, int field) const { return d_meta_ + 2 * p.tokens + field * p.entries; }
    const int* devWants(const Pass& p) const { return d_meta_ + 2 * p.tokens + 4 * p.entries; }

    bool check(std::string* err) const;
    bool loadTensors(TensorSource& s, std::string* err);
    bool allocate(const ModelOptions& o, std::string* err);
    bool packRows(TensorSource& s, const std::vector<std::pair<std::string, int>>& parts, int k, int align, Weight* out, std::string* err);
    bool loadNorm(TensorSource& s, const std::string& name, Norm* out, std::string* err);
    void* dmalloc(size_t bytes, bool zero);
    void makePass(const std::vector<StepEntry>& entries, const std::vector<int>& from, const std::vector<int>& count, Pass* p) const;
    int issue(const Pass& p, cudaStream_t st);          // the whole pass; launches, or -1
    int issueHead(const Pass& p, int row0, int rows, cudaStream_t st);
    int run(const Pass& p, float* logits, int* choice);
    size_t elem() const { return dtype_ == FLOAT ? 4 : 2; }
    int act() const { return dtype_ == FLOAT ? 0 : 3; }

    GpuControl gpu_;
    KvCache cache_;
    DecoderSpec spec_;
    DataType dtype_ = BFLOAT16;
    std::vector<Layer> layers_;
    Weight embed_, head_;
    Norm final_norm_;
    size_t weight_bytes_ = 0;
    int cap_ = 0, want_cap_ = 0;    // tokens a pass takes; wanted rows the head takes at once
    int ldw_ = 0, ld_qkvg_ = 0, ld_att_ = 0, ld_ff_ = 0, ld_eff_ = 0, ld_router_ = 0, ld_logits_ = 0, ld_first_ = 0, top_ = 0, max_experts_ = 0;
    float* x_ = nullptr;
    void *xn_ = nullptr, *qkvg_ = nullptr, *att_ = nullptr, *v_first_ = nullptr, *ff_ = nullptr, *ff_shared_ = nullptr;
    float* router_logits_ = nullptr;
    void *moe_x_ = nullptr, *moe_h_ = nullptr, *moe_y_ = nullptr;
    int *pair_row_ = nullptr, *row_token_ = nullptr, *choice_ = nullptr, *counters_ = nullptr, *group_offset_ = nullptr, *active_ = nullptr;
    float *pair_weight_ = nullptr, *shared_weight_ = nullptr;
    void* head_x_ = nullptr;
    float* logits_ = nullptr;
    int* d_choice_ = nullptr;
    float* d_best_ = nullptr;
    void* attn_work_ = nullptr;
    int* d_meta_ = nullptr;
    int* h_meta_ = nullptr;
    int* h_choice_ = nullptr;
    float* h_logits_ = nullptr;
    std::map<std::pair<int, int>, std::pair<cudaGraphExec_t, int>> graphs_;    // (entries, length bucket) -> graph, launches
    int last_launches_ = 0;
};

}    // namespace cccc
