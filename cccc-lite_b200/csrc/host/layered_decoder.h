// A decoder given as a list of layers: each a mixer (attention with separate key and value sizes, latent attention, an mLSTM)
// and a feed-forward (dense, or a mixture of experts with an optional shared one), over a residual stream in float.  Weights are BF16 (or, in
// the float mode, floats).  What a design fixes or configures is data here - a DecoderSpec that the design's own file
// builds from its config.json; the kernels are those of include/cccc_b200_decoder.h.
//
// Launches per layer of a decode step: norm (which first adds what the sublayer before left pending: experts' outputs, or a
// branch with a norm of its own), the mixer, o (added to the stream, or left pending), norm, then up and down, or router,
// choice, gate+up of the chosen experts and the shared one, down of both.  The mixer is q+k+v+gate, append and attention (which
// applies the output gate); or, for latent attention, both down projections, their norms and the cache row, the queries, the
// queries against the latent (or, in prompts, keys and values of all heads from the cached latents), attention, the values'
// projection and gate; or q+k+v+gate with the recurrence's own gates beside them as floats, and the recurrence.
#pragma once

#include "language_model.h"
#include "tensor_source.h"

#include "../../../include/cccc_b200_decoder.h"

#include <map>

namespace cccc
{

struct RotarySpec
{
    int dims = 0;    // 0: no rotation
    double base = 0.0;
    bool interleaved = false;
};

struct AttentionSpec
{
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1.0f;
    bool qk_norm = false;    // q and k heads to unit RMS
    bool v_mix = false;      // mix in the values of the first layer that has this set
    int window = 0;          // a token sees itself and the window - 1 before it; 0: all
    RotarySpec rot;
    std::string q, k, v, o;    // tensor names; v empty: the values are the keys as projected
    std::string gate, vmix;    // empty: no output gate; no mixing factor
    std::string q_norm, k_norm;    // weights of norms over the whole projections; empty: none
    std::string sink;              // scores in the softmax denominator; empty: none
};

// Keys and values of all heads come from one latent per token; the cache holds it and a rotated key part.
struct LatentSpec
{
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, q_rank = 0, kv_rank = 0, window = 0;
    float scale = 1.0f;
    RotarySpec rot;
    std::string dq, q_norm, uq, dkv, kv_norm, uk, uv, o;
    std::string gate;    // one per head; empty: none
};

struct MlstmSpec
{
    int heads = 0, dim = 0, vdim = 0;
    float cap = 1.0f;
    std::string q, k, v, gate, o, norm;
    std::string input, forget;    // with ".b" added, their biases
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
        DENSE,    // down(act(up x)), or down(act(gate x) * up x) for a gated activation
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
    enum Kind
    {
        ATTENTION,
        LATENT,
        MLSTM
    } kind = ATTENTION;
    std::string norm1, norm2;      // weights; with ".b" added, the biases of a layer norm
    std::string norm1b, norm2b;    // of the mixer's and the feed-forward's output; empty: none
    AttentionSpec attention;
    LatentSpec latent;
    MlstmSpec mlstm;
    MlpSpec mlp;
    int weights_of = -1;           // the layer whose tensors this one uses (its cache or state is its own)
};

struct DecoderSpec
{
    int vocab = 0, width = 0;
    float embed_scale = 1.0f, logit_scale = 1.0f, eps = 1e-5f;
    float logit_softcap = 0.0f;    // cap * tanh(logit / cap); 0: none
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
        Norm norm1, norm2, norm1b, norm2b;
        Weight in, o;    // q, k, v and output gate; or the latents' down projections and the heads' gates
        int k_off = 0, v_off = 0, g_off = 0;
        float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr;
        const void* rotary = nullptr;
        Weight uq, absorb, uk, uv;     // latent: a head's queries every q_step columns; absorb: each head's W_uk transposed
        int q_step = 0;
        int gates = 0, f_off = 0;      // mLSTM: first row of the gates in `in`, and the forget gates' distance from it
        float *gate_bias = nullptr, *head_norm = nullptr;
        int v_mix = 0;    // 1: the first mixing layer, 2: a later one
        float lambda = 0.f;
        Weight up, down;                                 // dense (up: gate rows ahead of it where the activation is gated)
        Weight router, experts_in, experts_out;          // experts one below the other: gate rows, then up rows
        Weight shared_in, shared_out;
    };
    // Entries of a pass that take the same kernels: those with few tokens come first.
    struct Part
    {
        int first_entry = 0, entries = 0, first_token = 0, tokens = 0, max_n = 0, max_len = 0;
        bool few = false;
    };
    // One pass: a ragged batch in the device's step arrays, laid out one behind the other.
    struct Pass
    {
        int tokens = 0, entries = 0, wants = 0;
        bool decode = false;    // one wanted token per entry
        std::vector<Part> parts;
        std::vector<std::pair<int, int>> asked;    // per wanted place: entry and index among its wants
        std::vector<int> pos, n;                   // per entry
        std::vector<int> host;
    };
    // What a pass' launches share.
    struct Issue
    {
        const Pass& p;
        cudaStream_t st;
        int bad = 0, n = 0;
        void ok(int rc)
        {
            bad += rc != 0;
            n++;
        }
    };
    const int* devIds(const Pass&) const { return d_meta_; }
    const int* devTokenEntry(const Pass& p) const { return d_meta_ + p.tokens; }
    const int* devEntries(const Pass& p, int field) const { return d_meta_ + 2 * p.tokens + field * p.entries; }
    const int* devWants(const Pass& p) const { return d_meta_ + 2 * p.tokens + 4 * p.entries; }
    // floor and pos2 of the entries' expanded keys, for the w-th of windows_
    const int* devExpanded(const Pass& p, int w, int field) const { return d_meta_ + 2 * p.tokens + 4 * p.entries + p.wants + (2 * w + field) * p.entries; }

    bool check(std::string* err) const;
    bool loadTensors(TensorSource& s, std::string* err);
    bool allocate(const ModelOptions& o, std::string* err);
    struct Rows
    {
        std::string name;
        int rows = 0, pieces = 1;    // pieces of rows / pieces rows, each padded
    };
    bool packRows(TensorSource& s, const std::vector<Rows>& parts, int k, int align, Weight* out, std::string* err);
    // the transpose of each of `pieces` blocks [rows][k], one below the other
    bool packTransposed(TensorSource& s, const std::string& name, int pieces, int rows, int k, Weight* out, std::string* err);
    bool upload(const std::string& name, const std::vector<uint16_t>& bits, size_t first, int rows, int k, size_t at, const Weight& w, std::string* err);
    bool loadVector(TensorSource& s, const std::vector<std::pair<std::string, int>>& parts, float** out, std::string* err);
    bool loadLayer(TensorSource& s, const LayerSpec& ls, Layer* L, std::string* err);
    bool loadMixer(TensorSource& s, const LayerSpec& ls, Layer* L, std::string* err);
    bool checkMixer(const LayerSpec& ls, const std::string& at, int* mixed, std::string* err) const;
    const void* rotaryTable(const RotarySpec& r, int dims, std::string* err);
    bool loadNorm(TensorSource& s, const std::string& name, Norm* out, std::string* err);
    bool allocateMixers(const ModelOptions& o, std::string* err);
    void* dmalloc(size_t bytes, bool zero);
    void makePass(const std::vector<StepEntry>& entries, const std::vector<int>& from, const std::vector<int>& count, Pass* p) const;
    int issue(const Pass& p, cudaStream_t st);          // the whole pass; launches, or -1
    int issueHead(const Pass& p, int row0, int rows, cudaStream_t st);
    // layered_mixers.cpp: xn_ -> att_, all but the output projection
    void issueAttention(Issue& r, int layer);
    void issueLatent(Issue& r, int layer);
    void issueLatentExpanded(Issue& r, int layer, const cuda_b200_batch& part);
    void issueMlstm(Issue& r, int layer);
    cuda_b200_linear dense(const Issue& r, const Weight& w, const void* X, int ldx, void* Y, int ldy) const;
    cuda_b200_batch batchOf(const Pass& p, const Part& part) const;
    cuda_b200_batch wholeBatch(const Pass& p) const;
    int expandedFloor(const Pass& p, int window, std::vector<int>* floor, std::vector<int>* pos2) const;
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
    static constexpr int kFewTokens = 8;    // tokens up to which an entry takes the kernels for few tokens
    int max_context_ = 0;
    int cap_ = 0, want_cap_ = 0;    // tokens a pass takes; wanted rows the head takes at once
    int ldw_ = 0, ld_in_ = 0, ld_att_ = 0, ld_ff_ = 0, ld_eff_ = 0, ld_router_ = 0, ld_logits_ = 0, ld_first_ = 0, top_ = 0, max_experts_ = 0;
    float* x_ = nullptr;
    void *xn_ = nullptr, *in_ = nullptr, *att_ = nullptr, *v_first_ = nullptr, *ff_ = nullptr, *ff_shared_ = nullptr;
    float* branch_ = nullptr;    // an output projection whose result is normalised before it is added
    // latent attention: query latents, queries, queries against the latent and their outputs (few tokens), gathered latents and
    // expanded keys and values (prompts)
    int ld_cq_ = 0, ld_q_ = 0, ld_ql_ = 0, ld_ol_ = 0, ld_c_ = 0, few_cap_ = 0, expand_cap_ = 0;
    void *cq_ = nullptr, *q_ = nullptr, *ql_ = nullptr, *ol_ = nullptr, *c_ = nullptr, *k_exp_ = nullptr, *v_exp_ = nullptr;
    int* zero_slots_ = nullptr;
    std::vector<int> windows_;    // the windows that layers with expanded keys have
    int ld_gates_ = 0;
    float *gates_ = nullptr, *mlstm_work_ = nullptr;
    std::map<std::pair<int, double>, const void*> rotary_;    // (dims, base) -> table
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
