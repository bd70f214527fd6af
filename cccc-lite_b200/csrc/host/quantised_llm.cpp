// The quantised cccc LLM (DecodeStep) behind the LanguageModel interface, for the registry, the scheduler and the command
// line.  config.json: {"architecture": "cccc-llm", "hidden", "n_heads", "n_kv_heads", "head_dim", "ffn", "vocab", "layers",
// "rope_theta", "eps", "qk_norm", and optionally "weights" (container file, default model.bin) and "weight_data_type"
// ("fp8_e4m3", "fp8_e5m2", "fp4_e2m1": quantise while loading)}.  Prompts go through the decode step token by token, as the
// generation loop of this model always did; sequences that decode together share a step.
#include "decode_step.h"
#include "language_model.h"

#include <algorithm>
#include <cstring>

namespace cccc
{

namespace
{
class QuantisedLlm : public LanguageModel
{
public:
    bool load(const ModelOptions& o, const Json& c, std::string* err)
    {
        if (o.dtype != BFLOAT16) { return fail(err, "this model runs in bfloat16 activations only"); }
        if (o.noise_weights) { return fail(err, "this model needs its weight file"); }
        ModelConfig m;
        m.hidden = (int)c["hidden"].number();
        m.n_heads = (int)c["n_heads"].number();
        m.n_kv_heads = (int)c["n_kv_heads"].number();
        m.head_dim = (int)c["head_dim"].number();
        m.ffn = (int)c["ffn"].number();
        m.vocab = (int)c["vocab"].number();
        m.layers = (int)c["layers"].number();
        m.rope_theta = (float)c["rope_theta"].number(10000.0);
        m.eps = (float)c["eps"].number(1e-6);
        m.qk_norm = c["qk_norm"].boolean();
        m.max_context = o.max_context;
        const std::string& t = c["weight_data_type"].string();
        if (t == "fp8_e4m3") { m.weight_data_type = FP8_E4M3; }
        else if (t == "fp8_e5m2") { m.weight_data_type = FP8_E5M2; }
        else if (t == "fp4_e2m1") { m.weight_data_type = FP4_E2M1; }
        else if (!t.empty()) { return fail(err, "no weight_data_type '" + t + "'"); }
        if (m.n_heads <= 0 || m.n_kv_heads <= 0 || m.ffn <= 0 || m.vocab <= 0) { return fail(err, "config.json lacks a size"); }
        const std::string path = o.dir + "/" + (c.has("weights") ? c["weights"].string() : "model.bin");
        BinFile f;
        if (gpu_.init(o.device) != 0) { return fail(err, "cannot open CUDA device " + std::to_string(o.device)); }
        if (!f.open(path)) { return fail(err, "cannot open '" + path + "'"); }
        vocab_ = m.vocab;
        batch_ = std::min(o.max_sequences, 32);
        return step_.load(&gpu_, f, m, batch_, nullptr, 0, err);
    }
    int vocab() const override { return vocab_; }
    KvCache& cache() override { return step_.cache(); }
    int launchesLastStep() const override { return launches_; }
    size_t weightBytes() const override { return step_.weightBytes(); }

    int step(const std::vector<StepEntry>& entries, float* logits, int* choice) override
    {
        if (!valid(entries)) { return -1; }
        launches_ = 0;
        std::vector<size_t> first(entries.size());
        size_t wanted = 0, longest = 0;
        for (size_t e = 0; e < entries.size(); e++)
        {
            first[e] = wanted;
            wanted += entries[e].want.size();
            longest = std::max(longest, entries[e].tokens.size());
        }
        std::vector<uint16_t> row(logits ? (size_t)batch_ * vocab_ : 0);
        for (size_t i = 0; i < longest; i++)    // the i-th tokens of all entries that have one
        {
            std::vector<int> ids, pos, slot, next;
            std::vector<size_t> owner;
            bool any = false;
            for (size_t e = 0; e < entries.size(); e++)
            {
                if (i >= entries[e].tokens.size()) { continue; }
                ids.push_back(entries[e].tokens[i]);
                slot.push_back(entries[e].slot);
                pos.push_back(cache().length(entries[e].slot));
                owner.push_back(e);
                any = any || std::count(entries[e].want.begin(), entries[e].want.end(), (int)i);
            }
            next.resize(ids.size());
            if (step_.step(ids.data(), pos.data(), (int)ids.size(), next.data(), nullptr, logits && any ? row.data() : nullptr, slot.data()) != 0) { return 1; }
            launches_ += step_.lastLaunches();
            for (size_t k = 0; k < owner.size(); k++)
            {
                const StepEntry& E = entries[owner[k]];
                cache().setLength(E.slot, pos[k] + 1);
                for (size_t w = 0; w < E.want.size(); w++)
                {
                    if (E.want[w] != (int)i) { continue; }
                    if (choice) { choice[first[owner[k]] + w] = next[k]; }
                    for (int v = 0; logits && v < vocab_; v++)
                    {
                        const uint32_t u = (uint32_t)row[k * vocab_ + v] << 16;
                        std::memcpy(logits + (first[owner[k]] + w) * vocab_ + v, &u, 4);
                    }
                }
            }
        }
        return 0;
    }

private:
    static bool fail(std::string* err, const std::string& what)
    {
        if (err) { *err = what; }
        return false;
    }
    GpuControl gpu_;
    DecodeStep step_;
    int vocab_ = 0, batch_ = 1, launches_ = 0;
};

const bool g_registered = ModelRegistry::add("cccc-llm", [](const ModelOptions& o, const Json& config, std::string* err) {
    std::unique_ptr<QuantisedLlm> m(new QuantisedLlm());
    if (!m->load(o, config, err)) { m.reset(); }
    return std::unique_ptr<LanguageModel>(std::move(m));
});
}    // namespace

}    // namespace cccc
