// What every served model offers - sequences in cache slots, steps over ragged batches of new tokens - and the registry
// that picks the model class by the architecture a model folder's config.json names.
#pragma once

#include "cccc_host.h"
#include "json.h"
#include "kv_cache.h"

#include <functional>
#include <memory>
#include <string>
#include <vector>

namespace cccc
{

// New tokens of one sequence: they continue what its slot holds.  `want`: places among them whose logits are asked for.
struct StepEntry
{
    int slot = -1;
    std::vector<int> tokens;
    std::vector<int> want;
};

class LanguageModel
{
public:
    virtual ~LanguageModel() = default;
    virtual int vocab() const = 0;
    virtual KvCache& cache() = 0;
    // Runs the entries' tokens.  For every wanted place, in the order of the entries and of `want`: logits (nullable) gets
    // a row of vocab() floats, choice (nullable) the id of the largest logit.  Returns 0; -1 for entries that cannot run
    // (a closed slot, one slot twice, a full cache, a token outside the vocabulary), nothing having run; 1 on a CUDA error.
    virtual int step(const std::vector<StepEntry>& entries, float* logits, int* choice) = 0;
    virtual int launchesLastStep() const { return 0; }
    virtual size_t weightBytes() const { return 0; }
    // Device time of one step in ms (the fastest of `repeat` runs of `inner` steps): `entries` sequences that hold `context`
    // tokens each get `tokens` more, with the logits of the last one.  < 0 where the model does not time itself.
    virtual float timeStep(int entries, int tokens, int context, int inner, int repeat)
    {
        (void)entries, (void)tokens, (void)context, (void)inner, (void)repeat;
        return -1.f;
    }

protected:
    // The checks of step() that every model needs.
    bool valid(const std::vector<StepEntry>& entries);
};

struct ModelOptions
{
    std::string dir;
    int device = 0;
    DataType dtype = BFLOAT16;      // FLOAT: everything in true 32-bit
    int max_context = 4096;         // rows of a cache slot
    int max_sequences = 1;          // cache slots
    int max_step_tokens = 4096;     // tokens one pass runs; longer steps run in several
    bool noise_weights = false;     // config.json only: seeded random weights
};

using ModelFactory = std::function<std::unique_ptr<LanguageModel>(const ModelOptions&, const Json& config, std::string* err)>;

class ModelRegistry
{
public:
    static bool add(const std::string& architecture, ModelFactory f);    // at static initialisation
    static std::vector<std::string> names();
    // Reads dir/config.json and makes the model its "architecture" names.
    static std::unique_ptr<LanguageModel> create(const ModelOptions& o, std::string* err);
};

}    // namespace cccc
