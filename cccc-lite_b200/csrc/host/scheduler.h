// Token generation over a LanguageModel: one sequence through the Generator loop, or many requests sharing the model's
// cache slots and steps.
#pragma once

#include "generate.h"
#include "language_model.h"

#include <deque>

namespace cccc
{

struct GenerateStats
{
    int rebuilds = 0, decode_steps = 0, prefill_tokens = 0;
};

// Generator (generate.h) over one cache slot of `m`, its prompts in portions of up to `portion` tokens.  ctx as there.
// Returns the generated ids; *failed is set when a step failed or no slot was free.
std::vector<int> generateWith(LanguageModel& m, std::vector<int>& ctx, const GenerateConfig& cfg, unsigned int seed, int max_new, int portion,
    GenerateStats* stats, bool* failed);

// Requests wait in order of arrival for a cache slot; every step carries one token of each sequence that decodes and, as
// far as the step's token budget goes, portions of the prompts that are still being read.
class Scheduler
{
public:
    struct Request
    {
        std::vector<int> prompt;
        SamplerConfig sampler;
        std::vector<int> eos_ids;
        int max_new = 16;
        unsigned int seed = 0;
    };
    struct Result
    {
        std::vector<int> tokens;    // EOS excluded
        bool rejected = false;      // empty, or longer than a cache slot
    };
    Scheduler(LanguageModel& m, int step_tokens) : m_(m), step_tokens_(step_tokens > 0 ? step_tokens : 1) {}
    int submit(Request r);              // the request's number
    bool step();                        // one step of the model; false when nothing is left to do, or on failure
    bool failed() const { return failed_; }
    int steps() const { return steps_; }
    const Result& result(int request) const { return results_[(size_t)request]; }

private:
    struct Live
    {
        int id = 0, slot = -1;
        Request r;
        size_t read = 0;    // prompt tokens already in the cache
        int next = -1;      // the token to decode
        std::vector<int> ctx;
        std::mt19937 rng;
    };
    LanguageModel& m_;
    int step_tokens_;
    std::deque<std::pair<int, Request>> waiting_;
    std::vector<Live> live_;
    std::vector<Result> results_;
    bool failed_ = false;
    int steps_ = 0;
};

}    // namespace cccc
