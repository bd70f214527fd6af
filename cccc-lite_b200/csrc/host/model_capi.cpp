// A C harness over the registry, the models and the generation loops, for the command-line programs and the tests (ctypes).
#include "scheduler.h"

#include <cstring>

using namespace cccc;

#define HOST_EXPORT extern "C" __attribute__((visibility("default")))

namespace
{
void setErr(char* err, int err_len, const std::string& e)
{
    if (err && err_len > 0)
    {
        std::strncpy(err, e.c_str(), (size_t)err_len - 1);
        err[err_len - 1] = '\0';
    }
}

SamplerConfig samplerOf(float temperature, int top_k, float top_p, float rep, const int* banned, int n_banned)
{
    SamplerConfig s;
    s.temperature = temperature;
    s.top_k = top_k;
    s.top_p = top_p;
    s.repetition_penalty = rep;
    s.banned_ids.assign(banned, banned + n_banned);
    return s;
}
}    // namespace

// names of the architectures this library and those loaded beside it know, separated by blanks
HOST_EXPORT int cccc_model_architectures(char* out, int len)
{
    std::string all;
    for (const auto& n : ModelRegistry::names()) { all += (all.empty() ? "" : " ") + n; }
    setErr(out, len, all);
    return (int)all.size();
}

HOST_EXPORT void* cccc_model_open(const char* dir, int device, int dtype, int max_context, int max_sequences, int max_step_tokens, int noise, char* err,
    int err_len)
{
    ModelOptions o;
    o.dir = dir;
    o.device = device;
    o.dtype = (DataType)dtype;
    o.max_context = max_context;
    o.max_sequences = max_sequences;
    o.max_step_tokens = max_step_tokens;
    o.noise_weights = noise != 0;
    std::string e;
    std::unique_ptr<LanguageModel> m = ModelRegistry::create(o, &e);
    if (!m) { setErr(err, err_len, e); }
    return m.release();
}
HOST_EXPORT void cccc_model_close(void* m) { delete (LanguageModel*)m; }
// what: 0 vocabulary, 1 rows of a cache slot, 2 cache slots, 3 launches of the last step, 4 weight bytes, 5 cache bytes
HOST_EXPORT unsigned long long cccc_model_info(void* m, int what)
{
    auto* l = (LanguageModel*)m;
    switch (what)
    {
    case 0: return (unsigned long long)l->vocab();
    case 1: return (unsigned long long)l->cache().rows();
    case 2: return (unsigned long long)l->cache().slots();
    case 3: return (unsigned long long)l->launchesLastStep();
    case 4: return l->weightBytes();
    case 5: return l->cache().bytes();
    default: return 0;
    }
}
HOST_EXPORT int cccc_model_open_slot(void* m) { return ((LanguageModel*)m)->cache().open(); }
HOST_EXPORT void cccc_model_close_slot(void* m, int slot) { ((LanguageModel*)m)->cache().close(slot); }
HOST_EXPORT int cccc_model_slot_length(void* m, int slot) { return ((LanguageModel*)m)->cache().length(slot); }

// n_entries entries: slot[e], n_tokens[e] of `tokens`, n_want[e] of `want` (one entry behind the other).
HOST_EXPORT int cccc_model_step(void* m, int n_entries, const int* slot, const int* n_tokens, const int* tokens, const int* n_want, const int* want,
    float* logits, int* choice)
{
    std::vector<StepEntry> entries((size_t)n_entries);
    for (int e = 0; e < n_entries; e++)
    {
        entries[e].slot = slot[e];
        entries[e].tokens.assign(tokens, tokens + n_tokens[e]);
        entries[e].want.assign(want, want + n_want[e]);
        tokens += n_tokens[e];
        want += n_want[e];
    }
    return ((LanguageModel*)m)->step(entries, logits, choice);
}

HOST_EXPORT float cccc_model_time_step(void* m, int entries, int tokens, int context, int inner, int repeat)
{
    return ((LanguageModel*)m)->timeStep(entries, tokens, context, inner, repeat);
}

// One sequence through the generation loop; gen: eos_n, eos ids..., think_open, think_close, sys_n, turn_n, T, T_kv.  Returns
// the number of ids (out gets up to out_cap), -1 when a step failed.  stats = rebuilds, decode steps, prefill tokens.
HOST_EXPORT int cccc_model_generate(void* m, int* ctx, int n_ctx, const int* gen, float temperature, int top_k, float top_p, float rep, const int* banned,
    int n_banned, unsigned int seed, int max_new, int portion, int* out, int out_cap, int* stats)
{
    GenerateConfig g;
    const int n = gen[0];
    g.eos_ids.assign(gen + 1, gen + 1 + n);
    const int* r = gen + 1 + n;
    g.think_open_id = r[0];
    g.think_close_id = r[1];
    g.sys_n = r[2];
    g.turn_n = r[3];
    g.T = r[4];
    g.T_kv = r[5];
    g.sampler = samplerOf(temperature, top_k, top_p, rep, banned, n_banned);
    std::vector<int> c(ctx, ctx + n_ctx);
    GenerateStats s;
    bool failed = false;
    const std::vector<int> got = generateWith(*(LanguageModel*)m, c, g, seed, max_new, portion, &s, &failed);
    if (failed) { return -1; }
    for (size_t i = 0; i < got.size() && i < (size_t)out_cap; i++) { out[i] = got[i]; }
    if (stats)
    {
        stats[0] = s.rebuilds;
        stats[1] = s.decode_steps;
        stats[2] = s.prefill_tokens;
    }
    return (int)got.size();
}

// Many prompts through the scheduler, all with one sampler (seeds seed, seed + 1, ...).  out: [n][max_new], n_out: tokens of
// each (-1: rejected).  Returns the steps it took, -1 when one failed.
HOST_EXPORT int cccc_model_generate_many(void* m, int n, const int* n_prompt, const int* prompts, float temperature, int top_k, float top_p, float rep,
    const int* banned, int n_banned, const int* eos, int n_eos, unsigned int seed, int max_new, int step_tokens, int* out, int* n_out)
{
    Scheduler s(*(LanguageModel*)m, step_tokens);
    for (int i = 0; i < n; i++)
    {
        Scheduler::Request r;
        r.prompt.assign(prompts, prompts + n_prompt[i]);
        prompts += n_prompt[i];
        r.sampler = samplerOf(temperature, top_k, top_p, rep, banned, n_banned);
        r.eos_ids.assign(eos, eos + n_eos);
        r.max_new = max_new;
        r.seed = seed + (unsigned int)i;
        s.submit(std::move(r));
    }
    while (s.step()) {}
    if (s.failed()) { return -1; }
    for (int i = 0; i < n; i++)
    {
        const auto& r = s.result(i);
        n_out[i] = r.rejected ? -1 : (int)r.tokens.size();
        for (size_t k = 0; k < r.tokens.size(); k++) { out[(size_t)i * max_new + k] = r.tokens[k]; }
    }
    return s.steps();
}
