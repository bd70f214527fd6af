#include "scheduler.h"

#include <algorithm>

namespace cccc
{

std::vector<int> generateWith(LanguageModel& m, std::vector<int>& ctx, const GenerateConfig& cfg, unsigned int seed, int max_new, int portion,
    GenerateStats* stats, bool* failed)
{
    int slot = m.cache().open();
    *failed = slot < 0;
    if (*failed) { return {}; }
    auto feed = [&](const int* tokens, int n, bool want, std::vector<float>* logits) {
        StepEntry e;
        e.slot = slot;
        e.tokens.assign(tokens, tokens + n);
        if (want) { e.want = { n - 1 }; }
        if (logits) { logits->resize((size_t)m.vocab()); }
        int choice = -1;
        if (m.step({ e }, want && logits ? logits->data() : nullptr, want ? &choice : nullptr) != 0) { *failed = true; }
        return choice;
    };
    Generator g(
        m.vocab(), [&](int token, int, std::vector<float>* logits) { return *failed ? -1 : feed(&token, 1, true, logits); },
        [&]() {
            m.cache().close(slot);
            slot = m.cache().open();
        },
        seed);
    g.setPrefill([&](const std::vector<int>& tokens, std::vector<float>* logits) {
        int next = -1;
        if (logits) { logits->assign((size_t)m.vocab(), 0.f); }
        for (size_t at = 0; at < tokens.size() && !*failed; at += (size_t)portion)
        {
            const int n = (int)std::min((size_t)portion, tokens.size() - at);
            const bool last = at + (size_t)n == tokens.size();
            next = feed(tokens.data() + at, n, last, last ? logits : nullptr);
        }
        return next;
    });
    // a failed step ends the loop at once: no id of the model is negative
    GenerateConfig c = cfg;
    c.eos_ids.push_back(-1);
    std::vector<int> out = g.generate(ctx, c, max_new);
    m.cache().close(slot);
    if (stats) { *stats = { g.rebuilds(), g.decodeSteps(), g.prefillTokens() }; }
    return out;
}

int Scheduler::submit(Request r)
{
    const int id = (int)results_.size();
    results_.emplace_back();
    if (r.prompt.empty() || (int)r.prompt.size() > m_.cache().rows()) { results_.back().rejected = true; }
    else { waiting_.emplace_back(id, std::move(r)); }
    return id;
}

bool Scheduler::step()
{
    if (failed_) { return false; }
    while (!waiting_.empty())
    {
        Live l;
        l.slot = m_.cache().open();
        if (l.slot < 0) { break; }
        l.id = waiting_.front().first;
        l.r = std::move(waiting_.front().second);
        waiting_.pop_front();
        l.ctx = l.r.prompt;
        l.rng.seed(l.r.seed);
        live_.push_back(std::move(l));
    }
    if (live_.empty()) { return false; }
    std::vector<StepEntry> entries;
    std::vector<size_t> owner;
    int room = step_tokens_;
    bool logits_needed = false;
    for (int pass = 0; pass < 2; pass++)    // decoding sequences first
    {
        for (size_t i = 0; i < live_.size(); i++)
        {
            Live& l = live_[i];
            const bool reading = l.read < l.r.prompt.size();
            if (reading != (pass == 1) || room <= 0) { continue; }
            StepEntry e;
            e.slot = l.slot;
            if (reading)
            {
                const size_t n = std::min((size_t)room, l.r.prompt.size() - l.read);
                e.tokens.assign(l.r.prompt.begin() + (long)l.read, l.r.prompt.begin() + (long)(l.read + n));
                l.read += n;
                if (l.read == l.r.prompt.size()) { e.want = { (int)n - 1 }; }
            }
            else
            {
                e.tokens = { l.next };
                e.want = { 0 };
            }
            room -= (int)e.tokens.size();
            logits_needed = logits_needed || (!e.want.empty() && l.r.sampler.needsLogits());
            entries.push_back(std::move(e));
            owner.push_back(i);
        }
    }
    int wanted = 0;
    for (const auto& e : entries) { wanted += (int)e.want.size(); }
    std::vector<float> logits(logits_needed ? (size_t)wanted * m_.vocab() : 0);
    std::vector<int> choice((size_t)wanted);
    if (m_.step(entries, logits_needed ? logits.data() : nullptr, wanted ? choice.data() : nullptr) != 0)
    {
        failed_ = true;
        for (auto& l : live_) { m_.cache().close(l.slot); }
        live_.clear();
        return false;
    }
    steps_++;
    int at = 0;
    for (size_t k = 0; k < entries.size(); k++)
    {
        if (entries[k].want.empty()) { continue; }
        Live& l = live_[owner[k]];
        int id = choice[(size_t)at];
        if (l.r.sampler.needsLogits())
        {
            std::vector<float> row(logits.begin() + (long)at * m_.vocab(), logits.begin() + (long)(at + 1) * m_.vocab());
            id = sampleLogits(row, l.r.sampler, l.ctx, l.rng);
        }
        at++;
        Result& res = results_[(size_t)l.id];
        const bool eos = id < 0 || std::find(l.r.eos_ids.begin(), l.r.eos_ids.end(), id) != l.r.eos_ids.end();
        if (!eos && (int)res.tokens.size() < l.r.max_new)
        {
            res.tokens.push_back(id);
            l.ctx.push_back(id);
            l.next = id;
        }
        if (eos || (int)res.tokens.size() >= l.r.max_new || m_.cache().length(l.slot) >= m_.cache().rows())
        {
            m_.cache().close(l.slot);
            l.slot = -1;
        }
    }
    live_.erase(std::remove_if(live_.begin(), live_.end(), [](const Live& l) { return l.slot < 0; }), live_.end());
    return !live_.empty() || !waiting_.empty();
}

}    // namespace cccc
