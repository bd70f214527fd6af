#include "language_model.h"

namespace cccc
{

bool LanguageModel::valid(const std::vector<StepEntry>& entries)
{
    std::vector<bool> seen((size_t)cache().slots(), false);
    for (const auto& e : entries)
    {
        if (!cache().isOpen(e.slot) || seen[e.slot] || cache().length(e.slot) + (int)e.tokens.size() > cache().rows()
            || e.want.size() > e.tokens.size())
        {
            return false;
        }
        seen[e.slot] = true;
        for (int t : e.tokens)
        {
            if (t < 0 || t >= vocab()) { return false; }
        }
        for (int w : e.want)
        {
            if (w < 0 || w >= (int)e.tokens.size()) { return false; }
        }
    }
    return true;
}

static std::map<std::string, ModelFactory>& registry()
{
    static std::map<std::string, ModelFactory> r;
    return r;
}

bool ModelRegistry::add(const std::string& architecture, ModelFactory f)
{
    registry()[architecture] = std::move(f);
    return true;
}

std::vector<std::string> ModelRegistry::names()
{
    std::vector<std::string> n;
    for (const auto& m : registry()) { n.push_back(m.first); }
    return n;
}

std::unique_ptr<LanguageModel> ModelRegistry::create(const ModelOptions& o, std::string* err)
{
    std::string text, e;
    Json config;
    const std::string path = o.dir + "/config.json";
    if (!readFile(path, &text))
    {
        if (err) { *err = "cannot read '" + path + "'"; }
        return nullptr;
    }
    if (!Json::parse(text, &config, &e))
    {
        if (err) { *err = "'" + path + "': " + e; }
        return nullptr;
    }
    const std::string& name = config["architecture"].string();
    auto it = registry().find(name);
    if (it == registry().end())
    {
        if (err)
        {
            *err = "no model class for architecture '" + name + "'; known:";
            for (const auto& m : registry()) { *err += " " + m.first; }
        }
        return nullptr;
    }
    return it->second(o, config, err);
}

}    // namespace cccc
