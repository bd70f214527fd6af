#include "design_config.h"

#include <cstdio>

namespace cccc
{

bool configError(std::string* err, const std::string& what)
{
    if (err) { *err = "config.json: " + what; }
    return false;
}

void warnUnknown(const Json& j, const std::string& where, const std::vector<std::string>& known)
{
    for (const auto& m : j.members())
    {
        bool found = false;
        for (const auto& k : known) { found = found || k == m.first; }
        if (!found) { std::fprintf(stderr, "config.json: %s%s%s is not known and ignored\n", where.c_str(), where.empty() ? "" : ".", m.first.c_str()); }
    }
}

bool registerLayered(const std::string& architecture, SpecReader read)
{
    return ModelRegistry::add(architecture, [read](const ModelOptions& o, const Json& config, std::string* err) {
        std::unique_ptr<LayeredDecoder> m(new LayeredDecoder());
        DecoderSpec spec;
        if (!read(config, &spec, err)) { return std::unique_ptr<LanguageModel>(); }
        if (o.noise_weights)
        {
            NoiseSource noise(1);
            if (!m->load(o, spec, noise, err)) { m.reset(); }
        }
        else
        {
            SafetensorsFile file;
            if (!file.open(o.dir + "/model.safetensors", err) || !m->load(o, spec, file, err)) { m.reset(); }
        }
        return std::unique_ptr<LanguageModel>(std::move(m));
    });
}

}    // namespace cccc
