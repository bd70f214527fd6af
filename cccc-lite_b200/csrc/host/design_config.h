// What the readers of designs' config.json files share.
#pragma once

#include "layered_decoder.h"

namespace cccc
{

// *err = what; false
bool configError(std::string* err, const std::string& what);
// Members a reader does not know: said on stderr, since the model may mean something by them.
void warnUnknown(const Json& j, const std::string& where, const std::vector<std::string>& known);
using SpecReader = bool (*)(const Json& config, DecoderSpec* spec, std::string* err);
// A LayeredDecoder of what `read` makes of config.json, with weights from model.safetensors (or seeded noise).
bool registerLayered(const std::string& architecture, SpecReader read);

}    // namespace cccc
