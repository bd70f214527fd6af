// Tazunex: mLSTM, sliding-window attention with sinks over its own keys as values, and latent attention, in any order; gated
// GELU feed-forwards; RMS norms before and after each; a shared embedding table, capped logits; layers that share tensors.
// Reads config.json into a DecoderSpec; everything else is LayeredDecoder.
#include "design_config.h"

namespace cccc
{

namespace
{
bool positive(const Json& j, const std::vector<std::string>& names, const std::string& at, std::string* err)
{
    for (const auto& n : names)
    {
        if (j[n].type() != Json::NUMBER || j[n].number() <= 0) { return configError(err, (at.empty() ? "" : at + ".") + n + " must be positive"); }
    }
    return true;
}

bool readRotary(const Json& r, const std::string& at, bool interleaved, RotarySpec* out, std::string* err)
{
    warnUnknown(r, at, { "base", "dims" });
    if (!positive(r, { "base", "dims" }, at, err)) { return false; }
    out->base = r["base"].number();
    out->dims = (int)r["dims"].number();
    out->interleaved = interleaved;
    return true;
}

bool readMixer(const Json& j, const std::string& at, const std::string& p, LayerSpec* L, std::string* err)
{
    const std::string type = j["type"].string(), where = at + ".mixer", x = p + ".mix.";
    const Json& m = j["mixer"];
    auto num = [&](const char* n) { return (int)m[n].number(); };
    if (type == "mlstm")
    {
        warnUnknown(m, where, { "heads", "dim", "vdim", "gate_cap" });
        if (!positive(m, { "heads", "dim", "vdim", "gate_cap" }, where, err)) { return false; }
        L->kind = LayerSpec::MLSTM;
        MlstmSpec& s = L->mlstm;
        s.heads = num("heads");
        s.dim = num("dim");
        s.vdim = num("vdim");
        s.cap = (float)m["gate_cap"].number();
        s.q = x + "q";
        s.k = x + "k";
        s.v = x + "v";
        s.gate = x + "g";
        s.o = x + "o";
        s.norm = x + "norm";
        s.input = x + "i";
        s.forget = x + "f";
        return true;
    }
    if (type != "attention" && type != "latent_attention") { return configError(err, at + ": no mixer of type '" + type + "'"); }
    warnUnknown(m["mask"], where + ".mask", { "size" });
    if (!positive(m, { "heads", "dim", "vdim" }, where, err) || !positive(m["mask"], { "size" }, where + ".mask", err)) { return false; }
    if (m["scale"].type() != Json::NUMBER) { return configError(err, where + ".scale is needed"); }
    const int window = (int)m["mask"]["size"].number();
    if (type == "attention")
    {
        warnUnknown(m, where, { "heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot" });
        L->kind = LayerSpec::ATTENTION;
        AttentionSpec& s = L->attention;
        if (!positive(m, { "kv_heads" }, where, err) || !readRotary(m["rot"], where + ".rot", false, &s.rot, err)) { return false; }
        s.heads = num("heads");
        s.kv_heads = num("kv_heads");
        s.dim = num("dim");
        s.vdim = num("vdim");
        s.scale = (float)m["scale"].number();
        s.window = window;
        s.q = x + "q";
        s.k = x + "k";    // no v: the values are the keys as projected
        s.o = x + "o";
        s.q_norm = x + "q.norm";
        s.k_norm = x + "k.norm";
        s.sink = x + "sink";
        return true;
    }
    warnUnknown(m, where, { "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask", "rot" });
    L->kind = LayerSpec::LATENT;
    LatentSpec& s = L->latent;
    if (!positive(m, { "rot_dim", "q_rank", "kv_rank" }, where, err) || !readRotary(m["rot"], where + ".rot", true, &s.rot, err)) { return false; }
    s.heads = num("heads");
    s.dim = num("dim");
    s.rot_dim = num("rot_dim");
    s.vdim = num("vdim");
    s.q_rank = num("q_rank");
    s.kv_rank = num("kv_rank");
    s.scale = (float)m["scale"].number();
    s.window = window;
    s.dq = x + "dq";
    s.q_norm = x + "dq.norm";
    s.uq = x + "uq";
    s.dkv = x + "dkv";
    s.kv_norm = x + "dkv.norm";
    s.uk = x + "uk";
    s.uv = x + "uv";
    s.gate = x + "g";
    s.o = x + "o";
    return true;
}

bool readSpec(const Json& c, DecoderSpec* s, std::string* err)
{
    warnUnknown(c, "", { "architecture", "layers", "logit_softcap", "norm", "vocab", "width" });
    if (!positive(c, { "vocab", "width", "logit_softcap" }, "", err)) { return false; }
    if (!c["layers"].size() || c["norm"]["eps"].type() != Json::NUMBER) { return configError(err, "norm.eps and layers are needed"); }
    s->vocab = (int)c["vocab"].number();
    s->width = (int)c["width"].number();
    s->eps = (float)c["norm"]["eps"].number();
    s->logit_softcap = (float)c["logit_softcap"].number();
    s->norm_kind = B200_NORM_RMS;
    s->embed = s->head = "embed";
    s->final_norm = "final.norm";
    for (size_t i = 0; i < c["layers"].size(); i++)
    {
        const Json& j = c["layers"][i];
        const std::string at = "layers[" + std::to_string(i) + "]", p = "l" + std::to_string(i);
        warnUnknown(j, at, { "type", "mixer", "mlp", "weights_of" });
        LayerSpec L;
        L.norm1 = p + ".norm1";
        L.norm2 = p + ".norm2";
        L.norm1b = p + ".norm1b";
        L.norm2b = p + ".norm2b";
        if (!j["weights_of"].isNull()) { L.weights_of = (int)j["weights_of"].number(-2); }
        if (!readMixer(j, at, p, &L, err)) { return false; }
        const Json& f = j["mlp"];
        if (!f.isNull())
        {
            if (f["kind"].string() != "dense") { return configError(err, at + ": no feed-forward of kind '" + f["kind"].string() + "'"); }
            warnUnknown(f, at + ".mlp", { "kind", "ff" });
            if (!positive(f, { "ff" }, at + ".mlp", err)) { return false; }
            L.mlp.kind = MlpSpec::DENSE;
            L.mlp.activation = B200_ACT_GELU_GATE;
            L.mlp.dense = { (int)f["ff"].number(), p + ".mlp.gate", p + ".mlp.up", p + ".mlp.down" };
        }
        s->layers.push_back(L);
    }
    return true;
}

const bool g_registered = registerLayered("Tazunex", readSpec);
}    // namespace

}    // namespace cccc
