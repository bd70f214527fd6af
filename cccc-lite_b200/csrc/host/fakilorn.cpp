// Fakilorn: attention without positions over unit-RMS queries and keys, values mixed with the first layer's, a sigmoid
// output gate; dense squared-ReLU or mixture-of-experts feed-forwards; layer norms; a scaled, shared embedding table.
// Reads config.json into a DecoderSpec; everything else is LayeredDecoder.
#include "design_config.h"

namespace cccc
{

namespace
{
ExpertSpec expert(const std::string& prefix, int ff) { return { ff, prefix + ".gate", prefix + ".up", prefix + ".down" }; }

bool readSpec(const Json& c, DecoderSpec* s, std::string* err)
{
    if (!c["layers"].size() || c["embedding"]["scale"].type() != Json::NUMBER || c["norm"]["eps"].type() != Json::NUMBER
        || c["logit_scale"].type() != Json::NUMBER)
    {
        return configError(err, "vocab, width, embedding.scale, norm.eps, logit_scale and layers are needed");
    }
    s->vocab = (int)c["vocab"].number();
    s->width = (int)c["width"].number();
    s->embed_scale = (float)c["embedding"]["scale"].number();
    s->logit_scale = (float)c["logit_scale"].number();
    s->eps = (float)c["norm"]["eps"].number();
    s->norm_kind = B200_NORM_LAYER;
    s->embed = s->head = "embed";
    s->final_norm = "final.norm";
    for (size_t i = 0; i < c["layers"].size(); i++)
    {
        const Json& j = c["layers"][i];
        const std::string at = "layers[" + std::to_string(i) + "]", p = "l" + std::to_string(i);
        if (j["type"].string() != "attention") { return configError(err, at + ": no mixer of type '" + j["type"].string() + "'"); }
        LayerSpec L;
        L.norm1 = p + ".norm1";
        L.norm2 = p + ".norm2";
        const Json& m = j["mixer"];
        warnUnknown(m, at + ".mixer", { "heads", "kv_heads", "dim", "vdim", "scale", "v_mix" });
        if (m["scale"].type() != Json::NUMBER) { return configError(err, at + ": mixer.scale is needed"); }
        AttentionSpec& a = L.attention;
        a.heads = (int)m["heads"].number();
        a.kv_heads = (int)m["kv_heads"].number();
        a.dim = (int)m["dim"].number();
        a.vdim = (int)m["vdim"].number();
        a.scale = (float)m["scale"].number();
        a.v_mix = m["v_mix"].boolean();
        a.qk_norm = true;
        a.q = p + ".mix.q";
        a.k = p + ".mix.k";
        a.v = p + ".mix.v";
        a.o = p + ".mix.o";
        a.gate = p + ".mix.g";
        a.vmix = p + ".mix.vmix";
        const Json& f = j["mlp"];
        const std::string kind = f["kind"].string();
        if (f.isNull()) { L.mlp.kind = MlpSpec::NONE; }
        else if (kind == "dense")
        {
            warnUnknown(f, at + ".mlp", { "kind", "ff" });
            L.mlp.kind = MlpSpec::DENSE;
            L.mlp.activation = B200_ACT_RELU2;
            L.mlp.dense = { (int)f["ff"].number(), "", p + ".mlp.up", p + ".mlp.down" };
        }
        else if (kind == "moe")
        {
            warnUnknown(f, at + ".mlp", { "kind", "router", "expert", "shared" });
            warnUnknown(f["router"], at + ".mlp.router", { "experts", "top" });
            warnUnknown(f["expert"], at + ".mlp.expert", { "ff" });
            warnUnknown(f["shared"], at + ".mlp.shared", { "ff" });
            L.mlp.kind = MlpSpec::MOE;
            L.mlp.top = (int)f["router"]["top"].number();
            L.mlp.router = p + ".mlp.router";
            for (int e = 0; e < (int)f["router"]["experts"].number(); e++)
            {
                L.mlp.experts.push_back(expert(p + ".mlp.e" + std::to_string(e), (int)f["expert"]["ff"].number()));
            }
            if (!f["shared"].isNull())
            {
                L.mlp.shared = expert(p + ".mlp.shared", (int)f["shared"]["ff"].number());
                if (L.mlp.shared.ff <= 0) { return configError(err, at + ": mlp.shared.ff must be positive"); }
                L.mlp.shared_gate = p + ".mlp.shared.sg";
            }
        }
        else { return configError(err, at + ": no feed-forward of kind '" + kind + "'"); }
        s->layers.push_back(L);
    }
    return true;
}

const bool g_registered = registerLayered("Fakilorn", readSpec);
}    // namespace

}    // namespace cccc
