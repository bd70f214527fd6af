#include "layered_decoder.h"

#include <algorithm>
#include <cstring>

namespace cccc
{

namespace
{
bool fail(std::string* err, const std::string& what)
{
    if (err) { *err = what; }
    return false;
}
int pad64(int n) { return (n + 63) / 64 * 64; }
float widen(uint16_t b)
{
    const uint32_t u = (uint32_t)b << 16;
    float f;
    std::memcpy(&f, &u, 4);
    return f;
}
constexpr int kStreamRows = 32;    // rows up to which the weight-streaming kernels (and the graphs) run a pass
}    // namespace

LayeredDecoder::~LayeredDecoder()
{
    if (gpu_.getDeviceID() < 0) { return; }
    gpu_.setAsCurrent();
    gpu_.synchronize();
    for (auto& g : graphs_) { cudaGraphExecDestroy(g.second.first); }
    if (h_meta_) { cudaFreeHost(h_meta_); }
    if (h_choice_) { cudaFreeHost(h_choice_); }
    if (h_logits_) { cudaFreeHost(h_logits_); }
}

void* LayeredDecoder::dmalloc(size_t bytes, bool zero)
{
    void* p = gpu_.malloc(bytes + 256);    // tiles may read a little past the last row
    if (p && zero) { cudaMemsetAsync(p, 0, bytes + 256, gpu_.stream()); }
    return p;
}

bool LayeredDecoder::check(std::string* err) const
{
    const DecoderSpec& s = spec_;
    if (s.vocab <= 0 || s.width <= 0 || s.layers.empty()) { return fail(err, "vocab, width and layers must be given"); }
    int mixed = -1;
    for (size_t i = 0; i < s.layers.size(); i++)
    {
        const AttentionSpec& a = s.layers[i].mixer;
        const std::string at = "layer " + std::to_string(i) + ": ";
        if (a.heads <= 0 || a.kv_heads <= 0 || a.dim <= 0 || a.vdim <= 0) { return fail(err, at + "heads, kv_heads, dim and vdim must be positive"); }
        if (a.heads % a.kv_heads) { return fail(err, at + "heads must be a multiple of kv_heads"); }
        if (a.v_mix)
        {
            if (mixed >= 0 && mixed != a.kv_heads * a.vdim) { return fail(err, at + "layers that mix values must have values of one size"); }
            mixed = a.kv_heads * a.vdim;
        }
        const MlpSpec& m = s.layers[i].mlp;
        if (m.kind == MlpSpec::DENSE && m.dense.ff <= 0) { return fail(err, at + "ff must be positive"); }
        if (m.kind == MlpSpec::MOE)
        {
            if (m.experts.empty() || m.top <= 0 || m.top > (int)m.experts.size()) { return fail(err, at + "top must lie between 1 and the number of experts"); }
            if (m.experts[0].ff <= 0 || m.shared.ff < 0) { return fail(err, at + "experts' ff must be positive"); }
        }
    }
    return true;
}

bool LayeredDecoder::load(const ModelOptions& o, const DecoderSpec& spec, TensorSource& source, std::string* err)
{
    spec_ = spec;
    dtype_ = o.dtype;
    if (dtype_ != BFLOAT16 && dtype_ != FLOAT) { return fail(err, "this model runs in bfloat16 or float32"); }
    if (!check(err)) { return false; }
    if (o.max_context <= 0 || o.max_sequences <= 0 || o.max_step_tokens <= 0) { return fail(err, "context, sequences and step tokens must be positive"); }
    if (gpu_.init(o.device) != 0) { return fail(err, "cannot open CUDA device " + std::to_string(o.device)); }
    cap_ = std::max(std::min(o.max_step_tokens, o.max_context * o.max_sequences), std::min(o.max_sequences, kStreamRows));
    if (!loadTensors(source, err) || !allocate(o, err)) { return false; }
    gpu_.synchronize();
    return cuda_b200_decoder_check("model load") == 0 ? true : fail(err, "a CUDA error while loading");
}

// Tensors [rows][k] one below the other, every one padded to a multiple of `align` rows; rows padded to 64 columns; zeros.
bool LayeredDecoder::packRows(TensorSource& s, const std::vector<std::pair<std::string, int>>& parts, int k, int align, Weight* out, std::string* err)
{
    size_t rows = 0;
    for (const auto& p : parts) { rows += (size_t)(p.second + align - 1) / align * align; }
    out->rows = (int)rows;
    out->k = k;
    out->ld = pad64(k);
    const size_t row_bytes = (size_t)out->ld * elem();
    out->w = dmalloc(rows * row_bytes, true);
    if (!out->w) { return fail(err, "no device memory for '" + parts[0].first + "'"); }
    gpu_.synchronize();
    std::vector<uint16_t> bits;
    std::vector<float> wide;
    size_t at = 0;
    for (const auto& p : parts)
    {
        if (!s.readBf16(p.first, { p.second, k }, &bits, err)) { return false; }
        const void* src = bits.data();
        if (dtype_ == FLOAT)
        {
            wide.resize(bits.size());
            for (size_t i = 0; i < bits.size(); i++) { wide[i] = widen(bits[i]); }
            src = wide.data();
        }
        if (cudaMemcpy2D((char*)out->w + at * row_bytes, row_bytes, src, (size_t)k * elem(), (size_t)k * elem(), (size_t)p.second, cudaMemcpyHostToDevice)
            != cudaSuccess)
        {
            return fail(err, "cannot copy '" + p.first + "' to the device");
        }
        weight_bytes_ += bits.size() * elem();
        at += (size_t)(p.second + align - 1) / align * align;
    }
    return true;
}

bool LayeredDecoder::loadNorm(TensorSource& s, const std::string& name, Norm* out, std::string* err)
{
    auto vec = [&](const std::string& n, float** dst) {
        std::vector<uint16_t> bits;
        if (!s.readBf16(n, { spec_.width }, &bits, err)) { return false; }
        std::vector<float> f(bits.size());
        for (size_t i = 0; i < f.size(); i++) { f[i] = widen(bits[i]); }
        *dst = (float*)dmalloc(f.size() * 4, false);
        if (!*dst || cudaMemcpy(*dst, f.data(), f.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess) { return fail(err, "no device memory for '" + n + "'"); }
        return true;
    };
    return vec(name, &out->w) && (spec_.norm_kind != B200_NORM_LAYER || vec(name + ".b", &out->b));
}

bool LayeredDecoder::loadTensors(TensorSource& s, std::string* err)
{
    const int W = spec_.width;
    if (!packRows(s, { { spec_.embed, spec_.vocab } }, W, 1, &embed_, err)) { return false; }
    head_ = embed_;
    if (spec_.head != spec_.embed && !packRows(s, { { spec_.head, spec_.vocab } }, W, 1, &head_, err)) { return false; }
    if (!loadNorm(s, spec_.final_norm, &final_norm_, err)) { return false; }
    bool mixing = false;
    layers_.resize(spec_.layers.size());
    for (size_t i = 0; i < layers_.size(); i++)
    {
        const LayerSpec& ls = spec_.layers[i];
        const AttentionSpec& a = ls.mixer;
        Layer& L = layers_[i];
        if (!loadNorm(s, ls.norm1, &L.norm1, err)) { return false; }
        std::vector<std::pair<std::string, int>> parts = { { a.q, a.heads * a.dim }, { a.k, a.kv_heads * a.dim }, { a.v, a.kv_heads * a.vdim } };
        if (!a.gate.empty()) { parts.emplace_back(a.gate, a.heads * a.vdim); }
        if (!packRows(s, parts, W, 8, &L.qkvg, err)) { return false; }
        auto pad8 = [](int n) { return (n + 7) / 8 * 8; };
        L.k_off = pad8(a.heads * a.dim);
        L.v_off = L.k_off + pad8(a.kv_heads * a.dim);
        L.g_off = L.v_off + pad8(a.kv_heads * a.vdim);
        L.n_qkvg = L.qkvg.rows;
        if (!packRows(s, { { a.o, W } }, a.heads * a.vdim, 1, &L.o, err)) { return false; }
        if (a.v_mix)
        {
            L.v_mix = mixing ? 2 : 1;
            mixing = true;
            if (L.v_mix == 2)
            {
                std::vector<uint16_t> b;
                if (!s.readBf16(a.vmix, {}, &b, err)) { return false; }
                L.lambda = widen(b[0]);
            }
        }
        const MlpSpec& m = ls.mlp;
        if (m.kind == MlpSpec::NONE) { continue; }
        if (!loadNorm(s, ls.norm2, &L.norm2, err)) { return false; }
        if (m.kind == MlpSpec::DENSE)
        {
            if (!packRows(s, { { m.dense.up, m.dense.ff } }, W, 1, &L.up, err) || !packRows(s, { { m.dense.down, W } }, m.dense.ff, 1, &L.down, err)) { return false; }
            continue;
        }
        parts = { { m.router, (int)m.experts.size() } };
        if (m.shared.ff) { parts.emplace_back(m.shared_gate, 1); }
        if (!packRows(s, parts, W, 1, &L.router, err)) { return false; }
        std::vector<std::pair<std::string, int>> in, out;
        for (const auto& e : m.experts)
        {
            in.emplace_back(e.gate, e.ff);
            in.emplace_back(e.up, e.ff);
            out.emplace_back(e.down, W);
        }
        if (!packRows(s, in, W, 1, &L.experts_in, err) || !packRows(s, out, m.experts[0].ff, 1, &L.experts_out, err)) { return false; }
        if (m.shared.ff
            && (!packRows(s, { { m.shared.gate, m.shared.ff }, { m.shared.up, m.shared.ff } }, W, 1, &L.shared_in, err)
                || !packRows(s, { { m.shared.down, W } }, m.shared.ff, 1, &L.shared_out, err)))
        {
            return false;
        }
    }
    return true;
}

bool LayeredDecoder::allocate(const ModelOptions& o, std::string* err)
{
    std::vector<KvLayerShape> shapes;
    int vdim = 0, qkvg = 0, att = 0, ff = 0, eff = 0, sff = 0, router = 0, first = 0;
    for (size_t i = 0; i < layers_.size(); i++)
    {
        const AttentionSpec& a = spec_.layers[i].mixer;
        const MlpSpec& m = spec_.layers[i].mlp;
        shapes.push_back({ a.kv_heads, a.dim, a.vdim });
        vdim = std::max(vdim, a.vdim);
        qkvg = std::max(qkvg, layers_[i].n_qkvg);
        att = std::max(att, a.heads * a.vdim);
        if (a.v_mix) { first = a.kv_heads * a.vdim; }
        if (m.kind == MlpSpec::DENSE) { ff = std::max(ff, m.dense.ff); }
        if (m.kind == MlpSpec::MOE)
        {
            eff = std::max(eff, m.experts[0].ff);
            sff = std::max(sff, m.shared.ff);
            router = std::max(router, layers_[i].router.rows);
            top_ = std::max(top_, m.top);
            max_experts_ = std::max(max_experts_, (int)m.experts.size());
        }
    }
    if (!cache_.init(&gpu_, shapes, (int)elem(), o.max_sequences, o.max_context, err)) { return false; }
    ldw_ = pad64(spec_.width);
    ld_qkvg_ = pad64(qkvg);
    ld_att_ = pad64(att);
    ld_ff_ = pad64(std::max(ff, sff));
    ld_eff_ = pad64(std::max(eff, 1));
    ld_router_ = pad64(std::max(router, 1));
    ld_logits_ = pad64(spec_.vocab);
    ld_first_ = pad64(std::max(first, 1));
    want_cap_ = std::min(cap_, 256);
    const size_t T = (size_t)cap_, P = T * top_, e = elem();
    bool ok = true;
    auto get = [&](size_t bytes) {
        void* p = dmalloc(bytes, true);
        ok = ok && p;
        return p;
    };
    x_ = (float*)get(T * ldw_ * 4);
    xn_ = get(T * ldw_ * e);
    qkvg_ = get(T * ld_qkvg_ * e);
    att_ = get(T * ld_att_ * e);
    v_first_ = get(T * ld_first_ * e);
    ff_ = get(T * ld_ff_ * e);
    if (top_)
    {
        router_logits_ = (float*)get(T * ld_router_ * 4);
        moe_x_ = get(P * ldw_ * e);
        moe_h_ = get(P * ld_eff_ * e);
        moe_y_ = get(P * ldw_ * e);
        pair_row_ = (int*)get(P * 4);
        row_token_ = (int*)get(P * 4);
        choice_ = (int*)get(P * 4);
        pair_weight_ = (float*)get(P * 4);
        shared_weight_ = (float*)get(T * 4);
        counters_ = (int*)get((size_t)max_experts_ * 4);
        group_offset_ = (int*)get((size_t)(max_experts_ + 1) * 4);
        active_ = (int*)get((size_t)max_experts_ * 4);
    }
    head_x_ = get((size_t)want_cap_ * ldw_ * e);
    logits_ = (float*)get((size_t)want_cap_ * ld_logits_ * 4);
    d_choice_ = (int*)get((size_t)want_cap_ * 4);
    d_best_ = (float*)get((size_t)want_cap_ * 4);
    attn_work_ = get(cuda_b200_attention_work_bytes((unsigned int)vdim));
    const size_t meta = 3 * T + 4 * T;
    d_meta_ = (int*)get(meta * 4);
    ok = ok && cudaMallocHost((void**)&h_meta_, meta * 4) == cudaSuccess && cudaMallocHost((void**)&h_choice_, (size_t)want_cap_ * 4) == cudaSuccess
        && cudaMallocHost((void**)&h_logits_, (size_t)want_cap_ * spec_.vocab * 4) == cudaSuccess;
    if (!ok) { return fail(err, "no memory for the step's buffers"); }
    return true;
}

void LayeredDecoder::makePass(const std::vector<StepEntry>& entries, const std::vector<int>& from, const std::vector<int>& count, Pass* p) const
{
    std::vector<int> ids, owner, slot, pos, start, n, wants;
    p->decode = true;
    for (size_t e = 0; e < entries.size(); e++)
    {
        if (count[e] == 0) { continue; }
        const StepEntry& E = entries[e];
        const int first = (int)ids.size(), index = (int)slot.size(), at = cache_.length(E.slot);
        slot.push_back(E.slot);
        pos.push_back(at);
        start.push_back(first);
        n.push_back(count[e]);
        for (int i = 0; i < count[e]; i++)
        {
            ids.push_back(E.tokens[from[e] + i]);
            owner.push_back(index);
        }
        size_t before = wants.size();
        for (int w : E.want)
        {
            if (w >= from[e] && w < from[e] + count[e]) { wants.push_back(first + w - from[e]); }
        }
        p->decode = p->decode && count[e] == 1 && wants.size() == before + 1;
        p->max_n = std::max(p->max_n, count[e]);
        p->max_len = std::max(p->max_len, at + count[e]);
    }
    p->tokens = (int)ids.size();
    p->entries = (int)slot.size();
    p->wants = (int)wants.size();
    p->decode = p->decode && p->tokens <= kStreamRows;
    for (auto* v : { &ids, &owner, &slot, &pos, &start, &n, &wants }) { p->host.insert(p->host.end(), v->begin(), v->end()); }
}

int LayeredDecoder::issueHead(const Pass& p, int row0, int rows, cudaStream_t st)
{
    const unsigned int PDL = 1u;
    int bad = 0, n = 0;
    auto ok = [&](int rc) {
        bad += rc != 0;
        n++;
    };
    cuda_b200_norm f = {};
    f.X = x_;
    f.weight = final_norm_.w;
    f.bias = final_norm_.b;
    f.out = head_x_;
    f.rows = devWants(p) + row0;
    f.n = (unsigned int)rows;
    f.width = (unsigned int)spec_.width;
    f.ldx = f.ldo = (unsigned int)ldw_;
    f.kind = spec_.norm_kind;
    f.eps = spec_.eps;
    ok(cuda_b200_norm_rows(act(), &f, st, PDL));
    cuda_b200_linear h = {};
    h.W = head_.w;
    h.X = head_x_;
    h.Y = logits_;
    h.rows = (unsigned int)rows;
    h.N = (unsigned int)spec_.vocab;
    h.K = (unsigned int)spec_.width;
    h.ldw = (unsigned int)head_.ld;
    h.ldx = (unsigned int)ldw_;
    h.ldy = (unsigned int)ld_logits_;
    h.alpha = spec_.logit_scale;
    ok(cuda_b200_linear_rows(act(), 1, &h, st, PDL, 0));
    ok(cuda_b200_argmax_f32(logits_, (unsigned int)rows, (unsigned int)spec_.vocab, (unsigned int)ld_logits_, d_choice_, d_best_, st, PDL));
    return bad ? -1 : n;
}

int LayeredDecoder::issue(const Pass& p, cudaStream_t st)
{
    const unsigned int PDL = 1u;
    const unsigned int T = (unsigned int)p.tokens, W = (unsigned int)spec_.width;
    const int out16 = act();
    const bool stream = dtype_ == BFLOAT16 && p.tokens <= kStreamRows;
    int bad = 0, n = 0;
    auto ok = [&](int rc) {
        bad += rc != 0;
        n++;
    };
    cuda_b200_batch b = {};
    b.slot = devEntries(p, 0);
    b.pos = devEntries(p, 1);
    b.start = devEntries(p, 2);
    b.n = devEntries(p, 3);
    b.token_entry = devTokenEntry(p);
    b.entries = (unsigned int)p.entries;
    b.tokens = T;
    b.max_n = (unsigned int)p.max_n;
    b.max_len = (unsigned int)p.max_len;
    auto dense = [&](const Weight& w, const void* X, int ldx, void* Y, int ldy) {
        cuda_b200_linear l = {};
        l.W = w.w;
        l.X = X;
        l.Y = Y;
        l.rows = T;
        l.N = (unsigned int)w.rows;
        l.K = (unsigned int)w.k;
        l.ldw = (unsigned int)w.ld;
        l.ldx = (unsigned int)ldx;
        l.ldy = (unsigned int)ldy;
        l.out_type = out16;
        l.alpha = 1.0f;
        return l;
    };
    auto into_stream = [&](const Weight& w, const void* X, int ldx) {
        cuda_b200_linear l = dense(w, X, ldx, x_, ldw_);
        l.out_type = 0;
        l.accumulate = 1;
        return l;
    };
    unsigned int pending = 0;    // experts' outputs per token that the stream still lacks
    auto norm = [&](const Norm& w, void* out) {
        cuda_b200_norm a = {};
        a.X = x_;
        a.weight = w.w;
        a.bias = w.b;
        a.out = out;
        a.Y = moe_y_;
        a.slot_row = pair_row_;
        a.slot_weight = pair_weight_;
        a.slots = pending;
        a.n = T;
        a.width = W;
        a.ldx = a.ldo = a.ldy = (unsigned int)ldw_;
        a.kind = spec_.norm_kind;
        a.eps = spec_.eps;
        ok(cuda_b200_norm_rows(act(), &a, st, PDL));
        pending = 0;
    };
    ok(cuda_b200_embed_f32(act(), devIds(p), embed_.w, (unsigned int)embed_.ld, x_, (unsigned int)ldw_, T, W, (unsigned int)spec_.vocab, spec_.embed_scale, st,
        PDL));
    for (size_t i = 0; i < layers_.size(); i++)
    {
        const Layer& L = layers_[i];
        const AttentionSpec& s = spec_.layers[i].mixer;
        const MlpSpec& m = spec_.layers[i].mlp;
        norm(L.norm1, xn_);
        cuda_b200_linear l = dense(L.qkvg, xn_, ldw_, qkvg_, ld_qkvg_);
        ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
        cuda_b200_attention a = {};
        a.qkvg = qkvg_;
        a.out = att_;
        a.k_cache = cache_.k((int)i);
        a.v_cache = cache_.v((int)i);
        a.v_first = v_first_;
        a.work = attn_work_;
        a.ld = (unsigned int)ld_qkvg_;
        a.ldo = (unsigned int)ld_att_;
        a.k_off = (unsigned int)L.k_off;
        a.v_off = (unsigned int)L.v_off;
        a.g_off = (unsigned int)L.g_off;
        a.v_first_ld = (unsigned int)ld_first_;
        a.H = (unsigned int)s.heads;
        a.Hkv = (unsigned int)s.kv_heads;
        a.dim = (unsigned int)s.dim;
        a.vdim = (unsigned int)s.vdim;
        a.k_ld = (unsigned int)cache_.kLd((int)i);
        a.v_ld = (unsigned int)cache_.vLd((int)i);
        a.T_max = (unsigned int)cache_.rows();
        a.slots = (unsigned int)cache_.slots();
        a.v_mix = L.v_mix;
        a.qk_norm = s.qk_norm;
        a.gate = !s.gate.empty();
        a.mix = L.lambda;
        a.eps = spec_.eps;
        a.scale = s.scale;
        ok(cuda_b200_attention_rows(act(), &a, &b, st, PDL, 0));
        l = into_stream(L.o, att_, ld_att_);
        ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
        if (m.kind == MlpSpec::NONE) { continue; }
        norm(L.norm2, xn_);
        if (m.kind == MlpSpec::DENSE)
        {
            l = dense(L.up, xn_, ldw_, ff_, ld_ff_);
            l.activation = m.activation;
            ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
            l = into_stream(L.down, ff_, ld_ff_);
            ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
            continue;
        }
        l = dense(L.router, xn_, ldw_, router_logits_, ld_router_);
        l.out_type = 0;
        ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
        const unsigned int E = (unsigned int)m.experts.size(), top = (unsigned int)m.top;
        const bool shared = m.shared.ff != 0;
        cuda_b200_route r = {};
        r.logits = router_logits_;
        r.pair_row = pair_row_;
        r.pair_weight = pair_weight_;
        r.row_token = row_token_;
        r.group_offset = group_offset_;
        r.active = active_;
        r.shared_weight = shared_weight_;
        r.choice = choice_;
        r.counters = counters_;
        r.n = T;
        r.ldl = (unsigned int)ld_router_;
        r.experts = E;
        r.top = top;
        r.active_cap = std::min(E, T * top);
        r.sg_col = shared ? (int)E : -1;
        ok(cuda_b200_route_rows(&r, st, PDL));
        auto grouped = [&](cuda_b200_linear* g, int group_rows) {
            g->rows = T * top;
            g->group_offset = group_offset_;
            g->groups = E;
            g->group_rows = (unsigned int)group_rows;
            g->group_max = T;
            g->active = active_;
            g->active_cap = r.active_cap;
        };
        const bool gathered = dtype_ == BFLOAT16 && !stream;
        if (gathered) { ok(cuda_b200_gather_rows(act(), xn_, (unsigned int)ldw_, row_token_, moe_x_, (unsigned int)ldw_, T * top, W, st, PDL)); }
        cuda_b200_linear in[2], out[2];
        in[0] = dense(L.experts_in, gathered ? moe_x_ : xn_, ldw_, moe_h_, ld_eff_);
        in[0].N = in[0].up_row = (unsigned int)m.experts[0].ff;
        in[0].activation = B200_ACT_SILU_GATE;
        grouped(&in[0], 2 * m.experts[0].ff);
        if (!gathered) { in[0].x_row = row_token_; }
        out[0] = dense(L.experts_out, moe_h_, ld_eff_, moe_y_, ldw_);
        out[0].N = W;
        grouped(&out[0], (int)W);
        if (shared)
        {
            in[1] = dense(L.shared_in, xn_, ldw_, ff_, ld_ff_);
            in[1].N = in[1].up_row = (unsigned int)m.shared.ff;
            in[1].activation = B200_ACT_SILU_GATE;
            out[1] = into_stream(L.shared_out, ff_, ld_ff_);
            out[1].row_scale = shared_weight_;
        }
        ok(cuda_b200_linear_rows(act(), shared ? 2 : 1, in, st, PDL, 0));
        ok(cuda_b200_linear_rows(act(), shared ? 2 : 1, out, st, PDL, 0));
        pending = top;
    }
    if (pending) { norm(Norm(), nullptr); }
    return bad ? -1 : n;
}

int LayeredDecoder::run(const Pass& p, float* logits, int* choice)
{
    cudaStream_t st = gpu_.stream();
    std::memcpy(h_meta_, p.host.data(), p.host.size() * 4);
    if (cudaMemcpyAsync(d_meta_, h_meta_, p.host.size() * 4, cudaMemcpyHostToDevice, st) != cudaSuccess) { return 1; }
    const unsigned long long before = cuda_b200_decoder_launches();
    const size_t V = (size_t)spec_.vocab;
    auto fetch = [&](int row0, int rows) {
        if (logits)
        {
            cudaMemcpy2DAsync(h_logits_, V * 4, logits_, (size_t)ld_logits_ * 4, V * 4, (size_t)rows, cudaMemcpyDeviceToHost, st);
        }
        if (choice) { cudaMemcpyAsync(h_choice_, d_choice_, (size_t)rows * 4, cudaMemcpyDeviceToHost, st); }
        if (cudaStreamSynchronize(st) != cudaSuccess) { return false; }
        if (logits) { std::memcpy(logits + (size_t)row0 * V, h_logits_, (size_t)rows * V * 4); }
        if (choice) { std::memcpy(choice + row0, h_choice_, (size_t)rows * 4); }
        return true;
    };
    if (p.decode && p.wants <= want_cap_)
    {
        // lengths up to a power of two share a graph
        Pass q = p;
        q.max_len = 64;
        while (q.max_len < p.max_len) { q.max_len *= 2; }
        q.max_len = std::min(q.max_len, cache_.rows());
        auto it = graphs_.find({ p.entries, q.max_len });
        if (it != graphs_.end())
        {
            if (cudaGraphLaunch(it->second.first, st) != cudaSuccess) { return 1; }
            last_launches_ += it->second.second;
            return fetch(0, p.wants) ? 0 : 1;
        }
        // the first step of this shape runs launch by launch (which also loads the kernels), then the launches are recorded
        if (issue(q, st) < 0 || issueHead(q, 0, q.wants, st) < 0) { return -1; }
        const int launches = (int)(cuda_b200_decoder_launches() - before);
        last_launches_ += launches;
        if (!fetch(0, p.wants)) { return 1; }
        cudaGraph_t graph = nullptr;
        cudaGraphExec_t exec = nullptr;
        if (cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal) != cudaSuccess) { return 1; }
        const bool recorded = issue(q, st) >= 0 && issueHead(q, 0, q.wants, st) >= 0;
        const cudaError_t e = cudaStreamEndCapture(st, &graph);
        const bool good = recorded && e == cudaSuccess && graph && cudaGraphInstantiate(&exec, graph, 0) == cudaSuccess;
        if (graph) { cudaGraphDestroy(graph); }
        if (!good)
        {
            cudaGetLastError();
            return 1;
        }
        graphs_[{ p.entries, q.max_len }] = { exec, launches };
        return 0;
    }
    if (issue(p, st) < 0) { return -1; }
    for (int r0 = 0; r0 < p.wants; r0 += want_cap_)
    {
        const int rows = std::min(want_cap_, p.wants - r0);
        if (issueHead(p, r0, rows, st) < 0) { return -1; }
        if ((logits || choice) && !fetch(r0, rows)) { return 1; }
    }
    last_launches_ += (int)(cuda_b200_decoder_launches() - before);
    // the pinned step arrays are reused by the next pass
    return cudaStreamSynchronize(st) == cudaSuccess ? 0 : 1;
}

int LayeredDecoder::step(const std::vector<StepEntry>& entries, float* logits, int* choice)
{
    if (!valid(entries)) { return -1; }
    gpu_.setAsCurrent();
    last_launches_ = 0;
    // passes of up to cap_ tokens; a long entry goes on in the next one.  Results are placed in the order asked for.
    std::vector<int> done(entries.size(), 0), first(entries.size(), 0);
    int wanted = 0;
    for (size_t e = 0; e < entries.size(); e++)
    {
        first[e] = wanted;
        wanted += (int)entries[e].want.size();
    }
    for (;;)
    {
        std::vector<int> count(entries.size(), 0);
        int room = cap_;
        for (size_t e = 0; e < entries.size(); e++)
        {
            count[e] = std::min(room, (int)entries[e].tokens.size() - done[e]);
            room -= count[e];
        }
        if (room == cap_) { break; }
        Pass p;
        makePass(entries, done, count, &p);
        std::vector<int> place;
        for (size_t e = 0; e < entries.size(); e++)
        {
            for (size_t w = 0; w < entries[e].want.size(); w++)
            {
                const int at = entries[e].want[w];
                if (at >= done[e] && at < done[e] + count[e]) { place.push_back(first[e] + (int)w); }
            }
        }
        std::vector<float> lg(logits && p.wants ? (size_t)p.wants * spec_.vocab : 0);
        std::vector<int> ch(choice ? p.wants : 0);
        const int rc = run(p, logits ? lg.data() : nullptr, choice ? ch.data() : nullptr);
        if (rc) { return rc; }
        for (size_t i = 0; i < place.size(); i++)
        {
            if (logits) { std::memcpy(logits + (size_t)place[i] * spec_.vocab, lg.data() + i * spec_.vocab, (size_t)spec_.vocab * 4); }
            if (choice) { choice[place[i]] = ch[i]; }
        }
        for (size_t e = 0; e < entries.size(); e++)
        {
            done[e] += count[e];
            if (count[e]) { cache_.setLength(entries[e].slot, cache_.length(entries[e].slot) + count[e]); }
        }
    }
    return cuda_b200_decoder_check("decoder step");
}

float LayeredDecoder::timeStep(int entries, int tokens, int context, int inner, int repeat)
{
    gpu_.setAsCurrent();
    if (entries <= 0 || tokens <= 0 || (long long)entries * tokens > cap_ || context + tokens > cache_.rows() || entries > cache_.slots()) { return -1.f; }
    std::vector<StepEntry> batch((size_t)entries);
    std::vector<int> from((size_t)entries, 0), count((size_t)entries, tokens);
    for (int e = 0; e < entries; e++)
    {
        batch[e].slot = cache_.open();
        if (batch[e].slot < 0) { return -1.f; }
        cache_.setLength(batch[e].slot, context);
        for (int i = 0; i < tokens; i++) { batch[e].tokens.push_back((int)(((long long)e * 7919 + (long long)i * 104729 + 17) % spec_.vocab)); }
        batch[e].want = { tokens - 1 };
    }
    Pass p;
    makePass(batch, from, count, &p);
    float best = -1.f;
    cudaStream_t st = gpu_.stream();
    cudaEvent_t a, z;
    cudaEventCreate(&a);
    cudaEventCreate(&z);
    std::vector<int> ch((size_t)p.wants);
    bool ok = p.wants <= want_cap_ && run(p, nullptr, ch.data()) == 0;
    auto g = graphs_.end();
    if (ok && p.decode)
    {
        for (auto it = graphs_.begin(); it != graphs_.end(); ++it)
        {
            if (it->first.first == entries && it->first.second >= std::min(p.max_len, cache_.rows()) && (g == graphs_.end() || it->first.second < g->first.second)) { g = it; }
        }
        ok = g != graphs_.end();
    }
    for (int r = 0; ok && r <= repeat; r++)    // the first run warms up
    {
        cudaEventRecord(a, st);
        for (int i = 0; i < inner && ok; i++)
        {
            ok = p.decode ? cudaGraphLaunch(g->second.first, st) == cudaSuccess : issue(p, st) >= 0 && issueHead(p, 0, p.wants, st) >= 0;
        }
        cudaEventRecord(z, st);
        ok = ok && cudaEventSynchronize(z) == cudaSuccess;
        float ms = 0.f;
        cudaEventElapsedTime(&ms, a, z);
        if (ok && r > 0 && (best < 0.f || ms / (float)inner < best)) { best = ms / (float)inner; }
    }
    cudaEventDestroy(a);
    cudaEventDestroy(z);
    for (auto& e : batch) { cache_.close(e.slot); }
    return ok && cuda_b200_decoder_check("timed step") == 0 ? best : -1.f;
}

}    // namespace cccc
