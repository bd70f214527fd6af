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
bool activationGated(int a) { return a == B200_ACT_SILU_GATE || a == B200_ACT_GELU_GATE; }
// Do two layers have tensors of the same shapes?
bool sameShape(const LayerSpec& a, const LayerSpec& b)
{
    auto key = [](const LayerSpec& l) {
        const AttentionSpec& x = l.attention;
        const LatentSpec& y = l.latent;
        const MlstmSpec& z = l.mlstm;
        return std::vector<int>{ (int)l.kind, x.heads, x.kv_heads, x.dim, x.vdim, y.heads, y.dim, y.rot_dim, y.vdim, y.q_rank, y.kv_rank, z.heads, z.dim, z.vdim,
            (int)l.mlp.kind, l.mlp.dense.ff, (int)l.mlp.experts.size(), l.mlp.shared.ff };
    };
    return key(a) == key(b);
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
        const std::string at = "layer " + std::to_string(i) + ": ";
        // layers may share tensors through one another, but not in a circle
        int own = (int)i;
        for (size_t hops = 0; s.layers[own].weights_of != -1; hops++)
        {
            own = s.layers[own].weights_of;
            if (own < 0 || own >= (int)s.layers.size() || hops >= s.layers.size()) { return fail(err, at + "weights_of must lead to a layer with tensors"); }
        }
        if (!sameShape(s.layers[i], s.layers[own])) { return fail(err, at + "differs from the layer whose tensors it uses"); }
        if (!checkMixer(s.layers[i], at, &mixed, err)) { return false; }
        const MlpSpec& m = s.layers[i].mlp;
        if (m.kind == MlpSpec::DENSE && m.dense.ff <= 0) { return fail(err, at + "ff must be positive"); }
        if (m.kind == MlpSpec::DENSE && activationGated(m.activation) != !m.dense.gate.empty()) { return fail(err, at + "a gated activation needs a gate, others take none"); }
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
    max_context_ = o.max_context;
    cap_ = std::max(std::min(o.max_step_tokens, o.max_context * o.max_sequences), std::min(o.max_sequences, kStreamRows));
    if (!loadTensors(source, err) || !allocate(o, err)) { return false; }
    gpu_.synchronize();
    return cuda_b200_decoder_check("model load") == 0 ? true : fail(err, "a CUDA error while loading");
}

// `rows` rows of k from the first-th element of `bits` to row `at` of w.
bool LayeredDecoder::upload(const std::string& name, const std::vector<uint16_t>& bits, size_t first, int rows, int k, size_t at, const Weight& w, std::string* err)
{
    const size_t row_bytes = (size_t)w.ld * elem();
    const void* src = bits.data() + first;
    std::vector<float> wide;
    if (dtype_ == FLOAT)
    {
        wide.resize((size_t)rows * k);
        for (size_t i = 0; i < wide.size(); i++) { wide[i] = widen(bits[first + i]); }
        src = wide.data();
    }
    weight_bytes_ += (size_t)rows * k * elem();
    return cudaMemcpy2D((char*)w.w + at * row_bytes, row_bytes, src, (size_t)k * elem(), (size_t)k * elem(), (size_t)rows, cudaMemcpyHostToDevice) == cudaSuccess
        || fail(err, "cannot copy '" + name + "' to the device");
}

// Tensors [rows][k] one below the other, every piece padded to a multiple of `align` rows; rows padded to 64 columns; zeros.
bool LayeredDecoder::packRows(TensorSource& s, const std::vector<Rows>& parts, int k, int align, Weight* out, std::string* err)
{
    auto padded = [&](int n) { return (size_t)(n + align - 1) / align * align; };
    size_t rows = 0;
    for (const auto& p : parts) { rows += padded(p.rows / p.pieces) * p.pieces; }
    out->rows = (int)rows;
    out->k = k;
    out->ld = pad64(k);
    out->w = dmalloc(rows * out->ld * elem(), true);
    if (!out->w) { return fail(err, "no device memory for '" + parts[0].name + "'"); }
    gpu_.synchronize();
    std::vector<uint16_t> bits;
    size_t at = 0;
    for (const auto& p : parts)
    {
        if (!s.readBf16(p.name, { p.rows, k }, &bits, err)) { return false; }
        const int piece = p.rows / p.pieces;
        for (int j = 0; j < p.pieces; j++)
        {
            if (!upload(p.name, bits, (size_t)j * piece * k, piece, k, at, *out, err)) { return false; }
            at += padded(piece);
        }
    }
    return true;
}

bool LayeredDecoder::packTransposed(TensorSource& s, const std::string& name, int pieces, int rows, int k, Weight* out, std::string* err)
{
    std::vector<uint16_t> bits, turned((size_t)pieces * rows * k);
    if (!s.readBf16(name, { (int64_t)pieces * rows, k }, &bits, err)) { return false; }
    for (int p = 0; p < pieces; p++)
    {
        for (int r = 0; r < rows; r++)
        {
            for (int c = 0; c < k; c++) { turned[((size_t)p * k + c) * rows + r] = bits[((size_t)p * rows + r) * k + c]; }
        }
    }
    out->rows = pieces * k;
    out->k = rows;
    out->ld = pad64(rows);
    out->w = dmalloc((size_t)out->rows * out->ld * elem(), true);
    if (!out->w) { return fail(err, "no device memory for '" + name + "'"); }
    gpu_.synchronize();
    return upload(name, turned, 0, out->rows, rows, 0, *out, err);
}

// Vectors one behind the other, as floats.
bool LayeredDecoder::loadVector(TensorSource& s, const std::vector<std::pair<std::string, int>>& parts, float** out, std::string* err)
{
    std::vector<float> f;
    std::vector<uint16_t> bits;
    for (const auto& p : parts)
    {
        if (!s.readBf16(p.first, { p.second }, &bits, err)) { return false; }
        for (uint16_t b : bits) { f.push_back(widen(b)); }
    }
    *out = (float*)dmalloc(f.size() * 4, false);
    return (*out && cudaMemcpy(*out, f.data(), f.size() * 4, cudaMemcpyHostToDevice) == cudaSuccess) || fail(err, "no device memory for '" + parts[0].first + "'");
}

bool LayeredDecoder::loadNorm(TensorSource& s, const std::string& name, Norm* out, std::string* err)
{
    return loadVector(s, { { name, spec_.width } }, &out->w, err)
        && (spec_.norm_kind != B200_NORM_LAYER || loadVector(s, { { name + ".b", spec_.width } }, &out->b, err));
}

bool LayeredDecoder::loadTensors(TensorSource& s, std::string* err)
{
    const int W = spec_.width;
    if (!packRows(s, { { spec_.embed, spec_.vocab } }, W, 1, &embed_, err)) { return false; }
    head_ = embed_;
    if (spec_.head != spec_.embed && !packRows(s, { { spec_.head, spec_.vocab } }, W, 1, &head_, err)) { return false; }
    if (!loadNorm(s, spec_.final_norm, &final_norm_, err)) { return false; }
    layers_.resize(spec_.layers.size());
    for (size_t i = 0; i < layers_.size(); i++)
    {
        if (spec_.layers[i].weights_of == -1 && !loadLayer(s, spec_.layers[i], &layers_[i], err)) { return false; }
    }
    bool mixing = false;
    for (size_t i = 0; i < layers_.size(); i++)
    {
        size_t own = i;
        while (spec_.layers[own].weights_of != -1) { own = (size_t)spec_.layers[own].weights_of; }
        if (own != i) { layers_[i] = layers_[own]; }
        const AttentionSpec& a = spec_.layers[i].attention;
        if (spec_.layers[i].kind != LayerSpec::ATTENTION || !a.v_mix) { continue; }
        layers_[i].v_mix = mixing ? 2 : 1;
        mixing = true;
        if (layers_[i].v_mix == 2)
        {
            std::vector<uint16_t> b;
            if (!s.readBf16(a.vmix, {}, &b, err)) { return false; }
            layers_[i].lambda = widen(b[0]);
        }
    }
    return true;
}

bool LayeredDecoder::loadLayer(TensorSource& s, const LayerSpec& ls, Layer* out, std::string* err)
{
    const int W = spec_.width;
    Layer& L = *out;
    if (!loadNorm(s, ls.norm1, &L.norm1, err) || !loadMixer(s, ls, &L, err)) { return false; }
    // a branch's norm has no bias
    if (!ls.norm1b.empty() && !loadVector(s, { { ls.norm1b, W } }, &L.norm1b.w, err)) { return false; }
    const MlpSpec& m = ls.mlp;
    if (m.kind == MlpSpec::NONE) { return true; }
    if (!loadNorm(s, ls.norm2, &L.norm2, err) || (!ls.norm2b.empty() && !loadVector(s, { { ls.norm2b, W } }, &L.norm2b.w, err))) { return false; }
    if (m.kind == MlpSpec::DENSE)
    {
        std::vector<Rows> up = { { m.dense.up, m.dense.ff } };
        if (!m.dense.gate.empty()) { up.insert(up.begin(), { m.dense.gate, m.dense.ff }); }
        return packRows(s, up, W, 1, &L.up, err) && packRows(s, { { m.dense.down, W } }, m.dense.ff, 1, &L.down, err);
    }
    std::vector<Rows> parts = { { m.router, (int)m.experts.size() } };
    if (m.shared.ff) { parts.push_back({ m.shared_gate, 1 }); }
    if (!packRows(s, parts, W, 1, &L.router, err)) { return false; }
    std::vector<Rows> in, down;
    for (const auto& e : m.experts)
    {
        in.push_back({ e.gate, e.ff });
        in.push_back({ e.up, e.ff });
        down.push_back({ e.down, W });
    }
    if (!packRows(s, in, W, 1, &L.experts_in, err) || !packRows(s, down, m.experts[0].ff, 1, &L.experts_out, err)) { return false; }
    return !m.shared.ff
        || (packRows(s, { { m.shared.gate, m.shared.ff }, { m.shared.up, m.shared.ff } }, W, 1, &L.shared_in, err)
            && packRows(s, { { m.shared.down, W } }, m.shared.ff, 1, &L.shared_out, err));
}

bool LayeredDecoder::allocate(const ModelOptions& o, std::string* err)
{
    int ff = 0, eff = 0, sff = 0, router = 0;
    bool branch = false;
    for (size_t i = 0; i < layers_.size(); i++)
    {
        const LayerSpec& ls = spec_.layers[i];
        const MlpSpec& m = ls.mlp;
        branch = branch || !ls.norm1b.empty() || !ls.norm2b.empty();
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
    if (!allocateMixers(o, err)) { return false; }
    ldw_ = pad64(spec_.width);
    ld_ff_ = pad64(std::max(ff, sff));
    ld_eff_ = pad64(std::max(eff, 1));
    ld_router_ = pad64(std::max(router, 1));
    ld_logits_ = pad64(spec_.vocab);
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
    if (branch) { branch_ = (float*)get(T * ldw_ * 4); }
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
    const size_t meta = 3 * T + 4 * T + 2 * windows_.size() * T;
    d_meta_ = (int*)get(meta * 4);
    ok = ok && cudaMallocHost((void**)&h_meta_, meta * 4) == cudaSuccess && cudaMallocHost((void**)&h_choice_, (size_t)want_cap_ * 4) == cudaSuccess
        && cudaMallocHost((void**)&h_logits_, (size_t)want_cap_ * spec_.vocab * 4) == cudaSuccess;
    if (!ok) { return fail(err, "no memory for the step's buffers"); }
    return true;
}

void LayeredDecoder::makePass(const std::vector<StepEntry>& entries, const std::vector<int>& from, const std::vector<int>& count, Pass* p) const
{
    std::vector<int> ids, owner, slot, start, wants, order;
    // entries of a few tokens first; the float mode has one kind of kernel
    for (int kind = 0; kind < 2; kind++)
    {
        for (size_t e = 0; e < entries.size(); e++)
        {
            const bool few = count[e] <= kFewTokens;
            if (count[e] != 0 && (kind == 0) == (few || dtype_ == FLOAT)) { order.push_back((int)e); }
        }
    }
    p->decode = true;
    for (int e : order)
    {
        const StepEntry& E = entries[e];
        const int first = (int)ids.size(), index = (int)slot.size(), at = cache_.length(E.slot);
        const bool few = count[e] <= kFewTokens || dtype_ == FLOAT;
        if (p->parts.empty() || p->parts.back().few != few)
        {
            Part part;
            part.few = few;
            part.first_entry = index;
            part.first_token = first;
            p->parts.push_back(part);
        }
        Part& part = p->parts.back();
        part.entries++;
        part.tokens += count[e];
        part.max_n = std::max(part.max_n, count[e]);
        part.max_len = std::max(part.max_len, at + count[e]);
        slot.push_back(E.slot);
        p->pos.push_back(at);
        start.push_back(first);
        p->n.push_back(count[e]);
        for (int i = 0; i < count[e]; i++)
        {
            ids.push_back(E.tokens[from[e] + i]);
            owner.push_back(index);
        }
        const size_t before = wants.size();
        for (size_t k = 0; k < E.want.size(); k++)
        {
            const int w = E.want[k];
            if (w >= from[e] && w < from[e] + count[e])
            {
                wants.push_back(first + w - from[e]);
                p->asked.emplace_back(e, (int)k);
            }
        }
        p->decode = p->decode && count[e] == 1 && wants.size() == before + 1;
    }
    p->tokens = (int)ids.size();
    p->entries = (int)slot.size();
    p->wants = (int)wants.size();
    p->decode = p->decode && p->tokens <= kStreamRows;
    for (auto* v : { &ids, &owner, &slot, &p->pos, &start, &p->n, &wants }) { p->host.insert(p->host.end(), v->begin(), v->end()); }
    if (dtype_ == FLOAT) { return; }
    for (int window : windows_)
    {
        std::vector<int> floor, pos2;
        expandedFloor(*p, window, &floor, &pos2);
        p->host.insert(p->host.end(), floor.begin(), floor.end());
        p->host.insert(p->host.end(), pos2.begin(), pos2.end());
    }
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
    h.cap = spec_.logit_softcap;
    if (h.cap > 0.f) { h.activation = B200_ACT_SOFTCAP; }
    ok(cuda_b200_linear_rows(act(), 1, &h, st, PDL, 0));
    ok(cuda_b200_argmax_f32(logits_, (unsigned int)rows, (unsigned int)spec_.vocab, (unsigned int)ld_logits_, d_choice_, d_best_, st, PDL));
    return bad ? -1 : n;
}

int LayeredDecoder::issue(const Pass& p, cudaStream_t st)
{
    const unsigned int PDL = 1u;
    const unsigned int T = (unsigned int)p.tokens, W = (unsigned int)spec_.width;
    const bool stream = dtype_ == BFLOAT16 && p.tokens <= kStreamRows;
    Issue r0{ p, st };
    auto ok = [&](int rc) { r0.ok(rc); };
    auto dense = [&](const Weight& w, const void* X, int ldx, void* Y, int ldy) { return this->dense(r0, w, X, ldx, Y, ldy); };
    auto into_stream = [&](const Weight& w, const void* X, int ldx) {
        cuda_b200_linear l = dense(w, X, ldx, x_, ldw_);
        l.out_type = 0;
        l.accumulate = 1;
        return l;
    };
    unsigned int pending = 0;           // experts' outputs per token that the stream still lacks
    const Norm* branch = nullptr;       // the norm of a branch that the stream still lacks
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
        if (branch)
        {
            a.branch = branch_;
            a.branch_weight = branch->w;
            a.ldb = (unsigned int)ldw_;
        }
        a.n = T;
        a.width = W;
        a.ldx = a.ldo = a.ldy = (unsigned int)ldw_;
        a.kind = spec_.norm_kind;
        a.eps = spec_.eps;
        ok(cuda_b200_norm_rows(act(), &a, st, PDL));
        pending = 0;
        branch = nullptr;
    };
    // a sublayer's last linear: onto the stream, or aside until the next norm
    auto output = [&](const Weight& w, const void* X, int ldx, const Norm& after) {
        cuda_b200_linear l = into_stream(w, X, ldx);
        if (after.w)
        {
            l.Y = branch_;
            l.accumulate = 0;
            branch = &after;
        }
        ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
    };
    ok(cuda_b200_embed_f32(act(), devIds(p), embed_.w, (unsigned int)embed_.ld, x_, (unsigned int)ldw_, T, W, (unsigned int)spec_.vocab, spec_.embed_scale, st,
        PDL));
    for (size_t i = 0; i < layers_.size(); i++)
    {
        const Layer& L = layers_[i];
        const MlpSpec& m = spec_.layers[i].mlp;
        norm(L.norm1, xn_);
        switch (spec_.layers[i].kind)
        {
        case LayerSpec::ATTENTION: issueAttention(r0, (int)i); break;
        case LayerSpec::LATENT: issueLatent(r0, (int)i); break;
        case LayerSpec::MLSTM: issueMlstm(r0, (int)i); break;
        }
        output(L.o, att_, ld_att_, L.norm1b);
        if (m.kind == MlpSpec::NONE) { continue; }
        norm(L.norm2, xn_);
        if (m.kind == MlpSpec::DENSE)
        {
            cuda_b200_linear l = dense(L.up, xn_, ldw_, ff_, ld_ff_);
            l.activation = m.activation;
            l.N = l.up_row = (unsigned int)m.dense.ff;
            ok(cuda_b200_linear_rows(act(), 1, &l, st, PDL, 0));
            output(L.down, ff_, ld_ff_, L.norm2b);
            continue;
        }
        cuda_b200_linear l = dense(L.router, xn_, ldw_, router_logits_, ld_router_);
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
    if (pending || branch) { norm(Norm(), nullptr); }
    return r0.bad ? -1 : r0.n;
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
        int& len = q.parts[0].max_len;
        len = 64;
        while (len < p.parts[0].max_len) { len *= 2; }
        len = std::min(len, cache_.rows());
        auto it = graphs_.find({ p.entries, len });
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
        graphs_[{ p.entries, len }] = { exec, launches };
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
        for (const auto& a : p.asked) { place.push_back(first[a.first] + a.second); }
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
            if (it->first.first == entries && it->first.second >= std::min(p.parts[0].max_len, cache_.rows()) && (g == graphs_.end() || it->first.second < g->first.second)) { g = it; }
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
