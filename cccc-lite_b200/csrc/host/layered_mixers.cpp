// The mixers of a LayeredDecoder: their checks, tensors, buffers and launches.
#include "layered_decoder.h"

#include <algorithm>
#include <cmath>

namespace cccc
{

namespace
{
bool fail(std::string* err, const std::string& what)
{
    if (err) { *err = what; }
    return false;
}
int pad(int n, int to) { return (n + to - 1) / to * to; }
constexpr unsigned int PDL = 1u;
constexpr int kExpandRows = 16384;    // cached rows that are expanded at a time, unless one sequence has more
}    // namespace

bool LayeredDecoder::checkMixer(const LayerSpec& ls, const std::string& at, int* mixed, std::string* err) const
{
    auto rotary = [&](const RotarySpec& r, int dim) {
        return r.dims == 0 || (r.dims > 0 && r.dims % 2 == 0 && r.dims <= dim && r.base > 0.0) || fail(err, at + "rot.dims must be even and no more than a head has");
    };
    if (ls.kind == LayerSpec::ATTENTION)
    {
        const AttentionSpec& a = ls.attention;
        if (a.heads <= 0 || a.kv_heads <= 0 || a.dim <= 0 || a.vdim <= 0) { return fail(err, at + "heads, kv_heads, dim and vdim must be positive"); }
        if (a.heads % a.kv_heads) { return fail(err, at + "heads must be a multiple of kv_heads"); }
        if (a.v.empty() && a.vdim != a.dim) { return fail(err, at + "values that are the keys must have their size"); }
        if (a.window < 0) { return fail(err, at + "a window cannot be negative"); }
        if (a.v_mix)
        {
            if (*mixed >= 0 && *mixed != a.kv_heads * a.vdim) { return fail(err, at + "layers that mix values must have values of one size"); }
            *mixed = a.kv_heads * a.vdim;
        }
        return rotary(a.rot, a.dim);
    }
    if (ls.kind == LayerSpec::LATENT)
    {
        const LatentSpec& a = ls.latent;
        if (a.heads <= 0 || a.dim <= 0 || a.rot_dim <= 0 || a.vdim <= 0 || a.q_rank <= 0 || a.kv_rank <= 0)
        {
            return fail(err, at + "heads, dim, rot_dim, vdim, q_rank and kv_rank must be positive");
        }
        if (a.window < 0) { return fail(err, at + "a window cannot be negative"); }
        if (a.rot.dims != a.rot_dim || !a.rot.interleaved) { return fail(err, at + "rot.dims must be rot_dim, its pairs side by side"); }
        return rotary(a.rot, a.rot_dim);
    }
    const MlstmSpec& a = ls.mlstm;
    if (a.heads <= 0 || a.dim <= 0 || a.vdim <= 0 || !(a.cap > 0.f)) { return fail(err, at + "heads, dim, vdim and the gates' cap must be positive"); }
    return true;
}

const void* LayeredDecoder::rotaryTable(const RotarySpec& r, int dims, std::string* err)
{
    auto it = rotary_.find({ dims, r.base });
    if (it != rotary_.end()) { return it->second; }
    void* t = dmalloc((size_t)max_context_ * dims / 2 * 8, false);
    if (!t || cuda_b200_rotary_table(t, (unsigned int)max_context_, (unsigned int)dims, r.base, gpu_.stream()) != 0)
    {
        fail(err, "no device memory for the table of rotations");
        return nullptr;
    }
    rotary_[{ dims, r.base }] = t;
    return t;
}

bool LayeredDecoder::loadMixer(TensorSource& s, const LayerSpec& ls, Layer* out, std::string* err)
{
    const int W = spec_.width;
    Layer& L = *out;
    if (ls.kind == LayerSpec::ATTENTION)
    {
        const AttentionSpec& a = ls.attention;
        const int q = a.heads * a.dim, k = a.kv_heads * a.dim, v = a.kv_heads * a.vdim;
        std::vector<Rows> parts = { { a.q, q }, { a.k, k } };
        L.k_off = pad(q, 8);
        L.v_off = L.k_off;
        L.g_off = L.k_off + pad(k, 8);
        if (!a.v.empty())
        {
            parts.push_back({ a.v, v });
            L.v_off = L.g_off;
            L.g_off += pad(v, 8);
        }
        if (!a.gate.empty()) { parts.push_back({ a.gate, a.heads * a.vdim }); }
        if (!packRows(s, parts, W, 8, &L.in, err) || !packRows(s, { { a.o, W } }, a.heads * a.vdim, 1, &L.o, err)) { return false; }
        if (!a.q_norm.empty() && !loadVector(s, { { a.q_norm, q } }, &L.q_norm, err)) { return false; }
        if (!a.k_norm.empty() && !loadVector(s, { { a.k_norm, k } }, &L.k_norm, err)) { return false; }
        if (!a.sink.empty() && !loadVector(s, { { a.sink, a.heads } }, &L.sink, err)) { return false; }
        return a.rot.dims == 0 || (L.rotary = rotaryTable(a.rot, a.rot.dims, err));
    }
    if (ls.kind == LayerSpec::LATENT)
    {
        const LatentSpec& a = ls.latent;
        std::vector<Rows> parts = { { a.dq, a.q_rank }, { a.dkv, a.kv_rank + a.rot_dim } };
        if (!a.gate.empty()) { parts.push_back({ a.gate, a.heads }); }
        L.k_off = pad(a.q_rank, 8);
        L.g_off = L.k_off + pad(a.kv_rank + a.rot_dim, 8);
        L.q_step = pad(a.dim + a.rot_dim, 16);
        return packRows(s, parts, W, 8, &L.in, err) && packRows(s, { { a.uq, a.heads * (a.dim + a.rot_dim), a.heads } }, a.q_rank, 16, &L.uq, err)
            && packTransposed(s, a.uk, a.heads, a.dim, a.kv_rank, &L.absorb, err) && packRows(s, { { a.uk, a.heads * a.dim } }, a.kv_rank, 1, &L.uk, err)
            && packRows(s, { { a.uv, a.heads * a.vdim } }, a.kv_rank, 1, &L.uv, err) && packRows(s, { { a.o, W } }, a.heads * a.vdim, 1, &L.o, err)
            && loadVector(s, { { a.q_norm, a.q_rank } }, &L.q_norm, err) && loadVector(s, { { a.kv_norm, a.kv_rank } }, &L.k_norm, err)
            && (L.rotary = rotaryTable(a.rot, a.rot_dim, err));
    }
    const MlstmSpec& a = ls.mlstm;
    const int qk = a.heads * a.dim, v = a.heads * a.vdim;
    L.k_off = pad(qk, 8);
    L.v_off = 2 * L.k_off;
    L.g_off = L.v_off + pad(v, 8);
    L.gates = L.g_off + pad(v, 8);
    L.f_off = pad(a.heads, 8);
    return packRows(s, { { a.q, qk }, { a.k, qk }, { a.v, v }, { a.gate, v }, { a.input, a.heads }, { a.forget, a.heads } }, W, 8, &L.in, err) && packRows(s, { { a.o, W } }, v, 1, &L.o, err)
        && loadVector(s, { { a.input + ".b", a.heads }, { a.forget + ".b", a.heads } }, &L.gate_bias, err) && loadVector(s, { { a.norm, v } }, &L.head_norm, err);
}

// The cache and the mixers' buffers.
bool LayeredDecoder::allocateMixers(const ModelOptions& o, std::string* err)
{
    std::vector<KvLayerShape> shapes;
    int vdim = 0, in = 0, att = 0, first = 0, cq = 0, q = 0, ql = 0, ol = 0, c = 0, window = 0, kx = 0, vx = 0, gates = 0;
    unsigned long long mlstm = 0;
    for (size_t i = 0; i < layers_.size(); i++)
    {
        const LayerSpec& ls = spec_.layers[i];
        in = std::max(in, layers_[i].in.rows);
        KvLayerShape shape;
        if (ls.kind == LayerSpec::ATTENTION)
        {
            const AttentionSpec& a = ls.attention;
            shape.kv_heads = a.kv_heads;
            shape.k_dim = a.dim;
            shape.v_dim = a.vdim;
            vdim = std::max(vdim, a.vdim);
            att = std::max(att, a.heads * a.vdim);
            if (a.v_mix) { first = a.kv_heads * a.vdim; }
        }
        else if (ls.kind == LayerSpec::LATENT)
        {
            const LatentSpec& a = ls.latent;
            shape.kv_heads = 1;
            shape.k_dim = a.kv_rank + a.rot_dim;
            vdim = std::max({ vdim, pad(a.kv_rank, 8), a.vdim });
            att = std::max(att, a.heads * a.vdim);
            cq = std::max(cq, a.q_rank);
            q = std::max(q, a.heads * layers_[i].q_step);
            ql = std::max(ql, a.heads * pad(a.kv_rank + a.rot_dim, 16));
            ol = std::max(ol, a.heads * pad(a.kv_rank, 8));
            c = std::max(c, a.kv_rank);
            kx = std::max(kx, a.heads * layers_[i].q_step);
            vx = std::max(vx, a.heads * pad(a.vdim, 16));
            const int w = a.window ? std::min(a.window, o.max_context) : o.max_context;
            window = std::max(window, w);
            if (std::find(windows_.begin(), windows_.end(), w) == windows_.end()) { windows_.push_back(w); }
        }
        else
        {
            const MlstmSpec& a = ls.mlstm;
            shape.state_floats = (size_t)a.heads * cuda_b200_mlstm_state_floats((unsigned int)a.dim, (unsigned int)a.vdim);
            att = std::max(att, a.heads * a.vdim);
            gates = std::max(gates, 2 * layers_[i].f_off);
            mlstm = std::max(mlstm, cuda_b200_mlstm_work_floats((unsigned int)cap_, (unsigned int)std::min(cap_, o.max_sequences), (unsigned int)a.heads, (unsigned int)a.dim, (unsigned int)a.vdim));
        }
        shapes.push_back(shape);
    }
    if (!cache_.init(&gpu_, shapes, (int)elem(), o.max_sequences, o.max_context, err)) { return false; }
    const size_t T = (size_t)cap_, e = elem();
    bool ok = true;
    auto get = [&](size_t bytes) {
        void* p = dmalloc(bytes, true);
        ok = ok && p;
        return p;
    };
    ld_in_ = pad(in, 64);
    ld_att_ = pad(att, 64);
    ld_first_ = pad(std::max(first, 1), 64);
    in_ = get(T * ld_in_ * e);
    att_ = get(T * ld_att_ * e);
    v_first_ = get(T * ld_first_ * e);
    attn_work_ = get(cuda_b200_attention_work_bytes((unsigned int)vdim));
    if (cq)
    {
        // prompts expand cached rows in BF16; the float mode keeps to the latent throughout
        const bool expands = dtype_ == BFLOAT16;
        few_cap_ = expands ? std::min(cap_, o.max_sequences * kFewTokens) : cap_;
        expand_cap_ = expands ? std::max(std::min(o.max_context, cap_ + window), std::min(kExpandRows, cap_ + o.max_sequences * window)) : 0;
        ld_cq_ = pad(cq, 64);
        ld_q_ = pad(q, 64);
        ld_ql_ = pad(ql, 64);
        ld_ol_ = pad(ol, 64);
        ld_c_ = pad(c, 64);
        const size_t F = (size_t)few_cap_, X = (size_t)expand_cap_;
        cq_ = get(T * ld_cq_ * e);
        q_ = get(T * ld_q_ * e);
        ql_ = get(F * ld_ql_ * e);
        ol_ = get(F * ld_ol_ * e);
        c_ = get(X * ld_c_ * e);
        k_exp_ = get(X * kx * e);
        v_exp_ = get(X * vx * e);
        zero_slots_ = (int*)get(T * 4);
    }
    if (gates)
    {
        ld_gates_ = pad(gates, 64);
        gates_ = (float*)get(T * ld_gates_ * 4);
        mlstm_work_ = (float*)get(mlstm * 4);
    }
    return ok || fail(err, "no memory for the mixers' buffers");
}

cuda_b200_linear LayeredDecoder::dense(const Issue& r, const Weight& w, const void* X, int ldx, void* Y, int ldy) const
{
    cuda_b200_linear l = {};
    l.W = w.w;
    l.X = X;
    l.Y = Y;
    l.rows = (unsigned int)r.p.tokens;
    l.N = (unsigned int)w.rows;
    l.K = (unsigned int)w.k;
    l.ldw = (unsigned int)w.ld;
    l.ldx = (unsigned int)ldx;
    l.ldy = (unsigned int)ldy;
    l.out_type = act();
    l.alpha = 1.0f;
    return l;
}

cuda_b200_batch LayeredDecoder::batchOf(const Pass& p, const Part& part) const
{
    cuda_b200_batch b = {};
    b.slot = devEntries(p, 0);
    b.pos = devEntries(p, 1);
    b.start = devEntries(p, 2);
    b.n = devEntries(p, 3);
    b.token_entry = devTokenEntry(p);
    b.entries = (unsigned int)part.entries;
    b.tokens = (unsigned int)part.tokens;
    b.max_n = (unsigned int)part.max_n;
    b.max_len = (unsigned int)part.max_len;
    b.first_entry = (unsigned int)part.first_entry;
    b.first_token = (unsigned int)part.first_token;
    return b;
}

cuda_b200_batch LayeredDecoder::wholeBatch(const Pass& p) const
{
    Part all;
    all.entries = p.entries;
    all.tokens = p.tokens;
    for (const Part& part : p.parts)
    {
        all.max_n = std::max(all.max_n, part.max_n);
        all.max_len = std::max(all.max_len, part.max_len);
    }
    return batchOf(p, all);
}

void LayeredDecoder::issueAttention(Issue& r, int layer)
{
    const Layer& L = layers_[layer];
    const AttentionSpec& s = spec_.layers[layer].attention;
    cuda_b200_linear l = dense(r, L.in, xn_, ldw_, in_, ld_in_);
    r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
    cuda_b200_attention a = {};
    a.qkvg = in_;
    a.out = att_;
    a.k_cache = cache_.k(layer);
    a.v_cache = cache_.v(layer);
    a.v_first = v_first_;
    a.work = attn_work_;
    a.q_norm = L.q_norm;
    a.k_norm = L.k_norm;
    a.rotary = L.rotary;
    a.sink = L.sink;
    a.ld = (unsigned int)ld_in_;
    a.ldo = (unsigned int)ld_att_;
    a.k_off = (unsigned int)L.k_off;
    a.v_off = (unsigned int)L.v_off;
    a.g_off = (unsigned int)L.g_off;
    a.v_first_ld = (unsigned int)ld_first_;
    a.H = (unsigned int)s.heads;
    a.Hkv = (unsigned int)s.kv_heads;
    a.dim = (unsigned int)s.dim;
    a.vdim = (unsigned int)s.vdim;
    a.k_ld = (unsigned int)cache_.kLd(layer);
    a.v_ld = (unsigned int)cache_.vLd(layer);
    a.T_max = (unsigned int)cache_.rows();
    a.slots = (unsigned int)cache_.slots();
    a.rot_dims = (unsigned int)s.rot.dims;
    a.window = (unsigned int)s.window;
    a.v_mix = L.v_mix;
    a.qk_norm = s.qk_norm;
    a.gate = !s.gate.empty();
    a.rot_interleaved = s.rot.interleaved;
    a.mix = L.lambda;
    a.eps = spec_.eps;
    a.scale = s.scale;
    for (const Part& part : r.p.parts)
    {
        const cuda_b200_batch b = batchOf(r.p, part);
        r.ok(cuda_b200_attention_rows(act(), &a, &b, r.st, PDL, 0));
    }
}

// A few tokens: the queries go to the latent's space, where attention has one key/value head of the cached rows.
void LayeredDecoder::issueLatent(Issue& r, int layer)
{
    const Layer& L = layers_[layer];
    const LatentSpec& s = spec_.layers[layer].latent;
    cuda_b200_linear l = dense(r, L.in, xn_, ldw_, in_, ld_in_);
    r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
    const cuda_b200_batch all = wholeBatch(r.p);
    cuda_b200_latent d = {};
    d.down = in_;
    d.cq = cq_;
    d.cache = cache_.k(layer);
    d.q_norm = L.q_norm;
    d.kv_norm = L.k_norm;
    d.rotary = L.rotary;
    d.ld = (unsigned int)ld_in_;
    d.ld_cq = (unsigned int)ld_cq_;
    d.kv_off = (unsigned int)L.k_off;
    d.q_rank = (unsigned int)s.q_rank;
    d.kv_rank = (unsigned int)s.kv_rank;
    d.rot_dim = (unsigned int)s.rot_dim;
    d.c_ld = (unsigned int)cache_.kLd(layer);
    d.T_max = (unsigned int)cache_.rows();
    d.eps = spec_.eps;
    r.ok(cuda_b200_latent_down(act(), &d, &all, r.st, PDL));
    l = dense(r, L.uq, cq_, ld_cq_, q_, ld_q_);
    r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
    const unsigned int H = (unsigned int)s.heads, step = (unsigned int)pad(s.kv_rank + s.rot_dim, 16);
    for (const Part& part : r.p.parts)
    {
        const cuda_b200_batch b = batchOf(r.p, part);
        if (!part.few && dtype_ == BFLOAT16)
        {
            issueLatentExpanded(r, layer, b);
            continue;
        }
        // tokens of this part come first in the pass (or are all of it): rows 0 .. tokens of ql and ol
        l = dense(r, L.absorb, q_, ld_q_, ql_, ld_ql_);
        l.rows = b.tokens;
        l.N = l.group_rows = (unsigned int)s.kv_rank;
        l.blocks = H;
        l.x_step = (unsigned int)L.q_step;
        l.y_step = step;
        r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
        r.ok(cuda_b200_latent_query(act(), q_, (unsigned int)ld_q_, (unsigned int)L.q_step, (unsigned int)s.dim, ql_, (unsigned int)ld_ql_, step,
            (unsigned int)s.kv_rank, H, (unsigned int)s.rot_dim, L.rotary, d.T_max, &b, r.st, PDL));
        cuda_b200_attention a = {};
        a.qkvg = ql_;
        a.out = ol_;
        a.k_cache = a.v_cache = cache_.k(layer);
        a.work = attn_work_;
        a.ld = (unsigned int)ld_ql_;
        a.ldo = (unsigned int)ld_ol_;
        a.H = H;
        a.Hkv = 1;
        a.dim = (unsigned int)(s.kv_rank + s.rot_dim);
        a.vdim = (unsigned int)pad(s.kv_rank, 8);    // columns behind the latent meet zero weights
        a.k_ld = a.v_ld = d.c_ld;
        a.T_max = d.T_max;
        a.slots = (unsigned int)cache_.slots();
        a.q_ld = step;
        a.window = (unsigned int)s.window;
        a.no_append = 1;
        a.scale = s.scale;
        r.ok(cuda_b200_attention_rows(act(), &a, &b, r.st, PDL, 0));
        l = dense(r, L.uv, ol_, ld_ol_, att_, ld_att_);
        l.rows = b.tokens;
        l.N = l.group_rows = (unsigned int)s.vdim;
        l.blocks = H;
        l.x_step = a.vdim;
        l.y_step = (unsigned int)s.vdim;
        if (!s.gate.empty())
        {
            l.head_gate = (const char*)in_ + (size_t)L.g_off * elem();
            l.ld_gate = (unsigned int)ld_in_;
        }
        r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
    }
}

// Where the entries' expanded rows go: entry e's first key that any of its tokens sees to floor[e], its first token to pos2[e].
// Returns all rows.  Entries go one behind the other inside runs of expand_cap_ rows.
int LayeredDecoder::expandedFloor(const Pass& p, int window, std::vector<int>* floor, std::vector<int>* pos2) const
{
    int at = 0, most = 0;
    for (int e = 0; e < p.entries; e++)
    {
        const int before = std::min(p.pos[e], window - 1), rows = before + p.n[e];
        const bool few = p.n[e] <= kFewTokens;
        if (!few && at + rows > expand_cap_) { at = 0; }
        floor->push_back(few ? 0 : at);
        pos2->push_back(few ? 0 : at + before);
        if (!few) { at += rows; }
        most = std::max(most, at);
    }
    return most;
}

// Prompts: keys and values of all heads from the cached latents that the part's tokens may read, then plain attention.
void LayeredDecoder::issueLatentExpanded(Issue& r, int layer, const cuda_b200_batch& part)
{
    const Layer& L = layers_[layer];
    const LatentSpec& s = spec_.layers[layer].latent;
    const int window = s.window ? std::min(s.window, max_context_) : max_context_;
    const int w = (int)(std::find(windows_.begin(), windows_.end(), window) - windows_.begin());
    const unsigned int H = (unsigned int)s.heads, step = (unsigned int)L.q_step, v_step = (unsigned int)pad(s.vdim, 16);
    std::vector<int> floor, pos2;
    expandedFloor(r.p, window, &floor, &pos2);
    r.ok(cuda_b200_latent_query(act(), q_, (unsigned int)ld_q_, step, (unsigned int)s.dim, q_, (unsigned int)ld_q_, step, (unsigned int)s.dim, H,
        (unsigned int)s.rot_dim, L.rotary, (unsigned int)cache_.rows(), &part, r.st, PDL));
    const int end = (int)(part.first_entry + part.entries);
    int token = (int)part.first_token;
    for (int e = (int)part.first_entry; e < end;)
    {
        Part run;    // entries whose rows fit together
        run.first_entry = e;
        run.first_token = token;
        int rows = 0, longest = 0;
        for (; e < end && (run.entries == 0 || floor[e] != 0); e++)
        {
            run.entries++;
            run.tokens += r.p.n[e];
            run.max_n = std::max(run.max_n, r.p.n[e]);
            rows = pos2[e] + r.p.n[e];
            longest = std::max(longest, rows - floor[e]);
        }
        token += run.tokens;
        run.max_len = rows;
        cuda_b200_batch b = batchOf(r.p, run);
        cuda_b200_expand x = {};
        x.cache = cache_.k(layer);
        x.c = c_;
        x.K = k_exp_;
        x.floor = devExpanded(r.p, w, 0);
        x.pos2 = devExpanded(r.p, w, 1);
        x.c_ld = (unsigned int)cache_.kLd(layer);
        x.T_max = (unsigned int)cache_.rows();
        x.kv_rank = (unsigned int)s.kv_rank;
        x.rot_dim = (unsigned int)s.rot_dim;
        x.ld_c = (unsigned int)ld_c_;
        x.k_ld = step;
        x.T = (unsigned int)expand_cap_;
        x.dim = (unsigned int)s.dim;
        x.heads = H;
        x.max_rows = (unsigned int)longest;
        r.ok(cuda_b200_latent_expand(act(), &x, &b, r.st, PDL));
        cuda_b200_linear l = dense(r, L.uk, c_, ld_c_, k_exp_, (int)step);
        l.rows = (unsigned int)rows;
        l.N = l.group_rows = (unsigned int)s.dim;
        l.blocks = H;
        l.y_step = x.T * step;
        r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
        l = dense(r, L.uv, c_, ld_c_, v_exp_, (int)v_step);
        l.rows = (unsigned int)rows;
        l.N = l.group_rows = (unsigned int)s.vdim;
        l.blocks = H;
        l.y_step = x.T * v_step;
        r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
        cuda_b200_attention a = {};
        a.qkvg = q_;
        a.out = att_;
        a.k_cache = k_exp_;
        a.v_cache = v_exp_;
        a.work = attn_work_;
        a.ld = (unsigned int)ld_q_;
        a.ldo = (unsigned int)ld_att_;
        a.H = a.Hkv = H;
        a.dim = (unsigned int)(s.dim + s.rot_dim);
        a.vdim = (unsigned int)s.vdim;
        a.k_ld = step;
        a.v_ld = v_step;
        a.T_max = x.T;
        a.slots = 1;
        a.q_ld = step;
        a.window = (unsigned int)s.window;
        a.no_append = 1;
        a.scale = s.scale;
        if (!s.gate.empty())
        {
            a.head_gate = (const char*)in_ + (size_t)L.g_off * elem();
            a.ld_gate = (unsigned int)ld_in_;
        }
        b.slot = zero_slots_;
        b.pos = devExpanded(r.p, w, 1);
        b.floor = devExpanded(r.p, w, 0);
        r.ok(cuda_b200_attention_rows(act(), &a, &b, r.st, PDL, 0));
    }
}

void LayeredDecoder::issueMlstm(Issue& r, int layer)
{
    const Layer& L = layers_[layer];
    const MlstmSpec& s = spec_.layers[layer].mlstm;
    cuda_b200_linear l = dense(r, L.in, xn_, ldw_, in_, ld_in_);
    l.Y_tail = gates_;
    l.tail = (unsigned int)L.gates;
    l.ld_tail = (unsigned int)ld_gates_;
    r.ok(cuda_b200_linear_rows(act(), 1, &l, r.st, PDL, 0));
    cuda_b200_mlstm a = {};
    a.qkvg = in_;
    a.gates = gates_;
    a.bias = L.gate_bias;
    a.norm = L.head_norm;
    a.out = att_;
    a.state = cache_.state(layer);
    a.work = mlstm_work_;
    a.ld = (unsigned int)ld_in_;
    a.ld_gates = (unsigned int)ld_gates_;
    a.ldo = (unsigned int)ld_att_;
    a.k_off = (unsigned int)L.k_off;
    a.v_off = (unsigned int)L.v_off;
    a.g_off = (unsigned int)L.g_off;
    a.f_off = (unsigned int)L.f_off;
    a.heads = (unsigned int)s.heads;
    a.dim = (unsigned int)s.dim;
    a.vdim = (unsigned int)s.vdim;
    a.cap = s.cap;
    a.eps = spec_.eps;
    a.q_scale = (float)(1.0 / std::sqrt((double)s.dim));
    for (const Part& part : r.p.parts)
    {
        const cuda_b200_batch b = batchOf(r.p, part);
        r.ok(cuda_b200_mlstm_rows(act(), &a, &b, r.st, PDL, 0));
    }
}

}    // namespace cccc
