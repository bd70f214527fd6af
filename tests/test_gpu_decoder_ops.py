"""The layer operations of include/cccc_b200_decoder.h, each alone, against numpy statements of the same mechanism."""
import numpy as np
import pytest

from __graft_entry__ import load_package
from oracle import fakilorn as F

pytestmark = pytest.mark.gpu

FLOAT, BF16 = 0, 3
TOL = {FLOAT: 2e-6, BF16: 6e-3}     # of the largest value of a row, against float64 on the same inputs


@pytest.fixture(scope="module")
def D():
    d = load_package().decoder_capi
    d.lib()
    return d


def dev(a, dtype=None):
    import torch

    t = torch.from_numpy(np.ascontiguousarray(a)).cuda()
    return t.to(torch.bfloat16 if dtype == BF16 else torch.float32) if dtype is not None else t


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def pad64(n):
    return (n + 63) // 64 * 64


def padded(a, dtype, ld=None, junk=0.0):
    """Rows of `a` in a device buffer of row stride ld (columns behind them hold `junk`)."""
    out = np.full((a.shape[0], ld or pad64(a.shape[1])), junk, np.float32)
    out[:, :a.shape[1]] = a
    return dev(out, dtype)


def rand(rng, *shape, dtype=BF16, scale=1.0):
    a = (scale * rng.standard_normal(shape)).astype(np.float32)
    return F.bf16_round(a).reshape(shape) if dtype == BF16 else a


def close(got, want, dtype, what="", factor=1.0):
    bar = factor * TOL[dtype] * np.maximum(np.abs(want).max(axis=-1, keepdims=True), 1e-6)
    assert np.all(np.isfinite(got)), what
    worst = float((np.abs(got - want) / bar).max())
    assert worst <= 1.0, (what, worst)


# ---- rows --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("width,n", [(200, 3), (97, 70), (1032, 5), (4096, 65), (3, 1)])
def test_norm_adds_branches_first(D, dtype, width, n):
    rng = np.random.default_rng(width + n)
    ld = pad64(width)
    x = (3 + 2 * rng.standard_normal((n, width))).astype(np.float32)
    w, b = rng.standard_normal(width).astype(np.float32), rng.standard_normal(width).astype(np.float32)
    slots, n_y = 3, 2 * n + 1
    y = rand(rng, n_y, width, dtype=dtype)
    rows = rng.integers(0, n_y, (n, slots)).astype(np.int32)
    wt = rng.standard_normal((n, slots)).astype(np.float32)
    for kind, eps in ((D.NORM_LAYER, 1e-3), (D.NORM_RMS, 0.5)):
        for with_slots in (False, True):
            X, out = padded(x, FLOAT, junk=1e9), padded(np.zeros((n, width)), dtype)
            Y, dr, dw, bw, bb = padded(y, dtype), dev(rows), dev(wt), dev(w), dev(b)
            a = D.fill(D.Norm, X=X, weight=bw, bias=bb, out=out, n=n, width=width, ldx=ld, ldo=ld, ldy=ld, kind=kind, eps=eps)
            want_x = x.astype(np.float64)
            if with_slots:
                a = D.fill(D.Norm, X=X, weight=bw, bias=bb, out=out, Y=Y, slot_row=dr, slot_weight=dw, n=n, width=width, ldx=ld, ldo=ld, ldy=ld, slots=slots,
                           kind=kind, eps=eps)
                want_x = want_x + (wt[:, :, None] * y[rows].astype(np.float64)).sum(1)
            assert D.norm(dtype, a) == 0 and D.check() == 0
            want = F.layer_norm(want_x, w, b, eps) if kind == D.NORM_LAYER else F.unit_rms(want_x, eps) * w
            close(host(X)[:, :width], want_x, FLOAT, "stream", 4)
            close(host(out)[:, :width], want, dtype, (kind, with_slots), 10 if dtype == FLOAT else 1)
            assert np.all(host(out)[:, width:] == 0) and np.all(host(X)[:, width + (-width) % 4:] == np.float32(1e9))


def test_norm_of_chosen_rows_leaves_the_stream(D):
    rng = np.random.default_rng(5)
    x = rng.standard_normal((9, 130)).astype(np.float32)
    rows = np.array([7, 0, 7, 3], np.int32)
    X, out, dr = padded(x, FLOAT), padded(np.zeros((4, 130)), BF16), dev(rows)
    assert D.norm(BF16, D.fill(D.Norm, X=X, out=out, rows=dr, n=4, width=130, ldx=192, ldo=192, kind=D.NORM_LAYER, eps=1e-5)) == 0
    close(host(out)[:, :130], F.layer_norm(x[rows].astype(np.float64), 1.0, 0.0, 1e-5), BF16)
    assert np.array_equal(host(X)[:, :130], x.astype(np.float64))


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
def test_embedding_is_scaled_in_float(D, dtype):
    rng = np.random.default_rng(6)
    table = rand(rng, 50, 77, dtype=dtype)
    ids = np.array([0, 49, 3, -1, 50, 3], np.int32)
    X, T, I = padded(np.ones((6, 77)), FLOAT), padded(table, dtype), dev(ids)
    assert D.embed(dtype, I, T, 128, X, 128, 6, 77, 50, 7.3) == 0
    want = np.stack([table[i] * np.float32(7.3) if 0 <= i < 50 else np.zeros(77, np.float32) for i in ids])
    assert np.array_equal(X.cpu().numpy()[:, :77], want)


def test_argmax_takes_the_first_largest(D):
    import torch

    rng = np.random.default_rng(7)
    a = rng.standard_normal((5, 5003)).astype(np.float32)
    a[0, [17, 4000]] = 9.0
    a[1, 5002] = 11.0
    a[2, :] = -np.inf
    a[3, :] = np.nan
    a[4, :100] = np.nan
    idx, val = torch.zeros(5, dtype=torch.int32, device="cuda"), torch.zeros(5, device="cuda")
    assert D.argmax(dev(a), 5, 5003, 5003, idx, val) == 0
    assert idx.tolist()[:4] == [17, 5002, 0, -1] and idx.tolist()[4] == 100 + int(np.argmax(a[4, 100:]))


# ---- linears -----------------------------------------------------------------------------------------
def act_ref(kind, a, up):
    return F.squared_relu(a) if kind == 1 else (F.silu(a) * up if kind == 2 else a)


KERNELS = {FLOAT: [0], BF16: [1, 2]}


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("rows,N,K", [(1, 40, 97), (5, 136, 200), (9, 16, 64), (17, 300, 520), (33, 72, 130), (130, 260, 200), (300, 640, 1032)])
@pytest.mark.parametrize("activation", [0, 1, 2])
def test_dense_linear(D, dtype, rows, N, K, activation):
    rng = np.random.default_rng(rows * 1000 + N + K)
    w, x = rand(rng, 2 * N if activation == 2 else N, K, dtype=dtype, scale=K ** -0.5), rand(rng, rows, K, dtype=dtype)
    W, X = padded(w, dtype), padded(x, dtype, junk=5.0)
    full = 0.7 * (x.astype(np.float64) @ w.T.astype(np.float64))
    want = act_ref(activation, full[:, :N], full[:, N:])
    rs = rng.uniform(0.5, 2, rows).astype(np.float32)
    start = rng.standard_normal((rows, N)).astype(np.float32)
    for kernel in KERNELS[dtype]:
        for out_type, accumulate, scaled in ((0, 0, False), (0, 1, True), (0, 1, False), (3, 0, False)):
            if dtype == FLOAT and out_type == 3:
                continue
            ldy = N + (-N) % 8 + 8
            Y, R = padded(start, out_type if out_type else FLOAT, ldy, junk=-3.0), dev(rs)
            a = D.fill(D.Linear, W=W, X=X, Y=Y, row_scale=R if scaled else None, rows=rows, N=N, K=K, ldw=pad64(K), ldx=pad64(K), ldy=ldy, up_row=N,
                       out_type=out_type, activation=activation, accumulate=accumulate, alpha=0.7)
            assert D.linear(dtype, [a], kernel=kernel) == 0 and D.check() == 0
            ref = want * rs[:, None] if scaled else want
            if accumulate:
                ref = ref + start
            # float results are the float sums of BF16-exact operands
            close(host(Y)[:, :N], ref, BF16 if out_type == 3 else FLOAT, (kernel, out_type, accumulate), 10)
            assert np.all(host(Y)[:, N:] == -3.0)


@pytest.mark.parametrize("tokens,E,top,ff,width", [(1, 8, 2, 40, 96), (7, 5, 3, 24, 200), (32, 16, 4, 72, 130), (90, 3, 1, 136, 64), (400, 9, 4, 200, 260),
                                                   (64, 1, 1, 32, 72)])
@pytest.mark.parametrize("dtype", [FLOAT, BF16])
def test_experts_from_router_to_stream(D, dtype, tokens, E, top, ff, width):
    """Routing, the grouped gated linears and the weighted addition, against the mixture written out."""
    import torch

    rng = np.random.default_rng(tokens + E)
    h = rand(rng, tokens, width, dtype=dtype)
    w = dict(router=rand(rng, E, width, dtype=dtype, scale=width ** -0.5), shared=dict(sg=rand(rng, 1, width, dtype=dtype, scale=width ** -0.5)))
    for j in range(E):
        w[f"e{j}"] = dict(gate=rand(rng, ff, width, dtype=dtype, scale=width ** -0.5), up=rand(rng, ff, width, dtype=dtype, scale=width ** -0.5),
                          down=rand(rng, width, ff, dtype=dtype, scale=ff ** -0.5))
    ldw, lde, P = pad64(width), pad64(ff), tokens * top
    X, S = padded(h, dtype, junk=1.0), padded(np.zeros((tokens, width)), FLOAT)
    z = np.concatenate([h @ w["router"].T, h @ w["shared"]["sg"].T], 1).astype(np.float32)
    Z = padded(z, FLOAT)
    i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device="cuda")
    pr, rt, ch, ctr, off, act = i32(P), i32(P), i32(P), i32(E), i32(E + 1), i32(E)
    pw, sw = torch.zeros(P, device="cuda"), torch.zeros(tokens, device="cuda")
    cap = min(E, P)
    r = D.fill(D.Route, logits=Z, pair_row=pr, pair_weight=pw, row_token=rt, group_offset=off, active=act, shared_weight=sw, choice=ch, counters=ctr, n=tokens,
               ldl=pad64(E + 1), experts=E, top=top, active_cap=cap, sg_col=E)
    assert D.route(r) == 0 and D.check() == 0
    idx, wt = F.route(z[:, :E].astype(np.float64), top)
    assert np.array_equal(ch.cpu().numpy().reshape(tokens, top), idx)
    assert np.allclose(pw.cpu().numpy().reshape(tokens, top), wt, rtol=1e-5, atol=1e-7)
    assert np.allclose(sw.cpu().numpy(), F.sigmoid(z[:, E].astype(np.float64)), rtol=1e-5)
    counts = np.bincount(idx.reshape(-1), minlength=E)
    assert np.array_equal(off.cpu().numpy(), np.concatenate([[0], np.cumsum(counts)]))
    live = np.nonzero(counts)[0]
    assert act.cpu().tolist()[:cap] == (list(live) + [-1] * cap)[:cap]
    rows = pr.cpu().numpy().reshape(tokens, top)
    assert sorted(rows.reshape(-1)) == list(range(P))
    owner = np.empty(P, int)
    for t in range(tokens):
        for s in range(top):
            owner[rows[t, s]] = idx[t, s]
            assert rt[int(rows[t, s])].item() == t
    assert np.all(np.diff(owner) >= 0)
    W1 = padded(np.concatenate([np.concatenate([w[f"e{j}"]["gate"], w[f"e{j}"]["up"]]) for j in range(E)]), dtype)
    W2 = padded(np.concatenate([w[f"e{j}"]["down"] for j in range(E)]), dtype)
    want = sum(np.where((idx == j).any(1), (wt * (idx == j)).sum(1), 0)[:, None] * F.gated_expert(h.astype(np.float64), {k: v.astype(np.float64) for k, v in w[f"e{j}"].items()})
               for j in range(E))
    for kernel in KERNELS[dtype]:
        if kernel == 1 and tokens > 100:
            continue
        H, Y = padded(np.full((P, ff), 9.0), dtype), padded(np.full((P, width), 9.0), dtype)
        G = padded(np.zeros((P, width)), dtype)
        x_in = X
        if kernel == 2:
            assert D.gather(dtype, X, ldw, rt, G, ldw, P, width) == 0
            assert np.array_equal(host(G)[:, :width], h[rt.cpu().numpy()].astype(np.float64))
            x_in = G
        grp = dict(rows=P, group_offset=off, groups=E, group_max=tokens, active=act, active_cap=cap, alpha=1.0, out_type=dtype)
        a = D.fill(D.Linear, W=W1, X=x_in, Y=H, x_row=None if kernel == 2 else rt, N=ff, K=width, ldw=ldw, ldx=ldw, ldy=lde, group_rows=2 * ff, up_row=ff,
                   activation=2, **grp)
        assert D.linear(dtype, [a], kernel=kernel) == 0
        b = D.fill(D.Linear, W=W2, X=H, Y=Y, N=width, K=ff, ldw=lde, ldx=lde, ldy=ldw, group_rows=width, **grp)
        assert D.linear(dtype, [b], kernel=kernel) == 0
        S.zero_()
        assert D.norm(dtype, D.fill(D.Norm, X=S, Y=Y, slot_row=pr, slot_weight=pw, n=tokens, width=width, ldx=ldw, ldo=ldw, ldy=ldw, slots=top, eps=1e-5)) == 0
        assert D.check() == 0
        close(host(S)[:, :width], want, dtype, kernel, 3 if dtype == BF16 else 10)


def test_a_group_of_members_is_the_separate_launches(D):
    rng = np.random.default_rng(11)
    x = rand(rng, 6, 288)
    X = padded(x, BF16)
    members, outs, wants = [], [], []
    for j, (N, act) in enumerate(((70, 0), (48, 2), (130, 1))):
        w = rand(rng, N * (2 if act == 2 else 1), 288, scale=0.05)
        W, Y = padded(w, BF16), padded(np.zeros((6, N)), FLOAT)
        full = x.astype(np.float64) @ w.T
        wants.append(act_ref(act, full[:, :N], full[:, N:]))
        members.append(D.fill(D.Linear, W=W, X=X, Y=Y, rows=6, N=N, K=288, ldw=320, ldx=320, ldy=pad64(N), up_row=N, activation=act, alpha=1.0))
        outs.append((W, Y, N))
    before = D.launches()
    assert D.linear(BF16, members, flags=1) == 0 and D.launches() == before + 1
    for (W, Y, N), want in zip(outs, wants):
        close(host(Y)[:, :N], want, FLOAT, N, 10)


def test_descriptors_that_are_not_taken(D):
    X = padded(np.ones((2, 64)), BF16)
    base = dict(W=X, X=X, Y=X, rows=2, N=2, K=64, ldw=64, ldx=64, ldy=64, alpha=1.0)
    for bad in (dict(ldw=72), dict(K=65), dict(X=X.data_ptr() + 2), dict(activation=5), dict(activation=4), dict(blocks=2, x_step=4), dict(accumulate=1, out_type=3), dict(W=None)):
        assert D.linear(BF16, [D.fill(D.Linear, **{**base, **bad})]) == -1, bad
    assert D.linear(FLOAT, [D.fill(D.Linear, **{**base, "out_type": 3})]) == -1
    assert D.linear(7, [D.fill(D.Linear, **base)]) == -1


# ---- attention ---------------------------------------------------------------------------------------
class Attn:
    """A batch over caches of several slots: device buffers, the call, and the reference result."""

    def __init__(self, D, dtype, H, Hkv, dim, vdim, entries, T_max=700, slots=4, scale=0.2, v_mix=0, qk_norm=1, gate=1, mix=0.3, seed=0):
        import torch

        self.D, self.dtype = D, dtype
        rng = np.random.default_rng(seed)
        self.H, self.Hkv, self.dim, self.vdim, self.entries, self.T_max, self.scale = H, Hkv, dim, vdim, entries, T_max, scale
        self.v_mix, self.qk_norm, self.gate, self.mix, self.eps = v_mix, qk_norm, gate, mix, 1e-2
        T = sum(n for _, _, n in entries)
        self.q, self.k = rand(rng, T, H, dim, dtype=dtype), rand(rng, T, Hkv, dim, dtype=dtype)
        self.v, self.g = rand(rng, T, Hkv, vdim, dtype=dtype), rand(rng, T, H, vdim, dtype=dtype)
        self.first = rand(rng, T, Hkv, vdim, dtype=dtype)
        self.kc, self.vc = rand(rng, slots, Hkv, T_max, dim, dtype=dtype), rand(rng, slots, Hkv, T_max, vdim, dtype=dtype)
        self.T, self.torch = T, torch

    def run(self, kernel=0):
        D, dt, T = self.D, self.dtype, self.T
        pad8 = lambda n: (n + 7) // 8 * 8
        H, G, d, dv = self.H, self.Hkv, self.dim, self.vdim
        k_off = pad8(H * d)
        v_off = k_off + pad8(G * d)
        g_off = v_off + pad8(G * dv)
        ld = pad64(g_off + H * dv)
        row = np.full((T, ld), 3.0, np.float32)
        row[:, :H * d] = self.q.reshape(T, -1)
        row[:, k_off:k_off + G * d] = self.k.reshape(T, -1)
        row[:, v_off:v_off + G * dv] = self.v.reshape(T, -1)
        row[:, g_off:g_off + H * dv] = self.g.reshape(T, -1)
        kl, vl = (n + (-n) % 16 for n in (d, dv))
        kc, vc = np.zeros(self.kc.shape[:3] + (kl,), np.float32), np.zeros(self.vc.shape[:3] + (vl,), np.float32)
        kc[..., :d], vc[..., :dv] = self.kc, self.vc
        self.x, self.K, self.V = dev(row, dt), dev(kc, dt), dev(vc, dt)
        self.out = padded(np.full((T, H * dv), -2.0), dt)
        self.fst = padded(self.first.reshape(T, -1), dt)
        self.work = self.torch.zeros(D.attention_work_bytes(dv), dtype=self.torch.uint8, device="cuda")
        a = D.fill(D.Attention, qkvg=self.x, out=self.out, k_cache=self.K, v_cache=self.V, v_first=self.fst, work=self.work, ld=ld, ldo=pad64(H * dv),
                   k_off=k_off, v_off=v_off, g_off=g_off, v_first_ld=pad64(G * dv), H=H, Hkv=G, dim=d, vdim=dv, k_ld=kl, v_ld=vl, T_max=self.T_max, slots=self.kc.shape[0],
                   v_mix=self.v_mix, qk_norm=self.qk_norm, gate=self.gate, mix=self.mix, eps=self.eps, scale=self.scale)
        n = [e[2] for e in self.entries]
        meta = [np.array(m, np.int32) for m in ([e[0] for e in self.entries], [e[1] for e in self.entries], np.concatenate([[0], np.cumsum(n)[:-1]]), n,
                                                np.repeat(np.arange(len(n)), n))]
        self.meta = [dev(m) for m in meta]
        b = D.fill(D.Batch, slot=self.meta[0], pos=self.meta[1], start=self.meta[2], n=self.meta[3], token_entry=self.meta[4], entries=len(n), tokens=T,
                   max_n=max(n), max_len=max(p + m for _, p, m in self.entries))
        assert D.attention(dt, a, b, kernel=kernel) == 0 and D.check() == 0
        return host(self.out)[:, :H * dv].reshape(T, H, dv)

    def reference(self):
        f8 = lambda a: a.astype(np.float64)
        q, k = f8(self.q), f8(self.k)
        if self.qk_norm:
            q, k = F.unit_rms(q, self.eps), F.unit_rms(k, self.eps)
        v = f8(self.v) if self.v_mix != 2 else F.mix_values(f8(self.v), f8(self.first), self.mix)
        if self.dtype == BF16:      # what the caches hold and the tensor cores read
            q, k, v = (F.bf16_round(a).astype(np.float64).reshape(a.shape) for a in (q, k, v))
        out, at = np.zeros((self.T, self.H, self.vdim)), 0
        self.k_new, self.v_new = k, v
        for slot, pos, n in self.entries:
            K = np.concatenate([f8(self.kc[slot, :, :pos]), k[at:at + n].transpose(1, 0, 2)], 1)
            V = np.concatenate([f8(self.vc[slot, :, :pos]), v[at:at + n].transpose(1, 0, 2)], 1)
            for j in range(n):
                for h in range(self.H):
                    kv = h // (self.H // self.Hkv)
                    s = K[kv, :pos + j + 1] @ q[at + j, h] * self.scale
                    p = np.exp(s - s.max())
                    out[at + j, h] = (p / p.sum()) @ V[kv, :pos + j + 1]
            at += n
        return out * F.sigmoid(f8(self.g)) if self.gate else out


KINDS = {FLOAT: [0], BF16: [1, 2, 3, 4, 5]}
SIZES = [(6, 2, 40, 24), (4, 4, 7, 5), (24, 1, 72, 136), (8, 2, 64, 56), (2, 1, 128, 128), (3, 3, 200, 16), (5, 1, 16, 256), (12, 3, 256, 72)]


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("H,Hkv,dim,vdim", SIZES)
def test_attention_sizes_and_ragged_batches(D, dtype, H, Hkv, dim, vdim):
    ragged, decoding = [(2, 130, 3), (0, 0, 37), (3, 333, 1), (1, 64, 18)], [(1, 600, 1), (3, 0, 1), (0, 15, 1), (2, 16, 1)]
    for v_mix, entries in ((0, ragged), (1, ragged), (2, ragged), (0, decoding), (1, decoding), (2, decoding)):
        a = Attn(D, dtype, H, Hkv, dim, vdim, entries, scale=0.3, v_mix=v_mix, seed=H * dim)
        want = a.reference()
        for kind in KINDS[dtype]:
            if kind == 4 and max(dim, vdim) > 128:
                continue
            got = a.run(kind)
            close(got.reshape(a.T, -1), want.reshape(a.T, -1), dtype, (kind, v_mix), 10 if dtype == FLOAT else 1.5)
            # the caches: new rows in place, everything else untouched, padding zero
            K, V, at = host(a.K), host(a.V), 0
            kc, vc = a.kc.astype(np.float64), a.vc.astype(np.float64)
            for slot, pos, n in a.entries:
                kc[slot, :, pos:pos + n] = a.k_new[at:at + n].transpose(1, 0, 2)
                vc[slot, :, pos:pos + n] = a.v_new[at:at + n].transpose(1, 0, 2)
                at += n
            step = 1e-6 if dtype == FLOAT else 2.0 ** -7
            assert np.abs(K[..., :dim] - kc).max() <= step * np.abs(kc).max() and np.abs(V[..., :vdim] - vc).max() <= step * np.abs(vc).max()
            old = np.ones(kc.shape[:3], bool)
            for slot, pos, n in a.entries:
                old[slot, :, pos:pos + n] = False
            assert np.array_equal(K[..., :dim][old], kc[old]) and np.array_equal(V[..., :vdim][old], vc[old])
            assert np.all(K[..., dim:] == 0) and np.all(V[..., vdim:] == 0)
            if v_mix == 1:
                assert np.array_equal(host(a.fst)[:, :Hkv * vdim].reshape(a.v.shape), a.v.astype(np.float64))


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("pos,n", [(600, 1), (600, 2), (0, 600), (511, 80), (63, 66)])
def test_one_key_stands_out(D, dtype, pos, n):
    """One key scores far above all others: whoever sees it returns its value, whoever does not, does not.  Keys at the
    start, at tile edges, the query's own and the one behind it."""
    spots = sorted({0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 255, 256, 511, 512, pos - 1, pos, pos + 1, pos + n - 1})
    for spot in (s for s in spots if 0 <= s < pos + n):
        a = Attn(D, dtype, 4, 2, 32, 32, [(1, pos, n)], scale=1.0, qk_norm=0, gate=0, seed=spot)
        u = np.zeros(32, np.float32)
        u[3] = 8.0
        a.q[:] = 0.25 * a.q + u
        if spot < pos:
            a.kc[1, :, spot], a.vc[1, :, spot] = u, 5.0
        else:
            a.k[spot - pos], a.v[spot - pos] = u, 5.0
        want = a.reference()
        for kind in KINDS[dtype]:
            if kind in (1, 4) and n > 100:
                continue
            got = a.run(kind)
            close(got.reshape(n, -1), want.reshape(n, -1), dtype, (kind, spot), 10 if dtype == FLOAT else 1.5)
            sees = np.arange(pos, pos + n) >= spot
            assert np.all(np.abs(got[sees] - 5.0) < 0.2) and (sees.all() or np.abs(got[~sees]).max() < 4.0)


def test_softmax_weights_are_not_rounded(D):
    """Thousands of near-equal weights, values that cancel all but a little: weights rounded to 16 bits would show."""
    T = 2048
    a = Attn(D, BF16, 8, 1, 64, 64, [(0, T - 1, 1)], T_max=T, slots=1, scale=0.05, qk_norm=0, gate=0, seed=3)
    a.vc[..., :] = 64.0 * np.where(np.arange(T) % 2, 1, -1)[None, None, :, None] + (np.arange(T) % 7 == 0)[None, None, :, None]
    a.vc = F.bf16_round(a.vc).reshape(a.vc.shape)
    want = a.reference()
    for kind in (1, 2, 3, 4, 5):
        assert np.abs(a.run(kind) - want).max() < 2.5e-3 * max(1.0, np.abs(want).max()), kind


def test_split_results_do_not_depend_on_the_splits(D):
    """The same query alone (many splits) and among thirty others (few): the same values up to float rounding."""
    one = Attn(D, BF16, 8, 2, 64, 56, [(3, 650, 1)], seed=4)
    many = Attn(D, BF16, 8, 2, 64, 56, [(s % 4, 100 + s, 1) for s in range(3)] + [(3, 650, 1)], slots=4, seed=5)
    many.kc, many.vc = one.kc, one.vc
    for name in ("q", "k", "v", "g"):
        getattr(many, name)[3] = getattr(one, name)[0]
    for kind in (1, 4):
        x, y = one.run(kind)[0], many.run(kind)[3]
        assert np.abs(x - y).max() <= 2.0 ** -8 * np.abs(x).max()
