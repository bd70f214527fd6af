"""The layer operations that Tazunex's mixers and norms are made of, each alone, every kernel of an operation on the same cases,
against the plain statements in oracle/tazunex.py."""
import numpy as np
import pytest

from __graft_entry__ import load_package
from oracle import tazunex as Z
from tests.test_gpu_decoder_ops import BF16, FLOAT, close, dev, host, pad64, padded, rand

pytestmark = pytest.mark.gpu

f8 = lambda a: np.asarray(a).astype(np.float64)
cut = lambda a, dtype: Z.bf16_round(a).astype(np.float64).reshape(np.shape(a)) if dtype == BF16 else f8(a)


@pytest.fixture(scope="module")
def D():
    d = load_package().decoder_capi
    d.lib()
    return d


def batch(D, entries, **more):
    """entries: (slot, position, tokens).  Returns (descriptor, what it points to)."""
    n = [e[2] for e in entries]
    meta = [dev(np.array(m, np.int32)) for m in ([e[0] for e in entries], [e[1] for e in entries], np.concatenate([[0], np.cumsum(n)[:-1]]), n,
                                                 np.repeat(np.arange(len(n)), n))]
    b = D.fill(D.Batch, slot=meta[0], pos=meta[1], start=meta[2], n=meta[3], token_entry=meta[4], entries=len(n), tokens=sum(n), max_n=max(n),
               max_len=max(p + m for _, p, m in entries), **more)
    return b, meta


# ---- norms, tables, linears ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("width,n", [(200, 3), (97, 70), (4096, 2), (5, 1)])
def test_norm_of_a_branch_ahead_of_the_norm(D, dtype, width, n):
    rng = np.random.default_rng(width)
    x, y = 2 * rng.standard_normal((n, width)).astype(np.float32), 9 * rng.standard_normal((n, width)).astype(np.float32)
    w, v = (rng.standard_normal(width).astype(np.float32) for _ in range(2))
    ld, eps = pad64(width), 0.3
    X, Y, out, dw, dv = padded(x, FLOAT, junk=1e9), padded(y, FLOAT, junk=1e9), padded(np.zeros((n, width)), dtype), dev(w), dev(v)
    a = D.fill(D.Norm, X=X, weight=dw, out=out, branch=Y, branch_weight=dv, n=n, width=width, ldx=ld, ldo=ld, ldb=ld, kind=D.NORM_RMS, eps=eps)
    assert D.norm(dtype, a) == 0 and D.check() == 0
    stream = f8(x) + Z.rms_norm(f8(y), v, eps)
    close(host(X)[:, :width], stream, FLOAT, "stream", 4)
    close(host(out)[:, :width], Z.rms_norm(stream, w, eps), dtype, "norm", 10 if dtype == FLOAT else 1)
    assert np.all(host(out)[:, width:] == 0)


def test_rotary_table_is_as_exact_as_floats_are(D):
    import torch

    for rows, dims, base in ((70000, 6, 1e4), (300, 128, 5e5)):
        t = torch.zeros(rows, dims // 2, 2, device="cuda")
        assert D.rotary_table(t, rows, dims, base) == 0 and D.check() == 0
        a = np.arange(rows)[:, None] * base ** (-2.0 * np.arange(dims // 2) / dims)
        assert np.abs(t.cpu().numpy() - np.stack([np.cos(a), np.sin(a)], 2)).max() < 1e-6


KERNELS = {FLOAT: [0], BF16: [1, 2]}


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("rows,N,K", [(1, 40, 97), (9, 136, 200), (33, 72, 130), (200, 260, 200)])
def test_gated_gelu_soft_cap_and_float_tail(D, dtype, rows, N, K):
    rng = np.random.default_rng(rows + N)
    w, x = rand(rng, 2 * N, K, dtype=dtype, scale=2 * K ** -0.5), rand(rng, rows, K, dtype=dtype)
    W, X = padded(w, dtype), padded(x, dtype, junk=3.0)
    z = f8(x) @ f8(w).T
    ldy = pad64(2 * N)
    base = dict(W=W, X=X, rows=rows, K=K, ldw=pad64(K), ldx=pad64(K), ldy=ldy, alpha=1.0)
    for kernel in KERNELS[dtype]:
        Y = padded(np.zeros((rows, N)), FLOAT, ldy, junk=-3.0)
        assert D.linear(dtype, [D.fill(D.Linear, Y=Y, N=N, up_row=N, activation=D.ACT_GELU_GATE, **base)], kernel=kernel) == 0
        close(host(Y)[:, :N], Z.gelu_tanh(z[:, :N]) * z[:, N:], FLOAT, ("gelu", kernel), 10)
        Y = padded(np.zeros((rows, N)), FLOAT, ldy, junk=-3.0)
        assert D.linear(dtype, [D.fill(D.Linear, Y=Y, N=N, activation=D.ACT_SOFTCAP, cap=1.7, **base)], kernel=kernel) == 0
        close(host(Y)[:, :N], Z.soft_cap(z[:, :N], 1.7), FLOAT, ("cap", kernel), 10)
        for tail in (8, N, 2 * N - 3):
            Y, Yt = padded(np.zeros((rows, 2 * N)), dtype, ldy, junk=-3.0), padded(np.zeros((rows, 2 * N)), FLOAT, ldy, junk=-4.0)
            assert D.linear(dtype, [D.fill(D.Linear, Y=Y, Y_tail=Yt, N=2 * N, tail=tail, ld_tail=ldy, out_type=dtype, **base)], kernel=kernel) == 0
            close(host(Y)[:, :tail], z[:, :tail], dtype, ("front", kernel, tail), 10 if dtype == FLOAT else 1)
            close(host(Yt)[:, :2 * N - tail], z[:, tail:], FLOAT, ("tail", kernel, tail), 10)
            assert np.all(host(Yt)[:, 2 * N:] == -4.0) and np.all(host(Y)[:, 2 * N:] == -3.0)


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("rows,blocks,N,K,x_step", [(1, 3, 40, 24, 32), (7, 5, 9, 100, 104), (40, 2, 130, 64, 80), (150, 6, 128, 200, 0), (300, 3, 72, 40, 48)])
def test_block_diagonal_linear_with_head_gates(D, dtype, rows, blocks, N, K, x_step):
    rng = np.random.default_rng(rows + blocks)
    w = rand(rng, blocks, N, K, dtype=dtype, scale=K ** -0.5)
    x = rand(rng, rows, max(x_step * blocks, K), dtype=dtype)
    g = rand(rng, rows, blocks, dtype=dtype)
    W, X, G = padded(w.reshape(-1, K), dtype), padded(x, dtype, pad64(x.shape[1]) + 64, junk=2.0), padded(g, dtype)
    y_step = N + 8
    ldy = pad64(blocks * y_step)
    cols = [x[:, b * x_step:b * x_step + K] for b in range(blocks)]
    z = np.stack([f8(c) @ f8(w[b]).T for b, c in enumerate(cols)], 1)
    for kernel in KERNELS[dtype]:
        if kernel == 1 and rows > 100:
            continue
        for gated in (False, True):
            Y = padded(np.full((rows, blocks * y_step), -3.0), dtype, ldy, junk=-3.0)
            a = D.fill(D.Linear, W=W, X=X, Y=Y, head_gate=G if gated else None, rows=rows, N=N, K=K, ldw=pad64(K), ldx=X.shape[1], ldy=ldy, blocks=blocks, group_rows=N,
                       x_step=x_step, y_step=y_step, ld_gate=G.shape[1], out_type=dtype, alpha=1.0)
            assert D.linear(dtype, [a], kernel=kernel) == 0 and D.check() == 0
            got = host(Y)[:, :blocks * y_step].reshape(rows, blocks, y_step)
            want = z * Z.sigmoid(f8(g))[:, :, None] if gated else z
            close(got[:, :, :N].reshape(rows, -1), want.reshape(rows, -1), dtype, (kernel, gated), 10 if dtype == FLOAT else 1)
            assert np.all(got[:, :, N:] == -3.0)


# ---- attention -----------------------------------------------------------------------------------------
class Attn:
    """Attention from projections on: q and k normalised over the whole projection and rotated, values = keys as projected, a
    window, sinks, gates per head."""

    def __init__(self, D, dtype, H, G, dim, window, rot, entries, interleaved=False, norm=True, sink=True, gate=True, T_max=700, slots=4, scale=0.3, seed=0):
        rng = np.random.default_rng(seed)
        self.D, self.dtype, self.H, self.G, self.dim, self.window, self.rot, self.entries = D, dtype, H, G, dim, window, rot, entries
        self.interleaved, self.T_max, self.scale, self.eps, self.base = interleaved, T_max, scale, 1e-2, 300.0
        T = self.T = sum(n for _, _, n in entries)
        self.q, self.k = rand(rng, T, H * dim, dtype=dtype), rand(rng, T, G * dim, dtype=dtype)
        self.qn, self.kn = (1 + 0.3 * rng.standard_normal(n * dim).astype(np.float32) if norm else None for n in (H, G))
        self.sink = 2 * rng.standard_normal(H).astype(np.float32) if sink else None
        self.g = rand(rng, T, H, dtype=dtype) if gate else None
        self.kc, self.vc = rand(rng, slots, G, T_max, dim, dtype=dtype), rand(rng, slots, G, T_max, dim, dtype=dtype)

    def run(self, kernel):
        import torch

        D, dt, T, H, G, d = self.D, self.dtype, self.T, self.H, self.G, self.dim
        k_off = (H * d + 7) // 8 * 8
        g_off = k_off + (G * d + 7) // 8 * 8
        ld, kl = pad64(g_off + H), d + (-d) % 16
        row = np.full((T, ld), 3.0, np.float32)
        row[:, :H * d], row[:, k_off:k_off + G * d] = self.q, self.k
        if self.g is not None:
            row[:, g_off:g_off + H] = self.g
        kc, vc = (np.zeros(c.shape[:3] + (kl,), np.float32) for c in (self.kc, self.vc))
        kc[..., :d], vc[..., :d] = self.kc, self.vc
        x, self.K, self.V, out = dev(row, dt), dev(kc, dt), dev(vc, dt), padded(np.full((T, H * d), -2.0), dt)
        work = torch.zeros(D.attention_work_bytes(d), dtype=torch.uint8, device="cuda")
        table = torch.zeros(self.T_max, max(1, self.rot // 2), 2, device="cuda")
        assert D.rotary_table(table, self.T_max, self.rot, self.base) == 0
        keep = [None if a is None else dev(a) for a in (self.qn, self.kn, self.sink)]
        gate = x.data_ptr() + g_off * x.element_size() if self.g is not None else None
        a = D.fill(D.Attention, qkvg=x, out=out, k_cache=self.K, v_cache=self.V, work=work, q_norm=keep[0], k_norm=keep[1], sink=keep[2], rotary=table, head_gate=gate,
                   ld=ld, ldo=pad64(H * d), k_off=k_off, v_off=k_off, H=H, Hkv=G, dim=d, vdim=d, k_ld=kl, v_ld=kl, T_max=self.T_max, slots=self.kc.shape[0],
                   rot_dims=self.rot, ld_gate=ld, window=self.window, rot_interleaved=int(self.interleaved), eps=self.eps, scale=self.scale)
        b, meta = batch(D, self.entries)
        assert D.attention(dt, a, b, kernel=kernel) == 0 and D.check() == 0
        return host(out)[:, :H * d].reshape(T, H, d)

    def reference(self):
        H, G, d = self.H, self.G, self.dim
        pos = np.concatenate([np.arange(p, p + n) for _, p, n in self.entries])
        q, k = f8(self.q), f8(self.k)
        if self.qn is not None:
            q, k = Z.rms_norm(q, self.qn, self.eps), Z.rms_norm(k, self.kn, self.eps)
        q, k = (Z.rotate(a.reshape(self.T, -1, d), pos, self.base, self.rot, self.interleaved) if self.rot else a.reshape(self.T, -1, d) for a in (q, k))
        q, k, v = cut(q, self.dtype), cut(k, self.dtype), f8(self.k).reshape(self.T, G, d)
        self.k_new, out, at = k, np.zeros((self.T, H, d)), 0
        for slot, p, n in self.entries:
            K = np.concatenate([f8(self.kc[slot, :, :p]).transpose(1, 0, 2), k[at:at + n]])
            V = np.concatenate([f8(self.vc[slot, :, :p]).transpose(1, 0, 2), v[at:at + n]])
            mask = Z.visible(p + n, self.window or 10 ** 9)
            Q = np.concatenate([np.zeros((p, H, d)), q[at:at + n]])
            out[at:at + n] = Z.softmax_attention(Q, K, V, self.scale, mask, self.sink)[p:]
            at += n
        return out * Z.sigmoid(f8(self.g))[:, :, None] if self.g is not None else out


KINDS = {FLOAT: [0], BF16: [0, 1, 2, 3, 4, 5]}


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("H,G,dim,rot,interleaved", [(6, 2, 40, 16, False), (4, 4, 10, 6, False), (5, 1, 72, 72, True), (3, 3, 200, 32, False), (8, 1, 128, 128, False)])
def test_norms_rotation_windows_and_sinks_in_ragged_batches(D, dtype, H, G, dim, rot, interleaved):
    ragged, decoding = [(2, 130, 3), (0, 0, 37), (3, 333, 1), (1, 64, 70)], [(1, 600, 1), (3, 0, 1), (0, 15, 1), (2, 16, 1)]
    for entries, window in ((ragged, 50), (decoding, 33), (ragged, 1), (decoding, 0)):
        a = Attn(D, dtype, H, G, dim, window, rot, entries, interleaved, seed=H * dim + window)
        want = a.reference()
        for kind in KINDS[dtype]:
            if kind == 4 and dim > 128:
                continue
            got = a.run(kind)
            close(got.reshape(a.T, -1), want.reshape(a.T, -1), dtype, (kind, window), 10 if dtype == FLOAT else 2)
            K, V, at = host(a.K)[..., :dim], host(a.V)[..., :dim], 0
            for slot, p, n in entries:      # keys turned, values as projected, everything else as it was
                step = 1e-5 if dtype == FLOAT else 2.0 ** -7
                assert np.abs(K[slot, :, p:p + n].transpose(1, 0, 2) - a.k_new[at:at + n]).max() < step * np.abs(a.k_new).max()
                assert np.array_equal(V[slot, :, p:p + n].transpose(1, 0, 2), f8(a.k[at:at + n]).reshape(n, G, dim))
                assert np.array_equal(K[slot, :, :p], f8(a.kc[slot, :, :p])) and np.array_equal(V[slot, :, p + n:], f8(a.vc[slot, :, p + n:]))
                at += n


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("pos,n", [(600, 1), (597, 4), (0, 600), (250, 200)])
@pytest.mark.parametrize("window", [1, 16, 63, 64, 65, 129, 500])
def test_one_key_inside_or_outside_the_window(D, dtype, pos, n, window):
    """A key far above all others, just inside the last row's window, just outside it, at tile borders: who sees it returns its value."""
    last = pos + n - 1
    for spot in sorted({last - window + 1, last - window, last - window + 2, last // 64 * 64, max(0, last // 64 * 64 - 1), pos}):
        if not 0 <= spot <= last:
            continue
        a = Attn(D, dtype, 4, 2, 32, window, 0, [(1, pos, n)], norm=False, sink=False, gate=False, scale=1.0, seed=spot)
        u = np.zeros(32, np.float32)
        u[3] = 8.0
        a.q[:] = (0.25 * a.q.reshape(n, 4, 32) + u).reshape(n, -1)
        a.q = Z.bf16_round(a.q).reshape(n, -1)
        if spot < pos:
            a.kc[1, :, spot], a.vc[1, :, spot] = u, 5.0
        else:
            a.k[spot - pos] = np.tile(u, 2)
        want = a.reference()
        value = np.full(32, 5.0) if spot < pos else u
        rows = np.arange(pos, pos + n)
        sees = (rows >= spot) & (rows - spot < window)
        assert sees[-1] == (spot > last - window)
        for kind in KINDS[dtype]:
            if kind in (1, 4) and n > 100:
                continue
            got = a.run(kind)
            close(got.reshape(n, -1), want.reshape(n, -1), dtype, (kind, spot), 10 if dtype == FLOAT else 2)
            near = np.abs(got - value).max(axis=(1, 2)) < 0.3
            assert np.array_equal(near, sees), (kind, spot)


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
def test_sinks_take_their_share(D, dtype):
    """Sinks far below, at and far above the scores, alone with one key and over many keys in splits."""
    for entries in ([(0, 0, 1), (1, 690, 1)], [(2, 5, 120)]):
        a = Attn(D, dtype, 4, 2, 24, 0, 0, entries, norm=False, gate=False, scale=0.4, seed=1)
        a.sink = np.array([-60.0, 0.0, 6.0, 60.0], np.float32)
        want = a.reference()
        for kind in KINDS[dtype]:
            got = a.run(kind)
            close(got.reshape(a.T, -1), want.reshape(a.T, -1), dtype, kind, 10 if dtype == FLOAT else 2)
            assert np.abs(got[:, 3]).max() < 1e-6 and np.abs(got[:, 0]).max() > 0.1


# ---- latent attention ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("q_rank,kv_rank,rot", [(72, 56, 8), (13, 11, 4), (200, 264, 64), (1536, 512, 64)])
def test_latent_rows_and_rotated_queries(D, dtype, q_rank, kv_rank, rot):
    import torch

    rng = np.random.default_rng(kv_rank)
    entries, T_max, heads, dim = [(1, 40, 3), (0, 0, 5)], 64, 3, 16
    T, kv_off, c_ld = 8, (q_rank + 7) // 8 * 8, kv_rank + rot + (-(kv_rank + rot)) % 16
    x = rand(rng, T, kv_off + kv_rank + rot, dtype=dtype, scale=3.0)
    qn, kn = (1 + 0.3 * rng.standard_normal(r).astype(np.float32) for r in (q_rank, kv_rank))
    X, cq, cache = padded(x, dtype), padded(np.full((T, q_rank), -1.0), dtype), padded(np.full((2 * T_max, c_ld), -5.0), dtype, c_ld)
    table = torch.zeros(T_max, rot // 2, 2, device="cuda")
    assert D.rotary_table(table, T_max, rot, 100.0) == 0
    b, meta = batch(D, entries)
    keep = [dev(qn), dev(kn)]
    a = D.fill(D.Latent, down=X, cq=cq, cache=cache, q_norm=keep[0], kv_norm=keep[1], rotary=table, ld=X.shape[1], ld_cq=cq.shape[1], kv_off=kv_off, q_rank=q_rank,
               kv_rank=kv_rank, rot_dim=rot, c_ld=c_ld, T_max=T_max, eps=0.1)
    assert D.latent_down(dtype, a, b) == 0 and D.check() == 0
    pos = np.array([40, 41, 42, 0, 1, 2, 3, 4])
    close(host(cq)[:, :q_rank], Z.rms_norm(f8(x[:, :q_rank]), qn, 0.1), dtype, "query latent", 10 if dtype == FLOAT else 1)
    rows = host(cache).reshape(2, T_max, c_ld)
    got = np.concatenate([rows[1, 40:43], rows[0, :5]])
    close(got[:, :kv_rank], Z.rms_norm(f8(x[:, kv_off:kv_off + kv_rank]), kn, 0.1), dtype, "latent", 10 if dtype == FLOAT else 1)
    turned = Z.rotate(f8(x[:, None, kv_off + kv_rank:]), pos, 100.0, rot, True)[:, 0]
    close(got[:, kv_rank:kv_rank + rot], turned, dtype, "rotated", 10 if dtype == FLOAT else 1)
    assert np.all(rows[0, 5:] == -5) and np.all(rows[1, :40] == -5) and np.all(got[:, kv_rank + rot:] == -5)
    # queries: the rotated parts of every head, elsewhere and in place
    q = rand(rng, T, heads * (dim + rot), dtype=dtype)
    want = Z.rotate(f8(q).reshape(T, heads, dim + rot)[..., dim:], pos, 100.0, rot, True)
    Q, out = padded(q, dtype), padded(np.full((T, heads * (rot + 8)), -1.0), dtype)
    for dst, step, off in ((out, rot + 8, 8), (Q, dim + rot, dim)):
        assert D.latent_query(dtype, Q, Q.shape[1], dim + rot, dim, dst, dst.shape[1], step, off, heads, rot, table, T_max, b) == 0 and D.check() == 0
        y = host(dst)[:, :heads * step].reshape(T, heads, step)
        close(y[..., off:off + rot].reshape(T, -1), want.reshape(T, -1), dtype, "query", 10 if dtype == FLOAT else 1)
    assert np.all(host(out)[:, :heads * (rot + 8)].reshape(T, heads, -1)[..., :8] == -1)
    assert np.array_equal(host(Q)[:, :heads * (dim + rot)].reshape(T, heads, -1)[..., :dim], f8(q).reshape(T, heads, -1)[..., :dim])


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
def test_expanding_cached_latents(D, dtype):
    """Rows of several sequences, from their windows' first on, one behind the other; rotated parts beside every head's key."""
    rng = np.random.default_rng(3)
    kv, rot, heads, dim, T_max, window = 24, 8, 3, 16, 50, 10
    entries = [(0, 30, 12), (1, 0, 20), (0, 0, 1)]
    c = rand(rng, 2, T_max, kv + rot, dtype=dtype)
    b, meta = batch(D, entries)
    before = [min(p, window - 1) for _, p, _ in entries]
    floor = np.cumsum([0] + [x + n for x, (_, _, n) in zip(before, entries)])
    cache, C_, K = padded(c.reshape(-1, kv + rot), dtype, 32), padded(np.full((64, kv), -1.0), dtype), padded(np.full((heads * 64, 32), -1.0), dtype, 32)
    keep = [dev(np.array(m, np.int32)) for m in (floor[:3], floor[:3] + before)]
    a = D.fill(D.Expand, cache=cache, c=C_, K=K, floor=keep[0], pos2=keep[1], c_ld=32, T_max=T_max, kv_rank=kv, rot_dim=rot, ld_c=C_.shape[1], k_ld=32, T=64, dim=dim,
               heads=heads, max_rows=21)
    assert D.latent_expand(dtype, a, b) == 0 and D.check() == 0
    want = np.concatenate([c[s, p - x:p + n] for (s, p, n), x in zip(entries, before)])
    assert np.array_equal(host(C_)[:len(want), :kv], f8(want[:, :kv])) and np.all(host(C_)[len(want):, :kv] == -1)
    k = host(K).reshape(heads, 64, 32)
    assert np.all(k[..., :dim] == -1)
    for h in range(heads):
        assert np.array_equal(k[h, :len(want), dim:dim + rot], f8(want[:, kv:]))


class LatentAttn:
    """Ready queries against latent rows: one key/value head, values the first columns of the key rows."""

    def __init__(self, D, dtype, H, dim, vdim, window, entries, T_max=900, slots=3, scale=0.2, sink=False, seed=0):
        rng = np.random.default_rng(seed)
        self.D, self.dtype, self.H, self.dim, self.vdim, self.window, self.entries, self.scale, self.T_max = D, dtype, H, dim, vdim, window, entries, scale, T_max
        self.T = sum(n for _, _, n in entries)
        self.q, self.c = rand(rng, self.T, H, dim, dtype=dtype), rand(rng, slots, T_max, dim, dtype=dtype)
        self.sink = 2 * rng.standard_normal(H).astype(np.float32) if sink else None

    def run(self, kernel, q_ld=None, floor=None, T=None):
        import torch

        D, dt, H = self.D, self.dtype, self.H
        q_ld = q_ld or self.dim + (-self.dim) % 16
        ld, c_ld = pad64(H * q_ld), self.dim + (-self.dim) % 16
        q = np.zeros((self.T, H, q_ld), np.float32)
        q[..., :self.dim] = self.q
        x, cache = padded(q.reshape(self.T, -1), dt, ld), padded(self.c.reshape(-1, self.dim), dt, c_ld)
        out = padded(np.full((self.T, H * self.vdim), -2.0), dt)
        work = torch.zeros(D.attention_work_bytes(self.vdim), dtype=torch.uint8, device="cuda")
        keep = [None if self.sink is None else dev(self.sink), None if floor is None else dev(np.array(floor, np.int32))]
        a = D.fill(D.Attention, qkvg=x, out=out, k_cache=cache, v_cache=cache, work=work, sink=keep[0], ld=ld, ldo=out.shape[1], H=H, Hkv=1, dim=self.dim, vdim=self.vdim,
                   k_ld=c_ld, v_ld=c_ld, T_max=self.T_max, slots=self.c.shape[0], q_ld=q_ld, window=self.window, no_append=1, scale=self.scale)
        b, meta = batch(D, self.entries, **({} if floor is None else dict(floor=keep[1])))
        assert D.attention(dt, a, b, kernel=kernel) == 0 and D.check() == 0
        return host(out)[:, :H * self.vdim].reshape(self.T, H, self.vdim)

    def reference(self, floor=None):
        out, at = np.zeros((self.T, self.H, self.vdim)), 0
        for e, (slot, p, n) in enumerate(self.entries):
            rows = f8(self.c[slot, :p + n])[:, None]
            mask = Z.visible(p + n, self.window or 10 ** 9)
            if floor is not None:
                mask = mask & (np.arange(p + n) >= floor[e])
            Q = np.concatenate([np.zeros((p, self.H, self.dim)), f8(self.q[at:at + n])])
            with np.errstate(invalid="ignore"):
                out[at:at + n] = Z.softmax_attention(Q, rows, rows[..., :self.vdim], self.scale, mask, self.sink)[p:]
            at += n
        return out


@pytest.mark.parametrize("dtype,kinds", [(FLOAT, [0]), (BF16, [0, 3, 6])])
@pytest.mark.parametrize("H,dim,vdim,window", [(6, 64, 56, 33), (3, 15, 11, 5), (32, 576, 512, 0), (5, 330, 264, 100), (40, 144, 128, 64), (1, 10, 8, 1), (2, 200, 72, 200)])
def test_latent_attention_of_few_tokens(D, dtype, kinds, H, dim, vdim, window):
    for entries in ([(0, 0, 1)], [(2, 700, 1), (0, 63, 1), (1, 64, 1)], [(1, 300, 8), (2, 5, 2), (0, 0, 8), ]):
        a = LatentAttn(D, dtype, H, dim, vdim, window, entries, sink=len(entries) == 3, scale=dim ** -0.5, seed=dim)
        want = a.reference()
        for kind in kinds:
            got = a.run(kind)
            close(got.reshape(a.T, -1), want.reshape(a.T, -1), dtype, (kind, len(entries)), 10 if dtype == FLOAT else 2)


@pytest.mark.parametrize("dtype,kinds", [(FLOAT, [0]), (BF16, [3, 6])])
@pytest.mark.parametrize("window", [0, 1, 64, 65, 300])
def test_one_latent_row_inside_or_outside_the_window(D, dtype, kinds, window):
    """Scores that grow by far more than the running maximum allows without rescaling; window edges; splits."""
    pos, n, dim, vdim = 640, 3, 48, 40
    last = pos + n - 1
    for spot in sorted({0, 63, 64, 320, last, last - 1} | ({last - window + 1, last - window, pos - window + 1} if window else set())):
        a = LatentAttn(D, dtype, 5, dim, vdim, window, [(1, pos, n)], scale=1.0, seed=spot)
        u = np.zeros(dim, np.float32)
        u[44] = 9.0
        a.q[:] = Z.bf16_round(0.2 * a.q + u).reshape(a.q.shape)
        a.c[1, spot], a.c[1, spot, :vdim] = u, 5.0
        want = a.reference()
        rows = np.arange(pos, pos + n)
        sees = (rows >= spot) & ((rows - spot < window) if window else True)
        for kind in kinds:
            got = a.run(kind)
            close(got.reshape(n, -1), want.reshape(n, -1), dtype, (kind, spot), 10 if dtype == FLOAT else 2)
            assert np.array_equal(np.abs(got - 5.0).max(axis=(1, 2)) < 0.3, sees), (kind, spot)


def test_keys_below_an_entrys_floor_are_not_seen(D):
    entries, floor = [(1, 130, 2), (1, 400, 1), (0, 70, 60)], [100, 385, 3]
    a = LatentAttn(D, BF16, 4, 64, 64, 50, entries, seed=2)
    want = a.reference(floor)
    for kind in (1, 2, 3, 4, 5, 6):
        got = a.run(kind, floor=floor)
        close(got.reshape(a.T, -1), want.reshape(a.T, -1), BF16, kind, 2)


# ---- mLSTM -------------------------------------------------------------------------------------------------
class Mlstm:
    """Sequences in slots, run in pieces; the plain recurrence over all their tokens."""

    def __init__(self, D, dtype, heads, dim, vdim, lengths, cap=8.0, slots=4, seed=0, forget=4.0):
        import torch

        rng = np.random.default_rng(seed)
        self.D, self.dtype, self.heads, self.dim, self.vdim, self.cap, self.eps = D, dtype, heads, dim, vdim, cap, 1e-3
        H, qk, v = heads, heads * dim, heads * vdim
        pad8 = lambda n: (n + 7) // 8 * 8
        self.off = [0, pad8(qk), 2 * pad8(qk), 2 * pad8(qk) + pad8(v)]
        self.f_off, self.ld = pad8(H), pad64(2 * pad8(qk) + 2 * pad8(v))
        self.bias, self.norm = rng.standard_normal(2 * H).astype(np.float32), 1 + 0.3 * rng.standard_normal(v).astype(np.float32)
        self.bias[H:] += forget
        self.seq = []
        for n in lengths:
            q = rand(rng, n, qk, dtype=dtype)
            k = rand(rng, n, qk, dtype=dtype, scale=0.5) + q       # scores that do not cancel
            k = Z.bf16_round(k).reshape(k.shape) if dtype == BF16 else k
            self.seq.append((q, k, rand(rng, n, v, dtype=dtype), rand(rng, n, v, dtype=dtype), 3 * rng.standard_normal((n, 2 * H)).astype(np.float32)))
        self.stride = D.mlstm_state_floats(dim, vdim)
        self.state = torch.full((slots, heads, self.stride), 7.0, device="cuda")       # an old sequence's
        self.at, self.torch = [0] * len(lengths), torch

    def run(self, pieces, kernel):
        """pieces: (sequence, slot, tokens).  Returns the outputs, one array per piece."""
        D, H, T = self.D, self.heads, sum(n for _, _, n in pieces)
        x, g = np.full((T, self.ld), 2.0, np.float32), np.full((T, pad64(2 * self.f_off)), 9.0, np.float32)
        row = 0
        for s, _, n in pieces:
            at = self.at[s]
            for part, off in zip(self.seq[s][:4], self.off):
                x[row:row + n, off:off + part.shape[1]] = part[at:at + n]
            gates = self.seq[s][4][at:at + n]
            g[row:row + n, :H], g[row:row + n, self.f_off:self.f_off + H] = gates[:, :H], gates[:, H:]
            row += n
        X, G, out = dev(x, self.dtype), dev(g), padded(np.full((T, H * self.vdim), -2.0), self.dtype)
        work = self.torch.full((D.mlstm_work_floats(T, len(pieces), H, self.dim, self.vdim),), float("nan"), device="cuda")
        keep = [dev(self.bias), dev(self.norm)]
        a = D.fill(D.Mlstm, qkvg=X, gates=G, bias=keep[0], norm=keep[1], out=out, state=self.state, work=work, ld=self.ld, ld_gates=g.shape[1], ldo=out.shape[1],
                   k_off=self.off[1], v_off=self.off[2], g_off=self.off[3], f_off=self.f_off, heads=H, dim=self.dim, vdim=self.vdim, cap=self.cap, eps=self.eps,
                   q_scale=self.dim ** -0.5)
        b, meta = batch(D, [(slot, self.at[s], n) for s, slot, n in pieces])
        assert D.mlstm(self.dtype, a, b, kernel=kernel) == 0 and D.check() == 0
        y, row, got = host(out), 0, []
        assert np.all(y[:, H * self.vdim:] == 0)
        for s, _, n in pieces:
            got.append(y[row:row + n, :H * self.vdim])
            self.at[s] += n
            row += n
        return got

    def reference(self, s):
        q, k, v, g, gates = (f8(a) for a in self.seq[s])
        T, H = len(q), self.heads
        z = Z.soft_cap(gates + self.bias, self.cap)
        o = Z.mlstm_recurrence(q.reshape(T, H, -1) * self.dim ** -0.5, k.reshape(T, H, -1), v.reshape(T, H, -1), z[:, :H], Z.log_sigmoid(z[:, H:]))
        return Z.rms_norm(o, 1.0, self.eps).reshape(T, -1) * self.norm * Z.sigmoid(g)

    def fits(self, kernel, n):
        if kernel == 2:
            return n <= 8 and self.dim <= 512
        return kernel != 3 or (self.dim % 16 == 0 and self.vdim % 8 == 0 and self.dim <= 256)


MSIZES = [(3, 40, 56), (2, 7, 5), (2, 48, 72), (1, 16, 8), (4, 64, 64), (2, 208, 320), (8, 256, 512), (1, 512, 24), (2, 136, 104), (1, 16, 1024)]


@pytest.mark.parametrize("dtype", [FLOAT, BF16])
@pytest.mark.parametrize("heads,dim,vdim", MSIZES)
def test_mlstm_in_pieces_of_every_kind(D, dtype, heads, dim, vdim):
    """Token by token, in small pieces, in chunks cut anywhere, by every kernel and by turns; states carried in slots."""
    total = 150 if dim * vdim > 40000 else 300
    plans = {"tokens": [1] * 40 + [8] * 50, "small": [2, 3, 8, 5, 1] * 60, "chunks": [total - 20, 20], "cut": [9, 128, 1, 70, 8, 33, 127] * 3}
    for name, plan in plans.items():
        m = Mlstm(D, dtype, heads, dim, vdim, [total], seed=dim)
        want = m.reference(0)
        kernels = [1] if dtype == FLOAT else [0, 1, 2, 3]
        got, turn = [], 0
        while m.at[0] < total:
            n = min(plan[turn % len(plan)], total - m.at[0])
            able = [k for k in kernels if m.fits(k, n)]
            got += m.run([(0, 2, n)], able[turn % len(able)])
            turn += 1
        e = np.abs(np.concatenate(got) - want).max(axis=1) / np.abs(want).max(axis=1)
        bar = 2e-5 if dtype == FLOAT else 8e-3
        assert np.quantile(e, 0.97) < bar and e.max() < 20 * bar, (name, int(e.argmax()), e.max(), np.quantile(e, 0.97))
        state = m.state.cpu().numpy()
        assert np.all(state[[0, 1, 3]] == 7.0) and np.all(np.isfinite(state))


@pytest.mark.parametrize("kernel", [0, 1, 2, 3])
def test_mlstm_entries_side_by_side(D, kernel):
    """Unequal entries in one launch, in any slots, beside one another in every way the scratch memory lays chunks out."""
    lengths = [8, 3, 8, 1] if kernel == 2 else [300, 5, 128, 129]
    m = Mlstm(D, BF16, 2, 32, 40, [2 * n for n in lengths], seed=5)
    want = [m.reference(s) for s in range(4)]
    order, slots = [2, 0, 3, 1], [1, 3, 0, 2]
    got = {s: [] for s in range(4)}
    for _ in range(2):
        for s, y in zip(order, m.run([(s, slots[s], lengths[s]) for s in order], kernel)):
            got[s].append(y)
    for s in range(4):
        e = np.abs(np.concatenate(got[s]) - want[s]).max(axis=1) / np.abs(want[s]).max(axis=1)
        assert np.median(e) < 8e-3 and e.max() < 0.1, (s, e.max())


@pytest.mark.parametrize("dtype,kernel", [(FLOAT, 1), (BF16, 1), (BF16, 2), (BF16, 3)])
def test_mlstm_gates_at_their_extremes(D, dtype, kernel):
    """Gates that shut, reset and keep everything: running maxima that fall below zero and jump, outputs that rest on the floor of the
    denominator, a key from the first token read by the last."""
    for what in ("reset", "shut", "keep"):
        n = 8 if kernel == 2 else 260
        m = Mlstm(D, dtype, 2, 32, 24, [n], cap=15.0, seed=7, forget=0.0)
        g = m.seq[0][4]
        if what == "reset":
            g[:, 2:] = 40.0
            g[n // 2 - 1, 2:] = -60.0
            g[n // 4, :2] = 30.0
        elif what == "shut":
            g[:, :2], g[:, 2:] = -60.0, -2.0
        else:
            g[:, :2], g[:, 2:] = -40.0, 60.0
            g[0, :2] = 30.0
        want = m.reference(0)
        got = np.concatenate(m.run([(0, 1, n)], kernel))
        e = np.abs(got - want).max(axis=1) / np.maximum(np.abs(want).max(axis=1), 1e-3)
        bar = 5e-5 if dtype == FLOAT else 1e-2
        assert np.quantile(e, 0.95) < bar and e.max() < 20 * bar, (what, e.max(), int(e.argmax()))
