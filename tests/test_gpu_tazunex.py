"""The Tazunex decoder through the serving interface - registry, loader, cache slots and recurrent states, steps, scheduler,
generation loop, command line - against the plain statement in oracle/tazunex.py, on small random models."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from __graft_entry__ import ROOT, load_package
from oracle import tazunex as Z

pytestmark = pytest.mark.gpu

# error of a row of logits (rms) over the logits' standard deviation: the worst row's, the median row's.  In 16 bits single rows are
# ill conditioned (where an mLSTM's scores cancel), the others are not.
BAR = {"float32": (3e-5, 1e-5), "bfloat16": (0.08, 0.015)}


def attn(heads, kv, dim, window, rot, scale=None, base=1e4):
    return "attention", dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale or dim ** -0.5, mask=dict(size=window), rot=dict(base=base, dims=rot))


def latent(heads, dim, rot, vdim, q_rank, kv_rank, window, scale=None, base=2e4):
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale or (dim + rot) ** -0.5,
                                    mask=dict(size=window), rot=dict(base=base, dims=rot))


def mlstm(heads, dim, vdim, cap=12.0):
    return "mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def config(width, vocab, layers, eps=1e-5, cap=20.0):
    out = []
    for L in layers:
        if isinstance(L, int):
            out.append(dict({k: v for k, v in out[L].items() if k != "weights_of"}, weights_of=L))
        else:
            (kind, mixer), ff = L
            out.append(dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=ff) if ff else None))
    return dict(architecture="Tazunex", width=width, vocab=vocab, norm=dict(eps=eps), logit_softcap=cap, layers=out)


CONFIGS = {
    # unlike layers, a layer without feed-forward, tensors shared directly and through another layer
    "mixed": config(200, 331, [(latent(5, 24, 8, 40, 72, 56, 33), 136), (mlstm(3, 40, 56), 88), (attn(6, 3, 48, 70, 16), None), 1, 3, 0, (mlstm(2, 136, 72), 64), 2]),
    # sizes that are multiples of nothing
    "odd": config(97, 53, [(attn(6, 2, 10, 9, 6), 33), (mlstm(3, 7, 5), 19), (latent(3, 9, 4, 7, 13, 11, 5), 21), (mlstm(5, 12, 20, 3.0), 27)], eps=1e-3),
    # large heads: 192-element keys, a latent of 264, states of 200 x 320
    "large": config(264, 410, [(latent(2, 128, 64, 128, 200, 264, 150), 96), (attn(4, 2, 192, 100, 192), 80), (mlstm(2, 200, 320), 72), (attn(2, 1, 264, 200, 8), 64)]),
    # one of everything
    "ones": config(64, 40, [(attn(1, 1, 16, 1, 16), 8), (latent(1, 16, 2, 8, 8, 8, 1), 8), (mlstm(1, 16, 24), 16)], cap=2.0),
}


@pytest.fixture(scope="module")
def serve():
    return load_package().serve


def write(d, c, w):
    (d / "config.json").write_text(json.dumps(c))
    Z.write_safetensors(str(d / "model.safetensors"), w)
    return str(d)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, c in CONFIGS.items():
        w = Z.random_weights(c, seed=len(name))
        out[name] = (write(tmp_path_factory.mktemp(name), c, w), c, w)
    return out


_known = {}


def forward(c, w, tokens):
    """The plain logits, once per model and prompt."""
    key = (json.dumps(c), tuple(tokens), float(np.abs(w["embed"]).sum()))
    if key not in _known:
        _known[key] = Z.forward(c, w, tokens)
    return _known[key]


def tokens_for(c, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, c["vocab"], n)]


def errors(got, want):
    return np.sqrt(((np.atleast_2d(got) - np.atleast_2d(want)) ** 2).mean(1)) / want.std()


def check(got, want, dtype, what="", factor=1.0):
    e = errors(got, want)
    assert e.max() < factor * BAR[dtype][0] and np.median(e) < factor * BAR[dtype][1], (what, e.max(), int(e.argmax()), np.median(e))


def feed(m, slot, tokens, cuts):
    rows, at = [], 0
    for n in cuts:
        n = min(n, len(tokens) - at)
        if n <= 0:
            break
        lg, _ = m.step([(slot, tokens[at:at + n], range(n))])
        rows.append(np.array(lg, np.float64).reshape(n, -1))
        at += n
    assert at == len(tokens)
    return np.concatenate(rows)


CUTS = {"whole": [10 ** 6], "tokens": [1] * 10 ** 4, "twos": [2, 3] * 10 ** 4, "unequal": [45, 2, 68, 33, 1, 1, 31, 64, 7, 9] * 100, "prompt then tokens": [150] + [1] * 10 ** 4,
        "eights and nines": [8, 9] * 1000}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_logits_do_not_depend_on_the_cuts(serve, folders, name, dtype):
    d, c, w = folders[name]
    tokens = tokens_for(c, 290, 1)
    want = forward(c, w, tokens)
    factor = 2.5 if name == "ones" else 1.0      # little but rounding there: single heads of few elements
    m = serve.Model(d, dtype=dtype, max_context=300, max_sequences=2, max_step_tokens=200)      # the whole prompt takes two passes
    ref = None
    for how, cuts in CUTS.items():
        slot = m.open_slot()
        got = feed(m, slot, tokens, cuts)
        assert m.slot_length(slot) == len(tokens)
        m.close_slot(slot)
        for part, rows in (("all", slice(None)), ("first", slice(0, 3)), ("last", slice(-3, None))):
            check(got[rows], want[rows], dtype, (how, part), factor * (1.0 if part == "all" else 2.0))
        ref = got if ref is None else ref
        check(got, ref, dtype, how, factor)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_sharp_attention_at_the_edge_of_the_window(serve, tmp_path, kind, dtype):
    """Token t's query is token t + 150's key: it reads that one and itself, where it stands inside the window."""
    window = 61
    layer = attn(4, 2, 32, window, 4, scale=0.7) if kind == "attention" else latent(4, 32, 4, 24, 48, 48, window, scale=0.7)
    c = config(128, 300, [(layer, None), (layer, 96)])
    w = Z.random_weights(c, 3)
    turn = np.linalg.qr(np.random.default_rng(4).standard_normal((128, 128)))[0]
    w["embed"] = np.random.default_rng(5).standard_normal((300, 128)) * 0.25
    w["embed"][150:] = w["embed"][:150] @ turn.T
    w["l0.norm1"][:] = 1.0
    w["l0.norm1b"] *= 4
    if kind == "attention":
        k = w["l0.mix.k"] @ turn
        w["l0.mix.q"] = np.concatenate([k[:32], k[:32], k[32:], k[32:]])
        w["l0.mix.q.norm"][:] = w["l0.mix.k.norm"][:] = 1.0
        w["l0.mix.sink"][:] = [-3, 0, 2, 9]
    else:
        w["l0.mix.dq"], w["l0.mix.dq.norm"] = w["l0.mix.dkv"][:48] @ turn, w["l0.mix.dkv.norm"].copy()
        w["l0.mix.uq"].reshape(4, 36, 48)[:, :32] = w["l0.mix.uk"].reshape(4, 32, 48)
    w = {n: Z.bf16_round(a).reshape(a.shape) for n, a in w.items()}
    tokens = [150 + int(t) for t in np.random.default_rng(2).permutation(150)[:110]]
    for g in [window - 1, window, 80, window + 1, 1, window - 2, 30] * 30:      # the partner of what stands so far back
        back = tokens[max(0, len(tokens) - g)]
        tokens.append(back - 150 if back >= 150 else back + 150)
    want = forward(c, w, tokens)
    # the case is as sharp as it is meant to be: another window gives other logits
    for by in (-1, 1):
        other = json.loads(json.dumps(c))
        for L in other["layers"]:
            L["mixer"]["mask"]["size"] += by
        far = np.sqrt(((forward(other, w, tokens) - want) ** 2).mean(1)) / want.std()
        assert (far > 0.2).mean() > 0.03
    m = serve.Model(write(tmp_path, c, w), dtype=dtype, max_context=512)
    for cuts in ([400], [100] + [1] * 230, [64] * 6, [2, 7] * 50):
        slot = m.open_slot()
        got = feed(m, slot, tokens, cuts)
        m.close_slot(slot)
        check(got, want, dtype, cuts[:2], 2.0)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_slots_and_reuse(serve, folders, dtype):
    """Requests of unequal length share steps, come and go, and take over slots: each gets the logits it gets alone."""
    d, c, w = folders["mixed"]
    rng = np.random.default_rng(9)
    m = serve.Model(d, dtype=dtype, max_context=160, max_sequences=3, max_step_tokens=128)
    todo = [tokens_for(c, n, 100 + n) for n in (1, 150, 37, 64, 5, 129, 90, 2, 160, 33)]
    want = [forward(c, w, t) for t in todo]
    live, queue, got, seen_slots = {}, list(range(len(todo))), {i: [] for i in range(len(todo))}, []
    while live or queue:
        while queue and len(live) < 3:
            live[queue.pop(0)] = [m.open_slot(), 0]
        entries, plan = [], []
        for i, (slot, at) in live.items():
            n = min(int(rng.choice([1, 1, 2, 3, 20, 70])), len(todo[i]) - at)
            entries.append((slot, todo[i][at:at + n], range(n)))
            plan.append((i, n))
            seen_slots.append((i, slot))
        lg, ch = m.step(entries, choice=True)
        rows, k = np.array(lg, np.float64).reshape(-1, c["vocab"]), 0
        assert list(np.argmax(rows, axis=1)) == ch
        for i, n in plan:
            got[i].append(rows[k:k + n])
            k += n
            live[i][1] += n
            if live[i][1] == len(todo[i]):
                m.close_slot(live[i][0])
                del live[i]
    assert len({s for _, s in seen_slots}) == 3 and len({(i, s) for i, s in seen_slots}) == len(todo)
    for i in range(len(todo)):
        check(np.concatenate(got[i]), want[i], dtype, i, 1.5)
    # entries that cannot run leave everything as it is, states included
    slot = m.open_slot()
    m.step([(slot, [1, 2], [])])
    for bad in ([(slot, [c["vocab"]], [0])], [(slot, [-1], [0])], [(slot, [1] * 159, [0])], [(slot, [1], [1])], [(slot, [1], [0]), (slot, [2], [0])]):
        with pytest.raises(RuntimeError, match="cannot run"):
            m.step(bad)
    assert m.slot_length(slot) == 2
    lg, _ = m.step([(slot, [3], [0])])
    check(np.array(lg, np.float64), forward(c, w, [1, 2, 3])[2], dtype, "kept", 3)
    m.close()


def test_many_prompts_in_one_step(serve, folders):
    """More expanded latent rows than go together at a time, chunks of many entries, beside sequences that decode."""
    d, c, w = folders["mixed"]
    m = serve.Model(d, max_context=64, max_sequences=40, max_step_tokens=96)
    todo = [tokens_for(c, 9 + 5 * (i % 10), i) for i in range(40)]
    slots = [m.open_slot() for _ in todo]
    m.step([(s, t[:-3], []) for s, t in zip(slots, todo)])
    lg, _ = m.step([(s, t[-3:] if i % 2 else t[-3:-1], [1]) for i, (s, t) in enumerate(zip(slots, todo))])
    rows = np.array(lg, np.float64).reshape(40, -1)
    check(rows, np.stack([forward(c, w, t)[-2] for t in todo]), "bfloat16")
    m.close()


def test_long_decoding(serve, folders):
    """Hundreds of tokens one by one, over changes of the split count, far past every window."""
    for name, n in (("odd", 500), ("large", 320)):
        d, c, w = folders[name]
        tokens = tokens_for(c, n, 4)
        want = forward(c, w, tokens)
        m = serve.Model(d, max_context=n)
        slot = m.open_slot()
        got = feed(m, slot, tokens, [1] * n)
        check(got, want, "bfloat16", name)
        with pytest.raises(RuntimeError, match="cannot run"):
            m.step([(slot, [0], [0])])
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_carries_a_token_from_far_back(serve, tmp_path, dtype):
    """Forget gates near one, input gates that open for one token only: what it wrote is read hundreds of tokens later."""
    c = config(96, 60, [(mlstm(2, 16, 24, 15.0), 32), (mlstm(2, 32, 16, 15.0), None)])
    w = Z.random_weights(c, 8)
    for i in range(2):
        w[f"l{i}.mix.f"][:], w[f"l{i}.mix.f.b"][:] = 0.0, 14.0
        w[f"l{i}.mix.i.b"][:] = -6.0
    tokens = tokens_for(c, 400, 6)
    other = [(tokens[0] + 1) % 60] + tokens[1:]
    want = forward(c, w, tokens)
    assert errors(forward(c, w, other)[-1], want[-1])[0] > 0.02
    m = serve.Model(write(tmp_path, c, w), dtype=dtype, max_context=400)
    for cuts in ([400], [130] + [1] * 270, [2, 77] * 20):
        slot = m.open_slot()
        check(feed(m, slot, tokens, cuts), want, dtype, cuts[:2])
        m.close_slot(slot)
    m.close()


def greedy(c, w, prompt, n):
    out = []
    for _ in range(n):
        out.append(int(np.argmax(Z.forward(c, w, prompt + out)[-1])))
    return out


def test_greedy_generation_loop_scheduler_and_command_line(serve, folders):
    d, c, w = folders["mixed"]
    prompts = [tokens_for(c, n, n) for n in (5, 61, 1, 18, 33)]
    want = [greedy(c, w, p, 8) for p in prompts]
    m = serve.Model(d, dtype="float32", max_context=128, max_sequences=2)
    for p, g in zip(prompts, want):
        ids, stats = m.generate(p, 8, portion=7)
        assert ids == g and stats["prefill_tokens"] == len(p) and stats["rebuilds"] == 0
    for budget in (3, 40, 1000):
        got, _ = m.generate_many(prompts + [[], [0] * 129], 8, step_tokens=budget)
        assert got[:5] == want and got[5:] == [None, None]
    a, _ = m.generate_many(prompts, 6, seed=3, sampler=dict(temperature=0.9, top_k=12))
    b, _ = m.generate_many(prompts, 6, seed=3, sampler=dict(temperature=0.9, top_k=12), step_tokens=5)
    assert a == b and a != [g[:6] for g in want]
    m.close()
    # in 16 bits every chosen token is at least nearly the largest
    m = serve.Model(d, max_context=128, max_sequences=3)
    got, _ = m.generate_many(prompts, 8, step_tokens=40)
    for p, ids in zip(prompts, got):
        z = Z.forward(c, w, p + ids)[len(p) - 1:-1]
        assert np.all(z[np.arange(8), ids] > z.max(1) - 0.1 * z.std())
    m.close()
    cmd = [sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", d, "--dtype", "float32", "--max-new", "8"]
    for p in prompts[:2]:
        cmd += ["--prompt", ",".join(map(str, p))]
    out = subprocess.run(cmd, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert [[int(x) for x in line.split(",")] for line in out.stdout.split()] == want[:2]


def test_trace_runner(serve, folders, tmp_path):
    d, c, w = folders["odd"]
    a, b = tokens_for(c, 40, 7), tokens_for(c, 9, 8)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:33], want=[0, 32])], end=[]), dict(step=1, entries=[dict(id="b", tokens=b, want=[8])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=a[33:39], want=[])], end=[]), dict(step=5, entries=[dict(id="a", tokens=a[39:], want=[0])], end=["a"])]
    for dtype in ("float32", "bfloat16"):
        out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "60"],
                             input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert out.returncode == 0, out.stderr
        assert [x for x in out.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 5"]
        za, zb = forward(c, w, a), forward(c, w, b)
        for step, want in ((0, za[[0, 32]]), (1, zb[[8]]), (5, za[[39]])):
            got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(-1, c["vocab"])
            assert got.shape == want.shape
            check(got, want, dtype, step, 3)
        assert not os.path.exists(tmp_path / "2.f32")
