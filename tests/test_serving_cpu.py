"""No GPU needed: the serving library's exports and registry, what it says about model folders it cannot serve, and the
plain decoder statement the GPU tests rest on."""
import importlib.util
import json
import os
import re

import numpy as np
import pytest

from __graft_entry__ import ROOT, load_package
from oracle import fakilorn as F
from oracle import tazunex as Z


def test_decoder_library_exports_its_header():
    d = load_package().decoder_capi
    L = d.lib()
    header = open(os.path.join(ROOT, "include", "cccc_b200_decoder.h")).read()
    declared = set(re.findall(r"C_EXPORT\s+[\w\s\*]+?\b(cuda_b200_\w+)\s*\(", header))
    assert declared == set(d.SYMBOLS)
    for name in declared:
        assert getattr(L, name) is not None


def test_all_architectures_are_registered():
    import ctypes as C

    s = load_package().serve
    buf = C.create_string_buffer(256)
    for name in ("Fakilorn", "Tazunex"):
        s.library(name).cccc_model_architectures(buf, 256)
        assert name in buf.value.decode().split()
    s.library("cccc-llm").cccc_model_architectures(buf, 256)
    assert {"Fakilorn", "Tazunex", "cccc-llm"} <= set(buf.value.decode().split())


BASE = dict(architecture="Fakilorn", width=48, vocab=20, embedding=dict(scale=2.0), logit_scale=1.0, norm=dict(eps=1e-5),
            layers=[dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.3, v_mix=True), mlp=dict(kind="dense", ff=24)),
                    dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.3, v_mix=True),
                         mlp=dict(kind="moe", router=dict(experts=3, top=2), expert=dict(ff=16), shared=dict(ff=8)))])


def changed(path, value):
    c = json.loads(json.dumps(BASE))
    at = c
    for p in path[:-1]:
        at = at[p]
    at[path[-1]] = value
    return c


@pytest.mark.parametrize("path,value,says", [
    (["architecture"], "Nobody", "no model class"),
    (["layers", 0, "type"], "scan", "no mixer of type 'scan'"),
    (["layers", 0, "mlp", "kind"], "sparse", "no feed-forward of kind 'sparse'"),
    (["layers", 1, "mixer", "heads"], 3, "multiple of kv_heads"),
    (["layers", 1, "mixer", "vdim"], 5, "values of one size"),
    (["layers", 1, "mlp", "router", "top"], 4, "top must lie between"),
    (["layers", 0, "mixer", "scale"], None, "scale is needed"),
    (["norm", "eps"], None, "are needed"),
    (["layers", 0, "mlp", "ff"], 0, "ff must be positive"),
])
def test_folders_that_cannot_be_served_say_why(tmp_path, path, value, says):
    c = changed(path, value)
    (tmp_path / "config.json").write_text(json.dumps(c))
    F.write_safetensors(str(tmp_path / "model.safetensors"), F.random_weights(BASE, 1))
    with pytest.raises(RuntimeError, match=says):
        load_package().serve.Model(str(tmp_path))


def test_a_folder_without_weights_or_with_broken_json(tmp_path):
    s = load_package().serve
    (tmp_path / "config.json").write_text(json.dumps(BASE))
    with pytest.raises(RuntimeError, match="cannot open"):
        s.Model(str(tmp_path))
    (tmp_path / "model.safetensors").write_bytes(b"\xff" * 40)
    with pytest.raises(RuntimeError, match="truncated"):
        s.Model(str(tmp_path))


def test_plain_decoder_is_causal_and_mixes_values():
    w = F.random_weights(BASE, 2)
    t = [int(v) for v in np.random.default_rng(0).integers(0, 20, 30)]
    z = F.forward(BASE, w, t)
    # a prefix gives the prefix of the logits
    assert np.allclose(F.forward(BASE, w, t[:11]), z[:11], atol=1e-10)
    # the first mixing layer's factor is unused, the second one's is not
    a, b = dict(w), dict(w)
    a["l0.mix.vmix"], b["l1.mix.vmix"] = np.float32(0.9), np.float32(0.9)
    assert np.array_equal(F.forward(BASE, a, t), z) and not np.allclose(F.forward(BASE, b, t), z)


TAZUNEX = dict(architecture="Tazunex", width=48, vocab=20, norm=dict(eps=1e-5), logit_softcap=9.0, layers=[
    dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=8, vdim=8, scale=0.3, mask=dict(size=7), rot=dict(base=100.0, dims=4)), mlp=dict(kind="dense", ff=24)),
    dict(type="latent_attention", mixer=dict(heads=3, dim=8, rot_dim=4, vdim=6, q_rank=10, kv_rank=12, scale=0.3, mask=dict(size=5), rot=dict(base=100.0, dims=4)),
         mlp=dict(kind="dense", ff=24)),
    dict(type="mlstm", mixer=dict(heads=2, dim=4, vdim=8, gate_cap=6.0), mlp=None),
    dict(type="mlstm", mixer=dict(heads=2, dim=4, vdim=8, gate_cap=6.0), mlp=None, weights_of=2)])


@pytest.mark.parametrize("path,value,says", [
    (["layers", 0, "type"], "scan", "no mixer of type 'scan'"),
    (["layers", 0, "mlp", "kind"], "moe", "no feed-forward of kind 'moe'"),
    (["layers", 0, "mixer", "heads"], 3, "multiple of kv_heads"),
    (["layers", 0, "mixer", "vdim"], 6, "must have their size"),
    (["layers", 0, "mixer", "mask"], None, "mask.size must be positive"),
    (["layers", 0, "mixer", "rot", "dims"], 5, "rot.dims must be even"),
    (["layers", 1, "mixer", "rot", "dims"], 2, "rot.dims must be rot_dim"),
    (["layers", 1, "mixer", "kv_rank"], 0, "kv_rank must be positive"),
    (["layers", 1, "mixer", "scale"], None, "scale is needed"),
    (["layers", 2, "mixer", "gate_cap"], 0, "gate_cap must be positive"),
    (["layers", 3, "weights_of"], 3, "must lead to a layer with tensors"),
    (["layers", 3, "weights_of"], 9, "must lead to a layer with tensors"),
    (["layers", 3, "weights_of"], 0, "differs from the layer whose tensors it uses"),
    (["layers", 3, "mixer", "dim"], 8, "differs from the layer whose tensors it uses"),
    (["logit_softcap"], None, "logit_softcap must be positive"),
])
def test_tazunex_folders_that_cannot_be_served_say_why(tmp_path, path, value, says):
    c = json.loads(json.dumps(TAZUNEX))
    at = c
    for p in path[:-1]:
        at = at[p]
    at[path[-1]] = value
    (tmp_path / "config.json").write_text(json.dumps(c))
    Z.write_safetensors(str(tmp_path / "model.safetensors"), Z.random_weights(TAZUNEX, 1))
    with pytest.raises(RuntimeError, match=says):
        load_package().serve.Model(str(tmp_path))


def test_plain_tazunex_is_causal_windowed_and_shares_tensors():
    w = Z.random_weights(TAZUNEX, 2)
    assert not [n for n in w if n.startswith("l3.")]
    t = [int(v) for v in np.random.default_rng(0).integers(0, 20, 30)]
    z = Z.forward(TAZUNEX, w, t)
    assert np.allclose(Z.forward(TAZUNEX, w, t[:11]), z[:11], atol=1e-9) and np.abs(z).max() < 9.0
    # attention alone sees as far as its windows reach, and no further
    c = dict(TAZUNEX, layers=TAZUNEX["layers"][:2])
    a, b = Z.forward(c, w, t), Z.forward(c, w, [(t[0] + 1) % 20] + t[1:])
    reach = 7 + 5 - 2
    assert not np.allclose(a[reach], b[reach]) and np.allclose(a[reach + 1:], b[reach + 1:], atol=1e-12)
    # a layer that shares tensors is a layer of its own
    own = dict(w, **{n.replace("l2.", "l3."): v for n, v in w.items() if n.startswith("l2.")})
    c = json.loads(json.dumps(TAZUNEX))
    del c["layers"][3]["weights_of"]
    assert np.array_equal(Z.forward(c, own, t), z)


def test_plain_tazunex_mechanisms_by_hand():
    assert np.allclose(Z.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 0.0), np.array([[3.0, 8.0]]) / np.sqrt(12.5))
    assert np.isclose(Z.gelu_tanh(1.0), 0.841192, atol=1e-6) and np.isclose(Z.soft_cap(1e9, 3.0), 3.0) and np.isclose(Z.log_sigmoid(0.0), -np.log(2.0))
    x = np.arange(6.0)[None, None]
    half, side = (Z.rotate(x, [1], 1.0, 4, inter)[0, 0] for inter in (False, True))
    c, s = np.cos(1.0), np.sin(1.0)
    assert np.allclose(half, [-2 * s, c - 3 * s, 2 * c, 3 * c + s, 4, 5]) and np.allclose(side, [-s, c, 2 * c - 3 * s, 3 * c + 2 * s, 4, 5])
    assert np.allclose(Z.rotate(x, [3], 16.0, 4, False)[0, 0][[1, 3]], [np.cos(0.75) - 3 * np.sin(0.75), 3 * np.cos(0.75) + np.sin(0.75)])
    assert Z.visible(4, 2).astype(int).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    q, k, v = np.ones((2, 1, 1)), np.array([[[0.0]], [[np.log(3.0)]]]), np.array([[[8.0]], [[0.0]]])
    assert np.allclose(Z.softmax_attention(q, k, v, 1.0, Z.visible(2, 2), [np.log(4.0)])[:, 0, 0], [8 / 5, 8 / 8])
    # one key, an open input gate, then a forget gate of one half: the running maximum starts at zero, not below
    st = (np.zeros((1, 1)), np.zeros(1), 0.0)
    st, o = Z.mlstm_step(st, np.array([2.0]), np.array([3.0]), np.array([5.0]), 1.0, -1.0)
    assert np.allclose([st[0][0, 0], st[1][0], st[2]], [15, 3, 1]) and np.allclose(o, 30 / (6 + 1e-6))
    st, o = Z.mlstm_step(st, np.array([0.1]), np.array([1.0]), np.array([1.0]), -9.0, np.log(0.5))
    m = 1 + np.log(0.5)
    assert np.isclose(st[2], m) and np.isclose(st[1][0], 3 + np.exp(-9 - m)) and np.allclose(o, 0.1 * st[0][0, 0] / (max(0.1 * st[1][0], np.exp(-m)) + 1e-6))


def test_plain_mechanisms_by_hand():
    assert np.allclose(F.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 1.0]), np.array([0.5, -0.5]), 3.0), [[0.5 - 1.0, -0.5 + 0.5]])
    assert np.allclose(F.unit_rms(np.array([[3.0, 4.0]]), 0.0), np.array([[3.0, 4.0]]) / np.sqrt(12.5))
    idx, wt = F.route(np.array([[0.0, np.log(3.0), -5.0]]), 2)
    assert idx.tolist() == [[1, 0]] and np.allclose(wt, [[0.75, 0.25]])
    q = np.array([[[1.0]], [[1.0]]])
    k = np.array([[[0.0]], [[np.log(3.0)]]])
    v = np.array([[[8.0]], [[0.0]]])
    assert np.allclose(F.causal_attention(q, k, v, 1.0, 1)[:, 0, 0], [8.0, 2.0])
    assert F.squared_relu(np.array([-2.0, 3.0])).tolist() == [0.0, 9.0]
    assert np.allclose(F.mix_values(2.0, 4.0, 0.25), 2.5)


def test_command_line_programs_load():
    for name in ("trace_run", "generate"):
        loader = importlib.machinery.SourceFileLoader(name, os.path.join(ROOT, "bin", name))
        spec = importlib.util.spec_from_loader(name, loader)
        m = importlib.util.module_from_spec(spec)
        loader.exec_module(m)
        assert os.access(os.path.join(ROOT, "bin", name), os.X_OK) and callable(m.main)
