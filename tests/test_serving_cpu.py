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


def test_decoder_library_exports_its_header():
    d = load_package().decoder_capi
    L = d.lib()
    header = open(os.path.join(ROOT, "include", "cccc_b200_decoder.h")).read()
    declared = set(re.findall(r"C_EXPORT\s+[\w\s\*]+?\b(cuda_b200_\w+)\s*\(", header))
    assert declared == set(d.SYMBOLS)
    for name in declared:
        assert getattr(L, name) is not None


def test_both_architectures_are_registered():
    import ctypes as C

    s = load_package().serve
    buf = C.create_string_buffer(256)
    s.library("Fakilorn").cccc_model_architectures(buf, 256)
    assert "Fakilorn" in buf.value.decode().split()
    s.library("cccc-llm").cccc_model_architectures(buf, 256)
    assert {"Fakilorn", "cccc-llm"} <= set(buf.value.decode().split())


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
