"""A plain, slow numpy statement of the Fakilorn decoder (no cache, no batching, whole sequences), one
function per mechanism, in float64 unless asked otherwise.  Test infrastructure only: the product path
(csrc/decoder, csrc/host) shares nothing with it.

config: the dict read from config.json.  weights: dict name -> numpy array (any float type).
"""
from __future__ import annotations

import json
import struct

import numpy as np


# ---- files -------------------------------------------------------------------------------------------
def bf16_round(a):
    """Nearest-even rounding of float values to bfloat16, returned as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    r = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return r.astype(np.uint32).view(np.float32)


def write_safetensors(path, tensors):
    """tensors: name -> float array holding bfloat16-exact values (stored as BF16)."""
    head, blobs, off = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a, dtype=np.float32)
        b = (np.ascontiguousarray(a).reshape(-1).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)


def read_safetensors(path):
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(data[lo:hi], np.uint16).astype(np.uint32) << 16).view(np.float32)
        elif t["dtype"] == "F32":
            a = np.frombuffer(data[lo:hi], np.float32)
        else:
            a = np.frombuffer(data[lo:hi], np.int32)
        out[name] = a.reshape(t["shape"])
    return out


# ---- mechanisms --------------------------------------------------------------------------------------
def layer_norm(x, w, b, eps):
    mu = x.mean(axis=-1, keepdims=True)
    d = x - mu
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w + b


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def causal_attention(q, k, v, scale, group):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads kv head h // group."""
    T, H, _ = q.shape
    out = np.empty((T, H, v.shape[2]), q.dtype)
    hidden = np.triu(np.ones((T, T), bool), 1)
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s[hidden] = -np.inf
        s -= s.max(axis=1, keepdims=True)
        p = np.exp(s)
        p /= p.sum(axis=1, keepdims=True)
        out[:, h] = p @ v[:, h // group]
    return out


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention_mixer(h, w, m, eps, v_first):
    """h [T, width]; w: tensors of the mixer; m: its config; v_first: values of the first mixing layer, or None when
    this layer is that one or does not mix.  Returns (output, the layer's own unmixed values)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w["q"].T).reshape(T, H, d), eps)
    k = unit_rms((h @ w["k"].T).reshape(T, G, d), eps)
    own = (h @ w["v"].T).reshape(T, G, dv)
    v = own if v_first is None else mix_values(own, v_first.reshape(own.shape), float(w["vmix"]))
    o = causal_attention(q, k, v, m["scale"], H // G).reshape(T, H * dv)
    o = o * sigmoid(h @ w["g"].T)
    return o @ w["o"].T, own


def dense_mlp(h, w):
    return squared_relu(h @ w["up"].T) @ w["down"].T


def gated_expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z, top):
    """Router logits [T, E] -> (chosen experts [T, top], weights [T, top])."""
    order = np.argsort(-z, axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(z, order, axis=1)
    e = np.exp(c - c.max(axis=1, keepdims=True))
    return order, e / e.sum(axis=1, keepdims=True)


def moe_mlp(h, w, m):
    """w: nested dict, 'router' [E, width], experts 'e<j>', 'shared' (with 'sg') where the config has one."""
    idx, wt = route(h @ w["router"].T, m["router"]["top"])
    out = np.zeros_like(h)
    for j in range(m["router"]["experts"]):
        rows, slot = np.nonzero(idx == j)
        if rows.size:
            out[rows] += wt[rows, slot][:, None] * gated_expert(h[rows], w[f"e{j}"])
    if m.get("shared"):
        out += sigmoid(h @ w["shared"]["sg"].T) * gated_expert(h, w["shared"])
    return out


# ---- the model ---------------------------------------------------------------------------------------
def _nest(weights, dtype):
    root = {}
    for name, a in weights.items():
        d = root
        *path, leaf = name.split(".")
        if leaf == "b" and path[-1].startswith("norm"):
            path, leaf = path[:-1], path[-1] + ".b"
        for p in path:
            d = d.setdefault(p, {})
        d[leaf] = np.asarray(a, dtype)
    return root


def forward(config, weights, tokens, dtype=np.float64, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out (a list) receives the residual stream after every layer."""
    w = _nest(weights, dtype)
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * dtype(config["embedding"]["scale"])
    v_first = None
    for i, L in enumerate(config["layers"]):
        t = w[f"l{i}"]
        mixes = bool(L["mixer"].get("v_mix"))
        y, own = attention_mixer(layer_norm(x, t["norm1"], t["norm1.b"], eps), t["mix"], L["mixer"], eps, v_first if mixes else None)
        if mixes and v_first is None:
            v_first = own
        x = x + y
        if L.get("mlp"):
            h = layer_norm(x, t["norm2"], t["norm2.b"], eps)
            x = x + (dense_mlp(h, t["mlp"]) if L["mlp"]["kind"] == "dense" else moe_mlp(h, t["mlp"], L["mlp"]))
        if layers_out is not None:
            layers_out.append(x.copy())
    f = w["final"]
    x = layer_norm(x, f["norm"], f["norm.b"], eps)
    return (x @ w["embed"].T) * dtype(config["logit_scale"])


# ---- random models for the tests ---------------------------------------------------------------------
def tensor_shapes(config):
    """name -> shape of every tensor a model of this config has."""
    W, out = config["width"], {"embed": (config["vocab"], config["width"])}

    def norm(name):
        out[name] = (W,)
        out[name + ".b"] = (W,)

    for i, L in enumerate(config["layers"]):
        m, p = L["mixer"], f"l{i}."
        norm(p + "norm1")
        out[p + "mix.q"] = (m["heads"] * m["dim"], W)
        out[p + "mix.k"] = (m["kv_heads"] * m["dim"], W)
        out[p + "mix.v"] = (m["kv_heads"] * m["vdim"], W)
        if m.get("v_mix"):
            out[p + "mix.vmix"] = ()
        out[p + "mix.g"] = (m["heads"] * m["vdim"], W)
        out[p + "mix.o"] = (W, m["heads"] * m["vdim"])
        f = L.get("mlp")
        if not f:
            continue
        norm(p + "norm2")
        if f["kind"] == "dense":
            out[p + "mlp.up"] = (f["ff"], W)
            out[p + "mlp.down"] = (W, f["ff"])
            continue
        out[p + "mlp.router"] = (f["router"]["experts"], W)
        groups = [(f"e{j}", f["expert"]["ff"]) for j in range(f["router"]["experts"])]
        if f.get("shared"):
            groups.append(("shared", f["shared"]["ff"]))
            out[p + "mlp.shared.sg"] = (1, W)
        for name, ff in groups:
            out[f"{p}mlp.{name}.gate"] = (ff, W)
            out[f"{p}mlp.{name}.up"] = (ff, W)
            out[f"{p}mlp.{name}.down"] = (W, ff)
    norm("final.norm")
    return out


def random_weights(config, seed, gain=1.0):
    """bfloat16-exact float32 tensors; linears N(0, gain / fan-in), norms near 1, mixing factors in (0, 1)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        a = rng.standard_normal(shape)
        if name == "embed":
            a = a / np.sqrt(shape[1])
        elif "norm" in name:
            a = 0.1 * a if name.endswith(".b") else 1.0 + 0.2 * a
        elif name.endswith("vmix"):
            a = rng.uniform(0.2, 0.8, shape)
        else:
            a = a * np.sqrt(gain / shape[1])
        out[name] = bf16_round(np.asarray(a, np.float32)).reshape(shape)
    return out
