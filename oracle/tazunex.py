"""A plain, slow numpy statement of the Tazunex decoder (no cache, no batching, whole sequences, the recurrence one
token after the other), one function per mechanism, in float64 unless asked otherwise.  Test infrastructure only: the
product path (csrc/decoder, csrc/host) shares nothing with it.

config: the dict read from config.json.  weights: dict name -> numpy array (any float type).
"""
from __future__ import annotations

import numpy as np

from oracle.fakilorn import bf16_round, write_safetensors  # noqa: F401  (files are written the same way)


# ---- mechanisms --------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def rotate(x, pos, base, dims, interleaved):
    """x [T, heads, d]: turns the first `dims` of d by pos * base^(-2i/dims), pair by pair."""
    i = np.arange(dims // 2)
    a = np.asarray(pos, np.float64)[:, None] * np.float64(base) ** (-2.0 * i / dims)
    c, s = np.cos(a)[:, None, :].astype(x.dtype), np.sin(a)[:, None, :].astype(x.dtype)
    first, second = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
    out = x.copy()
    out[..., first] = x[..., first] * c - x[..., second] * s
    out[..., second] = x[..., second] * c + x[..., first] * s
    return out


def visible(T, window):
    """[T, T]: may position i read position j."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < window)


def softmax_attention(q, k, v, scale, mask, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; head h reads k/v head h // (H / G).  sink [H]: a learned
    score that takes part in the denominator only."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        s = np.where(mask, (q[:, h] @ k[:, h // group].T) * scale, -np.inf)
        m = s.max(axis=1, keepdims=True)
        if sink is not None:
            m = np.maximum(m, sink[h])
        p = np.exp(s - m)
        z = p.sum(axis=1, keepdims=True)
        if sink is not None:
            z = z + np.exp(sink[h] - m)
        out[:, h] = (p / z) @ v[:, h // group]
    return out


def attention_mixer(h, w, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    raw = h @ w["k"].T
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, d)
    k = rms_norm(raw, w["k.norm"], eps).reshape(T, G, d)
    r = m["rot"]
    q, k = (rotate(a, np.arange(T), r["base"], r["dims"], False) for a in (q, k))
    o = softmax_attention(q, k, raw.reshape(T, G, d), m["scale"], visible(T, m["mask"]["size"]), w["sink"])
    return o.reshape(T, -1) @ w["o"].T


def latent_attention_mixer(h, w, m, eps):
    T, H, d, rd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(T, H, d + rd)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :R], w["dkv.norm"], eps)
    turn = lambda a: rotate(a, np.arange(T), m["rot"]["base"], rd, True)
    k_rot = turn(down[:, None, R:])
    k = np.concatenate([(c @ w["uk"].T).reshape(T, H, d), np.repeat(k_rot, H, axis=1)], axis=2)
    v = (c @ w["uv"].T).reshape(T, H, m["vdim"])
    q = np.concatenate([q[..., :d], turn(q[..., d:])], axis=2)
    o = softmax_attention(q, k, v, m["scale"], visible(T, m["mask"]["size"]))
    o = o * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, -1) @ w["o"].T


def mlstm_step(state, q, k, v, log_i, log_f):
    """One token of one head.  state: (S [d, dv], n [d], m).  Returns the new state and the output [dv]."""
    S, n, m = state
    m1 = max(log_f + m, log_i)
    keep, add = np.exp(log_f + m - m1), np.exp(log_i - m1)
    S = keep * S + add * np.outer(k, v)
    n = keep * n + add * k
    return (S, n, m1), (S.T @ q) / (max(abs(n @ q), np.exp(-m1)) + 1e-6)


def mlstm_recurrence(q, k, v, log_i, log_f):
    """q, k [T, H, d], v [T, H, dv], log gates [T, H] -> [T, H, dv]."""
    T, H, d = q.shape
    dt = q.dtype.type
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        st = (np.zeros((d, v.shape[2]), q.dtype), np.zeros(d, q.dtype), dt(0))
        for t in range(T):
            st, out[t, h] = mlstm_step(st, q[t, h], k[t, h], v[t, h], log_i[t, h], log_f[t, h])
    return out


def mlstm_gates(h, w, cap):
    log_i = soft_cap(h @ w["i"].T + w["i.b"], cap)
    log_f = log_sigmoid(soft_cap(h @ w["f"].T + w["f.b"], cap))
    return log_i, log_f


def mlstm_mixer(h, w, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, d) * h.dtype.type(d ** -0.5)
    k = (h @ w["k"].T).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, dv)
    log_i, log_f = mlstm_gates(h, w, m["gate_cap"])
    o = rms_norm(mlstm_recurrence(q, k, v, log_i, log_f), 1.0, eps).reshape(T, H * dv)
    return (o * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def gated_mlp(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer, "mlstm": mlstm_mixer}


# ---- the model ---------------------------------------------------------------------------------------
def owner(config, i):
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def part(weights, prefix, dtype):
    return {n[len(prefix):]: np.asarray(a, dtype) for n, a in weights.items() if n.startswith(prefix)}


def forward(config, weights, tokens, dtype=np.float64, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out (a list) receives the residual stream after every layer."""
    eps = dtype(config["norm"]["eps"])
    table = np.asarray(weights["embed"], dtype)
    x = table[np.asarray(tokens)]
    for i, L in enumerate(config["layers"]):
        p = f"l{owner(config, i)}."
        norm = lambda a, name: rms_norm(a, np.asarray(weights[p + name], dtype), eps)
        x = x + norm(MIXERS[L["type"]](norm(x, "norm1"), part(weights, p + "mix.", dtype), L["mixer"], eps), "norm1b")
        if L.get("mlp"):
            x = x + norm(gated_mlp(norm(x, "norm2"), part(weights, p + "mlp.", dtype)), "norm2b")
        if layers_out is not None:
            layers_out.append(x.copy())
    x = rms_norm(x, np.asarray(weights["final.norm"], dtype), eps)
    return soft_cap(x @ table.T, dtype(config["logit_softcap"]))


# ---- random models for the tests ---------------------------------------------------------------------
def mixer_shapes(kind, m, W):
    if kind == "attention":
        q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        return {"q": (q, W), "k": (k, W), "q.norm": (q,), "k.norm": (k,), "sink": (m["heads"],), "o": (W, m["heads"] * m["vdim"])}
    if kind == "latent_attention":
        H, R = m["heads"], m["kv_rank"]
        return {"dq": (m["q_rank"], W), "dq.norm": (m["q_rank"],), "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]), "dkv": (R + m["rot_dim"], W),
                "dkv.norm": (R,), "uk": (H * m["dim"], R), "uv": (H * m["vdim"], R), "g": (H, W), "o": (W, H * m["vdim"])}
    H, qk, v = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
    return {"q": (qk, W), "k": (qk, W), "v": (v, W), "g": (v, W), "o": (W, v), "norm": (v,), "i": (H, W), "i.b": (H,), "f": (H, W), "f.b": (H,)}


def tensor_shapes(config):
    """name -> shape of every tensor a model of this config has."""
    W = config["width"]
    out = {"embed": (config["vocab"], W), "final.norm": (W,)}
    for i, L in enumerate(config["layers"]):
        if owner(config, i) != i:
            continue
        p, f = f"l{i}.", L.get("mlp")
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        out.update({p + "mix." + n: s for n, s in mixer_shapes(L["type"], L["mixer"], W).items()})
        if f:
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.gate": (f["ff"], W), p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
    return out


def random_weights(config, seed):
    """bfloat16-exact float32 tensors: linears N(0, 1 / fan-in), norms near 1, forget gates that mostly keep.

    An mLSTM's output is divided by its own size, so where its scores q . k cancel, rounding decides its direction.  To keep
    these models well conditioned, tokens share a direction, the mLSTM's keys resemble its queries and branches are small."""
    rng = np.random.default_rng(seed)
    out = {}
    shared = 1.5 * rng.standard_normal(config["width"])
    for name, shape in tensor_shapes(config).items():
        a = rng.standard_normal(shape)
        if name.endswith(".f.b"):
            a = 3.0 + 2.0 * a
        elif "norm" in name.rsplit(".", 1)[-1]:
            a = 1.0 + 0.2 * a
            if name.endswith(("norm1b", "norm2b")):
                a = 0.3 * a
        elif name == "embed":
            a = 0.17 * (a + shared)
        elif len(shape) == 2:
            a = a / np.sqrt(shape[1]) * (3.0 if name.endswith((".mix.i", ".mix.f")) else 1.0)
        if name.endswith(".mix.k") and name[:-1] + "f" in tensor_shapes(config):
            a = 0.9 * out[name[:-1] + "q"] + 0.44 * a
        out[name] = bf16_round(np.asarray(a, np.float32)).reshape(shape)
    return out
