"""ctypes binding of include/cccc_b200_decoder.h (libcccc-b200-decoder.so).  Tensors are torch tensors that only hold device
memory, or raw pointers."""
from __future__ import annotations

import ctypes as C
import os

HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(HERE, "libcccc-b200-decoder.so")

FLOAT, BF16 = 0, 3
ACT_NONE, ACT_RELU2, ACT_SILU_GATE, ACT_GELU_GATE, ACT_SOFTCAP = 0, 1, 2, 3, 4
NORM_RMS, NORM_LAYER = 0, 1

_vp, _i, _u, _f = C.c_void_p, C.c_int, C.c_uint, C.c_float


def _struct(name, pointers, uints, ints=(), floats=()):
    return type(name, (C.Structure,), {"_fields_": [(n, _vp) for n in pointers] + [(n, _u) for n in uints] + [(n, _i) for n in ints] + [(n, _f) for n in floats]})


Norm = _struct("Norm", ("X", "weight", "bias", "out", "Y", "slot_row", "slot_weight", "rows", "branch", "branch_weight"), ("n", "width", "ldx", "ldo", "ldy", "slots", "ldb"), ("kind",), ("eps",))
Linear = _struct("Linear", ("W", "X", "Y", "row_scale", "group_offset", "x_row", "active", "head_gate", "Y_tail"),
                 ("rows", "N", "K", "ldw", "ldx", "ldy", "groups", "group_rows", "group_max", "up_row", "active_cap", "blocks", "x_step", "y_step",
                  "ld_gate", "tail", "ld_tail"), ("out_type", "activation", "accumulate"), ("alpha", "cap"))
Batch = _struct("Batch", ("slot", "pos", "start", "n", "token_entry", "floor"), ("entries", "tokens", "max_n", "max_len", "first_entry", "first_token"))
Attention = _struct("Attention", ("qkvg", "out", "k_cache", "v_cache", "v_first", "work", "q_norm", "k_norm", "rotary", "sink", "head_gate"),
                    ("ld", "ldo", "k_off", "v_off", "g_off", "v_first_ld", "H", "Hkv", "dim", "vdim", "k_ld", "v_ld", "T_max", "slots", "q_ld", "rot_dims", "ld_gate",
                     "window"), ("v_mix", "qk_norm", "gate", "rot_interleaved", "no_append"), ("mix", "eps", "scale"))
Latent = _struct("Latent", ("down", "cq", "cache", "q_norm", "kv_norm", "rotary"), ("ld", "ld_cq", "kv_off", "q_rank", "kv_rank", "rot_dim", "c_ld", "T_max"), (),
                 ("eps",))
Expand = _struct("Expand", ("cache", "c", "K", "floor", "pos2"), ("c_ld", "T_max", "kv_rank", "rot_dim", "ld_c", "k_ld", "T", "dim", "heads", "max_rows"))
Mlstm = _struct("Mlstm", ("qkvg", "gates", "bias", "norm", "out", "state", "work"), ("ld", "ld_gates", "ldo", "k_off", "v_off", "g_off", "f_off", "heads", "dim", "vdim"),
                (), ("cap", "eps", "q_scale"))
Route = _struct("Route", ("logits", "pair_row", "pair_weight", "row_token", "group_offset", "active", "shared_weight", "choice", "counters"),
                ("n", "ldl", "experts", "top", "active_cap"), ("sg_col",))

SYMBOLS = {
    "cuda_b200_embed_f32": (_i, [_i, _vp, _vp, _u, _vp, _u, _u, _u, _u, _f, _vp, _u]),
    "cuda_b200_norm_rows": (_i, [_i, C.POINTER(Norm), _vp, _u]),
    "cuda_b200_linear_rows": (_i, [_i, _u, C.POINTER(Linear), _vp, _u, _i]),
    "cuda_b200_attention_work_bytes": (C.c_ulonglong, [_u]),
    "cuda_b200_attention_rows": (_i, [_i, C.POINTER(Attention), C.POINTER(Batch), _vp, _u, _i]),
    "cuda_b200_rotary_table": (_i, [_vp, _u, _u, C.c_double, _vp]),
    "cuda_b200_latent_down": (_i, [_i, C.POINTER(Latent), C.POINTER(Batch), _vp, _u]),
    "cuda_b200_latent_query": (_i, [_i, _vp, _u, _u, _u, _vp, _u, _u, _u, _u, _u, _vp, _u, C.POINTER(Batch), _vp, _u]),
    "cuda_b200_latent_expand": (_i, [_i, C.POINTER(Expand), C.POINTER(Batch), _vp, _u]),
    "cuda_b200_mlstm_state_floats": (C.c_ulonglong, [_u, _u]),
    "cuda_b200_mlstm_work_floats": (C.c_ulonglong, [_u, _u, _u, _u, _u]),
    "cuda_b200_mlstm_rows": (_i, [_i, C.POINTER(Mlstm), C.POINTER(Batch), _vp, _u, _i]),
    "cuda_b200_route_rows": (_i, [C.POINTER(Route), _vp, _u]),
    "cuda_b200_gather_rows": (_i, [_i, _vp, _u, _vp, _vp, _u, _u, _u, _vp, _u]),
    "cuda_b200_argmax_f32": (_i, [_vp, _u, _u, _u, _vp, _vp, _vp, _u]),
    "cuda_b200_decoder_check": (_i, [C.c_char_p]),
    "cuda_b200_decoder_launches": (C.c_ulonglong, []),
}
_lib = None


def lib() -> C.CDLL:
    """The loaded library; compiled first where it is missing (it is the only implementation)."""
    global _lib
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            import importlib.util

            spec = importlib.util.spec_from_file_location("cccc_lite_b200_build", os.path.join(HERE, "build.py"))
            m = importlib.util.module_from_spec(spec)
            spec.loader.exec_module(m)
            m.build_decoder()
        L = C.CDLL(LIB_PATH)
        for name, (res, args) in SYMBOLS.items():
            fn = getattr(L, name)
            fn.restype, fn.argtypes = res, args
        _lib = L
    return _lib


def _ptr(t):
    return None if t is None else (t if isinstance(t, int) else t.data_ptr())


def _stream():
    import torch

    return torch.cuda.current_stream().cuda_stream


def fill(cls, **kw):
    """A descriptor from keyword arguments (tensors become pointers; keep them alive)."""
    a = cls()
    pointers = {n for n, t in cls._fields_ if t is _vp}
    for k, v in kw.items():
        setattr(a, k, _ptr(v) if k in pointers else v)
    return a


def embed(dtype, ids, table, ld_table, X, ldx, n, width, vocab, scale, flags=0):
    return lib().cuda_b200_embed_f32(dtype, _ptr(ids), _ptr(table), ld_table, _ptr(X), ldx, n, width, vocab, scale, _stream(), flags)


def norm(dtype, desc, flags=0):
    return lib().cuda_b200_norm_rows(dtype, C.byref(desc), _stream(), flags)


def linear(dtype, descs, flags=0, kernel=0):
    return lib().cuda_b200_linear_rows(dtype, len(descs), (Linear * len(descs))(*descs), _stream(), flags, kernel)


def attention(dtype, desc, batch, flags=0, kernel=0):
    return lib().cuda_b200_attention_rows(dtype, C.byref(desc), C.byref(batch), _stream(), flags, kernel)


def attention_work_bytes(vdim):
    return int(lib().cuda_b200_attention_work_bytes(vdim))


def rotary_table(table, rows, dims, base):
    return lib().cuda_b200_rotary_table(_ptr(table), rows, dims, base, _stream())


def latent_down(dtype, desc, batch, flags=0):
    return lib().cuda_b200_latent_down(dtype, C.byref(desc), C.byref(batch), _stream(), flags)


def latent_query(dtype, src, ld_src, src_step, src_off, dst, ld_dst, dst_step, dst_off, heads, rot_dim, rotary, T_max, batch, flags=0):
    return lib().cuda_b200_latent_query(dtype, _ptr(src), ld_src, src_step, src_off, _ptr(dst), ld_dst, dst_step, dst_off, heads, rot_dim, _ptr(rotary), T_max,
                                        C.byref(batch), _stream(), flags)


def latent_expand(dtype, desc, batch, flags=0):
    return lib().cuda_b200_latent_expand(dtype, C.byref(desc), C.byref(batch), _stream(), flags)


def mlstm_state_floats(dim, vdim):
    return int(lib().cuda_b200_mlstm_state_floats(dim, vdim))


def mlstm_work_floats(tokens, entries, heads, dim, vdim):
    return int(lib().cuda_b200_mlstm_work_floats(tokens, entries, heads, dim, vdim))


def mlstm(dtype, desc, batch, flags=0, kernel=0):
    return lib().cuda_b200_mlstm_rows(dtype, C.byref(desc), C.byref(batch), _stream(), flags, kernel)


def route(desc, flags=0):
    return lib().cuda_b200_route_rows(C.byref(desc), _stream(), flags)


def gather(dtype, X, ldx, row_token, out, ldo, n, width, flags=0):
    return lib().cuda_b200_gather_rows(dtype, _ptr(X), ldx, _ptr(row_token), _ptr(out), ldo, n, width, _stream(), flags)


def argmax(logits, rows, cols, ld, idx, val, flags=0):
    return lib().cuda_b200_argmax_f32(_ptr(logits), rows, cols, ld, _ptr(idx), _ptr(val), _stream(), flags)


def check(label="decoder"):
    return lib().cuda_b200_decoder_check(label.encode())


def launches():
    return int(lib().cuda_b200_decoder_launches())
