"""Serving a model folder (config.json + weights) from Python: builds and loads the library that holds the architecture,
and binds the C harness over the C++ registry, models, scheduler and generation loop (csrc/host/model_capi.cpp).  Standard
library only; everything that computes is in the library.
"""
from __future__ import annotations

import ctypes as C
import importlib.util
import json
import os
from array import array

HERE = os.path.dirname(os.path.abspath(__file__))
FLOAT32, BFLOAT16 = 0, 3
DTYPES = {"float32": FLOAT32, "bfloat16": BFLOAT16}
# architectures made of the decoder library's operations; the others need the quantized path's libraries as well
DECODER_ARCHITECTURES = ("Fakilorn", "Tazunex")

_vp, _i, _u, _f, _ip, _fp = C.c_void_p, C.c_int, C.c_uint, C.c_float, C.POINTER(C.c_int), C.POINTER(C.c_float)
SYMBOLS = {
    "cccc_model_architectures": (_i, [C.c_char_p, _i]),
    "cccc_model_open": (_vp, [C.c_char_p, _i, _i, _i, _i, _i, _i, C.c_char_p, _i]),
    "cccc_model_close": (None, [_vp]),
    "cccc_model_info": (C.c_ulonglong, [_vp, _i]),
    "cccc_model_open_slot": (_i, [_vp]),
    "cccc_model_close_slot": (None, [_vp, _i]),
    "cccc_model_slot_length": (_i, [_vp, _i]),
    "cccc_model_step": (_i, [_vp, _i, _ip, _ip, _ip, _ip, _ip, _fp, _ip]),
    "cccc_model_time_step": (_f, [_vp, _i, _i, _i, _i, _i]),
    "cccc_model_generate": (_i, [_vp, _ip, _i, _ip, _f, _i, _f, _f, _ip, _i, _u, _i, _i, _ip, _i, _ip]),
    "cccc_model_generate_many": (_i, [_vp, _i, _ip, _ip, _f, _i, _f, _f, _ip, _i, _ip, _i, _u, _i, _i, _ip, _ip]),
}
_libs: dict = {}


def _build_module():
    spec = importlib.util.spec_from_file_location("cccc_lite_b200_build", os.path.join(HERE, "build.py"))
    m = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(m)
    return m


def library(architecture: str) -> C.CDLL:
    """The library whose registry knows `architecture`, compiled first where it is missing or stale."""
    small = architecture in DECODER_ARCHITECTURES
    if small not in _libs:
        build = _build_module()
        path = build.build_decoder() if small else build.build()
        L = C.CDLL(path if small else build.HOST_LIB)
        for name, (res, args) in SYMBOLS.items():
            fn = getattr(L, name)      # the host library's own dependency provides them there
            fn.restype, fn.argtypes = res, args
        _libs[small] = L
    return _libs[small]


def _ints(values):
    values = list(values)
    return (C.c_int * max(1, len(values)))(*values)


def _sampler(sampler):
    s = dict(temperature=0.0, top_k=0, top_p=1.0, repetition_penalty=1.0, banned_ids=())
    s.update(sampler or {})
    return s["temperature"], s["top_k"], s["top_p"], s["repetition_penalty"], _ints(s["banned_ids"]), len(s["banned_ids"])


class Model:
    """A loaded model: cache slots, steps over ragged batches, generation."""

    def __init__(self, folder, dtype="bfloat16", device=0, max_context=4096, max_sequences=1, max_step_tokens=4096, noise_weights=False):
        with open(os.path.join(folder, "config.json")) as f:
            architecture = json.load(f).get("architecture", "")
        self.lib = library(architecture)
        err = C.create_string_buffer(1024)
        self.h = self.lib.cccc_model_open(os.fsencode(folder), device, DTYPES[dtype], max_context, max_sequences, max_step_tokens, int(noise_weights), err,
                                          1024)
        if not self.h:
            raise RuntimeError(err.value.decode())
        self.vocab = self.info(0)

    def info(self, what):
        return int(self.lib.cccc_model_info(self.h, what))

    def open_slot(self):
        slot = self.lib.cccc_model_open_slot(self.h)
        if slot < 0:
            raise RuntimeError("no free cache slot")
        return slot

    def close_slot(self, slot):
        self.lib.cccc_model_close_slot(self.h, slot)

    def slot_length(self, slot):
        return self.lib.cccc_model_slot_length(self.h, slot)

    def step(self, entries, logits=True, choice=False):
        """entries: (slot, tokens, want) triples.  Returns (logits, choices): a float array of wanted * vocab values and the
        ids of the largest logits, in the order of the entries and of their wanted places (None where not asked for)."""
        wanted = sum(len(w) for _, _, w in entries)
        lg = array("f", bytes(4 * wanted * self.vocab)) if logits else None
        ch = (C.c_int * max(1, wanted))() if choice else None
        lp = (C.c_float * len(lg)).from_buffer(lg) if logits and wanted else None
        rc = self.lib.cccc_model_step(self.h, len(entries), _ints(s for s, _, _ in entries), _ints(len(t) for _, t, _ in entries),
                                      _ints(x for _, t, _ in entries for x in t), _ints(len(w) for _, _, w in entries),
                                      _ints(x for _, _, w in entries for x in w), lp, ch)
        if rc != 0:
            raise RuntimeError("the step's entries cannot run" if rc == -1 else "a step failed")
        return lg, (list(ch[:wanted]) if choice else None)

    def time_step(self, entries, tokens, context, inner=10, repeat=5):
        """Device milliseconds of one step (see LanguageModel::timeStep)."""
        return self.lib.cccc_model_time_step(self.h, entries, tokens, context, inner, repeat)

    def generate(self, prompt, max_new, seed=0, sampler=None, eos_ids=(), portion=2048, T=0, T_kv=0, sys_n=0, turn_n=0):
        """One sequence through the generation loop (csrc/host/generate.h).  Returns (ids, stats)."""
        rows = self.info(1)
        gen = _ints([len(eos_ids), *eos_ids, -1, -1, sys_n, turn_n, T or rows, T_kv or rows])
        out, stats = (C.c_int * max(1, max_new))(), (C.c_int * 3)()
        n = self.lib.cccc_model_generate(self.h, _ints(prompt), len(prompt), gen, *_sampler(sampler), seed, max_new, portion, out, max_new, stats)
        if n < 0:
            raise RuntimeError("a step failed")
        return list(out[:n]), dict(rebuilds=stats[0], decode_steps=stats[1], prefill_tokens=stats[2])

    def generate_many(self, prompts, max_new, seed=0, sampler=None, eos_ids=(), step_tokens=2048):
        """Many prompts through the scheduler.  Returns (a list of ids per prompt, None for a rejected one; steps taken)."""
        n = len(prompts)
        out, n_out = (C.c_int * max(1, n * max_new))(), (C.c_int * max(1, n))()
        steps = self.lib.cccc_model_generate_many(self.h, n, _ints(len(p) for p in prompts), _ints(x for p in prompts for x in p), *_sampler(sampler),
                                                  _ints(eos_ids), len(eos_ids), seed, max_new, step_tokens, out, n_out)
        if steps < 0:
            raise RuntimeError("a step failed")
        return [list(out[i * max_new:i * max_new + n_out[i]]) if n_out[i] >= 0 else None for i in range(n)], steps

    def close(self):
        if self.h:
            self.lib.cccc_model_close(self.h)
            self.h = None
