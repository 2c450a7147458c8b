"""Binding of the decoder language models (include/voxtral_b200_lm.h).

    lm = LanguageModel("model_folder")            # config.json + model.safetensors
    seq = lm.open()
    logits = lm.step(seq, tokens, want=[-1])
    tokens = lm.generate(seq, prompt, 64)

The design is picked by config.json's "architecture". The symbols live in libvoxtral_b200.so and, for
programs that need nothing of the speech path, in libvb200_lm.so; either serves. There is no CPU
fallback: a missing library or a missing sm_100 GPU raises.
"""
import ctypes as C
import json
import os

import numpy as np

HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATHS = [os.path.join(HERE, "lib", n) for n in ("libvoxtral_b200.so", "libvb200_lm.so")]
DTYPES = {"bfloat16": 0, "float32": 1}


class Options(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("dtype", "max_seqs", "max_tokens", "block_rows")]


class Info(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("vocab", "width", "layers", "runs", "max_seqs", "max_tokens", "block_rows", "dtype")] + \
               [(n, C.c_size_t) for n in ("weight_bytes", "state_bytes_per_seq")]


_libs = {}


def lm_lib(path=None):
    """The shared library with the language-model entry points."""
    if path is None:
        path = next((p for p in LIB_PATHS if os.path.exists(p)), None)
        if path is None:
            raise RuntimeError(f"{LIB_PATHS[0]} is missing: run `python voxtral-tts.c_b200/build.py` (there is no CPU fallback)")
    if path in _libs:
        return _libs[path]
    L = C.CDLL(path)
    fp, vp = C.POINTER(C.c_float), C.c_void_p
    for name, res, args in (
            ("vb200_lm_open", vp, [C.c_char_p, C.POINTER(Options)]),
            ("vb200_lm_open_random", vp, [C.c_char_p, C.POINTER(Options), C.c_uint]),
            ("vb200_lm_check_config", C.c_int, [C.c_char_p]),
            ("vb200_lm_close", None, [vp]),
            ("vb200_lm_info", C.c_int, [vp, C.POINTER(Info)]),
            ("vb200_lm_error", C.c_char_p, []),
            ("vb200_lm_seq_open", C.c_int, [vp]),
            ("vb200_lm_seq_close", C.c_int, [vp, C.c_int]),
            ("vb200_lm_seq_length", C.c_int, [vp, C.c_int]),
            ("vb200_lm_step", C.c_int, [vp, C.c_int, vp, C.c_int, vp, C.c_int, vp]),
            ("vb200_lm_generate", C.c_int, [vp, C.c_int, vp, C.c_int, C.c_int, vp]),
            ("vb200_lm_last_ms", C.c_int, [vp, fp, fp]),
            ("vb200_lm_tap_enable", C.c_int, [vp, C.c_int]),
            ("vb200_lm_tap_read", C.c_int, [vp, vp, C.c_int])):
        fn = getattr(L, name)
        fn.restype, fn.argtypes = res, args
    _libs[path] = L
    return L


def check_config(config, lib_path=None):
    """Raises ValueError when the library cannot run this configuration (a dict or JSON text). Needs no GPU."""
    L = lm_lib(lib_path)
    text = config if isinstance(config, str) else json.dumps(config)
    if L.vb200_lm_check_config(text.encode()) != 0:
        raise ValueError(L.vb200_lm_error().decode())


def _ints(a):
    return np.ascontiguousarray(a, dtype=np.int32).reshape(-1)


def _ptr(a):
    return a.ctypes.data_as(C.c_void_p)


class LanguageModel:
    """A loaded decoder language model: slots for sequences, portions of tokens in, logits out."""

    def __init__(self, folder=None, dtype="bfloat16", max_seqs=1, max_tokens=0, block_rows=0, config=None, seed=0, lib_path=None):
        """folder: config.json + model.safetensors; or config (a dict) with hashed random weights."""
        self.L = lm_lib(lib_path)
        self.h = None
        opt = Options(DTYPES[dtype], max_seqs, max_tokens, block_rows)
        if folder is not None:
            self.h = self.L.vb200_lm_open(os.fsencode(folder), C.byref(opt))
        else:
            self.h = self.L.vb200_lm_open_random(json.dumps(config).encode(), C.byref(opt), seed)
        if not self.h:
            raise RuntimeError(self.L.vb200_lm_error().decode())
        self.info = Info()
        self.L.vb200_lm_info(self.h, C.byref(self.info))

    def _ok(self, rc):
        if rc < 0:
            raise RuntimeError(self.L.vb200_lm_error().decode())
        return rc

    def open(self):
        return self._ok(self.L.vb200_lm_seq_open(self.h))

    def release(self, seq):
        self._ok(self.L.vb200_lm_seq_close(self.h, seq))

    def length(self, seq):
        return self._ok(self.L.vb200_lm_seq_length(self.h, seq))

    def step(self, seq, tokens, want=()):
        """Feeds the next tokens; returns the logits [len(want), vocab] at the wanted places."""
        t, w = _ints(tokens), _ints([x + len(tokens) if x < 0 else x for x in want])
        out = np.empty((w.size, self.info.vocab), dtype=np.float32)
        self._ok(self.L.vb200_lm_step(self.h, seq, _ptr(t), t.size, _ptr(w) if w.size else None, w.size, _ptr(out) if w.size else None))
        return out

    def generate(self, seq, prompt, n_new):
        """Greedy continuation of a sequence by n_new tokens, the choice made on the device."""
        p, out = _ints(prompt), np.empty(n_new, dtype=np.int32)
        self._ok(self.L.vb200_lm_generate(self.h, seq, _ptr(p), p.size, n_new, _ptr(out)))
        return out.tolist()

    def last_ms(self):
        """(prompt, decoding) device milliseconds of the last generate call."""
        a, b = C.c_float(0), C.c_float(0)
        self._ok(self.L.vb200_lm_last_ms(self.h, C.byref(a), C.byref(b)))
        return a.value, b.value

    def tap(self, on=True):
        self._ok(self.L.vb200_lm_tap_enable(self.h, 1 if on else 0))

    def tap_read(self, n):
        """Residual stream after every layer run of the last step of n tokens: [runs, n, width]."""
        out = np.empty((self.info.runs, n, self.info.width), dtype=np.float32)
        self._ok(self.L.vb200_lm_tap_read(self.h, _ptr(out), n))
        return out

    def close(self):
        if self.h:
            self.L.vb200_lm_close(self.h)
            self.h = None

    def __enter__(self):
        return self

    def __exit__(self, *_):
        self.close()
