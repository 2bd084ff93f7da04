"""Decoder models described by a folder with config.json and model.safetensors (include/gptb200.h: gptb200_decoder_*).

A ctypes view like the rest of the package: weights, sequence states, steps, sampling and generation are in the library.
"""
from __future__ import annotations

import ctypes
import os

import numpy as np

from . import GptB200Error, build

DTYPES = {"bfloat16": 0, "float32": 1}

_lib = None


def load_library() -> ctypes.CDLL:
    """The library with the decoder models (built on demand when nothing current is there; there is no fallback)."""
    global _lib
    if _lib is not None:
        return _lib
    lib = ctypes.CDLL(build.decoder_library())
    vp, i, ip = ctypes.c_void_p, ctypes.c_int, ctypes.POINTER(ctypes.c_int)
    dp, sz, f32, ull, ll = ctypes.POINTER(ctypes.c_double), ctypes.c_size_t, ctypes.c_float, ctypes.c_ulonglong, ctypes.c_longlong
    sig = {
        "gptb200_decoder_check_config": (i, [ctypes.c_char_p, ctypes.c_char_p, sz]),
        "gptb200_decoder_load": (i, [ctypes.POINTER(vp), ctypes.c_char_p, i, i, vp, ctypes.c_char_p, sz]),
        "gptb200_decoder_destroy": (i, [vp]),
        "gptb200_decoder_context": (vp, [vp]),
        "gptb200_decoder_vocab": (i, [vp]),
        "gptb200_decoder_open": (i, [vp, i, ip]),
        "gptb200_decoder_close": (i, [vp, i]),
        "gptb200_decoder_length": (i, [vp, i]),
        "gptb200_decoder_set_option": (i, [vp, ctypes.c_char_p, i]),
        "gptb200_decoder_step": (i, [vp, i, vp, vp, vp, i, vp, vp]),
        "gptb200_decoder_generate": (i, [vp, i, vp, vp, i, f32, ull, vp]),
        "gptb200_rotary_frequencies": (i, [i, ctypes.c_double, dp, dp, dp]),
        "gptb200_linear_bf16": (i, [vp, i, vp, ll, vp, ll, vp, i, i, i, vp, i, i, vp, vp, i]),
        "gptb200_sample_rows": (i, [vp, vp, vp, i, i, ll, f32, ull, ull]),
        "gptb200_ctx_launch_count": (ll, [vp]),
        "gptb200_ctx_synchronize": (i, [vp]),
        "gptb200_last_error": (ctypes.c_char_p, [vp]),
    }
    for name, (res, args) in sig.items():
        fn = getattr(lib, name)
        fn.restype = res
        fn.argtypes = args
    _lib = lib
    return lib


def check_config(text: str) -> str:
    """Empty if the library can run a model with this config.json, else the reason (host only)."""
    buf = ctypes.create_string_buffer(512)
    rc = load_library().gptb200_decoder_check_config(text.encode(), buf, len(buf))
    return buf.value.decode() if rc != 0 else ""


def rotary_frequencies(rot: dict):
    """(frequencies of the rotated pairs, factor on cosine and sine) as the library computes them (host only)."""
    s = rot.get("scaling")
    four = (ctypes.c_double * 4)(*[float(s[k]) for k in ("factor", "original", "fast", "slow")]) if s else None
    freq, gain = (ctypes.c_double * (rot["dims"] // 2))(), ctypes.c_double()
    rc = load_library().gptb200_rotary_frequencies(rot["dims"], float(rot["base"]), four, freq, ctypes.byref(gain))
    if rc != 0:
        raise GptB200Error(rc, "gptb200_rotary_frequencies")
    return np.array(freq), gain.value


def _ints(values) -> np.ndarray:
    return np.ascontiguousarray(values, dtype=np.int32)


class Decoder:
    """One loaded model.  Sequences are numbers from open(); step() runs any mixture of them."""

    batched = True   # several sequences per step

    def __init__(self, folder: str, dtype: str = "bfloat16", device: int = 0, stream: int | None = None):
        if dtype not in DTYPES:
            raise ValueError(f"dtype must be one of {sorted(DTYPES)}")
        self._lib = load_library()
        self._d = ctypes.c_void_p()
        message = ctypes.create_string_buffer(512)
        rc = self._lib.gptb200_decoder_load(ctypes.byref(self._d), os.fspath(folder).encode(), DTYPES[dtype], device, ctypes.c_void_p(stream or 0), message, len(message))
        if rc != 0:
            raise GptB200Error(rc, "gptb200_decoder_load", message.value.decode())
        self.vocab = int(self._lib.gptb200_decoder_vocab(self._d))

    def close_model(self) -> None:
        if self._d:
            self._lib.gptb200_decoder_destroy(self._d)
            self._d = ctypes.c_void_p()

    def __del__(self):  # pragma: no cover - best effort
        try:
            self.close_model()
        except Exception:
            pass

    @property
    def context(self) -> int:
        return int(self._lib.gptb200_decoder_context(self._d))

    def _check(self, rc: int, what: str) -> None:
        if rc != 0:
            raise GptB200Error(rc, what, self._lib.gptb200_last_error(ctypes.c_void_p(self.context)).decode())

    def set_option(self, key: str, value: int) -> None:
        self._check(self._lib.gptb200_decoder_set_option(self._d, key.encode(), value), "gptb200_decoder_set_option")

    def launch_count(self) -> int:
        return int(self._lib.gptb200_ctx_launch_count(ctypes.c_void_p(self.context)))

    def open(self, max_len: int) -> int:
        slot = ctypes.c_int()
        self._check(self._lib.gptb200_decoder_open(self._d, max_len, ctypes.byref(slot)), "gptb200_decoder_open")
        return slot.value

    def close(self, seq: int) -> None:
        self._check(self._lib.gptb200_decoder_close(self._d, seq), "gptb200_decoder_close")

    def length(self, seq: int) -> int:
        return int(self._lib.gptb200_decoder_length(self._d, seq))

    def step(self, entries, want) -> np.ndarray:
        """entries: [(sequence, tokens)]; want: rows of the step (all tokens numbered through) -> logits [len(want), vocab] fp32."""
        slots, counts = _ints([s for s, _ in entries]), _ints([len(t) for _, t in entries])
        tokens = _ints(np.concatenate([_ints(t) for _, t in entries]))
        rows = _ints(want)
        out = np.empty((len(rows), self.vocab), np.float32)
        self._check(self._lib.gptb200_decoder_step(self._d, len(slots), slots.ctypes.data, counts.ctypes.data, tokens.ctypes.data, len(rows), rows.ctypes.data if len(rows) else None,
                                                   out.ctypes.data if len(rows) else None), "gptb200_decoder_step")
        return out

    def generate(self, seqs, first, steps: int, temperature: float = 0.0, seed: int = 0) -> np.ndarray:
        """steps tokens for every sequence after the token first[i]: int32 [steps, len(seqs)]; the last one is not run."""
        slots, tok = _ints(seqs), _ints(first)
        out = np.empty((steps, len(slots)), np.int32)
        self._check(self._lib.gptb200_decoder_generate(self._d, len(slots), slots.ctypes.data, tok.ctypes.data, steps, temperature, seed, out.ctypes.data), "gptb200_decoder_generate")
        return out
