"""ctypes view of the step executor's C interface (include/ckb200_model.h): the configuration struct, argument types of the
ckb200_model_* entry points, and the two pointer helpers every caller of the library's C ABI needs.  Python only passes
pointers and sizes; all work happens in libckb200.so."""
from __future__ import annotations

import ctypes as C

import numpy as np

c_float_p = C.POINTER(C.c_float)


def fptr(a: np.ndarray):
    """float* of a C-contiguous float32 array."""
    assert a.dtype == np.float32 and a.flags["C_CONTIGUOUS"]
    return a.ctypes.data_as(c_float_p)


def vptr(a: np.ndarray):
    """void* of a C-contiguous array."""
    assert a.flags["C_CONTIGUOUS"]
    return C.c_void_p(a.ctypes.data)


class CfgStruct(C.Structure):
    """CKB200ModelConfig, field for field."""
    _fields_ = [(n, C.c_int) for n in ("embed_dim", "num_heads", "num_kv_heads", "head_dim", "intermediate_size", "num_layers", "vocab_size", "max_seq_len")] + \
               [("rms_eps", C.c_float), ("rope_theta", C.c_float)] + \
               [(n, C.c_int) for n in ("fmt_q", "fmt_k", "fmt_v", "fmt_o", "fmt_gate_up", "fmt_down", "fmt_lm_head", "fmt_embedding", "tie_embeddings", "batch", "tp_rank", "tp_size")]


def make_cfg(cfg: dict, batch=1, tp_rank=0, tp_size=1) -> CfgStruct:
    """A configuration with tied embeddings (the LM head doubles as the token table) from a dict of the model fields."""
    s = CfgStruct()
    for k, v in cfg.items():
        setattr(s, k, v)
    s.fmt_embedding = cfg["fmt_lm_head"]
    s.tie_embeddings = 1
    s.batch, s.tp_rank, s.tp_size = batch, tp_rank, tp_size
    return s


_P, _I = C.c_void_p, C.c_int
_MODEL_API = {
    # function: (result, arguments)
    "ckb200_model_create": (_P, [C.POINTER(CfgStruct)]),
    "ckb200_model_free": (None, [_P]),
    "ckb200_model_open": (_P, [C.c_char_p, _I]),
    "ckb200_model_open_bump": (_P, [C.c_char_p, C.c_char_p, _I]),
    "ckb200_model_config": (C.POINTER(CfgStruct), [_P]),
    "ckb200_model_family": (C.c_char_p, [_P]),
    "ckb200_model_upload_tensor": (_I, [_P, _I, _I, _P, C.c_size_t]),
    "ckb200_model_tensor_bytes": (C.c_size_t, [_P, _I, _I]),
    "ckb200_model_kv_device": (_P, [_P, _I, _I]),
    "ckb200_model_kv_element_bytes": (_I, [_P]),
    "ckb200_model_logits_device": (_P, [_P]),
    "ckb200_model_set_pos": (_I, [_P, _I]),
    "ckb200_model_get_pos": (_I, [_P]),
    "ckb200_model_reset": (_I, [_P]),
    "ckb200_model_decode": (_I, [_P, _P, _P]),
    "ckb200_model_decode_repeat": (_I, [_P, _I]),
    "ckb200_model_prefill": (_I, [_P, _P, _I, _P]),
    "ckb200_model_extend": (_I, [_P, _P, _I, _P, _I, _P]),
    "ckb200_model_probe_residual": (_I, [_P, _P, _I]),
    "ckb200_model_fill_synthetic": (_I, [_P, C.c_ulonglong]),
    "ckb200_model_fill_kv_synthetic": (_I, [_P, _I, C.c_ulonglong]),
    "ckb200_model_weight_bytes": (C.c_size_t, [_P]),
    "ckb200_model_use_tp": (None, [_P]),
    "ckb200_tune_set": (_I, [C.c_char_p, _I]),
    "ckb200_last_error_message": (C.c_char_p, []),
    "ckb200_copy_to_device": (_I, [_P, _P, C.c_size_t]),
    "ckb200_copy_to_host": (_I, [_P, _P, C.c_size_t]),
}


def bind_model_api(lib):
    """Declare argument and result types of the ckb200_model_* functions on a ctypes handle of libckb200.so, or of a library that holds
    one model family (which lacks the other families' own functions)."""
    for name, (res, args) in _MODEL_API.items():
        try:
            f = getattr(lib, name)
        except AttributeError:
            continue
        f.restype, f.argtypes = res, args


class Session:
    """One sequence on an open model: tokens go in portion by portion, logits come out at the places asked for."""

    def __init__(self, lib, spec: str, max_tokens: int | None = None, float32: bool = False):
        bind_model_api(lib)
        self.lib = lib
        if max_tokens:
            lib.ckb200_tune_set(b"model_max_seq", max_tokens)
        lib.ckb200_tune_set(b"model_f32", int(float32))
        self.handle = lib.ckb200_model_open(spec.encode(), 1)
        if not self.handle:
            raise RuntimeError((lib.ckb200_last_error_message() or b"cannot open the model").decode())
        self.vocab = lib.ckb200_model_config(self.handle).contents.vocab_size

    def _check(self, rc: int) -> None:
        if rc:
            raise RuntimeError((self.lib.ckb200_last_error_message() or b"step failed").decode())

    def extend(self, tokens, want=()) -> np.ndarray:
        """The next tokens of the sequence; fp32 logits [len(want), vocab] at the places `want` among them, in that order."""
        ids = np.ascontiguousarray(tokens, dtype=np.int32)
        places = np.unique(np.asarray(want, dtype=np.int32))
        out = np.empty((len(places), self.vocab), dtype=np.float32)
        self._check(self.lib.ckb200_model_extend(self.handle, vptr(ids), len(ids), vptr(places) if len(places) else None, len(places), vptr(out) if len(places) else None))
        return out[np.searchsorted(places, np.asarray(want, dtype=np.int32))] if len(places) else out

    def reset(self) -> None:
        """Give back what the sequence holds; the next one starts at position 0."""
        self._check(self.lib.ckb200_model_reset(self.handle))

    def close(self) -> None:
        if self.handle:
            self.lib.ckb200_model_free(self.handle)
            self.handle = None
