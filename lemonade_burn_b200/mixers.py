"""Descriptions of the sequence mixers for the calls of include/lbk.h that run one alone."""
from __future__ import annotations

import ctypes as C
from typing import Optional, Sequence, Tuple

import numpy as np

from . import _lib


class LatentDesc(C.Structure):
    _fields_ = [(n, C.c_size_t) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")] + [("freq_dev", C.c_void_p), ("rot_factor", C.c_float)]


class RecurrenceDesc(C.Structure):
    _fields_ = [("delta", C.c_int)] + [(n, C.c_size_t) for n in ("heads", "kv_heads", "dim", "vdim", "taps")]


def rotation_frequencies(dims: int, base: float, yarn: Optional[Sequence[float]] = None) -> Tuple[np.ndarray, float]:
    """(frequency of each pair, factor on cos and sin); yarn: (factor, original, fast, slow)."""
    freq, factor = np.empty(dims // 2, dtype=np.float64), C.c_float()
    y = None if yarn is None else np.asarray(yarn, dtype=np.float64)
    _lib.check(_lib.load().lbk_rotation_frequencies(dims, base, None if y is None else y.ctypes.data_as(C.c_void_p), freq.ctypes.data_as(C.c_void_p),
                                                    C.cast(C.byref(factor), C.c_void_p)))
    return freq, float(factor.value)
