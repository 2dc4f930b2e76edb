"""Bindings of the boundary kernel of residuals with norms on both sides of a sublayer (``csrc/sandwich.cu``)."""
from __future__ import annotations

import ctypes

import torch

from . import lib as K
from .latent import _f32


class _Source(ctypes.Structure):
    _fields_ = [("y", ctypes.c_void_p), ("row_of", ctypes.c_void_p), ("slot_w", ctypes.c_void_p), ("slice", ctypes.c_longlong),
                ("row", ctypes.c_longlong), ("slots", ctypes.c_int), ("slices", ctypes.c_int), ("bf16", ctypes.c_int),
                ("factor", ctypes.c_float), ("norm", ctypes.c_void_p)]


def source(y, row_elems: int, *, slices: int = 1, slice_elems: int = 0, slots: int = 1, slot_w=None, row_of=None, factor: float = 1.0,
           norm=None) -> _Source:
    """What a sublayer left: value row ``r`` starts at ``r * row_elems`` of ``y`` and has ``slices`` slices ``slice_elems`` apart; a
    row is the sum of its slots weighted by ``slot_w`` (slot ``s`` of row ``i``: value row ``row_of[i * slots + s]``, or
    ``i * slots + s``), times ``factor``; ``norm``: weight of an RMS norm ahead of the factor (two sources only)."""
    ptr = lambda t: 0 if t is None else t.data_ptr()        # noqa: E731
    s = _Source(ptr(y), ptr(row_of), ptr(slot_w), slice_elems, row_elems, slots, slices, int(y.dtype == torch.bfloat16), factor, ptr(norm))
    s.tensors = (y, row_of, slot_w, norm)       # alive as long as the source
    return s


def boundary(sources, *, m: int, width: int, groups: int, eps: float, post, next, x_in, x_out, h, vocab: int = 0, flag=None):
    """``x_out = x_in + G(y) * post`` and ``h = G(x_out) * next``, with y the sum of the ``sources``.  ``x_in`` / ``post`` None: none
    of it; ``x_out`` None: the residual ends here; ``vocab``: value rows are tokens."""
    arr = (_Source * len(sources))(*sources)
    K._check(K.lib().b2_sandwich(ctypes.byref(arr), len(sources), vocab, K._p(flag), m, width, h.shape[-1], groups, ctypes.c_float(eps),
                                 K._p(post), K._p(next), K._p(x_in), K._p(x_out), K._p(h), _f32(h), K._stream()), "sandwich")
