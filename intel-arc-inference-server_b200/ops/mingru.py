"""Binding of the minGRU kernels (``csrc/mingru.cu``)."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def scan(part, s: int, m: int, col: int, width: int, w, req, pos, n1: int, segs, n_segs: int, mult: float, state, out):
    """fp32 slices ``[s][m][part columns]`` with gate | candidate | output gate from column ``col``; rows before ``n1`` one by
    one, the rest as segments.  ``out``: rows whose first ``width`` columns are written, times ``mult``."""
    K._check(K.lib().b2_mingru(K._p(part), s, m, part.shape[1], col, width, K._p(w.bias_z), K._p(w.bias_x), K._p(req), K._p(pos), n1,
                               K._p(segs), n_segs, ctypes.c_float(mult), K._p(state), K._p(out), out.stride(0), _f32(out),
                               K._stream()), "mingru")
    K.launch_count += int(0 < n1 < m)
