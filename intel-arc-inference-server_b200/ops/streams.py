"""Bindings of the residual-stream kernel (``csrc/streams.cu``).

``embed`` starts the streams of a step's rows, ``boundary`` adds a sublayer's result to them; both leave what the next
sublayer reads in ``h`` (norm with one number, or with a factor per column; ``mu`` / ``prev``: token shift against the row
before, or the layer's state -- with ``mu`` ``[planes][ld]`` one shifted result per plane in ``h`` ``[planes * m][ld]``).
``next_h`` [slots][ld] holds the last unshifted row of every sequence until the boundary with ``commit`` stores it.
``again`` (embedding table, tokens) and ``add`` [ld] are added to the streams ahead of the norm."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def _launch(y, slices, table, tokens, freq, flag, m, streams, width, req, pos, x_in, x_out, w_mix, w_out, scale, mult, w_in, norm,
            eps, h, mu, prev, next_h, commit, bias, add, again):
    ld = h.shape[1]
    planes = 1 if mu is None or mu.dim() == 1 else mu.shape[0]
    K._check(K.lib().b2_streams(K._p(y), ctypes.c_longlong(m * ld), slices, K._p(table), K._p(tokens), K._p(freq),
                                table.shape[0] if table is not None else 0, _f32(table) if table is not None else 0, K._p(flag),
                                K._p(req), K._p(pos), m, streams, width, ld, K._p(x_in), K._p(x_out), K._p(w_mix), K._p(w_out),
                                K._p(scale), ctypes.c_float(mult), K._p(w_in), K._p(norm), int(norm.numel() > 1), ctypes.c_float(eps),
                                K._p(h), _f32(h), K._p(mu), planes, K._p(prev), K._p(next_h), K._p(commit), K._p(bias), K._p(add),
                                int(again), K._stream()), "streams")


def embed(table, tokens, freq, flag, *, m, streams, width, req, pos, eps, norm, h, x_out, w_in=None, mu=None, prev=None, next_h=None,
          add=None, again=None):
    """Streams = embedding row + sines and cosines of ``pos * freq`` (fp64 angles per position; None: none)."""
    if again is not None:
        raise ValueError("the streams start as the embedding row")
    _launch(None, 0, table, tokens, freq, flag, m, streams, width, req, pos, None, x_out, None, None, None, 0.0, w_in, norm, eps, h,
            mu, prev, next_h, None, None, add, False)


def boundary(y, slices: int, w, q: int, mult: float, *, m, streams, width, req, pos, eps, x_in, x_out, norm, h, w_in=None, mu=None,
             prev=None, next_h=None, commit=None, bias=None, add=None, again=None, freq=None):
    """``y``: fp32 slices [slices][m][ld] of sublayer ``q`` (0: mixer, 1: feed-forward) of the layer with
    ``models.weights.StreamWeights`` ``w`` (None: one stream that keeps itself); ``bias`` [ld] of its linear; ``x_out`` None: the
    streams end here."""
    table, tokens = again or (None, None)
    mix, out, scale = (w.w_mix[q], w.w_out[q], w.scale[q]) if w is not None else (None, None, None)
    _launch(y, slices, table, tokens, freq, None, m, streams, width, req, pos, x_in, x_out, mix, out, scale, mult,
            w_in, norm, eps, h, mu, prev, next_h, commit, bias, add, again is not None)
