"""Bindings of the residual-stream kernel (``csrc/streams.cu``).

``embed`` starts the streams of a step's rows, ``boundary`` adds a sublayer's result to them; both leave what the next
sublayer reads in ``h`` (norm with one number; ``mu`` / ``prev``: token shift against the row before, or the layer's state).
``next_h`` [slots][ld] holds the last unshifted row of every sequence until the boundary with ``commit`` stores it."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def _launch(y, slices, embed, tokens, freq, flag, m, streams, width, req, pos, x_in, x_out, w_mix, w_out, scale, mult, w_in, norm,
            eps, h, mu, prev, next_h, commit):
    ld = h.shape[1]
    K._check(K.lib().b2_streams(K._p(y), ctypes.c_longlong(m * ld), slices, K._p(embed), K._p(tokens), K._p(freq),
                                embed.shape[0] if embed is not None else 0, _f32(embed) if embed is not None else 0, K._p(flag),
                                K._p(req), K._p(pos), m, streams, width, ld, K._p(x_in), K._p(x_out), K._p(w_mix), K._p(w_out),
                                K._p(scale), ctypes.c_float(mult), K._p(w_in), K._p(norm), ctypes.c_float(eps), K._p(h), _f32(h),
                                K._p(mu), K._p(prev), K._p(next_h), K._p(commit), K._stream()), "streams")


def embed(table, tokens, freq, flag, *, m, streams, width, req, pos, eps, norm, h, x_out, w_in=None, mu=None, prev=None, next_h=None):
    """Streams = embedding row + sines and cosines of ``pos * freq`` (fp64 angles per position; None: none)."""
    _launch(None, 0, table, tokens, freq, flag, m, streams, width, req, pos, None, x_out, None, None, None, 0.0, w_in, norm, eps, h,
            mu, prev, next_h, None)


def boundary(y, slices: int, w, q: int, mult: float, *, m, streams, width, req, pos, eps, x_in, x_out, norm, h, w_in=None, mu=None,
             prev=None, next_h=None, commit=None):
    """``y``: fp32 slices [slices][m][ld] of sublayer ``q`` (0: mixer, 1: feed-forward) of the layer with
    ``models.weights.StreamWeights`` ``w``; ``x_out`` None: the streams end here."""
    _launch(y, slices, None, None, None, None, m, streams, width, req, pos, x_in, x_out, w.w_mix[q], w.w_out[q], w.scale[q], mult,
            w_in, norm, eps, h, mu, prev, next_h, commit)
