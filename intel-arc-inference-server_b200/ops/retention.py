"""Bindings of the fixed-decay recurrence (``csrc/retention.cu``).  ``g``: ``models.retention.RetentionGeometry``, ``a``:
``models.config.Retention``; ``part``: fp32 slices of a projection whose columns from ``col`` are q | k | v | gate; ``rope``: (cos, sin)
``[positions][pairs]``; ``decay`` fp32 ``[2][heads]``: the decays and their log2; ``state`` ``[slots][heads * dk * dv]`` fp32; ``out``:
rows whose first ``g.heads * g.dv`` columns are written, times ``mult``."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def step(part, s: int, m: int, col: int, g, a, req, pos, rope, eps: float, mult: float, decay, state, out):
    """Rows in order, one token at a time."""
    K._check(K.lib().b2_retention_step(K._p(part), s, m, part.shape[1], col, g.heads, g.dk, g.dv, a.vdim, K._p(req), K._p(pos), K._p(rope[0]),
                                       K._p(rope[1]), rope[0].shape[1], ctypes.c_float(a.dim ** -0.5), ctypes.c_float(eps),
                                       ctypes.c_float(mult), K._p(decay), K._p(state), K._p(out), out.stride(0), _f32(out), K._stream()),
             "retention_step")


def chunks_ok(g) -> bool:
    return bool(K.lib().b2_retention_chunks_ok(g.dk, g.dv))


def wants_raw(g) -> bool:
    return bool(K.lib().b2_retention_raw(g.dk, g.dv))


def chunk_rows() -> int:
    return K.lib().b2_retention_chunk_rows()


def segments(part, m: int, col: int, g, a, t, pos, rope, eps: float, mult: float, decay, state, kv, raw, out):
    """Prompt segments (``t``: ``runtime.batch.ChunkPlan`` in chunks of ``chunk_rows()``); ``kv``: fp32, ``t.chunks * heads`` states;
    ``raw``: fp32 ``[m][heads * dv]`` where ``wants_raw``."""
    K._check(K.lib().b2_retention_segments(K._p(part), m, part.shape[1], col, g.heads, g.dk, g.dv, a.vdim, K._p(pos), K._p(t.segs), t.n_segs,
                                           t.most, K._p(rope[0]), K._p(rope[1]), rope[0].shape[1], ctypes.c_float(a.dim ** -0.5),
                                           ctypes.c_float(eps), ctypes.c_float(mult), K._p(decay), K._p(state), K._p(kv), K._p(raw),
                                           K._p(out), out.stride(0), K._stream()), "retention_segments")
    K.launch_count += 2 + int(raw is not None)      # sums, scan, rows (and the head norm)
