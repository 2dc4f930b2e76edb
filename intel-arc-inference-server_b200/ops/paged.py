"""Bindings of the grouped-query attention over pages (``csrc/paged.cu``) and of its prompt form
(``csrc/attn_prefill.cu``).  ``g``: ``models.grouped.GroupedGeometry``; ``slope2`` / ``sink2``: distance bias and sinks per
head times log2 e, or None; ``logb``: (r1, r2) of a logarithmic distance bias, or None; ``chunk`` 0: no chunks; ``out``: rows
whose first ``g.heads * g.dv`` columns are written, times ``mult``."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def append(part, s: int, m: int, g, with_kv: bool, req, pos, block_table, q, k, v):
    """fp32 slices of the projection: queries to ``q``, keys and values into the pages."""
    K._check(K.lib().b2_kv_append(K._p(part), 0, s, m, g.nq, g.kv_heads, g.dk, g.dv, int(with_kv), K._p(req), K._p(pos),
                                  K._p(block_table), block_table.shape[1], K._p(q), K._p(k), K._p(v), _f32(q), K._stream()),
             "kv_append")


def append_rows(qkv, m: int, g, req, pos, block_table, k, v):
    """bf16 rows q | k | v: keys and values into the pages."""
    K._check(K.lib().b2_kv_append(K._p(qkv), 1, 1, m, g.nq, g.kv_heads, g.dk, g.dv, 1, K._p(req), K._p(pos), K._p(block_table),
                                  block_table.shape[1], None, K._p(k), K._p(v), 0, K._stream()), "kv_append_rows")


def norm(part, s: int, m: int, g, a, w, eps: float, req, pos, block_table, q, k, v):
    """fp32 slices ``[s][m][part columns]`` whose first columns are q | k | v: biases, norms and query temperature of
    ``models.config.GroupedAttention`` ``a`` with ``models.weights.GroupedWeights`` ``w``; queries to ``q``, keys and values
    into the pages."""
    K._check(K.lib().b2_kv_norm(K._p(part), s, m, part.shape[1], g.heads, g.kv_heads, g.dk, g.dv, a.dim, a.vdim, K._p(w.bias),
                                K._p(w.q_norm), K._p(w.k_norm), int(a.v_norm), ctypes.c_float(eps), ctypes.c_float(a.temp),
                                a.temp_every, K._p(req), K._p(pos), K._p(block_table), block_table.shape[1], K._p(q), K._p(k),
                                K._p(v), _f32(q), K._stream()), "kv_norm")


def rows_ok(g) -> bool:
    return bool(K.lib().b2_paged_rows_ok(g.dk, g.dv))


def rows(q, k, v, m: int, g, req, pos, block_table, nsplit: int, chunk: int, scale: float, slope2, sink2, o_part, ml_part, out,
         logb=None, mult: float = 1.0):
    r1, r2 = logb or (None, None)
    K._check(K.lib().b2_paged_rows(K._p(q), q.stride(0), K._p(k), K._p(v), m, g.heads, g.kv_heads, g.dk, g.dv, K._p(req), K._p(pos),
                                   K._p(block_table), block_table.shape[1], nsplit, chunk, ctypes.c_float(scale), K._p(slope2),
                                   K._p(sink2), K._p(r1), K._p(r2), K._p(o_part), K._p(ml_part), K._p(out), out.stride(0),
                                   ctypes.c_float(mult), K._stream()), "paged_rows")
    if nsplit > 1:
        K.launch_count += 1      # the merge


def simple(q, k, v, m: int, g, req, pos, block_table, chunk: int, scale: float, slope2, sink2, out, logb=None, mult: float = 1.0):
    r1, r2 = logb or (None, None)
    K._check(K.lib().b2_paged_simple(K._p(q), q.stride(0), K._p(k), K._p(v), m, g.heads, g.kv_heads, g.dk, g.dv, K._p(req), K._p(pos),
                                     K._p(block_table), block_table.shape[1], chunk, ctypes.c_float(scale), K._p(slope2), K._p(sink2),
                                     K._p(r1), K._p(r2), K._p(out), out.stride(0), ctypes.c_float(mult), _f32(out), K._stream()),
             "paged_simple")


def segments_per_tile(g) -> int:
    """Query rows one CTA of the prompt attention serves (0: the sizes are outside its forms)."""
    return K.lib().b2_attn_segments_per_tile(g.dk, g.dv)


def attn_segments(q, k, v, block_table, out, tiles, n_tiles: int, q_rows: int, g, scale: float, chunk: int, slope2, sink2,
                  logb=None, mult: float = 1.0):
    r1, r2 = logb or (None, None)
    K._check(K.lib().b2_attn_prefill_segments(K._p(q), q.stride(0), K._p(k), K._p(v), K._p(block_table), block_table.shape[1],
                                              K._p(out), K._p(tiles), n_tiles, q_rows, g.heads, g.kv_heads, g.dk, g.dv, k.shape[0],
                                              ctypes.c_float(scale), chunk, K._p(slope2), K._p(sink2), K._p(r1), K._p(r2), out.stride(0),
                                              ctypes.c_float(mult), K._stream()), "attn_prefill_segments")
