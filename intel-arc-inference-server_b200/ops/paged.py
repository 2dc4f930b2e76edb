"""Bindings of the grouped-query attention over pages (``csrc/paged.cu``) and of its prompt form
(``csrc/attn_prefill.cu``).  ``g``: ``models.grouped.GroupedGeometry``; ``slope2`` / ``sink2``: distance bias and sinks per
head times log2 e, or None; ``logb``: (r1, r2) of a logarithmic distance bias, or None; ``chunk`` 0: no chunks; ``out``: rows
whose first ``g.heads * g.dv`` columns are written, times ``mult``; ``extra``: ``Extra``, or None."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from . import lib as K
from .latent import _f32


class _AttnExtra(ctypes.Structure):
    _fields_ = [(n, ctypes.c_void_p) for n in ("cos", "sin", "vcos", "vsin")] + [(n, ctypes.c_int) for n in ("rd", "vd", "tied", "gate_col")] \
        + [("gate", ctypes.c_void_p)] + [(n, ctypes.c_int) for n in ("ldg", "window", "pool", "slots")] + [("pk", ctypes.c_void_p), ("pv", ctypes.c_void_p)]


class _SegExtra(ctypes.Structure):
    _fields_ = [(n, ctypes.c_int) for n in ("window", "pool", "pool_rows")] + [(n, ctypes.c_void_p) for n in ("pool_row", "pk", "pv", "cos", "sin")] \
        + [("half", ctypes.c_int), ("gate", ctypes.c_void_p), ("ldg", ctypes.c_int)]


def _ptr(t) -> int:
    return 0 if t is None else t.data_ptr()


@dataclass
class Extra:
    """What an attention call has beyond plain causal keys: rotations (tables ``[positions][pairs]`` of cosines and sines, of pairs
    of neighbouring dimensions) of queries and keys and of values -- the latter's results are turned back --, values that are the
    unrotated keys, gates of the results (``[rows][heads * dv]``; columns from ``gate_col`` of the projection), a window, and pooled
    blocks of ``pool`` positions before it (planes ``[page][kv head][slots][..]``)."""
    rot: Optional[tuple] = None
    vrot: Optional[tuple] = None
    tied: bool = False
    gate: Optional[torch.Tensor] = None
    gate_col: int = 0
    window: int = 0
    pool: int = 0
    pk: Optional[torch.Tensor] = None
    pv: Optional[torch.Tensor] = None

    def _struct(self) -> _AttnExtra:
        c, s = self.rot or (None, None)
        vc, vs = self.vrot or (None, None)
        return _AttnExtra(_ptr(c), _ptr(s), _ptr(vc), _ptr(vs), 0 if c is None else 2 * c.shape[1], 0 if vc is None else 2 * vc.shape[1],
                          int(self.tied), self.gate_col, _ptr(self.gate), 0 if self.gate is None else self.gate.stride(0), self.window,
                          self.pool, self.pk.shape[2] if self.pool else 0, _ptr(self.pk), _ptr(self.pv))


def _extra(x: Optional[Extra]):
    return None if x is None else ctypes.byref(x._struct())


def append(part, s: int, m: int, g, with_kv: bool, req, pos, block_table, q, k, v):
    """fp32 slices of the projection: queries to ``q``, keys and values into the pages."""
    K._check(K.lib().b2_kv_append(K._p(part), 0, s, m, g.nq, g.kv_heads, g.dk, g.dv, int(with_kv), K._p(req), K._p(pos),
                                  K._p(block_table), block_table.shape[1], K._p(q), K._p(k), K._p(v), _f32(q), K._stream()),
             "kv_append")


def append_rows(qkv, m: int, g, req, pos, block_table, k, v):
    """bf16 rows q | k | v: keys and values into the pages."""
    K._check(K.lib().b2_kv_append(K._p(qkv), 1, 1, m, g.nq, g.kv_heads, g.dk, g.dv, 1, K._p(req), K._p(pos), K._p(block_table),
                                  block_table.shape[1], None, K._p(k), K._p(v), 0, K._stream()), "kv_append_rows")


def norm(part, s: int, m: int, g, a, w, eps: float, req, pos, block_table, q, k, v, extra: Optional[Extra] = None):
    """fp32 slices ``[s][m][part columns]`` whose first columns are q | k | v (tied values: q | k): biases, norms, rotations and
    query temperature of ``models.config.GroupedAttention`` ``a`` with ``models.weights.GroupedWeights`` ``w``; queries to ``q``,
    keys and values into the pages, gates to ``extra.gate``, pooled blocks that end at one of the rows to their planes."""
    K._check(K.lib().b2_kv_norm(K._p(part), s, m, part.shape[1], g.heads, g.kv_heads, g.dk, g.dv, a.dim, a.vdim, K._p(w.bias),
                                K._p(w.q_norm), K._p(w.k_norm), int(a.v_norm), ctypes.c_float(eps), ctypes.c_float(a.temp),
                                a.temp_every, K._p(req), K._p(pos), K._p(block_table), block_table.shape[1], K._p(q), K._p(k),
                                K._p(v), _f32(q), _extra(extra), K._stream()), "kv_norm")


def pool_gather(req, block, n: int, g, block_table, pool: int, pk, pv, k, v):
    """Pooled blocks ``block[i]`` of slots ``req[i]`` as rows ``k`` ``[n][kv heads * dk]``, ``v`` ``[n][kv heads * dv]``."""
    K._check(K.lib().b2_pool_gather(K._p(req), K._p(block), n, K._p(block_table), block_table.shape[1], g.kv_heads, g.dk, g.dv, pool,
                                    pk.shape[2], K._p(pk), K._p(pv), K._p(k), K._p(v), K._stream()), "pool_gather")


def rows_ok(g) -> bool:
    return bool(K.lib().b2_paged_rows_ok(g.dk, g.dv))


def rows(q, k, v, m: int, g, req, pos, block_table, nsplit: int, chunk: int, scale: float, slope2, sink2, o_part, ml_part, out,
         logb=None, mult: float = 1.0, extra: Optional[Extra] = None):
    r1, r2 = logb or (None, None)
    K._check(K.lib().b2_paged_rows(K._p(q), q.stride(0), K._p(k), K._p(v), m, g.heads, g.kv_heads, g.dk, g.dv, K._p(req), K._p(pos),
                                   K._p(block_table), block_table.shape[1], nsplit, chunk, ctypes.c_float(scale), K._p(slope2),
                                   K._p(sink2), K._p(r1), K._p(r2), K._p(o_part), K._p(ml_part), K._p(out), out.stride(0),
                                   ctypes.c_float(mult), _extra(extra), K._stream()), "paged_rows")
    if nsplit > 1:
        K.launch_count += 1      # the merge


def simple(q, k, v, m: int, g, req, pos, block_table, chunk: int, scale: float, slope2, sink2, out, logb=None, mult: float = 1.0,
           extra: Optional[Extra] = None):
    r1, r2 = logb or (None, None)
    K._check(K.lib().b2_paged_simple(K._p(q), q.stride(0), K._p(k), K._p(v), m, g.heads, g.kv_heads, g.dk, g.dv, K._p(req), K._p(pos),
                                     K._p(block_table), block_table.shape[1], chunk, ctypes.c_float(scale), K._p(slope2), K._p(sink2),
                                     K._p(r1), K._p(r2), K._p(out), out.stride(0), ctypes.c_float(mult), _f32(out), _extra(extra),
                                     K._stream()), "paged_simple")


def segments_per_tile(g) -> int:
    """Query rows one CTA of the prompt attention serves (0: the sizes are outside its forms)."""
    return K.lib().b2_attn_segments_per_tile(g.dk, g.dv)


def attn_segments(q, k, v, block_table, out, tiles, n_tiles: int, q_rows: int, g, scale: float, chunk: int, slope2, sink2,
                  logb=None, mult: float = 1.0, extra: Optional[Extra] = None, pooled=None):
    """``extra.gate``: rows as in ``q``; ``pooled``: (rows of pooled keys, of pooled values, first row of every tile's sequence)."""
    r1, r2 = logb or (None, None)
    x = None
    if extra is not None:
        pk, pv, first = pooled or (None, None, None)
        vc, vs = extra.vrot or (None, None)
        x = _SegExtra(extra.window, extra.pool, 0 if pk is None else pk.shape[0], _ptr(first), _ptr(pk), _ptr(pv), _ptr(vc), _ptr(vs),
                      0 if vc is None else vc.shape[1], _ptr(extra.gate), 0 if extra.gate is None else extra.gate.stride(0))
    K._check(K.lib().b2_attn_prefill_segments(K._p(q), q.stride(0), K._p(k), K._p(v), K._p(block_table), block_table.shape[1],
                                              K._p(out), K._p(tiles), n_tiles, q_rows, g.heads, g.kv_heads, g.dk, g.dv, k.shape[0],
                                              ctypes.c_float(scale), chunk, K._p(slope2), K._p(sink2), K._p(r1), K._p(r2), out.stride(0),
                                              ctypes.c_float(mult), None if x is None else ctypes.byref(x), K._stream()),
             "attn_prefill_segments")
