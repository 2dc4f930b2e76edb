"""Bindings of the recurrences with a decay per key channel (``csrc/channel_rec.cu``).  ``act``: prepared fp32 rows
(``act_cols`` columns); ``lr``: (fp32 slices, their number) of the second half of the low-rank projections, or None, and the
kernel takes the dots from their weight ``w2`` itself."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def act_cols(hq: int, h: int, dk: int, dv: int) -> int:
    """Columns of a prepared row: q | k | decay | v | gate | two numbers per head, each padded to fours."""
    return 2 * hq * dk + h * (dk + 2 * dv) + 2 * ((h + 3) // 4 * 4)


def fused(dk: int, dv: int) -> bool:
    """Rows one by one: the scan norms and gates its rows itself."""
    return bool(K.lib().b2_channel_fused(dk, dv))


def lowrank_rows(part, s: int, m: int, cols, ranks, kp: int, tanh: bool, out):
    """First halves (columns ``cols[i]`` .. + ``ranks[i]`` of the projection's slices) as rows ``[planes][m][kp]`` fp32, or
    bf16 ``[planes][m][2 kp]`` in two limbs."""
    two = len(cols) > 1
    K._check(K.lib().b2_lowrank_rows(K._p(part), s, m, part.shape[1], len(cols), cols[0], ranks[0], cols[1] if two else 0,
                                     ranks[1] if two else 0, kp, int(tanh), K._p(out), _f32(out), K._stream()), "lowrank_rows")


def _second(lr):
    return (K._p(lr[0]), lr[1]) if lr is not None else (None, 0)


def delta_prep(part, s: int, m: int, g, a, w, req, pos, conv_state, conv_next, lr, act):
    """``g``: ``models.channel_delta.DeltaGeometry``, ``a``: ``ChannelDelta``, ``w``: ``DeltaWeights``."""
    ptr, n = _second(lr)
    K._check(K.lib().b2_delta_prep(K._p(part), s, m, part.shape[1], g.kv_heads, g.heads, g.dk, g.dv, a.dim, g.col_b, g.col_a1, a.a_rank,
                                   g.col_g1, a.g_rank, K._p(req), K._p(pos), g.taps, K._p(w.conv), K._p(conv_state), K._p(conv_next),
                                   K._p(w.neg_a), K._p(w.dt_bias), ptr, n, K._p(w.second), g.kp, w.second.stride(0), K._p(act),
                                   _f32(w.second), K._stream()), "delta_prep")


def wkv_prep(part, s: int, m: int, g, a, w, lr, act):
    """``g``: ``models.wkv.WkvGeometry``, ``a``: ``Wkv``, ``w``: ``WkvWeights``."""
    ptr, n = _second(lr)
    K._check(K.lib().b2_wkv_prep(K._p(part), s, m, part.shape[1], g.heads, g.d, a.w_rank, K._p(w.u), K._p(w.w0), ptr, n, K._p(w.second),
                                 g.kp, w.second.stride(0), K._p(act), _f32(w.second), K._stream()), "wkv_prep")


def block_bytes(delta: bool, dk: int, dv: int) -> int:
    """Workspace of the tensor-core form per (16 rows of a segment, head); 0: the sizes are outside it."""
    return K.lib().b2_channel_block_bytes(int(delta), dk, dv)


def scan(act, delta: bool, m: int, hq: int, h: int, dk: int, dv: int, vdim: int, req, pos, t, state, norm, eps: float, raw, out,
         conv_next=None, conv_state=None, ws=None):
    """The recurrence over prepared rows, head norm and gate.  ``t``: the rows' segments (``runtime.batch.ChunkPlan``), or None: a
    sequence per run of equal ``req``; ``ws`` (segments; uint8, ``4 * t.chunks * h`` blocks): on the tensor cores."""
    elems = conv_state[0].numel() if conv_state is not None else 0
    K._check(K.lib().b2_channel_scan(K._p(act), int(delta), m, hq, h, dk, dv, vdim, K._p(req), K._p(pos), K._p(t.segs if t else None),
                                     t.n_segs if t else 0, t.chunks if t else 0, t.most if t else 0, K._p(state), K._p(conv_next),
                                     K._p(conv_state), elems, K._p(norm), ctypes.c_float(eps), K._p(ws),
                                     ctypes.c_longlong(ws.numel() if ws is not None else 0), K._p(raw), K._p(out), _f32(out), K._stream()),
             "channel_scan")
    K.launch_count += int(t is not None or not fused(dk, dv)) + int(ws is not None)
