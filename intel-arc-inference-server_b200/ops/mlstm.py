"""Bindings of the mLSTM kernels (``csrc/mlstm.cu``).  ``g``: ``models.mlstm.MlstmGeometry``, ``a``: ``MatrixLstm``;
``state`` [slots][g.state_elems] fp32."""
from __future__ import annotations

import ctypes

from . import lib as K
from .latent import _f32


def step(part, s: int, m: int, n: int, g, a, req, pos, gate_bias, eps: float, norm, state, out):
    """Rows in order, one token at a time; ``part``: fp32 slices [s][m][n] of the projection."""
    K._check(K.lib().b2_mlstm_step(K._p(part), s, m, n, g.heads, g.dk, g.dv, a.dim, a.vdim, K._p(req), K._p(pos), K._p(gate_bias),
                                   ctypes.c_float(a.gate_cap), ctypes.c_float(eps), K._p(norm), K._p(state), K._p(out), _f32(out),
                                   K._stream()), "mlstm_step")


def chunks_ok(g) -> bool:
    return bool(K.lib().b2_mlstm_chunks_ok(g.dk, g.dv))


def segments(proj, z, rows: int, g, a, t, pos, gate_bias, eps: float, norm, state, gates, raw, out):
    """Prompt segments (``t``: ``runtime.batch.ChunkPlan``) in chunks of 64 rows."""
    K._check(K.lib().b2_mlstm_segments(K._p(proj), proj.stride(0), K._p(z), z.stride(0), rows, g.heads, g.dk, g.dv, a.dim, a.vdim,
                                       K._p(t.segs), t.n_segs, t.chunks, t.most, K._p(pos), K._p(gate_bias),
                                       ctypes.c_float(a.gate_cap), ctypes.c_float(eps), K._p(norm), K._p(state), K._p(gates),
                                       K._p(raw), K._p(out), K._stream()), "mlstm_segments")
    K.launch_count += 2      # gates, scan, output
