"""mLSTM mixers: a matrix memory per head with exponential gates, one fp32 state per sequence and layer.

Rows of a step update the state token by token (``step``); long segments of a prompt go through the chunked form on the
tensor cores (``segments``), whose gates come from a GEMM of their own with fp32 results.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import gemm as G
from ..ops import mlstm as R
from .config import MatrixLstm, ModelConfig
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, pad64
from .weights import MlstmWeights


@dataclass(frozen=True)
class MlstmGeometry:
    """Kernel sizes: ``dk`` / ``dv`` columns of a head's keys / values; the projection's rows are q | k | v | output gate of
    all heads, then the input and forget gates."""
    heads: int
    dk: int
    dv: int

    @staticmethod
    def of(a: MatrixLstm) -> "MlstmGeometry":
        return MlstmGeometry(a.heads, pad64(a.dim), pad64(a.vdim))

    @property
    def n(self) -> int:
        return 2 * self.heads * (self.dk + self.dv)

    @property
    def gates(self) -> int:
        return (2 * self.heads + 7) // 8 * 8

    @property
    def state_elems(self) -> int:
        """Per value block of 32: S [dk][32], n [dk], the running maximum and padding."""
        return self.heads * (self.dv // 32) * (self.dk * 33 + 4)


def shapes(cfg: ModelConfig, p: str, a: MatrixLstm) -> dict:
    h, n = cfg.hidden, a.heads
    return {p + "q": (n * a.dim, h), p + "k": (n * a.dim, h), p + "v": (n * a.vdim, h), p + "g": (n * a.vdim, h),
            p + "o": (h, n * a.vdim), p + "norm": (n * a.vdim,), p + "i": (n, h), p + "i.b": (n,),
            p + "f": (n, h), p + "f.b": (n,)}


def assemble(t, p: str, a: MatrixLstm) -> MlstmWeights:
    """``t``: ``listed.Assembler``."""
    g, n = MlstmGeometry.of(a), a.heads
    parts = [t.heads(t.t(p + "" + x), n, [(size, pad)], t.wp)
             for x, size, pad in (("q", a.dim, g.dk), ("k", a.dim, g.dk), ("v", a.vdim, g.dv), ("g", a.vdim, g.dv))]
    gates = torch.cat([t.t(p + "i"), t.t(p + "f")])
    norm = torch.zeros(n, g.dv, dtype=torch.float32, device=t.device)
    norm[:, : a.vdim] = t.vec(p + "norm").view(n, a.vdim)
    return MlstmWeights(torch.cat(parts + [t.padded(gates, pad64(2 * n), t.wp)]), torch.cat([t.vec(p + "i.b"), t.vec(p + "f.b")]),
                        norm.view(-1), t.out_proj(p + "o", n, a.vdim, g.dv))


def weight_elems(cfg: ModelConfig, a: MatrixLstm) -> int:
    g = MlstmGeometry.of(a)
    return pad64(cfg.hidden) * (g.n + pad64(2 * a.heads) + a.heads * g.dv)


def scratch_elems(cfg: ModelConfig, a: MatrixLstm, rows: int, keys: int) -> int:
    g = MlstmGeometry.of(a)
    return rows * (9 * (g.n + pad64(2 * a.heads)) + 3 * a.heads * g.dv) + (rows // 64 + rows // 32 + 1) * 256 * a.heads


def page_planes(a: MatrixLstm) -> dict:
    return {}


def state_shapes(a: MatrixLstm) -> dict:
    return {"mlstm": (MlstmGeometry.of(a).state_elems,)}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: MatrixLstm, w: MlstmWeights):
        self.ll, self.li, self.a, self.w, self.g = ll, li, a, w, MlstmGeometry.of(a)
        chunks = ll.device.type == "cuda" and not ll.f32 and R.chunks_ok(self.g)
        self.forms = [("chunks",)] if chunks else []

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """The recurrence over the step's rows: fp32 slices of its output projection."""
        ll, a, g, w, eps = self.ll, self.a, self.g, self.w, self.ll.cfg.rms_eps
        state = kv.states[f"mlstm{self.li}"][0]
        h = sc.get("h", m, ll.wp)
        out = sc.get("mlstm_out", m, g.heads * g.dv)
        n1 = m if plan is None or not self.forms else plan.n_single
        if n1:
            part, s = ll.linear(sc, "mlstm_in", w.proj, h, n1)
            R.step(part, s, n1, w.proj.shape[0], g, a, rows.req, rows.pos, w.gate_bias, eps, w.norm, state, out)
        if n1 < m:
            t, n = plan.tables[self.forms[0]], m - n1
            proj, z = sc.get("mlstm_rows", n, g.n), sc.get("mlstm_gates", n, g.gates, torch.float32)
            G.gemm_bf16(h[n1:], w.proj[: g.n], proj)
            G.gemm_bf16(h[n1:], w.proj[g.n: g.n + g.gates], z, epi=G.EPI_F32)
            R.segments(proj, z, n, g, a, t, rows.pos[n1:], w.gate_bias, eps, w.norm, state,
                       sc.get("mlstm_chunks", t.chunks * g.heads, 256, torch.float32),
                       sc.get("mlstm_raw", n, g.heads * g.dv, torch.float32), out[n1:])
        return ll.linear(sc, "o", w.o, out, m)
