"""Retention mixers: linear attention with a fixed decay per head and no softmax, one fp32 matrix per head, sequence and layer.

Rows of a step update the state token by token; long segments of a prompt are cut into chunks whose products all run side by side
on the tensor cores, with one pass over the chunks' states in between.  Queries and keys are rotated where they are used, from the
projection's fp32 values."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import retention as R
from .config import ModelConfig, Retention
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, pad64, pair_order
from .weights import RetentionWeights


@dataclass(frozen=True)
class RetentionGeometry:
    """Kernel sizes: ``dk`` / ``dv`` columns of a head's keys / values; the projection's rows are q | k | v | gate of all heads."""
    heads: int
    dk: int
    dv: int

    @staticmethod
    def of(a: Retention) -> "RetentionGeometry":
        dk = pad64(a.dim)
        return RetentionGeometry(a.heads, dk if dk <= 256 else 384 if dk <= 384 else 512, pad64(a.vdim))

    @property
    def n(self) -> int:
        return 2 * self.heads * (self.dk + self.dv)


def shapes(cfg: ModelConfig, p: str, a: Retention) -> dict:
    h, qk, v = cfg.hidden, a.heads * a.dim, a.heads * a.vdim
    return {p + "q": (qk, h), p + "k": (qk, h), p + "v": (v, h), p + "g": (v, h), p + "o": (h, v)}


def assemble(t, p: str, a: Retention) -> RetentionWeights:
    """``t``: ``listed.Assembler``."""
    g, order = RetentionGeometry.of(a), pair_order(a.rot.dims, a.dim)
    parts = [t.heads(t.t(p + x), a.heads, [(size, pad)], t.wp, order if x in "qk" else None)
             for x, size, pad in (("q", a.dim, g.dk), ("k", a.dim, g.dk), ("v", a.vdim, g.dv), ("g", a.vdim, g.dv))]
    decay = torch.tensor([list(a.decay), [math.log2(d) if d > 0 else float("-inf") for d in a.decay]], dtype=torch.float32, device=t.device)
    return RetentionWeights(t.stack(parts), t.out_proj(p + "o", a.heads, a.vdim, g.dv), decay)


def weight_elems(cfg: ModelConfig, a: Retention) -> int:
    g = RetentionGeometry.of(a)
    return pad64(cfg.hidden) * (g.n + g.heads * g.dv)


def scratch_elems(cfg: ModelConfig, a: Retention, rows: int, keys: int) -> int:
    g = RetentionGeometry.of(a)
    chunks = rows // 128 + rows // 32 + 1 if rows > 64 and g.dk <= 256 else 0        # segments of 32 rows and more
    return rows * (9 * g.n + 2 * g.heads * g.dv) + chunks * g.heads * g.dk * g.dv


def page_planes(a: Retention) -> dict:
    return {}


def state_shapes(a: Retention) -> dict:
    g = RetentionGeometry.of(a)
    return {"retention": (g.heads * g.dk * g.dv,)}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: Retention, w: RetentionWeights):
        self.ll, self.li, self.a, self.w, self.g = ll, li, a, w, RetentionGeometry.of(a)
        self.rope = ll.rotation(a.rot)
        self.cols, self.out_cols = self.g.n, self.g.heads * self.g.dv      # columns of its projection, and of its rows
        chunks = ll.device.type == "cuda" and not ll.f32 and R.chunks_ok(self.g)
        self.forms = [("chunks", R.chunk_rows())] if chunks else []
        self.raw = bool(chunks) and R.wants_raw(self.g)

    def core(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan], part, s: int, col: int, out,
             mult: float = 1.0):
        """From its columns ``col`` .. of the projection's fp32 slices to its rows ``out``, times ``mult``."""
        a, g, w, eps = self.a, self.g, self.w, self.ll.cfg.rms_eps
        state = kv.states[f"retention{self.li}"][0]
        n1 = m if plan is None or not self.forms else plan.n_single
        if n1:
            R.step(part, s, n1, col, g, a, rows.req, rows.pos, self.rope, eps, mult, w.decay, state, out)
        if n1 < m:
            t = plan.tables[self.forms[0]]
            states = sc.get("retention_chunks", t.chunks, g.heads * g.dk * g.dv, torch.float32)
            raw = sc.get("retention_raw", m - n1, g.heads * g.dv, torch.float32) if self.raw else None
            R.segments(part[n1:], m - n1, col, g, a, t, rows.pos[n1:], self.rope, eps, mult, w.decay, state, states, raw, out[n1:])

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """The recurrence over the step's rows: fp32 slices of its output projection."""
        ll, w = self.ll, self.w
        part, s = ll.linear(sc, "retention_in", w.proj, sc.get("h", m, ll.wp), m)
        out = sc.get("retention_out", m, self.out_cols)
        self.core(sc, m, rows, block_table, kv, plan, part, s, 0, out)
        return ll.linear(sc, "o", w.o, out, m)
