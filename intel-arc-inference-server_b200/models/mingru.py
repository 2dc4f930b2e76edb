"""minGRU mixers: an elementwise recurrence whose gates read the current token only; one fp32 number per channel, sequence and
layer.  Rows of a step are walked in order; long segments of a prompt in blocks of rows that are reduced side by side."""
from __future__ import annotations

from typing import Optional

from ..ops import mingru as R
from .config import MinGru, ModelConfig
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, pad64
from .weights import MinGruWeights


def shapes(cfg: ModelConfig, p: str, a: MinGru) -> dict:
    h, n = cfg.hidden, a.width
    return {p + "z": (n, h), p + "z.b": (n,), p + "x": (n, h), p + "x.b": (n,), p + "g": (n, h), p + "o": (h, n)}


def assemble(t, p: str, a: MinGru) -> MinGruWeights:
    """``t``: ``listed.Assembler``."""
    n = pad64(a.width)
    return MinGruWeights(t.stack([t.padded(t.t(p + x), n, t.wp) for x in "zxg"]), t.padded(t.t(p + "o"), t.wp, n),
                         t.vec(p + "z.b", n), t.vec(p + "x.b", n))


def weight_elems(cfg: ModelConfig, a: MinGru) -> int:
    return 4 * pad64(cfg.hidden) * pad64(a.width)


def scratch_elems(cfg: ModelConfig, a: MinGru, rows: int, keys: int) -> int:
    return rows * 9 * 3 * pad64(a.width) + rows * pad64(a.width)


def page_planes(a: MinGru) -> dict:
    return {}


def state_shapes(a: MinGru) -> dict:
    return {"gru": (pad64(a.width),)}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: MinGru, w: MinGruWeights):
        self.ll, self.li, self.a, self.w = ll, li, a, w
        self.n = pad64(a.width)
        self.cols = 3 * self.n                  # columns of its projection, and of what its output projection reads
        self.out_cols = self.n
        self.forms = [("chunks",)] if ll.device.type == "cuda" else []

    def core(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan], part, s: int, col: int, out,
             mult: float = 1.0):
        """From its columns ``col`` .. of the projection's fp32 slices to its rows ``out``, times ``mult``."""
        n1 = m if plan is None else plan.n_single
        t = plan.tables[self.forms[0]] if n1 < m else None
        R.scan(part, s, m, col, self.n, self.w, rows.req, rows.pos, n1, t.segs if t else None, t.n_segs if t else 0, mult,
               kv.states[f"gru{self.li}"][0], out)

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """The recurrence over the step's rows: fp32 slices of its output projection."""
        ll, w = self.ll, self.w
        part, s = ll.linear(sc, "gru_in", w.proj, sc.get("h", m, ll.wp), m)
        out = sc.get("gru_out", m, self.n)
        self.core(sc, m, rows, block_table, kv, plan, part, s, 0, out)
        return ll.linear(sc, "o", w.o, out, m)
