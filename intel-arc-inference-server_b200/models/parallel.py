"""Two mixers side by side on the same input.  Their input projections are one linear, and so are their output projections:
each mixer leaves its rows, times its scale, in its own columns of what the output projection reads.  Where each mixer's result
goes through a norm of its own the output projections stay apart (one launch over two planes of rows when they read equally many
columns), and the results are handed to the residual's boundary kernel, which norms and adds them.

Both mixers are of kinds with a ``core`` (from columns of a projection to rows): ``grouped``, ``retention``, ``mingru``."""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import sandwich as S
from .config import ModelConfig, ParallelMixer, SandwichBlock
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, kind, pad64
from .weights import GroupedWeights, ParallelWeights


def _sides(a: ParallelMixer):
    return ("left", a.left), ("right", a.right)


def shapes(cfg: ModelConfig, p: str, a: ParallelMixer) -> dict:
    out = {}
    for side, m in _sides(a):
        out.update(kind(m).shapes(cfg, f"{p}{side}.", m))
        if a.normed:
            out[f"{p}{side}.out"] = (cfg.hidden,)
    return out


def assemble(t, p: str, a: ParallelMixer) -> ParallelWeights:
    """``t``: ``listed.Assembler``."""
    parts, projs, outs = [], [], []
    for side, m in _sides(a):
        w = kind(m).assemble(t, f"{p}{side}.", m)
        name = "qkv" if isinstance(w, GroupedWeights) else "proj"
        projs.append(getattr(w, name))
        outs.append(w.o)
        setattr(w, name, None)
        w.o = None
        parts.append(w)
    if a.normed:
        norms = [t.vec(f"{p}{side}.out", t.wp) for side, _ in _sides(a)]
        if outs[0].shape == outs[1].shape:
            return ParallelWeights(torch.cat(projs), torch.cat(outs), *parts, norms)
        return ParallelWeights(torch.cat(projs), None, *parts, norms, outs)
    return ParallelWeights(torch.cat(projs), torch.cat(outs, dim=1).contiguous(), *parts)


def weight_elems(cfg: ModelConfig, a: ParallelMixer) -> int:
    return sum(kind(m).weight_elems(cfg, m) for _, m in _sides(a))


def scratch_elems(cfg: ModelConfig, a: ParallelMixer, rows: int, keys: int) -> int:
    return sum(kind(m).scratch_elems(cfg, m, rows, keys) for _, m in _sides(a)) + (rows * 18 * pad64(cfg.hidden) if a.normed else 0)


def page_planes(a: ParallelMixer) -> dict:
    return {n: v for _, m in _sides(a) for n, v in kind(m).page_planes(m).items()}


def state_shapes(a: ParallelMixer) -> dict:
    return {n: v for _, m in _sides(a) for n, v in kind(m).state_shapes(m).items()}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: ParallelMixer, w: ParallelWeights):
        self.ll, self.a, self.w = ll, a, w
        self.sides = [kind(m).Mixer(ll, li, m, sw) for m, sw in ((a.left, w.left), (a.right, w.right))]
        self.forms = [f for s in self.sides for f in s.forms]
        if a.normed and not isinstance(ll.cfg.block, SandwichBlock):
            raise ValueError(f"{ll.cfg.name}: mixers with results normed one by one need the residual with norms on both sides")

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """Both mixers over the step's rows: fp32 slices of the output projection, or the two results as sources of the boundary."""
        ll, w, a = self.ll, self.w, self.a
        part, s = ll.linear(sc, "parallel_in", w.proj, sc.get("h", m, ll.wp), m)
        if a.normed:
            return self._apart(sc, m, rows, block_table, kv, plan, part, s), 0
        out = sc.get("parallel_out", m, w.o.shape[1])
        col = at = 0
        for mixer, mult in zip(self.sides, (a.left_scale, a.right_scale)):
            mixer.core(sc, m, rows, block_table, kv, plan, part, s, col, out[:, at:], mult)
            col, at = col + mixer.cols, at + mixer.out_cols
        return ll.linear(sc, "o", w.o, out, m)

    def _apart(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan], part, s: int) -> list:
        ll, w, a, wp = self.ll, self.w, self.a, self.ll.wp
        left, right = self.sides
        if w.outs is None:
            x = sc.get("parallel_planes", 2 * m, left.out_cols, mult=2).view(2, m, left.out_cols)
            outs = [x[0], x[1]]
        else:
            outs = [sc.get(f"parallel_{side}", m, mixer.out_cols) for side, mixer in (("left", left), ("right", right))]
        left.core(sc, m, rows, block_table, kv, plan, part, s, 0, outs[0])
        right.core(sc, m, rows, block_table, kv, plan, part, s, left.cols, outs[1])
        if w.outs is None:
            y, n = ll.linear_planes(sc, "parallel_o", w.o, x, wp, m)
            results = [(y.view(-1)[i * wp:], n, 2 * wp) for i in range(2)]
        else:
            results = []
            for side, o, x in zip(("left", "right"), w.outs, outs):
                y, n = ll.linear(sc, f"o_{side}", o, x, m)
                results.append((y, n, wp))
        return [S.source(y, row, slices=n, slice_elems=m * row, factor=f, norm=g)
                for (y, n, row), f, g in zip(results, (a.left_scale, a.right_scale), w.norms)]
