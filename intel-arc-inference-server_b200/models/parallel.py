"""Two mixers side by side on the same input.  Their input projections are one linear, and so are their output projections:
each mixer leaves its rows, times its scale, in its own columns of what the output projection reads.

Both mixers are of kinds with a ``core`` (from columns of a projection to rows): ``grouped``, ``mingru``."""
from __future__ import annotations

from typing import Optional

import torch

from .config import ModelConfig, ParallelMixer
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, kind
from .weights import GroupedWeights, ParallelWeights


def _sides(a: ParallelMixer):
    return ("left", a.left), ("right", a.right)


def shapes(cfg: ModelConfig, p: str, a: ParallelMixer) -> dict:
    out = {}
    for side, m in _sides(a):
        out.update(kind(m).shapes(cfg, f"{p}{side}.", m))
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
    return ParallelWeights(torch.cat(projs), torch.cat(outs, dim=1).contiguous(), *parts)


def weight_elems(cfg: ModelConfig, a: ParallelMixer) -> int:
    return sum(kind(m).weight_elems(cfg, m) for _, m in _sides(a))


def scratch_elems(cfg: ModelConfig, a: ParallelMixer, rows: int, keys: int) -> int:
    return sum(kind(m).scratch_elems(cfg, m, rows, keys) for _, m in _sides(a))


def page_planes(a: ParallelMixer) -> dict:
    return {n: v for _, m in _sides(a) for n, v in kind(m).page_planes(m).items()}


def state_shapes(a: ParallelMixer) -> dict:
    return {n: v for _, m in _sides(a) for n, v in kind(m).state_shapes(m).items()}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: ParallelMixer, w: ParallelWeights):
        self.ll, self.a, self.w = ll, a, w
        self.sides = [kind(m).Mixer(ll, li, m, sw) for m, sw in ((a.left, w.left), (a.right, w.right))]
        self.forms = [f for s in self.sides for f in s.forms]

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """Both mixers over the step's rows: fp32 slices of the output projection."""
        ll, w, a = self.ll, self.w, self.a
        part, s = ll.linear(sc, "parallel_in", w.proj, sc.get("h", m, ll.wp), m)
        out = sc.get("parallel_out", m, w.o.shape[1])
        col = at = 0
        for mixer, mult in zip(self.sides, (a.left_scale, a.right_scale)):
            mixer.core(sc, m, rows, block_table, kv, plan, part, s, col, out[:, at:], mult)
            col, at = col + mixer.cols, at + mixer.out_cols
        return ll.linear(sc, "o", w.o, out, m)
