"""Residual with a norm on both sides of every sublayer: the layer loop of models with a ``SandwichBlock``.

One kernel per sublayer boundary folds what a sublayer left (a linear's slices, the experts' weighted slots, or two mixers'
results, each with a norm of its own), norms it, adds it to the fp32 residual and norms that for the next sublayer; the first one
starts the residual from the embedding, the last one makes the head's input."""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import sandwich as S
from .config import DenseFfn
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows


class SandwichWalk:
    def __init__(self, ll: ListedLayers):
        self.ll, self.cfg = ll, ll.cfg
        if ll.cfg.loop is not None or ll.cfg.shift_runs:
            raise ValueError(f"{ll.cfg.name}: looped layers and shifted inputs need the pre-normed residual")

    def _fold(self, y, s: int, m: int):
        """Sources of a linear's slices, or of what a mixer with several results returned."""
        if isinstance(y, list):
            return y
        return [S.source(y, self.ll.wp, slices=s, slice_elems=m * self.ll.wp)]

    def run(self, m: int, rows: StepRows, block_table, kv, sc: ListedScratch, flag, plan: Optional[BatchPlan] = None) -> torch.Tensor:
        """All layers for ``m`` rows; returns the head's input of every row."""
        ll, cfg, b = self.ll, self.cfg, self.cfg.block
        x, h = sc.get("resid", m, ll.wp, torch.float32), sc.get("h", m, ll.wp)
        layers = ll.w.layers
        common = dict(m=m, width=cfg.hidden, groups=b.groups, eps=cfg.rms_eps)

        def reads(i: int) -> dict:
            """What the sublayer after the boundary reads: layer ``i``'s mixer, or the head."""
            if i == len(layers):
                return dict(next=ll.w.final_norm, h=sc.get("head_rows", m, ll.wp), x_out=None)
            return dict(next=layers[i].input_norm, h=h, x_out=x)
        S.boundary([S.source(ll.w.embed, ll.wp, row_of=rows.token, factor=b.scale)], post=None, x_in=None, vocab=cfg.vocab, flag=flag,
                   **common, **reads(0))
        for i, (spec, lw) in enumerate(zip(cfg.layer_specs, layers)):
            y, s = ll.mixers[i].run(sc, m, rows, block_table, kv, plan)
            after = reads(i + 1) if spec.ffn is None else dict(next=lw.post_norm, h=h, x_out=x)
            S.boundary(self._fold(y, s, m), post=lw.behind[0], x_in=x, **common, **after)
            if spec.ffn is None:
                continue
            if isinstance(spec.ffn, DenseFfn):
                src = self._fold(*ll.dense(sc, spec.ffn, lw.dense, m), m)
            else:
                src = [S.source(**ll.experts(sc, spec.ffn, lw.moe, m))]
            S.boundary(src, post=lw.behind[1], x_in=x, **common, **reads(i + 1))
        return sc.get("head_rows", m, ll.wp)
