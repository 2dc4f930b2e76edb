"""Residual of several streams (hyper-connections) around pre-normed sublayers: the layer loop of models with a
``StreamBlock``.

One kernel per sublayer boundary adds a sublayer's result to the streams and makes what the next sublayer reads (norm, token
shift); the first one starts the streams from the embedding, the last one makes the head's input.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import streams as S
from .config import DenseFfn, LayerSpec, ModelConfig
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows
from .weights import StreamWeights


def _sublayers(spec: LayerSpec):
    return (1,) if spec.ffn is None else (1, 2)


def shapes(cfg: ModelConfig, p: str, spec: LayerSpec) -> dict:
    b, out = cfg.block, {}
    for q in _sublayers(spec):
        out.update({f"{p}hc{q}.in": (b.streams,), f"{p}hc{q}.out": (b.streams,), f"{p}hc{q}.mix": (b.streams, b.streams)})
        if b.scale:
            out[f"{p}ls{q}"] = (cfg.hidden,)
    if b.shift:
        out[p + "shift"] = (cfg.hidden,)
    return out


def assemble(t, p: str, spec: LayerSpec) -> StreamWeights:
    """``t``: ``listed.Assembler``."""
    b, subs = t.cfg.block, _sublayers(spec)
    return StreamWeights([t.vec(f"{p}hc{q}.in") for q in subs], [t.vec(f"{p}hc{q}.out") for q in subs],
                         [t.vec(f"{p}hc{q}.mix") for q in subs], [t.vec(f"{p}ls{q}", t.wp) if b.scale else None for q in subs],
                         t.vec(p + "shift", t.wp) if b.shift else None)


def plain_value(cfg: ModelConfig, name: str, shape: tuple) -> Optional[torch.Tensor]:
    """Random-init models: streams that keep themselves and share what is read and written evenly; half a token shift."""
    last = name.rsplit(".", 1)[-1]
    if cfg.block is None:
        return None
    if ".hc" in name:
        s = cfg.block.streams
        return torch.eye(s) if last == "mix" else torch.full(shape, 1.0 / s if last == "in" else 1.0)
    if last == "shift":
        return torch.full(shape, 0.5)
    return torch.zeros(shape) if last == "b" else None


class StreamWalk:
    def __init__(self, ll: ListedLayers):
        self.ll, self.cfg = ll, ll.cfg
        b, width = ll.cfg.block, ll.cfg.hidden
        if any(s.ffn is not None and not isinstance(s.ffn, DenseFfn) for s in ll.cfg.layer_specs):
            raise ValueError(f"{ll.cfg.name}: residual streams take dense feed-forwards")
        self.freq = None
        if b.sinusoid:
            self.freq = torch.tensor([b.sinusoid ** (-2.0 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64,
                                     device=ll.device)

    def run(self, m: int, rows: StepRows, block_table, kv, sc: ListedScratch, flag, plan: Optional[BatchPlan] = None) -> torch.Tensor:
        """All layers for ``m`` rows; returns the head's input of every row."""
        ll, cfg, b = self.ll, self.cfg, self.cfg.block
        x = [sc.get(f"streams{i}", m, b.streams * ll.wp, torch.float32) for i in range(2)]
        h = sc.get("h", m, ll.wp)
        shift = kv.states.get("shift")
        layers = ll.w.layers
        last = len(layers) - 1
        common = dict(m=m, streams=b.streams, width=cfg.hidden, req=rows.req, pos=rows.pos, eps=cfg.rms_eps,
                      next_h=kv.shift_next)

        def reads(li: int, ffn: bool) -> dict:
            """What the sublayer after the boundary reads: layer ``li``'s feed-forward or mixer, or the head."""
            if li > last:
                return dict(norm=ll.w.final_norm, h=sc.get("head_rows", m, ll.wp), x_out=None)
            lw = layers[li]
            out = dict(w_in=lw.streams.w_in[ffn], norm=lw.post_norm if ffn else lw.input_norm, h=h)
            if b.shift and not ffn:
                out.update(mu=lw.streams.shift, prev=shift[li])
            return out

        S.embed(ll.w.embed, rows.token, self.freq, flag, x_out=x[0], **common, **reads(0, False))
        i = 0
        for li, (spec, lw) in enumerate(zip(cfg.layer_specs, layers)):
            for q in range(1 if spec.ffn is None else 2):
                y, s = ll.dense(sc, spec.ffn, lw.dense, m) if q else ll.mixers[li].run(sc, m, rows, block_table, kv, plan)
                after = reads(li, True) if not q and spec.ffn is not None else reads(li + 1, False)
                S.boundary(y, s, lw.streams, q, b.mult, x_in=x[i], **{"x_out": x[i ^ 1], **common, **after},
                           commit=shift[li] if b.shift and not q else None)
                i ^= 1
        return sc.get("head_rows", m, ll.wp)
