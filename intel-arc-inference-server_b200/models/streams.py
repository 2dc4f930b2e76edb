"""Residual of several streams (hyper-connections), or of one, around pre-normed sublayers: the layer loop of models with a
``StreamBlock``.

One kernel per sublayer boundary adds a sublayer's result to the streams and makes what the next sublayer reads (norm, token
shift, one or several mixes with the previous token's row); the first one starts the streams from the embedding, the last one
makes the head's input.  Ahead of a pass over a looped range of layers the boundary adds the pass's vector and the embedding
row.
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
    if not b.mixing:
        return out
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
    if cfg.block.columns:      # norms, biases and mixes of models with plain residuals
        if last == "A_log":
            return torch.log(torch.linspace(1.0, 8.0, shape[0]))
        if last in ("dt_bias", "w0"):
            return torch.full(shape, -3.0)
        if last in ("norm1", "norm2", "b") and len(shape) == 1 or name == "final.norm":
            return torch.zeros(shape)
        if ".mu." in name:
            return torch.full(shape, 0.5)
        if last in ("r1", "r2"):
            return torch.full(shape, 1.0 if last == "r1" else 0.1)
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
        if not b.mixing and (b.streams != 1 or b.scale or b.shift):
            raise ValueError(f"{ll.cfg.name}: a residual without mixing is one plain stream")
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
        layers, runs = ll.w.layers, cfg.layer_runs
        shift = dict(zip(cfg.shift_runs, kv.states["shift"])) if cfg.shift_runs else {}
        common = dict(m=m, streams=b.streams, width=cfg.hidden, req=rows.req, pos=rows.pos, eps=cfg.rms_eps,
                      next_h=kv.shift_next)

        def reads(j: int, ffn: bool) -> dict:
            """What the sublayer after the boundary reads: run ``j``'s feed-forward or mixer, or the head."""
            if j == len(runs):
                return dict(norm=ll.w.final_norm, h=sc.get("head_rows", m, ll.wp), x_out=None)
            li, begins = runs[j]
            lw = layers[li]
            out = dict(w_in=lw.streams.w_in[ffn] if b.mixing else None, norm=lw.post_norm if ffn else lw.input_norm, h=h)
            if j in shift and not ffn:
                planes = getattr(cfg.layer_specs[li].mixer, "shifts", 0)
                out.update(mu=lw.mixer.shift if planes else lw.streams.shift, prev=shift[j])
                if planes:
                    out["h"] = ll.shifted(sc, planes, m)
            if begins >= 0 and not ffn:         # a pass over the looped layers starts
                out["add"] = ll.w.loop_step[begins]
                if begins:
                    out["again"] = (ll.w.embed, rows.token)
            return out

        S.embed(ll.w.embed, rows.token, self.freq, flag, x_out=x[0], **common, **reads(0, False))
        i = 0
        for j, (li, _) in enumerate(runs):
            spec, lw = cfg.layer_specs[li], layers[li]
            for q in range(1 if spec.ffn is None else 2):
                y, s = ll.dense(sc, spec.ffn, lw.dense, m) if q else ll.mixers[j].run(sc, m, rows, block_table, kv, plan)
                after = reads(j, True) if not q and spec.ffn is not None else reads(j + 1, False)
                S.boundary(y, s, lw.streams, q, b.mult, x_in=x[i], **{"x_out": x[i ^ 1], **common, **after}, freq=self.freq,
                           commit=None if q else shift.get(j), bias=lw.dense.down_bias if q else None)
                i ^= 1
        return sc.get("head_rows", m, ll.wp)
