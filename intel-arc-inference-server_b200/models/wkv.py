"""Time-mixing mixers (wkv): five inputs, each its own mix of the token's row and the one before (made by the residual's
boundary kernel), one fp32 matrix per head, sequence and layer.  The recurrence shares its kernels with ``channel_delta``."""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import channel_rec as R
from ..ops import gemm as G
from ..ops import latent as L
from .channel_delta import block_elems, pad_key, scan_rows, second_half
from .config import ModelConfig, Wkv
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, pad64
from .weights import WkvWeights

INPUTS = "rkvgw"


@dataclass(frozen=True)
class WkvGeometry:
    """Kernel sizes; the projection's rows are r | k | v | gate (``heads * d`` each) | first half of the decay."""
    heads: int
    d: int
    kp: int
    n: int

    @staticmethod
    def of(a: Wkv) -> "WkvGeometry":
        d = pad_key(a.dim)
        return WkvGeometry(a.heads, d, pad64(max(a.w_rank, 1)), 4 * a.heads * d + pad64(max(a.w_rank, 1)))

    @property
    def hd(self) -> int:
        return self.heads * self.d

    @property
    def act(self) -> int:
        return R.act_cols(self.heads, self.heads, self.d, self.d)


def shapes(cfg: ModelConfig, p: str, a: Wkv) -> dict:
    h, n = cfg.hidden, a.heads * a.dim
    return {**{p + "mu." + x: (h,) for x in INPUTS}, **{p + x: (n, h) for x in "rkvg"}, p + "w1": (a.w_rank, h), p + "w2": (n, a.w_rank),
            p + "w0": (n,), p + "u": (a.heads, a.dim), p + "norm": (n,), p + "o": (h, n)}


def tensor_sizes(p: str, a: Wkv, shape) -> Wkv:
    return dataclasses.replace(a, w_rank=shape(p + "w1")[0])


def assemble(t, p: str, a: Wkv) -> WkvWeights:
    """``t``: ``listed.Assembler``."""
    g = WkvGeometry.of(a)
    proj = t.zeros(g.n, t.wp)
    proj[: 4 * g.hd] = t.stack([t.heads(t.t(p + x), a.heads, [(a.dim, g.d)], t.wp) for x in "rkvg"])
    proj[4 * g.hd: 4 * g.hd + a.w_rank] = t.padded(t.t(p + "w1"), a.w_rank, t.wp)
    vec = lambda x: t.fp32_heads(p + x, a.heads, a.dim, g.d, 1).reshape(-1).contiguous()       # noqa: E731
    return WkvWeights(proj, torch.stack([t.vec(p + "mu." + x, t.wp) for x in INPUTS]), vec("u"), vec("w0"),
                      second_half(t, ((p + "w2", a.heads, a.dim, g.d),), g.kp), vec("norm"), t.out_proj(p + "o", a.heads, a.dim, g.d))


def weight_elems(cfg: ModelConfig, a: Wkv) -> int:
    g = WkvGeometry.of(a)
    return pad64(cfg.hidden) * (g.n + g.hd) + 2 * g.hd * g.kp


def scratch_elems(cfg: ModelConfig, a: Wkv, rows: int, keys: int) -> int:
    g = WkvGeometry.of(a)
    return rows * (5 * pad64(cfg.hidden) + 9 * g.n + g.kp + g.hd + g.act + 2 * g.hd) + block_elems(rows, a.heads, g.d, g.d)


def page_planes(a: Wkv) -> dict:
    return {}


def state_shapes(a: Wkv) -> dict:
    g = WkvGeometry.of(a)
    return {"wkv": (g.heads * g.d * g.d,)}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: Wkv, w: WkvWeights):
        self.ll, self.li, self.a, self.w, self.g = ll, li, a, w, WkvGeometry.of(a)
        if ll.cfg.block is None:
            raise ValueError(f"{ll.cfg.name}: time mixing needs the pre-normed residual, which makes its shifted inputs")
        self.forms = [("chunks",)] if ll.device.type == "cuda" else []

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """The recurrence over the step's rows: fp32 slices of its output projection."""
        ll, a, g, w = self.ll, self.a, self.g, self.w
        x = ll.shifted(sc, len(INPUTS), m).view(len(INPUTS), m, ll.wp)
        part, s = ll.linear_planes(sc, "wkv_in", w.proj, x, g.hd, m)
        lr = None
        if not ll.f32 and m > L.GEMV_ROWS:
            y, z = sc.get("lowrank", m, 2 * g.kp), sc.get("wkv_second", m, g.hd, torch.float32)
            R.lowrank_rows(part, s, m, (4 * g.hd,), (a.w_rank,), g.kp, True, y)
            G.gemm_bf16(y, w.second, z, epi=G.EPI_F32)
            lr = (z, 1)
        act = sc.get("wkv_act", m, g.act, torch.float32)
        R.wkv_prep(part, s, m, g, a, w, lr, act)
        return scan_rows(ll, sc, plan, m, rows, act, False, g.heads, g.heads, g.d, g.d, a.dim, w, kv.states[f"wkv{self.li}"][0], "wkv")
