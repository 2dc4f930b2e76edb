"""Delta-rule mixers with one decay per head and key channel: one fp32 matrix per head, sequence and layer, and the last inputs
of the short convolutions.

Everything that enters the recurrence is prepared for all rows at once (``ops/csrc/channel_rec.cu``); the recurrence walks the
rows of a sequence in order with the state in registers.  The second halves of the low-rank projections (decays, output gate)
are taken inside the preparation for a few rows, by GEMMs over two bf16 limbs for more.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import channel_rec as R
from ..ops import gemm as G
from ..ops import latent as L
from .config import ChannelDelta, ModelConfig
from .listed import BatchPlan, ListedLayers, ListedScratch, StepRows, pad64
from .weights import DeltaWeights


def pad_key(n: int) -> int:
    """Key dims of a recurrent head in the kernels."""
    return pad64(n) if n <= 256 else 384 if n <= 384 else 512


@dataclass(frozen=True)
class DeltaGeometry:
    """Kernel sizes; the projection's rows are q | k | v | step sizes | first halves of decay and gate."""
    heads: int
    kv_heads: int
    dk: int
    dv: int
    taps: int
    kp: int                       # columns of the low-rank rows
    n: int                        # rows of the projection
    a_rank: int

    @staticmethod
    def of(a: ChannelDelta) -> "DeltaGeometry":
        dk, dv = pad_key(a.dim), pad64(a.vdim)
        n = 2 * a.kv_heads * dk + a.heads * dv + a.heads + a.a_rank + a.g_rank
        return DeltaGeometry(a.heads, a.kv_heads, dk, dv, 4 if a.conv <= 4 else 8 if a.conv <= 8 else 16,
                             pad64(max(a.a_rank, a.g_rank, 1)), pad64(n), a.a_rank)

    @property
    def channels(self) -> int:
        """Columns that go through the convolution."""
        return 2 * self.kv_heads * self.dk + self.heads * self.dv

    @property
    def col_b(self) -> int:
        return self.channels

    @property
    def col_a1(self) -> int:
        return self.channels + self.heads

    @property
    def col_g1(self) -> int:
        return self.col_a1 + self.a_rank

    @property
    def second(self) -> int:
        return self.heads * (self.dk + self.dv)

    @property
    def act(self) -> int:
        return R.act_cols(self.kv_heads, self.heads, self.dk, self.dv)


def shapes(cfg: ModelConfig, p: str, a: ChannelDelta) -> dict:
    h, qk, v = cfg.hidden, a.kv_heads * a.dim, a.heads * a.vdim
    return {p + "q": (qk, h), p + "q.conv": (qk, a.conv), p + "k": (qk, h), p + "k.conv": (qk, a.conv), p + "v": (v, h),
            p + "v.conv": (v, a.conv), p + "b": (a.heads, h), p + "A_log": (a.heads,), p + "norm": (a.vdim,), p + "a1": (a.a_rank, h),
            p + "a2": (a.heads * a.dim, a.a_rank), p + "dt_bias": (a.heads * a.dim,), p + "g1": (a.g_rank, h), p + "g2": (v, a.g_rank),
            p + "o": (h, v)}


def tensor_sizes(p: str, a: ChannelDelta, shape) -> ChannelDelta:
    return dataclasses.replace(a, a_rank=shape(p + "a1")[0], g_rank=shape(p + "g1")[0])


def second_half(t, parts, kp: int) -> torch.Tensor:
    """Second halves of low-rank projections one below the other; in bf16 twice side by side, for activations in two limbs."""
    w = t.stack([t.heads(t.t(name), heads, [(size, pad)], kp) for name, heads, size, pad in parts])
    return w if t.dtype == torch.float32 else torch.cat([w, w], dim=1).contiguous()


def assemble(t, p: str, a: ChannelDelta) -> DeltaWeights:
    """``t``: ``listed.Assembler``."""
    g = DeltaGeometry.of(a)
    sides = (("q", a.kv_heads, a.dim, g.dk), ("k", a.kv_heads, a.dim, g.dk), ("v", a.heads, a.vdim, g.dv))
    proj = t.zeros(g.n, t.wp)
    rows = t.stack([t.heads(t.t(p + x), n, [(size, pad)], t.wp) for x, n, size, pad in sides]
                   + [t.padded(t.t(p + x), n, t.wp) for x, n in (("b", a.heads), ("a1", a.a_rank), ("g1", a.g_rank))])
    proj[: len(rows)] = rows
    conv = torch.zeros(g.taps, g.channels, dtype=torch.float32, device=t.device)      # shorter ones: zeros at the old end
    conv[g.taps - a.conv:] = torch.cat([t.fp32_heads(p + x + ".conv", n, size, pad, a.conv) for x, n, size, pad in sides]).T
    norm = torch.zeros(a.heads, g.dv, dtype=torch.float32, device=t.device)
    norm[:, : a.vdim] = t.vec(p + "norm")
    return DeltaWeights(proj, conv.contiguous(), torch.exp(t.vec(p + "A_log")),
                        t.fp32_heads(p + "dt_bias", a.heads, a.dim, g.dk, 1).reshape(-1).contiguous(),
                        second_half(t, ((p + "a2", a.heads, a.dim, g.dk), (p + "g2", a.heads, a.vdim, g.dv)), g.kp), norm.view(-1),
                        t.out_proj(p + "o", a.heads, a.vdim, g.dv))


def weight_elems(cfg: ModelConfig, a: ChannelDelta) -> int:
    g = DeltaGeometry.of(a)
    return pad64(cfg.hidden) * (g.n + a.heads * g.dv) + 2 * g.second * g.kp + 2 * g.taps * g.channels


def scratch_elems(cfg: ModelConfig, a: ChannelDelta, rows: int, keys: int) -> int:
    g = DeltaGeometry.of(a)
    return rows * (9 * g.n + 2 * g.kp + g.second + g.act + 2 * g.heads * g.dv) + max(rows, 64) * (g.taps - 1) * g.channels \
        + block_elems(rows, a.heads, g.dk, g.dv)


def block_elems(rows: int, heads: int, dk: int, dv: int) -> int:
    """32-bit words of the tensor-core form's workspace (at least 32 rows per segment: twice the rows' chunks at most)."""
    return 0 if dk > 256 else (2 * rows // 16 + 4) * heads * (6 * 16 * (dk + 8) // 2 + dk + 384 + 20 * dv)


def page_planes(a: ChannelDelta) -> dict:
    return {}


def state_shapes(a: ChannelDelta) -> dict:
    g = DeltaGeometry.of(a)
    return {"delta": (g.heads * g.dk * g.dv,), "conv": (g.taps - 1, g.channels)}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: ChannelDelta, w: DeltaWeights):
        self.ll, self.li, self.a, self.w, self.g = ll, li, a, w, DeltaGeometry.of(a)
        self.forms = [("chunks",)] if ll.device.type == "cuda" else []

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """The recurrence over the step's rows: fp32 slices of its output projection."""
        ll, a, g, w = self.ll, self.a, self.g, self.w
        state, conv = kv.states[f"delta{self.li}"][0], kv.states[f"conv{self.li}"][0]
        part, s = ll.linear(sc, "delta_in", w.proj, sc.get("h", m, ll.wp), m)
        lr = None
        if not ll.f32 and m > L.GEMV_ROWS:
            x = sc.get("lowrank", 2 * m, 2 * g.kp, mult=2)
            R.lowrank_rows(part, s, m, (g.col_a1, g.col_g1), (a.a_rank, a.g_rank), g.kp, False, x)
            y, n = sc.get("delta_second", m, g.second, torch.float32), g.heads * g.dk
            G.gemm_bf16(x[:m], w.second[:n], y[:, :n], epi=G.EPI_F32)
            G.gemm_bf16(x[m:], w.second[n:], y[:, n:], epi=G.EPI_F32)
            lr = (y, 1)
        act = sc.get("delta_act", m, g.act, torch.float32)
        nxt = sc.get("conv_next", conv.shape[0], conv[0].numel(), torch.float32)
        R.delta_prep(part, s, m, g, a, w, rows.req, rows.pos, conv, nxt, lr, act)
        return scan_rows(ll, sc, plan, m, rows, act, True, g.kv_heads, g.heads, g.dk, g.dv, a.vdim, w, state, "delta", nxt, conv)


def scan_rows(ll, sc, plan, m: int, rows: StepRows, act, delta: bool, hq: int, h: int, dk: int, dv: int, vdim: int, w, state, name: str,
              conv_next=None, conv_state=None):
    """The recurrence over prepared rows, rows one by one and prompt segments, and its output projection."""
    n1 = m if plan is None else plan.n_single
    out = sc.get(name + "_out", m, h * dv)
    raw = sc.get(name + "_raw", m, h * dv, torch.float32) if n1 < m or not R.fused(dk, dv) else None
    sizes = (hq, h, dk, dv, vdim)
    if n1:
        R.scan(act, delta, n1, *sizes, rows.req, rows.pos, None, state, w.norm, ll.cfg.rms_eps, raw, out, conv_next, conv_state)
    if n1 < m:
        t, block = plan.tables[("chunks",)], 0 if ll.f32 else R.block_bytes(delta, dk, dv)
        ws = sc.get("channel_blocks", 4 * t.chunks * h, block, torch.uint8).view(-1) if block else None
        R.scan(act[n1:], delta, m - n1, *sizes, rows.req[n1:], rows.pos[n1:], t, state, w.norm, ll.cfg.rms_eps, raw[n1:], out[n1:],
               conv_next, conv_state, ws)
    return ll.linear(sc, "o", w.o, out, m)
