"""Grouped-query attention mixers over paged keys and values of any head size; optional rotation, distance bias (linear or
logarithmic), chunked mask, window with pooled blocks before it, sinks, biases and norms of queries, keys and values, query
temperature, rotated values, values that are the keys, gated results, and layers that read another layer's keys and values.

Rows of a step are attended one by one (split-KV kernel) or, for long segments of a prompt, in query tiles by the tcgen05
prompt attention straight over the pages.  The projection of a prompt stays in the GEMM's bf16 rows: the prompt attention
reads its queries there.  With biases, norms or rotations the projection is fp32 instead, and a kernel of its own makes query
rows and fills the pages (``core``, which also serves a mixer beside another one).

Pooled blocks are planes of the page pool: a block lies in the page of its last position, so what a page holds depends on the
positions up to its end alone.  The step that brings a block's last position writes it.
"""
from __future__ import annotations

import dataclasses
import math
from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import gemm as G
from ..ops import latent as L
from ..ops import paged as P
from .config import GroupedAttention, ModelConfig, Rotary
from .listed import SMS, BatchPlan, ListedLayers, ListedScratch, StepRows, pad64, pair_order
from .weights import GroupedWeights

LOG2E = math.log2(math.e)


@dataclass(frozen=True)
class GroupedGeometry:
    """Kernel sizes: ``dk`` / ``dv`` columns of a key / value head."""
    heads: int
    kv_heads: int
    dk: int
    dv: int

    @staticmethod
    def of(a: GroupedAttention) -> "GroupedGeometry":
        return GroupedGeometry(a.heads, a.kv_heads, pad64(a.dim), pad64(a.vdim))

    @property
    def nq(self) -> int:
        return self.heads * self.dk

    @property
    def groups(self) -> int:
        """CTAs per row and split of the row attention: 16 query heads of one key/value head each."""
        return self.kv_heads * ((self.heads // self.kv_heads + 15) // 16)

    @property
    def nkv(self) -> int:
        return self.kv_heads * (self.dk + self.dv)


def shapes(cfg: ModelConfig, p: str, a: GroupedAttention) -> dict:
    h = cfg.hidden
    out = {p + "q": (a.heads * a.dim, h), p + "o": (h, a.heads * a.vdim)}
    if a.kv_from < 0:
        out[p + "k"] = (a.kv_heads * a.dim, h)
        if not a.tied:
            out[p + "v"] = (a.kv_heads * a.vdim, h)
    if a.gate:
        out[p + "g"] = (a.heads * a.vdim, h)
    if a.sink:
        out[p + "sink"] = (a.heads,)
    if a.qkv_bias:
        out.update({p + n + ".b": (h * d,) for n, h, d in (("q", a.heads, a.dim), ("k", a.kv_heads, a.dim), ("v", a.kv_heads, a.vdim))})
    if a.qk_norm:
        out.update({p + "q.norm": (a.dim,), p + "k.norm": (a.dim,)})
    if a.log_bias:
        out.update({p + "r1": (a.heads,), p + "r2": (a.heads,)})
    return out


def assemble(t, p: str, a: GroupedAttention) -> GroupedWeights:
    """``t``: ``listed.Assembler``."""
    g = GroupedGeometry.of(a)
    order = pair_order(a.rot.dims, a.dim) if a.rot is not None else None
    v_order = order if a.tied else pair_order(a.vdim, a.vdim) if a.rot_values else None
    parts = [t.heads(t.t(p + "q"), a.heads, [(a.dim, g.dk)], t.wp, order)]
    if a.kv_from < 0:
        parts.append(t.heads(t.t(p + "k"), a.kv_heads, [(a.dim, g.dk)], t.wp, order))
        if not a.tied:
            parts.append(t.heads(t.t(p + "v"), a.kv_heads, [(a.vdim, g.dv)], t.wp, v_order))
    if a.gate:
        parts.append(t.heads(t.t(p + "g"), a.heads, [(a.vdim, g.dv)], t.wp, v_order))
    slope2 = None
    if a.bias:
        slope2 = torch.tensor([2.0 ** (-a.bias * (h + 1) / a.heads) * LOG2E for h in range(a.heads)], dtype=torch.float32, device=t.device)
    sink2 = t.vec(p + "sink") * LOG2E if a.sink else None
    w = GroupedWeights(torch.cat(parts), t.out_proj(p + "o", a.heads, a.vdim, g.dv, v_order), slope2, sink2)
    if a.qkv_bias:
        w.bias = torch.cat([t.fp32_heads(p + n + ".b", h, d, pad, 1).reshape(-1) for n, h, d, pad in (
            ("q", a.heads, a.dim, g.dk), ("k", a.kv_heads, a.dim, g.dk), ("v", a.kv_heads, a.vdim, g.dv))])
    if a.qk_norm:
        w.q_norm, w.k_norm = (t.vec(p + n + ".norm", g.dk) for n in "qk")
        if order is not None:
            w.q_norm, w.k_norm = (torch.cat([x[: a.dim][order], x[a.dim:]]) for x in (w.q_norm, w.k_norm))
    if a.log_bias:
        w.r1, w.r2 = t.vec(p + "r1"), t.vec(p + "r2")
    return w


def weight_elems(cfg: ModelConfig, a: GroupedAttention) -> int:
    g = GroupedGeometry.of(a)
    return pad64(cfg.hidden) * (proj_cols(g, a) + g.heads * g.dv)


def proj_cols(g: GroupedGeometry, a: GroupedAttention) -> int:
    """Columns of the input projection: q | k | v | gate, those that there are."""
    return gate_col(g, a) + (g.heads * g.dv if a.gate else 0)


def gate_col(g: GroupedGeometry, a: GroupedAttention) -> int:
    return g.nq + (g.kv_heads * (g.dk + (0 if a.tied else g.dv)) if a.kv_from < 0 else 0)


def scratch_elems(cfg: ModelConfig, a: GroupedAttention, rows: int, keys: int) -> int:
    g = GroupedGeometry.of(a)
    return rows * (9 * max(proj_cols(g, a), g.nq + g.nkv) + g.nq + (3 if a.gate else 2) * g.heads * g.dv)  \
        + max(rows, Mixer.partials(g)) * (g.dv + 2) + (keys // a.pool * g.nkv if a.pool else 0)


def page_planes(a: GroupedAttention) -> dict:
    """Plane name -> (heads, columns), or (heads, columns, rows per page) where a page does not hold a row per position."""
    g = GroupedGeometry.of(a)
    out = {} if a.kv_from >= 0 else {"k": (g.kv_heads, g.dk), "v": (g.kv_heads, g.dv)}
    if a.pool:
        out.update(pk=(g.kv_heads, g.dk, a.pool_slots), pv=(g.kv_heads, g.dv, a.pool_slots))
    return out


def state_shapes(a: GroupedAttention) -> dict:
    return {}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: GroupedAttention, w: GroupedWeights):
        self.ll, self.li, self.a, self.w, self.g = ll, li, a, w, GroupedGeometry.of(a)
        self.src = li if a.kv_from < 0 else a.kv_from
        on_gpu = ll.device.type == "cuda" and not ll.f32
        self.tile_rows = P.segments_per_tile(self.g) if on_gpu else 0
        self.rows_form = on_gpu and P.rows_ok(self.g)
        form = ("pooled", a.window, a.pool, self.tile_rows) if a.window else ("tiles", a.chunk, self.tile_rows)
        self.forms = [form] if self.tile_rows else []
        self.rot = ll.rotation(a.rot) if a.rot is not None else None
        self.vrot = ll.rotation(Rotary(a.vdim, a.rot.base)) if a.rot_values else None
        self.plain = a.rot is None and not a.gate and not a.tied and not a.window          # nothing of ``ops.paged.Extra``
        self.normed = a.qkv_bias or a.qk_norm or a.v_norm or a.temp != 0.0 or not self.plain
        if self.normed and a.kv_from >= 0:
            raise ValueError("layers on another layer's keys have neither biases, norms nor rotations of their own")
        if a.window and (a.chunk or a.bias or a.log_bias):
            raise ValueError("a window has neither chunks nor a distance bias beside it")
        self.cols = proj_cols(self.g, a)        # columns of its projection, and of its rows
        self.out_cols = self.g.heads * self.g.dv
        self.logb = (w.r1, w.r2) if a.log_bias else None

    def nsplit(self, m: int) -> int:
        """KV splits of the row attention: about two CTAs per SM, at least two pages per warp of a split."""
        a = self.a
        keys = min(a.chunk or a.window or self.ll.max_pos, self.ll.max_pos)
        if a.pool:
            keys += (self.ll.max_pos - keys) // a.pool
        return max(1, min(64, 2 * SMS // (m * self.g.groups), keys // 128))

    @staticmethod
    def partials(g: GroupedGeometry) -> int:
        """Most (row, head, split) partials a call with several splits leaves."""
        return (2 * SMS // g.groups + 1) * g.heads

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """Attention of the step's rows: fp32 slices of its output projection."""
        ll, g, w = self.ll, self.g, self.w
        own = self.a.kv_from < 0
        k, v = kv.pages[f"k{self.src}"], kv.pages[f"v{self.src}"]
        h = sc.get("h", m, ll.wp)
        out = sc.get("attn", m, g.heads * g.dv)
        if self.normed:
            part, s = ll.linear(sc, "qkv", w.qkv, h, m)
            self.core(sc, m, rows, block_table, kv, plan, part, s, 0, out)
            return ll.linear(sc, "o", w.o, out, m)
        if ll.f32 or m <= L.GEMV_ROWS:
            part, s = ll.linear(sc, "qkv", w.qkv, h, m)
            q = sc.get("q_rows", m, g.nq)
            P.append(part, s, m, g, own, rows.req, rows.pos, block_table, q, k, v)
        else:
            q = sc.get("qkv_rows", m, w.qkv.shape[0])
            G.gemm_bf16(h, w.qkv, q)
            if own:
                P.append_rows(q, m, g, rows.req, rows.pos, block_table, k, v)
        self.attend(sc, m, rows, block_table, plan, q, k, v, out)
        return ll.linear(sc, "o", w.o, out, m)

    def core(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan], part, s: int, col: int, out,
             mult: float = 1.0):
        """From its columns of the projection's fp32 slices, which come first, to its rows ``out``, times ``mult``."""
        if col:
            raise ValueError("the columns of an attention mixer come first")
        a, g, k, v = self.a, self.g, kv.pages[f"k{self.li}"], kv.pages[f"v{self.li}"]
        q, extra = sc.get("q_rows", m, g.nq), None
        if not self.plain:
            gate = sc.get("attn_gate", m, g.heads * g.dv) if a.gate else None
            extra = P.Extra(self.rot, self.vrot, a.tied, gate, gate_col(g, a), a.window, a.pool, kv.pages.get(f"pk{self.li}"),
                            kv.pages.get(f"pv{self.li}"))
        P.norm(part, s, m, g, a, self.w, self.ll.cfg.rms_eps, rows.req, rows.pos, block_table, q, k, v, extra)
        self.attend(sc, m, rows, block_table, plan, q, k, v, out, mult, extra)

    def attend(self, sc: ListedScratch, m: int, rows: StepRows, block_table, plan: Optional[BatchPlan], q, k, v, out, mult: float = 1.0,
               extra: Optional[P.Extra] = None):
        """Attention of query rows ``q`` over the pages, which hold the step's keys and values already."""
        a, g, w = self.a, self.g, self.w
        more = dict(logb=self.logb, mult=mult, extra=extra)
        n1 = m if plan is None or not self.tile_rows else plan.n_single
        if n1 and self.rows_form:
            ns, cap = self.nsplit(n1), self.partials(g)
            op = sc.get(f"o_part{cap}", cap, g.dv, torch.float32) if ns > 1 else None      # layers of other heads have their own
            ml = sc.get(f"ml_part{cap}", cap, 2, torch.float32) if ns > 1 else None
            P.rows(q, k, v, n1, g, rows.req, rows.pos, block_table, ns, a.chunk, a.scale, w.slope2, w.sink2, op, ml, out, **more)
        elif n1:
            P.simple(q, k, v, n1, g, rows.req, rows.pos, block_table, a.chunk, a.scale, w.slope2, w.sink2, out, **more)
        if n1 < m:
            t = plan.tables[self.forms[0]]
            if extra is not None:
                if extra.gate is not None:
                    more["extra"] = dataclasses.replace(extra, gate=extra.gate[n1:])
                if a.pool and t.n_pool:
                    pk, pv = sc.get("pool_k", t.n_pool, g.kv_heads * g.dk), sc.get("pool_v", t.n_pool, g.kv_heads * g.dv)
                    P.pool_gather(t.preq, t.block, t.n_pool, g, block_table, a.pool, extra.pk, extra.pv, pk, pv)
                    more["pooled"] = (pk, pv, t.first)
            P.attn_segments(q[n1:], k, v, block_table, out[n1:], t.tiles, t.n_tiles, m - n1, g, a.scale, a.chunk, w.slope2, w.sink2, **more)
