"""Latent-attention mixers: queries and keys / values go through low-rank latents; the cache holds the key-value latent and
one rotated key part shared by the heads.

Attention has two forms with the same cache: decode rows work against the key-value latent itself (W_uk moved to the query,
W_uv behind the softmax); long segments of a prompt expand keys and values of their window by GEMMs and run the tcgen05
prompt attention.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import gemm as G
from ..ops import latent as L
from .config import LatentAttention, ModelConfig
from .listed import SMS, BatchPlan, ListedLayers, ListedScratch, StepRows, pad64
from .oracle import rope_tables
from .weights import LatentWeights


@dataclass(frozen=True)
class LatentGeometry:
    """Kernel sizes of a mixer: ``dn`` / ``rp`` / ``dv`` columns of a head's unrotated, rotated and value part, ``qp`` /
    ``kvp`` columns of the latents; a cache row is ``kvp + rp`` elements."""
    heads: int
    q_rank: int
    qp: int
    kv_rank: int
    kvp: int
    rot: int
    rp: int
    dn: int
    dv: int
    rope_dims: int

    @staticmethod
    def of(a: LatentAttention) -> "LatentGeometry":
        dv = pad64(a.vdim)
        return LatentGeometry(a.heads, a.q_rank, pad64(a.q_rank), a.kv_rank, pad64(a.kv_rank), a.rot_dim,
                              max(64, pad64(a.rot_dim)), pad64(a.dim), 256 if dv == 192 else dv, a.rope_dims)

    @property
    def lc(self) -> int:
        return self.kvp + self.rp

    @property
    def n_down(self) -> int:
        return self.qp + self.kvp + self.rp

    @property
    def dk(self) -> int:
        return self.dn + self.rp


# ------------------------------------------------------------------ weights and sizes
def shapes(cfg: ModelConfig, p: str, a: LatentAttention) -> dict:
    h = cfg.hidden
    return {p + "dq": (a.q_rank, h), p + "dq.norm": (a.q_rank,), p + "uq": (a.heads * (a.dim + a.rot_dim), a.q_rank),
            p + "dkv": (a.kv_rank + a.rot_dim, h), p + "dkv.norm": (a.kv_rank,), p + "uk": (a.heads * a.dim, a.kv_rank),
            p + "uv": (a.heads * a.vdim, a.kv_rank), p + "o": (h, a.heads * a.vdim)}


def assemble(t, p: str, a: LatentAttention) -> LatentWeights:
    """``t``: ``listed.Assembler``."""
    g, h = LatentGeometry.of(a), t.cfg.hidden
    down, dkv = t.zeros(g.n_down, t.wp), t.t(p + "dkv")
    down[: a.q_rank, :h] = t.t(p + "dq")
    down[g.qp: g.qp + a.kv_rank, :h] = dkv[: a.kv_rank]
    down[g.qp + g.kvp: g.qp + g.kvp + a.rot_dim, :h] = dkv[a.kv_rank:]
    return LatentWeights(down, t.vec(p + "dq.norm"), t.vec(p + "dkv.norm"),
                         t.heads(t.t(p + "uq"), a.heads, [(a.dim, g.dn), (a.rot_dim, g.rp)], g.qp),
                         t.heads(t.t(p + "uk"), a.heads, [(a.dim, g.dn)], g.kvp),
                         t.heads(t.t(p + "uv"), a.heads, [(a.vdim, g.dv)], g.kvp), t.out_proj(p + "o", a.heads, a.vdim, g.dv))


def weight_elems(cfg: ModelConfig, a: LatentAttention) -> int:
    g, wp = LatentGeometry.of(a), pad64(cfg.hidden)
    return g.n_down * wp + g.heads * (g.dk * g.qp + (g.dn + g.dv) * g.kvp + wp * g.dv)


def scratch_elems(cfg: ModelConfig, a: LatentAttention, rows: int, keys: int) -> int:
    g = LatentGeometry.of(a)
    return rows * (9 * (g.n_down + g.heads * g.dk) + g.heads * (g.lc + 2 * g.dv)) + max(rows, SMS) * g.heads * (g.kvp + 2) \
        + keys * (g.lc + g.heads * (g.dn + g.dv)) + rows * g.heads * g.dk


def page_planes(a: LatentAttention) -> dict:
    """Per position: plane name -> (heads, columns); 0 heads: rows shared by the heads."""
    return {"latent": (0, LatentGeometry.of(a).lc)}


def state_shapes(a: LatentAttention) -> dict:
    return {}


class Mixer:
    def __init__(self, ll: ListedLayers, li: int, a: LatentAttention, w: LatentWeights):
        self.ll, self.li, self.a, self.w, self.g = ll, li, a, w, LatentGeometry.of(a)
        key = ("rope", a.rope_dims, a.rope_base)
        if key not in ll.shared:
            c, sn = rope_tables(a.rope_dims, a.rope_base, ll.max_pos)
            ll.shared[key] = (c.to(ll.device).contiguous(), sn.to(ll.device).contiguous())
        self.rope = ll.shared[key]
        on_gpu = ll.device.type == "cuda" and not ll.f32
        self.tile_rows = L.prefill_rows_per_tile(self.g) if on_gpu else 0     # query rows per tile of the prompt attention
        self.rows_form = on_gpu and L.rows_ok(self.g)
        self.forms = [("keys", a.window, self.tile_rows)] if self.tile_rows else []

    def nsplit(self, m: int) -> int:
        """KV splits of the decode attention: about one CTA per SM, at least one key tile per split."""
        if not self.rows_form:
            return 1
        a = self.a
        keys = min(a.window, self.ll.max_pos) if a.window else self.ll.max_pos
        groups = (a.heads + 31) // 32 if a.heads > 16 else 1
        return max(1, min(64, SMS // (m * groups), (keys + 63) // 64))

    def run(self, sc: ListedScratch, m: int, rows: StepRows, block_table, kv, plan: Optional[BatchPlan]):
        """Latent attention of the step's rows: fp32 slices of its output projection."""
        ll, a, g, w, cache = self.ll, self.a, self.g, self.w, kv.pages[f"latent{self.li}"]
        h = sc.get("h", m, ll.wp)
        part, s = ll.linear(sc, "down", w.down, h, m)
        cq = sc.get("cq", m, g.qp)
        rope = self.rope
        L.prep(part, s, m, g, w.q_norm, w.kv_norm, ll.cfg.rms_eps, rows.req, rows.pos, block_table, rope, cq, cache)
        out = sc.get("attn", m, g.heads * g.dv)
        n1 = m if plan is None or not self.tile_rows else plan.n_single
        if n1:
            q, s = ll.linear(sc, "q", w.uq, cq, n1)
            ql = sc.get("ql", n1, g.heads * g.lc)
            L.absorb(q, s, n1, g, w.uk, rows.pos, rope, ql)
            ns = self.nsplit(n1)
            cap = max(n1 * ns, SMS) if sc.fixed else n1 * ns
            op = sc.get("o_part", cap, g.heads * g.kvp, torch.float32)
            ml = sc.get("ml_part", cap, g.heads * 2, torch.float32)
            if self.rows_form:
                L.rows(ql, cache, n1, g, rows.req, rows.pos, block_table, op, ml, ns, a.window, a.scale)
            else:
                L.simple(ql, cache, n1, g, rows.req, rows.pos, block_table, op, ml, a.window, a.scale)
            L.merge(op, ml, n1, g, ns, w.uv, out)
        if n1 < m:
            self._prompt_attention(sc, a, g, w, cq[n1:], m - n1, rows.pos[n1:], block_table, cache,
                                   plan.tables[self.forms[0]], rope, out[n1:])
        return ll.linear(sc, "o", w.o, out, m)

    def _prompt_attention(self, sc, a, g, w, cq, m, pos, block_table, cache, kp, rope, out):
        q = sc.get("q_prompt", m, g.heads * g.dk)
        G.gemm_bf16(cq, w.uq, q)
        L.rope_q(q, pos, m, g, rope)
        n = kp.n_keys
        c, kr = sc.get("key_c", n, g.kvp), sc.get("key_rot", n, g.rp)
        k, v = sc.get("k", n, g.heads * g.dn), sc.get("v", n, g.heads * g.dv)
        L.gather(cache, kp.kreq, kp.kpos, n, block_table, g, c, kr)
        G.gemm_bf16(c, w.uk, k)
        G.gemm_bf16(c, w.uv, v)
        L.attn_prefill_rows(q, k, kr, v, out, kp.tiles, kp.n_tiles, m, n, g, a.scale, a.window)
