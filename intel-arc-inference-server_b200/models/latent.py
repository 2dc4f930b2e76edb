"""Models that list their layers: latent-attention mixers, routed experts over unquantised weights, layer norms on the
sublayers' outputs, an fp32 residual stream.

This module holds the mechanisms: the padded geometry of a mixer, the assembly of weights from checkpoint tensors, the
scratch of a step, and one function per sublayer that enqueues its kernels for the rows of a step.  ``DecoderModel``
walks the layers (``listed_walk``); ``Engine`` gives it the rows of a decode step (control block, CUDA graphs) or of a
mixed batch (``runtime/batch.py``).

Kernel sizes are whole 64s: weights are padded with zeros when they are loaded (rows and columns), and padded
activation columns are zero; norms, rotations and scales use the true sizes.

Few rows (up to 16) take the weight-streaming GEMVs, more rows the tcgen05 GEMMs.  Attention has two forms with the same
cache: decode rows work against the key-value latent itself (W_uk moved to the query, W_uv behind the softmax); long
segments of a prompt expand keys and values of their window by GEMMs and run the tcgen05 prompt attention.  Models whose
weights are fp32 run everything in 32-bit (no reduced-precision product anywhere).
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

import torch

from ..ops import gemm as G
from ..ops import latent as L
from ..ops import lib as K
from ..ops import moe as M
from .config import ExpertFfn, LatentAttention, ModelConfig
from .oracle import rope_tables
from .weights import ExpertStack, LatentWeights, LayerWeights, ModelWeights, interleave16

SMS = 148
# Experts of more rows than this go through the expert-sorted grouped GEMMs, which read every chosen expert once; the
# GEMVs read one expert per (row, slot).
EXPERT_GEMV_ROWS = int(os.environ.get("B2_EXPERT_GEMV_ROWS", "4"))


def pad64(n: int) -> int:
    return (n + 63) // 64 * 64


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


# ------------------------------------------------------------------ weights
def tensor_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    """Checkpoint tensors of a listed model, by name."""
    h = cfg.hidden
    out = {"embed": (cfg.vocab, h), "final.norm": (h,), "head": (cfg.vocab, h)}
    for i, s in enumerate(cfg.layer_specs):
        p, a, f = f"l{i}.", s.mixer, s.ffn
        out.update({p + "norm1": (h,), p + "mix.dq": (a.q_rank, h), p + "mix.dq.norm": (a.q_rank,),
                    p + "mix.uq": (a.heads * (a.dim + a.rot_dim), a.q_rank), p + "mix.dkv": (a.kv_rank + a.rot_dim, h),
                    p + "mix.dkv.norm": (a.kv_rank,), p + "mix.uk": (a.heads * a.dim, a.kv_rank),
                    p + "mix.uv": (a.heads * a.vdim, a.kv_rank), p + "mix.o": (h, a.heads * a.vdim)})
        if f is not None:
            out[p + "norm2"] = (h,)
            out[p + "mlp.router"] = (f.experts, h)
            for e in range(f.experts):
                out.update({f"{p}mlp.e{e}.gate": (f.ff, h), f"{p}mlp.e{e}.up": (f.ff, h), f"{p}mlp.e{e}.down": (h, f.ff)})
    return out


def assemble(cfg: ModelConfig, get: Callable[[str], torch.Tensor], device, dtype=torch.bfloat16) -> ModelWeights:
    """Kernel-layout weights from checkpoint tensors (``get(name)``)."""
    wp = pad64(cfg.hidden)

    def t(name):
        return get(name).to(device=device, dtype=dtype)

    def vec(name):
        return get(name).float().to(device).contiguous()

    def padded(w, rows, cols):
        out = torch.zeros(rows, cols, dtype=dtype, device=device)
        out[: w.shape[0], : w.shape[1]] = w
        return out

    def heads(w, n, parts, cols):
        """Head-major rows: each head's parts (true size, padded size) in turn."""
        out = torch.zeros(n, sum(p for _, p in parts), cols, dtype=dtype, device=device)
        v = w.reshape(n, sum(s for s, _ in parts), w.shape[1])
        src = dst = 0
        for size, pad in parts:
            out[:, dst: dst + size, : w.shape[1]] = v[:, src: src + size]
            src, dst = src + size, dst + pad
        return out.reshape(-1, cols)

    layers = []
    for i, s in enumerate(cfg.layer_specs):
        p, a, f, g = f"l{i}.", s.mixer, s.ffn, LatentGeometry.of(s.mixer)
        down = torch.zeros(g.n_down, wp, dtype=dtype, device=device)
        dkv = t(p + "mix.dkv")
        down[: a.q_rank, : cfg.hidden] = t(p + "mix.dq")
        down[g.qp: g.qp + a.kv_rank, : cfg.hidden] = dkv[: a.kv_rank]
        down[g.qp + g.kvp: g.qp + g.kvp + a.rot_dim, : cfg.hidden] = dkv[a.kv_rank:]
        o = torch.zeros(wp, a.heads, g.dv, dtype=dtype, device=device)
        o[: cfg.hidden, :, : a.vdim] = t(p + "mix.o").reshape(cfg.hidden, a.heads, a.vdim)
        mix = LatentWeights(down, vec(p + "mix.dq.norm"), vec(p + "mix.dkv.norm"),
                            heads(t(p + "mix.uq"), a.heads, [(a.dim, g.dn), (a.rot_dim, g.rp)], g.qp),
                            heads(t(p + "mix.uk"), a.heads, [(a.dim, g.dn)], g.kvp),
                            heads(t(p + "mix.uv"), a.heads, [(a.vdim, g.dv)], g.kvp), o.reshape(wp, a.heads * g.dv))
        lw = LayerWeights(input_norm=vec(p + "norm1"), post_norm=vec(p + "norm2") if f is not None else None, qkv=None, o=None,
                          latent=mix)
        if f is not None:
            ffp = pad64(f.ff)
            gu = torch.zeros(f.experts, 2 * ffp, wp, dtype=dtype, device=device)
            dn = torch.zeros(f.experts, wp, ffp, dtype=dtype, device=device)
            for e in range(f.experts):
                q = f"{p}mlp.e{e}."
                gu[e] = interleave16(padded(t(q + "gate"), ffp, wp), padded(t(q + "up"), ffp, wp))
                dn[e, : cfg.hidden, : f.ff] = t(q + "down")
            lw.moe = ExpertStack(padded(t(p + "mlp.router"), (f.experts + 7) // 8 * 8, wp), gu, dn)
        layers.append(lw)
    return ModelWeights(cfg, padded(t("embed"), cfg.vocab, wp), padded(t("head"), cfg.vocab, wp), vec("final.norm"), layers)


def random_listed_weights(cfg: ModelConfig, device="cpu", seed: int = 0, std: float = 0.02,
                          dtype=torch.bfloat16) -> ModelWeights:
    shapes = tensor_shapes(cfg)
    g = torch.Generator(device=device)
    g.manual_seed(seed)

    def get(name):
        shape = shapes[name]
        if len(shape) == 1:
            return torch.ones(shape, device=device)
        return torch.empty(shape, dtype=torch.bfloat16, device=device).normal_(0, std if name == "head" else shape[1] ** -0.5, generator=g)
    return assemble(cfg, get, device, dtype)


def padded_weight_elems(cfg: ModelConfig) -> int:
    """Elements of the assembled weights (host arithmetic, the memory planner's figure)."""
    wp, n = pad64(cfg.hidden), 2 * cfg.vocab * pad64(cfg.hidden)
    for s in cfg.layer_specs:
        g, f = LatentGeometry.of(s.mixer), s.ffn
        n += g.n_down * wp + g.heads * (g.dk * g.qp + (g.dn + g.dv) * g.kvp + wp * g.dv)
        if f is not None:
            n += (f.experts + 7) // 8 * 8 * wp + 3 * f.experts * pad64(f.ff) * wp
    return n


def step_scratch_elems(cfg: ModelConfig, rows: int, keys: int = 0) -> int:
    """Upper bound, in 32-bit words, of what a step of ``rows`` rows allocates (``keys``: expanded key rows)."""
    wp, n = pad64(cfg.hidden), 0
    for s in cfg.layer_specs:
        g, f = LatentGeometry.of(s.mixer), s.ffn
        one = rows * (9 * (g.n_down + g.heads * g.dk) + 10 * wp + g.heads * (g.lc + 2 * g.dv))
        one += max(rows, SMS) * g.heads * (g.kvp + 2) + keys * (g.lc + g.heads * (g.dn + g.dv)) + rows * g.heads * g.dk
        if f is not None:
            slots = rows * f.top + (f.experts + 1) * 128
            one += slots * (4 * wp + pad64(f.ff)) + rows * f.experts
        n = max(n, one)
    # layers of unequal sizes keep scratch of their own
    return n * len(set(cfg.layer_specs)) + rows * wp * 4


# ------------------------------------------------------------------ scratch of a step
class ListedScratch:
    """Activations of a step by name.  The decode step's (``fixed`` rows) are allocated once, because captured graphs
    keep their addresses; a mixed batch's grow with the largest batch."""

    def __init__(self, device, dtype, fixed: int = 0):
        self.device, self.dtype, self.fixed = device, dtype, fixed
        self._t: Dict[tuple, torch.Tensor] = {}

    def get(self, name: str, rows: int, cols: int, dtype=None, mult: int = 1) -> torch.Tensor:
        """``[rows][cols]`` view; ``mult``: value rows per row of the step.  New memory is zeroed: padding that nothing
        writes is zero and stale rows are finite."""
        dtype = dtype or self.dtype
        key = (name, cols, mult, dtype)
        t = self._t.get(key)
        need = max(rows, self.fixed * mult) * cols
        if t is None or t.numel() < need:
            if self.fixed and t is not None:
                raise RuntimeError(f"the decode step's scratch {name!r} cannot grow under captured graphs")
            t = self._t[key] = torch.zeros(need, dtype=dtype, device=self.device)
        return t[: rows * cols].view(rows, cols)

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._t.values())


@dataclass
class StepRows:
    """The rows of a step: device int32 arrays of request slots, positions and tokens."""
    req: torch.Tensor
    pos: torch.Tensor
    token: torch.Tensor


@dataclass
class KeyPlan:
    """Prompt segments of a batch for one (window, rows per tile): the cache rows whose keys and values the segments see
    and the query tiles over them."""
    n_keys: int
    kreq: torch.Tensor
    kpos: torch.Tensor
    n_tiles: int
    tiles: torch.Tensor


@dataclass
class BatchPlan:
    """How a mixed batch's rows are attended: rows before ``n_single`` one by one over the latent, the rest by prompt
    segments (``keys[(window, rows per tile)]``)."""
    n_single: int
    keys: Dict[tuple, KeyPlan]


class ListedLayers:
    """Sublayer functions of a listed model over one device's weights."""

    def __init__(self, weights: ModelWeights, max_pos: int):
        self.w, self.cfg = weights, weights.cfg
        self.device, self.dtype = weights.embed.device, weights.embed.dtype
        self.f32 = self.dtype == torch.float32
        self.wp = weights.embed.shape[1]
        self.geo = [LatentGeometry.of(s.mixer) for s in self.cfg.layer_specs]
        self.max_pos = max_pos
        self._rope: Dict[tuple, tuple] = {}
        for s in self.cfg.layer_specs:
            key = (s.mixer.rope_dims, s.mixer.rope_base)
            if key not in self._rope:
                c, sn = rope_tables(key[0], key[1], max_pos)
                self._rope[key] = (c.to(self.device).contiguous(), sn.to(self.device).contiguous())
        self._splits: Dict[tuple, int] = {}
        self._rows_form: Dict[LatentGeometry, bool] = {}
        self._tile_rows: Dict[LatentGeometry, int] = {}

    # ---------------------------------------------------------------- pieces
    def rope(self, a: LatentAttention):
        return self._rope[(a.rope_dims, a.rope_base)]

    def tile_rows(self, g: LatentGeometry) -> int:
        """Query rows per tile of the expanded prompt attention, 0 when this mixer has none."""
        if self.f32:
            return 0
        if g not in self._tile_rows:
            self._tile_rows[g] = L.prefill_rows_per_tile(g)
        return self._tile_rows[g]

    def rows_form(self, g: LatentGeometry) -> bool:
        if g not in self._rows_form:
            self._rows_form[g] = not self.f32 and L.rows_ok(g)
        return self._rows_form[g]

    def nsplit(self, a: LatentAttention, g: LatentGeometry, m: int) -> int:
        """KV splits of the decode attention: about one CTA per SM, at least one key tile per split."""
        if not self.rows_form(g):
            return 1
        keys = min(a.window, self.max_pos) if a.window else self.max_pos
        groups = (a.heads + 31) // 32 if a.heads > 16 else 1
        return max(1, min(64, SMS // (m * groups), (keys + 63) // 64))

    def linear(self, sc: ListedScratch, name: str, w: torch.Tensor, x: torch.Tensor, m: int):
        """fp32 ``x[:m] @ w.T`` as (slices [s][m][n], s)."""
        n, k = w.shape
        if self.f32 or m > L.GEMV_ROWS:
            out = sc.get(name, m, n, torch.float32)
            if self.f32:
                L.linear_f32(x, w, out, m)
            else:
                G.gemm_bf16(x[:m], w, out, epi=G.EPI_F32)
            return out, 1
        s = self._splits.get((n, k))
        if s is None:
            s = self._splits[(n, k)] = L.gemv_splits(n, k)
        out = sc.get(name, m * s, n, torch.float32, mult=s)
        L.gemv_bf16(w, x, out, m, n, k, s)
        return out, s

    # ---------------------------------------------------------------- mixer
    def mixer(self, sc: ListedScratch, li: int, m: int, rows: StepRows, block_table, cache, plan: Optional[BatchPlan]):
        """Latent attention of the step's rows: fp32 slices of its output projection."""
        a, g, w = self.cfg.layer_specs[li].mixer, self.geo[li], self.w.layers[li].latent
        h = sc.get("h", m, self.wp)
        part, s = self.linear(sc, "down", w.down, h, m)
        cq = sc.get("cq", m, g.qp)
        rope = self.rope(a)
        L.prep(part, s, m, g, w.q_norm, w.kv_norm, self.cfg.rms_eps, rows.req, rows.pos, block_table, rope, cq, cache)
        out = sc.get("attn", m, g.heads * g.dv)
        tile_rows = self.tile_rows(g)
        n1 = m if plan is None or not tile_rows else plan.n_single
        if n1:
            q, s = self.linear(sc, "q", w.uq, cq, n1)
            ql = sc.get("ql", n1, g.heads * g.lc)
            L.absorb(q, s, n1, g, w.uk, rows.pos, rope, ql)
            ns = self.nsplit(a, g, n1)
            cap = max(n1 * ns, SMS) if sc.fixed else n1 * ns
            op = sc.get("o_part", cap, g.heads * g.kvp, torch.float32)
            ml = sc.get("ml_part", cap, g.heads * 2, torch.float32)
            if self.rows_form(g):
                L.rows(ql, cache, n1, g, rows.req, rows.pos, block_table, op, ml, ns, a.window, a.scale)
            else:
                L.simple(ql, cache, n1, g, rows.req, rows.pos, block_table, op, ml, a.window, a.scale)
            L.merge(op, ml, n1, g, ns, w.uv, out)
        if n1 < m:
            self._prompt_attention(sc, a, g, w, cq[n1:], m - n1, rows.pos[n1:], block_table, cache,
                                   plan.keys[(a.window, tile_rows)], rope, out[n1:])
        return self.linear(sc, "o", w.o, out, m)

    def _prompt_attention(self, sc, a, g, w, cq, m, pos, block_table, cache, kp: KeyPlan, rope, out):
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

    # ---------------------------------------------------------------- feed-forward
    def experts(self, sc: ListedScratch, f: ExpertFfn, w: ExpertStack, m: int):
        """Routed experts of the step's rows: arguments of ``sublayer_norm`` that describe the weighted slots."""
        k, wp, er = f.top, self.wp, w.router.shape[0]
        ffp = w.down.shape[2]
        i32, f32 = torch.int32, torch.float32
        h = sc.get("h", m, wp)
        logits = sc.get("router", m, er, f32)
        idx, wt = sc.get("topk_idx", m, k, i32), sc.get("topk_w", m, k, f32)
        few = m <= EXPERT_GEMV_ROWS
        if not self.f32 and m <= L.GEMV_ROWS:
            M.router_rows(w.router, h, logits, m, f.experts, wp, er, f.experts, k, False, False, idx, wt,
                          sc.get("ticket", 1, 1, i32), rule=f.rule)
        else:
            if self.f32:
                L.linear_f32(h, w.router, logits, m)
            else:
                G.gemm_bf16(h, w.router, logits, epi=G.EPI_F32)
            M.route(logits, er, m, f.experts, k, idx, wt, rule=f.rule)
        if self.f32:
            act, y = sc.get("act", m * k, ffp, mult=k), sc.get("y", m * k, wp, mult=k)
            L.linear_f32_experts(w.gate_up, idx.view(-1), m * k, h, k, act, True)
            L.linear_f32_experts(w.down, idx.view(-1), m * k, act, 1, y, False)
            return dict(y=y, slots=k, row_elems=wp, slot_w=wt)
        if few:
            act = sc.get("act", m * k, ffp, mult=k)
            L.gemv_bf16_experts(w.gate_up, idx, m * k, h, k, act, 2 * ffp, wp, epi=L.EPI_SILU)
            s = self._splits.get((wp, ffp, "experts"))
            if s is None:
                s = self._splits[(wp, ffp, "experts")] = min(2, L.gemv_splits(wp, ffp))
            y = sc.get("y", m * k * s, wp, f32, mult=k * s)
            L.gemv_bf16_experts(w.down, idx, m * k, act, 1, y, wp, ffp, splits=s)
            return dict(y=y, slots=k, slices=s, row_elems=s * wp, slice_elems=wp, slot_w=wt)
        # expert-sorted rows in blocks of 128 for the grouped GEMMs; counts stay on the device
        e = f.experts
        blk = (m * k + 127) // 128 + e
        cap = (max(m, sc.fixed) * k + 127) // 128 + e
        meta = sc.get(f"moe_tables_{e}_{k}", 2 * e + 3 * cap + 2, 1, i32).view(-1)
        counts, base, n_blk = meta[:e], meta[e: 2 * e], meta[2 * e: 2 * e + 1]
        total, tabs = meta[2 * e + 1: 2 * e + 2], meta[2 * e + 2:]
        be, br, bn = tabs[:blk], tabs[cap: cap + blk], tabs[2 * cap: 2 * cap + blk]
        rank, row_of = sc.get("moe_rank", m, k, i32), sc.get("moe_row", m, k, i32)
        xs, act, y = (sc.get(f"{nm}_{e}_{k}" if sc.fixed else nm, cap * 128, c) for nm, c in (("moe_x", wp), ("moe_act", ffp), ("moe_y", wp)))
        counts.zero_()
        M.sort(idx, m, k, e, blk, counts, rank, base, be, br, bn, n_blk, total)
        M.scatter(idx, rank, base, m, k, h, wp, row_of, xs)
        blocks = (be, br, bn, n_blk, blk)
        G.gemm_grouped_bf16(xs, w.gate_up, act, blocks, epi=G.EPI_SILU_MUL)
        G.gemm_grouped_bf16(act, w.down, y, blocks)
        return dict(y=y, slots=k, row_elems=wp, slot_w=wt, row_of=row_of)
