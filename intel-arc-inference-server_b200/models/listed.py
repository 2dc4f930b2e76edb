"""Models that list their layers: what every such model shares.

A layer is a mixer and a feed-forward (``LayerSpec``).  Each kind of mixer has a module of its own (``latent``, ``grouped``,
``mlstm``, ``retention``, ``mingru``, ``channel_delta``, ``wkv``; ``parallel``: two of them side by side) with the same functions: ``shapes`` and
``assemble`` (checkpoint tensors, kernel-layout weights), ``tensor_sizes`` (sizes that only the tensors give; not every kind has
some), ``weight_elems`` and ``scratch_elems`` (the planner's figures), ``page_planes`` (what it keeps per position in the page
pool), ``state_shapes`` (what it keeps per sequence) and ``Mixer``, whose ``run`` enqueues its kernels for the rows of a step and
whose ``forms`` are the tables it wants of a mixed batch's prompt segments.  Pages and states belong to layer runs
(``ModelConfig.layer_runs``): a layer that runs several times in a step has several, and a layer that uses another one's weights
(``LayerSpec.weights_of``) has its own.
The residual around the sublayers is ``streams.StreamWalk``, ``sandwich.SandwichWalk`` or the layer-normed single stream of
``DecoderModel.listed_walk``.  ``Engine`` gives both the rows of a decode step (control block, CUDA graphs) or of a mixed
batch (``runtime/batch.py``).

Kernel sizes are whole 64s: weights are padded with zeros when they are loaded (rows and columns), and padded activation
columns are zero; norms, rotations and scales use the true sizes.

Few rows (up to 16) take the weight-streaming GEMVs, more rows the tcgen05 GEMMs.  Models whose weights are fp32 run
everything in 32-bit (no reduced-precision product anywhere).
"""
from __future__ import annotations

import dataclasses
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

import torch

from ..ops import gemm as G
from ..ops import latent as L
from ..ops import moe as M
from .config import (ChannelDelta, DenseFfn, ExpertFfn, GroupedAttention, LatentAttention, MatrixLstm, MinGru, ModelConfig,
                     ParallelMixer, Retention, Rotary, SandwichBlock, Wkv)
from .weights import DenseWeights, ExpertStack, LayerWeights, ModelWeights, interleave16

SMS = 148
# Experts of more rows than this go through the expert-sorted grouped GEMMs, which read every chosen expert once; the
# GEMVs read one expert per (row, slot).
EXPERT_GEMV_ROWS = int(os.environ.get("B2_EXPERT_GEMV_ROWS", "4"))


def pad64(n: int) -> int:
    return (n + 63) // 64 * 64


def kind(mixer):
    """The module of a mixer's kind."""
    from . import channel_delta, grouped, latent, mingru, mlstm, parallel, retention, wkv
    return {LatentAttention: latent, GroupedAttention: grouped, MatrixLstm: mlstm, Retention: retention, MinGru: mingru,
            ParallelMixer: parallel, ChannelDelta: channel_delta, Wkv: wkv}[type(mixer)]


def pair_order(dims: int, size: int) -> list:
    """Order of a head's dimensions in the kernels, which rotate neighbours: i and i + dims / 2 next to each other, then the rest."""
    return [i + half for i in range(dims // 2) for half in (0, dims // 2)] + list(range(dims, size))


def sizes_in_tensors(cfg: ModelConfig) -> bool:
    """Some of the model's sizes are given by its tensors only."""
    return any(hasattr(kind(s.mixer), "tensor_sizes") for s in cfg.layer_specs)


def with_tensor_sizes(cfg: ModelConfig, shape: Callable[[str], tuple]) -> ModelConfig:
    """The configuration with the sizes that only the checkpoint's tensors give (``shape(name)``)."""
    specs = []
    for i, s in enumerate(cfg.layer_specs):
        sizes = getattr(kind(s.mixer), "tensor_sizes", None)
        specs.append(s if sizes is None else dataclasses.replace(s, mixer=sizes(f"l{i}.mix.", s.mixer, shape)))
    return dataclasses.replace(cfg, layer_specs=tuple(specs))


# ------------------------------------------------------------------ weights
def tensor_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    """Checkpoint tensors of a listed model, by name."""
    from . import streams
    h, behind = cfg.hidden, isinstance(cfg.block, SandwichBlock)
    norm = (h,) if cfg.block is None or cfg.block.columns or behind else ()

    def feed(p, ff, gated):
        out.update({p + "up": (ff, h), p + "down": (h, ff)})
        if gated:
            out[p + "gate"] = (ff, h)
    out = {"embed": (cfg.vocab, h), "final.norm": norm, "head": (cfg.vocab, h)}
    for i, s in enumerate(cfg.layer_specs):
        p, f = f"l{i}.", s.ffn
        if s.weights_of >= 0:
            continue
        out[p + "norm1"] = norm
        out.update(kind(s.mixer).shapes(cfg, p + "mix.", s.mixer))
        if behind:
            out.update({p + f"norm{q}b": norm for q in ((1,) if f is None else (1, 2))})
        elif cfg.block is not None:
            out.update(streams.shapes(cfg, p, s))
        if f is None:
            continue
        out[p + "norm2"] = norm
        if isinstance(f, DenseFfn):
            feed(p + "mlp.", f.ff, not f.relu2)
            if f.bias:
                out.update({p + "mlp.gate.b": (f.ff,), p + "mlp.up.b": (f.ff,), p + "mlp.down.b": (h,)})
        else:
            out[p + "mlp.router"] = (f.experts, h)
            for e in range(f.experts):
                feed(f"{p}mlp.e{e}.", f.ff, not f.relu2)
            if f.shared:
                feed(p + "mlp.shared.", f.shared, not f.relu2)
    if cfg.loop is not None:
        out["loop.step"] = (cfg.loop.times, h)
    return out


class Assembler:
    """Checkpoint tensors (``get(name)``) in kernel layout on one device."""

    def __init__(self, cfg: ModelConfig, get: Callable[[str], torch.Tensor], device, dtype):
        self.cfg, self.get, self.device, self.dtype = cfg, get, device, dtype
        self.wp = pad64(cfg.hidden)

    def t(self, name: str) -> torch.Tensor:
        return self.get(name).to(device=self.device, dtype=self.dtype)

    def vec(self, name: str, cols: int = 0) -> torch.Tensor:
        """fp32 vector (or single number), padded with zeros to ``cols``."""
        v = self.get(name).float().to(self.device).reshape(-1)
        if cols > len(v):
            v = torch.cat([v, torch.zeros(cols - len(v), device=self.device)])
        return v.contiguous()

    def norm(self, name: str) -> torch.Tensor:
        """Norm weights as factors."""
        if isinstance(self.cfg.block, SandwichBlock):
            return self.vec(name, self.wp)
        if self.cfg.block is None or not self.cfg.block.columns:
            return self.vec(name)
        return self.vec(name, self.wp) + (torch.arange(self.wp, device=self.device) < self.cfg.hidden)

    def stack(self, parts) -> torch.Tensor:
        return torch.cat(parts).contiguous()

    def fp32_heads(self, name: str, n: int, size: int, pad: int, cols: int) -> torch.Tensor:
        """fp32 ``[n * pad][cols]`` from head-major rows."""
        out = torch.zeros(n, pad, cols, dtype=torch.float32, device=self.device)
        out[:, :size] = self.get(name).float().to(self.device).reshape(n, size, cols)
        return out.reshape(n * pad, cols)

    def zeros(self, *shape) -> torch.Tensor:
        return torch.zeros(*shape, dtype=self.dtype, device=self.device)

    def padded(self, w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
        out = self.zeros(rows, cols)
        out[: w.shape[0], : w.shape[1]] = w
        return out

    def heads(self, w: torch.Tensor, n: int, parts, cols: int, order=None) -> torch.Tensor:
        """Head-major rows: each head's parts (true size, padded size) in turn; ``order``: of a head's rows."""
        out = self.zeros(n, sum(p for _, p in parts), cols)
        v = w.reshape(n, sum(s for s, _ in parts), w.shape[1])
        if order is not None:
            v = v[:, order]
        src = dst = 0
        for size, pad in parts:
            out[:, dst: dst + size, : w.shape[1]] = v[:, src: src + size]
            src, dst = src + size, dst + pad
        return out.reshape(-1, cols)

    def out_proj(self, name: str, heads: int, size: int, pad: int, order=None) -> torch.Tensor:
        """Output projection over concatenated heads: [wp][heads * pad]; ``order``: of a head's columns."""
        o, w = self.zeros(self.wp, heads, pad), self.t(name).reshape(self.cfg.hidden, heads, size)
        o[: self.cfg.hidden, :, :size] = w if order is None else w[..., order]
        return o.reshape(self.wp, heads * pad)

    def gate_up(self, p: str, ffp: int, gated: bool = True, lo: int = 0) -> torch.Tensor:
        """What a feed-forward's hidden columns ``lo`` .. are made with."""
        gate, up = (self.padded(self.t(p + n)[lo: lo + ffp], ffp, self.wp) if n == "up" or gated else None for n in ("gate", "up"))
        return interleave16(gate, up) if gated else up

    def down(self, p: str, ffp: int, lo: int = 0) -> torch.Tensor:
        return self.padded(self.t(p + "down")[:, lo: lo + ffp], self.wp, ffp)


def assemble(cfg: ModelConfig, get: Callable[[str], torch.Tensor], device, dtype=torch.bfloat16) -> ModelWeights:
    """Kernel-layout weights from checkpoint tensors (``get(name)``)."""
    from . import streams
    a = Assembler(cfg, get, device, dtype)
    wp, layers = a.wp, []
    for i, s in enumerate(cfg.layer_specs):
        p, f = f"l{i}.", s.ffn
        if s.weights_of >= 0:
            layers.append(None)
            continue
        lw = LayerWeights(input_norm=a.norm(p + "norm1"), post_norm=a.norm(p + "norm2") if f is not None else None, qkv=None, o=None)
        lw.mixer = kind(s.mixer).assemble(a, p + "mix.", s.mixer)
        if cfg.block is not None and cfg.block.mixing:
            lw.streams = streams.assemble(a, p, s)
        if isinstance(cfg.block, SandwichBlock):
            lw.behind = (a.norm(p + "norm1b"), a.norm(p + "norm2b") if f is not None else None)
        if isinstance(f, DenseFfn):
            ffp = pad64(f.ff)
            lw.dense = DenseWeights(a.gate_up(p + "mlp.", ffp, not f.relu2), a.down(p + "mlp.", ffp))
            if f.bias:
                lw.dense.bias = interleave16(a.vec(p + "mlp.gate.b", ffp)[:, None], a.vec(p + "mlp.up.b", ffp)[:, None]).view(-1).contiguous()
                lw.dense.down_bias = a.vec(p + "mlp.down.b", wp)
        elif f is not None:
            ffp = pad64(f.ff)
            held = f.experts + f.shared_slots
            gu, dn = a.zeros(held, (1 if f.relu2 else 2) * ffp, wp), a.zeros(held, wp, ffp)
            for e in range(held):      # a shared expert is as many of the common width as its hidden columns fill
                q, lo = (f"{p}mlp.e{e}.", 0) if e < f.experts else (p + "mlp.shared.", (e - f.experts) * ffp)
                gu[e] = a.gate_up(q, ffp, not f.relu2, lo)
                dn[e] = a.down(q, ffp, lo)
            lw.moe = ExpertStack(a.padded(a.t(p + "mlp.router"), (f.experts + 7) // 8 * 8, wp), gu, dn)
        layers.append(lw)
    for i, s in enumerate(cfg.layer_specs):
        j = i
        while cfg.layer_specs[j].weights_of >= 0:
            j = cfg.layer_specs[j].weights_of
        layers[i] = layers[j]
    w = ModelWeights(cfg, a.padded(a.t("embed"), cfg.vocab, wp), a.padded(a.t("head"), cfg.vocab, wp), a.norm("final.norm"), layers)
    if cfg.loop is not None:
        w.loop_step = torch.zeros(cfg.loop.times, wp, dtype=torch.float32, device=device)
        w.loop_step[:, : cfg.hidden] = get("loop.step").float().to(device)
    return w


def random_listed_weights(cfg: ModelConfig, device="cpu", seed: int = 0, std: float = 0.02,
                          dtype=torch.bfloat16) -> ModelWeights:
    from . import streams
    shapes = tensor_shapes(cfg)
    g = torch.Generator(device=device)
    g.manual_seed(seed)

    def get(name):
        shape = shapes[name]
        plain = streams.plain_value(cfg, name, shape)
        if plain is not None:
            return plain.to(device)
        if len(shape) < 2:
            return torch.ones(shape, device=device)
        return torch.empty(shape, dtype=torch.bfloat16, device=device).normal_(0, std if name == "head" else shape[1] ** -0.5, generator=g)
    return assemble(cfg, get, device, dtype)


def padded_weight_elems(cfg: ModelConfig) -> int:
    """Elements of the assembled weights (host arithmetic, the memory planner's figure)."""
    wp, n = pad64(cfg.hidden), 2 * cfg.vocab * pad64(cfg.hidden)
    for s in cfg.layer_specs:
        f = s.ffn
        if s.weights_of >= 0:
            continue
        n += kind(s.mixer).weight_elems(cfg, s.mixer)
        if f is not None:
            each = (2 if f.relu2 else 3) * pad64(f.ff) * wp
            n += each if isinstance(f, DenseFfn) else (f.experts + 7) // 8 * 8 * wp + (f.experts + f.shared_slots) * each
    return n


def state_elems(cfg: ModelConfig) -> int:
    """fp32 elements of one sequence's recurrent states."""
    n = 0
    for s in cfg.run_specs:
        for shape in kind(s.mixer).state_shapes(s.mixer).values():
            size = 1
            for d in shape:
                size *= d
            n += size
    return n


def step_scratch_elems(cfg: ModelConfig, rows: int, keys: int = 0) -> int:
    """Upper bound, in 32-bit words, of what a step of ``rows`` rows allocates (``keys``: expanded key rows)."""
    wp, n = pad64(cfg.hidden), 0
    for s in cfg.layer_specs:
        f = s.ffn
        one = rows * 10 * wp + kind(s.mixer).scratch_elems(cfg, s.mixer, rows, keys)
        if isinstance(f, DenseFfn):
            one += rows * 3 * pad64(f.ff)
        elif f is not None:
            slots = rows * (f.top + f.shared_slots) + (f.experts + f.shared_slots + 1) * 128
            one += slots * (4 * wp + pad64(f.ff)) + rows * f.experts
        n = max(n, one)
    # layers of unequal sizes keep scratch of their own
    n = n * len({(s.mixer, s.ffn) for s in cfg.layer_specs}) + rows * wp * 4
    return n + (rows * wp * (2 * cfg.block.streams + 2) if cfg.block is not None else 0)


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
    """The rows of a step: device int32 arrays of request slots, positions and tokens.  Rows of a request are consecutive."""
    req: torch.Tensor
    pos: torch.Tensor
    token: torch.Tensor

    def tail(self, n: int) -> "StepRows":
        return StepRows(self.req[n:], self.pos[n:], self.token[n:])


@dataclass
class BatchPlan:
    """How a mixed batch's rows are handled: rows before ``n_single`` one by one, the rest as prompt segments, described by
    one table per form the model's mixers use (``tables[form]``, see ``runtime/batch.py``)."""
    n_single: int
    tables: Dict[tuple, object]


class ListedLayers:
    """Mixers and feed-forwards of a listed model over one device's weights."""

    def __init__(self, weights: ModelWeights, max_pos: int):
        self.w, self.cfg = weights, weights.cfg
        self.device, self.dtype = weights.embed.device, weights.embed.dtype
        self.f32 = self.dtype == torch.float32
        self.wp = weights.embed.shape[1]
        self.max_pos = max_pos
        self.shared: Dict[tuple, object] = {}        # what layers of equal sizes share (angle tables and the like)
        self._splits: Dict[tuple, int] = {}
        if self.cfg.loop is not None and (self.cfg.block is None or any(getattr(s.mixer, "kv_from", -1) >= 0 for s in self.cfg.layer_specs)):
            raise ValueError(f"{self.cfg.name}: layers that run several times need the pre-normed residual and keys of their own")
        self.mixers = [kind(self.cfg.layer_specs[i].mixer).Mixer(self, j, self.cfg.layer_specs[i].mixer, weights.layers[i].mixer)
                       for j, (i, _) in enumerate(self.cfg.layer_runs)]

    def rotation(self, rot: Rotary):
        """(cos, sin) tables ``[positions][pairs]``, angles in double precision."""
        if rot not in self.shared:
            freq, amp = rot.frequencies()
            angle = torch.arange(self.max_pos, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None, :]
            self.shared[rot] = tuple((f(angle) * amp).float().to(self.device).contiguous() for f in (torch.cos, torch.sin))
        return self.shared[rot]

    def forms(self):
        """Tables the mixers want of a mixed batch's prompt segments."""
        return sorted({f for m in self.mixers for f in m.forms})

    def shifted(self, sc: ListedScratch, planes: int, m: int) -> torch.Tensor:
        """``[planes * m][wp]``: what a mixer with several shifted inputs reads."""
        return sc.get(f"h_shift{planes}", planes * m, self.wp, mult=planes)

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
        s = self.splits(n, k)
        out = sc.get(name, m * s, n, torch.float32, mult=s)
        L.gemv_bf16(w, x, out, m, n, k, s)
        return out, s

    def linear_planes(self, sc: ListedScratch, name: str, w: torch.Tensor, x: torch.Tensor, plane_rows: int, m: int):
        """``linear`` with activations ``x`` ``[planes][m][k]``: weight rows ``n`` read plane ``min(n // plane_rows, planes - 1)``."""
        n, k = w.shape
        if self.f32 or m > L.GEMV_ROWS:
            out, last = sc.get(name, m, n, torch.float32), x.shape[0] - 1
            for i in range(x.shape[0]):
                lo, hi = i * plane_rows, n if i == last else (i + 1) * plane_rows
                if self.f32:
                    L.linear_f32(x[i], w[lo:hi], out[:, lo:hi], m)
                else:
                    G.gemm_bf16(x[i], w[lo:hi], out[:, lo:hi], epi=G.EPI_F32)
            return out, 1
        s = self.splits(n, k)
        out = sc.get(name, m * s, n, torch.float32, mult=s)
        L.gemv_bf16_planes(w, x, plane_rows, out, m, n, k, s)
        return out, s

    def splits(self, n: int, k: int) -> int:
        s = self._splits.get((n, k))
        if s is None:
            s = self._splits[(n, k)] = L.gemv_splits(n, k)
        return s

    # ---------------------------------------------------------------- feed-forwards
    def dense(self, sc: ListedScratch, f: DenseFfn, w: DenseWeights, m: int):
        """Feed-forward of the step's rows: fp32 slices of its down projection (without its bias)."""
        h = sc.get("h", m, self.wp)
        n = w.gate_up.shape[0]
        if f.relu2:
            act = sc.get("ffn_act", m, n)
            if self.f32:
                L.linear_f32(h, w.gate_up, act, m, squared=True)
            elif m <= L.GEMV_ROWS:
                L.gemv_bf16(w.gate_up, h, act, m, n, self.wp, epi=L.EPI_RELU2)
            else:
                G.gemm_bf16(h, w.gate_up, act, epi=G.EPI_RELU2)
            return self.linear(sc, "ffn_down", w.down, act, m)
        act = sc.get("ffn_act", m, n // 2)
        if self.f32:
            gu = sc.get("gate_up", m, n)
            L.linear_f32(h, w.gate_up, gu, m)
            L.glu_rows_f32(gu, act, m, n, f.limit, f.alpha, f.shift, f.gelu, w.bias)
        elif m <= L.GEMV_ROWS:
            L.gemv_bf16_glu(w.gate_up, h, act, m, n, self.wp, f.limit, f.alpha, f.shift, f.gelu, w.bias)
        else:
            G.gemm_glu(h, w.gate_up, act, f.limit, f.alpha, f.shift, f.gelu, w.bias)
        return self.linear(sc, "ffn_down", w.down, act, m)

    def experts(self, sc: ListedScratch, f: ExpertFfn, w: ExpertStack, m: int):
        """Routed experts of the step's rows (and the shared one, as slots with weight one): arguments of ``sublayer_norm`` that
        describe the weighted slots."""
        shared = f.shared_slots
        k, wp, er = f.top + shared, self.wp, w.router.shape[0]
        ffp = w.down.shape[2]
        i32, f32 = torch.int32, torch.float32
        h = sc.get("h", m, wp)
        logits = sc.get("router", m, er, f32)
        idx, wt = sc.get("topk_idx", m, k, i32), sc.get("topk_w", m, k, f32)
        few = m <= EXPERT_GEMV_ROWS
        if not self.f32 and m <= L.GEMV_ROWS:
            M.router_rows(w.router, h, logits, m, f.experts, wp, er, f.experts, f.top, shared, False, idx, wt,
                          sc.get("ticket", 1, 1, i32), rule=f.rule)
        else:
            if self.f32:
                L.linear_f32(h, w.router, logits, m)
            else:
                G.gemm_bf16(h, w.router, logits, epi=G.EPI_F32)
            M.route(logits, er, m, f.experts, f.top, idx, wt, rule=f.rule, shared=shared)
        if self.f32:
            act, y = sc.get("act", m * k, ffp, mult=k), sc.get("y", m * k, wp, mult=k)
            L.linear_f32_experts(w.gate_up, idx.view(-1), m * k, h, k, act, L.ACT_RELU2 if f.relu2 else L.ACT_SILU)
            L.linear_f32_experts(w.down, idx.view(-1), m * k, act, 1, y, L.ACT_NONE)
            return dict(y=y, slots=k, row_elems=wp, slot_w=wt)
        if few:
            act = sc.get("act", m * k, ffp, mult=k)
            L.gemv_bf16_experts(w.gate_up, idx, m * k, h, k, act, w.gate_up.shape[1], wp, epi=L.EPI_RELU2 if f.relu2 else L.EPI_SILU)
            s = self._splits.get((wp, ffp, "experts"))
            if s is None:
                s = self._splits[(wp, ffp, "experts")] = min(2, L.gemv_splits(wp, ffp))
            y = sc.get("y", m * k * s, wp, f32, mult=k * s)
            L.gemv_bf16_experts(w.down, idx, m * k, act, 1, y, wp, ffp, splits=s)
            return dict(y=y, slots=k, slices=s, row_elems=s * wp, slice_elems=wp, slot_w=wt)
        # expert-sorted rows in blocks of 128 for the grouped GEMMs; counts stay on the device
        e = f.experts + shared
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
        G.gemm_grouped_bf16(xs, w.gate_up, act, blocks, epi=G.EPI_RELU2 if f.relu2 else G.EPI_SILU_MUL)
        G.gemm_grouped_bf16(act, w.down, y, blocks)
        return dict(y=y, slots=k, row_elems=wp, slot_w=wt, row_of=row_of)
