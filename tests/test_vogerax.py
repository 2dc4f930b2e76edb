"""Vogerax on the GPU against the plain reference (tests/vogerax_oracle.py): every mechanism alone, then whole models served in
32-bit (sharp) and in bf16, in prompts, portions, decode steps, mixed batches and reused pages and slots."""
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import vogerax_oracle as O
from b200serve.models.config import (DenseFfn, ExpertFfn, GroupedAttention, LayerSpec, ParallelMixer, Retention, Rotary, SandwichBlock,
                                     listed_config, preset)

pytestmark = pytest.mark.gpu
DEV = "cuda"
F32, BF16, F64 = torch.float32, torch.bfloat16, torch.float64


def rel(got, ref):
    return float((got.double().cpu() - ref.double().cpu()).pow(2).mean().sqrt() / ref.double().pow(2).mean().sqrt().cpu())


def worst_row(got, ref):
    got, ref = got.double().cpu().flatten(1), ref.double().cpu().flatten(1)
    return float(((got - ref).pow(2).mean(-1) / ref.pow(2).mean(-1)).sqrt().max())


def gen(seed):
    return torch.Generator().manual_seed(seed)


def i32(v):
    return torch.tensor(np.asarray(v), dtype=torch.int32, device=DEV)


def pad_cols(t, ld):
    out = torch.zeros(*t.shape[:-1], ld, dtype=t.dtype)
    out[..., : t.shape[-1]] = t
    return out


def runs_rows(runs):
    """(slot, position) of every row of runs (slot, first position, rows)."""
    return [(s, p + i) for s, p, n in runs for i in range(n)]


def slices_of(full, slices, seed=1):
    """fp32 slices that add up to ``full``."""
    part = torch.randn(slices, *full.shape, generator=gen(seed))
    part[-1] = full - part[:-1].sum(0)
    return part.to(DEV)


def tables(freq, n, amp=1.0):
    a = torch.arange(n, dtype=F64)[:, None] * torch.as_tensor(freq, dtype=F64)[None]
    return tuple((f(a) * amp).float().to(DEV).contiguous() for f in (torch.cos, torch.sin))


def order(dims, size):
    """Kernel order of a head's dimensions: rotated pairs are neighbours."""
    return [i + h for i in range(dims // 2) for h in (0, dims // 2)] + list(range(dims, size))


# ------------------------------------------------------------------ residual
@pytest.mark.parametrize("width,ld,groups", [(72, 128, 1), (72, 128, 9), (210, 256, 3), (1500, 1536, 4), (1500, 1536, 500), (5000, 5056, 2), (2048, 2048, 16)])
@pytest.mark.parametrize("m", [1, 5, 70])
def test_boundary(width, ld, groups, m):
    """x + G(y) post, G of that for the next sublayer: slices, weighted slots in any rows, two normed results, bf16 values."""
    from b200serve.ops import sandwich as S
    g, eps = gen(width + m + groups), 0.2
    rnd = lambda *s: torch.randn(*s, generator=g)                                  # noqa: E731
    x, post, nxt = rnd(m, width), rnd(width), rnd(width)
    scale = torch.rand(width, generator=g) ** 2 * 3       # parts of unequal size: a column in the wrong group shows
    norm = lambda v, w: O.group_norm(v, w.double(), eps, groups)                   # noqa: E731

    def check(sources, y, h_dtype=F32, **kw):
        xo = torch.full((m, ld), float("nan"), device=DEV)
        h = torch.full((m, ld), float("nan"), dtype=h_dtype, device=DEV)
        S.boundary(sources, m=m, width=width, groups=groups, eps=eps, post=pad_cols(post, ld).to(DEV), next=pad_cols(nxt, ld).to(DEV),
                   x_in=pad_cols(x, ld).to(DEV), x_out=xo, h=h, **kw)
        want = x.double() + norm(y, post)
        assert worst_row(xo[:, :width], want) < 1e-5 and torch.all(xo[:, width:] == 0)
        assert worst_row(h[:, :width], norm(want, nxt)) < (1e-5 if h_dtype == F32 else 6e-3) and torch.all(h[:, width:] == 0)
    for s in (1, 3):
        y = rnd(s, m, width) * scale
        check([S.source(pad_cols(y, ld).to(DEV), ld, slices=s, slice_elems=m * ld)], y.double().sum(0), BF16 if s == 1 else F32)
    # weighted slots: rows in order with slices; sorted rows in bf16
    k, s = 3, 2
    y, w = rnd(m * k, s, width) * scale, torch.rand(m, k, generator=g)
    check([S.source(pad_cols(y, ld).to(DEV), s * ld, slices=s, slice_elems=ld, slots=k, slot_w=w.to(DEV))],
          (w.double()[..., None] * y.double().sum(1).view(m, k, width)).sum(1))
    perm, yb = torch.randperm(m * k, generator=g), (rnd(m * k, width) * scale).bfloat16()
    check([S.source(pad_cols(yb, ld).to(DEV), ld, slots=k, slot_w=w.to(DEV), row_of=i32(perm))], (w.double()[..., None] * yb.double()[perm].view(m, k, width)).sum(1))
    # two results, each through a norm of its own, side by side in the slices
    two, gains = rnd(2, m, 2, width) * scale, rnd(2, width)
    t = pad_cols(two, ld).to(DEV).view(2, m, 2 * ld)
    check([S.source(t.view(-1)[i * ld:], 2 * ld, slices=2, slice_elems=m * 2 * ld, factor=f, norm=pad_cols(gains[i], ld).to(DEV)) for i, f in ((0, 0.5), (1, -1.5))],
          sum(f * O.rms(two[:, :, i].double().sum(0), eps) * gains[i].double() for i, f in ((0, 0.5), (1, -1.5))))


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_first_boundary(dtype):
    from b200serve.ops import sandwich as S
    width, ld, vocab, n = 90, 128, 25, 12
    table, nxt = torch.randn(vocab, width, generator=gen(3)).to(dtype), torch.randn(width, generator=gen(4))
    tok, flag = torch.randint(0, vocab, (n,), generator=gen(5)), torch.zeros(1, dtype=torch.int32, device=DEV)
    tok[:2] = torch.tensor([vocab - 1, 0])
    out = lambda t: torch.full((n, ld), float("nan"), dtype=t, device=DEV)         # noqa: E731
    xo, h = out(F32), out(dtype)
    emb = pad_cols(table, ld).to(DEV)
    run = lambda t: S.boundary([S.source(emb, ld, row_of=i32(t), factor=3.0)], m=n, width=width, groups=5, eps=1e-5, post=None,   # noqa: E731
                               next=pad_cols(nxt, ld).to(DEV), x_in=None, x_out=xo, h=h, vocab=vocab, flag=flag)
    run(tok)
    x = table[tok].double() * 3
    assert rel(xo[:, :width], x) < 1e-6 and rel(h[:, :width], O.group_norm(x, nxt.double(), 1e-5, 5)) < (1e-5 if dtype == F32 else 5e-3) and int(flag) == 0
    bad = tok.clone()
    bad[4] = vocab               # outside: reads row 0, and says so
    run(bad)
    assert int(flag) == 1 and rel(xo[4, :width], table[0].double() * 3) < 1e-6


# ------------------------------------------------------------------ feed-forwards
def test_squared_relu_products():
    from b200serve.ops import gemm as G, latent as L
    k, n = 192, 160
    w = torch.randn(n, k, generator=gen(1)) * 0.2
    for m in (1, 7, 16, 40, 300):
        x = torch.randn(m, k, generator=gen(m))
        out = torch.full((m, n), float("nan"), device=DEV)
        L.linear_f32(x.to(DEV), w.to(DEV), out, m, squared=True)
        assert rel(out, O.relu2(x.double() @ w.double().T)) < 1e-5
        xb, wb, ob = x.bfloat16().to(DEV), w.bfloat16().to(DEV), torch.full((m, n), float("nan"), dtype=BF16, device=DEV)
        if m <= 16:
            L.gemv_bf16(wb, xb, ob, m, n, k, epi=L.EPI_RELU2)
        else:
            G.gemm_bf16(xb, wb, ob, epi=G.EPI_RELU2)
        ref = O.relu2(xb.double().cpu() @ wb.double().cpu().T)
        assert rel(ob, ref) < 5e-3 and torch.equal(ob.cpu() == 0, ref.bfloat16() == 0)


@pytest.mark.parametrize("experts,top,ff,shared", [(12, 3, 80, 150), (5, 5, 64, 64), (9, 1, 128, 0), (40, 2, 200, 100), (64, 8, 72, 700)])
@pytest.mark.parametrize("m", [1, 4, 5, 16, 17, 150])
def test_routed_and_shared_experts(experts, top, ff, shared, m):
    """The feed-forward of a layer through its GEMV, sorted and 32-bit forms, and the boundary that weighs its slots."""
    from b200serve.models.listed import ListedLayers, ListedScratch, assemble, tensor_shapes
    from b200serve.ops import sandwich as S
    width = 130
    f = ExpertFfn(experts, top, ff, "softmax", relu2=True, shared=shared)
    cfg = listed_config("ffn", "Vogerax", (LayerSpec(GroupedAttention(1, 1, 8, 8, 1.0, rot=Rotary(8, 10.0), tied=True), f),), width, 20, 1e-5, SandwichBlock(2))
    raw = {n: torch.randn(s, generator=gen(len(n))) * (s[1] ** -0.5 if len(s) > 1 else 1.0) for n, s in tensor_shapes(cfg).items()}
    raw = {n: t.bfloat16().float() for n, t in raw.items()}
    raw["l0.mlp.router"] *= 4
    h = torch.randn(m, width, generator=gen(m)).bfloat16()
    js = cfg.to_listed_config()["layers"][0]["mlp"]
    y = O.routed({k: v.double() for k, v in raw.items()}, "l0.mlp.", js, h.double())
    ones = torch.ones(width, dtype=F64)
    for dtype in (F32, BF16):
        ll = ListedLayers(assemble(cfg, lambda n: raw[n], DEV, dtype), 64)
        sc = ListedScratch(torch.device(DEV), dtype)
        sc.get("h", m, ll.wp).copy_(pad_cols(h.float(), ll.wp))
        x = torch.zeros(m, ll.wp, device=DEV)
        w = pad_cols(torch.ones(width), ll.wp).to(DEV)
        S.boundary([S.source(**ll.experts(sc, f, ll.w.layers[0].moe, m))], m=m, width=width, groups=1, eps=0.0, post=w, next=w, x_in=x, x_out=x,
                   h=torch.empty(m, ll.wp, dtype=dtype, device=DEV))
        # rounding may only swap experts whose scores are that close
        assert worst_row(x[:, :width], O.group_norm(y, ones, 0.0, 1)) < (2e-5 if dtype == F32 else 0.03), dtype


# ------------------------------------------------------------------ what attention caches
# (heads, kv heads, dim, vdim, rotated dims): one, a few and more than sixteen heads on a key head
CACHED = [(6, 2, 40, 72, 24), (4, 4, 128, 128, 128), (18, 1, 72, 136, 2), (1, 1, 200, 40, 100), (3, 3, 16, 256, 16), (2, 1, 300, 520, 300)]


@pytest.mark.parametrize("shape", CACHED)
@pytest.mark.parametrize("kind", ["gated", "tied"])
@pytest.mark.parametrize("pool", [0, 1, 3, 16, 20])
def test_what_the_cache_holds(shape, kind, pool):
    """Norms, rotations, gates and pooled blocks of several requests in one step, whose earlier positions came with other steps."""
    from b200serve.models.grouped import GroupedGeometry
    from b200serve.models.weights import GroupedWeights
    from b200serve.ops import paged as P
    heads, kv, dim, vdim, rd = shape
    tied = kind == "tied"
    vdim = dim if tied else vdim
    a = GroupedAttention(heads, kv, dim, vdim, 1.0, rot=Rotary(rd, 1e4), qk_norm=not tied, tied=tied, rot_values=not tied, gate=not tied,
                         window=1 if pool else 0, pool=pool)
    g, eps, slots, blocks = GroupedGeometry.of(a), 0.1, 4, 6
    steps = [[(2, 0, 37), (0, 0, 5)], [(0, 5, 1), (2, 37, 1), (3, 0, 1)], [(3, 1, 2), (0, 6, 30), (2, 38, 3)], [(0, 36, 1), (3, 3, 40), (2, 41, 22)]]
    ends = {2: 63, 0: 37, 3: 43}
    gsd = gen(heads + dim)
    raw = {s: {n: torch.randn(t, c, d, generator=gsd) for n, c, d in (("q", heads, dim), ("k", kv, dim), ("v", kv, vdim), ("g", heads, vdim))}
           for s, t in ends.items()}
    qn, kn = torch.rand(dim, generator=gsd) + 0.5, torch.rand(dim, generator=gsd) + 0.5
    ok, ov = order(rd, dim), order(rd, dim) if tied else order(vdim, vdim)
    vec = lambda t: None if tied else pad_cols(t[ok], g.dk).to(DEV)                 # noqa: E731
    w = GroupedWeights(None, None, None, None, None, vec(qn), vec(kn))
    bt = (torch.randperm(slots * blocks, generator=gsd) + 1).view(slots, blocks).to(torch.int32).to(DEV).contiguous()
    freq = O.frequencies(rd, 1e4)
    vfreq = O.frequencies(vdim, 1e4)

    def reference(s):
        pos, r = torch.arange(ends[s]), {n: t.double() for n, t in raw[s].items()}
        q, k, v = r["q"], r["k"], r["k"] if tied else O.rotate(r["v"], pos, vfreq)
        if not tied:
            q, k = O.rms(q, eps) * qn.double(), O.rms(k, eps) * kn.double()
        return O.rotate(q, pos, freq)[..., ok], O.rotate(k, pos, freq)[..., ok], v[..., ov], torch.sigmoid(r["g"])[..., ov]
    ref = {s: reference(s) for s in ends}
    for dtype, tol in ((F32, 1e-5), (BF16, 4e-3)):
        planes = {n: torch.full((slots * blocks + 1, kv, 16 if len(n) == 1 else a.pool_slots, g.dk if n[-1] == "k" else g.dv), float("nan"), dtype=dtype, device=DEV)
                  for n in ("k", "v") + (("pk", "pv") if pool else ())}
        got_q, got_g = {s: [] for s in ends}, {s: [] for s in ends}
        for i, runs in enumerate(steps):
            at = runs_rows(runs)
            m, sl = len(at), 1 if len(at) > 16 else 2 + i % 2
            cols = []
            for s, p in at:
                r = raw[s]
                row = [pad_cols(r["q"][p][:, ok], g.dk).flatten(), pad_cols(r["k"][p][:, ok], g.dk).flatten()]
                if not tied:
                    row += [pad_cols(r["v"][p][:, ov], g.dv).flatten(), pad_cols(r["g"][p][:, ov], g.dv).flatten()]
                cols.append(torch.cat(row + [torch.full((8,), 7.0)]))
            part = slices_of(torch.stack(cols), sl, seed=i).view(sl * m, -1)
            gate = None if tied else torch.full((m, heads * g.dv), float("nan"), dtype=dtype, device=DEV)
            extra = P.Extra(tables(freq, 64), None if tied else tables(vfreq, 64), tied, gate, g.nq + g.nkv, a.window, pool, planes.get("pk"), planes.get("pv"))
            q = torch.full((m, g.nq), float("nan"), dtype=dtype, device=DEV)
            P.norm(part, sl, m, g, a, w, eps, i32([s for s, _ in at]), i32([p for _, p in at]), bt, q, planes["k"], planes["v"], extra)
            for j, (s, _) in enumerate(at):
                got_q[s].append(q[j].view(heads, g.dk))
                if not tied:
                    got_g[s].append(gate[j].view(heads, g.dv))
        for s, n in ends.items():
            q, k, v, gt = ref[s]
            assert rel(torch.stack(got_q[s])[..., :dim], q) < tol and torch.all(torch.stack(got_q[s])[..., dim:] == 0)
            if not tied:
                assert rel(torch.stack(got_g[s])[..., :vdim], gt) < tol
            kk, vv = (torch.stack([planes[x][int(bt[s, p // 16]), :, p % 16] for p in range(n)]) for x in "kv")
            assert rel(kk[..., :dim], k) < tol and rel(vv[..., :vdim], v) < tol and torch.all(kk[..., dim:] == 0) and torch.all(vv[..., vdim:] == 0)
            for b in range(n // pool if pool else 0):       # means of what the cache holds, exactly those
                e = b * pool + pool - 1
                for held, x in ((kk, "pk"), (vv, "pv")):
                    have = planes[x][int(bt[s, e // 16]), :, (e % 16) // pool]
                    want = held[b * pool: e + 1].double().mean(0)
                    assert float((have.double() - want).abs().max()) <= 2e-6 * float(want.abs().max()) + float(want.abs().max()) * (0 if dtype == F32 else 2 ** -8)


# ------------------------------------------------------------------ attention
class Attn:
    """Cached keys and values of two requests behind a scattered page table, with their pooled blocks."""

    def __init__(self, shape, n, dtype, window=0, pool=0, turned=False, gate=False, sink=False, seed=0):
        from b200serve.models.grouped import GroupedGeometry
        g = gen(seed)
        heads, kv, dim, vdim = shape
        self.a = a = GroupedAttention(heads, kv, dim, vdim, 0.8 * dim ** -0.5, window=window, pool=pool)
        self.g, self.n, self.dtype, self.turned, self.gated = GroupedGeometry.of(a), n, dtype, turned, gate
        blocks = (n + 15) // 16
        self.bt = (torch.randperm(2 * blocks, generator=g) + 1).view(2, blocks).to(torch.int32).to(DEV).contiguous()
        self.k, self.v = torch.randn(2, n, kv, dim, generator=g).to(dtype), torch.randn(2, n, kv, vdim, generator=g).to(dtype)
        self.sink = torch.rand(heads, generator=g) * 4 if sink else None
        self.rest = 3e4            # what unseen blocks and keys hold: it would show
        self.turn = O.frequencies(vdim, 500.0) if turned else None
        self.fill()

    def fill(self):
        a, g, n = self.a, self.g, self.n
        pages = self.bt.numel() + 1
        self.kc, self.vc = (torch.zeros(pages, a.kv_heads, 16, c, dtype=self.dtype, device=DEV) for c in (g.dk, g.dv))
        for r in range(2):
            page, off = self.bt[r].long()[torch.arange(n, device=DEV) // 16], torch.arange(n, device=DEV) % 16
            self.kc[page, :, off, : a.dim], self.vc[page, :, off, : a.vdim] = self.k[r].to(DEV), self.v[r].to(DEV)
        self.pk = self.pv = None
        if a.pool:
            # blocks of their own, so that a block read in a token's place (or the other way) shows
            nb = n // a.pool
            g2 = gen(77)
            self.bk, self.bv = torch.randn(2, nb, a.kv_heads, a.dim, generator=g2).to(self.dtype), torch.randn(2, nb, a.kv_heads, a.vdim, generator=g2).to(self.dtype)
            self.pk, self.pv = (torch.zeros(pages, a.kv_heads, a.pool_slots, c, dtype=self.dtype, device=DEV) for c in (g.dk, g.dv))
            self.put_blocks()

    def put_blocks(self):
        a = self.a
        e = (torch.arange(self.n // a.pool, device=DEV) + 1) * a.pool - 1
        for r in range(2):
            page, slot = self.bt[r].long()[e // 16], (e % 16) // a.pool
            self.pk[page, :, slot, : a.dim], self.pv[page, :, slot, : a.vdim] = self.bk[r].to(DEV), self.bv[r].to(DEV)

    def reference(self, q, req, pos, gate):
        a, out = self.a, {}
        for r in sorted(set(req)):
            i = [j for j, x in enumerate(req) if x == r]
            p = torch.tensor([pos[j] for j in i])
            k, v, seen = self.k[r].double(), self.v[r].double(), O.causal(p, self.n)
            if a.window:
                seen, far = O.window_and_blocks(p, self.n, a.window, a.pool or self.n + 1)
                if a.pool:
                    k, v, seen = torch.cat([k, self.bk[r].double()]), torch.cat([v, self.bv[r].double()]), torch.cat([seen, far], dim=1)
            o = O.attend(q[i].double(), k, v, seen, a.scale, None if self.sink is None else self.sink.double())
            if self.turned:            # kernel order: neighbours
                ov = order(a.vdim, a.vdim)
                inv = torch.argsort(torch.tensor(ov))
                o = O.rotate(o[..., inv], -p, self.turn)[..., ov]
            out.update(zip(i, o))
        o = torch.stack([out[j] for j in range(len(req))])
        return o * gate.double() if self.gated else o

    def extra(self, gate):
        from b200serve.ops import paged as P
        a, rows = self.a, None
        if self.gated:
            rows = torch.zeros(len(gate), self.g.heads * self.g.dv + 32, dtype=self.dtype, device=DEV)      # rows inside wider ones
            rows[:, : self.g.heads * self.g.dv] = pad_cols(gate, self.g.dv).flatten(1).to(self.dtype)
        return P.Extra(None, tables(self.turn, self.n) if self.turned else None, False, rows, 0, a.window, a.pool, self.pk, self.pv)

    def padded_q(self, q):
        return pad_cols(q.to(self.dtype).float(), self.g.dk).to(self.dtype).view(len(q), -1).to(DEV).contiguous()

    def out(self, m):
        wide = torch.full((m, self.g.heads * self.g.dv + 64), float("nan"), dtype=self.dtype, device=DEV)
        return wide, wide[:, : self.g.heads * self.g.dv]

    def cut(self, wide, mult):
        v = wide[:, : self.g.heads * self.g.dv].reshape(len(wide), self.g.heads, self.g.dv)
        assert torch.all(v[..., self.a.vdim:] == 0) and torch.all(torch.isnan(wide[:, self.g.heads * self.g.dv:]))
        return v[..., : self.a.vdim].float() / mult

    def sink2(self):
        return None if self.sink is None else (self.sink * 1.4426950408889634).to(DEV)

    def rows(self, q, req, pos, gate, nsplit=0, mult=0.5):
        from b200serve.ops import paged as P
        g, m = self.g, len(pos)
        wide, out = self.out(m)
        args = (self.padded_q(q), self.kc, self.vc, m, g, i32(req), i32(pos), self.bt)
        more = dict(mult=mult, extra=self.extra(gate))
        if nsplit:
            op, ml = (torch.full((m * nsplit * g.heads, c), float("nan"), device=DEV) for c in (g.dv, 2))
            P.rows(*args, nsplit, 0, self.a.scale, None, self.sink2(), op, ml, out, **more)
        else:
            P.simple(*args, 0, self.a.scale, None, self.sink2(), out, **more)
        return self.cut(wide, mult)

    def segments(self, q, segs, gate, mult=2.0):
        from b200serve.ops import paged as P
        from b200serve.runtime.batch import segment_blocks, segment_tiles
        a, g, per = self.a, self.g, P.segments_per_tile(self.g)
        pooled = None
        if a.window:
            tiles, first, preq, block = segment_blocks(segs, a.window, a.pool, per)
            if len(block):
                pk, pv = (torch.full((len(block), g.kv_heads * c), float("nan"), dtype=BF16, device=DEV) for c in (g.dk, g.dv))
                P.pool_gather(i32(preq), i32(block), len(block), g, self.bt, a.pool, self.pk, self.pv, pk, pv)
                pooled = (pk, pv, i32(first))
        else:
            tiles = segment_tiles(segs, 0, per)
        wide, out = self.out(len(q))
        P.attn_segments(self.padded_q(q), self.kc, self.vc, self.bt, out, i32(tiles).view(-1), len(tiles), len(q), g, a.scale, 0, None,
                        self.sink2(), mult=mult, extra=self.extra(gate), pooled=pooled)
        return self.cut(wide, mult)

    def spike(self, q, row, req, key, over=9.0, block=False):
        """Makes every head's score at one key (or block) stand out."""
        a = self.a
        kk = (self.bk if block else self.k)[req, key].double().repeat_interleave(a.heads // a.kv_heads, dim=0)
        q[row] = (over / a.scale * kk / kk.pow(2).sum(-1, keepdim=True)).float()

    def gates(self, m):
        return torch.rand(m, self.a.heads, self.a.vdim, generator=gen(9)).to(self.dtype).float()


SHAPES = [(6, 2, 40, 72), (4, 4, 128, 128), (18, 1, 72, 136), (1, 1, 200, 40), (40, 2, 64, 192), (3, 3, 16, 256), (8, 4, 256, 130)]
MASKS = [(70, 6), (16, 16), (33, 20), (1, 1), (48, 8), (100, 0), (130, 40)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,pool", MASKS)
def test_windowed_rows(shape, window, pool):
    """Every row asks for one key or block just inside or just outside of what it sees."""
    cases = []              # (position, request, key, is it a block)
    for i, pos in enumerate((0, 15, 16, 95, 160, 255, 298, 299)):
        r, lo = i % 2, max(0, pos - window + 1)
        cases += [(pos, r, k, False) for k in (pos, lo, lo - 1, 0) if k >= 0]
        if pool:
            seen = lo // pool
            cases += [(pos, r, b, True) for b in (0, seen - 1, seen) if 0 <= b < 300 // pool]
    req, pos = [c[1] for c in cases], [c[0] for c in cases]
    for dtype, splits in ((BF16, (0, 1, 3, 32)), (F32, (0,))):
        t = Attn(shape, 300, dtype, window, pool, seed=shape[0])
        q = torch.randn(len(cases), t.a.heads, t.a.dim, generator=gen(3))
        for i, (_, r, key, block) in enumerate(cases):
            t.spike(q, i, r, key, block=block)
        q, gate = q.to(dtype).float(), t.gates(len(cases))
        ref = t.reference(q, req, pos, gate)
        for ns in splits:
            got = t.rows(q, req, pos, gate, ns)
            for i in range(len(cases)):
                assert rel(got[i], ref[i]) < (2e-5 if dtype == F32 else 0.02), (dtype, ns, cases[i])


@pytest.mark.parametrize("shape", SHAPES + [(2, 1, 192, 64), (2, 2, 130, 200), (2, 1, 64, 64), (4, 2, 190, 192), (2, 1, 256, 180)])
@pytest.mark.parametrize("window,pool", [(70, 6), (16, 16), (200, 4), (300, 0), (1, 1), (129, 40)])
def test_windowed_prompt_segments(shape, window, pool):
    t = Attn(shape, 600, BF16, window, pool, seed=shape[2])
    segs = [(0, 0, 300), (1, 217, 37), (0, 300, 290)]
    at = runs_rows(segs)
    q = torch.randn(len(at), t.a.heads, t.a.dim, generator=gen(5))
    for row in range(3, len(at), 7):                # inside and outside of both edges, in turn
        r, pos = at[row]
        lo = max(0, pos - window + 1)
        seen = lo // pool if pool else 0
        options = [(k, False) for k in (lo, lo - 1, pos) if k >= 0] + [(b, True) for b in (seen - 1, seen, 0) if pool and 0 <= b < 600 // pool]
        key, block = options[row % len(options)]
        t.spike(q, row, r, key, block=block)
    q, gate = q.bfloat16().float(), t.gates(len(at))
    got, ref = t.segments(q, segs, gate), t.reference(q, [r for r, _ in at], [p for _, p in at], gate)
    assert rel(got, ref) < 8e-3 and worst_row(got, ref) < 0.04


@pytest.mark.parametrize("shape", SHAPES + [(2, 2, 130, 200), (4, 2, 48, 34)])
def test_rotated_values_sinks_and_gates(shape):
    """Results turned back by the row's position, gated, with a sink per head; each alone and together."""
    for turned, gate, sink in ((True, True, True), (True, False, False), (False, True, False), (False, False, True)):
        t = Attn(shape, 300, BF16, turned=turned, gate=gate, sink=sink, seed=shape[1])
        pos, req = [0, 1, 15, 17, 49, 130, 299, 298], [0, 1, 0, 1, 0, 1, 0, 1]
        q = torch.randn(len(pos), t.a.heads, t.a.dim, generator=gen(3))
        t.spike(q, 5, 1, 0)
        t.spike(q, 6, 0, 16)
        q, gates = q.bfloat16().float(), t.gates(len(pos))
        ref = t.reference(q, req, pos, gates)
        for ns in (0, 1, 3, 32):
            assert worst_row(t.rows(q, req, pos, gates, ns), ref) < 0.02, (turned, gate, sink, ns)
        segs = [(1, 0, 150), (0, 170, 130)]
        at = runs_rows(segs)
        q, gates = torch.randn(280, t.a.heads, t.a.dim, generator=gen(5)).bfloat16().float(), t.gates(280)
        got, ref = t.segments(q, segs, gates), t.reference(q, [r for r, _ in at], [p for _, p in at], gates)
        assert rel(got, ref) < 8e-3 and worst_row(got, ref) < 0.03, (turned, gate, sink)
        t = Attn(shape, 100, F32, turned=turned, gate=gate, sink=sink, seed=shape[1])
        q, gates = torch.randn(6, t.a.heads, t.a.dim, generator=gen(3)), t.gates(6)
        pos = [0, 1, 15, 16, 64, 99]
        assert rel(t.rows(q, [1] * 6, pos, gates), t.reference(q, [1] * 6, pos, gates)) < 1e-5


def test_far_blocks_among_hundreds():
    """One block thousands of positions back carries the row's weight; its neighbours and the tokens around it do not."""
    t = Attn((32, 8, 64, 64), 2500, BF16, 128, 8, seed=2)
    pos, blocks = [2499, 2400, 2048, 1300], [3, 1, 16, 100]
    q = torch.randn(4, 32, 64, generator=gen(1)) * 0.2
    for i in range(4):
        t.spike(q, i, 1, blocks[i], over=14.0, block=True)
    q, gate = q.bfloat16().float(), t.gates(4)
    ref = t.reference(q, [1] * 4, pos, gate)
    for ns in (0, 1, 9, 40):
        assert worst_row(t.rows(q, [1] * 4, pos, gate, ns), ref) < 0.02
    qs = torch.randn(100, 32, 64, generator=gen(6)) * 0.2
    for row, b in ((99, 5), (0, 63), (50, 64), (98, (2498 - 127) // 8 - 1)):
        t.spike(qs, row, 1, b, over=14.0, block=True)
    qs, gate = qs.bfloat16().float(), t.gates(100)
    assert worst_row(t.segments(qs, [(1, 2400, 100)], gate), t.reference(qs, [1] * 100, list(range(2400, 2500)), gate)) < 0.03


# ------------------------------------------------------------------ retention
# (heads, dim, vdim, rotated dims): value dims of one CTA and of several, key dims beyond the tensor-core form
CELLS = [(3, 56, 40, 32), (2, 128, 128, 128), (1, 64, 200, 64), (2, 200, 128, 24), (4, 16, 384, 8), (2, 130, 64, 130), (1, 96, 512, 0), (2, 300, 100, 40), (1, 400, 64, 2)]


class Cell:
    def __init__(self, shape, slots=4, decay=None, eps=0.05):
        from b200serve.models.retention import RetentionGeometry
        h, dim, vdim, rd = shape
        decay = decay or [1 - 2.0 ** -(1 + 2 * i) for i in range(h)]
        self.a, self.eps = Retention(h, dim, vdim, tuple(decay), Rotary(rd, 300.0)), eps
        self.g = RetentionGeometry.of(self.a)
        self.rope = tables(O.frequencies(rd, 300.0), 1024) if rd else (torch.zeros(1024, 0, device=DEV),) * 2
        self.decay = torch.tensor(decay, dtype=F64)
        self.table = torch.stack([self.decay, torch.log2(self.decay)]).float().to(DEV)
        self.state = torch.full((slots, h * self.g.dk * self.g.dv), float("nan"), device=DEV)      # a sequence starts from zeros by itself

    def inputs(self, t, seed):
        a, g = self.a, gen(seed)
        return {n: torch.randn(t, a.heads, d, generator=g) for n, d in (("q", a.dim), ("k", a.dim), ("v", a.vdim), ("g", a.vdim))}

    def reference(self, x):
        a, pos, d = self.a, torch.arange(len(x["q"])), {n: t.double() for n, t in x.items()}
        f = O.frequencies(a.rot.dims, 300.0)
        o, s = O.retention_scan(O.rotate(d["q"], pos, f), O.rotate(d["k"], pos, f) * a.dim ** -0.5, d["v"], self.decay)
        return O.rms(o, self.eps) * O.silu(d["g"]), s

    def part(self, x, rows, slices, before=4):
        """The projection's slices for rows of ``x``, with other columns around them."""
        a, g, ok = self.a, self.g, order(self.a.rot.dims, self.a.dim)
        cols = [torch.full((len(rows), before), 9.0)]
        for n, pad in (("q", g.dk), ("k", g.dk), ("v", g.dv), ("g", g.dv)):
            t = torch.stack([x[r][n][p] for r, p in rows])
            cols.append(pad_cols(t[..., ok] if n in "qk" else t, pad).flatten(1))
        return slices_of(torch.cat(cols + [torch.full((len(rows), 8), 9.0)], dim=1), slices).view(slices * len(rows), -1)

    def run(self, x, runs, dtype, chunked, slices=1, mult=1.5):
        from b200serve.ops import retention as R
        from b200serve.runtime.batch import ChunkPlan, segment_chunks
        a, g, rows = self.a, self.g, runs_rows(runs)
        m, req, pos = len(rows), i32([r for r, _ in rows]), i32([p for _, p in rows])
        wide = torch.full((m, g.heads * g.dv + 64), float("nan"), dtype=dtype, device=DEV)
        out = wide[:, : g.heads * g.dv]
        part = self.part(x, rows, slices)
        if chunked:
            per = R.chunk_rows()
            segs, chunks = segment_chunks(runs, per)
            t = ChunkPlan(len(segs), i32(segs).view(-1), chunks, max((s[1] + per - 1) // per for s in segs))
            kv = torch.full((chunks, g.heads * g.dk * g.dv), float("nan"), device=DEV)
            raw = torch.full((m, g.heads * g.dv), float("nan"), device=DEV) if R.wants_raw(g) else None
            R.segments(part, m, 4, g, a, t, pos, self.rope, self.eps, mult, self.table, self.state, kv, raw, out)
        else:
            R.step(part, slices, m, 4, g, a, req, pos, self.rope, self.eps, mult, self.table, self.state, out)
        v = out.reshape(m, g.heads, g.dv)
        assert torch.all(v[..., a.vdim:] == 0) and torch.all(torch.isnan(wide[:, g.heads * g.dv:]))
        return v[..., : a.vdim].float() / mult

    def held(self, slot):
        a, g, ok = self.a, self.g, order(self.a.rot.dims, self.a.dim)
        return self.state[slot].view(g.heads, g.dk, g.dv)[:, : a.dim, : a.vdim].cpu()[:, torch.argsort(torch.tensor(ok))]


@pytest.mark.parametrize("shape", CELLS)
def test_retention_token_by_token(shape):
    c = Cell(shape)
    ends = {0: 40, 2: 9, 3: 25}
    x = {s: c.inputs(n, s) for s, n in ends.items()}
    ref = {s: c.reference(x[s]) for s in ends}
    for dtype, tol in ((F32, 1e-5), (BF16, 5e-3)):
        got = {s: [] for s in ends}
        for i, runs in enumerate(([(2, 0, 4), (0, 0, 1)], [(0, 1, 20), (3, 0, 1), (2, 4, 5)], [(3, 1, 24), (0, 21, 19)])):
            o, j = c.run(x, runs, dtype, False, 1 + 2 * i), 0
            for s, _, n in runs:
                got[s].append(o[j: j + n])
                j += n
        for s in ends:
            assert worst_row(torch.cat(got[s]), ref[s][0]) < 3 * tol and rel(torch.cat(got[s]), ref[s][0]) < tol
            assert rel(c.held(s), ref[s][1]) < 1e-5
        assert torch.all(torch.isnan(c.state[1]))


@pytest.mark.parametrize("shape", [s for s in CELLS if s[1] <= 256])
@pytest.mark.parametrize("cuts", [(400,), (128, 129, 143), (32, 2, 33, 100, 1, 232), (1, 399)])
def test_retention_in_chunks(shape, cuts):
    """Segments of several requests side by side, cut at and off the chunks' edges, with tokens in between."""
    c = Cell(shape)
    x = {s: c.inputs(400, 10 + s) for s in (0, 3)}
    x[1] = c.inputs(150, 5)
    ref = {s: c.reference(x[s]) for s in x}
    got, at = {s: [] for s in x}, 0
    for i, n in enumerate(cuts):
        runs = [(3, at, n)] + ([(1, 0, 150)] if i == 0 else []) + [(0, at, n)]
        o, j = c.run(x, runs, BF16, n > 2), 0
        for s, _, k in runs:
            got[s].append(o[j: j + k])
            j += k
        at += n
    for s in x:
        assert rel(torch.cat(got[s]), ref[s][0]) < 5e-3 and worst_row(torch.cat(got[s]), ref[s][0]) < 0.02
        assert rel(c.held(s), ref[s][1]) < 5e-3         # values are bf16


def test_decays_at_their_ends():
    """No decay at all, hardly any, nearly everything and everything at once: exact powers whatever the distance."""
    decay = [1.0, 1 - 2.0 ** -14, 0.01, 0.0]
    for chunked, dtype in ((False, F32), (True, BF16)):
        c = Cell((4, 64, 64, 64), decay=decay)
        x = {0: c.inputs(300, 1)}
        ref, state = c.reference(x[0])
        got = torch.cat([c.run(x, [(0, 0, 257)], dtype, chunked), c.run(x, [(0, 257, 43)], dtype, chunked)])
        for h in range(4):
            assert worst_row(got[:, h], ref[:, h]) < (2e-5 if dtype == F32 else 0.02), h
            assert rel(c.held(0)[h], state[h]) < (1e-5 if dtype == F32 else 5e-3), h


def test_a_far_token_in_the_state():
    """One loud token hundreds of rows back, asked for by a late query: its weight is the decay to the power of the distance."""
    c = Cell((2, 64, 128, 0), decay=[0.999, 0.99], eps=1e-12)
    x = {0: c.inputs(500, 3)}
    for n in "kv":
        x[0][n] *= 1e-3
    x[0]["k"][37], x[0]["v"][37] = torch.randn(2, 64, generator=gen(1)), torch.randn(2, 128, generator=gen(2))
    x[0]["q"][400:] = x[0]["k"][37]
    ref, _ = c.reference(x[0])
    got = c.run(x, [(0, 0, 500)], BF16, True)
    assert worst_row(got[400:], ref[400:]) < 0.01


# ------------------------------------------------------------------ whole models
def att(h, g, dim, scale, rot, window, pool):
    return GroupedAttention(h, g, dim, dim, scale, rot=rot, tied=True, window=window, pool=pool)


def par(h, g, dim, vdim, scale, rot, right):
    return ParallelMixer(GroupedAttention(h, g, dim, vdim, scale, sink=True, qk_norm=True, rot=rot, rot_values=True, gate=True), right, 0.5, 0.5, True)


def odd_config():
    """Sizes that fit no tile, single heads, heads outside the tensor-core forms, a window of one position, blocks longer than a
    page, pairs of one dimension, weights used by earlier and by several layers, unequal output projections."""
    a = att(5, 1, 24, 0.3, Rotary(2, 50.0, 3.0), 1, 5)
    b = par(3, 3, 300, 270, 0.06, Rotary(100, 1e4, 2.0, 40, 8.0, 1.0), Retention(1, 24, 34, (0.93,), Rotary(24, 100.0)))
    return listed_config("vogerax-odd", "Vogerax", (
        LayerSpec(a, None, 2), LayerSpec(b, DenseFfn(40, relu2=True)), LayerSpec(a, None), LayerSpec(att(18, 1, 300, 0.05, Rotary(300, 1e3, 1.0), 45, 37), ExpertFfn(5, 5, 24, relu2=True, score="softmax", shared=200)),
        LayerSpec(b, DenseFfn(40, relu2=True), 1), LayerSpec(a, None, 0),
        LayerSpec(par(20, 1, 34, 10, 0.4, Rotary(6, 1e4, 16.0, 64, 4.0, 0.5), Retention(3, 270, 150, (0.5, 0.99, 1.0), Rotary(200, 1e4, 5.0))), None)),
        150, 333, 1e-3, SandwichBlock(15, 0.3))


def one_config():
    """As small as it gets: one group, one expert, blocks of one position, equal sizes."""
    return listed_config("vogerax-one", "Vogerax", (
        LayerSpec(att(2, 2, 64, 0.2, Rotary(64, 1e4), 64, 1), ExpertFfn(1, 1, 64, relu2=True, score="softmax", shared=64)),
        LayerSpec(par(2, 2, 64, 64, 0.2, Rotary(64, 1e4), Retention(2, 64, 64, (0.9, 0.99), Rotary(64, 1e4))), ExpertFfn(8, 1, 64, relu2=True, score="softmax"))),
        64, 100, 1e-5, SandwichBlock(1, 1.0))


def wide_config():
    """Heads of several blocks, a plain window, full attention whose values are the keys, more experts than a step has rows."""
    return listed_config("vogerax-wide", "Vogerax", (
        LayerSpec(att(4, 2, 190, 0.1, Rotary(64, 1e5, 4.0), 90, 0), ExpertFfn(48, 6, 100, relu2=True, score="softmax", shared=90)),
        LayerSpec(par(6, 2, 130, 128, 0.1, Rotary(130, 1e4, 4.0, 100), Retention(4, 128, 192, (0.97, 0.8, 0.99, 0.999), Rotary(128, 1e5))), DenseFfn(300, relu2=True)),
        LayerSpec(att(4, 4, 64, 0.15, Rotary(32, 1e4), 0, 0), None), LayerSpec(att(8, 2, 96, 0.12, Rotary(96, 1e4, 2.0), 100, 12), DenseFfn(64, relu2=True))),
        1280, 211, 1e-6, SandwichBlock(5, 20.0))


def lively(name, t):
    """Random weights that make the mechanisms matter: peaked attention near and far, sinks that take a share, gates that open and
    close, norms and routers with character."""
    last, g = name.rsplit(".", 1)[-1], gen(len(name) + t.numel())
    uni = lambda lo, hi: lo + (hi - lo) * torch.rand(t.shape, generator=g)         # noqa: E731
    if last == "sink":
        return uni(-1.0, 4.0)
    if last == "norm" and ".left." in name:
        return uni(0.7, 2.0)
    if last in ("norm1b", "norm2b", "out"):
        return uni(-1.0, 1.0)
    if last in ("q", "k") and ".left." not in name:
        return t * 1.6
    return t * 2.0 if last == "router" else t


class Model:
    def __init__(self, cfg, path):
        from b200serve.utils.synth import write_listed
        self.cfg, self.json, self.path = cfg, cfg.to_listed_config(), str(path / "snap")
        self.w = {k: v.double() for k, v in write_listed(cfg, self.path, seed=len(cfg.name), make=lively).items()}
        self.weights, self.known = {}, {}

    def logits(self, ids):
        key = tuple(ids)
        if key not in self.known:
            self.known[key] = O.forward(self.w, self.json, list(ids))
        return self.known[key]

    def engine(self, dtype, max_seqs=4, max_len=512, num_pages=None, **kw):
        from b200serve.loader.loader import load
        from b200serve.runtime.engine import Engine
        if dtype not in self.weights:
            self.weights[dtype] = load(self.path, device=DEV, dtype=dtype, report=None)
        return Engine(self.weights[dtype], max_seqs=max_seqs, max_len=max_len, num_pages=num_pages, **kw)

    def prompt(self, n, seed=0):
        return torch.randint(0, self.cfg.vocab, (n,), generator=gen(1000 * n + seed)).tolist()


@pytest.fixture(scope="module", params=["mini", "odd", "one", "wide"])
def model(request, tmp_path_factory):
    cfg = {"mini": lambda: preset("vogerax-mini"), "odd": odd_config, "one": one_config, "wide": wide_config}[request.param]()
    return Model(cfg, tmp_path_factory.mktemp(request.param))


def close(got, ref, dtype):
    """In bf16 a token whose experts' scores are a rounding apart may go to another expert: a few positions may be further off."""
    got, ref = got.double().cpu(), ref.double()
    r = ((got - ref).pow(2).mean(-1) / ref.pow(2).mean(-1)).sqrt()
    if dtype == "float32":
        assert float(r.max()) < 1e-4, (float(r.max()), int(r.argmax()), float(r.median()))
    else:
        few = torch.sort(r).values[: max(1, int(0.95 * len(r)))]
        assert float(r.median()) < (0.03 if len(r) > 9 else 0.08) and float(few.max()) < 0.12 and float(r.max()) < 0.5, (float(r.max()), int(r.argmax()), float(r.median()))


DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 2, 17, 64, 65, 230])
def test_prompt_in_one_step(model, dtype, n):
    eng = model.engine(dtype)
    ids = model.prompt(n)
    close(eng.forward_batch([(1, ids, list(range(n)))]), model.logits(ids), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_token_by_token_equals_the_prompt(model, dtype):
    ids = model.prompt(230)
    eng = model.engine(dtype)
    lg = torch.cat([eng.forward_batch([(0, [t], [0])]).clone() for t in ids])
    close(lg, model.logits(ids), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2] * 20 + [3, 5, 7, 100, 75], [33, 32, 31, 64, 1, 65, 4], [100, 2, 2, 96, 30], [16, 16, 15, 17, 166], [69, 1, 1, 1, 158]])
def test_portions(model, dtype, cuts):
    ids = model.prompt(230)
    eng = model.engine(dtype)
    out, at = [], 0
    for c in cuts:
        out.append(eng.forward_batch([(2, ids[at: at + c], list(range(c)))]).clone())
        at += c
    assert at == len(ids)
    close(torch.cat(out), model.logits(ids), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_and_reused_pages(model, dtype):
    """Unequal requests in one batch, portions beside decode rows, requests that pause; a pool just large enough, whose
    pages and slots are freed and taken again."""
    eng = model.engine(dtype, num_pages=1 + (512 // 16))
    prompts = [model.prompt(n, seed=n) for n in (200, 35, 90, 3, 150, 61, 1, 120)]
    rng = np.random.default_rng(5)
    live, got, nxt, free = {}, {}, 0, [0, 1, 2, 3]
    used = set()
    while nxt < len(prompts) or live:
        while nxt < len(prompts) and free and sum(len(prompts[i]) + 16 for i, _ in live.values()) + len(prompts[nxt]) < 480:
            live[free.pop(0)] = (nxt, 0)
            got[nxt] = []
            nxt += 1
        batch = []
        for s, (i, at) in list(live.items()):
            if len(live) > 1 and rng.random() < 0.2:
                continue                       # left out of this step
            c = min(len(prompts[i]) - at, int(rng.choice([1, 1, 2, 13, 40, 77])))
            batch.append((s, prompts[i][at: at + c], list(range(c))))
        if not batch:
            continue
        lg, j = eng.forward_batch(batch).clone(), 0
        for s, toks, _ in batch:
            i, at = live[s]
            got[i].append(lg[j: j + len(toks)])
            j += len(toks)
            live[s] = (i, at + len(toks))
            if live[s][1] == len(prompts[i]):
                used.update(eng.pool.table(s))
                eng.reset(s)
                free.append(s)
                del live[s]
    assert len(used) < sum((len(p) + 15) // 16 for p in prompts)       # pages did come back
    for i, p in enumerate(prompts):
        close(torch.cat(got[i]), model.logits(p), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_above_the_runners_limit(model, dtype):
    """A step of more tokens than one batch holds runs as several, in order."""
    eng = model.engine(dtype)
    eng._batch_runner().max_tokens = 96
    a, b, c = model.prompt(150, seed=1), model.prompt(90, seed=2), model.prompt(1, seed=3)
    lg = eng.forward_batch([(0, a, [0, 95, 96, 149]), (3, b, [89, 0]), (1, c, [0])])
    close(lg, torch.cat([model.logits(a)[[0, 95, 96, 149]], model.logits(b)[[89, 0]], model.logits(c)]), dtype)


def near_best(ref, new, dtype):
    """Every token is the reference's choice for the tokens before it, or within rounding of it."""
    gap = ref.max(-1).values - ref[torch.arange(len(new)), torch.tensor(new)]
    if dtype == "float32":
        assert float(gap.max()) < 1e-3
    else:
        assert float(gap.median()) < 0.05 * float(ref.std()) and float(gap.max()) < float(ref.std())


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_greedy_generation(model, dtype):
    """``Engine.generate``: prompt pass, then captured decode steps; the logits of the last step too."""
    ids = model.prompt(70)
    eng = model.engine(dtype)
    new = eng.generate(ids, 130)
    ref = model.logits(ids + new[:-1])[len(ids) - 1:]
    near_best(ref, new, dtype)
    close(eng.logits(1), ref[-1:], dtype)
    assert eng.steps_replayed >= 129


@pytest.mark.parametrize("dtype", DTYPES)
def test_decode_steps_of_several_requests(model, dtype):
    """Captured steps that advance by themselves, requests at different depths."""
    eng = model.engine(dtype)
    prompts = {s: model.prompt(n, seed=s) for s, n in ((0, 100), (2, 7), (3, 63))}
    first = {s: eng.prefill(s, p) for s, p in prompts.items()}
    eng.decode_begin(list(prompts), [first[s] for s in prompts])
    new = {s: [first[s]] for s in prompts}
    for _ in range(20):
        for s, t in zip(prompts, eng.decode_step()):
            new[s].append(t)
    for s, p in prompts.items():
        near_best(model.logits(p + new[s][:-1])[len(p) - 1:], new[s], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_more_requests_than_a_gemv_takes(model, dtype):
    """Thirty requests in one decode step."""
    eng = model.engine(dtype, max_seqs=30, max_len=64)
    prompts = [model.prompt(3 + i, seed=i) for i in range(30)]
    eng.forward_batch([(i, p[:-1], []) for i, p in enumerate(prompts)])
    lg = eng.forward_batch([(i, p[-1:], [0]) for i, p in enumerate(prompts)])
    close(lg, torch.stack([model.logits(p)[-1] for p in prompts]), dtype)


def test_rows_taken_back(model):
    """Rejected rows leave pages, blocks and state as if they had never run, in row steps and in mixed batches."""
    from b200serve.runtime.engine import Row
    ids = model.prompt(120)
    eng = model.engine("float32")
    eng.forward_batch([(0, ids[:100], [])])
    eng.forward_rows([Row(0, 100, ids[100])] + [Row(0, 101 + i, 5 + i) for i in range(8)])
    eng.truncate(0, 101)
    eng.forward_batch([(1, model.prompt(80), []), (0, ids[101:104] + [7, 8], [])])
    eng.truncate(0, 104)
    close(eng.forward_batch([(0, ids[104:], list(range(16)))]), model.logits(ids)[104:], "float32")
    with pytest.raises(NotImplementedError):
        eng.truncate(0, 50)
    eng.truncate(0, 0)
    close(eng.forward_batch([(0, ids[:30], [29])]), model.logits(ids)[29:30], "float32")


def test_saved_sessions(model):
    ids = model.prompt(200)
    eng = model.engine("float32")
    eng.forward_batch([(0, ids[:96], [])])
    blob = eng.save_kv(0, 0, 96)
    eng.reset()
    eng.forward_batch([(1, model.prompt(60), [])])
    eng.load_kv(3, blob)
    close(eng.forward_batch([(3, ids[96:], [103])]), model.logits(ids)[-1:], "float32")


def test_buffers_stay_within_the_planners_figures(model):
    from b200serve.runtime import memory_plan as MP
    from b200serve.runtime.buffer_registry import audit
    for dtype in DTYPES:
        eng = model.engine(dtype)
        for s in range(4):
            eng.prefill(s, model.prompt(40 + s))
        eng.forward_batch([(s, [1, 2, 3], [0]) for s in range(4)])
        audit(eng.model.buf, eng.kv, eng.cfg, eng.kv_dtype, eng.max_seqs)
        eng.forward_batch([(s, model.prompt(60), []) for s in range(4)])
        assert eng._batch_runner().scratch.nbytes <= 4 * MP.prefill_scratch_bytes(eng.cfg, 240, "listed")
        assert all(t.dtype == (F32 if dtype == "float32" else BF16) for t in eng.kv.pages.values())
        assert all(t.dtype == F32 for t in eng.kv.states.values())


@pytest.mark.parametrize("spec", ["off", "lookup"])
def test_served_over_http(model, spec):
    """Concurrent requests through the server: prompt chunks and decode rows share batches, drafts are taken back, tokens
    are the reference's."""
    import http.client
    import threading
    from b200serve.server.adapter import EngineAdapter
    from b200serve.server.app import Server, ServerOptions
    from b200serve.server.chat_template import ChatTemplate
    from b200serve.server.iface import ByteTok
    eng = model.engine("float32")
    adapter = EngineAdapter(eng)
    calls = []
    inner = adapter.step_mixed
    adapter.step_mixed = lambda slot, ids, rows: calls.append((len(ids), len(rows))) or inner(slot, ids, rows)
    srv = Server(adapter, ByteTok(), ChatTemplate(), ServerOptions(model_name="m", prefill_chunk=48, max_queue=8, spec=spec,
                                                                   spec_max=4 if spec != "off" else 0)).start()
    res = {}

    def post(i, ids, extra):
        c = http.client.HTTPConnection("127.0.0.1", srv.port, timeout=60)
        c.request("POST", "/v1/completions", json.dumps({"prompt": ids, "max_tokens": 16, "temperature": 0, "ignore_eos": True,
                                                         "return_token_ids": True, **extra}), {"Content-Type": "application/json"})
        r = c.getresponse()
        res[i] = (r.status, json.loads(r.read().decode()))
        c.close()
    prompts = [(model.prompt(9, seed=3) * 40)[:n] for n in (90, 200, 20, 110)]
    try:
        ts = [threading.Thread(target=post, args=(i, p, {})) for i, p in enumerate(prompts)]
        for t in ts:
            t.start()
        for t in ts:
            t.join()
        for i, p in enumerate(prompts):
            status, body = res[i]
            assert status == 200, body
            new = body["choices"][0]["token_ids"]
            assert len(new) == 16
            near_best(model.logits(p + new[:-1])[len(p) - 1:], new, "float32")
        assert calls
        for i in (10, 11):                     # sampled: the same seed draws the same tokens
            post(i, prompts[0], {"temperature": 0.9, "top_k": 50, "seed": 4})
        assert res[10][1]["choices"][0]["token_ids"] == res[11][1]["choices"][0]["token_ids"]
    finally:
        srv.stop()


def test_trace_replay_program(model, tmp_path):
    """The trace program in a process of its own: admission, a pause, release and reuse of slots, wanted places."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    a, b = model.prompt(90, seed=1), model.prompt(70, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:80], "want": [0, 79]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[80:81], "want": [0]}, {"id": "b", "tokens": b[:67], "want": [66, 5]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[67:], "want": []}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[81:], "want": [8]}, {"id": "c", "tokens": b[:3], "want": [2]}], "end": ["a", "c"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model.path, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = model.logits(a), model.logits(b)
    for i, ref in ((0, la[[0, 79]]), (1, torch.stack([la[80], lb[66], lb[5]])), (3, torch.stack([la[89], lb[2]]))):
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, model.cfg.vocab)
        close(got, ref, "float32")


def test_mechanisms_in_other_company():
    """The new mechanisms under the other residuals and beside the other kinds of layers: they are not tied to one design."""
    from b200serve.models.config import LatentAttention, MatrixLstm, MinGru, StreamBlock
    from b200serve.models.listed import random_listed_weights
    from b200serve.runtime.engine import Engine
    ff, up = DenseFfn(64), DenseFfn(96, relu2=True)
    near, gated = att(4, 2, 40, 0.2, Rotary(16, 1e4, 2.0), 24, 5), par(4, 2, 64, 64, 0.2, Rotary(64, 1e4, 4.0, 64), None).left
    ret = Retention(2, 64, 72, (0.9, 0.99), Rotary(32, 1e3))
    moe = ExpertFfn(6, 2, 64, "sigmoid", renorm=True, relu2=True, shared=100)
    streams = listed_config("medley", "Napadra", (LayerSpec(near, ff), LayerSpec(ret, up), LayerSpec(ParallelMixer(gated, ret, 0.7, 1.2), None),
                                                  LayerSpec(ParallelMixer(dataclasses.replace(near, qkv_bias=True, v_norm=True), MinGru(40), 1.0, 0.5), up)), 128, 200, 1e-5, StreamBlock(2, 0.6))
    normed = listed_config("medley2", "Mumusun", (LayerSpec(ret, moe), LayerSpec(gated, up), LayerSpec(near, None)), 128, 200, 1e-5)
    latent = LatentAttention(4, 64, 32, 64, 128, 96, 0.1, 32, 1e4, 48)
    two = listed_config("medley3", "Vogerax", (LayerSpec(latent, ExpertFfn(6, 2, 64, "sigmoid", renorm=True)), LayerSpec(MatrixLstm(2, 64, 64, 5.0), ff),
                                               LayerSpec(ParallelMixer(gated, ret, 0.7, 1.2), moe)), 128, 200, 1e-5, SandwichBlock(4, 2.0))
    ids = torch.randint(0, 200, (150,), generator=gen(1)).tolist()
    for cfg in (streams, normed, two):
        out = {}
        for dt in (F32, BF16):
            eng = Engine(random_listed_weights(cfg, DEV, 3, dtype=dt, std=0.1), max_seqs=2, max_len=256)
            whole = eng.forward_batch([(0, ids, list(range(150)))]).clone()
            one = torch.cat([eng.forward_batch([(1, [t], [0])]).clone() for t in ids])
            if dt == F32:
                close(one, whole.double().cpu(), "float32")
            out[dt] = whole, one
        for got in out[BF16]:           # random routers are close calls: a few tokens go to other experts
            d = ((got - out[F32][0]).pow(2).mean(-1) / out[F32][0].pow(2).mean(-1)).sqrt().sort().values.cpu()
            assert float(d[75]) < 0.03 and float(d[120]) < 0.12, (cfg.name, d[75], d[120])


def test_blocks_of_models_without_a_state(tmp_path):
    """A model of windowed layers alone can be rewound anywhere, and its pages can be kept and shared: blocks lie in the pages whose
    positions they end in."""
    from b200serve.runtime.engine import Engine
    a = [att(4, 2, 40, 0.3, Rotary(16, 1e4, 2.0), 24, pool) for pool in (5, 16, 37)]
    m = Model(listed_config("vogerax-near", "Vogerax", [LayerSpec(x, DenseFfn(72, relu2=True)) for x in a], 96, 120, 1e-5, SandwichBlock(2, 4.0)), tmp_path)
    eng = m.engine("float32")
    assert not eng.cfg.recurrent and isinstance(eng, Engine)
    ids, other = m.prompt(200), m.prompt(200, seed=1)
    eng.forward_batch([(0, ids[:150] + other[:40], [])])
    eng.truncate(0, 150)                   # in the middle of a page and of blocks
    close(eng.forward_batch([(0, ids[150:], list(range(50)))]), m.logits(ids)[150:], "float32")
    blob = eng.save_kv(0, 0, 96)           # whole pages of a longer sequence
    eng.reset()
    eng.forward_batch([(2, other[:70], [])])
    eng.load_kv(1, blob)
    mixed = ids[:96] + other[:90]
    out = [eng.forward_batch([(1, mixed[p: p + n], list(range(n)))]).clone() for p, n in ((96, 1), (97, 2), (99, 87))]
    close(torch.cat(out), m.logits(mixed)[96:], "float32")
