"""Pefulorn on the GPU against the plain reference (tests/pefulorn_oracle.py): every mechanism alone, then whole models served
in 32-bit (sharp) and in bf16, in prompts, portions, decode steps, mixed batches and reused pages and slots."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pefulorn_oracle as O
from b200serve.models.config import (ChannelDelta, DenseFfn, GroupedAttention, LayerLoop, LayerSpec, MinGru, ParallelMixer, StreamBlock,
                                     Wkv, listed_config, preset)

pytestmark = pytest.mark.gpu
DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16


def rel(got, ref):
    return float((got.double().cpu() - ref.double().cpu()).pow(2).mean().sqrt() / ref.double().pow(2).mean().sqrt().cpu())


def gen(seed):
    return torch.Generator().manual_seed(seed)


def i32(v):
    return torch.tensor(np.asarray(v), dtype=torch.int32, device=DEV)


def pad_cols(t, ld):
    out = torch.zeros(*t.shape[:-1], ld)
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


def segments(runs):
    from b200serve.runtime.batch import CHUNK, ChunkPlan, segment_chunks
    segs, chunks = segment_chunks(runs)
    return ChunkPlan(len(segs), i32(segs).view(-1), chunks, max((s[1] + CHUNK - 1) // CHUNK for s in segs))


# ------------------------------------------------------------------ residual
RUNS = {1: [(0, 9, 1)], 5: [(2, 0, 1), (0, 5, 3), (1, 40, 1)], 70: [(1, 0, 40), (0, 3, 29), (2, 7, 1)],
        1400: [(0, 64, 700), (3, 0, 650), (1, 2, 50)]}


@pytest.mark.parametrize("width,ld", [(72, 128), (200, 256), (1500, 1536), (5000, 5056)])
@pytest.mark.parametrize("m", sorted(RUNS))
@pytest.mark.parametrize("planes", [0, 1, 5])
def test_plain_residual_boundary(width, ld, m, planes):
    """x + y + bias, what comes ahead of a pass, a norm with a factor per column, several mixes with the row before."""
    from b200serve.ops import streams as S
    g, runs, eps = gen(width + m), RUNS[m], 0.2
    at = runs_rows(runs)
    req, pos = [r for r, _ in at], [p for _, p in at]
    n, slots, vocab = len(at), 4, 30
    rnd = lambda *s: torch.randn(*s, generator=g)                                  # noqa: E731
    x, y, bias, add, norm = rnd(n, width), rnd(3 if n < 100 else 1, n, width), rnd(width), rnd(width), rnd(width)
    mu, prev, table, tok = torch.rand(max(planes, 1), width, generator=g), rnd(slots, width), rnd(vocab, width).bfloat16(), torch.randint(0, vocab, (n,), generator=g)
    for ahead in (False, True):
        ref = x.double() + y.double().sum(0) + bias.double()
        if ahead:
            ref = ref + add.double() + table[tok].double()
        h = O.rms(ref, eps) * norm.double()
        before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
        for i, (r, p) in enumerate(at):
            if i == 0 or at[i - 1][0] != r:
                before[i] = prev[r].double() if p else 0
        want = [h] if not planes else [h + (before - h) * mu[k].double() for k in range(planes)]
        x_out = torch.full((n, ld), float("nan"), device=DEV)
        out = torch.full((max(planes, 1) * n, ld), float("nan"), device=DEV)
        nxt = pad_cols(rnd(slots, width), ld).to(DEV)
        held, commit = nxt.clone(), torch.zeros_like(nxt)
        kw = dict(m=n, streams=1, width=width, req=i32(req), pos=i32(pos), eps=eps, x_in=pad_cols(x, ld).to(DEV), norm=pad_cols(norm, ld).to(DEV),
                  bias=pad_cols(bias, ld).to(DEV))
        if ahead:
            kw.update(add=pad_cols(add, ld).to(DEV), again=(pad_cols(table.float(), ld).bfloat16().to(DEV), i32(tok)))
        if planes:
            m_ = pad_cols(mu, ld).to(DEV)
            kw.update(mu=m_ if planes > 1 else m_[0].contiguous(), prev=pad_cols(prev, ld).to(DEV), next_h=nxt, commit=commit)
        S.boundary(pad_cols(y, ld).to(DEV), len(y), None, 0, 1.0, x_out=x_out, h=out, **kw)
        assert rel(x_out[:, :width], ref) < 1e-6 and torch.all(x_out[:, width:] == 0)
        for k, w in enumerate(want):
            got = out[k * n: (k + 1) * n]
            assert rel(got[:, :width], w) < 3e-6 and torch.all(got[:, width:] == 0)
            worst = (got[:, :width].double().cpu() - w).pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()
            assert float(worst.max()) < 2e-5, int(worst.argmax())
        if planes:
            for r in range(slots):
                if r in req:
                    last = max(i for i, q in enumerate(req) if q == r)
                    assert torch.equal(commit[r], held[r]) and rel(nxt[r, :width], h[last]) < 1e-5
                else:
                    assert torch.equal(nxt[r], held[r]) and torch.all(commit[r] == 0)


def test_first_boundary_with_a_pass_and_mixes():
    """A model whose first layer starts a pass and reads shifted inputs."""
    from b200serve.ops import streams as S
    width, ld, vocab, n = 90, 128, 25, 12
    g = gen(3)
    table, add, mu, norm = (torch.randn(vocab, width, generator=g).bfloat16(), torch.randn(width, generator=g), torch.rand(5, width, generator=g),
                            torch.randn(width, generator=g))
    tok, flag = torch.randint(0, vocab, (n,), generator=g), torch.zeros(1, dtype=torch.int32, device=DEV)
    x_out, h, nxt = torch.empty(n, ld, device=DEV), torch.empty(5 * n, ld, device=DEV), torch.zeros(1, ld, device=DEV)
    S.embed(pad_cols(table.float(), ld).bfloat16().to(DEV), i32(tok), None, flag, m=n, streams=1, width=width, req=i32([0] * n), pos=i32(range(n)),
            eps=1e-5, norm=pad_cols(norm, ld).to(DEV), h=h, x_out=x_out, mu=pad_cols(mu, ld).to(DEV), prev=torch.full((1, ld), 9.0, device=DEV),
            next_h=nxt, add=pad_cols(add, ld).to(DEV))
    x = table[tok].double() + add.double()
    hr = O.rms(x, 1e-5) * norm.double()
    assert rel(x_out[:, :width], x) < 1e-6 and rel(nxt[0, :width], hr[-1]) < 1e-5 and int(flag) == 0
    for k in range(5):
        assert rel(h[k * n: (k + 1) * n, :width], hr + (O.previous(hr) - hr) * mu[k].double()) < 3e-6


# ------------------------------------------------------------------ linears
def test_gelu_products_with_biases():
    from b200serve.models.weights import interleave16
    from b200serve.ops import gemm as G, latent as L
    g = gen(4)
    k, ff = 192, 160
    gate, up = torch.randn(ff, k, generator=g) * 0.2, torch.randn(ff, k, generator=g) * 0.2
    ba, bb = torch.randn(ff, generator=g), torch.randn(ff, generator=g)
    bias = interleave16(ba[:, None], bb[:, None]).view(-1).to(DEV)
    ref = lambda x, a, b: O.gelu_tanh(x @ a.T + ba.double()) * (x @ b.T + bb.double())       # noqa: E731
    inf = float("inf")
    for m in (1, 7, 16, 40, 300):
        x = torch.randn(m, k, generator=g)
        w = interleave16(gate, up)
        out = torch.empty(m, ff, device=DEV)
        L.glu_rows_f32((x @ w.T).to(DEV).contiguous(), out, m, 2 * ff, inf, 1.0, 0.0, True, bias)
        assert rel(out, ref(x.double(), gate.double(), up.double())) < 1e-5
        xb, wb = x.bfloat16().to(DEV), w.bfloat16().to(DEV).contiguous()
        ob = torch.full((m, ff), float("nan"), dtype=BF16, device=DEV)
        if m <= 16:
            L.gemv_bf16_glu(wb, xb, ob, m, 2 * ff, k, inf, 1.0, 0.0, True, bias)
        else:
            G.gemm_glu(xb, wb, ob, inf, 1.0, 0.0, True, bias)
        assert rel(ob, ref(xb.double().cpu(), gate.bfloat16().double(), up.bfloat16().double())) < 5e-3
    big = torch.tensor([[60.0] * 16 + [1.0] * 16, [-60.0] * 16 + [1.0] * 16], device=DEV)      # far ends: x and 0
    out = torch.empty(2, 16, device=DEV)
    L.glu_rows_f32(big, out, 2, 32, inf, 1.0, 0.0, True, None)
    assert torch.all(out[0] == 60) and torch.all(out[1] == 0)


@pytest.mark.parametrize("rows,n", [(128, 5 * 128), (192, 4 * 192 + 64), (64, 4 * 64 + 320)])
def test_linear_over_planes(rows, n):
    from b200serve.ops import gemm as G, latent as L
    k, planes = 256, 5
    w = torch.randn(n, k, generator=gen(1)) * 0.1
    which = torch.clamp(torch.arange(n) // rows, max=planes - 1)
    for m in (1, 5, 8, 13, 16):
        x = torch.randn(planes, m, k, generator=gen(m))
        ref = torch.einsum("nk,nmk->mn", w.bfloat16().double(), x.bfloat16().double()[which])
        for s in (1, 2):
            out = torch.full((s * m, n), float("nan"), device=DEV)
            L.gemv_bf16_planes(w.bfloat16().to(DEV), x.bfloat16().to(DEV), rows, out, m, n, k, s)
            assert rel(out.view(s, m, n).sum(0), ref) < 1e-5
    m, x = 70, torch.randn(planes, 70, k, generator=gen(9))
    for dtype, tol in ((F32, 1e-6), (BF16, 1e-5)):
        wd, xd, out = w.to(dtype).to(DEV), x.to(dtype).to(DEV), torch.full((m, n), float("nan"), device=DEV)
        for i in range(planes):                    # columns of one result, as the layers use them
            lo, hi = i * rows, n if i == planes - 1 else (i + 1) * rows
            if dtype == F32:
                L.linear_f32(xd[i], wd[lo:hi], out[:, lo:hi], m)
            else:
                G.gemm_bf16(xd[i], wd[lo:hi], out[:, lo:hi], epi=G.EPI_F32)
        assert rel(out, torch.einsum("nk,nmk->mn", wd.double().cpu(), xd.double().cpu()[which])) < tol


# ------------------------------------------------------------------ attention
# (heads, kv heads, dim, vdim): one, a few and more than sixteen heads on a key head, every block count of a key and a value
SHAPES = [(6, 2, 40, 72), (4, 4, 128, 128), (18, 1, 72, 136), (1, 1, 200, 40), (40, 2, 64, 192), (3, 3, 16, 256), (8, 4, 256, 130)]


class Attn:
    """Cached keys and values of two requests behind a scattered page table, a logarithmic distance bias."""

    def __init__(self, shape, n, dtype, seed=0):
        from b200serve.models.grouped import GroupedGeometry
        g = gen(seed)
        heads, kv, dim, vdim = shape
        self.a = a = GroupedAttention(heads, kv, dim, vdim, 0.8 * dim ** -0.5, log_bias=True)
        self.g, self.n, self.dtype = GroupedGeometry.of(a), n, dtype
        blocks = (n + 15) // 16
        self.bt = (torch.randperm(2 * blocks, generator=g) + 1).view(2, blocks).to(torch.int32).to(DEV).contiguous()
        self.k, self.v = torch.randn(2, n, kv, dim, generator=g).to(dtype), torch.randn(2, n, kv, vdim, generator=g).to(dtype)
        self.r1, self.r2 = torch.rand(heads, generator=g) * 2, torch.rand(heads, generator=g) ** 3 * 2
        self.kc, self.vc = (torch.zeros(2 * blocks + 1, kv, 16, c, dtype=dtype, device=DEV) for c in (self.g.dk, self.g.dv))
        for r in range(2):
            for p in range(n):
                page = int(self.bt[r, p // 16])
                self.kc[page, :, p % 16, :dim] = self.k[r, p].to(DEV)
                self.vc[page, :, p % 16, :vdim] = self.v[r, p].to(DEV)

    def reference(self, q, req, pos):
        out = {}
        for r in sorted(set(req)):
            i = [j for j, x in enumerate(req) if x == r]
            o = O.log_bias_attention(q[i].double(), self.k[r].double(), self.v[r].double(), torch.tensor([pos[j] for j in i]),
                                     torch.arange(self.n), self.a.scale, self.r1.double(), self.r2.double())
            out.update(zip(i, o))
        return torch.stack([out[j] for j in range(len(req))])

    def padded_q(self, q):
        return pad_cols(q.to(self.dtype).float(), self.g.dk).to(self.dtype).view(len(q), -1).to(DEV).contiguous()

    def out(self, m, dtype):
        """Rows inside wider ones."""
        wide = torch.full((m, self.g.heads * self.g.dv + 64), float("nan"), dtype=dtype, device=DEV)
        return wide, wide[:, : self.g.heads * self.g.dv]

    def cut(self, wide, mult):
        v = wide[:, : self.g.heads * self.g.dv].reshape(len(wide), self.g.heads, self.g.dv)
        assert torch.all(v[..., self.a.vdim:] == 0) and torch.all(torch.isnan(wide[:, self.g.heads * self.g.dv:]))
        return v[..., : self.a.vdim].float() / mult

    def rows(self, q, req, pos, nsplit=0, mult=0.5):
        from b200serve.ops import paged as P
        g, m = self.g, len(pos)
        wide, out = self.out(m, self.dtype)
        args = (self.padded_q(q), self.kc, self.vc, m, g, i32(req), i32(pos), self.bt)
        more = dict(logb=(self.r1.to(DEV), self.r2.to(DEV)), mult=mult)
        if nsplit:
            op, ml = (torch.full((m * nsplit * g.heads, c), float("nan"), device=DEV) for c in (g.dv, 2))
            P.rows(*args, nsplit, 0, self.a.scale, None, None, op, ml, out, **more)
        else:
            P.simple(*args, 0, self.a.scale, None, None, out, **more)
        return self.cut(wide, mult)

    def segments(self, q, segs, mult=2.0):
        from b200serve.ops import paged as P
        from b200serve.runtime.batch import segment_tiles
        tiles = segment_tiles(segs, 0, P.segments_per_tile(self.g))
        wide, out = self.out(len(q), BF16)
        P.attn_segments(self.padded_q(q), self.kc, self.vc, self.bt, out, i32(tiles).view(-1), len(tiles), len(q), self.g, self.a.scale, 0,
                        None, None, logb=(self.r1.to(DEV), self.r2.to(DEV)), mult=mult)
        return self.cut(wide, mult)

    def spike(self, q, row, req, key, pos, over=9.0):
        """Makes every head's score at one key stand out against the bias of its place."""
        a = self.a
        kk = self.k[req, key].double().repeat_interleave(a.heads // a.kv_heads, dim=0)
        want = over + O.log_bias(torch.tensor(float(pos - key)).double(), self.r1.double(), self.r2.double())
        q[row] = (want[:, None] / a.scale * kk / kk.pow(2).sum(-1, keepdim=True)).float()


@pytest.mark.parametrize("shape", SHAPES)
def test_attention_of_rows(shape):
    pos = [0, 1, 15, 16, 17, 49, 64, 130, 299, 299, 32, 131]
    req = [0, 1, 0, 1, 1, 0, 0, 1, 0, 1, 1, 0]
    for dtype, splits in ((BF16, (0, 1, 3, 32)), (F32, (0,))):
        t = Attn(shape, 300, dtype, seed=shape[0])
        q = torch.randn(len(pos), t.a.heads, t.a.dim, generator=gen(3)).to(dtype).float()
        t.spike(q, 7, 1, 0, 130)                  # the first key, a page's last and first key, the row's own
        t.spike(q, 8, 0, 15, 299)
        t.spike(q, 9, 1, 16, 299)
        t.spike(q, 11, 0, 131, 131)
        q = q.to(dtype).float()
        ref = t.reference(q, req, pos)
        for ns in splits:
            got = t.rows(q, req, pos, ns)
            for i in range(len(pos)):
                assert rel(got[i], ref[i]) < (1e-5 if dtype == F32 else 0.02), (dtype, ns, i)
            assert rel(got, ref) < (1e-5 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("shape", SHAPES + [(2, 1, 192, 64), (2, 2, 130, 200), (2, 1, 64, 64), (4, 2, 190, 192), (2, 1, 256, 180)])
def test_attention_of_prompt_segments(shape):
    t = Attn(shape, 600, BF16, seed=shape[2])
    segs = [(0, 0, 300), (1, 217, 37), (0, 300, 290)]
    at = runs_rows(segs)
    q = torch.randn(len(at), t.a.heads, t.a.dim, generator=gen(5))
    for row, key in ((1, 0), (63, 63), (64, 0), (65, 64), (129, 127), (255, 1), (256, 255), (299, 16), (300, 200), (336, 0), (500, 3), (626, 589)):
        t.spike(q, row, at[row][0], key, at[row][1])
    q = q.bfloat16().float()
    got = t.segments(q, segs)
    ref = t.reference(q, [r for r, _ in at], [p for _, p in at])
    assert rel(got, ref) < 8e-3
    worst = ((got.double().cpu() - ref).pow(2).mean((1, 2)) / ref.pow(2).mean((1, 2))).sqrt()
    assert float(worst.max()) < 0.04, int(worst.argmax())


def test_far_keys_among_hundreds():
    """A key thousands of positions back carries the row's weight against what its distance costs."""
    t = Attn((32, 8, 64, 64), 2500, BF16, seed=2)
    pos, keys = [2499, 2400, 2048, 1300], [3, 1, 16, 1023]
    q = torch.randn(4, 32, 64, generator=gen(1)) * 0.2
    for i in range(4):
        t.spike(q, i, 1, keys[i], pos[i], over=14.0)
    q = q.bfloat16().float()
    ref = t.reference(q, [1] * 4, pos)
    for ns in (0, 1, 9, 40):
        assert rel(t.rows(q, [1] * 4, pos, ns), ref) < 0.02
    qs = torch.randn(100, 32, 64, generator=gen(6)) * 0.2
    t.spike(qs, 99, 1, 5, 2499, over=14.0)
    qs = qs.bfloat16().float()
    assert rel(t.segments(qs, [(1, 2400, 100)])[99], t.reference(qs, [1] * 100, list(range(2400, 2500)))[99]) < 0.02


def test_distance_bias_shows_in_equal_keys():
    """With equal keys the weights are the bias alone: a distance that is one off would show."""
    t = Attn((4, 1, 64, 64), 200, F32, seed=4)
    t.k[:] = t.k[:1, :1]
    t.kc[1:] = pad_cols(t.k[0, 0], 64).view(1, 1, 1, 64).to(DEV)
    t.r1, t.r2 = torch.tensor([0.0, 1.0, 4.0, 2.0]), torch.tensor([1.0, 2.0, 0.5, 40.0])
    q = torch.randn(3, 4, 64, generator=gen(1))
    assert rel(t.rows(q, [0, 1, 1], [0, 3, 199]), t.reference(q, [0, 1, 1], [0, 3, 199])) < 1e-5


# sizes up to eight quads per lane
@pytest.mark.parametrize("shape", SHAPES[:4] + [(2, 1, 300, 520), (1, 1, 1000, 16)])
@pytest.mark.parametrize("bias,qk_norm,v_norm,temp,every", [(True, True, True, 0.5, 7), (False, False, True, 0.0, 1), (True, True, False, 1.5, 1),
                                                            (True, False, False, 0.3, 100)])
def test_heads_with_biases_norms_and_temperature(shape, bias, qk_norm, v_norm, temp, every):
    from b200serve.models.grouped import GroupedGeometry
    from b200serve.models.weights import GroupedWeights
    from b200serve.ops import paged as P
    heads, kv, dim, vdim = shape
    a = GroupedAttention(heads, kv, dim, vdim, 1.0, qkv_bias=bias, qk_norm=qk_norm, v_norm=v_norm, temp=temp, temp_every=every)
    g, rg, eps = GroupedGeometry.of(a), gen(heads + dim), 0.03
    blocks = 20
    bt = (torch.randperm(2 * blocks, generator=rg) + 1).view(2, blocks).to(torch.int32).to(DEV).contiguous()
    req, pos = [1, 0, 1, 1, 0], [300, 0, every - 1, min(every, 318), 17]
    m, sides = 5, (("q", heads, dim, g.dk), ("k", kv, dim, g.dk), ("v", kv, vdim, g.dv))
    raw = {n: torch.randn(m, h, d, generator=rg) for n, h, d, _ in sides}
    b = {n: torch.randn(h, d, generator=rg) for n, h, d, _ in sides}
    wn = {n: torch.randn(dim, generator=rg) for n in "qk"}
    ref = {}
    for n, _, _, _ in sides:
        x = raw[n].double() + (b[n].double() if bias else 0)
        if n == "v":
            x = O.rms(x, eps) if v_norm else x
        elif qk_norm:
            x = O.rms(x, eps) * wn[n].double()
        if n == "q":
            x = x * O.temperature(torch.tensor(pos), temp, every)[:, None, None]
        ref[n] = x
    full = torch.cat([pad_cols(raw[n], p).view(m, -1) for n, _, _, p in sides] + [torch.full((m, 192), 5.0)], dim=1)
    w = GroupedWeights(None, None, None, None)
    if bias:
        w.bias = torch.cat([pad_cols(b[n], p).view(-1) for n, _, _, p in sides]).to(DEV)
    if qk_norm:
        w.q_norm, w.k_norm = (pad_cols(wn[n], g.dk).to(DEV) for n in "qk")
    for dtype, tol in ((F32, 2e-6), (BF16, 4e-3)):
        for s in (1, 3):
            q = torch.full((m, g.nq), float("nan"), dtype=dtype, device=DEV)
            k, v = (torch.full((2 * blocks + 1, kv, 16, c), float("nan"), dtype=dtype, device=DEV) for c in (g.dk, g.dv))
            P.norm(slices_of(full, s).view(s * m, -1), s, m, g, a, w, eps, i32(req), i32(pos), bt, q, k, v)
            q = q.view(m, heads, g.dk)
            assert rel(q[..., :dim], ref["q"]) < tol and torch.all(q[..., dim:].float().abs() < 1e-4)
            for i in range(m):
                page, off = int(bt[req[i], pos[i] // 16]), pos[i] % 16
                assert rel(k[page, :, off, :dim], ref["k"][i]) < tol and rel(v[page, :, off, :vdim], ref["v"][i]) < tol
            assert int((~torch.isnan(k[:, 0, :, 0])).sum()) == m


# ------------------------------------------------------------------ minGRU
class Gru:
    def __init__(self, width, slots=4, seed=0):
        from b200serve.models.weights import MinGruWeights
        g = gen(seed)
        self.width, self.n = width, (width + 63) // 64 * 64
        self.bz, self.bx = torch.randn(width, generator=g), torch.randn(width, generator=g) * 0.3
        self.w = MinGruWeights(None, None, pad_cols(self.bz, self.n).to(DEV), pad_cols(self.bx, self.n).to(DEV))
        self.state = torch.full((slots, self.n), float("nan"), device=DEV)        # a sequence starts from zeros by itself

    def inputs(self, t, seed):
        g = gen(seed)
        return torch.randn(3, t, self.width, generator=g) * torch.tensor([3.0, 1.5, 1.0])[:, None, None]

    def reference(self, x):
        s, _ = O.min_gru_scan(x[0].double() + self.bz.double(), x[1].double() + self.bx.double())
        return s * O.silu(x[2].double())

    def run(self, runs, n1, dtype, slices=1, col=64, mult=0.7):
        """``runs``: (slot, first position, inputs); the first ``n1`` rows one by one, the other runs as segments."""
        from b200serve.ops import mingru as R
        at = runs_rows([(s, p, x.shape[1]) for s, p, x in runs])
        m = len(at)
        full = torch.full((m, col + 3 * self.n), 3.0)
        for i in range(3):
            full[:, col + i * self.n: col + (i + 1) * self.n] = pad_cols(torch.cat([x[i] for _, _, x in runs]), self.n)
        t, seen = None, 0
        if n1 < m:
            segs = []
            for s, p, x in runs:
                if seen >= n1:
                    segs.append((s, p, x.shape[1]))
                seen += x.shape[1]
            t = segments(segs)
        wide = torch.full((m, self.n + 64), float("nan"), dtype=dtype, device=DEV)
        R.scan(slices_of(full, slices).view(slices * m, -1), slices, m, col, self.n, self.w, i32([s for s, _ in at]), i32([p for _, p in at]), n1,
               t.segs if t else None, t.n_segs if t else 0, mult, self.state, wide[:, 64:])
        assert torch.all(wide[:, 64 + self.width:] == 0) and torch.all(torch.isnan(wide[:, :64]))
        return wide[:, 64: 64 + self.width].double().cpu() / mult


@pytest.mark.parametrize("width", [1, 40, 64, 200, 1000])
@pytest.mark.parametrize("cuts", [(400,), (128, 129, 143), (1, 130, 2, 64, 203), (33, 40, 327)])
def test_gated_recurrence(width, cuts):
    for dtype, tol in ((F32, 2e-6), (BF16, 5e-3)):
        t = Gru(width, seed=width)
        x, y = t.inputs(400, 1), t.inputs(400, 2)
        ref, ref2 = t.reference(x), t.reference(y)
        at = 0
        for n in cuts:
            runs = [(1, at, x[:, at: at + n]), (3, at, y[:, at: at + n])]
            if n < 32:
                got = t.run(runs, 2 * n, dtype, slices=3)
            elif n == 40:                          # one sequence row by row, the other as a segment
                got = t.run(runs, n, dtype)
            else:
                got = t.run(runs, 0, dtype)
            assert rel(got, torch.cat([ref[at: at + n], ref2[at: at + n]])) < tol, (at, n)
            at += n
        again = t.inputs(3, 99)                    # a slot that is used again starts from zeros
        assert rel(t.run([(1, 0, again)], 3, dtype), t.reference(again)) < tol and torch.isnan(t.state[0]).all()


def test_gates_at_their_ends():
    """Gates nearly shut keep an early value for hundreds of rows, gates nearly open forget at once."""
    t = Gru(64, seed=5)
    t.bz[:] = 0
    t.w.bias_z.zero_()
    x = t.inputs(500, 1)
    x[0] = -30.0
    x[0, 3], x[0, 200, ::2], x[2] = 4.0, 30.0, 2.0
    x[1, 10:20] = 90.0
    x[1, 20:30] = -90.0
    ref = t.reference(x)
    got = t.run([(0, 0, x)], 0, F32)
    assert float(((got - ref).abs() / ref.abs().clamp(min=1e-30)).max()) < 1e-5
    assert rel(t.run([(2, 0, x)], 500, F32), ref) < 1e-6 and rel(t.run([(1, 0, x)], 0, BF16), ref) < 5e-3


# ------------------------------------------------------------------ recurrences with channel decays
# (key heads, heads, key dims, value dims): every count of dims per lane, one head, shared key heads, values beyond one CTA's head
CELLS = [(1, 1, 16, 40), (2, 2, 64, 64), (3, 6, 100, 128), (1, 4, 128, 130), (2, 2, 190, 70), (2, 2, 256, 128), (1, 2, 250, 300), (1, 1, 300, 48),
         (1, 2, 500, 512)]


class Cell:
    """Prepared rows made directly."""

    def __init__(self, shape, delta, slots=4, seed=0):
        from b200serve.models.channel_delta import pad_key
        from b200serve.ops import channel_rec as R
        g = gen(seed)
        self.hq, self.h, self.dim, self.vdim = shape
        self.delta, self.dk = delta, pad_key(self.dim)
        self.dv = (self.vdim + 63) // 64 * 64
        self.cols = R.act_cols(self.hq, self.h, self.dk, self.dv)
        self.norm = torch.randn(self.h, self.vdim, generator=g)
        self.normp = pad_cols(self.norm, self.dv).view(-1).to(DEV)
        self.state = torch.full((slots, self.h * self.dk * self.dv), float("nan"), device=DEV)

    def inputs(self, t, seed, decay=None):
        g = gen(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)                              # noqa: E731
        x = dict(q=O.unit(rnd(t, self.hq, self.dim)), k=O.unit(rnd(t, self.hq, self.dim)), v=rnd(t, self.h, self.vdim), z=rnd(t, self.h, self.vdim),
                 g=torch.rand(t, self.h, self.dim, generator=g) ** 0.2 if decay is None else torch.full((t, self.h, self.dim), decay),
                 s1=torch.rand(t, self.h, generator=g), u=rnd(self.h, self.dim))
        return x

    def reference(self, x, eps=0.02):
        rep = lambda y: y.double().repeat_interleave(self.h // self.hq, dim=1)     # noqa: E731
        q, k, v, g = rep(x["q"]), rep(x["k"]), x["v"].double(), x["g"].double()
        if self.delta:
            o, _ = O.delta_scan(q, k, v, g, x["s1"].double())
        else:
            o, _ = O.wkv_scan(q, k, v, g, torch.zeros(self.h, self.dim, dtype=torch.float64))
            o = o + x["s1"].double()[:, :, None] * v
        return O.rms(o, eps) * self.norm.double() * x["z"].double()

    def act(self, x):
        t = len(x["q"])
        pad4 = lambda y: pad_cols(y, (y.shape[1] + 3) // 4 * 4)                    # noqa: E731
        s2 = torch.full((t, self.h), float("nan"))
        s2[:, : self.hq] = (x["q"].double() * x["k"].double()).sum(-1).float()
        g = torch.rand(t, self.h, self.dk, generator=gen(7))         # decays of padding dims do not matter
        g[..., : self.dim] = x["g"]
        parts = [pad_cols(x["q"], self.dk), pad_cols(x["k"], self.dk), g, pad_cols(x["v"], self.dv), pad_cols(x["z"], self.dv)]
        out = torch.cat([y.reshape(t, -1) for y in parts] + [pad4(x["s1"]), pad4(s2)], dim=1)
        assert out.shape[1] == self.cols
        return out

    def run(self, runs, dtype, seg, eps=0.02, tc=False):
        from b200serve.ops import channel_rec as R
        at = runs_rows([(s, p, len(x["q"])) for s, p, x in runs])
        m = len(at)
        act = torch.cat([self.act(x) for _, _, x in runs]).to(DEV)
        t = segments([(s, p, len(x["q"])) for s, p, x in runs]) if seg else None
        raw = torch.full((m, self.h * self.dv), float("nan"), device=DEV)
        out = torch.full((m, self.h * self.dv), float("nan"), dtype=dtype, device=DEV)
        R.scan(act, self.delta, m, self.hq, self.h, self.dk, self.dv, self.vdim, i32([s for s, _ in at]), i32([p for _, p in at]), t,
               self.state, self.normp, eps, raw, out, ws=self.workspace(t) if tc else None)
        v = out.view(m, self.h, self.dv)
        assert torch.all(v[..., self.vdim:] == 0)
        return v[..., : self.vdim]

    def workspace(self, t):
        from b200serve.ops import channel_rec as R
        return torch.full((4 * t.chunks * self.h * R.block_bytes(self.delta, self.dk, self.dv),), 0xFF, dtype=torch.uint8, device=DEV)


def cut_inputs(x, lo, hi):
    return {k: v[lo:hi] if k != "u" else v for k, v in x.items()}


def row_errors(got, ref):
    return ((got.double().cpu() - ref).pow(2).mean((1, 2)) / ref.pow(2).mean((1, 2))).sqrt()


@pytest.mark.parametrize("shape", CELLS)
@pytest.mark.parametrize("delta", [True, False])
def test_channel_recurrence(shape, delta):
    """Rows one by one (several of a sequence, sequences beside each other) and segments of any cut follow one walk over the whole
    sequence; a slot that is used again starts from zeros."""
    if not delta:
        shape = (shape[1],) + shape[1:]
    for cuts in ((70,), (33, 1, 36), (2, 1, 3, 64), (40, 17, 13), (1,) * 6 + (32, 32)):
        c = Cell(shape, delta, seed=shape[2])
        x, y = c.inputs(70, 1), c.inputs(70, 2)
        ref, ref2 = c.reference(x), c.reference(y)
        at = 0
        for n in cuts:
            runs = [(2, at, cut_inputs(x, at, at + n)), (0, at, cut_inputs(y, at, at + n))]
            got = c.run(runs, F32, n >= 32)
            assert float(row_errors(got, torch.cat([ref[at: at + n], ref2[at: at + n]])).max()) < 3e-5, (cuts, at, n)
            at += n
        assert torch.isnan(c.state[1]).all()
    again = c.inputs(37, 9)
    for seg in (False, True):
        assert float(row_errors(c.run([(2, 0, again)], BF16, seg), c.reference(again)).max()) < 6e-3


@pytest.mark.parametrize("shape", [s for s in CELLS if s[2] <= 256])
@pytest.mark.parametrize("delta", [True, False])
def test_channel_recurrence_on_tensor_cores(shape, delta):
    """Segments in chunks of sixteen rows, the last one cut anywhere, between rows one by one; several sequences."""
    if not delta:
        shape = (shape[1],) + shape[1:]
    for cuts in ((200,), (64, 1, 33, 47, 3, 52), (100, 100), (32, 168)):
        c = Cell(shape, delta, seed=shape[2])
        xs = {s: c.inputs(200, s) for s in (0, 3)}
        ref = {s: c.reference(x) for s, x in xs.items()}
        at = 0
        for n in cuts:
            runs = [(s, at, cut_inputs(x, at, at + n)) for s, x in xs.items()]
            got = c.run(runs, F32, n >= 32, tc=n >= 32)
            assert float(row_errors(got, torch.cat([ref[s][at: at + n] for s in xs])).max()) < 2e-4, (cuts, at, n)
            at += n
        assert torch.isnan(c.state[1]).all()


@pytest.mark.parametrize("delta", [True, False])
def test_decays_at_their_ends(delta):
    """Decays of nearly one remember a strong early write for hundreds of rows, decays of nearly zero forget it at once, mixed
    channels do both."""
    for decay in (0.9999, 1e-8, 0.0, None):
        c = Cell((2, 2, 96, 64), delta, seed=3)
        x = c.inputs(420, 5, decay)
        if decay is None:
            x["g"][:, :, ::2], x["g"][:, :, 1::2] = 1.0, 1e-20
        x["s1"][:] = 0.02
        x["v"][10:] *= 0.05
        x["v"][5] *= 40
        x["s1"][5] = 1.0
        x["q"][5:] = x["k"][5]                     # late rows ask for the early write
        ref = c.reference(x)
        for seg, tc in ((False, False), (True, False), (True, True)):
            assert float(row_errors(c.run([(1, 0, x)], F32, seg, tc=tc), ref).max()) < 5e-4, (decay, seg, tc)


def prep_model(mixer, taps_seed=0):
    """Weights of one mixer in a 64-wide model, fp32 and bf16 from the same bf16 values, with their reference tensors."""
    from b200serve.models.listed import Assembler, kind
    cfg = listed_config("one", "Pefulorn", (LayerSpec(mixer, None),), 64, 50, 1e-5,
                        StreamBlock(1, 1.0, shift=False, scale=False, sinusoid=0.0, mixing=False, columns=True))
    g, raw = gen(taps_seed + 5), {}
    for n, s in kind(mixer).shapes(cfg, "l0.mix.", mixer).items():
        raw[n] = (torch.randn(s, generator=g) * (0.5 if len(s) == 1 else s[1] ** -0.5)).bfloat16()
    w = {d: kind(mixer).assemble(Assembler(cfg, lambda n: raw[n], DEV, d), "l0.mix.", mixer) for d in (F32, BF16)}
    return {k: v.double() for k, v in raw.items()}, w


@pytest.mark.parametrize("mixer", [ChannelDelta(4, 2, 40, 72, 1, 5, 9), ChannelDelta(2, 2, 64, 64, 2, 64, 64), ChannelDelta(3, 1, 130, 40, 3, 80, 20),
                                   ChannelDelta(2, 2, 96, 200, 4, 16, 150), ChannelDelta(1, 1, 300, 64, 6, 30, 31), ChannelDelta(2, 1, 16, 300, 11, 8, 8)])
def test_what_enters_the_delta_rule(mixer):
    """Convolution with its state over any cut, unit norms, step sizes, decays and gates, from dots and from GEMMs."""
    from b200serve.models.channel_delta import DeltaGeometry
    from b200serve.ops import channel_rec as R
    a, g, p = mixer, DeltaGeometry.of(mixer), "l0.mix."
    raw, w = prep_model(mixer, a.conv)
    t = 150
    h = {s: torch.randn(t, 64, generator=gen(s)).bfloat16().float() for s in (0, 2)}
    ref = {}
    for s in h:
        x = h[s].double()
        q, k, v = (O.silu(O.causal_conv(x @ raw[p + n].T, raw[p + n + ".conv"])) for n in "qkv")
        q, k = (O.unit(y.reshape(t, a.kv_heads, a.dim)) for y in (q, k))
        q = q * a.dim ** -0.5
        ref[s] = dict(q=q, k=k, v=v.reshape(t, a.heads, a.vdim), s1=torch.sigmoid(x @ raw[p + "b"].T), s2=(q * k).sum(-1),
                      g=O.channel_decay(x @ raw[p + "a1"].T @ raw[p + "a2"].T, raw[p + "A_log"], raw[p + "dt_bias"], a.heads),
                      z=torch.sigmoid(x @ raw[p + "g1"].T @ raw[p + "g2"].T).reshape(t, a.heads, a.vdim))
    for dtype, form in ((F32, "dots"), (BF16, "dots"), (BF16, "gemm")):
        conv = torch.full((3, g.taps - 1, g.channels), float("nan"), device=DEV)
        at = 0
        for n in (1, 2, 40, 3, 1, 70, 1, 32):
            runs = [(2, at, n), (0, at, n)]
            x = torch.cat([h[s][at: at + n] for s, _, _ in runs]).double()
            m = len(x)
            full = (x @ w[F32].proj.double().cpu().T).float()
            nxt = torch.full_like(conv, float("nan")).view(3, -1)
            slices = 2 if m < 17 else 1
            part = slices_of(full, slices).view(slices * m, -1)
            lr = None
            if form == "gemm":
                from b200serve.ops import gemm as G
                low, y, nk = torch.empty(2 * m, 2 * g.kp, dtype=BF16, device=DEV), torch.empty(m, g.second, device=DEV), g.heads * g.dk
                R.lowrank_rows(part, slices, m, (g.col_a1, g.col_g1), (a.a_rank, a.g_rank), g.kp, False, low)
                for lo, hi, x_ in ((0, nk, low[:m]), (nk, g.second, low[m:])):
                    G.gemm_bf16(x_, w[BF16].second[lo:hi], y[:, lo:hi], epi=G.EPI_F32)
                lr = (y, 1)
            act = torch.full((m, g.act), float("nan"), device=DEV)
            rows = runs_rows(runs)
            R.delta_prep(part, slices, m, g, a, w[dtype], i32([s for s, _ in rows]), i32([q for _, q in rows]), conv, nxt, lr, act)
            conv[[0, 2]] = nxt.view_as(conv)[[0, 2]]
            assert torch.isnan(nxt[1]).all()
            cuts = act.double().cpu().split([g.kv_heads * g.dk] * 2 + [g.heads * g.dk, g.heads * g.dv, g.heads * g.dv] + [(g.heads + 3) // 4 * 4] * 2, dim=1)
            names = (("q", g.kv_heads, g.dk, a.dim), ("k", g.kv_heads, g.dk, a.dim), ("g", g.heads, g.dk, a.dim), ("v", g.heads, g.dv, a.vdim),
                     ("z", g.heads, g.dv, a.vdim))
            for got, (name, heads, pad, size) in zip(cuts, names):
                want = torch.cat([ref[s][name][at: at + n] for s, _, _ in runs])
                got = got.reshape(m, heads, pad)
                assert float(row_errors(got[..., :size], want).max()) < 2e-4, (name, form, at, n)
                if name in "qkv":
                    assert torch.all(got[..., size:] == 0)
            for got, name in zip(cuts[5:], ("s1", "s2")):
                want = torch.cat([ref[s][name][at: at + n] for s, _, _ in runs])
                assert float((got[:, : want.shape[1]] - want).abs().max()) < 2e-5, name
            at += n
        assert at == t


@pytest.mark.parametrize("mixer", [Wkv(3, 40, 9), Wkv(2, 64, 64), Wkv(1, 128, 100), Wkv(2, 200, 3), Wkv(1, 300, 20)])
def test_what_enters_the_time_mixing(mixer):
    from b200serve.models.wkv import WkvGeometry
    from b200serve.ops import channel_rec as R
    a, g, p = mixer, WkvGeometry.of(mixer), "l0.mix."
    raw, w = prep_model(mixer)
    for dtype, m in ((F32, 3), (F32, 90), (BF16, 1), (BF16, 16), (BF16, 90)):
        x = torch.randn(5, m, 64, generator=gen(m)).double()
        sides = [(x[i] @ raw[p + n].T).reshape(m, a.heads, a.dim) for i, n in enumerate("rkvg")]
        low = x[4] @ raw[p + "w1"].T
        decay = torch.exp(-torch.exp(torch.tanh(low) @ raw[p + "w2"].T + raw[p + "w0"])).reshape(m, a.heads, a.dim)
        full = torch.cat([pad_cols(y.float(), g.d).view(m, -1) for y in sides] + [pad_cols(low.float(), g.n - 4 * g.hd)], dim=1)
        s = 3 if m < 17 else 1
        part, act, lr = slices_of(full, s).view(s * m, -1), torch.full((m, g.act), float("nan"), device=DEV), None
        if dtype == BF16 and m > 16:
            from b200serve.ops import gemm as G
            y, z = torch.empty(m, 2 * g.kp, dtype=BF16, device=DEV), torch.empty(m, g.hd, device=DEV)
            R.lowrank_rows(part, s, m, (4 * g.hd,), (a.w_rank,), g.kp, True, y)
            G.gemm_bf16(y, w[BF16].second, z, epi=G.EPI_F32)
            lr = (z, 1)
        R.wkv_prep(part, s, m, g, a, w[dtype], lr, act)
        cuts = act.double().cpu().split([g.hd] * 5 + [(g.heads + 3) // 4 * 4] * 2, dim=1)
        for got, want in zip(cuts, (sides[0], sides[1], decay, sides[2], O.silu(sides[3]))):
            assert float(row_errors(got.reshape(m, a.heads, g.d)[..., : a.dim], want).max()) < 2e-4
        want = (sides[0] * raw[p + "u"] * sides[1]).sum(-1)
        assert float((cuts[5][:, : a.heads] - want).abs().max()) < 1e-5 * float(want.abs().max()) + 1e-6


# ------------------------------------------------------------------ whole models
PLAIN = StreamBlock(1, 1.0, shift=False, scale=False, sinusoid=0.0, mixing=False, columns=True)


def attention_beside_gru(heads, kv, dim, vdim, scale, width, coef, every, scales):
    return ParallelMixer(GroupedAttention(heads, kv, dim, vdim, scale, log_bias=True, qkv_bias=True, qk_norm=True, v_norm=True, temp=coef,
                                          temp_every=every), MinGru(width), *scales)


def odd_config():
    """Sizes that fit no tile, time mixing first, single heads, heads outside the tensor-core forms and beyond one CTA, one tap and
    many, the loop at the end, layers without feed-forwards in a row."""
    ff = lambda n: DenseFfn(n, gelu=True, bias=True)                               # noqa: E731
    return listed_config("pefulorn-odd", "Pefulorn", (
        LayerSpec(Wkv(1, 24, 7), None), LayerSpec(Wkv(2, 150, 3), ff(40)), LayerSpec(ChannelDelta(4, 1, 8, 150, 1, 3, 80), None),
        LayerSpec(attention_beside_gru(18, 1, 24, 34, 0.3, 40, 1.2, 3, (0.5, 2.0)), None), LayerSpec(ChannelDelta(1, 1, 270, 20, 7, 100, 4), ff(24)),
        LayerSpec(attention_beside_gru(3, 3, 300, 270, 0.07, 8, 0.2, 64, (-1.0, 0.7)), ff(72))), 150, 333, 1e-3, PLAIN, LayerLoop(4, 6, 2))


def one_config():
    """One pass over everything, a feed-forward only at the end."""
    return listed_config("pefulorn-one", "Pefulorn", (
        LayerSpec(ChannelDelta(2, 2, 64, 64, 4, 16, 16), None), LayerSpec(attention_beside_gru(2, 2, 64, 64, 0.2, 64, 0.0, 1, (1.0, 1.0)), None),
        LayerSpec(Wkv(1, 64, 16), DenseFfn(64, gelu=True, bias=True))), 64, 100, 1e-5, PLAIN, LayerLoop(0, 3, 1))


def flat_config():
    """No loop at all; wide heads; two attention layers with the same value size and other heads."""
    ff = DenseFfn(64, gelu=True, bias=True)
    return listed_config("pefulorn-flat", "Pefulorn", (
        LayerSpec(attention_beside_gru(4, 2, 190, 130, 0.1, 130, 0.6, 20, (0.9, 1.1)), ff), LayerSpec(Wkv(3, 128, 40), ff),
        LayerSpec(ChannelDelta(2, 1, 256, 128, 3, 40, 24), ff), LayerSpec(attention_beside_gru(3, 3, 64, 150, 0.15, 64, 0.4, 50, (1.0, 0.6)), None)),
        320, 211, 1e-6, PLAIN)


def lively(name, t):
    """Random weights that make the mechanisms matter: norms around zero, peaked attention at every distance, decays of every
    length, gates that open and close, mixes of every degree."""
    last, g = name.rsplit(".", 1)[-1], gen(len(name) + t.numel())
    uni = lambda lo, hi: lo + (hi - lo) * torch.rand(t.shape, generator=g)         # noqa: E731
    if name == "final.norm" or last in ("norm1", "norm2"):
        return 0.2 * torch.randn(t.shape, generator=g)
    if last == "norm" and ".left." in name:
        return uni(1.0, 2.5)
    if last in ("r1", "r2"):
        return uni(0.0, 1.5) if last == "r1" else uni(0.02, 1.0)
    if ".mu." in name:
        return uni(0.0, 1.0)
    if last == "A_log":
        return uni(-2.0, 1.0)
    if last in ("dt_bias", "w0"):
        return uni(-4.0, 0.5)
    if last == "conv":
        return torch.randn(t.shape, generator=g) * 0.6
    if name.endswith("z.b"):
        return uni(-4.0, 1.0)
    if last == "b" and t.dim() == 1:
        return 0.5 * torch.randn(t.shape, generator=g)
    if name == "loop.step":
        return torch.randn(t.shape, generator=g) * 0.5
    return t


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


@pytest.fixture(scope="module", params=["mini", "odd", "one", "flat"])
def model(request, tmp_path_factory):
    cfg = {"mini": lambda: preset("pefulorn-mini"), "odd": odd_config, "one": one_config, "flat": flat_config}[request.param]()
    return Model(cfg, tmp_path_factory.mktemp(request.param))


def close(got, ref, dtype):
    got, ref = got.double().cpu(), ref.double()
    r = ((got - ref).pow(2).mean(-1) / ref.pow(2).mean(-1)).sqrt()
    if dtype == "float32":
        assert float(r.max()) < 1e-4, (float(r.max()), int(r.argmax()), float(r.median()))
    else:
        assert float(r.median()) < 0.03 and float(r.max()) < 0.1, (float(r.max()), int(r.argmax()), float(r.median()))


DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 2, 17, 64, 65, 230])
def test_prompt_in_one_step(model, dtype, n):
    eng = model.engine(dtype)
    ids = model.prompt(n)
    close(eng.forward_batch([(1, ids, list(range(n)))]), model.logits(ids), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_token_by_token_equals_the_prompt(model, dtype):
    ids = model.prompt(150)
    eng = model.engine(dtype)
    lg = torch.cat([eng.forward_batch([(0, [t], [0])]).clone() for t in ids])
    close(lg, model.logits(ids), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2] * 20 + [3, 5, 7, 100, 83], [33, 32, 31, 64, 1, 65, 12], [100, 2, 2, 96, 38], [16, 16, 15, 17, 174],
                                  [238]])
def test_portions(model, dtype, cuts):
    ids = model.prompt(238)
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_greedy_generation(model, dtype):
    """``Engine.generate`` (prompt pass, then captured decode steps): every token is the reference's choice for the
    tokens before it, or within rounding of it; the logits of the last step too."""
    ids = model.prompt(70)
    eng = model.engine(dtype)
    new = eng.generate(ids, 130)
    ref = model.logits(ids + new[:-1])[len(ids) - 1:]
    gap = ref.max(-1).values - ref[torch.arange(len(new)), torch.tensor(new)]
    assert float(gap.max()) < (1e-3 if dtype == "float32" else 0.2 * float(ref.std()))
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
        ref = model.logits(p + new[s][:-1])[len(p) - 1:]
        gap = ref.max(-1).values - ref[torch.arange(21), torch.tensor(new[s])]
        assert float(gap.max()) < (1e-3 if dtype == "float32" else 0.2 * float(ref.std())), s


@pytest.mark.parametrize("dtype", DTYPES)
def test_more_requests_than_a_gemv_takes(model, dtype):
    """Thirty requests in one decode step."""
    eng = model.engine(dtype, max_seqs=30, max_len=64)
    prompts = [model.prompt(3 + i, seed=i) for i in range(30)]
    eng.forward_batch([(i, p[:-1], []) for i, p in enumerate(prompts)])
    lg = eng.forward_batch([(i, p[-1:], [0]) for i, p in enumerate(prompts)])
    close(lg, torch.stack([model.logits(p)[-1] for p in prompts]), dtype)


def test_rows_taken_back(model):
    """Rejected rows leave pages and state as if they had never run, in row steps and in mixed batches; a state cannot be
    rewound further."""
    from b200serve.runtime.engine import Row
    ids = model.prompt(120)
    eng = model.engine("float32")
    eng.forward_batch([(0, ids[:100], [])])
    eng.forward_rows([Row(0, 100, ids[100]), Row(0, 101, 5), Row(0, 102, 6)])
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
            ref = model.logits(p + new[:-1])[len(p) - 1:]
            assert float((ref.max(-1).values - ref[torch.arange(16), torch.tensor(new)]).max()) < 1e-3
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
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model.path, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=240)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        la, lb = model.logits(a), model.logits(b)
        for i, ref in ((0, la[[0, 79]]), (1, torch.stack([la[80], lb[66], lb[5]])), (3, torch.stack([la[89], lb[2]]))):
            got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, model.cfg.vocab)
            close(got, ref, dtype)


def test_mechanisms_in_other_company():
    """The new kinds of layers over several learned residual streams and under the layer-normed residual: mechanisms are not tied to
    one design."""
    from b200serve.models.config import MatrixLstm
    from b200serve.models.listed import random_listed_weights
    from b200serve.runtime.engine import Engine
    ff, gate = DenseFfn(64), DenseFfn(96, gelu=True, bias=True)
    delta, both = ChannelDelta(2, 1, 40, 72, 3, 8, 12), attention_beside_gru(4, 2, 64, 64, 0.2, 100, 0.5, 9, (0.7, 1.2))
    streams = listed_config("medley", "Napadra", (LayerSpec(delta, ff), LayerSpec(both, gate), LayerSpec(MatrixLstm(2, 64, 64, 5.0), None),
                                                  LayerSpec(MinGru(40), gate)), 128, 200, 1e-5, StreamBlock(3, 0.6), LayerLoop(1, 3, 2))
    normed = listed_config("medley2", "Mumusun", (LayerSpec(delta, ff), LayerSpec(both, ff), LayerSpec(MinGru(72), None)), 128, 200, 1e-5)
    mixes = listed_config("medley3", "Napadra", (LayerSpec(Wkv(2, 40, 8), ff), LayerSpec(both.left, None)), 128, 200, 1e-5, StreamBlock(2, 0.5, shift=False))
    ids = torch.randint(0, 200, (150,), generator=gen(1)).tolist()
    for cfg in (streams, normed, mixes):
        out = {}
        for dt in (F32, BF16):
            eng = Engine(random_listed_weights(cfg, DEV, 3, dtype=dt, std=0.1), max_seqs=2, max_len=256)
            whole = eng.forward_batch([(0, ids, list(range(150)))]).clone()
            one = torch.cat([eng.forward_batch([(1, [t], [0])]).clone() for t in ids])
            close(one, whole.double().cpu(), "float32" if dt == F32 else "bfloat16")
            out[dt] = whole
        close(out[BF16][:40], out[F32][:40].double().cpu(), "bfloat16")
