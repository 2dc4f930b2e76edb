"""Mumusun on the GPU against the plain reference (tests/mumusun_oracle.py): every mechanism alone, then whole models
served in 32-bit (sharp) and in bf16, in prompts, portions, decode steps, mixed batches and reused pages and slots."""
import json
import subprocess
import sys
import os

import numpy as np
import pytest
import torch

import mumusun_oracle as O
from b200serve.models.config import ExpertFfn, LatentAttention, LayerSpec, listed_config, preset

pytestmark = pytest.mark.gpu
DEV = "cuda"


def rel(got, ref):
    return float((got.double().cpu() - ref.double().cpu()).pow(2).mean().sqrt() / ref.double().pow(2).mean().sqrt().cpu())


def gen(seed):
    return torch.Generator().manual_seed(seed)


# ------------------------------------------------------------------ linears
@pytest.mark.parametrize("m", [1, 3, 8, 9, 16])
@pytest.mark.parametrize("n,k", [(64, 64), (320, 1984), (96, 448), (2112, 2048)])
def test_gemv_bf16(m, n, k):
    from b200serve.ops import latent as L
    g = gen(m * n + k)
    x, w = (torch.randn(m, k, generator=g) * 0.5).bfloat16().to(DEV), (torch.randn(n, k, generator=g) * 0.1).bfloat16().to(DEV)
    ref = x.double() @ w.double().T
    s = L.gemv_splits(n, k)
    out = torch.full((s, m, n), float("nan"), device=DEV)
    L.gemv_bf16(w, x, out, m, n, k, s)
    assert rel(out.sum(0), ref) < 1e-5
    ob = torch.empty(m, n, dtype=torch.bfloat16, device=DEV)
    L.gemv_bf16(w, x, ob, m, n, k, 1, L.EPI_BF16)
    assert rel(ob, ref) < 4e-3
    act = torch.empty(m, n // 2, dtype=torch.bfloat16, device=DEV)
    L.gemv_bf16(w, x, act, m, n, k, 1, L.EPI_SILU)
    v = ref.view(m, n // 32, 2, 16)
    assert rel(act, (O.silu(v[:, :, 0]) * v[:, :, 1]).reshape(m, n // 2)) < 4e-3
    # a row's bits do not depend on the rows beside it
    one = torch.empty(s, 1, n, device=DEV)
    L.gemv_bf16(w, x[m - 1:], one, 1, n, k, s)
    assert torch.equal(one[:, 0], out[:, m - 1])


@pytest.mark.parametrize("f32", [False, True])
def test_expert_rows(f32):
    from b200serve.models.weights import interleave16
    from b200serve.ops import latent as L
    g = gen(5)
    e, ff, h, m, k = 5, 128, 192, 3, 2
    dt = torch.float32 if f32 else torch.bfloat16
    x = torch.randn(m, h, generator=g).to(dt).to(DEV)
    gate, up = (torch.randn(e, ff, h, generator=g).mul(0.1).to(dt).to(DEV) for _ in range(2))
    down = torch.randn(e, h, ff, generator=g).mul(0.1).to(dt).to(DEV)
    ids = torch.tensor([4, 0, 2, 2, 1, 3], dtype=torch.int32, device=DEV)
    gu = torch.stack([interleave16(gate[i], up[i]) for i in range(e)]).contiguous()
    act = torch.empty(m * k, ff, dtype=dt, device=DEV)
    y = torch.empty(m * k, h, device=DEV)
    if f32:
        L.linear_f32_experts(gu, ids, m * k, x, k, act, True)
        L.linear_f32_experts(down, ids, m * k, act, 1, y, False)
    else:
        L.gemv_bf16_experts(gu, ids, m * k, x, k, act, 2 * ff, h, epi=L.EPI_SILU)
        L.gemv_bf16_experts(down, ids, m * k, act, 1, y, h, ff)
    for b in range(m * k):
        i = int(ids[b])
        w = {"gate": gate[i].double(), "up": up[i].double(), "down": down[i].double()}
        assert rel(y[b], O.expert(w, "", x[b // k].double())) < (1e-5 if f32 else 6e-3)


def test_linear_f32():
    from b200serve.ops import latent as L
    g = gen(6)
    for m, n, k in ((1, 64, 64), (70, 333, 192), (129, 1000, 64)):
        a, w = torch.randn(m, k, generator=g).to(DEV), torch.randn(n, k, generator=g).to(DEV)
        c = torch.empty(m, n, device=DEV)
        L.linear_f32(a, w, c, m)
        assert rel(c, a.double() @ w.double().T) < 1e-6


# ------------------------------------------------------------------ norms and the residual
@pytest.mark.parametrize("width,ld", [(200, 256), (1500, 1536), (5000, 5056)])
@pytest.mark.parametrize("m", [1, 5, 70])
def test_sublayer_norm(width, ld, m):
    from b200serve.ops import latent as L
    g = gen(width + m)
    x0 = torch.randn(m, ld, generator=g)
    x0[:, width:] = 0
    w = torch.randn(width, generator=g)
    eps = 0.3                              # large enough that leaving it out, or putting it elsewhere, shows

    def check(ref, **kw):
        x, h = x0.to(DEV).clone(), torch.full((m, ld), float("nan"), dtype=torch.bfloat16, device=DEV)
        L.sublayer_norm(m=m, width=width, w=w.to(DEV), eps=eps, x=x, h=h, **kw)
        want = x0[:, :width].double() + O.layer_norm(ref.double(), w.double(), eps)
        assert rel(x[:, :width], want) < 1e-6 and torch.all(x[:, width:] == 0) and torch.all(h[:, width:] == 0)
        assert torch.equal(h, x.bfloat16())
        own = torch.full((m, ld), float("nan"), device=DEV)
        hf = torch.empty(m, ld, device=DEV)
        L.sublayer_norm(m=m, width=width, w=w.to(DEV), eps=eps, x=own, h=hf, add=False, **kw)
        assert rel(own[:, :width], O.layer_norm(ref.double(), w.double(), eps)) < 1e-6 and torch.equal(hf, own)

    y = 0.4 * torch.randn(3, m, ld, generator=g) + 0.7      # a mean well away from zero
    check(y.sum(0)[:, :width], y=y.to(DEV), slices=3, slice_elems=m * ld, row_elems=ld)
    k = 3
    ys, wt = torch.randn(m * k, 2, ld, generator=g), torch.rand(m, k, generator=g)
    ref = (ys.sum(1).view(m, k, ld) * wt[..., None]).sum(1)[:, :width]
    check(ref, y=ys.to(DEV), slots=k, slices=2, slice_elems=ld, row_elems=2 * ld, slot_w=wt.to(DEV))
    yb = torch.randn(m * k + 40, ld, generator=g).bfloat16()
    rows = torch.randperm(m * k + 40, generator=g)[: m * k].to(torch.int32)
    ref = (yb[rows.long()].double().view(m, k, ld) * wt[..., None]).sum(1)[:, :width]
    check(ref, y=yb.to(DEV), slots=k, row_elems=ld, slot_w=wt.to(DEV), row_of=rows.to(DEV))


def test_layer_norm_of_selected_rows_and_embedding():
    from b200serve.ops import latent as L
    g = gen(9)
    x, w = torch.randn(7, 128, generator=g) + 2, torch.randn(100, generator=g)
    sel = torch.tensor([6, 0, 3], dtype=torch.int32, device=DEV)
    h = torch.empty(3, 128, device=DEV)
    L.layer_norm_rows(x.to(DEV), sel, w.to(DEV), 0.2, 3, 100, h)
    assert rel(h[:, :100], O.layer_norm(x[[6, 0, 3], :100].double(), w.double(), 0.2)) < 1e-6 and torch.all(h[:, 100:] == 0)
    e = torch.randn(11, 128, generator=g).bfloat16().to(DEV)
    xo, ho = torch.empty(2, 128, device=DEV), torch.empty(2, 128, dtype=torch.bfloat16, device=DEV)
    flag = torch.zeros(1, dtype=torch.int32, device=DEV)
    L.embed_rows(e, torch.tensor([10, 4], dtype=torch.int32, device=DEV), 2, xo, ho, flag)
    assert torch.equal(xo, e[[10, 4]].float()) and torch.equal(ho, e[[10, 4]]) and int(flag) == 0
    L.embed_rows(e, torch.tensor([11, -1], dtype=torch.int32, device=DEV), 2, xo, ho, flag)
    assert int(flag) == 1


def test_row_argmax_takes_the_lower_of_equal_logits():
    from b200serve.ops import latent as L
    lg = torch.zeros(2, 1000, device=DEV)
    lg[0, [900, 31, 700]] = 2.0
    val, idx = torch.empty(2, device=DEV), torch.empty(2, dtype=torch.int32, device=DEV)
    L.row_argmax(lg, 2, 1000, val, idx)
    assert idx.tolist() == [31, 0] and val.tolist() == [2.0, 0.0]


# ------------------------------------------------------------------ router
@pytest.mark.parametrize("e,top,groups,keep", [(12, 3, 3, 1), (16, 4, 4, 2), (10, 2, 1, 1), (8, 2, 8, 2), (96, 6, 8, 8), (1, 1, 1, 1),
                                               (500, 8, 20, 3)])
def test_router_groups(e, top, groups, keep):
    from b200serve.ops import moe as M
    g = gen(e)
    t, h = 13, 64
    z = torch.randn(t, e, generator=g) * 2
    idx, wt = torch.empty(t, top, dtype=torch.int32, device=DEV), torch.empty(t, top, device=DEV)
    rule = (1, groups, keep, 0)
    M.route(z.to(DEV).contiguous(), e, t, e, top, idx, wt, rule=rule)
    r = {"experts": e, "top": top, "groups": {"count": groups, "keep": keep}}
    for i in range(t):
        want = O.route(z[i].double(), r)
        assert idx[i].tolist() == [a for a, _ in want]
        assert torch.allclose(wt[i].cpu().double(), torch.stack([b for _, b in want]), rtol=1e-5)
    # the decode form: logits and routing in one launch
    er = (e + 7) // 8 * 8
    x = torch.randn(t, h, generator=g).bfloat16().to(DEV)
    w = torch.zeros(er, h, dtype=torch.bfloat16)
    w[:e] = (torch.randn(e, h, generator=g) * 0.3).bfloat16()
    logits, ticket = torch.empty(t, er, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    M.router_rows(w.to(DEV), x, logits, t, e, h, er, e, top, False, False, idx, wt, ticket, rule=rule)
    assert rel(logits[:, :e], x.double().cpu() @ w[:e].double().T) < 1e-5 and int(ticket) == 0
    for i in range(t):
        want = O.route(logits[i, :e].double().cpu(), r)
        assert idx[i].tolist() == [a for a, _ in want]
        assert torch.allclose(wt[i].cpu().double(), torch.stack([b for _, b in want]), rtol=1e-5)


def test_router_softmax_scores_without_renormalisation():
    from b200serve.ops import moe as M
    z = torch.randn(4, 40, generator=gen(1))
    idx, wt = torch.empty(4, 5, dtype=torch.int32, device=DEV), torch.empty(4, 5, device=DEV)
    M.route(z.to(DEV), 40, 4, 40, 5, idx, wt, rule=(0, 1, 1, 0))
    p, i = torch.softmax(z.double(), -1).topk(5, dim=-1)
    assert torch.equal(idx.cpu().long(), i) and torch.allclose(wt.cpu().double(), p, rtol=1e-4)


# ------------------------------------------------------------------ latent attention, mechanism by mechanism
# (heads, dim, rot_dim, vdim, kv_rank, q_rank, rope dims)
SHAPES = [(6, 40, 24, 72, 160, 100, 24), (16, 128, 64, 128, 512, 256, 64), (20, 72, 16, 48, 64, 72, 8), (1, 16, 8, 200, 320, 64, 8),
          (40, 64, 64, 64, 192, 128, 32)]


def mixer_of(shape, window, base=3e4):
    heads, dim, rot, vdim, rank, q_rank, rd = shape
    return LatentAttention(heads, dim, rot, vdim, rank, q_rank, 0.7 * (dim + rot) ** -0.5, rd, base, window)


def as_dict(a):
    return {"heads": a.heads, "dim": a.dim, "rot_dim": a.rot_dim, "vdim": a.vdim, "kv_rank": a.kv_rank, "scale": a.scale,
            "rot": {"dims": a.rope_dims, "base": a.rope_base}, "mask": {"size": a.window} if a.window else None}


class Attn:
    """One mixer with random weights, a scattered page table, and ``n`` positions of two requests in its cache."""

    def __init__(self, shape, window, n, dtype, seed=0):
        from b200serve.models.latent import LatentGeometry
        from b200serve.models.listed import assemble, tensor_shapes
        from b200serve.models.oracle import rope_tables
        g = gen(seed)
        self.a = a = mixer_of(shape, window)
        self.g = LatentGeometry.of(a)
        width = 80
        self.cfg = listed_config("one", "Mumusun", [LayerSpec(a, None)], width, 16, 1e-5)
        raw = {k: (1 + 0.3 * torch.randn(s, generator=g) if len(s) == 1 else torch.randn(s, generator=g) * s[1] ** -0.5).bfloat16()
               for k, s in tensor_shapes(self.cfg).items()}
        self.raw = {k: v.double() for k, v in raw.items()}
        self.w = assemble(self.cfg, lambda k: raw[k], DEV, dtype).layers[0].mixer
        self.dtype, self.n = dtype, n
        blocks = (n + 15) // 16
        perm = torch.randperm(2 * blocks, generator=g) + 1
        self.bt = perm.view(2, blocks).to(torch.int32).to(DEV).contiguous()
        self.cache = torch.zeros(2 * blocks + 1, 16, self.g.lc, dtype=dtype, device=DEV)
        c, s = rope_tables(a.rope_dims, a.rope_base, n)
        self.rope = (c.to(DEV), s.to(DEV))
        self.c = torch.randn(2, n, a.kv_rank, generator=g).to(dtype)              # latents and rotated key parts as cached
        self.kr = torch.randn(2, n, a.rot_dim, generator=g).to(dtype)
        for r in range(2):
            for p in range(n):
                row = self.cache[int(self.bt[r, p // 16]), p % 16]
                row[: a.kv_rank] = self.c[r, p].to(DEV)
                row[self.g.kvp: self.g.kvp + a.rot_dim] = self.kr[r, p].to(DEV)

    def reference(self, q, req, pos):
        """Attention output rows [len(pos)][heads][vdim] for unrotated queries ``q`` [rows][heads][dim + rot]."""
        a, w = self.a, self.raw
        p = "l0.mix."
        out = []
        for r in sorted(set(req)):
            i = [j for j, x in enumerate(req) if x == r]
            pp = torch.tensor([pos[j] for j in i])
            c, kr = self.c[r].double(), self.kr[r].double()
            k = torch.cat([(c @ w[p + "uk"].T).reshape(self.n, a.heads, a.dim),
                           kr[:, None].expand(self.n, a.heads, a.rot_dim)], -1)
            v = (c @ w[p + "uv"].T).reshape(self.n, a.heads, a.vdim)
            qq = q[i].double()
            qq = torch.cat([qq[..., : a.dim], O.rotate(qq[..., a.dim:], pp, a.rope_dims, a.rope_base)], -1)
            o = O.softmax_attention(qq, k, v, O.visible(pp, torch.arange(self.n), a.window), a.scale)
            out += list(zip(i, o))
        return torch.stack([o for _, o in sorted(out, key=lambda t: t[0])])

    def padded_q(self, q, dtype):
        a, g = self.a, self.g
        out = torch.zeros(len(q), a.heads, g.dk, dtype=dtype)
        out[..., : a.dim], out[..., g.dn: g.dn + a.rot_dim] = q[..., : a.dim], q[..., a.dim:]
        return out.reshape(len(q), -1).to(DEV)

    def rows(self, q, req, pos, nsplit, simple=False):
        from b200serve.ops import latent as L
        a, g, m = self.a, self.g, len(pos)
        rq, ps = (torch.tensor(x, dtype=torch.int32, device=DEV) for x in (req, pos))
        ql = torch.empty(m, a.heads * g.lc, dtype=self.dtype, device=DEV)
        L.absorb(self.padded_q(q, torch.float32), 1, m, g, self.w.uk, ps, self.rope, ql)
        op = torch.full((m * nsplit, a.heads * g.kvp), float("nan"), device=DEV)
        ml = torch.full((m * nsplit, a.heads * 2), float("nan"), device=DEV)
        if simple:
            L.simple(ql, self.cache, m, g, rq, ps, self.bt, op, ml, a.window, a.scale)
        else:
            L.rows(ql, self.cache, m, g, rq, ps, self.bt, op, ml, nsplit, a.window, a.scale)
        out = torch.full((m, a.heads * g.dv), float("nan"), dtype=self.dtype, device=DEV)
        L.merge(op, ml, m, g, nsplit, self.w.uv, out)
        v = out.view(m, a.heads, g.dv)
        assert torch.all(v[..., a.vdim:] == 0)
        return v[..., : a.vdim]

    def spike(self, q, row, req, key, gain=6.0):
        """Makes the scores of ``row``'s heads stand out at one key (through the rotated part's shared key)."""
        a = self.a
        kk = (self.c[req, key].double() @ self.raw["l0.mix.uk"].T).reshape(a.heads, a.dim)
        q[row, :, : a.dim] = (gain / (a.scale * kk.pow(2).sum(-1, keepdim=True).clamp_min(1e-3)) * kk * 2).float()
        q[row, :, a.dim:] *= 0.1


def test_down_projection_latents_and_cache_rows():
    from b200serve.ops import latent as L
    for shape in SHAPES:
        for dtype in (torch.float32, torch.bfloat16):
            t = Attn(shape, 0, 40, dtype)
            a, g, eps = t.a, t.g, 0.05
            m, s = 3, 2
            part = torch.zeros(s, m, g.n_down)
            raw = torch.randn(s, m, a.q_rank + a.kv_rank + a.rot_dim, generator=gen(2))
            part[..., : a.q_rank] = raw[..., : a.q_rank]
            part[..., g.qp: g.qp + a.kv_rank] = raw[..., a.q_rank: a.q_rank + a.kv_rank]
            part[..., g.qp + g.kvp: g.qp + g.kvp + a.rot_dim] = raw[..., a.q_rank + a.kv_rank:]
            req, pos = [1, 0, 1], [37, 0, 16]
            cq = torch.empty(m, g.qp, dtype=dtype, device=DEV)
            cache = torch.full_like(t.cache, float("nan"))
            L.prep(part.to(DEV), s, m, g, t.w.q_norm, t.w.kv_norm, eps, torch.tensor(req, dtype=torch.int32, device=DEV),
                   torch.tensor(pos, dtype=torch.int32, device=DEV), t.bt, t.rope, cq, cache)
            v = raw.double().sum(0)
            tol = 1e-6 if dtype == torch.float32 else 4e-3
            assert rel(cq[:, : a.q_rank], O.rms_norm(v[:, : a.q_rank], t.raw["l0.mix.dq.norm"], eps)) < tol
            c = O.rms_norm(v[:, a.q_rank: a.q_rank + a.kv_rank], t.raw["l0.mix.dkv.norm"], eps)
            kr = O.rotate(v[:, a.q_rank + a.kv_rank:], torch.tensor(pos), a.rope_dims, a.rope_base)
            for i in range(m):
                row = cache[int(t.bt[req[i], pos[i] // 16]), pos[i] % 16]
                assert rel(row[: a.kv_rank], c[i]) < tol and rel(row[g.kvp: g.kvp + a.rot_dim], kr[i]) < tol
                assert torch.all(row[a.kv_rank: g.kvp] == 0) and torch.all(row[g.kvp + a.rot_dim:] == 0)
            assert int((~torch.isnan(cache[..., 0])).sum()) == m          # nothing else was written


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [0, 1, 33, 130])
def test_decode_attention_forms(shape, window):
    n = 300
    for dtype, simple, nsplits in ((torch.bfloat16, False, (1, 3, 32)), (torch.bfloat16, True, (1,)), (torch.float32, True, (1,))):
        t = Attn(shape, window, n, dtype, seed=shape[0])
        pos = [0, 15, 16, 63, 64, 130, 299, 299, 32, 129]
        req = [0, 1, 0, 1, 1, 0, 0, 1, 0, 1]
        q = torch.randn(len(pos), t.a.heads, t.a.dim + t.a.rot_dim, generator=gen(3))
        ref = t.reference(q, req, pos)
        for ns in nsplits:
            got = t.rows(q, req, pos, ns, simple)
            assert rel(got, ref) < (1e-5 if dtype == torch.float32 else 8e-3), (dtype, simple, ns)


@pytest.mark.parametrize("shape", SHAPES[:3])
@pytest.mark.parametrize("window", [48, 64, 100])
def test_window_edges_in_decode_rows(shape, window):
    """One key carries nearly all of a row's weight: just inside the window it must be seen, just outside it must not."""
    n, pos = 260, 257
    t = Attn(shape, window, n, torch.bfloat16, seed=7)
    keys = [pos - window + 1, pos - window, pos, pos - 1, pos - 15, pos - 16, pos - 17, max(0, pos - window - 16)]
    q = torch.randn(len(keys), t.a.heads, t.a.dim + t.a.rot_dim, generator=gen(4))
    for i, k in enumerate(keys):
        t.spike(q, i, 0, k)
    ref = t.reference(q, [0] * len(keys), [pos] * len(keys))
    import dataclasses
    wrong = dataclasses.replace(t.a, window=window + 1)
    keep, t.a = t.a, wrong
    off_by_one = t.reference(q, [0] * len(keys), [pos] * len(keys))
    t.a = keep
    assert rel(off_by_one[1], ref[1]) > 0.3          # the reference itself tells the two windows apart
    for ns in (1, 2, 7):
        got = t.rows(q, [0] * len(keys), [pos] * len(keys), ns)
        for i in range(len(keys)):
            assert rel(got[i], ref[i]) < 0.03, (i, ns)


def run_prompt(t, q, segs):
    """The expanded prompt attention over segments (request, first position, rows) of ``q``."""
    from b200serve.ops import gemm as G
    from b200serve.ops import latent as L
    from b200serve.runtime.batch import segment_keys
    a, g = t.a, t.g
    per = L.prefill_rows_per_tile(g)
    if not per:
        return None
    m = len(q)
    pos = torch.cat([torch.arange(p, p + n) for _, p, n in segs]).to(torch.int32).to(DEV)
    qp = t.padded_q(q, torch.bfloat16).contiguous()
    L.rope_q(qp, pos, m, g, t.rope)
    kreq, kpos, tiles = segment_keys(segs, a.window, per)
    i32 = lambda v: torch.tensor(np.asarray(v), dtype=torch.int32, device=DEV)     # noqa: E731
    n = len(kreq)
    c, kr = torch.empty(n, g.kvp, dtype=torch.bfloat16, device=DEV), torch.empty(n, g.rp, dtype=torch.bfloat16, device=DEV)
    k, v = (torch.zeros(n, a.heads * d, dtype=torch.bfloat16, device=DEV) for d in (g.dn, g.dv))
    L.gather(t.cache, i32(kreq), i32(kpos), n, t.bt, g, c, kr)
    G.gemm_bf16(c, t.w.uk, k)
    G.gemm_bf16(c, t.w.uv, v)
    out = torch.full((m, a.heads * g.dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    L.attn_prefill_rows(qp, k, kr, v, out, i32(tiles).view(-1), len(tiles), m, n, g, a.scale, a.window)
    return out.view(m, a.heads, g.dv)[..., : a.vdim]


# more forms of the prompt kernel: key / value blocks of 64 (3, 1), (4, 1), (4, 2), (2, 4), (3, 4), (4, 4)
PROMPT_SHAPES = SHAPES + [(3, 128, 32, 64, 64, 64, 32), (2, 192, 40, 40, 64, 64, 40), (2, 130, 40, 128, 64, 64, 40),
                          (2, 100, 64, 256, 64, 64, 64), (2, 190, 64, 140, 64, 64, 64)]


@pytest.mark.parametrize("shape", PROMPT_SHAPES)
@pytest.mark.parametrize("window", [0, 2, 64, 150])
def test_prompt_attention(shape, window):
    n = 600
    t = Attn(shape, window, n, torch.bfloat16, seed=shape[1])
    segs = [(0, 0, 300), (1, 217, 37), (0, 300, 290)]
    rows = sum(x[2] for x in segs)
    q = torch.randn(rows, t.a.heads, t.a.dim + t.a.rot_dim, generator=gen(5))
    at = {}
    for r, p, cnt in segs:
        for i in range(cnt):
            at[len(at)] = (r, p + i)
    for row in (200, 299, 310, 336, 337, 500, rows - 1):      # rows whose weight sits on a key at the window's edge
        r, p = at[row]
        w = window or 190
        t.spike(q, row, r, max(0, p - w + (row % 2)))
    got = run_prompt(t, q, segs)
    if got is None:
        assert shape[1] + shape[2] > 256 or shape[3] > 256
        return
    ref = t.reference(q, [at[i][0] for i in range(rows)], [at[i][1] for i in range(rows)])
    assert rel(got, ref) < 8e-3
    worst = ((got.double().cpu() - ref).pow(2).mean((1, 2)) / ref.pow(2).mean((1, 2))).sqrt()
    assert float(worst.max()) < 0.05, int(worst.argmax())


# ------------------------------------------------------------------ whole models
def odd_config():
    """Sizes that fit no tile, single heads and experts, equal groups, a window of one, rotated part only half rotated."""
    m = LatentAttention
    return listed_config("mumusun-odd", "Mumusun", (
        LayerSpec(m(1, 20, 6, 12, 40, 24, 0.3, 4, 500.0, 1), ExpertFfn(1, 1, 24)),
        LayerSpec(m(18, 24, 10, 34, 72, 56, 0.2, 10, 1e4, 50), None),
        LayerSpec(m(2, 200, 24, 150, 600, 80, 0.1, 24, 1e4, 70), ExpertFfn(8, 3, 40, groups=8, keep=3)),
        LayerSpec(m(5, 32, 16, 192, 100, 64, 0.15, 16, 100.0, 0), ExpertFfn(4, 4, 16, groups=2, keep=2))), 200, 333, 1e-3)


CODE = 12      # leading residual columns that hold a token's code, see `coded`


def sharpen(name, t):
    """Peaked attention, so that the edges of windows matter."""
    return t * 3 if name.endswith("dq.norm") else t


def coded(name, t):
    """Weights for bf16: rounding must not flip a routing decision, or rows would differ by whole experts.  The first
    columns of an embedding are +-1, no sublayer adds to them, and routers read them alone: router logits are then the
    same in every element type, and still differ from token to token."""
    t = t.clone()
    if name == "embed":
        t[:, :CODE] = t[:, :CODE].sign()
    elif name.endswith("norm1") or name.endswith("norm2"):
        t[:CODE] = 0
    elif name.endswith("router"):
        t[:, CODE:] = 0
        t[:, :CODE] *= 8
    return t * 1.5 if name.endswith("dq.norm") else t


class Model:
    def __init__(self, cfg, path):
        from b200serve.utils.synth import write_listed
        self.cfg, self.json = cfg, cfg.to_listed_config()
        self.path = {"float32": str(path / "sharp"), "bfloat16": str(path / "coded")}
        self.w = {}
        for dtype, make in (("float32", sharpen), ("bfloat16", coded)):
            raw = write_listed(cfg, self.path[dtype], seed=len(cfg.name), make=make)
            self.w[dtype] = {k: v.double() for k, v in raw.items()}
        self.weights = {}
        self.known = {}

    def logits(self, ids, dtype):
        key = (dtype, *ids)
        if key not in self.known:
            self.known[key] = O.forward(self.w[dtype], self.json, list(ids))
        return self.known[key]

    def engine(self, dtype, max_seqs=4, max_len=512, num_pages=None, **kw):
        from b200serve.loader.loader import load
        from b200serve.runtime.engine import Engine
        if dtype not in self.weights:
            self.weights[dtype] = load(self.path[dtype], device=DEV, dtype=dtype, report=None)
        return Engine(self.weights[dtype], max_seqs=max_seqs, max_len=max_len, num_pages=num_pages, **kw)

    def prompt(self, n, seed=0):
        return torch.randint(0, self.cfg.vocab, (n,), generator=gen(1000 * n + seed)).tolist()


@pytest.fixture(scope="module", params=["mini", "odd"])
def model(request, tmp_path_factory):
    cfg = preset("mumusun-mini") if request.param == "mini" else odd_config()
    return Model(cfg, tmp_path_factory.mktemp(request.param))


def close(got, ref, dtype):
    got, ref = got.double().cpu(), ref.double()
    r = ((got - ref).pow(2).mean(-1) / ref.pow(2).mean(-1)).sqrt()
    limit = 1e-4 if dtype == "float32" else 0.06
    assert float(r.max()) < limit, (float(r.max()), int(r.argmax()), float(r.median()))


DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 2, 17, 64, 65, 230])
def test_prompt_in_one_step(model, dtype, n):
    eng = model.engine(dtype)
    ids = model.prompt(n)
    close(eng.forward_batch([(1, ids, list(range(n)))]), model.logits(ids, dtype), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_token_by_token_equals_the_prompt(model, dtype):
    ids = model.prompt(150)
    eng = model.engine(dtype)
    lg = torch.cat([eng.forward_batch([(0, [t], [0])]).clone() for t in ids])
    close(lg, model.logits(ids, dtype), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2] * 20 + [3, 5, 7, 100, 83], [33, 32, 31, 64, 1, 65, 12], [100, 2, 2, 96, 38], [16, 16, 15, 17, 174]])
def test_portions(model, dtype, cuts):
    ids = model.prompt(238)
    eng = model.engine(dtype)
    out, at = [], 0
    for c in cuts:
        out.append(eng.forward_batch([(2, ids[at: at + c], list(range(c)))]).clone())
        at += c
    assert at == len(ids)
    close(torch.cat(out), model.logits(ids, dtype), dtype)


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
            left = len(prompts[i]) - at
            c = min(left, int(rng.choice([1, 1, 2, 13, 40, 77])))
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
        close(torch.cat(got[i]), model.logits(p, dtype), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_request_does_not_depend_on_its_company(model, dtype):
    """The same request alone and beside others: the same to rounding (bits, where the same kernels serve both)."""
    ids = model.prompt(40)
    eng = model.engine(dtype)
    eng.forward_batch([(0, ids[:-1], [])])
    alone = eng.forward_batch([(0, ids[-1:], [0])]).clone()
    eng.reset(0)
    eng.forward_batch([(3, ids[:-1], []), (1, model.prompt(50), []), (2, model.prompt(70), [])])
    company = eng.forward_batch([(1, [5], []), (3, ids[-1:], [0]), (2, [6, 7, 8], [])]).clone()
    close(company, alone.double().cpu(), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_greedy_generation(model, dtype):
    """``Engine.generate`` (prompt pass, then captured decode steps): every token is the reference's choice for the
    tokens before it, or within rounding of it; the logits of the last step too."""
    ids = model.prompt(70)
    eng = model.engine(dtype)
    new = eng.generate(ids, 130)
    ref = model.logits(ids + new[:-1], dtype)[len(ids) - 1:]
    gap = ref.max(-1).values - ref[torch.arange(len(new)), torch.tensor(new)]
    assert float(gap.max()) < (1e-3 if dtype == "float32" else 0.2 * float(ref.std()))
    close(eng.logits(1), ref[-1:], dtype)
    assert eng.steps_replayed >= 129


def test_truncate_and_go_on(model):
    ids = model.prompt(120)
    eng = model.engine("float32")
    eng.forward_batch([(0, ids[:100] + model.prompt(60, seed=1), [])])
    eng.truncate(0, 100)
    close(eng.forward_batch([(0, ids[100:], list(range(20)))]), model.logits(ids, "float32")[100:], "float32")


def test_saved_pages_and_prefix_store(model):
    from b200serve.server.prefix import PrefixStore
    ids = model.prompt(200)
    eng = model.engine("float32")
    eng.forward_batch([(0, ids[:96], [])])
    blob = eng.save_kv(0, 0, 96)
    eng.load_kv(1, blob)
    close(eng.forward_batch([(1, ids[96:], [103])]), model.logits(ids, "float32")[-1:], "float32")
    eng.reset()
    store = PrefixStore(eng, host_gb=0.02, block_tokens=32)
    eng.reset(2)
    assert store.begin(2, ids) == 0
    eng.prefill(2, ids)
    store.after_prefill(2, ids)
    store.end(2, ids)
    more = ids[:160] + model.prompt(30, seed=9)
    hit = store.begin(3, more)
    assert hit >= 128
    close(eng.forward_batch([(3, more[hit:], [len(more) - hit - 1])]), model.logits(more, "float32")[-1:], "float32")


def test_weights_in_both_element_types_run_what_they_say(model):
    e32, e16 = model.engine("float32"), model.engine("bfloat16")
    assert e32.kv_dtype == "f32" and all(t.dtype == torch.float32 for t in e32.kv.pages.values())
    assert e16.kv_dtype == "bf16" and all(t.dtype == torch.bfloat16 for t in e16.kv.pages.values())


def test_served_over_http(model):
    """Concurrent requests through the server: prompt chunks and decode rows share batches, tokens are the reference's."""
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
    srv = Server(adapter, ByteTok(), ChatTemplate(), ServerOptions(model_name="m", prefill_chunk=48, max_queue=8)).start()
    res = {}

    def post(i, ids, extra):
        c = http.client.HTTPConnection("127.0.0.1", srv.port, timeout=60)
        c.request("POST", "/v1/completions", json.dumps({"prompt": ids, "max_tokens": 24, "temperature": 0, "ignore_eos": True,
                                                         "return_token_ids": True, **extra}), {"Content-Type": "application/json"})
        r = c.getresponse()
        res[i] = (r.status, json.loads(r.read().decode()))
        c.close()
    prompts = [model.prompt(n, seed=3) for n in (90, 200, 20, 170, 33, 110)]
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
            assert len(new) == 24
            ref = model.logits(p + new[:-1], "float32")[len(p) - 1:]
            assert float((ref.max(-1).values - ref[torch.arange(24), torch.tensor(new)]).max()) < 1e-3
        assert calls and max(n for _, n in calls) >= 1
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
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model.path["float32"], "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not os.path.exists(tmp_path / "2.f32")
    la, lb = model.logits(a, "float32"), model.logits(b, "float32")
    for i, ref in ((0, la[[0, 79]]), (1, torch.stack([la[80], lb[66], lb[5]])), (3, torch.stack([la[89], lb[2]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4")).view(-1, model.cfg.vocab)
        close(got, ref, "float32")
