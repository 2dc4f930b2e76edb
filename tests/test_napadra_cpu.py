"""Napadra without a GPU: the plain reference by hand, configuration, checkpoint layout, batch tables, planning."""
import json
import math

import pytest
import torch

import napadra_oracle as O
from b200serve.models.config import GroupedAttention, MatrixLstm, ModelConfig, preset

F64 = torch.float64


def test_oracle_mechanisms_by_hand():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    assert torch.allclose(O.rms(x, 0.5), x / math.sqrt(13.0))
    p = O.sinusoid(torch.tensor([0, 7]), 4)
    want = [math.sin(7), math.cos(7), math.sin(0.07), math.cos(0.07)]
    assert torch.allclose(p[0], torch.tensor([0.0, 1.0, 0.0, 1.0], dtype=F64)) and torch.allclose(p[1], torch.tensor(want, dtype=F64))
    h = torch.tensor([[1.0, 2.0], [5.0, 6.0]], dtype=F64)
    assert torch.allclose(O.token_shift(h, torch.tensor([0.0, 0.25], dtype=F64)), torch.tensor([[1.0, 1.5], [5.0, 5.0]], dtype=F64))
    s = torch.stack([h, 10 * h])
    mix = torch.tensor([[1.0, 2.0], [0.0, 0.5]], dtype=F64)       # from, to
    out = O.streams_out(s, mix, torch.tensor([1.0, 3.0], dtype=F64), h, 0.5)
    assert torch.allclose(out[0], 1.5 * h) and torch.allclose(out[1], (2 + 5 + 1.5) * h)
    assert torch.allclose(O.streams_in(s, torch.tensor([2.0, 0.1], dtype=F64)), 3 * h)
    assert torch.allclose(O.alibi_slopes(4), torch.tensor([2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8], dtype=F64))
    vis = O.same_chunk(torch.tensor([5, 6]), torch.arange(8), 3)
    assert vis[0].tolist() == [False] * 3 + [True] * 3 + [False] * 2 and vis[1].tolist() == [False] * 6 + [True, False]
    g = O.clamped_glu(torch.tensor([9.0, -1.0], dtype=F64), torch.tensor([-9.0, 0.5], dtype=F64), 2.0)
    assert torch.allclose(g, torch.tensor([2 / (1 + math.exp(-3.404)) * -1.0, -1 / (1 + math.exp(1.702)) * 1.5], dtype=F64))


def test_oracle_attention_by_hand():
    """Two heads on one key head, two keys, scores, bias and sink written out."""
    q, k = torch.tensor([[[1.0], [2.0]]], dtype=F64), torch.tensor([[[3.0]], [[1.0]]], dtype=F64)
    v, sink = torch.tensor([[[1.0]], [[10.0]]], dtype=F64), torch.tensor([0.3, -0.2], dtype=F64)
    o = O.sink_attention(q, k, v, torch.tensor([1]), torch.arange(2), None, 0.5, sink)[0, :, 0]
    for h, (qq, slope) in enumerate(((1.0, 2.0 ** -4), (2.0, 2.0 ** -8))):
        a, b = math.exp(qq * 3 * 0.5 - slope), math.exp(qq * 1 * 0.5)
        assert math.isclose(float(o[h]), (a + 10 * b) / (a + b + math.exp(float(sink[h]))), rel_tol=1e-12)
    one = O.sink_attention(q, k, v, torch.tensor([1]), torch.arange(2), 1, 0.5, sink)[0, 0, 0]      # its own chunk only
    assert math.isclose(float(one), 10 * math.exp(0.5) / (math.exp(0.5) + math.exp(0.3)), rel_tol=1e-12)


def test_oracle_recurrence_by_hand():
    """The running maximum cancels out of everything but the floor of the denominator."""
    g = torch.Generator().manual_seed(1)
    t, a, b = 9, 3, 2
    q, k, v = (torch.randn(t, 1, n, generator=g, dtype=F64) for n in (a, a, b))
    i, f = O.mlstm_gates(torch.randn(t, 1, generator=g, dtype=F64) * 4, torch.randn(t, 1, generator=g, dtype=F64) * 4, 2.5)
    assert float(i.abs().max()) < 2.5 and float(f.max()) < 0
    out, (s, n, m) = O.mlstm_scan(q, k, v, i, f)
    for j in range(t):
        w = [math.exp(float(f[r + 1: j + 1].sum() + i[r])) for r in range(j + 1)]
        num = sum(w[r] * float(k[r, 0] @ q[j, 0]) * v[r, 0] for r in range(j + 1))
        den = sum(w[r] * float(k[r, 0] @ q[j, 0]) for r in range(j + 1))
        top = max([float(f[: j + 1].sum())] + [float(f[r + 1: j + 1].sum() + i[r]) for r in range(j + 1)])
        want = num * math.exp(-top) / (max(abs(den) * math.exp(-top), math.exp(-top)) + 1e-6)
        assert torch.allclose(out[j, 0], want)
    half, state = O.mlstm_scan(q[:4], k[:4], v[:4], i[:4], f[:4])
    rest, _ = O.mlstm_scan(q[4:], k[4:], v[4:], i[4:], f[4:], state)
    assert torch.allclose(torch.cat([half, rest]), out)


def test_config_round_trip_and_refusals():
    for name in ("napadra-mini", "napadra-7b"):
        c = preset(name)
        back = ModelConfig.from_hf_config(json.loads(json.dumps(c.to_hf_config())))
        assert back.layer_specs == c.layer_specs and back.block == c.block and back.recurrent
        assert (back.hidden, back.vocab, back.rms_eps) == (c.hidden, c.vocab, c.rms_eps)
    d = preset("napadra-mini").to_hf_config()

    def layer(i, **kw):
        return lambda x: x["layers"][i]["mixer"].update(kw)
    for edit in (lambda x: x["layers"][0].update(type="mamba"), lambda x: x["layers"][0]["mlp"].update(kind="moe"), layer(0, kv_heads=4),
                 layer(4, kv_from=1), layer(4, kv_from=4), layer(4, kv_from=2), layer(5, kv_from=4), layer(1, vdim=600),
                 lambda x: x.update(streams=9), lambda x: x.update(streams=0)):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(bad)
    c = ModelConfig.from_hf_config(d)
    assert c.layer_specs[5].mixer.chunk == 0 and c.layer_specs[4].mixer.kv_from == 0
    assert not preset("mumusun-mini").recurrent and preset("small-hybrid").recurrent


@pytest.fixture(scope="module")
def snapshot(tmp_path_factory):
    from b200serve.utils.synth import write_listed
    path = str(tmp_path_factory.mktemp("mini"))
    return path, write_listed(preset("napadra-mini"), path, seed=3)


def test_loaded_weights_compute_the_layer(snapshot):
    """The padded kernel layout, multiplied out plainly, is the reference's layer."""
    from b200serve.loader.loader import load
    from b200serve.models.grouped import GroupedGeometry, LOG2E
    from b200serve.models.mlstm import MlstmGeometry
    from b200serve.models.weights import deinterleave16
    path, raw = snapshot
    w = load(path, device="cpu", dtype="float32", report=None)
    cfg, n = w.cfg, 30
    ref = {k: v.double() for k, v in raw.items()}
    h = torch.randn(n, cfg.hidden, generator=torch.Generator().manual_seed(1)).double()
    hp = torch.zeros(n, w.embed.shape[1], dtype=F64)
    hp[:, : cfg.hidden] = h
    pos, kept_ref, kept = torch.arange(n), {}, {}
    for i, (spec, lw, js) in enumerate(zip(cfg.layer_specs, w.layers, cfg.to_listed_config()["layers"])):
        a, m, p = spec.mixer, lw.mixer, f"l{i}.mix."
        if isinstance(a, GroupedAttention):
            g = GroupedGeometry.of(a)
            y = hp @ m.qkv.double().T
            q = y[:, : g.nq].view(n, a.heads, g.dk)
            if a.kv_from < 0:
                kept[i] = y[:, g.nq:].split([a.kv_heads * g.dk, a.kv_heads * g.dv], dim=1)
            k, v = (t.view(n, a.kv_heads, -1) for t in kept[i if a.kv_from < 0 else a.kv_from])
            assert torch.all(k[..., a.dim:] == 0) and torch.all(v[..., a.vdim:] == 0)
            assert torch.allclose(m.slope2.double() / LOG2E, O.alibi_slopes(a.heads))
            o = O.sink_attention(q, k, v, pos, pos, a.chunk or None, a.scale, m.sink2.double() / LOG2E)
            want = O.attention(ref, p, i if a.kv_from < 0 else a.kv_from, js["mixer"], h, kept_ref)
        else:
            g = MlstmGeometry.of(a)
            y = hp @ m.proj.double().T
            q, k, v, z = (t.view(n, a.heads, -1) for t in y[:, : g.n].split([a.heads * g.dk] * 2 + [a.heads * g.dv] * 2, dim=1))
            zi, zf = (y[:, g.n + j * a.heads: g.n + (j + 1) * a.heads] + m.gate_bias[j * a.heads: (j + 1) * a.heads].double() for j in (0, 1))
            o, _ = O.mlstm_scan(q * a.dim ** -0.5, k, v, *O.mlstm_gates(zi, zf, a.gate_cap))
            o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / a.vdim + cfg.rms_eps) * m.norm.view(a.heads, -1).double() * torch.sigmoid(z)
            want = O.mlstm(ref, p, js["mixer"], cfg.rms_eps, h)
        got = o.reshape(n, -1) @ m.o.double().T
        assert torch.allclose(got[:, : cfg.hidden], want, rtol=1e-5, atol=1e-6) and torch.all(got[:, cfg.hidden:] == 0)
        if spec.ffn is not None:
            gu = deinterleave16(hp @ lw.dense.gate_up.double().T)
            got = O.clamped_glu(*gu, spec.ffn.limit) @ lw.dense.down.double().T
            assert torch.allclose(got[:, : cfg.hidden], O.dense(ref, f"l{i}.mlp.", js["mlp"], h), rtol=1e-5, atol=1e-6)
        subs = (1,) if spec.ffn is None else (1, 2)
        for q, s in enumerate(subs):
            assert torch.equal(lw.streams.w_mix[q].view(cfg.block.streams, -1).double(), ref[f"l{i}.hc{s}.mix"])
            assert torch.equal(lw.streams.scale[q][: cfg.hidden].double(), ref[f"l{i}.ls{s}"]) and torch.all(lw.streams.scale[q][cfg.hidden:] == 0)


def test_loader_names_every_tensor_that_does_not_fit(snapshot, tmp_path):
    from safetensors.torch import save_file
    from b200serve.loader.loader import load
    path, raw = snapshot
    t = {k: v.clone() for k, v in raw.items() if k not in ("l1.mix.f.b", "l4.hc2.mix")}
    t["l0.shift"] = t["l0.shift"][:-1].clone()
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(preset("napadra-mini").to_hf_config()))
    with pytest.raises(ValueError) as e:
        load(str(tmp_path), device="cpu", report=None)
    assert all(x in str(e.value) for x in ("l1.mix.f.b: missing", "l4.hc2.mix: missing", "l0.shift: shape"))
    assert "l4.mix.k" not in str(e.value)            # a layer on another layer's keys has no projections of its own


def test_segment_tables():
    from b200serve.runtime.batch import segment_chunks, segment_tiles
    segs = [(2, 0, 300), (0, 77, 40), (1, 500, 130)]
    owner = [(s, p + i) for s, p, n in segs for i in range(n)]
    for chunk in (0, 1, 64, 200, 333):
        for per in (128, 256):
            seen = []
            for q0, rows, pos, slot in segment_tiles(segs, chunk, per):
                assert 1 <= rows <= per and all(owner[q0 + r] == (slot, pos + r) for r in range(rows))
                if chunk > per:
                    assert pos // chunk == (pos + rows - 1) // chunk
                seen += range(q0, q0 + rows)
            assert sorted(seen) == list(range(len(owner)))
    rows, chunks = segment_chunks(segs)
    assert rows == [(0, 300, 2, 0), (300, 40, 0, 5), (340, 130, 1, 6)] and chunks == 9


def test_planner_counts_pages_and_states():
    from b200serve.models.decoder import KVCache
    from b200serve.runtime import memory_plan as MP
    cfg = preset("napadra-mini")
    for form in ("bf16", "f32"):
        kv = KVCache(cfg, cfg.n_layers, 9, "cpu", form, n_slots=3)
        assert sum(t.numel() * t.element_size() for t in kv.page_tensors().values()) == 9 * MP.kv_bytes_per_page(cfg, form)
        held = sum(t.numel() * 4 for t in kv.states.values()) + kv.shift_next.numel() * 4
        assert held <= 3 * MP.state_bytes_per_slot(cfg) <= 2.1 * held
    assert set(kv.pages) == {"k0", "v0", "k2", "v2", "k5", "v5"} and set(kv.states) == {"mlstm1", "mlstm3", "shift"}
    with pytest.raises(ValueError):
        KVCache(cfg, cfg.n_layers, 9, "cpu", "int8")
    saved = kv.save_states(1)
    for t in kv.states.values():
        t.fill_(1)
    kv.load_states(1, saved)
    assert all(float(t[:, 1].abs().sum()) == 0 and float(t[:, 2].min()) == 1 for t in kv.states.values())
    big = preset("napadra-7b")
    assert MP.weight_bytes(big) >= 2 * big.param_count()
    a, b = MP.plan(big, 1, 16384), MP.plan(big, 8, 16384)
    assert b.total - a.total >= 7 * MP.state_bytes_per_slot(big)
    with pytest.raises(ValueError):
        MP.plan(big, 8, 65536, budget=20 * 2 ** 30)


def test_random_weights_and_refusals():
    from b200serve.cli import common
    from b200serve.models.weights import random_weights
    cfg = preset("napadra-mini")
    w = random_weights(cfg, seed=1)
    assert w.nbytes() > 2 * cfg.param_count() * 0.9 and torch.equal(w.layers[0].streams.w_mix[0].view(3, 3), torch.eye(3))
    with pytest.raises(ValueError):
        cfg.tp_shard(2)
    assert common.parallel_auto(preset("napadra-7b"), 8, 180 * 2 ** 30) == "1"
    with pytest.raises(SystemExit):
        common.load_model("napadra-mini", "cpu", int8_head=True)
    assert isinstance(cfg.layer_specs[1].mixer, MatrixLstm)
