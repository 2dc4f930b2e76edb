"""Pefulorn without a GPU: the plain reference by hand, configuration, checkpoint layout, order of layers, planning."""
import dataclasses
import json
import math

import pytest
import torch

import pefulorn_oracle as O
from b200serve.models.config import ChannelDelta, LayerLoop, ModelConfig, ParallelMixer, Wkv, preset

F64 = torch.float64


def gen(seed):
    return torch.Generator().manual_seed(seed)


def test_oracle_mechanisms_by_hand():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    assert torch.allclose(O.norm_one_plus(x, torch.tensor([0.0, 1.0], dtype=F64), 0.5), x / math.sqrt(13.0) * torch.tensor([1.0, 2.0]))
    assert torch.allclose(O.unit(x), x / math.sqrt(25 + 1e-6))
    g = float(O.gelu_tanh(torch.tensor(0.7, dtype=F64)))
    assert math.isclose(g, 0.35 * (1 + math.tanh(math.sqrt(2 / math.pi) * (0.7 + 0.044715 * 0.343))), rel_tol=1e-12)
    y = O.causal_conv(torch.tensor([[1.0], [10.0], [100.0]], dtype=F64), torch.tensor([[0.5, 2.0]], dtype=F64))
    assert y[:, 0].tolist() == [2.0, 20.5, 205.0]
    assert O.causal_conv(torch.ones(2, 1, dtype=F64), torch.ones(1, 5, dtype=F64))[:, 0].tolist() == [1.0, 2.0]
    d = O.channel_decay(torch.tensor([[0.3, -2.0]], dtype=F64), torch.tensor([0.5], dtype=F64), torch.tensor([0.1, 0.2], dtype=F64), 1)
    assert math.isclose(float(d[0, 0, 0]), math.exp(-math.exp(0.5) * math.log1p(math.exp(0.4))), rel_tol=1e-12)
    t = O.temperature(torch.tensor([0, 6, 7, 20]), 0.5, 7)
    assert torch.allclose(t, torch.tensor([1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(4)], dtype=F64))
    s, last = O.min_gru_scan(torch.tensor([[0.0], [2.0]], dtype=F64), torch.tensor([[1.0], [-1.0]], dtype=F64))
    z = 1 / (1 + math.exp(-2))
    assert torch.allclose(s[:, 0], torch.tensor([0.75, (1 - z) * 0.75 + z / (1 + math.e)], dtype=F64)) and torch.equal(last, s[-1])


def test_oracle_attention_by_hand():
    q, k = torch.tensor([[[1.0], [2.0]]], dtype=F64), torch.tensor([[[3.0]], [[1.0]]], dtype=F64)
    v, r1, r2 = torch.tensor([[[1.0]], [[10.0]]], dtype=F64), torch.tensor([0.7, 2.0], dtype=F64), torch.tensor([0.5, 3.0], dtype=F64)
    o = O.log_bias_attention(q, k, v, torch.tensor([1]), torch.arange(2), 0.5, r1, r2)[0, :, 0]
    for h, qq in enumerate((1.0, 2.0)):
        a, b = math.exp(qq * 1.5) * (1 + float(r2[h])) ** -float(r1[h]), math.exp(qq * 0.5)
        assert math.isclose(float(o[h]), (a + 10 * b) / (a + b), rel_tol=1e-12)


def test_oracle_recurrences_by_hand():
    """Sums over earlier rows written out; a sequence cut in two is the same sequence."""
    g = gen(1)
    t, a, b = 7, 3, 2
    q, k, v = (torch.randn(t, 1, n, generator=g, dtype=F64) for n in (a, a, b))
    w = torch.rand(t, 1, a, generator=g, dtype=F64)
    u = torch.randn(1, a, generator=g, dtype=F64)
    out, state = O.wkv_scan(q, k, v, w, u)
    for j in range(t):
        want = (q[j, 0] * u[0] * k[j, 0]).sum() * v[j, 0]
        for r in range(j):
            want = want + (q[j, 0] * k[r, 0] * w[r + 1: j, 0].prod(0)).sum() * v[r, 0]
        assert torch.allclose(out[j, 0], want)
    half, st = O.wkv_scan(q[:4], k[:4], v[:4], w[:4], u)
    assert torch.allclose(torch.cat([half, O.wkv_scan(q[4:], k[4:], v[4:], w[4:], u, st)[0]]), out)
    beta = torch.rand(t, 1, generator=g, dtype=F64)
    out, state = O.delta_scan(q, k, v, w, beta)
    wrote = []
    for j in range(t):
        seen = sum(((k[j, 0] * k[r, 0] * w[r + 1: j + 1, 0].prod(0)).sum() * wrote[r] for r in range(j)), torch.zeros(b, dtype=F64))
        wrote.append(beta[j, 0] * (v[j, 0] - seen))
        want = sum((q[j, 0] * k[r, 0] * w[r + 1: j + 1, 0].prod(0)).sum() * wrote[r] for r in range(j + 1))
        assert torch.allclose(out[j, 0], want)


def test_order_of_layers():
    c = dataclasses.replace(preset("pefulorn-mini"), loop=LayerLoop(1, 3, 2))
    assert c.layer_runs == ((0, -1), (1, 0), (2, -1), (1, 1), (2, -1), (3, -1), (4, -1), (5, -1))
    js = c.to_listed_config()
    assert [(i, -1 if b is None else b) for i, b in O.order_of(js)] == list(c.layer_runs)
    assert dataclasses.replace(c, loop=None).layer_runs == tuple((i, -1) for i in range(6))
    assert [c.run_specs[j].mixer for j in c.shift_runs] == [c.layer_specs[i].mixer for i in (2, 2, 4)]
    assert c.kv_bytes_per_token() == 2 * sum(s.mixer.kv_elems for s in c.run_specs)
    once = dataclasses.replace(c, loop=None)
    assert c.weight_bytes_per_token() > once.weight_bytes_per_token() and c.param_count() == once.param_count()


def test_config_round_trip_and_refusals():
    for name in ("pefulorn-mini", "pefulorn-7b"):
        c = preset(name)
        back = ModelConfig.from_hf_config(json.loads(json.dumps(c.to_hf_config())))
        bare = [dataclasses.replace(s, mixer=dataclasses.replace(s.mixer, **{f.name: 0 for f in dataclasses.fields(s.mixer) if f.name.endswith("_rank")}))
                for s in c.layer_specs]           # ranks are in the tensors
        assert list(back.layer_specs) == bare and (back.block, back.loop) == (c.block, c.loop) and back.recurrent
        assert (back.hidden, back.vocab, back.rms_eps) == (c.hidden, c.vocab, c.rms_eps)
    d = preset("pefulorn-mini").to_hf_config()

    def mixer(i, **kw):
        return lambda x: x["layers"][i]["mixer"].update(kw)
    for edit in (lambda x: x["layers"][0].update(type="mamba"), lambda x: x["layers"][0]["mlp"].update(kind="moe"), mixer(1, kv_heads=4),
                 mixer(1, conv=0), mixer(1, conv=17), mixer(2, dim=600), mixer(1, vdim=513), lambda x: x["loop"].update(stop=7),
                 lambda x: x["loop"].update(times=0), lambda x: x["loop"].update(start=4), lambda x: x["layers"][0]["mixer"]["left"].update(kv_heads=4),
                 lambda x: x["layers"][0]["mixer"]["left"].update(dim=1025)):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(bad)
    for value in (None, "absent"):
        e = json.loads(json.dumps(d))
        if value is None:
            e["loop"] = None
        else:
            del e["loop"]
        assert ModelConfig.from_hf_config(e).loop is None
    del d["layers"][0]["mixer"]["left"]["q_temp"]
    assert ModelConfig.from_hf_config(d).layer_specs[0].mixer.left.temp == 0.0


@pytest.fixture(scope="module")
def snapshot(tmp_path_factory):
    from b200serve.utils.synth import write_listed
    path = str(tmp_path_factory.mktemp("mini"))
    return path, write_listed(preset("pefulorn-mini"), path, seed=3, make=lambda n, t: t - 1 if "norm" in n and ".mix." not in n else t)


def test_sizes_come_from_the_tensors(snapshot):
    from b200serve.cli.common import peek_config
    path, raw = snapshot
    assert peek_config(path).layer_specs == preset("pefulorn-mini").layer_specs
    assert raw["l1.mix.a1"].shape[0] != raw["l1.mix.g1"].shape[0]


def test_loaded_weights_compute_the_layer(snapshot):
    """The padded kernel layout, multiplied out plainly, is the reference's layer."""
    from b200serve.loader.loader import load
    from b200serve.models.channel_delta import DeltaGeometry
    from b200serve.models.grouped import GroupedGeometry
    from b200serve.models.weights import deinterleave16
    from b200serve.models.wkv import WkvGeometry
    path, raw = snapshot
    w = load(path, device="cpu", dtype="float32", report=None)
    cfg, n, eps = w.cfg, 20, w.cfg.rms_eps
    assert cfg.layer_specs == preset("pefulorn-mini").layer_specs
    ref = {k: v.double() for k, v in raw.items()}
    h = torch.randn(n, cfg.hidden, generator=gen(1)).double()

    def pad(x, cols):
        out = torch.zeros(len(x), cols, dtype=F64)
        out[:, : x.shape[1]] = x
        return out
    wp = w.embed.shape[1]
    hp, pos = pad(h, wp), torch.arange(n)
    norm = lambda o, dims: o / torch.sqrt((o * o).sum(-1, keepdim=True) / dims + eps)        # noqa: E731
    for i, (spec, lw, js) in enumerate(zip(cfg.layer_specs, w.layers, cfg.to_listed_config()["layers"])):
        a, m, p = spec.mixer, lw.mixer, f"l{i}.mix."
        if isinstance(a, ChannelDelta):
            g = DeltaGeometry.of(a)
            y = hp @ m.proj.double().T
            c = O.silu(O.causal_conv(y[:, : g.channels], m.conv.double().T))
            q, k, v = c.split([g.kv_heads * g.dk] * 2 + [g.heads * g.dv], dim=1)
            q, k = (O.unit(x.view(n, g.kv_heads, g.dk)).repeat_interleave(g.heads // g.kv_heads, dim=1) for x in (q, k))
            low = [pad(y[:, col: col + r], g.kp) for col, r in ((g.col_a1, a.a_rank), (g.col_g1, a.g_rank))]
            z, gate = low[0] @ m.second[: g.heads * g.dk].double().T, low[1] @ m.second[g.heads * g.dk:].double().T
            decay = torch.exp(-m.neg_a.double()[:, None] * torch.nn.functional.softplus(z + m.dt_bias.double()).view(n, g.heads, g.dk))
            o, _ = O.delta_scan(q * a.dim ** -0.5, k, v.view(n, g.heads, g.dv), decay, torch.sigmoid(y[:, g.col_b: g.col_b + g.heads]))
            got = norm(o, a.vdim).reshape(n, -1) * m.norm.double() * torch.sigmoid(gate) @ m.o.double().T
            want = O.channel_delta(ref, p, js["mixer"], eps, h)
        elif isinstance(a, Wkv):
            g = WkvGeometry.of(a)
            mix = hp + (O.previous(hp) - hp) * m.shift.double()[:, None]
            rows = m.proj.double()
            r, k, v, gate = ((mix[j] @ rows[j * g.hd: (j + 1) * g.hd].T) for j in range(4))
            low = pad(torch.tanh(mix[4] @ rows[4 * g.hd: 4 * g.hd + a.w_rank].T), g.kp)
            decay = torch.exp(-torch.exp(low @ m.second.double().T + m.w0.double()))
            o, _ = O.wkv_scan(*(x.view(n, g.heads, g.d) for x in (r, k, v, decay)), m.u.view(g.heads, g.d).double())
            got = norm(o, a.dim).reshape(n, -1) * m.norm.double() * O.silu(gate) @ m.o.double().T
            want = O.wkv(ref, p, js["mixer"], eps, h)
        else:
            assert isinstance(a, ParallelMixer)
            left, g = a.left, GroupedGeometry.of(a.left)
            y = hp @ m.proj.double().T
            qkv = y[:, : g.nq + g.nkv] + m.left.bias.double()
            q, k, v = qkv.split([g.nq, g.kv_heads * g.dk, g.kv_heads * g.dv], dim=1)
            q = norm(q.view(n, g.heads, g.dk), left.dim) * m.left.q_norm.double() * O.temperature(pos, left.temp, left.temp_every)[:, None, None]
            k, v = norm(k.view(n, -1, g.dk), left.dim) * m.left.k_norm.double(), norm(v.view(n, -1, g.dv), left.vdim)
            o = O.log_bias_attention(q, k, v, pos, pos, left.scale, m.left.r1.double(), m.left.r2.double()).reshape(n, -1)
            z, u, gate = y[:, g.nq + g.nkv:].chunk(3, dim=1)
            s, _ = O.min_gru_scan(z + m.right.bias_z.double(), u + m.right.bias_x.double())
            got = torch.cat([a.left_scale * o, a.right_scale * s * O.silu(gate)], dim=1) @ m.o.double().T
            want = O.parallel(ref, p, js["mixer"], eps, h)
        assert torch.allclose(got[:, : cfg.hidden], want, rtol=1e-5, atol=1e-6), type(a)
        assert torch.all(got[:, cfg.hidden:] == 0)
        if spec.ffn is not None:
            gu = deinterleave16(hp @ lw.dense.gate_up.double().T + lw.dense.bias.double())
            got = O.gelu_tanh(gu[0]) * gu[1] @ lw.dense.down.double().T + lw.dense.down_bias.double()
            assert torch.allclose(got[:, : cfg.hidden], O.dense(ref, f"l{i}.mlp.", h), rtol=1e-5, atol=1e-6)
            assert torch.equal(lw.post_norm[: cfg.hidden].double(), (1 + ref[f"l{i}.norm2"].float()).double()) and torch.all(lw.post_norm[cfg.hidden:] == 0)
    assert torch.equal(w.loop_step[:, : cfg.hidden].double(), ref["loop.step"])


def test_low_rank_weights_in_two_limbs(snapshot):
    """bf16 models hold the second halves twice side by side."""
    from b200serve.loader.loader import load
    w, f = (load(snapshot[0], device="cpu", dtype=d, report=None) for d in ("bfloat16", "float32"))
    for i in (1, 2):
        a, b = w.layers[i].mixer.second.float(), f.layers[i].mixer.second
        assert torch.equal(a[:, : b.shape[1]], b) and torch.equal(a[:, b.shape[1]:], b)


def test_loader_names_every_tensor_that_does_not_fit(snapshot, tmp_path):
    from safetensors.torch import save_file
    from b200serve.loader.loader import load
    path, raw = snapshot
    t = {k: v.clone() for k, v in raw.items() if k not in ("l1.mix.a1", "l0.mix.right.x.b", "loop.step")}
    t["l2.mix.w2"] = t["l2.mix.w2"][:, :-1].clone()
    t["l0.mlp.down.b"] = t["l0.mlp.down.b"][:-1].clone()
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(preset("pefulorn-mini").to_hf_config()))
    with pytest.raises(ValueError) as e:
        load(str(tmp_path), device="cpu", report=None)
    for x in ("l1.mix.a1: missing", "l0.mix.right.x.b: missing", "loop.step: missing", "l2.mix.w2: shape", "l0.mlp.down.b: shape"):
        assert x in str(e.value)


def test_planner_counts_pages_and_states_of_runs():
    from b200serve.models.decoder import KVCache
    from b200serve.runtime import memory_plan as MP
    cfg = preset("pefulorn-mini")
    for form in ("bf16", "f32"):
        kv = KVCache(cfg, cfg.n_layers, 9, "cpu", form, n_slots=3)
        assert sum(t.numel() * t.element_size() for t in kv.page_tensors().values()) == 9 * MP.kv_bytes_per_page(cfg, form)
        held = sum(t.numel() * 4 for t in kv.states.values()) + kv.shift_next.numel() * 4
        assert held <= 3 * MP.state_bytes_per_slot(cfg) <= 2.1 * held
    # layer 3 (attention beside a minGRU) runs three times, as do the delta-rule and time-mixing layers before it
    assert set(kv.pages) == {f"{x}{j}" for x in "kv" for j in (0, 3, 6, 9)}
    assert {n for n in kv.states if n.startswith("wkv")} == {"wkv2", "wkv5", "wkv8", "wkv10"}
    assert len(kv.states["shift"]) == 4 and {"delta1", "conv4", "delta7", "delta11", "gru9"} <= set(kv.states)
    big = preset("pefulorn-7b")
    assert MP.weight_bytes(big) >= 2 * big.param_count()
    assert MP.plan(big, 8, 16384).total - MP.plan(big, 1, 16384).total >= 7 * MP.state_bytes_per_slot(big)


def test_random_weights_and_refusals():
    from b200serve.cli import common
    from b200serve.models.config import LayerSpec, StreamBlock, listed_config
    from b200serve.models.listed import ListedLayers, random_listed_weights
    from b200serve.models.weights import random_weights
    cfg = preset("pefulorn-mini")
    w = random_weights(cfg, seed=1)
    assert w.nbytes() > 2 * cfg.param_count() * 0.9 and w.loop_step.shape == (3, 256)
    assert torch.equal(w.layers[0].input_norm, (torch.arange(256) < 200).float())       # norms around one
    with pytest.raises(ValueError):
        cfg.tp_shard(2)
    assert common.parallel_auto(preset("pefulorn-7b"), 8, 180 * 2 ** 30) == "1"
    with pytest.raises(SystemExit):
        common.load_model("pefulorn-mini", "cpu", int8_head=True)
    specs = (LayerSpec(Wkv(2, 64, 16), None),)
    for bad in (listed_config("a", "Mumusun", specs, 64, 50, 1e-5), listed_config("b", "Mumusun", cfg.layer_specs[1:2], 64, 50, 1e-5, loop=LayerLoop(0, 1, 2))):
        with pytest.raises(ValueError):         # shifted inputs and passes need the pre-normed residual
            ListedLayers(random_listed_weights(bad), 64)
    plain = StreamBlock(2, 1.0, shift=False, scale=False, sinusoid=0.0, mixing=False, columns=True)
    from b200serve.models.streams import StreamWalk
    with pytest.raises(ValueError):
        StreamWalk(ListedLayers(random_listed_weights(listed_config("c", "Pefulorn", specs, 64, 50, 1e-5, plain)), 64))
