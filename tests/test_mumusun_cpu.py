"""Mumusun without a GPU: configuration, checkpoint layout, batch tables, planning, the scheduler's mixed steps."""
import dataclasses
import json

import numpy as np
import pytest
import torch

import mumusun_oracle as O
from b200serve.models.config import ModelConfig, preset


def test_oracle_mechanisms_by_hand():
    x = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    assert torch.allclose(O.layer_norm(x, torch.tensor([1.0, 2.0], dtype=torch.float64), 3.0), torch.tensor([[-0.5, 1.0]], dtype=torch.float64))
    assert torch.allclose(O.rms_norm(x, torch.ones(2, dtype=torch.float64), 4.0), x / 3.0)
    v = torch.tensor([[1.0, 0.0, 0.0, 2.0, 9.0]], dtype=torch.float64)      # pairs (0, 2) and (1, 3); element 4 passes
    r = O.rotate(v, torch.tensor([2]), 4, 100.0)[0]
    a, b = 2.0, 0.2
    want = torch.tensor([np.cos(a), -2 * np.sin(b), np.sin(a), 2 * np.cos(b), 9.0])
    assert torch.allclose(r, want)
    vis = O.visible(torch.tensor([5]), torch.arange(8), 3)[0].tolist()
    assert vis == [False, False, False, True, True, True, False, False]
    z = torch.tensor([3.0, -9.0, 2.0, 2.0, 2.9, 2.9], dtype=torch.float64)   # groups of two: best sums 2 (4, 5) then 1 (2, 3)
    got = O.route(z, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert [e for e, _ in got] == [4, 5, 2] and torch.allclose(got[0][1], torch.sigmoid(z[4]))


def test_config_round_trip_and_refusals():
    for name in ("mumusun-mini", "mumusun-16b"):
        c = preset(name)
        d = json.loads(json.dumps(c.to_hf_config()))
        back = ModelConfig.from_hf_config(d)
        assert back.layer_specs == c.layer_specs and (back.hidden, back.vocab, back.rms_eps) == (c.hidden, c.vocab, c.rms_eps)
    d = preset("mumusun-mini").to_hf_config()
    for edit in (lambda x: x["layers"][0].update(type="recurrent"), lambda x: x["layers"][0]["mlp"].update(kind="dense"),
                 lambda x: x["layers"][0]["mlp"]["router"].update(top=9), lambda x: x["layers"][0]["mixer"]["rot"].update(dims=34)):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(bad)
    free = json.loads(json.dumps(d))
    free["layers"][0]["mixer"].pop("mask")
    assert ModelConfig.from_hf_config(free).layer_specs[0].mixer.window == 0


@pytest.fixture(scope="module")
def snapshot(tmp_path_factory):
    from b200serve.utils.synth import write_listed
    path = str(tmp_path_factory.mktemp("mini"))
    return path, write_listed(preset("mumusun-mini"), path, seed=3)


def test_loaded_weights_compute_the_layer(snapshot):
    """The padded kernel layout, multiplied out plainly, is the reference's layer: attention against the latent, experts
    from the interleaved stack."""
    from b200serve.loader.loader import load
    from b200serve.models.latent import LatentGeometry
    from b200serve.models.weights import deinterleave16
    path, raw = snapshot
    w = load(path, device="cpu", dtype="float32", report=None)
    cfg, n = w.cfg, 50
    ref = {k: v.double() for k, v in raw.items()}
    h = torch.randn(n, cfg.hidden, generator=torch.Generator().manual_seed(1)).double()
    hp = torch.zeros(n, w.embed.shape[1], dtype=torch.float64)
    hp[:, : cfg.hidden] = h
    pos = torch.arange(n)
    for i, (spec, lw, js) in enumerate(zip(cfg.layer_specs, w.layers, cfg.to_listed_config()["layers"])):
        a, g, m = spec.mixer, LatentGeometry.of(spec.mixer), lw.mixer
        d = hp @ m.down.double().T
        assert torch.all(d[:, a.q_rank: g.qp] == 0) and torch.all(d[:, g.qp + a.kv_rank: g.qp + g.kvp] == 0)
        cq = torch.zeros(n, g.qp, dtype=torch.float64)
        cq[:, : a.q_rank] = O.rms_norm(d[:, : a.q_rank], m.q_norm.double(), cfg.rms_eps)
        c = torch.zeros(n, g.kvp, dtype=torch.float64)
        c[:, : a.kv_rank] = O.rms_norm(d[:, g.qp: g.qp + a.kv_rank], m.kv_norm.double(), cfg.rms_eps)
        kr = O.rotate(d[:, g.qp + g.kvp: g.qp + g.kvp + a.rot_dim], pos, a.rope_dims, a.rope_base)
        q = (cq @ m.uq.double().T).view(n, a.heads, g.dk)
        qa = torch.einsum("nhd,hdr->nhr", q[..., : g.dn], m.uk.double().view(a.heads, g.dn, g.kvp))
        qr = O.rotate(q[..., g.dn: g.dn + a.rot_dim], pos, a.rope_dims, a.rope_base)
        o = O.softmax_attention(torch.cat([qa, qr], -1), torch.cat([c, kr], -1)[:, None].expand(-1, a.heads, -1),
                                c[:, None].expand(-1, a.heads, -1), O.visible(pos, pos, a.window), a.scale)
        v = torch.einsum("nhr,hvr->nhv", o, m.uv.double().view(a.heads, g.dv, g.kvp)).reshape(n, -1)
        out = v @ m.o.double().T
        want = O.latent_attention(ref, f"l{i}.mix.", js["mixer"], cfg.rms_eps, h, pos)
        assert torch.allclose(out[:, : cfg.hidden], want, atol=1e-6) and torch.all(out[:, cfg.hidden:] == 0)
        if spec.ffn is None:
            assert lw.moe is None and lw.post_norm is None
            continue
        y = torch.zeros(n, w.embed.shape[1], dtype=torch.float64)
        z = hp @ lw.moe.router.double().T
        for t in range(n):
            for e, s in O.route(z[t, : spec.ffn.experts], js["mlp"]["router"]):
                gate, up = deinterleave16(lw.moe.gate_up[e].double() @ hp[t])
                y[t] += s * (lw.moe.down[e].double() @ (O.silu(gate) * up))
        assert torch.allclose(y[:, : cfg.hidden], O.moe(ref, f"l{i}.mlp.", js["mlp"], h), atol=1e-6)


def test_loader_names_every_tensor_that_does_not_fit(snapshot, tmp_path):
    from b200serve.loader.loader import load
    from b200serve.utils.safetensors_io import save_file
    path, raw = snapshot
    bad = dict(raw)
    bad.pop("l1.mix.uk")
    bad["l0.norm2"] = torch.ones(7, dtype=torch.bfloat16)
    save_file(bad, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(open(path + "/config.json").read())
    with pytest.raises(ValueError) as e:
        load(str(tmp_path), device="cpu", report=None)
    assert "l1.mix.uk: missing" in str(e.value) and "l0.norm2: shape" in str(e.value)
    with pytest.raises(ValueError):
        load(path, device="cpu", tp=(0, 2), report=None)
    with pytest.raises(ValueError):
        load(path, device="cpu", int8_head=True, report=None)


def test_segment_keys_cover_what_rows_see():
    from b200serve.runtime.batch import segment_keys
    segs = [(2, 0, 300), (0, 77, 40), (1, 500, 130)]
    for window in (0, 1, 64, 333):
        for per in (128, 256):
            kreq, kpos, tiles = segment_keys(segs, window, per)
            owner = [(s, p + i) for s, p, n in segs for i in range(n)]
            seen = set()
            for q0, rows, rel, krow in tiles:
                assert 1 <= rows <= per
                for r in range(rows):
                    slot, pos = owner[q0 + r]
                    seen.add(q0 + r)
                    first = max(0, pos - window + 1) if window else 0
                    # the row's own key, and the first one it sees, are where the tile says
                    own = krow + rel + r
                    assert (kreq[own], kpos[own]) == (slot, pos)
                    assert (kreq[own - (pos - first)], kpos[own - (pos - first)]) == (slot, first)
            assert seen == set(range(len(owner)))


def test_batch_tables_number_single_rows_first():
    from b200serve.runtime.batch import BatchRunner
    b = BatchRunner.__new__(BatchRunner)
    form = ("keys", 64, 256)
    b.forms = [form]
    host, spans, tables = b._tables([(1, 9, [5]), (3, 0, [7, 8])], [(0, 100, list(range(40)))], np.asarray([2, 42]))
    cut = lambda s: host[s[0]: s[0] + s[1]].tolist()     # noqa: E731
    assert cut(spans["req"])[:4] == [1, 3, 3, 0] and cut(spans["pos"])[:4] == [9, 0, 1, 100]
    assert cut(spans["token"])[:4] == [5, 7, 8, 0] and cut(spans["want"]) == [2, 42]
    used = []
    t = tables[form](lambda span: used.append(span) or cut(span))
    assert t.n_keys == 40 + 63 and t.kpos[0] == 37 and t.n_tiles == 1 and t.tiles == [0, 40, 63, 0]
    assert all(s[0] % 4 == 0 for s in (*spans.values(), *used))


def test_planner_counts_pages_and_refuses():
    from b200serve.models.decoder import KVCache
    from b200serve.runtime import memory_plan as MP
    cfg = preset("mumusun-mini")
    for form in ("bf16", "f32"):
        kv = KVCache(cfg, cfg.n_layers, 9, "cpu", form)
        held = sum(t.numel() * t.element_size() for t in kv.page_tensors().values())
        assert held == 9 * MP.kv_bytes_per_page(cfg, form)
        assert all(t.shape[1] == 9 for t in kv.page_tensors().values())
    with pytest.raises(ValueError):
        KVCache(cfg, cfg.n_layers, 9, "cpu", "int8")
    big = preset("mumusun-16b")
    assert MP.weight_bytes(big) >= 2 * big.param_count()
    p = MP.plan(big, 8, 65536, budget=180 * 2 ** 30)
    assert p.resident_bf16 == 0 and p.num_pages == 8 * 4096 + 1
    with pytest.raises(ValueError):
        MP.plan(big, 8, 65536, budget=20 * 2 ** 30)


def test_step_scratch_stays_within_the_planner_figure():
    from b200serve.models.listed import ListedScratch
    sc = ListedScratch("cpu", torch.float32, fixed=8)
    a = sc.get("x", 3, 16)
    assert a.shape == (3, 16) and sc.get("x", 8, 16).data_ptr() == a.data_ptr()
    assert sc.get("x", 2, 32).data_ptr() != a.data_ptr()            # another width is another buffer
    with pytest.raises(RuntimeError):
        sc.get("x", 9, 16)                                          # captured graphs hold its address
    free = ListedScratch("cpu", torch.float32)
    free.get("x", 4, 4)[:] = 1
    assert torch.all(free.get("x", 40, 4) == 0)


def test_not_sliced_over_gpus():
    from b200serve.cli import common
    cfg = preset("mumusun-16b")
    with pytest.raises(ValueError):
        cfg.tp_shard(2)
    assert common.parallel_auto(cfg, 8, 180 * 2 ** 30) == "1"
    with pytest.raises(SystemExit):
        common.parallel_auto(cfg, 8, 16 * 2 ** 30)
    with pytest.raises(SystemExit):
        common.load_model("tiny-dense", "cpu", dtype="float32")
    with pytest.raises(SystemExit):
        common.load_model("mumusun-mini", "cpu", int8_head=True)


def test_trace_flags_and_admission():
    from b200serve.cli import trace as T
    from b200serve.cli.flags import parse
    f = parse(T.TraceFlags, ["--model", "m", "--dtype", "float32", "--out", "o", "--max-tokens", "640"], "trace_run", "x")
    assert (f.model, f.dtype, f.out, f.max_tokens) == ("m", "float32", "o", 640)

    class Eng:
        max_seqs = 2
        log = []

        def reset(self, s):
            self.log.append(("reset", s))

        def forward_batch(self, batch):
            self.log.append(batch)
    r = T.Replay(Eng())
    r.step([{"id": "x", "tokens": [1, 2], "want": [1]}, {"id": "y", "tokens": [3]}])
    assert Eng.log[-1] == [(0, [1, 2], [1]), (1, [3], [])]
    with pytest.raises(RuntimeError):
        r.step([{"id": "z", "tokens": [1]}])
    r.end("x")
    r.step([{"id": "z", "tokens": [4]}, {"id": "y", "tokens": [5]}])
    assert Eng.log[-1] == [(0, [4], []), (1, [5], [])]


def test_scheduler_runs_prompt_chunks_and_decode_rows_as_one_batch():
    """A server over an engine with mixed batches makes one call per tick where another engine gets two, with the same
    tokens."""
    import http.client
    import threading
    from b200serve.server.app import Server, ServerOptions
    from b200serve.server.chat_template import ChatTemplate
    from b200serve.server.iface import ByteTok, MockEngine

    def serve(mixed):
        eng = MockEngine(vocab_size=259, max_len=2048, max_seqs=3, step_delay=0.002)
        eng.mixed_batches = mixed
        srv = Server(eng, ByteTok(), ChatTemplate(), ServerOptions(prefill_chunk=16)).start()
        out = {}

        def post(i):
            c = http.client.HTTPConnection("127.0.0.1", srv.port, timeout=30)
            c.request("POST", "/v1/completions", json.dumps({"prompt": [3 + i] * (30 + 50 * i), "max_tokens": 40, "temperature": 0,
                                                             "ignore_eos": True, "return_token_ids": True}),
                      {"Content-Type": "application/json"})
            out[i] = json.loads(c.getresponse().read())["choices"][0]["token_ids"]
        ts = [threading.Thread(target=post, args=(i,)) for i in range(3)]
        for t in ts:
            t.start()
        for t in ts:
            t.join()
        srv.stop()
        return out, getattr(eng, "mixed_steps", 0)
    plain, none = serve(False)
    both, some = serve(True)
    assert none == 0 and some > 0 and plain == both and all(len(v) == 40 for v in both.values())


def test_a_failed_mixed_step_fails_its_requests_only():
    import http.client
    from b200serve.server.app import Server, ServerOptions
    from b200serve.server.chat_template import ChatTemplate
    from b200serve.server.iface import ByteTok, MockEngine
    eng = MockEngine(vocab_size=259, max_len=2048, max_seqs=2, step_delay=0.01)
    eng.mixed_batches = True
    real = eng.step_mixed

    def failing(slot, ids, rows):
        eng.step_mixed = real
        raise RuntimeError("lost")
    eng.step_mixed = failing
    srv = Server(eng, ByteTok(), ChatTemplate(), ServerOptions(prefill_chunk=16)).start()

    def post(n, out):
        c = http.client.HTTPConnection("127.0.0.1", srv.port, timeout=30)
        c.request("POST", "/v1/completions", json.dumps({"prompt": [9] * n, "max_tokens": 60, "temperature": 0, "ignore_eos": True}),
                  {"Content-Type": "application/json"})
        out.append(c.getresponse().status)
    import threading
    a, b, c = [], [], []
    t = [threading.Thread(target=post, args=(10, a)), threading.Thread(target=post, args=(200, b))]
    for x in t:
        x.start()
    for x in t:
        x.join()
    post(20, c)
    srv.stop()
    assert sorted(a + b) in ([500, 500], [200, 500]) and c == [200]
