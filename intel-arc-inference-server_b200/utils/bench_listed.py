"""Throughput of models that list their layers, beside the framework's closest other model at equal size.

Decode: captured steps of 1, 8, 16 and 64 requests at one depth (one row each, positions advance on the device).  Prompt:
whole prompt passes through ``Engine.prefill``.  Both are timed with CUDA events after warm-up; the weights a step reads
are far more than the L2 holds.  The comparison models have the framework's W4A16 weights.
"""
from __future__ import annotations

import dataclasses

import torch

from ..models.config import (DenseFfn, GroupedAttention, LayerSpec, MatrixLstm, ModelConfig, listed_config, pefulorn_like,
                             preset, vogerax_like)
from ..models.weights import random_weights
from ..ops import lib as K
from ..runtime.engine import Engine


def mumusun_sizes():
    """(latent-attention mixture of experts, grouped-query mixture of experts) pairs: the same width, layers, experts, experts
    per token, query heads and window."""
    out = []
    big = preset("mumusun-16b")
    spec = big.layer_specs[0]
    small = dataclasses.replace(spec, mixer=dataclasses.replace(spec.mixer, heads=8, q_rank=768, kv_rank=256, window=2048),
                                ffn=dataclasses.replace(spec.ffn, experts=32, top=4, ff=768, groups=4, keep=2))
    wide = dataclasses.replace(spec, mixer=dataclasses.replace(spec.mixer, heads=32), ffn=dataclasses.replace(spec.ffn, ff=2048))
    for cfg in (big, listed_config("mumusun-2b", "Mumusun", (small,) * 24, 1024, 65536, 1e-6),
                listed_config("mumusun-wide-12l", "Mumusun", (wide,) * 12, 4096, 102400, 1e-6)):
        a, f = cfg.layer_specs[0].mixer, cfg.layer_specs[0].ffn
        out.append((cfg, ModelConfig(f"gqa-moe-like-{cfg.name}", cfg.n_layers, cfg.hidden, a.heads, max(1, a.heads // 4), 128, 0,
                                     cfg.vocab, n_experts=f.experts, top_k=f.top, expert_ffn=f.ff, shared_ffn=0,
                                     sliding_window=a.window, architecture="B200MoeForCausalLM")))
    return out


def napadra_sizes():
    """(mLSTM and chunked attention over residual streams, gated delta-net and softmax attention) pairs: the same width,
    layers, feed-forwards, attention heads, and key and value dimensions of the recurrent layers; every second layer is
    recurrent.  Contexts stay inside one chunk, so the attention layers of both see every earlier position."""
    out = []
    big = preset("napadra-7b")

    def like(name, width, layers, heads, kv, rec, ff, vocab):
        f, specs = DenseFfn(ff, 7.0, 1.702, 1.0), []
        att = GroupedAttention(heads, kv, 128, 128, 128 ** -0.5, 8192, 8.0, True)
        for i in range(0, layers, 4):
            specs += [LayerSpec(rec, f)] * 2 + [LayerSpec(att, f), LayerSpec(dataclasses.replace(att, kv_from=i + 2), f)]
        return listed_config(name, "Napadra", specs, width, vocab, 1e-5, big.block)
    for cfg in (big, like("napadra-1b", 2048, 24, 16, 4, MatrixLstm(16, 128, 128, 15.0), 5632, 64000),
                like("napadra-wide-8l", 8192, 8, 64, 8, MatrixLstm(16, 256, 512, 15.0), 22016, 64000)):
        r, a, f = cfg.layer_specs[0].mixer, cfg.layer_specs[2].mixer, cfg.layer_specs[0].ffn
        out.append((cfg, ModelConfig(f"hybrid-like-{cfg.name}", cfg.n_layers, cfg.hidden, a.heads, a.kv_heads, 128, f.ff, cfg.vocab,
                                     full_attn_every=2, gdn_k_heads=r.heads * r.dim // 128, gdn_v_heads=r.heads * r.vdim // 128,
                                     architecture="B200HybridForCausalLM")))
    return out


def pefulorn_sizes():
    """(delta rule with channel decays, time mixing and attention beside a minGRU; gated delta-net and softmax attention) pairs:
    the same width, layers, feed-forwards, attention heads and recurrent heads; three layers of four are recurrent."""
    out = []
    for cfg in (preset("pefulorn-7b"), pefulorn_like("pefulorn-1b", 2048, 24, 16, 4, 5632, 64000, 64),
                pefulorn_like("pefulorn-wide-8l", 8192, 8, 64, 8, 22016, 64000)):
        a, f = cfg.layer_specs[3].mixer.left, cfg.layer_specs[0].ffn
        out.append((cfg, ModelConfig(f"hybrid-like-{cfg.name}", cfg.n_layers, cfg.hidden, a.heads, a.kv_heads, 128, f.ff, cfg.vocab,
                                     full_attn_every=4, gdn_k_heads=a.heads, gdn_v_heads=a.heads,
                                     architecture="B200HybridForCausalLM")))
    return out


def vogerax_sizes():
    """(windowed attention with pooled blocks, gated attention beside retention and ungated experts; grouped-query mixture of
    experts) pairs: the same width, layers, query and key heads, window, experts, experts per token and weights per expert (two
    matrices here, three there); every fourth layer sees the whole context."""
    out = []
    for cfg in (preset("vogerax-16b"), vogerax_like("vogerax-2b", 1024, 24, 8, 2, 768, 32, 4, 65536, 1024),
                vogerax_like("vogerax-wide-12l", 4096, 12, 32, 8, 1536, 64, 6, 102400)):
        a, f = cfg.layer_specs[0].mixer, cfg.layer_specs[0].ffn
        ff = f.ff * 2 // 3 // 64 * 64
        out.append((cfg, ModelConfig(f"gqa-moe-like-{cfg.name}", cfg.n_layers, cfg.hidden, a.heads, a.kv_heads, 128, 0, cfg.vocab,
                                     n_experts=f.experts, top_k=f.top, expert_ffn=ff, shared_ffn=2 * ff, sliding_window=a.window,
                                     full_attn_every=4, architecture="B200MoeForCausalLM")))
    return out


SIZES = {"mumusun": mumusun_sizes, "napadra": napadra_sizes, "pefulorn": pefulorn_sizes, "vogerax": vogerax_sizes}


def _timed(fn, warm: int, reps: int) -> float:
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps


def bench_model(cfg: ModelConfig, depth: int = 4096, prompt: int = 4096, rows=(1, 8, 16, 64), steps: int = 32, warm: int = 4) -> dict:
    w = random_weights(cfg, device="cuda", seed=0, exact=False)
    g = torch.Generator().manual_seed(0)
    ids = torch.randint(0, cfg.vocab, (max(depth, prompt),), generator=g).tolist()
    out = {}
    need = depth + (steps + warm + 2) * 2 + 64
    eng = Engine(w, max_seqs=max(rows), max_len=max(need, prompt + 64))
    first = eng.prefill(0, ids[:depth])
    for s in range(1, max(rows)):       # the other requests start from a copy of the first one's pages
        eng._ensure_pages(s, depth)
        src, dst = (torch.tensor(eng.pool.table(i)[: (depth + 15) // 16], device="cuda") for i in (0, s))
        for t in eng.kv.page_tensors().values():
            t.index_copy_(1, dst, t.index_select(1, src))
        eng.seq_len[s] = depth
    states = eng.kv.save_states(0)
    for m in rows:
        for s in range(m):
            if eng.kv.states:           # positions after ``depth`` are written again; the state goes back to what it was
                eng.kv.load_states(s, states)
                eng.seq_len[s] = depth
            else:
                eng.truncate(s, depth)
        # unlike tokens, so that the rows' experts differ
        eng.decode_begin(list(range(m)), [(first + 997 * i) % cfg.vocab for i in range(m)])
        ms = _timed(lambda: eng.decode_step(read=False), warm, steps)
        out[f"decode_rows_{m}"] = {"ms_per_step": ms, "tokens_per_s": m * 1e3 / ms, "launches_per_step": eng.launches(m, True)}

    def one_prompt():
        eng.reset(0)
        eng.prefill(0, ids[:prompt])
    ms = _timed(one_prompt, 3, 4)
    out[f"prefill_{prompt}"] = {"ms": ms, "tokens_per_s": prompt * 1e3 / ms}
    K.check_status()
    out["config"] = {"layers": cfg.n_layers, "hidden": cfg.hidden, "depth": depth, "params_b": cfg.param_count() / 1e9,
                     "l2": "weights larger than L2", "weights": "bf16" if cfg.layer_specs else "W4A16"}
    eng.close()
    return out


def run(release=lambda: None, family: str = "mumusun", which=None) -> dict:
    out = {}
    for cfg, other in SIZES[family]():
        if which and cfg.name != which:
            continue
        for c in (cfg, other):
            out[c.name] = bench_model(c)
            release()
    return out
