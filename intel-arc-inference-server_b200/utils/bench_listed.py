"""Throughput of models that list their layers, beside the framework's closest other model at equal size.

Decode: captured steps of 1, 8, 16 and 64 requests at one depth (one row each, positions advance on the device).  Prompt:
whole prompt passes through ``Engine.prefill``.  Both are timed with CUDA events after warm-up; the weights a step reads
are far more than the L2 holds.  The comparison model has the same width, layers, experts, experts per token, query heads
and window, grouped-query attention instead of latents, and the framework's W4A16 weights.
"""
from __future__ import annotations

import dataclasses

import torch

from ..models.config import ModelConfig, listed_config, preset
from ..models.weights import random_weights
from ..ops import lib as K
from ..runtime.engine import Engine


def sizes():
    """(listed model, closest model) pairs."""
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
    for m in rows:
        for s in range(m):
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


def run(release=lambda: None, which=None) -> dict:
    out = {}
    for cfg, other in sizes():
        if which and cfg.name != which:
            continue
        for c in (cfg, other):
            out[c.name] = bench_model(c)
            release()
    return out
