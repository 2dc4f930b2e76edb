"""``trace_run``: replays a trace of token ids through the serving engine and writes logits (nothing is sampled).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

The entries of a step are one ``Engine.forward_batch``: portions of prompts beside single tokens, each continuing its
request.  ``want`` names places among an entry's tokens whose logits go to ``DIR/<step>.f32`` (fp32, [wanted, vocab]);
``end`` releases requests.  After every step "done <step>" is printed.  The page pool holds ``--max-tokens`` positions and
there are four sequence slots, so pages and slots are used again.  ``--dtype float32`` serves the model in 32-bit; exit
code 3 when its family has no 32-bit form.
"""
from __future__ import annotations

import json
import os
import sys
from dataclasses import dataclass
from typing import Dict, Optional

from .flags import flag, parse

SLOTS = 4


@dataclass
class TraceFlags:
    model: Optional[str] = flag(None, "folder with config.json and model.safetensors")
    dtype: str = flag("bfloat16", "element type of weights, cache and activations", ["bfloat16", "float32"])
    out: Optional[str] = flag(None, "folder the logits are written to")
    max_tokens: int = flag(4096, "most tokens live requests hold at any time")


class Replay:
    """Requests by name on an engine's slots."""

    def __init__(self, engine):
        self.e = engine
        self.slot: Dict[str, int] = {}
        self.free = list(range(engine.max_seqs))

    def step(self, entries):
        batch = []
        for en in entries:
            rid = en["id"]
            if rid not in self.slot:
                if not self.free:
                    raise RuntimeError(f"request {rid!r}: all {self.e.max_seqs} sequence slots are taken")
                self.slot[rid] = self.free.pop(0)
                self.e.reset(self.slot[rid])
            batch.append((self.slot[rid], en["tokens"], en.get("want", [])))
        return self.e.forward_batch(batch)

    def end(self, rid):
        slot = self.slot.pop(rid)
        self.e.reset(slot)
        self.free.append(slot)


def main(argv=None) -> int:
    f = parse(TraceFlags, argv, "trace_run", __doc__)
    if not f.model or not f.out:
        raise SystemExit("--model and --out are needed")
    from .common import hardware_gate, peek_config
    cfg = peek_config(f.model)
    if f.dtype == "float32" and not cfg.layer_specs:
        sys.stderr.write(f"{cfg.name}: this family is served in bfloat16 only\n")
        return 3
    import torch
    from ..loader.loader import load
    from ..runtime.engine import PAGE, Engine
    hardware_gate(1)
    torch.cuda.set_device(0)
    weights = load(f.model, device="cuda", dtype=f.dtype)
    tokens = -(-f.max_tokens // PAGE) * PAGE
    engine = Engine(weights, max_seqs=SLOTS, max_len=tokens, num_pages=tokens // PAGE + 1)
    replay = Replay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = replay.step(st["entries"])
        if any(en.get("want") for en in st["entries"]):
            logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(f.out, f"{st['step']}.f32"))
        for rid in st.get("end", []):
            replay.end(rid)
        sys.stdout.write(f"done {st['step']}\n")
        sys.stdout.flush()
    return 0
