"""Mixed batches: prompt portions of some requests beside decode rows of others, as one walk over the layers.

The decode step's control block holds 64 rows.  A batch here has a row table of its own (slot, position, token per row),
uploaded with one copy together with everything else the kernels need: the wanted rows, and for every window of the
model the cache rows the prompt segments see and their query tiles.  Entries of fewer than ``SEGMENT`` tokens are attended
row by row over the latent, longer ones as prompt segments over expanded keys and values; both kinds share every linear
and every expert of the step.  The walk itself is ``DecoderModel.listed_walk``, as in decode steps.

Takes the place of the reference's chunk walk (src/runtime/prefill/step.cc:102-319) for models that list their layers.
"""
from __future__ import annotations

from typing import List, Optional, Sequence, Tuple

import numpy as np
import torch

from ..models.latent import BatchPlan, KeyPlan, ListedScratch, StepRows
from ..ops import lib as K

SEGMENT = 32        # tokens from which an entry is attended as a prompt segment
ALIGN = 4           # int32 words: table parts start on 16-byte boundaries


def segment_keys(segments: Sequence[Tuple[int, int, int]], window: int, per: int):
    """Key rows and query tiles of prompt segments (slot, first position, rows): the slots and positions of every key some
    row of its segment sees, segment after segment, and tiles of at most ``per`` query rows as (first query row, rows,
    position of that row and key row of position 0, both counted from the segment's first key)."""
    kreq, kpos, tiles = [], [], []
    krow = qrow = 0
    for slot, p, n in segments:
        lo = max(0, p - window + 1) if window else 0       # first position any of the segment's rows sees
        kreq.append(np.full(p + n - lo, slot))
        kpos.append(np.arange(lo, p + n))
        tiles += [(qrow + r, min(per, n - r), p + r - lo, krow) for r in range(0, n, per)]
        krow += p + n - lo
        qrow += n
    tiles.sort(key=lambda t: -(t[2] + t[1]))               # tiles with many keys first
    return np.concatenate(kreq), np.concatenate(kpos), tiles


class BatchRunner:
    def __init__(self, engine, max_tokens: int = 4096):
        self.eng, self.max_tokens = engine, max_tokens
        ll = engine.model.listed
        self.scratch = ListedScratch(engine.device, ll.dtype)
        # forms of the expanded attention the model's layers use: (window, query rows per tile)
        self.forms = sorted({(s.mixer.window, ll.tile_rows(g)) for s, g in zip(engine.cfg.layer_specs, ll.geo) if ll.tile_rows(g)})

    # ------------------------------------------------------------------ tables
    def _tables(self, singles, segments, want: np.ndarray):
        """Host tables of a batch as one int32 array, and where their parts are.  ``singles`` / ``segments``: (slot,
        first position, tokens); rows are numbered singles first."""
        parts: List[np.ndarray] = []

        def add(a) -> Tuple[int, int]:
            off = sum(len(x) for x in parts)
            a = np.asarray(a, dtype=np.int32).ravel()
            pad = -len(a) % ALIGN
            parts.append(np.concatenate([a, np.zeros(pad, np.int32)]) if pad else a)
            return off, len(a)

        both = singles + segments
        spans = {"req": add(np.concatenate([np.full(len(t), s) for s, _, t in both])),
                 "pos": add(np.concatenate([np.arange(p, p + len(t)) for _, p, t in both])),
                 "token": add(np.concatenate([np.asarray(t) for _, _, t in both])), "want": add(want)}
        keys = {}
        for window, per in self.forms if segments else ():
            kreq, kpos, tiles = segment_keys([(s, p, len(t)) for s, p, t in segments], window, per)
            keys[(window, per)] = (len(kreq), add(kreq), add(kpos), len(tiles), add(tiles))
        return np.concatenate(parts), spans, keys

    def _walk(self, entries: Sequence[Tuple[int, List[int]]], want: Sequence[Tuple[int, int]]):
        """One batch: ``entries`` (slot, tokens) through all layers, K / V appended.  ``want``: (entry, place) pairs.
        Returns (residual rows, device indices of the wanted ones)."""
        eng, m = self.eng, self.eng.model
        slots = [s for s, _ in entries]
        if len(set(slots)) != len(slots):
            raise ValueError("a batch holds at most one entry per sequence")
        for s, t in entries:
            eng._ensure_pages(s, eng.seq_len[s] + len(t))
        seg = [bool(self.forms) and len(t) >= SEGMENT for _, t in entries]
        order = [i for i in range(len(entries)) if not seg[i]] + [i for i in range(len(entries)) if seg[i]]
        start, n = {}, 0
        for i in order:
            start[i] = n
            n += len(entries[i][1])
        item = lambda i: (entries[i][0], eng.seq_len[entries[i][0]], entries[i][1])   # noqa: E731
        singles, segments = [item(i) for i in order if not seg[i]], [item(i) for i in order if seg[i]]
        host, spans, keys = self._tables(singles, segments, np.asarray([start[i] + j for i, j in want], dtype=np.int32))
        dev = torch.from_numpy(host).pin_memory().to(eng.device, non_blocking=True)
        cut = lambda span: dev[span[0]: span[0] + span[1]]                              # noqa: E731
        rows = StepRows(cut(spans["req"]), cut(spans["pos"]), cut(spans["token"]))
        plan = BatchPlan(sum(len(t) for _, _, t in singles),
                         {f: KeyPlan(nk, cut(a), cut(b), nt, cut(c)) for f, (nk, a, b, nt, c) in keys.items()})
        resid = self.scratch.get("resid", n, m.listed.wp, torch.float32)
        m.listed_walk(n, rows, eng.block_table, eng.kv, self.scratch, resid, plan)
        for s, t in entries:
            eng.seq_len[s] += len(t)
        return resid, cut(spans["want"])

    # ------------------------------------------------------------------ whole steps
    def run(self, entries: Sequence[Tuple[int, List[int], List[int]]]) -> torch.Tensor:
        """``Engine.forward_batch`` for any number of tokens; more than ``max_tokens`` run as several batches."""
        eng = self.eng
        total = sum(len(w) for _, _, w in entries)
        out = self.scratch.get("logits", max(total, 1), eng.cfg.vocab, torch.float32)
        where, n = {}, 0            # (entry, place) -> rows of out
        for i, (_, _, ws) in enumerate(entries):
            for w in ws:
                where.setdefault((i, w), []).append(n)
                n += 1
        cut = [0] * len(entries)
        while any(cut[i] < len(t) for i, (_, t, _) in enumerate(entries)):
            room, now = self.max_tokens, []
            for i, (s, t, _) in enumerate(entries):
                k = min(room, len(t) - cut[i])
                if k > 0:
                    now.append((i, cut[i], k))
                    room -= k
            want = [(j, w - lo) for j, (i, lo, k) in enumerate(now) for w in sorted(set(entries[i][2])) if lo <= w < lo + k]
            dst = [where[(now[j][0], w + now[j][1])] for j, w in want]
            resid, sel = self._walk([(entries[i][0], entries[i][1][lo: lo + k]) for i, lo, k in now], want)
            self._logits(resid, sel, dst, out)
            for i, lo, k in now:
                cut[i] = lo + k
        return out[:total]

    def _logits(self, resid, sel, dst, out):
        m = self.eng.model
        step = m.buf.max_rows
        for c0 in range(0, len(dst), step):
            d = dst[c0: c0 + step]
            n = len(d)
            straight = d == [[d[0][0] + i] for i in range(n)]
            lg = out[d[0][0]: d[0][0] + n] if straight else self.scratch.get("logits_part", n, self.eng.cfg.vocab, torch.float32)
            m.listed_logits(resid, sel[c0: c0 + n], n, self.scratch, lg)
            if not straight:
                for i, rows in enumerate(d):
                    for r in rows:
                        out[r].copy_(lg[i])

    def prefill(self, slot: int, ids: List[int], chunk: Optional[int] = None) -> int:
        """``Engine.prefill``: portions of at most ``chunk`` tokens; the last row's logits go to ``buf.logits[0]``."""
        eng, m = self.eng, self.eng.model
        chunk = min(chunk or self.max_tokens, self.max_tokens)
        for c0 in range(0, len(ids), chunk):
            part = ids[c0: c0 + chunk]
            last = c0 + chunk >= len(ids)
            resid, sel = self._walk([(slot, part)], [(0, len(part) - 1)] if last else [])
        m.listed_logits(resid, sel, 1, self.scratch, m.buf.logits)
        K.argmax_finish(m.buf.cand_val, m.buf.cand_idx, m.buf.ncand, 1, eng.ctrl, False)
        return eng._read_out(1)[0]
