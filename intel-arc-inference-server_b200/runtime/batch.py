"""Mixed batches: prompt portions of some requests beside decode rows of others, as one walk over the layers.

The decode step's control block holds 64 rows.  A batch here has a row table of its own (slot, position, token per row),
uploaded with one copy together with everything else the kernels need: the wanted rows, and for every form of prompt
segments the model's mixers use (``Mixer.forms``) a table of its own.  Entries of fewer than ``SEGMENT`` tokens are handled
row by row, longer ones as prompt segments; both kinds share every linear and every expert of the step.  The walk itself is
``DecoderModel.listed_walk``, as in decode steps.

Forms: ``("keys", window, rows per tile)`` lists the cache rows the segments see, to be expanded, and query tiles over them;
``("tiles", chunk, rows per tile)`` query tiles over the pages; ``("pooled", window, pool, rows per tile)`` query tiles and the pooled
blocks that rows of a segment see before their window; ``("chunks",)`` the segments of a recurrence, in chunks of 64 rows or
``("chunks", rows)``.

Takes the place of the reference's chunk walk (src/runtime/prefill/step.cc:102-319) for models that list their layers.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import numpy as np
import torch

from ..models.listed import BatchPlan, ListedScratch, StepRows
from ..ops import lib as K

SEGMENT = 32        # tokens from which an entry is handled as a prompt segment
CHUNK = 64          # rows of a recurrence's chunk
ALIGN = 4           # int32 words: table parts start on 16-byte boundaries


@dataclass
class KeyPlan:
    """Cache rows whose keys and values the segments see, and the query tiles over them."""
    n_keys: int
    kreq: torch.Tensor
    kpos: torch.Tensor
    n_tiles: int
    tiles: torch.Tensor


@dataclass
class TilePlan:
    """Query tiles over the pages."""
    n_tiles: int
    tiles: torch.Tensor


@dataclass
class PoolPlan:
    """Query tiles over a window of the pages and the pooled blocks before it: slots and blocks of the segments' pooled rows, one
    segment after another, and the first row of every tile's segment."""
    n_tiles: int
    tiles: torch.Tensor
    n_pool: int
    preq: torch.Tensor
    block: torch.Tensor
    first: torch.Tensor


@dataclass
class ChunkPlan:
    """Segments of a recurrence: [n][4] (first row, rows, slot, first chunk); chunks in total and in the longest one."""
    n_segs: int
    segs: torch.Tensor
    chunks: int
    most: int


def segment_tiles(segments: Sequence[Tuple[int, int, int]], chunk: int, per: int):
    """Query tiles of prompt segments (slot, first position, rows) as (first query row, rows, position of that row, slot):
    at most ``per`` rows, and none across a border of chunks that hold more rows than a tile."""
    tiles, qrow = [], 0
    for slot, p, n in segments:
        r = 0
        while r < n:
            c = min(per, n - r)
            if chunk > per:
                c = min(c, chunk - (p + r) % chunk)
            tiles.append((qrow + r, c, p + r, slot))
            r += c
        qrow += n
    keys = lambda t: t[2] % chunk + t[1] if chunk else t[2] + t[1]     # noqa: E731
    tiles.sort(key=lambda t: -keys(t))                     # tiles with many keys first
    return tiles


def segment_chunks(segments: Sequence[Tuple[int, int, int]], per: int = CHUNK):
    """Prompt segments of a recurrence as (first row, rows, slot, first chunk), and the number of chunks."""
    out, row, chunks = [], 0, 0
    for slot, _, n in segments:
        out.append((row, n, slot, chunks))
        row += n
        chunks += (n + per - 1) // per
    return out, chunks


def segment_blocks(segments: Sequence[Tuple[int, int, int]], window: int, pool: int, per: int):
    """Query tiles as in ``segment_tiles``, every tile's first pooled row, and the slots and numbers of the blocks that the segments'
    last rows see, one segment after another."""
    preq, block, tiles = [], [], []
    qrow = rows = 0
    for slot, p, n in segments:
        blocks = max(0, p + n - window) // pool if pool else 0
        preq.append(np.full(blocks, slot))
        block.append(np.arange(blocks))
        tiles += [(qrow + r, min(per, n - r), p + r, slot, rows) for r in range(0, n, per)]
        qrow += n
        rows += blocks
    cost = lambda t: min(t[2], window) + t[1] + (max(0, t[2] + t[1] - window) // pool if pool else 0)      # noqa: E731
    tiles.sort(key=lambda t: -cost(t))                     # tiles with many keys first
    return [t[:4] for t in tiles], [t[4] for t in tiles], np.concatenate(preq), np.concatenate(block)


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
        self.forms = ll.forms()

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
        segs, tables = [(s, p, len(t)) for s, p, t in segments], {}
        for form in self.forms if segments else ():
            if form[0] == "keys":
                kreq, kpos, tiles = segment_keys(segs, form[1], form[2])
                k, t = (add(kreq), add(kpos)), add(tiles)
                tables[form] = lambda cut, n=len(kreq), k=k, nt=len(tiles), t=t: KeyPlan(n, cut(k[0]), cut(k[1]), nt, cut(t))
            elif form[0] == "tiles":
                tiles = segment_tiles(segs, form[1], form[2])
                tables[form] = lambda cut, nt=len(tiles), t=add(tiles): TilePlan(nt, cut(t))
            elif form[0] == "pooled":
                tiles, first, preq, block = segment_blocks(segs, *form[1:])
                where = add(tiles), add(preq), add(block), add(first)
                tables[form] = lambda cut, nt=len(tiles), n=len(block), w=where: PoolPlan(nt, cut(w[0]), n, cut(w[1]), cut(w[2]), cut(w[3]))
            else:
                per = form[1] if len(form) > 1 else CHUNK
                rows, chunks = segment_chunks(segs, per)
                most = max((n + per - 1) // per for _, _, n in segs)
                tables[form] = lambda cut, n=len(rows), t=add(rows), c=chunks, most=most: ChunkPlan(n, cut(t), c, most)
        return np.concatenate(parts), spans, tables

    def _walk(self, entries: Sequence[Tuple[int, List[int]]], want: Sequence[Tuple[int, int]]):
        """One batch: ``entries`` (slot, tokens) through all layers, K / V appended.  ``want``: (entry, place) pairs.
        Returns (the walk's rows, device indices of the wanted ones)."""
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
        host, spans, tables = self._tables(singles, segments, np.asarray([start[i] + j for i, j in want], dtype=np.int32))
        dev = torch.from_numpy(host).pin_memory().to(eng.device, non_blocking=True)
        cut = lambda span: dev[span[0]: span[0] + span[1]]                              # noqa: E731
        rows = StepRows(cut(spans["req"]), cut(spans["pos"]), cut(spans["token"]))
        plan = BatchPlan(sum(len(t) for _, _, t in singles), {f: make(cut) for f, make in tables.items()})
        resid = self.scratch.get("resid", n, m.listed.wp, torch.float32) if m.streams is None else None
        final = m.listed_walk(n, rows, eng.block_table, eng.kv, self.scratch, resid, plan)
        for s, t in entries:
            eng.seq_len[s] += len(t)
        return final, cut(spans["want"])

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
            final, sel = self._walk([(entries[i][0], entries[i][1][lo: lo + k]) for i, lo, k in now], want)
            self._logits(final, sel, dst, out)
            for i, lo, k in now:
                cut[i] = lo + k
        return out[:total]

    def _logits(self, final, sel, dst, out):
        m = self.eng.model
        step = m.buf.max_rows
        for c0 in range(0, len(dst), step):
            d = dst[c0: c0 + step]
            n = len(d)
            straight = d == [[d[0][0] + i] for i in range(n)]
            lg = out[d[0][0]: d[0][0] + n] if straight else self.scratch.get("logits_part", n, self.eng.cfg.vocab, torch.float32)
            m.listed_logits(final, sel[c0: c0 + n], n, self.scratch, lg)
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
            final, sel = self._walk([(slot, part)], [(0, len(part) - 1)] if last else [])
        m.listed_logits(final, sel, 1, self.scratch, m.buf.logits)
        K.argmax_finish(m.buf.cand_val, m.buf.cand_idx, m.buf.ncand, 1, eng.ctrl, False)
        return eng._read_out(1)[0]
