"""Single-GPU engine: sequence slots, paged KV, control block, CUDA-graph replay.

The role of the reference's ``runtime::Engine`` (src/runtime/engine.h:52-690):
ingest a prompt, replay decode steps, verify draft rows, keep per-sequence
state in slots.  Here a "captured command list" is a ``torch.cuda.CUDAGraph``
per (row count, advance) pair; the device control block carries positions and
tokens from one replay to the next, so plain decode needs no host write between
steps.  Host-side bookkeeping (sequence lengths, page tables) is deterministic
from the number of steps, so the host never reads the device to know where a
sequence is.
"""
from __future__ import annotations

import gc
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from ..models.config import ModelConfig
from ..models.decoder import DecoderModel, KVCache, attn_splits
from ..models.weights import ModelWeights
from ..ops import lib as K
from ..utils.staging import Staged
from .kv_pool import KvPool

PAGE = 16


@dataclass
class Row:
    slot: int
    pos: int
    token: int
    block: int = 0      # 1: a block drafter's row, which attends to all positions of its request's rows in the step


def _starts(entries) -> List[int]:
    """Index of every entry's first token in the flattened step."""
    out, n = [], 0
    for _, toks, _ in entries:
        out.append(n)
        n += len(toks)
    return out


class Engine:
    def __init__(self, weights: ModelWeights, max_seqs: int = 1, max_len: int = 4096, kv_dtype: str = "bf16",
                 max_rows: int = 64, use_graphs: bool = True, int8_head: bool = False, num_pages: Optional[int] = None,
                 nsplit_attn: int = 0, prefill_backend: str = "auto", tp=None, nccl=None,
                 extra_kv_layers: int = 0):
        """``tp``: wires of a tensor-parallel group; every rank builds the same Engine over its weight shard and
        is driven with the same calls (same rows, same order) -- the step's kernels do the crossings."""
        self.cfg = cfg = weights.cfg
        self.tp = tp if tp is not None and tp.world > 1 else None
        self.device = weights.embed.device
        self.max_seqs, self.max_len, self.max_rows = max_seqs, max_len, max_rows
        if cfg.layer_specs and weights.embed.dtype == torch.float32:
            kv_dtype = "f32"        # a model served in 32-bit keeps its cache in 32-bit
        self.max_blocks = (max_len + PAGE - 1) // PAGE
        if num_pages is None:
            num_pages = max_seqs * self.max_blocks + 1
        if not nsplit_attn:     # sized for contexts near the longest one the engine holds
            nsplit_attn = attn_splits(cfg.n_kv_heads, max_len)
        self.model = DecoderModel(weights, max_rows=max_rows, max_pos=max_len, nsplit_attn=nsplit_attn,
                                  int8_head=int8_head, tp=self.tp, nccl=nccl)
        self.kv = KVCache(cfg, cfg.n_layers + extra_kv_layers, num_pages, self.device, kv_dtype,   # + draft-head layers
                          n_slots=max_seqs)
        self.kv_dtype = kv_dtype
        self.pool = KvPool(num_pages, max_seqs, self.max_blocks)
        self.ctrl = torch.zeros(K.CTRL_WORDS, dtype=torch.int32, device=self.device)
        # pinned staging rings: a queued non-blocking copy may run long after the host moved on (see utils/staging.py)
        self.ctrl_stage = Staged((K.CTRL_WORDS,), torch.int32)
        self.table_stage = Staged((self.max_blocks,), torch.int32, depth=4)
        self.out_host = torch.zeros(K.CTRL_WORDS, dtype=torch.int32).pin_memory()
        self.block_table = torch.zeros(max_seqs, self.max_blocks, dtype=torch.int32, device=self.device)
        self.seq_len = [0] * max_seqs
        self._snap = None           # (rows, {slot: recurrent state before them}) of the last step of a recurrent model
        self.use_graphs = use_graphs
        self.graphs: Dict[Tuple[int, bool, bool], torch.cuda.CUDAGraph] = {}
        self._one_request = False   # the rows last written are consecutive positions of one request
        self.prefill_backend = prefill_backend
        self._prefill = None
        self.steps_replayed = 0
        self.last_prefill_row = 0
        # failure latch (the reference's TpEngine keeps `broken_` until reset(): src/runtime/tp_engine.cc:203-256,418-424)
        self.broken: Optional[str] = None
        if self.device.type == "cuda":
            K.arm_failure_word()
        import os
        if os.environ.get("B200SERVE_AUDIT", "0") == "1":     # every buffer has a planner entry (see buffer_registry.py)
            from .buffer_registry import audit
            audit(self.model.buf, self.kv, cfg, kv_dtype, max_seqs)
        self._batch = None          # runner of mixed batches (models that list their layers)
        self.launches_per_step: Dict[Tuple[int, bool, bool], int] = {}

    def close(self):
        """Releases the cross-GPU buffers of a tensor-parallel engine (mapped peer memory)."""
        torch.cuda.synchronize(self.device)
        self.graphs.clear()
        if self._prefill is not None and hasattr(self._prefill, "close"):
            self._prefill.close()
        self._prefill = None
        if self.tp is not None:
            self.tp.close()
            self.tp = self.model.tp = None

    # ------------------------------------------------------------------ slots and pages
    def reset(self, slot: Optional[int] = None):
        slots = range(self.max_seqs) if slot is None else [slot]
        for s in slots:
            self.pool.release(s)
            self.seq_len[s] = 0
            self.kv.reset_slot(s)       # recurrent state

    def truncate(self, slot: int, length: int):
        """Drop everything after ``length`` positions (rejected draft rows)."""
        assert length <= self.seq_len[slot]
        replay = rest = None
        if length == 0 < self.seq_len[slot]:
            self.kv.reset_slot(slot)
        elif length < self.seq_len[slot] and self.kv.states:
            # A recurrent state cannot be rewound.  The last multi-row step left a copy of the slot's state from
            # before its rows (the reference snapshots its GDN state the same way around verify rows): put it
            # back and run the rows that stay once more.
            snap = self._snap
            rows = [] if snap is None else [r for r in snap[0] if r.slot == slot]
            if not rows or slot not in snap[1] or length < rows[0].pos or self.seq_len[slot] != rows[-1].pos + 1:
                raise NotImplementedError("a recurrent state can only be rewound to a position inside the last multi-row "
                                          "step (prefix reuse is not available for recurrent families)")
            self.kv.load_states(slot, snap[1][slot])
            replay = [r for r in rows if r.pos < length]
            self.seq_len[slot] = rows[0].pos
            # one rewind per step and slot; the step's other slots can still be rewound
            rest = ([r for r in snap[0] if r.slot != slot], {s: v for s, v in snap[1].items() if s != slot})
        self.seq_len[slot] = min(self.seq_len[slot], length)
        self.pool.truncate(slot, (length + PAGE - 1) // PAGE)
        if replay:
            self.forward_rows(replay, advance=False, read=False)
        if rest is not None:
            self._snap = rest

    def _ensure_pages(self, slot: int, upto_len: int):
        if upto_len > self.max_len:
            raise ValueError(f"sequence of {upto_len} positions exceeds max_len {self.max_len}")
        want = (upto_len + PAGE - 1) // PAGE
        try:
            changed = self.pool.ensure(slot, want)
        except MemoryError:
            # the pool is short of pages: whoever keeps finished sessions and cached blocks on the device (the prefix
            # store) gives some back -- cached blocks go to the host tier, idle sessions leave, least recently used
            # first -- and the request goes on; only when that does not cover it does the request fail
            hook = getattr(self, "on_pool_pressure", None)
            need = want - len(self.pool.table(slot))
            if hook is None or not hook(slot, need):
                raise
            changed = self.pool.ensure(slot, want)
        if changed:
            row = self.pool.table(slot)
            host = self.table_stage.begin()
            host[: len(row)] = torch.from_numpy(np.asarray(row, dtype=np.int32))
            self.table_stage.push(self.block_table[slot, : len(row)], host[: len(row)])

    def _write_rows(self, rows: Sequence[Row]):
        m = len(rows)
        c = self.ctrl_stage.begin()
        c[K.CTRL_N_ROWS] = m
        for i, r in enumerate(rows):
            c[K.CTRL_ROW_REQ + i] = r.slot
            c[K.CTRL_ROW_POS + i] = r.pos
            c[K.CTRL_CUR_TOKEN + i] = r.token
            c[K.CTRL_ROW_BLOCK + i] = r.block
        self._one_request = all(r.slot == rows[0].slot and r.pos == rows[0].pos + i for i, r in enumerate(rows))
        self.ctrl_stage.push(self.ctrl)

    # ------------------------------------------------------------------ session snapshots
    def save_kv(self, slot: int, begin: int, end: int) -> dict:
        """The KV of positions ``[begin, end)`` of ``slot`` (whole pages: both multiples of 16, or ``end`` the
        sequence length) as pinned host tensors in page order -- the reference's ``save_kv`` (src/runtime/engine.h:170-209);
        the layout is ``[layer][page][kv head][16][head dim]`` per tensor and does not depend on the parallel mode."""
        if begin % PAGE or (end % PAGE and end != self.seq_len[slot]) or not 0 <= begin <= end <= self.seq_len[slot]:
            raise ValueError("save_kv takes whole pages inside the sequence")
        if self.kv.states and end != self.seq_len[slot]:
            raise ValueError("save_kv: a recurrent model's snapshot ends at the sequence end (its state is the one after the "
                             "last position)")
        pages = list(self.pool.table(slot))[begin // PAGE: (end + PAGE - 1) // PAGE]
        idx = torch.as_tensor(pages, device=self.device, dtype=torch.int64)
        tensors = self.kv.page_tensors()
        out = {"begin": begin, "end": end, "kv_dtype": self.kv_dtype}
        for name, t in self.kv.states.items():      # the recurrent state after position end - 1
            host = torch.empty((t.shape[0],) + tuple(t.shape[2:]), dtype=t.dtype).pin_memory()
            host.copy_(t[:, slot], non_blocking=True)
            out[name] = host
        for name, t in tensors.items():
            host = torch.empty((t.shape[0], len(pages)) + tuple(t.shape[2:]), dtype=t.dtype).pin_memory()
            host.copy_(t.index_select(1, idx), non_blocking=True)
            out[name] = host
        torch.cuda.current_stream().synchronize()
        return out

    def load_kv(self, slot: int, blob: dict):
        """Puts a ``save_kv`` blob back at its positions; the slot must hold exactly ``blob["begin"]`` positions."""
        begin, end = blob["begin"], blob["end"]
        if blob["kv_dtype"] != self.kv_dtype or self.seq_len[slot] != begin:
            raise ValueError("load_kv: the slot must end where the blob begins and use the same KV form")
        self._ensure_pages(slot, end)
        pages = list(self.pool.table(slot))[begin // PAGE: (end + PAGE - 1) // PAGE]
        idx = torch.as_tensor(pages, device=self.device, dtype=torch.int64)
        tensors = self.kv.page_tensors()
        for name, t in tensors.items():
            t.index_copy_(1, idx, blob[name].to(self.device, non_blocking=True))
        if self.kv.states:
            if any(name not in blob for name in self.kv.states):
                raise ValueError("load_kv: the blob holds no recurrent state for this model")
            self.kv.load_states(slot, blob)
            self._snap = None
        self.seq_len[slot] = end

    # ------------------------------------------------------------------ running a step
    def _enqueue(self, m: int, advance: bool):
        self.model.step_rows(m, self.ctrl, self.block_table, self.max_blocks, self.kv, advance,
                             one_request=self._one_request)

    def _run(self, m: int, advance: bool):
        if not self.use_graphs:
            self._enqueue(m, advance)
            return
        key = (m, advance, self._one_request)
        g = self.graphs.get(key)
        if g is None:
            # warm-up outside capture (sets function attributes, allocates split-K scratch), then
            # restore the control block the warm-up advanced
            saved = self.ctrl.clone()
            # KV appends repeat harmlessly; a recurrent update does not: the state is put back
            saved_states = {n: t.clone() for n, t in self.kv.states.items()}
            n0 = K.launch_count
            self._enqueue(m, advance)
            self.launches_per_step[key] = K.launch_count - n0
            torch.cuda.current_stream().synchronize()
            self.ctrl.copy_(saved)
            for n, t in saved_states.items():
                self.kv.states[n].copy_(t)
            g = torch.cuda.CUDAGraph()
            # no garbage collection while the stream captures: a dead engine's graphs and buffers released in the middle
            # of it abort the process
            collects = gc.isenabled()
            gc.disable()
            try:
                with torch.cuda.graph(g):
                    self._enqueue(m, advance)
            finally:
                if collects:
                    gc.enable()
            self.ctrl.copy_(saved)
            self.graphs[key] = g
        g.replay()
        self.steps_replayed += 1

    def launches(self, m: int, advance: bool = True) -> int:
        """Kernel launches of one captured step of ``m`` rows (0 before the first such step)."""
        return max((v for (mm, adv, _), v in self.launches_per_step.items() if mm == m and adv == advance), default=0)

    # ------------------------------------------------------------------ failure latch
    def require_ok(self):
        if self.broken is not None:
            raise K.KernelError(f"engine is latched after a failed step ({self.broken}); call reset_failure()")

    def check_failed(self, what: str = "step"):
        """After a synchronize: if any kernel's bounded wait ran out during the work just finished, latch the engine and
        raise an error that names the unit, the code and where it gave up (rank, tile).  The step's outputs are garbage."""
        if not K.failed_fast():
            return
        st = K.status()
        rank = self.tp.rank if self.tp is not None else (self.model.nccl[0] if self.model.nccl is not None else 0)
        self.broken = f"{what} on rank {rank}: " + ", ".join(
            f"{u}: code {v['code']} detail {v['detail']:#x} ({v['count']} waits)" for u, v in st.items())
        raise K.KernelError(f"device kernels gave up on a bounded wait during {self.broken}")

    def reset_failure(self):
        """Clears the status words, the whole-step kernel's barrier words and the wires' flags and call counters, and
        releases the latch.  Under tensor parallelism every rank must call it before the next step."""
        torch.cuda.synchronize(self.device)
        K.status_clear()
        self.model.mega_reset()
        if self.tp is not None:
            self.tp.reset()
        torch.cuda.synchronize(self.device)
        self.broken = None

    def _read_out(self, m: int) -> List[int]:
        self.out_host.copy_(self.ctrl, non_blocking=True)
        torch.cuda.current_stream().synchronize()
        self.check_failed()
        return self.out_host[K.CTRL_OUT_TOKEN: K.CTRL_OUT_TOKEN + m].tolist()

    # ------------------------------------------------------------------ public API
    def forward_rows(self, rows: Sequence[Row], advance: bool = False, read: bool = True):
        """Run arbitrary rows (verify, batched decode, chunked ingest). KV of each row is appended."""
        self.require_ok()
        for r in rows:
            self._ensure_pages(r.slot, r.pos + 1)
        self._snapshot(rows)
        self._write_rows(rows)
        self._run(len(rows), advance)
        for r in rows:
            self.seq_len[r.slot] = max(self.seq_len[r.slot], r.pos + 1)
        return self._read_out(len(rows)) if read else None

    def _snapshot(self, rows: Sequence[Row]):
        """Keeps the recurrent state from before a step's rows, so that its last rows can be taken back (``truncate``)."""
        self._snap = None
        if self.kv.states and rows:
            runs = [r.slot for i, r in enumerate(rows) if i == 0 or r.slot != rows[i - 1].slot]
            if len(set(runs)) != len(runs):
                raise ValueError("a recurrent model's step holds a sequence's rows one after another")
            several = {r.slot for i, r in enumerate(rows) if i and r.slot == rows[i - 1].slot}
            if several:       # a lone row of a sequence is its next token, never a draft
                self._snap = ([r for r in rows if r.slot in several], {s: self.kv.save_states(s) for s in sorted(several)})

    def logits(self, m: int) -> torch.Tensor:
        """fp32 logits of the last step's rows (device tensor view)."""
        return self.model.buf.logits[:m]

    @property
    def mixed_batches(self) -> bool:
        """Prompt portions and decode rows of several requests run as one batch of any size (``forward_batch``)."""
        return bool(self.cfg.layer_specs)

    def forward_batch(self, entries: Sequence[Tuple[int, Sequence[int], Sequence[int]]]) -> torch.Tensor:
        """One step over ``entries`` (slot, next tokens, wanted places among them): prompt portions beside decode rows of
        other requests, each continuing its slot.  Returns the fp32 logits of the wanted places [n][vocab], in order
        (a device tensor, valid until the next step)."""
        self.require_ok()
        entries = [(s, list(t), list(w)) for s, t, w in entries if len(t)]
        n = sum(len(t) for _, t, _ in entries)
        if n == 0:
            return self.logits(0)
        if n > self.max_rows and self.mixed_batches:
            # rows of entries short enough to be a decode step's can be taken back afterwards, as in ``forward_rows``
            self._snapshot([Row(s, self.seq_len[s] + i, t) for s, toks, _ in entries if 1 < len(toks) <= 16
                            for i, t in enumerate(toks)])
            out = self._batch_runner().run(entries)
            self.check_failed_sync("batch")
            return out
        got = []
        todo = [Row(s, self.seq_len[s] + i, t) for s, toks, _ in entries for i, t in enumerate(toks)]
        want = [j + w for j, (_, toks, ws) in zip(_starts(entries), entries) for w in ws]
        for c0 in range(0, n, self.max_rows):      # models without mixed batches: row steps
            part = todo[c0: c0 + self.max_rows]
            self.forward_rows(part, advance=False, read=False)
            sel = [w - c0 for w in want if c0 <= w < c0 + len(part)]
            if sel:
                got.append(self.logits(len(part))[sel] if n > self.max_rows or sel != list(range(len(part)))
                           else self.logits(len(part)))
        self.check_failed_sync("batch")
        return torch.cat(got) if len(got) > 1 else (got[0] if got else self.logits(0))

    def argmax(self, logits: torch.Tensor) -> List[int]:
        """Arg-max of fp32 logit rows (ties to the lower id)."""
        from ..ops import latent as L
        m, n = logits.shape
        val = torch.empty(m, dtype=torch.float32, device=logits.device)
        idx = torch.empty(m, dtype=torch.int32, device=logits.device)
        L.row_argmax(logits, m, n, val, idx)
        return idx.tolist()

    def check_failed_sync(self, what: str):
        torch.cuda.current_stream().synchronize()
        self.check_failed(what)

    def _batch_runner(self):
        if self._batch is None:
            from .batch import BatchRunner
            self._batch = BatchRunner(self)
        return self._batch

    def prefill(self, slot: int, ids: Sequence[int], chunk: Optional[int] = None) -> int:
        """Ingest ``ids`` after the slot's current length; returns the greedy next token."""
        self.require_ok()
        ids = list(ids)
        if self.mixed_batches and len(ids) > self.max_rows:
            self.last_prefill_row = 0
            self._snap = None
            return self._batch_runner().prefill(slot, ids, chunk)
        if self._use_tc_prefill(len(ids)):
            if self._prefill is None:
                if self.tp is not None:
                    from ..parallel.tp_prefill import TpPrefillRunner
                    self._prefill = TpPrefillRunner(self)
                elif self.model.nccl is not None:
                    from ..parallel.tp_prefill import NcclPrefillRunner
                    self._prefill = NcclPrefillRunner(self, self.model.nccl[2])
                else:
                    from .prefill import PrefillRunner
                    self._prefill = PrefillRunner(self)
            self.last_prefill_row = 0      # row of model.buf.logits that holds the prompt's last position
            tok = self._prefill.run(slot, ids, chunk)
            self.check_failed("prompt pass")
            return tok
        start = self.seq_len[slot]
        out = None
        for c0 in range(0, len(ids), self.max_rows):
            part = ids[c0: c0 + self.max_rows]
            rows = [Row(slot, start + c0 + i, t) for i, t in enumerate(part)]
            last = c0 + self.max_rows >= len(ids)
            out = self.forward_rows(rows, advance=False, read=last)
            hook = getattr(self, "on_chunk_hidden", None)
            if hook is not None:
                hook(None, slot, part, start + c0, self.model.buf.resid[: len(part)])
        self.last_prefill_row = len(out) - 1
        return out[-1]

    def _use_tc_prefill(self, n: int) -> bool:
        """Prompt chunks longer than the row kernels take go through the tcgen05 path when the shape
        has one (head size 128, bf16 KV, dense FFN or MoE with a grouped path)."""
        if self.prefill_backend == "rows" or n <= self.max_rows or self.mixed_batches:
            return False
        if self.cfg.n_gdn_layers and (self.kv.kv_int8 or self.tp is not None or self.model.nccl is not None):
            return False        # hybrid models: the layer-major int8-KV pass and the parallel runners know no GDN layers
        # an int8 KV cache: the one-GPU runner's layer-major pass, or the tensor-parallel runner's bf16 scratch of
        # the request; the NCCL comparison build has neither
        ok = self.cfg.head_dim == 128 and (not self.kv.kv_int8 or self.model.nccl is None)
        if not ok and self.prefill_backend != "auto":
            raise ValueError(f"prefill backend {self.prefill_backend!r} needs head_dim 128 (and a bf16 KV cache under "
                             "tensor parallelism)")
        return ok

    def decode_begin(self, slots: Sequence[int], tokens: Sequence[int]):
        """Arm plain decode: one row per slot, starting with ``tokens`` at each slot's current length."""
        rows = [Row(s, self.seq_len[s], t) for s, t in zip(slots, tokens)]
        self._write_rows(rows)
        self._decode_slots = list(slots)

    def decode_step(self, read: bool = True):
        """One replay of the armed decode rows; the device advances tokens and positions itself."""
        self.require_ok()
        slots = self._decode_slots
        for s in slots:
            self._ensure_pages(s, self.seq_len[s] + 1)
        self._run(len(slots), True)
        for s in slots:
            self.seq_len[s] += 1
        return self._read_out(len(slots)) if read else None

    def generate(self, ids: Sequence[int], n_new: int, slot: int = 0) -> List[int]:
        """Greedy: prefill ``ids`` then ``n_new`` tokens; returns the new tokens."""
        self.reset(slot)
        first = self.prefill(slot, ids)
        out = [first]
        if n_new > 1:
            self.decode_begin([slot], [first])
            for _ in range(n_new - 1):
                out.append(self.decode_step()[0])
        return out
