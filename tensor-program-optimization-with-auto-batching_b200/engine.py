"""What every served model shares: the staged rows of a pass, prompt passes, decode steps, and captured decode steps.

:class:`EngineBase` drives a model's ``forward`` -- the only part a model design writes itself -- over a paged cache:
``extend`` / ``prefill`` run portions of prompts of any length cut into passes of ``max_rows`` rows, ``decode`` one token
per sequence, ``capture_decode`` / :class:`DecodeSession` the same as a CUDA graph
(``tvm/llama_auto_batcher/llama_exec_graph.py:58-141``).
"""
from __future__ import annotations

import numpy as np
import torch

from . import ops
from .kv_cache import PagedCache


class EngineBase:
    """Row buffers of one pass and the loops around ``forward``.  A subclass provides

    ``forward(T, fused_append, use_lora, lm_rows, n_lm, hidden)`` over the first T staged rows (``tokens``, ``slots`` =
    adapter slots, ``row_slot`` = cache slots, ``row_pos``), returning (logits, next tokens);
    ``_begin_prompt_pass(chunk)`` / ``_end_prompt_pass()`` around the forward of a prompt pass, ``chunk`` a list of
    (sequence id, first row, rows, position of the first row);
    ``_check_prompt_status()`` after the last pass of a call."""

    def __init__(self, model, kv: PagedCache, max_rows: int):
        self.m, self.kv, self.max_rows = model, kv, int(max_rows)
        dev, T = model.device, self.max_rows
        i32 = dict(dtype=torch.int32, device=dev)
        self.logits = torch.zeros(T, model.V, dtype=torch.float32, device=dev)
        self.next_tok = torch.zeros(T, **i32)
        self.tokens = torch.zeros(T, **i32)
        self.slots = torch.full((T,), -1, **i32)
        self.row_slot = torch.zeros(T, **i32)
        self.row_pos = torch.zeros(T, **i32)
        self.last_rows = torch.zeros(T, **i32)
        self.iota = torch.arange(T, **i32)
        self.n_distinct = 0  # distinct adapters among the rows staged for the next pass (set with self.slots)
        self.max_keys = kv.max_pages * kv.page_size  # bound of the context of the rows staged for the next pass
        self.ws_linear = None

    def forward(self, T, fused_append, use_lora=True, lm_rows=None, n_lm=None, hidden=None):
        raise NotImplementedError

    def _begin_prompt_pass(self, chunk):
        pass

    def _end_prompt_pass(self):
        pass

    def _check_prompt_status(self):
        pass

    def status_word(self) -> int:
        """Status word of the projection kernels' scratch (synchronises): non-zero after a bounded wait expired
        somewhere since the buffer was last cleared; the outputs since then are undefined."""
        return ops.status_word(self.ws_linear)

    def check_status(self):
        """Raises if a projection kernel gave up a bounded wait, after re-zeroing the scratch (arrival counters of
        split tiles may be stale after such a failure) so that the engine stays usable."""
        st = self.status_word()
        if st:
            self.ws_linear.zero_()
            raise RuntimeError(f"mlora: a projection kernel gave up a bounded wait (status bits {st:#x}); "
                               "the results of this pass are undefined")

    def _stage(self, dst, values, dtype):
        t = torch.as_tensor(np.asarray(values), dtype=dtype)
        dst[: t.numel()].copy_(t.pin_memory(), non_blocking=True)

    def extend(self, seq_ids, portions, adapter_slots=None, want=None, use_lora=True):
        """Runs the next tokens (``portions``: lists of token ids) of already-added sequences from wherever each stands,
        cut into passes of at most ``max_rows`` rows.  ``want[i]``: places inside portion i whose logits are asked for
        (default: its last token).  Returns (logits [n, V] fp32, next tokens [n] int32), rows in the order of the
        sequences and of their places."""
        kv, dev = self.kv, self.m.device
        if adapter_slots is None:
            adapter_slots = [-1] * len(seq_ids)
        if want is None:
            want = [[len(p) - 1] for p in portions]
        first_out = np.cumsum([0] + [len(w) for w in want]).tolist()
        out_logits = torch.empty(first_out[-1], self.m.V, dtype=torch.float32, device=dev)
        out_tok = torch.empty(first_out[-1], dtype=torch.int32, device=dev)
        # rows: (seq index, position) in sequence order, cut into chunks
        pending = [(i, 0) for i in range(len(seq_ids)) if len(portions[i])]
        while pending:
            rows_left = self.max_rows
            chunk = []  # (seq index, start, n)
            nxt = []
            for i, start in pending:
                n_total = len(portions[i])
                if rows_left == 0:
                    nxt.append((i, start))
                    continue
                n = min(rows_left, n_total - start)
                chunk.append((i, start, n))
                rows_left -= n
                if start + n < n_total:
                    nxt.append((i, start + n))
            pending = nxt
            T = sum(n for _, _, n in chunk)
            toks = np.concatenate([np.asarray(portions[i][s:s + n], dtype=np.int32) for i, s, n in chunk])
            slots = np.concatenate([np.full(n, adapter_slots[i], dtype=np.int32) for i, _, n in chunk])
            passes, a = [], 0
            for i, _, n in chunk:
                passes.append((seq_ids[i], a, n, kv.length(seq_ids[i])))
                a += n
            row_slot, row_pos = kv.begin_forward([seq_ids[i] for i, _, _ in chunk], [n for _, _, n in chunk])
            self._stage(self.tokens, toks, torch.int32)
            self._stage(self.slots, slots, torch.int32)
            self.n_distinct = len({int(s) for s in slots if s >= 0})
            self.max_keys = max(p0 + n for _, _, n, p0 in passes)
            self.row_slot[:T].copy_(row_slot)
            self.row_pos[:T].copy_(row_pos)
            rows, dest, row_of = [], [], {}
            for (i, s, n), (_, r0, _, _) in zip(chunk, passes):
                for k, w in enumerate(want[i]):
                    if s <= w < s + n:
                        r = r0 + w - s
                        if r not in row_of:
                            row_of[r] = len(rows)
                            rows.append(r)
                        dest.append((first_out[i] + k, row_of[r]))
            self._begin_prompt_pass(passes)
            self._stage(self.last_rows, rows or [T - 1], torch.int32)
            lg, tk = self.forward(T, False, use_lora, self.last_rows, max(len(rows), 1))
            if rows:
                to, src = torch.tensor(dest, device=dev).unbind(1)
                out_logits[to] = lg[src]
                out_tok[to] = tk[src]
            kv.end_forward()
            self._end_prompt_pass()
        self.check_status()  # (synchronises; prefill is not the latency-critical call)
        self._check_prompt_status()
        return out_logits, out_tok

    def prefill(self, seq_ids, prompts, adapter_slots, use_lora=True):
        """Prefill whole prompts (lists of token ids) of already-added sequences, chunked to
        max_rows rows per pass.  Returns (logits [n_seq,V] fp32, next tokens [n_seq] int32)."""
        return self.extend(seq_ids, prompts, adapter_slots, use_lora=use_lora)

    def decode(self, seq_ids, tokens, adapter_slots, use_lora=True):
        """One eager decode step (host builds the row tables, as the reference's executor does)."""
        B = len(seq_ids)
        row_slot, row_pos = self.kv.begin_forward(seq_ids, [1] * B)
        self.max_keys = max(self.kv.length(s) for s in seq_ids) + 1
        self._stage(self.tokens, tokens, torch.int32)
        self._stage(self.slots, adapter_slots, torch.int32)
        self.n_distinct = len({int(s) for s in adapter_slots if s >= 0})
        self.row_slot[:B].copy_(row_slot)
        self.row_pos[:B].copy_(row_pos)
        out = self.forward(B, True, use_lora)
        self.kv.end_forward()
        return out

    # -- CUDA-graph decode: the whole step, including position bookkeeping, is one graph ---------------
    def capture_decode(self, seq_ids, adapter_slots, use_lora=True, reserve_tokens=0, feed_back=True):
        """Capture a decode step for this batch.  Rows follow ``seq_ids``; each replay consumes
        self.tokens[:B] (device) and leaves greedy tokens in self.next_tok[:B]."""
        B, kv = len(seq_ids), self.kv
        for sid in seq_ids:
            kv.reserve(sid, kv.length(sid) + reserve_tokens + 1)
        self._stage(self.row_slot, [kv.slot(s) for s in seq_ids], torch.int32)
        self._stage(self.slots, adapter_slots, torch.int32)
        self.n_distinct = len({int(s) for s in adapter_slots if s >= 0})
        self.max_keys = max(kv.tokens_reserved(s) for s in seq_ids)
        torch.cuda.synchronize()
        saved, undo = kv.seq_lens.clone(), kv.snapshot(seq_ids)

        def step():
            ops.kv_begin_decode(self.row_slot[:B], kv.seq_lens, self.row_pos[:B])
            self.forward(B, True, use_lora)
            if feed_back:  # the greedy tokens become the next step's input without leaving the device
                self.tokens[:B].copy_(self.next_tok[:B])

        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            step()  # warm-up outside capture (lazy module loading, attribute setting)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            step()
        kv.seq_lens.copy_(saved)  # warm-up advanced the device lengths (and states); capture itself runs nothing
        undo()
        torch.cuda.synchronize()
        return DecodeGraph(self, g, list(seq_ids), B)


class PlainEngine(EngineBase):
    """What the designs without adapters share: projections in the model's precision, buffers grown on demand, the status word
    of kernels with bounded waits.  ``linears``: (in, out) of every projection of a pass."""

    def __init__(self, model, kv: PagedCache, max_rows: int, linears, work_bytes: int = 0):
        super().__init__(model, kv, max_rows)
        lib, T = ops._lib.lib(), self.max_rows
        # (some projections have more rows than the pass: scratch no longer grows beyond 128)
        need = max([work_bytes] + [lib.mlora_linear_workspace(max(T, 128), k, n) for k, n in linears])
        self.ws_linear = ops.new_workspace(need, model.device)
        self.status = torch.zeros(1, dtype=torch.int32, device=model.device)
        self._buf, self._retired = {}, []

    # -- buffers that only some passes need, grown on demand (never while a graph is being captured: its warm-up run
    # -- has the same sizes); outgrown ones stay alive for the graphs that hold their addresses -------------------
    def _grow(self, name, numel, dtype=None):
        t = self._buf.get(name)
        if t is None or t.numel() < numel:
            if t is not None:
                self._retired.append(t)
            t = self._buf[name] = torch.zeros(numel, dtype=dtype or self.m.dtype, device=self.m.device)
        return t[:numel]

    def check_status(self):
        super().check_status()
        if int(self.status.item()):
            self.status.zero_()
            raise RuntimeError("mlora: an attention kernel gave up a bounded wait; this pass's results are undefined")

    def _linear(self, x, W, out, flags=0):
        if self.m.dtype == torch.float32:  # (OUT_F32: what it writes anyway)
            return ops.linear_f32(x, W, flags & ~ops.OUT_F32, out=out)
        return ops.linear(x, W, flags=flags, out=out, work=self.ws_linear)


class DecodeGraph:
    def __init__(self, engine, graph, seq_ids, B):
        self.engine, self.graph, self.seq_ids, self.B = engine, graph, seq_ids, B
        self._headroom = 0  # replays known to be covered by reserved pages (re-counted when it runs out)

    def replay(self):
        """One token for every row: consumes engine.tokens[:B], leaves greedy tokens in
        engine.next_tok[:B] (and, when captured with feed_back, back in engine.tokens).
        The step appends one token per sequence through block-table entries that must exist already:
        pages are reserved here when the host allocator still has some, else the replay is refused."""
        kv = self.engine.kv
        if self._headroom <= 0:
            for sid in self.seq_ids:
                kv.reserve(sid, kv.length(sid) + 1)  # raises when the pool or the row's table is exhausted
            self._headroom = min(kv.tokens_reserved(sid) - kv.length(sid) for sid in self.seq_ids)
        self._headroom -= 1
        self.graph.replay()
        self.engine.kv.note_device_decode(self.seq_ids)


class DecodeSession:
    """The batched greedy loop of one fused decode node (``tvm/llama_auto_batcher/llama_exec_graph.py:102-141``)
    with the batch state on the device: sequences finish on their end-of-sequence token or their own
    ``max_gen_len`` and leave the batch without the host rebuilding anything.  Every step is a CUDA-graph replay
    of ``decode_step_begin -> forward -> decode_step_end`` captured for a bucket of rows (powers of two up to the
    node's size); the host only learns the live count (4 bytes, every ``sync_every`` steps) to pick the bucket and
    to stop, and reads all generated tokens once at the end.

    ``seq_ids`` must already be in bucketing order (``LlamaSeqInfo.order_seqs``): rows of one adapter adjacent."""

    def __init__(self, engine: EngineBase, seq_ids, adapter_slots, first_tokens, max_gen, eos_id=None, use_lora=True):
        self.eng, self.seq_ids, self.use_lora = engine, list(seq_ids), use_lora
        kv, dev, n = engine.kv, engine.m.device, len(seq_ids)
        self.n = n
        self.max_len = int(max(max_gen)) + 1  # (a sequence always takes part in the node's first step)
        i32 = lambda v: torch.as_tensor(np.asarray(v, dtype=np.int32)).pin_memory().to(dev, non_blocking=True)
        self.live = torch.ones(n, dtype=torch.int32, device=dev)
        self.seq_slot = i32([kv.slot(s) for s in seq_ids])
        self.adapter_slot = i32(adapter_slots)
        self.last_tok = i32(first_tokens)
        self.max_gen = i32(max_gen)
        self.gen_count = torch.ones(n, dtype=torch.int32, device=dev)  # the prefill's token is the first one
        self.out_tokens = torch.zeros(n, self.max_len, dtype=torch.int32, device=dev)
        self.out_tokens[:, 0] = self.last_tok
        self.row_src = torch.full((max(n, 1),), -1, dtype=torch.int32, device=dev)
        self.n_live = torch.zeros(1, dtype=torch.int32, device=dev)
        self._n_live_host = torch.zeros(1, dtype=torch.int32).pin_memory()
        self.eos_id = -1 if eos_id is None else int(eos_id)
        self.n_distinct = len({int(a) for a in adapter_slots if a >= 0})
        for sid, g in zip(seq_ids, max_gen):
            kv.reserve(sid, kv.length(sid) + int(g) + 1)
        self.max_keys = max((kv.tokens_reserved(sid) for sid in seq_ids), default=1)
        self._graphs = {}
        self.steps = 0
        self.d2h_bytes = 0

    def _step(self, rows):
        e = self.eng
        ops.decode_step_begin(self.live, self.seq_slot, self.adapter_slot, self.last_tok, rows, e.kv.seq_lens,
                              self.row_src, e.row_slot, e.row_pos, e.slots, e.tokens, self.n_live)
        e.n_distinct, e.max_keys = self.n_distinct, self.max_keys
        e.forward(rows, True, self.use_lora)
        ops.decode_step_end(self.row_src, e.next_tok, rows, self.live, self.last_tok, self.gen_count, self.max_gen,
                            self.out_tokens, self.eos_id, self.n_live)

    def _graph(self, rows):
        g = self._graphs.get(rows)
        if g is not None:
            return g
        e = self.eng
        state = (self.live, self.last_tok, self.gen_count, self.out_tokens, e.kv.seq_lens, self.n_live)
        saved, undo = [t.clone() for t in state], e.kv.snapshot(self.seq_ids)
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            self._step(rows)  # warm-up outside capture; its effects are undone below
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            self._step(rows)
        for t, s in zip(state, saved):
            t.copy_(s)
        undo()
        torch.cuda.synchronize()
        self._graphs[rows] = g
        return g

    @staticmethod
    def bucket(n_live, n):
        """Rows of the step that serves ``n_live`` live sequences: the next power of two, capped at the node's size."""
        b = 1
        while b < n_live:
            b *= 2
        return min(b, n)

    def run(self, sync_every=1):
        """Runs until every sequence has finished.  Returns the token lists (first token included) in the order of
        ``seq_ids``."""
        bound = self.n  # upper bound of the live count (sequences only ever leave)
        while bound > 0:
            g = self._graph(self.bucket(bound, self.n))
            for _ in range(max(1, sync_every)):
                g.replay()
                self.steps += 1
            self._n_live_host.copy_(self.n_live, non_blocking=True)
            torch.cuda.current_stream().synchronize()
            self.d2h_bytes += 4
            bound = int(self._n_live_host[0])
        counts = self.gen_count.cpu().tolist()
        toks = self.out_tokens.cpu().tolist()
        self.d2h_bytes += 4 * (self.n + self.out_tokens.numel())
        for sid, c in zip(self.seq_ids, counts):
            self.eng.kv.note_device_decode([sid], c - 1)
        return [t[:c] for t, c in zip(toks, counts)]
