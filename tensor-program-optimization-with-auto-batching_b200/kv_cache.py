"""Paged caches: device pages + block tables, host-side page allocator.

Stands in for the object ``vm["create_paged_kv_cache"]`` returns and for the
``vm.builtin.kv_state_*`` functions the reference executor calls
(``tvm/llama_auto_batcher/llama_exec_graph.py:38-46,66,75-79,85,121-127``;
cache parameters ``tvm/llama_auto_batcher/llama_for_causal_lm.py:148-174``).

:class:`PagedCache` is the bookkeeping, shared by all kinds of cache: a block table ``[max_batch, max_pages]``
int32 and ``seq_lens [max_batch]`` int32.  Page ids are handed out by a host
free list; the device tables are refreshed with small async copies when they
change.  A decode step captured in a CUDA graph advances ``seq_lens`` on the
device itself (``mlora_kv_begin_decode``), so pages for the tokens a graph
will append must be reserved ahead with :meth:`reserve`.
"""
from __future__ import annotations

import numpy as np
import torch

from . import ops


class PagedCache:
    """Sequences, slots, page ids and block table; what a page holds is up to the subclass."""

    def __init__(self, max_batch, max_total_seq_len, prefill_chunk_size, page_size, device, max_seq_len=None):
        if page_size not in (16, 32):
            raise ValueError("page_size must be 16 or 32")
        self.max_batch, self.page_size = int(max_batch), int(page_size)
        self.prefill_chunk_size = int(prefill_chunk_size)
        self.device = torch.device(device)
        ps = self.page_size
        # every sequence may leave one page partly filled
        self.n_pages = (int(max_total_seq_len) + ps - 1) // ps + self.max_batch
        per_seq = int(max_seq_len) if max_seq_len else int(max_total_seq_len)
        self.max_pages = min((per_seq + ps - 1) // ps + 1, self.n_pages)
        self.block_table = torch.zeros(self.max_batch, self.max_pages, dtype=torch.int32, device=self.device)
        self.seq_lens = torch.zeros(self.max_batch, dtype=torch.int32, device=self.device)
        # host mirrors; device refreshes go through a fresh pinned staging tensor per copy, so a
        # later host-side update can never race with an asynchronous copy still in the stream
        self._bt_host = np.zeros((self.max_batch, self.max_pages), dtype=np.int32)
        self._len_host = np.zeros(self.max_batch, dtype=np.int32)
        self._free = list(range(self.n_pages - 1, -1, -1))
        self._slot_of = {}           # sid -> slot
        self._free_slots = list(range(self.max_batch - 1, -1, -1))
        self._n_pages_of = {}        # sid -> pages held
        self._pending = None

    # -- sequences -----------------------------------------------------------------------------
    def add_sequence(self, sid):
        if sid in self._slot_of:
            raise ValueError(f"sequence {sid} is already in the cache")
        if not self._free_slots:
            raise RuntimeError("no free sequence slot (max_batch reached)")
        slot = self._free_slots.pop()
        self._slot_of[sid] = slot
        self._n_pages_of[sid] = 0
        self._len_host[slot] = 0
        self._push(self.seq_lens[slot:slot + 1], self._len_host[slot:slot + 1])
        return slot

    def _push(self, dst, src_np):
        dst.copy_(torch.from_numpy(np.ascontiguousarray(src_np)).pin_memory(), non_blocking=True)

    def remove_sequence(self, sid):
        slot = self._slot_of.pop(sid)
        n = self._n_pages_of.pop(sid)
        self._free.extend(int(p) for p in self._bt_host[slot, :n].tolist()[::-1])
        self._free_slots.append(slot)

    def slot(self, sid):
        return self._slot_of[sid]

    def length(self, sid):
        return int(self._len_host[self._slot_of[sid]])

    def tokens_reserved(self, sid):
        """Tokens the pages held by ``sid`` have room for."""
        return self._n_pages_of[sid] * self.page_size

    def reserve(self, sid, n_tokens):
        """Make sure pages exist for ``n_tokens`` total tokens of sequence ``sid``."""
        slot = self._slot_of[sid]
        need = (int(n_tokens) + self.page_size - 1) // self.page_size
        have = self._n_pages_of[sid]
        if need <= have:
            return
        if need > self.max_pages:
            raise RuntimeError(f"sequence {sid} needs {need} pages, block table holds {self.max_pages}")
        if need - have > len(self._free):
            raise RuntimeError("paged KV cache is out of pages")
        for p in range(have, need):
            self._bt_host[slot, p] = self._free.pop()
        self._n_pages_of[sid] = need
        self._push(self.block_table[slot, have:need], self._bt_host[slot, have:need])

    # -- the reference's forward protocol -------------------------------------------------------------
    def begin_forward(self, seq_ids, append_lens):
        """Reserve pages for the rows of this forward and return (row_slot, row_pos) device tensors:
        one row per appended token, sequences in the order given."""
        seq_ids = [int(s) for s in seq_ids]
        append_lens = [int(a) for a in append_lens]
        slots, pos = [], []
        for sid, a in zip(seq_ids, append_lens):
            slot = self._slot_of[sid]
            n0 = int(self._len_host[slot])
            self.reserve(sid, n0 + a)
            slots.extend([slot] * a)
            pos.extend(range(n0, n0 + a))
        self._pending = (seq_ids, append_lens)
        row_slot = torch.tensor(slots, dtype=torch.int32).pin_memory().to(self.device, non_blocking=True)
        row_pos = torch.tensor(pos, dtype=torch.int32).pin_memory().to(self.device, non_blocking=True)
        return row_slot, row_pos

    def end_forward(self):
        seq_ids, append_lens = self._pending
        self._pending = None
        for sid, a in zip(seq_ids, append_lens):
            slot = self._slot_of[sid]
            self._len_host[slot] += a
        slots = sorted(self._slot_of[s] for s in seq_ids)
        lo, hi = slots[0], slots[-1] + 1
        self._push(self.seq_lens[lo:hi], self._len_host[lo:hi])

    def note_device_decode(self, seq_ids, n_steps=1):
        """Tell the host mirror that a captured decode step advanced these sequences on the device."""
        for sid in seq_ids:
            self._len_host[self._slot_of[int(sid)]] += n_steps

    def snapshot(self, seq_ids):
        """Whatever a step of these sequences changes and running it again would not put right (pages are simply written
        again): a function that puts it back."""
        return lambda: None

    # -- checks used by tests ---------------------------------------------------------------------
    def _gather_pages(self, pages, sid):
        """The first ``length(sid)`` rows of a sequence out of ``pages`` [n_pages, page_size, ...]."""
        slot = self._slot_of[sid]
        n = int(self._len_host[slot])
        n_pg = (n + self.page_size - 1) // self.page_size
        idx = torch.from_numpy(self._bt_host[slot, :n_pg].astype(np.int64)).to(self.device)
        return pages[idx].flatten(0, 1)[:n]


class PagedKVCache(PagedCache):
    """Keys and values per layer and head: ``[n_layers, 2, n_pages, Hkv, page_size, D]`` bf16."""

    def __init__(self, n_layers, n_kv_heads, head_dim, max_batch, max_total_seq_len, prefill_chunk_size,
                 page_size, device, max_seq_len=None):
        super().__init__(max_batch, max_total_seq_len, prefill_chunk_size, page_size, device, max_seq_len)
        self.n_layers, self.Hkv, self.D = n_layers, n_kv_heads, head_dim
        self.pages = torch.zeros(n_layers, 2, self.n_pages, n_kv_heads, self.page_size, head_dim, dtype=torch.bfloat16,
                                 device=self.device)

    # -- layer views -----------------------------------------------------------------------------
    def k_pages(self, layer):
        return self.pages[layer, 0]

    def v_pages(self, layer):
        return self.pages[layer, 1]

    def gather(self, sid, layer):
        """(K, V) of a sequence as dense [n, Hkv, D] tensors (block-table gather)."""
        return [self._gather_pages(self.pages[layer, kv].transpose(1, 2), sid) for kv in (0, 1)]


class PagedLatentCache(PagedCache):
    """One latent vector per token for every layer that computes latents: ``[n_pages, page_size, pitch]`` per such
    layer, a page in the tiled order of ``csrc/latent.cuh`` (:meth:`untile`).  Layers that attend to another layer's latents hold nothing and read that layer's pages.

    ``ranks``: layer -> kv_rank of the layers that own latents (the pitch is the rank rounded up to 64)."""

    def __init__(self, ranks, max_batch, max_total_seq_len, prefill_chunk_size, page_size, device, max_seq_len=None,
                 dtype=torch.bfloat16):
        super().__init__(max_batch, max_total_seq_len, prefill_chunk_size, page_size, device, max_seq_len)
        self.ranks = dict(ranks)
        self.pages = {l: torch.zeros(self.n_pages, self.page_size, -(-r // 64) * 64, dtype=dtype, device=self.device)
                      for l, r in self.ranks.items()}

    def latent_pages(self, layer):
        return self.pages[layer]

    def gather(self, sid, layer):
        """Latents of a sequence, dense [n, kv_rank]."""
        return self._gather_pages(self.untile(self.pages[layer]), sid)[:, :self.ranks[layer]]

    @staticmethod
    def untile(pages):
        """Row-major copy of ``pages`` [n_pages, page_size, pitch] stored as [page_size / 8][pitch / 64][8][8 chunks][8]
        with chunk c of row r at place c ^ r."""
        n, ps, pitch = pages.shape
        r = torch.arange(8, device=pages.device)
        t = pages.reshape(n, ps // 8, pitch // 64, 8, 8, 8)[:, :, :, r[:, None], r[:, None] ^ r[None, :]]
        return t.transpose(2, 3).reshape(n, ps, pitch)


class HybridCache(PagedCache):
    """Layers that keep keys and values per token (pages) beside layers that keep a state of fixed size per sequence.

    ``attention``: entry -> (kv heads, head size as stored); ``states``: entry -> {name: (shape of one sequence, dtype)}, stored
    as [max_batch, *shape] by the sequence's slot.  An entry is one run of a layer: a layer that runs several times has as many.
    A state is not cleared when a slot changes hands: whoever reads it takes position 0 as a start from zero."""

    def __init__(self, attention, states, max_batch, max_total_seq_len, prefill_chunk_size, page_size, device, max_seq_len=None,
                 dtype=torch.bfloat16):
        super().__init__(max_batch, max_total_seq_len, prefill_chunk_size, page_size, device, max_seq_len)
        self.pages = {e: torch.zeros(2, self.n_pages, h, self.page_size, d, dtype=dtype, device=self.device)
                      for e, (h, d) in attention.items()}
        self.states = {e: {name: torch.zeros(self.max_batch, *shape, dtype=dt, device=self.device)
                           for name, (shape, dt) in entry.items()} for e, entry in states.items()}

    def k_pages(self, entry):
        return self.pages[entry][0]

    def v_pages(self, entry):
        return self.pages[entry][1]

    def state(self, entry, name):
        return self.states[entry][name]

    def gather(self, sid, entry):
        """(K, V) of a sequence as dense [n, kv heads, head size] tensors."""
        return [self._gather_pages(p.transpose(1, 2), sid) for p in self.pages[entry]]

    def snapshot(self, seq_ids):
        slots = torch.tensor([self._slot_of[int(s)] for s in seq_ids], dtype=torch.int64, device=self.device)
        saved = [(t, t.index_select(0, slots)) for entry in self.states.values() for t in entry.values()]

        def restore():
            for t, old in saved:
                t.index_copy_(0, slots, old)
        return restore


# The three global functions of the reference's runtime, same names and argument order.
def kv_state_add_sequence(kv: PagedCache, sid):
    kv.add_sequence(int(sid))


def kv_state_begin_forward(kv: PagedCache, seq_ids, append_lens):
    kv._rows = kv.begin_forward(list(seq_ids), list(append_lens))


def kv_state_end_forward(kv: PagedCache):
    kv.end_forward()
    kv._rows = None
