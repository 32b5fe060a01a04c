"""Paged KV cache of all layers of one rank plus the page table / lengths of the running batch.

Every model family describes what its layers store (``cfg.cache_layout``: heads, key and value sizes, element type, how
far back a position looks); pages of 16 tokens (``rt.page_size``) are handed out per sequence and shared by all layers,
i.e. page *p* of a sequence is record *p* of every layer's storage.  Layers that look back only to the start of their
own chunk let go of older tokens: when no layer can see a page any more it returns to the free list (``retire``).

Beside the pages every sequence slot has a fixed-size fp32 state per layer (``cfg.state_layout``: the previous token's row
of a token shift, the state of a recurrence).  Kernels take a sequence's state as zero at position 0, so a slot needs no
clearing between sequences, and change it only where ``active`` says that the slot takes part in the step."""
from __future__ import annotations

import torch

from ..ops import attention as A
from .config import CacheSpec, ModelConfig, RuntimeConfig

_DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def _record(s: CacheSpec | None, page_size: int) -> int:
    return s.kv_heads * page_size * (s.dk + s.dv) if s is not None else 0


def _states(cfg) -> list[dict[str, int]]:
    return cfg.state_layout() if hasattr(cfg, "state_layout") else []


class KVState:
    @staticmethod
    def pool_pages(cfg, rt: RuntimeConfig, num_seqs: int, max_seq_len: int) -> int:
        """Pages the free list starts with: what the slots can hold at once, unless ``rt.kv_pool_tokens`` says less."""
        ps = rt.page_size
        per_seq = (max_seq_len + ps - 1) // ps
        chunks = [s.chunk for s in cfg.cache_layout(rt) if s is not None]
        if all(chunks):
            # what lies before the oldest visible chunk is given back between portions of a prompt
            per_seq = min(per_seq, (max(chunks, default=0) + rt.max_prefill_tokens + ps - 1) // ps + 2)
        total = num_seqs * per_seq
        if rt.kv_pool_tokens > 0:
            total = min(total, (rt.kv_pool_tokens + ps - 1) // ps + 2 * num_seqs)
        return total

    @staticmethod
    def nbytes(cfg, rt: RuntimeConfig, num_seqs: int, max_seq_len: int) -> int:
        """Device bytes of a cache for ``num_seqs`` sequences of up to ``max_seq_len`` tokens (storage + tables)."""
        max_pages = (max_seq_len + rt.page_size - 1) // rt.page_size
        pages = KVState.pool_pages(cfg, rt, num_seqs, max_seq_len) + 1
        layout = cfg.cache_layout(rt)
        size = max((_DTYPES[s.dtype].itemsize for s in layout if s is not None), default=0)
        states = sum(n for run in _states(cfg) for n in run.values()) * num_seqs * 4
        return sum(_record(s, rt.page_size) for s in layout) * pages * size + states + num_seqs * max_pages * 4 + num_seqs * 8 + 3 * 1024

    def __init__(self, cfg: ModelConfig, rt: RuntimeConfig, device, num_seqs: int, max_seq_len: int, alloc=None):
        """``alloc(shape, dtype) -> zeroed tensor``: where the cache lives (the rank's HBM arena); default torch.zeros.

        Pages are handed out on demand (``admit`` as a sequence grows) from a host-side free list.  The last page is
        a scratch page no sequence owns: the page-table rows of empty slots point at it, so a kernel that runs over
        an empty slot of the batch has somewhere harmless to write."""
        if alloc is None:
            def alloc(shape, dtype):
                return torch.zeros(shape, dtype=dtype, device=device)
        self.page_size = rt.page_size
        self.num_seqs = num_seqs
        self.max_pages = (max_seq_len + rt.page_size - 1) // rt.page_size
        self.num_pages = self.pool_pages(cfg, rt, num_seqs, max_seq_len) + 1
        self.scratch_page = self.num_pages - 1
        self.layout = cfg.cache_layout(rt)
        assert len({s.dtype for s in self.layout if s is not None}) <= 1
        sizes = [_record(s, rt.page_size) * self.num_pages for s in self.layout]
        dtype = next((s.dtype for s in self.layout if s is not None), rt.dtype)
        self.storage = alloc((max(1, sum(sizes)),), _DTYPES[dtype])
        self.layers, at = [], 0
        for s, n in zip(self.layout, sizes):
            self.layers.append(A.PagedKVCache(self.num_pages, s.kv_heads, rt.page_size, device, storage=self.storage[at:at + n],
                                              dk=s.dk, dv=s.dv) if s is not None else None)
            at += n
        # [sequence][numbers] per run and name; the numbers of a run are multiples of eight
        self.states: list[dict[str, torch.Tensor]] = []
        layout = _states(cfg)
        flat, at = alloc((max(1, sum(n for run in layout for n in run.values()) * num_seqs),), torch.float32), 0
        for run in layout:
            self.states.append({})
            for name, n in run.items():
                self.states[-1][name] = flat[at:at + n * num_seqs].view(num_seqs, n)
                at += n * num_seqs
        self.active = alloc((num_seqs,), torch.int32)         # 1: the slot takes part in the next decode step
        self.page_table = alloc((num_seqs, self.max_pages), torch.int32)
        self.seq_lens = alloc((num_seqs,), torch.int32)
        self.free_pages = list(range(self.num_pages - 2, -1, -1))
        self.owned: dict[int, list[int]] = {}       # page ids of a slot in token order; -1: given back by ``retire``
        self._retired: dict[int, int] = {}          # leading entries of ``owned`` that are -1
        # host mirror of the page table: rows are edited here; ``flush`` sends a snapshot (a ring of pinned buffers, so
        # that a copy still queued on the stream never sees an edit that belongs to a later step)
        self.table_host = torch.full((num_seqs, self.max_pages), self.scratch_page, dtype=torch.int32)
        self._cuda = torch.cuda.is_available() and torch.device(device).type == "cuda"
        self._ring = [(self.table_host.clone().pin_memory(), torch.cuda.Event()) for _ in range(4)] if self._cuda else []
        self._turn = 0
        self._dirty = True
        self.pages_high_water = 0

    def admit(self, seq: int, n_tokens: int) -> None:
        """Make sure sequence slot ``seq`` owns pages for ``n_tokens`` tokens (grows, never shrinks)."""
        need = (n_tokens + self.page_size - 1) // self.page_size
        if need > self.max_pages:
            raise RuntimeError(f"{n_tokens} tokens exceed the {self.max_pages * self.page_size} a page-table row can describe")
        have = self.owned.setdefault(seq, [])
        if need - len(have) > len(self.free_pages):
            raise RuntimeError("KV cache exhausted")
        while len(have) < need:
            self.table_host[seq, len(have)] = self.free_pages[-1]
            have.append(self.free_pages.pop())
            self._dirty = True
        self.pages_high_water = max(self.pages_high_water, self.num_pages - 1 - len(self.free_pages))

    def first_visible(self, pos: int) -> int:
        """Oldest position that some layer of a token at ``pos`` (or any later one) can still see."""
        return min(((pos - pos % s.chunk) if s.chunk else 0 for s in self.layout if s is not None), default=pos)

    def retire(self, seq: int, pos: int) -> None:
        """The next token of slot ``seq`` goes to position ``pos``: pages that lie wholly before everything it can see
        return to the free list."""
        pages = self.owned.get(seq)
        if not pages:
            return
        n0, n1 = self._retired.get(seq, 0), min(self.first_visible(pos) // self.page_size, len(pages))
        for i in range(n0, n1):
            self.free_pages.append(pages[i])
            pages[i] = -1
        if n1 > n0:
            self.table_host[seq, n0:n1] = self.scratch_page
            self._retired[seq] = n1
            self._dirty = True

    def release(self, seq: int) -> None:
        """Give the pages of slot ``seq`` back; its page-table row points at the scratch page again."""
        pages = self.owned.pop(seq, [])
        self._retired.pop(seq, None)
        if pages:
            self.free_pages.extend(p for p in reversed(pages) if p >= 0)
            self.table_host[seq].fill_(self.scratch_page)
            self._dirty = True

    def flush(self) -> None:
        """Copy the page table to the device if a row changed since the last flush (asynchronous, stream-ordered)."""
        if not self._dirty:
            return
        if self._cuda:
            buf, done = self._ring[self._turn]
            self._turn = (self._turn + 1) % len(self._ring)
            done.synchronize()                       # its previous copy has left the buffer
            buf.copy_(self.table_host)
            self.page_table.copy_(buf, non_blocking=True)
            done.record()
        else:
            self.page_table.copy_(self.table_host)
        self._dirty = False

    def pages_in_use(self) -> int:
        return self.num_pages - 1 - len(self.free_pages)
