"""Paged KV cache.

The reference keeps Python lists of per-layer block objects and concatenates them on every read
(model/core/cache.py:535-868, read path :824-835); its unified manager is lossy by default (H2O,
quantisation, eviction; cache.py:1886-2038).  Here the cache is two device tensors per layer
``[num_blocks, block_size, n_kv_head, head_dim]`` plus an int32 block table per sequence; the decode kernel
reads pages in place.  ``YvPagedLayeredCache`` keeps the same pages, tables and free list for layer runs that each store
what they need (keys and values of sizes of their own, or one latent row per token), and gives pages back once every
layer's window has passed them.  The cache is exact; eviction policies (LRU of whole sequences, sliding window) are
opt-in helpers that only edit block tables.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import numpy as np
import torch


RELEASED = -1      # table entry of a page that was given back because no later token can see it


@dataclass
class YvCacheConfig:
    block_size: int = 64
    num_blocks: int = 1024
    max_blocks_per_seq: int = 2048
    dtype: torch.dtype = torch.bfloat16
    sliding_window: Optional[int] = None      # keep only the last N tokens addressable (opt-in, lossy)


class YvBlockAllocator:
    """Free-list allocator of cache pages with reference counts (prefix sharing)."""

    def __init__(self, num_blocks: int):
        self.num_blocks = num_blocks
        self.free: List[int] = list(range(num_blocks - 1, -1, -1))
        self.refs: Dict[int, int] = {}

    def available(self) -> int:
        return len(self.free)

    def alloc(self) -> int:
        if not self.free:
            raise MemoryError("paged KV cache is out of blocks")
        b = self.free.pop()
        self.refs[b] = 1
        return b

    def share(self, b: int) -> int:
        self.refs[b] += 1
        return b

    def release(self, b: int) -> None:
        self.refs[b] -= 1
        if self.refs[b] == 0:
            del self.refs[b]
            self.free.append(b)


class YvPagedKVCache:
    """Block pool for all layers of one model replica plus per-sequence block tables (host side)."""

    def __init__(self, n_layer: int, n_kv_head: int, head_dim: int, cfg: YvCacheConfig, device: torch.device):
        self.cfg, self.device = cfg, device
        self.n_layer, self.hk, self.d = n_layer, n_kv_head, head_dim
        shape = (cfg.num_blocks, cfg.block_size, n_kv_head, head_dim)
        self.k = [torch.zeros(shape, dtype=cfg.dtype, device=device) for _ in range(n_layer)]
        self.v = [torch.zeros(shape, dtype=cfg.dtype, device=device) for _ in range(n_layer)]
        self.alloc = YvBlockAllocator(cfg.num_blocks)
        self.tables: Dict[int, List[int]] = {}       # seq id -> physical blocks
        self.lengths: Dict[int, int] = {}
        self.layer_offset = 0                         # first global layer index held by this pipeline stage
        # tokens (the query's own included) that the widest layer still reads; None = every token stays addressable
        self.reach: Optional[int] = None

    def layer(self, idx: int) -> Tuple[torch.Tensor, torch.Tensor]:
        return self.k[idx - self.layer_offset], self.v[idx - self.layer_offset]

    def bytes(self) -> int:
        return 2 * self.n_layer * self.k[0].numel() * self.k[0].element_size()

    # ---- sequence management (host) ---------------------------------------------------------------
    def add_sequence(self, seq_id: int) -> None:
        self.tables[seq_id] = []
        self.lengths[seq_id] = 0

    def free_sequence(self, seq_id: int) -> None:
        for b in self.tables.pop(seq_id, []):
            if b != RELEASED:
                self.alloc.release(b)
        self.lengths.pop(seq_id, None)

    def release_passed(self, seq_id: int) -> int:
        """Give back the pages that no token from here on can see (all layers windowed; see ``reach``).  Their table
        entries stay as placeholders, so that page i keeps holding tokens ``i * block_size ...``.  One page of slack
        is kept for callers that step back a few tokens.  Returns the number of pages freed."""
        if self.reach is None:
            return 0
        bs, tbl = self.cfg.block_size, self.tables[seq_id]
        last = (self.lengths[seq_id] - self.reach + 1 - bs) // bs          # pages below this one are out of reach
        freed = 0
        for i in range(min(last, len(tbl)) - 1, -1, -1):
            if tbl[i] == RELEASED:
                break                                                     # everything in front of it has gone before
            self.alloc.release(tbl[i])
            tbl[i] = RELEASED
            freed += 1
        return freed

    def fork(self, src: int, dst: int) -> None:
        """Share all full blocks of ``src`` with ``dst`` (prefix caching / beam search)."""
        self.tables[dst] = [b if b == RELEASED else self.alloc.share(b) for b in self.tables[src]]
        self.lengths[dst] = self.lengths[src]

    def can_append(self, seq_id: int, n_tokens: int) -> bool:
        need = self._blocks_needed(seq_id, n_tokens)
        return need <= self.alloc.available()

    def _blocks_needed(self, seq_id: int, n_tokens: int) -> int:
        bs = self.cfg.block_size
        have = len(self.tables[seq_id])
        total = (self.lengths[seq_id] + n_tokens + bs - 1) // bs
        return max(0, total - have)

    def append_slots(self, seq_id: int, n_tokens: int) -> List[int]:
        """Reserve room for ``n_tokens`` new tokens; returns their flat slot ids (block * block_size + offset)."""
        bs = self.cfg.block_size
        self.release_passed(seq_id)
        for _ in range(self._blocks_needed(seq_id, n_tokens)):
            self.tables[seq_id].append(self.alloc.alloc())
        start = self.lengths[seq_id]
        tbl = self.tables[seq_id]
        slots = [tbl[(start + i) // bs] * bs + (start + i) % bs for i in range(n_tokens)]
        self.lengths[seq_id] = start + n_tokens
        return slots

    def slots(self, seq_id: int, lo: int, hi: int) -> np.ndarray:
        """Flat slot ids of the tokens lo .. hi - 1 (which must not have been given back)."""
        bs = self.cfg.block_size
        pos = np.arange(lo, hi)
        pages = np.asarray(self.tables[seq_id], dtype=np.int64)[pos // bs]
        if pages.size and int(pages.min()) < 0:
            raise IndexError(f"sequence {seq_id}: tokens {lo}..{hi - 1} reach into released pages")
        return pages * bs + pos % bs

    def block_table_tensor(self, seq_ids: List[int], width: Optional[int] = None) -> torch.Tensor:
        width = width or max(1, max(len(self.tables[s]) for s in seq_ids))
        t = torch.zeros(len(seq_ids), width, dtype=torch.int32)
        for i, s in enumerate(seq_ids):
            tbl = self.tables[s]
            if self.cfg.sliding_window is not None:
                keep = (self.cfg.sliding_window + self.cfg.block_size - 1) // self.cfg.block_size + 1
                tbl = tbl[-keep:]
            t[i, : len(tbl)] = torch.tensor(tbl, dtype=torch.int32)
        return t.to(self.device, non_blocking=True)

    def seq_lens_tensor(self, seq_ids: List[int]) -> torch.Tensor:
        return torch.tensor([self.lengths[s] for s in seq_ids], dtype=torch.int32).to(self.device, non_blocking=True)

    # ---- checkpoint / restore (reference cache.py:2394-2430) ------------------------------------------------
    def state(self) -> Dict[str, object]:
        return {"tables": {k: list(v) for k, v in self.tables.items()}, "lengths": dict(self.lengths),
                "k": [t.cpu() for t in self.k], "v": [None if t is None else t.cpu() for t in self.v]}

    def load_state(self, st: Dict[str, object]) -> None:
        self.tables = {int(k): list(v) for k, v in st["tables"].items()}      # type: ignore[union-attr]
        self.lengths = {int(k): int(v) for k, v in st["lengths"].items()}     # type: ignore[union-attr]
        used = {b for t in self.tables.values() for b in t if b != RELEASED}
        self.alloc = YvBlockAllocator(self.cfg.num_blocks)
        self.alloc.free = [b for b in range(self.cfg.num_blocks - 1, -1, -1) if b not in used]
        self.alloc.refs = {b: sum(b in t for t in self.tables.values()) for b in used}
        for mine, saved in ((self.k, st["k"]), (self.v, st["v"])):
            for t, src in zip(mine, saved):                                    # type: ignore[arg-type]
                if t is not None:
                    t.copy_(src)


class YvPagedLayeredCache(YvPagedKVCache):
    """Pages whose contents differ from layer run to layer run.  Layout i is ``{"row": n}`` (one row of n numbers per
    token) or ``{"heads": g, "dim": d, "vdim": e}`` (keys ``[num_blocks, block_size, g, d]`` and values ``[.., g, e]``)."""

    def __init__(self, layouts: List[Dict[str, int]], cfg: YvCacheConfig, device: torch.device, reach: Optional[int] = None):
        self.cfg, self.device = cfg, device
        self.n_layer = len(layouts)
        self.hk = max(m.get("heads", 1) for m in layouts)
        self.d = max(m["row"] if "row" in m else max(m["dim"], m["vdim"]) for m in layouts)
        page = lambda *tail: torch.zeros(cfg.num_blocks, cfg.block_size, *tail, dtype=cfg.dtype, device=device)
        self.k = [page(m["row"]) if "row" in m else page(m["heads"], m["dim"]) for m in layouts]
        self.v = [None if "row" in m else page(m["heads"], m["vdim"]) for m in layouts]
        self.alloc = YvBlockAllocator(cfg.num_blocks)
        self.tables, self.lengths = {}, {}
        self.layer_offset = 0
        self.reach = reach

    def rows(self, idx: int) -> torch.Tensor:
        if self.v[idx - self.layer_offset] is not None:
            raise TypeError("this layer stores keys and values: use layer()")
        return self.k[idx - self.layer_offset]

    def layer(self, idx: int):
        if self.v[idx - self.layer_offset] is None:
            raise TypeError("this layer stores one row per token: use rows()")
        return super().layer(idx)

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.k + self.v if t is not None)


def cache_for_model(cfg, device: torch.device, num_blocks: int, block_size: Optional[int] = None, tp_size: int = 1,
                    n_layer: Optional[int] = None, dtype: torch.dtype = torch.bfloat16) -> YvPagedKVCache:
    cc = YvCacheConfig(block_size=block_size or cfg.kv_cache_block_size, num_blocks=num_blocks, dtype=dtype)
    if cfg.layer_specs:
        from .registry import cache_layout
        layouts, reach = cache_layout(cfg)
        return YvPagedLayeredCache(layouts, cc, device, reach)
    return YvPagedKVCache(n_layer or cfg.n_layer, cfg.n_kv_head // tp_size, cfg.head_dim, cc, device)
