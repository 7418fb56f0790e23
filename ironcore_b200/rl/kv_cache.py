"""Paged caches: fixed-size pages, a host-side free list, per-sequence page tables.

:class:`PagedCache` owns sequences and pages; what a page holds is up to the subclass. ``block_table[seq, i]`` is the
physical block of a sequence's i-th page and ``seq_lens[seq]`` its current length; both live on the device and are
updated in place, so a captured CUDA graph of the decode step keeps reading the current state.

* :class:`BlockKVCache` — keys and values, pools ``[num_blocks, block_size, kv_heads, head_dim]`` per layer.
* :class:`LayerCache` — whatever the mixer of a layer run declares: rows per token, fixed-size states per sequence."""

from __future__ import annotations

from typing import Dict, Iterable, List, Optional, Sequence, Tuple

import torch


class PagedCache:
    def __init__(self, num_blocks: int, block_size: int, max_seqs: int, max_seq_len: int, device):
        if block_size % 16:
            raise ValueError("block_size must be a multiple of 16")
        self.num_blocks, self.block_size = num_blocks, block_size
        self.max_seqs, self.max_seq_len = max_seqs, max_seq_len
        self.max_blocks_per_seq = (max_seq_len + block_size - 1) // block_size
        self.device = torch.device(device)
        self.block_table = torch.zeros((max_seqs, self.max_blocks_per_seq), dtype=torch.int32, device=self.device)
        self.seq_lens = torch.zeros(max_seqs, dtype=torch.int32, device=self.device)
        self.reset()

    # ---- sequences (host side) ----
    def reset(self):
        self._free: List[int] = list(range(self.num_blocks - 1, -1, -1))
        self._owned: List[List[int]] = [[] for _ in range(self.max_seqs)]
        self._dropped = [0] * self.max_seqs              # leading pages given back because no layer can see them
        self._host_lens = [0] * self.max_seqs
        self._idle: List[int] = list(range(self.max_seqs - 1, -1, -1))
        self.seq_lens.zero_()

    def acquire(self) -> int:
        """A sequence number nobody uses."""
        if not self._idle:
            raise RuntimeError("all cache sequences are in use")
        return self._idle.pop()

    def release(self, seq: int):
        """Give back a sequence obtained from :meth:`acquire` with everything it holds."""
        self.free(seq)
        self._idle.append(seq)

    def length(self, seq: int) -> int:
        return self._host_lens[seq]

    def advance(self, seq: int, new_len: int):
        """Host-side record of a sequence's length (``seq_lens`` is advanced by the step itself)."""
        self._host_lens[seq] = new_len

    # ---- pages (host side) ----
    @property
    def free_blocks(self) -> int:
        return len(self._free)

    def reserve(self, seq: int, new_len: int):
        """Make sure sequence ``seq`` owns enough pages for ``new_len`` tokens."""
        self.reserve_many([(seq, new_len)])

    def reserve_all(self, num_seqs: int, new_len: int):
        """:meth:`reserve` for sequences 0..num_seqs-1."""
        self.reserve_many([(s, new_len) for s in range(num_seqs)])

    def reserve_many(self, wanted: Iterable[Tuple[int, int]]):
        """:meth:`reserve` for several (sequence, length) pairs with one table update; all or nothing."""
        plan = []
        total = 0
        for seq, new_len in wanted:
            need = (new_len + self.block_size - 1) // self.block_size
            if need > self.max_blocks_per_seq:
                raise RuntimeError(f"sequence {seq} exceeds the cache's max_seq_len")
            have = self._dropped[seq] + len(self._owned[seq])
            if need > have:
                plan.append((seq, have, need))
                total += need - have
        if total > len(self._free):
            raise RuntimeError("KV cache is out of blocks")
        rows, cols, blocks = [], [], []
        for seq, have, need in plan:
            for page in range(have, need):
                blk = self._free.pop()
                self._owned[seq].append(blk)
                rows.append(seq)
                cols.append(page)
                blocks.append(blk)
        if rows:
            index = torch.tensor([rows, cols, blocks], dtype=torch.int64).to(self.device)
            self.block_table[index[0], index[1]] = index[2].to(torch.int32)

    def drop_before(self, seq: int, position: int):
        """Give back the pages of ``seq`` that end at or before ``position`` (no later token sees them)."""
        n = position // self.block_size - self._dropped[seq]
        if n > 0:
            self._free.extend(reversed(self._owned[seq][:n]))
            del self._owned[seq][:n]
            self._dropped[seq] += n

    def free(self, seq: int):
        self._free.extend(reversed(self._owned[seq]))
        self._owned[seq] = []
        self._dropped[seq] = 0
        self._host_lens[seq] = 0
        self.seq_lens[seq] = 0

    # ---- slot mapping ----
    def slots_for(self, seq_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """Flat cache slots (block * block_size + offset) for tokens at ``positions`` of ``seq_ids``."""
        page = (positions // self.block_size).long()
        blk = self.block_table[seq_ids.long(), page].long()
        return blk * self.block_size + (positions % self.block_size).long()

    def visible_from(self, position: int) -> int:
        """First token that any layer reads for a token at ``position``."""
        return 0


class BlockKVCache(PagedCache):
    def __init__(self, num_layers: int, kv_heads: int, head_dim: int, num_blocks: int, block_size: int = 16,
                 max_seqs: int = 128, max_seq_len: int = 1024, dtype=torch.bfloat16, device="cuda"):
        super().__init__(num_blocks, block_size, max_seqs, max_seq_len, device)
        self.num_layers, self.kv_heads, self.head_dim, self.dtype = num_layers, kv_heads, head_dim, dtype
        shape = (num_blocks, block_size, kv_heads, head_dim)
        self.k = [torch.zeros(shape, dtype=dtype, device=self.device) for _ in range(num_layers)]
        self.v = [torch.zeros(shape, dtype=dtype, device=self.device) for _ in range(num_layers)]

    def bytes_per_token(self) -> int:
        return 2 * self.num_layers * self.kv_heads * self.head_dim * torch.empty((), dtype=self.dtype).element_size()


class LayerCache(PagedCache):
    """``rows[run][name]``: [num_blocks * block_size, width]; ``states[run][name]``: [max_seqs, ...], one per sequence, as
    the run's :class:`~ironcore_b200.layers.mixer.CacheSpec` in ``specs`` declares them. Pages that no layer reads any more
    go back to the free list while a sequence is still running. A state belongs to whoever holds the sequence number;
    mixers take it for zeros at position 0."""

    def __init__(self, specs: Sequence, *, max_seqs: int, max_seq_len: int, block_size: int = 16,
                 num_blocks: Optional[int] = None, dtype=torch.bfloat16, device="cuda"):
        if num_blocks is None:
            num_blocks = max_seqs * ((max_seq_len + block_size - 1) // block_size)
        super().__init__(num_blocks, block_size, max_seqs, max_seq_len, device)
        self.specs, self.dtype = list(specs), dtype
        self.rows: List[Dict[str, torch.Tensor]] = [
            {name: torch.zeros((num_blocks * block_size, w), dtype=dtype, device=self.device) for name, w in s.rows.items()}
            for s in self.specs]
        self.states: List[Dict[str, torch.Tensor]] = [
            {name: torch.zeros((max_seqs, *shape), dtype=dt or dtype, device=self.device)
             for name, (shape, dt) in s.states.items()} for s in self.specs]

    def visible_from(self, position: int) -> int:
        reach = [lo for lo in (s.visible_from(position) for s in self.specs) if lo is not None]
        return min(reach) if reach else position

    def bytes_per_token(self) -> int:
        return sum(sum(s.rows.values()) for s in self.specs) * torch.empty((), dtype=self.dtype).element_size()

    def bytes_per_sequence(self) -> int:
        """Fixed-size states of one sequence."""
        return sum(t[0].numel() * t.element_size() for run in self.states for t in run.values())
