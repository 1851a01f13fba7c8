"""Paged KV cache: a pool of fixed-size blocks with reference counts and copy-on-write forks, per-sequence block
tables and a prefix cache keyed by hashed token chunks. Same concepts as the reference's NumPy implementation
(interface_bindings/paged_attention.py:43-427: ``KVBlockPool``, ``PagedKVCache``, ``PrefixCache``), with the K/V
storage living on the GPU in the layout the decode kernel reads ([blocks, block_size, Hkv, D] per layer)."""
from __future__ import annotations

import hashlib
from collections import OrderedDict
from typing import Dict, List, Optional, Tuple

import numpy as np
import torch

from ..ops.ragged import as_mask


class KVBlockPool:
    """Block id allocator with refcounts (shared prefixes) and copy-on-write."""

    def __init__(self, num_blocks: int):
        self.num_blocks = num_blocks
        self.free: List[int] = list(range(num_blocks - 1, -1, -1))
        self.ref = [0] * num_blocks
        self.reclaim = None     # callable(n) -> blocks freed; set by the cache that owns prefix entries

    def allocate(self) -> int:
        if not self.free and self.reclaim is not None:
            self.reclaim(1)
        if not self.free:
            raise MemoryError("KV block pool exhausted")
        b = self.free.pop()
        self.ref[b] = 1
        return b

    def share(self, b: int) -> int:
        self.ref[b] += 1
        return b

    def release(self, b: int) -> None:
        self.ref[b] -= 1
        if self.ref[b] == 0:
            self.free.append(b)
        elif self.ref[b] < 0:
            raise RuntimeError(f"double free of KV block {b}")

    @property
    def num_free(self) -> int:
        return len(self.free)


class PrefixCache:
    """Maps a hash of (all tokens up to the end of a full block) to the block that holds their K/V. Entries are
    kept in least-recently-used order; the cache never pins more than ``max_entries`` blocks (by default half of
    the pool) and gives blocks back on demand (``evict``) when the pool runs short."""

    def __init__(self, pool: KVBlockPool, block_size: int, max_entries: Optional[int] = None):
        if max_entries is None:
            max_entries = max(1, min(4096, pool.num_blocks // 2))
        self.pool, self.block_size, self.max_entries = pool, block_size, max_entries
        self.table: "OrderedDict[bytes, int]" = OrderedDict()

    @staticmethod
    def _hash(prev: bytes, chunk) -> bytes:
        h = hashlib.blake2b(digest_size=16)
        h.update(prev)
        h.update(bytes(str(list(chunk)), "ascii"))
        return h.digest()

    def match(self, tokens) -> Tuple[List[int], List[bytes]]:
        """Longest cached run of full blocks; returns (block ids with a new reference each, their keys)."""
        blocks, keys, prev = [], [], b""
        for i in range(0, len(tokens) - len(tokens) % self.block_size, self.block_size):
            key = self._hash(prev, tokens[i: i + self.block_size])
            b = self.table.get(key)
            if b is None:
                break
            self.table.move_to_end(key)
            blocks.append(self.pool.share(b))
            keys.append(key)
            prev = key
        return blocks, keys

    def insert(self, tokens, block_ids) -> None:
        prev = b""
        for j, i in enumerate(range(0, len(tokens) - len(tokens) % self.block_size, self.block_size)):
            key = self._hash(prev, tokens[i: i + self.block_size])
            if key in self.table:
                self.table.move_to_end(key)
            elif j < len(block_ids):
                if len(self.table) >= self.max_entries:
                    _, old = self.table.popitem(last=False)
                    self.pool.release(old)
                self.table[key] = self.pool.share(block_ids[j])
            prev = key

    def evictable(self) -> int:
        """Blocks that only the cache still holds."""
        return sum(1 for b in self.table.values() if self.pool.ref[b] == 1)

    def evict(self, n: int) -> int:
        """Give back up to ``n`` blocks that no running sequence shares, least recently used first."""
        freed = 0
        for key in list(self.table):
            if freed >= n:
                break
            b = self.table[key]
            if self.pool.ref[b] == 1:
                del self.table[key]
                self.pool.release(b)
                freed += 1
        return freed


class PagedKVCache:
    """``layer_shapes`` (one ``(kv heads, key size, value size)`` per layer) replaces ``num_kv_heads`` / ``head_dim`` for
    models whose layers differ or whose keys and values have different sizes."""

    def __init__(self, num_layers, num_blocks, block_size, num_kv_heads=0, head_dim=0, dtype=torch.bfloat16, device="cuda",
                 enable_prefix_cache=True, layer_shapes=None):
        self.block_size, self.num_layers = block_size, num_layers
        self.pool = KVBlockPool(num_blocks)
        shapes = layer_shapes if layer_shapes is not None else [(num_kv_heads, head_dim, head_dim)] * num_layers
        self.k = [torch.zeros(num_blocks, block_size, h, dk, dtype=dtype, device=device) for h, dk, _ in shapes]
        self.v = [torch.zeros(num_blocks, block_size, h, dv, dtype=dtype, device=device) for h, _, dv in shapes]
        self.tables: Dict[int, List[int]] = {}
        self.lens: Dict[int, int] = {}
        self.prefix = PrefixCache(self.pool, block_size) if enable_prefix_cache else None
        if self.prefix is not None:
            self.pool.reclaim = self.prefix.evict

    def blocks_for(self, n_tokens: int) -> int:
        """Most blocks a sequence of ``n_tokens`` holds at any time."""
        return (n_tokens + self.block_size - 1) // self.block_size

    def blocks_held(self, seq_id: int) -> int:
        """Blocks in the tables of a sequence."""
        return len(self.tables.get(seq_id, ()))

    def available_blocks(self) -> int:
        """Free blocks plus those the prefix cache would give back."""
        return self.pool.num_free + (self.prefix.evictable() if self.prefix is not None else 0)

    def make_room(self, n: int) -> bool:
        """Evict prefix entries until ``n`` blocks are free; False if that is not possible."""
        short = n - self.pool.num_free
        if short > 0 and self.prefix is not None:
            self.prefix.evict(short)
        return self.pool.num_free >= n

    # ---- sequences
    def add_sequence(self, seq_id: int, tokens=None) -> int:
        """Registers a sequence; returns how many prompt tokens are already covered by cached prefix blocks."""
        blocks = []
        if self.prefix is not None and tokens is not None:
            blocks, _ = self.prefix.match(tokens)
            # always leave at least one token to compute so that the model produces logits
            while blocks and len(blocks) * self.block_size >= len(tokens):
                self.pool.release(blocks.pop())
        self.tables[seq_id] = blocks
        self.lens[seq_id] = len(blocks) * self.block_size
        return self.lens[seq_id]

    def reserve(self, seq_id: int, n_new: int) -> List[int]:
        """Slots (block * block_size + offset) for the next ``n_new`` tokens, allocating / copying blocks as needed."""
        table, n = self.tables[seq_id], self.lens[seq_id]
        slots = []
        for i in range(n, n + n_new):
            bi, off = divmod(i, self.block_size)
            if bi == len(table):
                table.append(self.pool.allocate())
            elif self.pool.ref[table[bi]] > 1:      # shared block about to be written: copy on write
                new = self.pool.allocate()
                for l in range(self.num_layers):
                    self.k[l][new].copy_(self.k[l][table[bi]])
                    self.v[l][new].copy_(self.v[l][table[bi]])
                self.pool.release(table[bi])
                table[bi] = new
            slots.append(table[bi] * self.block_size + off)
        self.lens[seq_id] = n + n_new
        return slots

    def fork(self, src_id: int, dst_id: int) -> None:
        self.tables[dst_id] = [self.pool.share(b) for b in self.tables[src_id]]
        self.lens[dst_id] = self.lens[src_id]

    def free_sequence(self, seq_id: int, tokens=None) -> None:
        table = self.tables.pop(seq_id, [])
        n = self.lens.pop(seq_id, 0)
        if self.prefix is not None and tokens is not None:
            self.prefix.insert(tokens[:n], table)
        for b in table:
            self.pool.release(b)

    def block_table_tensor(self, seq_ids, device=None) -> Tuple[torch.Tensor, torch.Tensor]:
        mb = max(1, max(len(self.tables[s]) for s in seq_ids))
        bt = torch.zeros(len(seq_ids), mb, dtype=torch.int32)
        for i, s in enumerate(seq_ids):
            t = self.tables[s]
            bt[i, : len(t)] = torch.tensor(t, dtype=torch.int32)
        lens = torch.tensor([self.lens[s] for s in seq_ids], dtype=torch.int32)
        dev = device or self.k[0].device
        return bt.to(dev), lens.to(dev)

    def gather(self, layer: int, seq_id: int, n: Optional[int] = None):
        """Contiguous [n, Hkv, D] K and V of a sequence (used when a prefill chunk attends to cached tokens)."""
        n = self.lens[seq_id] if n is None else n
        blocks = torch.tensor(self.tables[seq_id][: (n + self.block_size - 1) // self.block_size], dtype=torch.long,
                              device=self.k[layer].device)
        k = self.k[layer][blocks].reshape(-1, *self.k[layer].shape[2:])[:n]
        v = self.v[layer][blocks].reshape(-1, *self.v[layer].shape[2:])[:n]
        return k, v


class ChunkedKVCache(PagedKVCache):
    """Paged cache of layers in which a position sees a bounded stretch of positions (``masks``: the masks that occur, see
    ``ops.ragged``; an integer stands for chunks of that length). Positions behind the last needed one are never stored, and
    blocks that fall behind it go back to the pool. Block tables start at block ``base[seq]``. Masks that average older blocks
    of positions keep one entry per average; these live in blocks of the same pool, listed per block length in ``averages``,
    and stay as long as the sequence. Without them a sequence holds a bounded number of blocks however long it grows."""

    def __init__(self, layer_shapes, masks, num_blocks, block_size, dtype=torch.bfloat16, device="cuda"):
        super().__init__(len(layer_shapes), num_blocks, block_size, dtype=dtype, device=device, enable_prefix_cache=False,
                         layer_shapes=layer_shapes)
        self.masks = list(dict.fromkeys(masks))
        self.rules = [as_mask(m) for m in self.masks]
        self.pools = tuple(sorted({m.pool for m in self.rules if m.pool}))
        self.base: Dict[int, int] = {}
        self.averages: Dict[int, Dict[int, List[int]]] = {p: {} for p in self.pools}

    @property
    def sizes(self) -> List[int]:
        """Most positions that each mask reaches back, ascending."""
        return sorted(m.span for m in self.rules)

    @property
    def table_width(self) -> int:
        """Blocks that the stored positions of one sequence can touch."""
        return (self.sizes[-1] + self.block_size - 2) // self.block_size + 1 if self.rules else 0

    def average_blocks(self, n_tokens: int, pool: int) -> int:
        """Cache blocks that hold the averages of ``n_tokens`` tokens in blocks of ``pool``."""
        return (n_tokens // pool + self.block_size - 1) // self.block_size

    def blocks_for(self, n_tokens: int) -> int:
        return min(super().blocks_for(n_tokens), self.table_width) + sum(self.average_blocks(n_tokens, p) for p in self.pools)

    def blocks_held(self, seq_id: int) -> int:
        return super().blocks_held(seq_id) + sum(len(t.get(seq_id, ())) for t in self.averages.values())

    def first_visible(self, pos: int) -> int:
        """Earliest position that any layer still needs at ``pos``."""
        return min(m.first(pos) for m in self.rules) if self.rules else pos + 1

    def add_sequence(self, seq_id: int, tokens=None) -> int:
        self.tables[seq_id], self.lens[seq_id], self.base[seq_id] = [], 0, 0
        for t in self.averages.values():
            t[seq_id] = []
        return 0

    def reserve(self, seq_id: int, n_new: int) -> List[int]:
        """Cache entries of the next ``n_new`` tokens; -1 for tokens that no later token needs. Also makes room for the
        averages that these tokens complete."""
        n, table, base = self.lens[seq_id], self.tables[seq_id], self.base[seq_id]
        end = n + n_new
        keep = self.first_visible(end - 1)
        new_base = keep // self.block_size
        while table and base < new_base:
            self.pool.release(table.pop(0))
            base += 1
        if not table:
            base = max(base, new_base)
        first = max(n, keep)
        while first < end and base + len(table) <= (end - 1) // self.block_size:   # first == end: no layer keeps keys
            table.append(self.pool.allocate())
        for p, t in self.averages.items():
            while len(t[seq_id]) < self.average_blocks(end, p):
                t[seq_id].append(self.pool.allocate())
        self.base[seq_id], self.lens[seq_id] = base, end
        return [-1] * (first - n) + self.entries(seq_id, first, end)

    def average_entries(self, seq_id: int, pool: int, lo: int, hi: int) -> List[int]:
        """Entries of the averages of blocks [lo, hi) of ``pool`` positions."""
        table, bs = self.averages[pool][seq_id], self.block_size
        i = np.arange(lo, hi)
        return (np.asarray(table, dtype=np.int64)[i // bs] * bs + i % bs).tolist() if hi > lo else []

    def entries(self, seq_id: int, lo: int, hi: int) -> List[int]:
        """Entries of the stored positions [lo, hi)."""
        table, base, bs = self.tables[seq_id], self.base[seq_id], self.block_size
        if hi - lo == 1:
            return [table[lo // bs - base] * bs + lo % bs]
        p = np.arange(lo, hi)
        return (np.asarray(table, dtype=np.int64)[p // bs - base] * bs + p % bs).tolist() if hi > lo else []

    def fork(self, src_id: int, dst_id: int) -> None:
        raise NotImplementedError("a chunked cache does not share blocks between sequences")

    def free_sequence(self, seq_id: int, tokens=None) -> None:
        self.base.pop(seq_id, None)
        for t in self.averages.values():
            for b in t.pop(seq_id, ()):
                self.pool.release(b)
        super().free_sequence(seq_id)


class HybridCache(ChunkedKVCache):
    """Memory of models that mix recurrent layers and attention of bounded reach: the block pool of the attention layers and one
    slot of fixed-size state per live sequence (``state_spec``: per layer, name -> (shape, dtype) of one slot). A slot is
    never cleared: the kernels start a sequence's first portion from an empty state whatever the slot holds."""

    def __init__(self, kv_shapes, masks, state_spec, max_sequences, num_blocks, block_size=16, dtype=torch.bfloat16,
                 device="cuda"):
        super().__init__(kv_shapes, masks, num_blocks, block_size, dtype, device)
        self.free_slots = list(range(max_sequences - 1, -1, -1))
        self.slots: Dict[int, int] = {}
        self.state = [{k: torch.zeros(max_sequences, *shape, dtype=dt, device=device) for k, (shape, dt) in spec.items()}
                      for spec in state_spec]

    def add_sequence(self, seq_id: int, tokens=None) -> int:
        if not self.free_slots:
            raise MemoryError("no free state slot")
        self.slots[seq_id] = self.free_slots.pop()
        return super().add_sequence(seq_id, tokens)

    def free_sequence(self, seq_id: int, tokens=None) -> None:
        if seq_id in self.slots:
            self.free_slots.append(self.slots.pop(seq_id))
        super().free_sequence(seq_id)
