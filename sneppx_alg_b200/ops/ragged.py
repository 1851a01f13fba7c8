"""Ragged batches: portions of several sequences packed row after row, with the index arrays that the kernels of the
hybrid decoders read. All arrays of a batch travel to the device in one copy."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import numpy as np
import torch

from . import _lib


RECUR_CHUNK = 16     # tokens per chunk of the recurrence kernels


@dataclass(frozen=True)
class Chunk:
    """Position p sees the positions of its own chunk of ``size`` up to itself."""

    size: int
    pool = 0

    def first(self, pos: int) -> int:
        """Earliest position whose key a token at ``pos`` needs."""
        return pos // self.size * self.size

    @property
    def span(self) -> int:
        """Most positions between ``first(pos)`` and ``pos``, both included."""
        return self.size


@dataclass(frozen=True)
class PooledWindow:
    """Position p sees the last ``size`` positions one by one and, before them, whole blocks of ``pool`` positions as one
    averaged key and value each. Keys of an unfinished block are kept until its average is formed."""

    size: int
    pool: int

    def first(self, pos: int) -> int:
        return max(0, min(pos - self.size + 1, pos // self.pool * self.pool))

    @property
    def span(self) -> int:
        return max(self.size, self.pool)

    def blocks_seen(self, pos: int) -> int:
        """Averaged blocks that a token at ``pos`` sees."""
        return max(0, pos - self.size + 1) // self.pool


def as_mask(m):
    """A chunk length stands for its ``Chunk``."""
    return Chunk(m) if isinstance(m, int) else m


@dataclass
class ChunkView:
    """Packed keys and values of one mask: per sequence the averaged blocks (masks that pool: all complete ones, those that
    this portion completes last), then the earlier positions that the portion's first tokens still see, then the portion.
    Rows of earlier work are copied from the cache: ``gather_entry`` -> ``gather_row``."""

    rows: int
    kv_row: torch.Tensor        # [T] packed row of each token
    kv_base: torch.Tensor       # [n] row that position 0 of the sequence would have
    gather_entry: torch.Tensor
    gather_row: torch.Tensor
    tiles: Optional[torch.Tensor] = None   # [n_tiles, 2]: portion, first row of the portion in the tile
    n_tiles: int = 0
    pool_base: Optional[torch.Tensor] = None     # [n] row of each sequence's first averaged block
    pool_src: Optional[torch.Tensor] = None      # blocks completed by this batch: row of the first token,
    pool_row: Optional[torch.Tensor] = None      # row of the average,
    pool_entry: Optional[torch.Tensor] = None    # cache entry of the average
    n_pool: int = 0


class RaggedBatch:
    """``decode``: one token per sequence; keys are then read from the block pool through ``block_table``."""

    def __init__(self):
        self.n = self.T = 0
        self.decode = False
        self.views: Dict[int, ChunkView] = {}
        self.want = None

    def struct(self) -> "_lib.SxRagged":
        r = _lib.SxRagged()
        r.cu, r.pos0, r.slot = self.cu.data_ptr(), self.pos0.data_ptr(), self.slot.data_ptr()
        r.tok_seq, r.tok_pos, r.n = self.tok_seq.data_ptr(), self.tok_pos.data_ptr(), self.n
        return r

    def chunks(self) -> "_lib.SxChunks":
        c = _lib.SxChunks()
        c.seq, c.start, c.first, c.n = self.chunk_seq.data_ptr(), self.chunk_start.data_ptr(), self.chunk_first.data_ptr(), self.n_chunks
        return c

    @classmethod
    def prompt(cls, device, tokens: List[List[int]], pos0: List[int], slots: List[int], entries: List[List[int]],
               earlier: Dict[object, List[List[int]]], want: List[int], tile_rows: int = 128, averages=None,
               segment_rows: int = 512) -> "RaggedBatch":
        """``earlier[mask][i]``: cache entries of the positions before sequence i's portion that its first token still
        needs (a chunk length may stand for its mask). ``averages[mask][i]``: for masks that pool, the cache entries of the
        averaged blocks complete before the portion and of those that it completes. ``want``: rows whose logits are asked
        for. ``segment_rows``: length of the segments that a scan may run side by side."""
        b = cls()
        b.n, b.T = len(tokens), sum(len(t) for t in tokens)
        lens = np.array([len(t) for t in tokens], dtype=np.int32)
        cu = np.zeros(b.n + 1, dtype=np.int32)
        np.cumsum(lens, out=cu[1:])
        p0 = np.array(pos0, dtype=np.int32)
        seq = np.repeat(np.arange(b.n, dtype=np.int32), lens)
        local = np.arange(b.T, dtype=np.int32) - cu[seq]
        parts = [np.concatenate([np.asarray(t, dtype=np.int32) for t in tokens]), cu, p0, np.array(slots, dtype=np.int32), seq,
                 p0[seq] + local, np.concatenate([np.asarray(e, dtype=np.int32) for e in entries]),
                 np.asarray(want, dtype=np.int32)]
        tiles = np.array([(i, r) for i in range(b.n) for r in range(0, int(lens[i]), tile_rows)], dtype=np.int32)
        parts.append(tiles.reshape(-1))
        per = (lens + RECUR_CHUNK - 1) // RECUR_CHUNK
        first = np.zeros(b.n + 1, dtype=np.int32)
        np.cumsum(per, out=first[1:])
        chunk_seq = np.repeat(np.arange(b.n, dtype=np.int32), per)
        parts += [chunk_seq, (np.arange(first[-1], dtype=np.int32) - first[chunk_seq]) * RECUR_CHUNK, first]
        b.n_chunks = int(first[-1])
        per = (lens + segment_rows - 1) // segment_rows
        seg_first = np.zeros(b.n + 1, dtype=np.int32)
        np.cumsum(per, out=seg_first[1:])
        parts += [np.repeat(np.arange(b.n, dtype=np.int32), per), seg_first]
        b.n_segments, b.segment_rows = int(seg_first[-1]), segment_rows
        views, none = [], np.zeros(0, np.int32)
        cat = lambda xs: np.concatenate([np.asarray(x, dtype=np.int32) for x in xs]) if xs else none  # noqa: E731
        for key in earlier:
            mask = as_mask(key)
            carry = np.array([len(e) for e in earlier[key]], dtype=np.int32)
            done, new = zip(*averages[key]) if mask.pool else ([()] * b.n, [()] * b.n)
            n_done, n_new = (np.array([len(e) for e in x], dtype=np.int32) for x in (done, new))
            start = np.zeros(b.n + 1, dtype=np.int32)
            np.cumsum(n_done + n_new + carry + lens, out=start[1:])
            kept = start[:-1] + n_done + n_new                      # packed row of the first earlier position
            row0 = kept + carry                                     # packed row of the portion's first token
            parts += [row0[seq] + local, row0 - p0, cat([e for i in range(b.n) for e in (done[i], earlier[key][i])]),
                      cat([r for i in range(b.n) for r in (start[i] + np.arange(n_done[i]), kept[i] + np.arange(carry[i]))])]
            if mask.pool:
                first_new = p0 // mask.pool
                assert (n_done == first_new).all() and (n_new == (p0 + lens) // mask.pool - first_new).all()
                parts += [start[:-1],
                          cat([row0[i] - p0[i] + (first_new[i] + np.arange(n_new[i])) * mask.pool for i in range(b.n)]),
                          cat([start[i] + n_done[i] + np.arange(n_new[i]) for i in range(b.n)]), cat(list(new))]
            views.append((key, int(start[-1]), int(n_new.sum())))
        dev = cls._upload(device, parts)
        b.ids, b.cu, b.pos0, b.slot, b.tok_seq, b.tok_pos, b.entry, b.want, tl, b.chunk_seq, b.chunk_start, b.chunk_first = dev[:12]
        b.seg_seq, b.seg_first = dev[12:14]
        at = 14
        for key, rows, n_pool in views:
            v = b.views[key] = ChunkView(rows, *dev[at: at + 4], tl, len(tiles))
            at += 4
            if as_mask(key).pool:
                v.pool_base, v.pool_src, v.pool_row, v.pool_entry = dev[at: at + 4]
                v.n_pool = n_pool
                at += 4
        if len(want) == b.T:
            b.want = None
        b.n_want = len(want)
        return b

    @staticmethod
    def _upload(device, parts):
        offs, n = [], 0
        for p in parts:
            offs.append(n)
            n += (len(p) + 3) // 4 * 4          # every array starts 16-byte aligned
        host = torch.zeros(max(n, 1), dtype=torch.int32)
        if torch.device(device).type == "cuda":
            host = host.pin_memory()
        hv = host.numpy()
        for p, o in zip(parts, offs):
            hv[o:o + len(p)] = p
        buf = host.to(device, non_blocking=True)
        return [buf[o:o + len(p)] for p, o in zip(parts, offs)]

    @classmethod
    def decode_layout(cls, n: int, width: int, pools=(), pool_width: int = 0):
        """Offsets of the decode arrays in one int32 buffer of ``length`` entries: (slices, length). ``pools``: block
        lengths of the masks that pool, each with a table of ``pool_width`` cache blocks of averages."""
        names = [("ids", n), ("pos0", n), ("slot", n), ("entry", n), ("block_base", n), ("cu", n + 1), ("tok_seq", n),
                 ("block_table", n * width)]
        for p in pools:
            names += [(("pool_entry", p), n), (("pool_table", p), n * pool_width)]
        out, o = {}, 0
        for name, k in names:
            out[name] = slice(o, o + k)
            o += (k + 3) // 4 * 4
        return out, max(o, 1)

    @classmethod
    def decode_views(cls, buf: torch.Tensor, n: int, width: int, pools=(), pool_width: int = 0) -> "RaggedBatch":
        """Decode batch over a device buffer laid out by ``decode_layout``."""
        lay, _ = cls.decode_layout(n, width, pools, pool_width)
        b = cls()
        b.n = b.T = b.n_want = n
        b.decode = True
        b.pool_entry, b.pool_table, b.pool_width = {}, {}, pool_width
        for name, sl in lay.items():
            if isinstance(name, tuple):
                getattr(b, name[0])[name[1]] = buf[sl]
            else:
                setattr(b, name, buf[sl])
        b.tok_pos, b.table_width = b.pos0, width
        return b

    @classmethod
    def fill_decode(cls, hv, n: int, width: int, ids, pos, slots, entries, tables, bases, pools=None, pool_width: int = 0) -> None:
        """Writes the host side of a decode buffer; rows past the sequences given are padding (slot and entry -1).
        ``pools[length]``: (cache entry of the average that each token completes or -1, tables of averages)."""
        pools = pools or {}
        lay, _ = cls.decode_layout(n, width, tuple(pools), pool_width)
        k = len(ids)
        hv[:] = 0
        hv[lay["slot"]] = -1
        hv[lay["entry"]] = -1
        for name, vals in (("ids", ids), ("pos0", pos), ("slot", slots), ("entry", entries), ("block_base", bases)):
            hv[lay[name].start: lay[name].start + k] = vals
        hv[lay["cu"]] = np.arange(n + 1, dtype=np.int32)
        hv[lay["tok_seq"]] = np.arange(n, dtype=np.int32)
        grids = [("block_table", width, tables)] if width else []
        for p, (done, tabs) in pools.items():
            e = lay["pool_entry", p]
            hv[e] = -1
            hv[e.start: e.start + k] = done
            grids.append((("pool_table", p), pool_width, tabs))
        for name, w, rows in grids:
            bt = hv[lay[name]].reshape(n, w)
            for i, t in enumerate(rows):
                bt[i, :len(t)] = t
