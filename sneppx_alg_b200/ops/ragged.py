"""Ragged batches: portions of several sequences packed row after row, with the index arrays that the kernels of the
hybrid decoders read. All arrays of a batch travel to the device in one copy."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import numpy as np
import torch

from . import _lib


RECUR_CHUNK = 16     # tokens per chunk of the recurrence kernels


@dataclass
class ChunkView:
    """Packed keys and values of one chunk length: rows of the portion, preceded by the rows of earlier positions that
    the portion's first tokens still see (copied from the cache: ``gather_entry`` -> ``gather_row``)."""

    rows: int
    kv_row: torch.Tensor        # [T] packed row of each token
    kv_base: torch.Tensor       # [n] row that position 0 of the sequence would have
    gather_entry: torch.Tensor
    gather_row: torch.Tensor
    tiles: Optional[torch.Tensor] = None   # [n_tiles, 2]: portion, first row of the portion in the tile
    n_tiles: int = 0


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
               earlier: Dict[int, List[List[int]]], want: List[int], tile_rows: int = 128) -> "RaggedBatch":
        """``earlier[size][i]``: cache entries of the positions before sequence i's portion that lie in the same chunk of
        that length. ``want``: rows whose logits are asked for."""
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
        sizes = sorted(earlier)
        rows = []
        for size in sizes:
            carry = np.array([len(e) for e in earlier[size]], dtype=np.int32)
            start = np.zeros(b.n + 1, dtype=np.int32)
            np.cumsum(carry + lens, out=start[1:])
            row0 = start[:-1] + carry                               # packed row of the portion's first token
            parts += [row0[seq] + local, row0 - p0,
                      np.concatenate([np.asarray(e, dtype=np.int32) for e in earlier[size]]) if carry.sum() else np.zeros(0, np.int32),
                      np.concatenate([start[i] + np.arange(carry[i], dtype=np.int32) for i in range(b.n)])]
            rows.append(int(start[-1]))
        dev = cls._upload(device, parts)
        b.ids, b.cu, b.pos0, b.slot, b.tok_seq, b.tok_pos, b.entry, b.want, tl, b.chunk_seq, b.chunk_start, b.chunk_first = dev[:12]
        for i, size in enumerate(sizes):
            r, base, ge, gr = dev[12 + 4 * i: 16 + 4 * i]
            b.views[size] = ChunkView(rows[i], r, base, ge, gr, tl, len(tiles))
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
    def decode_layout(cls, n: int, width: int):
        """Offsets of the decode arrays in one int32 buffer of ``length`` entries: (slices, length)."""
        names = [("ids", n), ("pos0", n), ("slot", n), ("entry", n), ("block_base", n), ("cu", n + 1), ("tok_seq", n),
                 ("block_table", n * width)]
        out, o = {}, 0
        for name, k in names:
            out[name] = slice(o, o + k)
            o += (k + 3) // 4 * 4
        return out, max(o, 1)

    @classmethod
    def decode_views(cls, buf: torch.Tensor, n: int, width: int) -> "RaggedBatch":
        """Decode batch over a device buffer laid out by ``decode_layout``."""
        lay, _ = cls.decode_layout(n, width)
        b = cls()
        b.n = b.T = b.n_want = n
        b.decode = True
        for name, sl in lay.items():
            setattr(b, name, buf[sl])
        b.tok_pos, b.table_width = b.pos0, width
        return b

    @classmethod
    def fill_decode(cls, hv, n: int, width: int, ids, pos, slots, entries, tables, bases) -> None:
        """Writes the host side of a decode buffer; rows past the sequences given are padding (slot and entry -1)."""
        lay, _ = cls.decode_layout(n, width)
        k = len(ids)
        hv[:] = 0
        hv[lay["slot"]] = -1
        hv[lay["entry"]] = -1
        for name, vals in (("ids", ids), ("pos0", pos), ("slot", slots), ("entry", entries), ("block_base", bases)):
            hv[lay[name].start: lay[name].start + k] = vals
        hv[lay["cu"]] = np.arange(n + 1, dtype=np.int32)
        hv[lay["tok_seq"]] = np.arange(n, dtype=np.int32)
        if width:
            bt = hv[lay["block_table"]].reshape(n, width)
            for i, t in enumerate(tables):
                bt[i, :len(t)] = t
