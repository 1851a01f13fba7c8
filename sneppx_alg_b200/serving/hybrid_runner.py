"""Runs a hybrid decoder (recurrent layers and attention of bounded reach, ``models/hybrid.py``) for the engine: prompts of
any lengths packed into one ragged batch, portions of a prompt from the state earlier portions left, and decode steps that
replay one CUDA graph per batch bucket. A sequence's memory is one state slot plus the cache blocks of the positions that
its next token needs and of its averaged blocks (``serving.kv_cache.HybridCache``)."""
from __future__ import annotations

from typing import List, Sequence, Tuple

import torch

from ..ops.gemm import static_weights
from ..ops.ragged import RaggedBatch
from .kv_cache import HybridCache


class HybridRunner:
    ragged_prefill = True       # prefill_batch takes prompts of different lengths
    max_portion = 16384         # prompt tokens of one sequence per pass (bounds the activations of very long prompts)

    def __init__(self, model, cache: HybridCache):
        self.model, self.cache = model, cache
        self._graphs = None

    @property
    def device(self):
        return self.model.embed.device

    # ------------------------------------------------------------------ one step
    @torch.no_grad()
    def step(self, entries: Sequence[Tuple[int, List[int], Sequence[int]]]):
        """``entries``: (sequence, its next tokens, places among them whose logits are wanted). All entries run as one
        batch; returns the wanted logits in order, [wanted, vocab] fp32."""
        if all(len(toks) == 1 for _, toks, _ in entries):
            logits = self.decode([s for s, _, _ in entries], [t[0] for _, t, _ in entries])
            keep = [i for i, (_, _, want) in enumerate(entries) for _ in want]
            return logits if keep == list(range(len(entries))) else logits[keep]
        cache = self.cache
        pos0 = [cache.lens[s] for s, _, _ in entries]
        earlier = {m: [cache.entries(s, r.first(p), p) for (s, _, _), p in zip(entries, pos0)]
                   for m, r in zip(cache.masks, cache.rules)}
        slots = [cache.reserve(s, len(t)) for s, t, _ in entries]
        averages = {m: [(cache.average_entries(s, r.pool, 0, p // r.pool),
                         cache.average_entries(s, r.pool, p // r.pool, (p + len(t)) // r.pool)) for (s, t, _), p in zip(entries, pos0)]
                    for m, r in zip(cache.masks, cache.rules) if r.pool}
        want, row = [], 0
        for _, toks, w in entries:
            want += [row + (i if i >= 0 else len(toks) + i) for i in w]
            row += len(toks)
        batch = RaggedBatch.prompt(self.device, [t for _, t, _ in entries], pos0, [cache.slots[s] for s, _, _ in entries], slots,
                                   earlier, want, averages=averages)
        return self.model.step(batch, cache)

    def prefill(self, seq_id: int, tokens: List[int], start: int):
        """Prompt tokens [start, len) of one sequence, long ones in portions; logits of the last position."""
        while len(tokens) - start > self.max_portion:
            self.step([(seq_id, tokens[start: start + self.max_portion], ())])
            start += self.max_portion
        return self.step([(seq_id, tokens[start:], (-1,))])

    def prefill_batch(self, seq_ids: List[int], prompts: List[List[int]]):
        """Whole prompts in one pass; logits of the last position of each, [n, V]."""
        return self.step([(s, p, (-1,)) for s, p in zip(seq_ids, prompts)])

    # ------------------------------------------------------------------ decode
    def enable_graphs(self, max_batch: int, max_len: int = 0):
        """Capture the decode step per batch bucket (1, 2, 4, .. max_batch). All inputs of a step sit in one int32 buffer
        filled by one host -> device copy; its size depends on what the masks reach, not on how long sequences get, except
        for the tables of averaged blocks, whose width is bucketed too (a graph is captured when one is outgrown)."""
        if self.device.type != "cuda":
            return
        self._buckets, b = [], 1
        while b < max_batch:
            self._buckets.append(b)
            b *= 2
        self._buckets.append(max_batch)
        self._graphs = {}

    def _body(self, batch):
        with static_weights():
            return self.model.step(batch, self.cache)

    def _graph_for(self, n, pool_width):
        g = self._graphs.get((n, pool_width))
        if g is not None:
            return g
        width, pools = self.cache.table_width, self.cache.pools
        _, length = RaggedBatch.decode_layout(n, width, pools, pool_width)
        host = torch.zeros(length, dtype=torch.int32).pin_memory()
        hv = host.numpy()
        # padding only: the warm-up writes no state
        RaggedBatch.fill_decode(hv, n, width, [], [], [], [], [], [], {p: ([], []) for p in pools}, pool_width)
        buf = host.to(self.device)
        batch = RaggedBatch.decode_views(buf, n, width, pools, pool_width)
        side = torch.cuda.Stream(device=self.device)
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            for _ in range(2):
                self._body(batch)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, capture_error_mode="thread_local"):   # other threads (HTTP handlers) may call CUDA
            out = self._body(batch)
        g = self._graphs[n, pool_width] = dict(graph=graph, host=host, hv=hv, buf=buf, out=out)
        return g

    def _pool_width(self, seq_ids) -> int:
        """Blocks of averages per table: the longest table, up to a power of two."""
        most = max((len(t[s]) for t in self.cache.averages.values() for s in seq_ids), default=0)
        return max(4, 1 << (most - 1).bit_length()) if self.cache.pools else 0

    @torch.no_grad()
    def decode(self, seq_ids: List[int], last_tokens: List[int]):
        """One token for each sequence; logits [B, V]."""
        cache, B, width = self.cache, len(seq_ids), self.cache.table_width
        pos = [cache.lens[s] for s in seq_ids]
        entries = [cache.reserve(s, 1)[0] for s in seq_ids]
        pools = {p: ([cache.average_entries(s, p, q // p, q // p + 1)[0] if (q + 1) % p == 0 else -1 for s, q in zip(seq_ids, pos)],
                     [cache.averages[p][s] for s in seq_ids]) for p in cache.pools}
        pw = self._pool_width(seq_ids)
        args = (last_tokens, pos, [cache.slots[s] for s in seq_ids], entries, [cache.tables[s] for s in seq_ids],
                [cache.base[s] for s in seq_ids], pools, pw)
        if self._graphs is not None and B <= self._buckets[-1]:
            n = next(b for b in self._buckets if b >= B)
            g = self._graph_for(n, pw)
            torch.cuda.current_stream().synchronize()      # the previous step's copy has left the pinned buffer
            RaggedBatch.fill_decode(g["hv"], n, width, *args)
            g["buf"].copy_(g["host"], non_blocking=True)
            g["graph"].replay()
            return g["out"][:B].clone()
        _, length = RaggedBatch.decode_layout(B, width, cache.pools, pw)
        host = torch.zeros(length, dtype=torch.int32)
        RaggedBatch.fill_decode(host.numpy(), B, width, *args)
        return self.model.step(RaggedBatch.decode_views(host.to(self.device), B, width, cache.pools, pw), cache)
