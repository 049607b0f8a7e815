"""Cache of the layer-list decoders, and the description of one batch of a step.

``StepCache`` gives every attention run 16-token pages (one page table for all runs) of keys and values, with head counts and sizes
of its own, or of latents, and every recurrent run a slot per sequence: the delta-rule state in fp32 and the ring of the short
convolutions' last inputs. A layer that is run several times has one pool or one state per run. Slots follow their sequence when
rows are swapped, and need no clearing: a sequence that starts at position 0 reads neither. When every attention run has a window
or a chunked mask, the pages that none of them can reach any more go back to the pool as the sequence grows.

``StepBatch`` packs the new tokens of several sequences (any number each) into one row of tokens and puts everything the
kernels need to know about them on the device in one copy."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence

import numpy as np
import torch

from ..ops.delta_rule import CHUNK
from ..ops.kv_attention import first_visible
from .kv_cache import PAGE, PagedRows


@dataclass(frozen=True)
class KeyValues:
    """Cache of one attention run: heads and (padded) head size of its keys and values, and the positions it can see."""
    heads: int
    dim: int
    window: Optional[int] = None
    chunk: Optional[int] = None


@dataclass(frozen=True)
class Latents:
    """Cache of one attention run over latents of (padded) ``rank`` numbers."""
    rank: int
    window: Optional[int] = None
    chunk: Optional[int] = None


class StepBatch:
    """``tokens[i]`` are the next tokens of cache row ``rows[i]``, which holds ``start[i]`` already. ``want``: packed indices
    whose logits are asked for (None: the last token of every sequence)."""

    def __init__(self, cache: "StepCache", tokens: Sequence[Sequence[int]], start: Sequence[int], rows: Sequence[int],
                 want: Optional[Sequence[int]] = None, vocab: Optional[int] = None):
        lens = [len(t) for t in tokens]
        if not lens or min(lens) < 1:
            raise ValueError("a step needs at least one token per sequence")
        if len(set(rows)) != len(rows) or min(rows) < 0 or max(rows) >= cache.max_batch:
            raise ValueError(f"bad cache rows {list(rows)}")
        flat = np.concatenate([np.asarray(t, dtype=np.int64) for t in tokens])
        if vocab is not None and not (0 <= flat.min() and flat.max() < vocab):
            raise ValueError(f"token id outside the vocabulary of {vocab}")
        self.n, self.T, self.max_len = len(lens), len(flat), max(lens)
        self.host_rows, self.host_start, self.lens = list(rows), [int(s) for s in start], lens
        self.max_pos = max(s + n for s, n in zip(self.host_start, lens))
        self.single = self.max_len == 1              # one token per sequence: the decode kernels
        self.fresh = not any(self.host_start)        # whole prompts: nothing is read from the cache
        self.device = cache.device
        want = np.cumsum(lens) - 1 if want is None else np.asarray(want, dtype=np.int64)
        self.n_want = len(want)
        self.want_all = self.n_want == self.T and bool((want == np.arange(self.T)).all())
        self.n_chunks = sum(-(-n // CHUNK) for n in lens)      # the delta rule advances chunk by chunk inside a portion
        self._buf = torch.empty(5 * self.n + 2 + 3 * self.T + self.n_chunks + self.n_want, dtype=torch.int32, device=self.device)
        self._views()
        self._fill(cache, flat, want)

    def _views(self):
        sizes = [self.n, self.n, self.n, self.n + 1, self.n + 1, self.n_chunks, self.T, self.T, self.T, self.n_want]
        (self.start, self.rows, self.slots, self.cu, self.cu_chunk, self.chunk_seq, self.ids, self.tok_seq, self.tok_pos,
         self.want) = torch.split(self._buf[:sum(sizes)], sizes)

    def _fill(self, cache, flat, want):
        lens, start = np.asarray(self.lens), np.asarray(self.host_start)
        seqs, chunks = np.arange(self.n), -(-lens // CHUNK)
        ends = lambda n: np.concatenate(([0], np.cumsum(n)))
        cu = ends(lens)
        seq = np.repeat(seqs, lens)
        parts = (start, self.host_rows, [cache.slot_of(r) for r in self.host_rows], cu, ends(chunks), np.repeat(seqs, chunks), flat, seq,
                 start[seq] + np.arange(self.T) - cu[seq], want)
        host = torch.empty(self._buf.numel(), dtype=torch.int32, pin_memory=self.device.type == "cuda")
        np.concatenate(parts, out=host.numpy(), casting="unsafe")
        self._buf.copy_(host, non_blocking=True)

    def refill(self, cache, tokens: Sequence[int], start: Sequence[int], rows: Sequence[int]):
        """Same shape, next step (one token per sequence): new values in the same device memory (a captured graph reads it)."""
        self.host_rows, self.host_start = list(rows), [int(s) for s in start]
        self.max_pos = max(self.host_start) + 1
        self._fill(cache, np.asarray(tokens), np.arange(self.n))


class StepCache(PagedRows):
    """``kv``: ``KeyValues`` per attention run; ``latents``: ``Latents`` per run of attention over latents; ``states``: ``DeltaShape``
    per recurrent run. ``rewind``: how many of a sequence's last tokens ``truncate`` must be able to drop (their pages are kept)."""

    def __init__(self, max_batch: int, max_seq: int, device, dtype=torch.bfloat16, num_pages: Optional[int] = None, kv: Sequence[KeyValues] = (),
                 latents: Sequence[Latents] = (), states: Sequence = ()):
        super().__init__(max_batch, max_seq, device, num_pages)
        self.dtype, self.rewind = dtype, 0
        self.kv = [torch.zeros(self.num_pages, s.heads, 2, PAGE, s.dim, dtype=dtype, device=self.device) for s in kv]
        self.latent = [torch.zeros(self.num_pages, PAGE, s.rank, dtype=dtype, device=self.device) for s in latents]
        self.state = [torch.zeros(max_batch, s.H, s.D, s.Dv, dtype=torch.float32, device=self.device) for s in states]
        self.ring = [torch.zeros(max_batch, s.taps, s.channels, dtype=torch.float32, device=self.device) for s in states]
        self._slot = list(range(max_batch))
        self.masks = sorted({(s.window or 0, s.chunk or 0) for s in (*kv, *latents)})

    def slot_of(self, row: int) -> int:
        return self._slot[row]

    def bytes_per_token(self) -> int:
        return sum(p.numel() // (self.num_pages * PAGE) * p.element_size() for p in self.kv + self.latent)

    def state_bytes(self) -> int:
        """Bytes of one sequence's recurrent states and convolution inputs."""
        return sum(t[0].numel() * 4 for t in self.state + self.ring)

    def first_needed(self, n: int) -> int:
        """The first cached position that a token at position ``n`` or later sees in any run."""
        return min((first_visible(n, w, c) for w, c in self.masks), default=0)

    def swap(self, a: int, b: int):
        super().swap(a, b)
        self._slot[a], self._slot[b] = self._slot[b], self._slot[a]

    def truncate(self, b: int, new_len: int):
        if new_len == 0:
            self.free(b)
        elif new_len != self._host_lens[b]:
            if self.state:
                raise RuntimeError("a recurrent state cannot be rewound")
            if self.first_needed(new_len) < self._released[b] * PAGE or new_len > self._host_lens[b]:
                raise RuntimeError(f"pages of a sequence of {self._host_lens[b]} tokens that one of {new_len} needs have been given back")
            super().truncate(b, new_len)

    def commit(self, batch_ids: List[int], new_lens: List[int]):
        for b, n in zip(batch_ids, new_lens):
            self._host_lens[b] = n
            self.release_before(b, self.first_needed(max(0, n - self.rewind)))

    def free(self, b: int):
        self._free.extend(reversed(self._host_pages[b][self._released[b]:]))
        self._host_pages[b], self._released[b], self._host_lens[b] = [], 0, 0
