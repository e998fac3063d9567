"""Cache manager and batch layout of decoders that mix paged attention with recurrent state.

``HybridCache`` owns, for every layer run of a model, what its run spec allocates: a K / V pool or a pool of latents (pages
addressed through ONE block table per sequence, shared by all attention runs) or slot-indexed recurrent state; it hands out
pages and slots.
``HybridSequence`` is one request's share of it. ``RaggedBatch`` describes one step: for every sequence the tokens it
brings, single decoded tokens first, then portions of prompts; all index arrays travel in one host-to-device copy.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from ..ops.masks import Mask, Window
from ..ops.rotary import Rotary
from .kv_cache import BlockAllocator


@dataclass(frozen=True)
class PagedRun:
    """Storage of one attention run: K and V pages of ``head_dim`` columns per key head. A run that rotates also gets the angles of
    its positions; one of the runs that share their first one's values (``mixes_values``) also gets that run's V pages (None for the
    first)."""
    kv_heads: int
    head_dim: int
    rotary: Optional[Rotary] = None
    mixes_values: bool = False

    def allocate(self, c: "HybridCache") -> tuple:
        shape = (c.num_blocks, self.kv_heads, c.block_size, self.head_dim)
        k, v = (torch.zeros(shape, dtype=c.dtype, device=c.device) for _ in range(2))
        if self.rotary is None and not self.mixes_values:
            return k, v
        first = None
        if self.mixes_values:
            if c.first_values is None:
                c.first_values = v
            else:
                first = c.first_values
        return k, v, c.angles(self.rotary) if self.rotary is not None else None, first


@dataclass(frozen=True)
class LatentRun:
    """Storage of one latent attention run: pages of one ``width``-column row per token, and the angles of its positions."""
    width: int
    rotary: Rotary

    def allocate(self, c: "HybridCache") -> tuple:
        return torch.zeros((c.num_blocks, c.block_size, self.width), dtype=c.dtype, device=c.device), c.angles(self.rotary)


@dataclass(frozen=True)
class StateRun:
    """Storage of one recurrent run: per slot the tail of its convolution's inputs (the model's dtype; absent without a
    convolution) and a recurrent state (fp32); the angles of its positions where it rotates anything."""
    state: tuple
    conv: Optional[tuple] = None
    rotary: Optional[Rotary] = None

    def allocate(self, c: "HybridCache") -> tuple:
        out = []
        if self.conv is not None:
            out.append(torch.zeros((c.max_sequences, *self.conv), dtype=c.dtype, device=c.device))
        out.append(torch.zeros((c.max_sequences, *self.state), dtype=torch.float32, device=c.device))
        if self.rotary is not None:
            out.append(c.angles(self.rotary))
        return tuple(out)


@dataclass(frozen=True)
class PairRun:
    """Storage of two mixers side by side."""
    left: object
    right: object

    def allocate(self, c: "HybridCache") -> tuple:
        return self.left.allocate(c), self.right.allocate(c)


class HybridCache:
    quantized = False

    def __init__(self, runs: Sequence, num_blocks: int, block_size: int, max_sequences: int, max_len: int, dtype, device):
        if num_blocks <= 0 or block_size <= 0 or max_sequences <= 0 or max_len <= 0:
            raise ValueError("HybridCache: sizes must be positive")
        self.num_blocks, self.block_size, self.max_sequences, self.max_len = num_blocks, block_size, max_sequences, max_len
        self.device, self.dtype = torch.device(device), dtype
        self.max_blocks = (max_len + block_size - 1) // block_size
        self.allocator = BlockAllocator(num_blocks)
        self.slot_allocator = BlockAllocator(max_sequences)
        self.tables = np.zeros((max_sequences, self.max_blocks), dtype=np.int32)   # row = the sequence's slot
        self._angles: Dict[Rotary, torch.Tensor] = {}
        self.first_values: Optional[torch.Tensor] = None      # V pages of the first run that mixes values
        self.runs: List[tuple] = [r.allocate(self) for r in runs]

    def angles(self, rotary: Rotary) -> torch.Tensor:
        """(cos, sin) of every position the cache can hold; one table for all runs that rotate alike."""
        if rotary not in self._angles:
            self._angles[rotary] = rotary.table(self.max_len, self.device)
        return self._angles[rotary]

    def tensors(self, run) -> list:
        """The tensors of one run's storage."""
        if isinstance(run, tuple):
            return [t for part in run for t in self.tensors(part)]
        return [run] if run is not None else []

    def nbytes(self) -> int:
        unique = {t.data_ptr(): t for t in self.tensors(tuple(self.runs)) if t.numel()}
        return sum(t.numel() * t.element_size() for t in unique.values())

    def can_admit(self) -> bool:
        """A slot is free (pages are the caller's business)."""
        return self.slot_allocator.num_free() > 0

    def blocks_for(self, n: int) -> int:
        return (n + self.block_size - 1) // self.block_size


class HybridSequence:
    """Pages and slot of one sequence. The slot is taken with the first tokens and given back by ``reset``."""

    def __init__(self, cache: HybridCache):
        self.cache = cache
        self.slot = -1
        self.blocks: List[int] = []
        self.length = 0

    def current_len(self) -> int:
        return self.length

    def max_len(self) -> int:
        return self.cache.max_len

    def reserve(self, n: int) -> None:
        """Makes room for ``n`` more tokens. Takes nothing when it raises."""
        c = self.cache
        total = self.length + n
        if total > c.max_len:
            raise RuntimeError(f"cache overflow: {self.length} + {n} > max_len {c.max_len}")
        need = c.blocks_for(total) - len(self.blocks)
        if need > c.allocator.num_free():
            raise RuntimeError(f"out of KV blocks: {need} needed, {c.allocator.num_free()} free")
        if self.slot < 0:
            if c.slot_allocator.num_free() == 0:
                raise RuntimeError("out of state slots")
            self.slot = c.slot_allocator.allocate()
            c.tables[self.slot] = 0
        for _ in range(need):
            b = c.allocator.allocate()
            c.tables[self.slot, len(self.blocks)] = b
            self.blocks.append(b)

    def release_to(self, blocks: int, slot: int) -> None:
        """Undoes a ``reserve`` that found ``blocks`` pages and this slot."""
        while len(self.blocks) > blocks:
            self.cache.allocator.free(self.blocks.pop())
        if slot < 0 and self.slot >= 0:
            self.cache.slot_allocator.free(self.slot)
            self.slot = -1

    def advance(self, n: int) -> None:
        self.length += n

    def reset(self) -> None:
        for b in self.blocks:
            self.cache.allocator.free(b)
        self.blocks = []
        if self.slot >= 0:
            self.cache.slot_allocator.free(self.slot)
        self.slot = -1
        self.length = 0


@dataclass
class Segments:
    """A step's prompt rows for one mask, cut at the chunk edges if it has chunks: query and key offsets of every piece, where each
    row's key goes on the key axis, and which pooled keys are copied in front of it."""
    n: int
    max_q: int
    keys: int
    n_gather: int
    host: List[np.ndarray]
    cu_q: Optional[torch.Tensor] = None
    cu_k: Optional[torch.Tensor] = None
    stage_rows: Optional[torch.Tensor] = None
    gather_dst: Optional[torch.Tensor] = None
    gather_src: Optional[torch.Tensor] = None


def cut_segments(portions, mask: Mask, slot_of) -> Segments:
    """``portions``: (pos0, n) of every prompt portion in row order; ``slot_of(i, positions)`` gives pool slots of portion
    i's sequence. Mask 0: one piece per portion with everything before it in front; a window: one piece with what its first
    row sees in front."""
    cu_q, cu_k, stage, dst, src = [0], [0], [], [], []
    row = key = 0
    window = mask.size if isinstance(mask, Window) else 0
    chunk = 0 if window else mask
    for i, (p0, n) in enumerate(portions):
        first = max(0, p0 - window + 1) if window else p0 // chunk * chunk if chunk > 0 else 0
        before = p0 - first
        if before:
            dst.append(np.arange(key, key + before, dtype=np.int32))
            src.append(slot_of(i, np.arange(first, p0)))
        stage.append(np.arange(key + before, key + before + n, dtype=np.int32))
        if chunk > 0:
            ends = np.append(np.arange(first + chunk, p0 + n, chunk), p0 + n)
        else:
            ends = np.array([p0 + n])
        cu_q.extend((ends - p0 + row).tolist())
        cu_k.extend((ends - first + key).tolist())
        row += n
        key += before + n
    q = np.asarray(cu_q, dtype=np.int32)
    cat = lambda a: np.concatenate(a).astype(np.int32) if a else np.zeros(0, dtype=np.int32)   # noqa: E731
    host = [q, np.asarray(cu_k, dtype=np.int32), cat(stage), cat(dst), cat(src)]
    return Segments(len(cu_q) - 1, int(np.diff(q).max()) if len(q) > 1 else 0, key, len(host[3]), host)


@dataclass
class Tiles:
    """A step's prompt portions cut into tiles of a fixed number of tokens, each portion from its first row: the portion of
    every tile, and the first tile of every portion."""
    n: int
    seq: Optional[torch.Tensor] = None
    first: Optional[torch.Tensor] = None


class RaggedBatch:
    """One step. ``entries``: (sequence, token ids); the sequences' pages are reserved here and their lengths advanced by
    ``commit`` once the step has been launched. Rows are ordered with single tokens first; ``row_of[i]`` is the first row
    of entry i. ``want`` [i]: places among entry i's tokens whose logits are asked for, answered in entry order. ``masks``:
    attention masks, ``tiles``: tile sizes that the model's mixers ask for (``segments``, ``tiles``)."""

    def __init__(self, cache: HybridCache, entries, want=None, masks: Sequence[Mask] = (), max_len: int = 0,
                 tiles: Sequence[int] = ()):
        self.cache = cache
        entries = [(s, np.asarray(t, dtype=np.int32)) for s, t in entries]
        if any(len(t) == 0 for _, t in entries):
            raise ValueError("RaggedBatch: an entry without tokens")
        if len({id(s) for s, _ in entries}) != len(entries):
            raise ValueError("RaggedBatch: a sequence appears twice")
        bs = cache.block_size
        taken = []
        try:
            for s, t in entries:
                before = (len(s.blocks), s.slot)
                s.reserve(len(t))
                taken.append((s, before))
        except Exception:
            for s, (nb, slot) in taken:        # a step that does not fit leaves no trace
                s.release_to(nb, slot)
            raise
        order = sorted(range(len(entries)), key=lambda i: len(entries[i][1]) > 1)
        self.entries = entries
        seqs = [entries[i][0] for i in order]
        toks = [entries[i][1] for i in order]
        n = np.array([len(t) for t in toks], dtype=np.int64)
        row0 = np.concatenate([[0], np.cumsum(n)])
        self.n_decode = nd = int((n == 1).sum())
        self.n_prompts = len(seqs) - nd
        self.rows = T = int(row0[-1])
        self.row_of = np.zeros(len(entries), dtype=np.int64)
        self.row_of[np.array(order, dtype=np.int64)] = row0[:-1]
        pos0 = np.array([s.length for s in seqs], dtype=np.int64)
        slot = np.array([s.slot for s in seqs], dtype=np.int64)
        seq_of = np.repeat(np.arange(len(seqs)), n)
        positions = np.arange(T) - row0[:-1][seq_of] + pos0[seq_of]
        pool_slots = cache.tables[slot[seq_of], positions // bs].astype(np.int64) * bs + positions % bs
        need = int((pos0 + n).max())
        self.max_len = max(max_len, need) if max_len else -(-need // 256) * 256   # (bounds the key split; coarse on purpose)
        tables = cache.tables[slot][:, :cache.blocks_for(need)]
        rows = []
        for i in range(len(entries)):
            w = (want[i] if want is not None else ())
            for k in w:
                if not 0 <= k < len(entries[i][1]):
                    raise ValueError("RaggedBatch: a wanted place outside its entry")
                rows.append(self.row_of[i] + k)
        self.n_want = len(rows)
        self._spans = list(zip(row0[:-1].tolist(), n.tolist(), slot.tolist(), pos0.tolist()))
        segs: Dict[Mask, Segments] = {}
        if self.n_prompts:
            pslots = slot[nd:]

            def slot_of(i, p):
                return cache.tables[pslots[i], p // bs] * bs + p % bs
            for c in masks:
                segs[c] = cut_segments(list(zip(pos0[nd:].tolist(), n[nd:].tolist())), c, slot_of)
        nblk = (n[nd:] + 3) // 4                  # the recurrence takes four tokens of a portion at once
        fields = {
            "tokens": np.concatenate(toks), "positions": positions, "slots": pool_slots, "seq_of": seq_of, "tables": tables,
            "state_slots": slot, "lens": pos0[:nd] + 1, "cu": row0[nd:] - row0[nd], "pos0": pos0[nd:],
            "blk_seq": np.repeat(np.arange(self.n_prompts), nblk), "blk0": np.concatenate([[0], np.cumsum(nblk)]), "want": np.asarray(rows, dtype=np.int64),
        }
        self._tiles: Dict[int, Tiles] = {}
        if self.n_prompts:
            for size in tiles:
                per = -(-n[nd:] // size)
                self._tiles[size] = Tiles(int(per.sum()))
                fields[f"seq:{size}"] = np.repeat(np.arange(self.n_prompts), per)
                fields[f"first:{size}"] = np.concatenate([[0], np.cumsum(per)])
        pieces = list(segs.values())
        for i, sg in enumerate(pieces):
            for name, a in zip(("cu_q", "cu_k", "stage_rows", "gather_dst", "gather_src"), sg.host):
                fields[f"{name}:{i}"] = a
        flat = np.concatenate([np.ascontiguousarray(a, dtype=np.int32).reshape(-1) for a in fields.values()])
        host = torch.from_numpy(flat)
        if cache.device.type == "cuda":
            dev = host.pin_memory().to(cache.device, non_blocking=True)
        else:
            dev = host
        at = 0
        for name, a in fields.items():
            t = dev[at:at + a.size].view(a.shape)
            at += a.size
            if ":" in name:
                f, c = name.split(":")
                setattr(self._tiles[int(c)] if f in ("seq", "first") else pieces[int(c)], f, t)
            else:
                setattr(self, name, t)
        self._segs = segs

    def segments(self, mask: Mask) -> Segments:
        return self._segs[mask]

    def tiles(self, size: int) -> Tiles:
        return self._tiles[size]

    def spans(self):
        """(first row, rows, slot, position of the first row) of every sequence, in row order."""
        return self._spans

    def commit(self) -> None:
        for s, t in self.entries:
            s.advance(len(t))


class DecodeBatch:
    """A step of ``rows`` single tokens with device arrays at fixed addresses, for captured launches: packed int32 rows
    [token, position, pool slot, length, state slot, table...]; a row without a sequence has position and slots -1 and length 0."""
    HEAD = 5
    n_prompts = 0

    def __init__(self, packed: torch.Tensor, max_len: int):
        self.packed, self.max_len = packed, max_len
        self.rows = self.n_decode = self.n_want = packed.shape[0]
        self.want = None

    def unpack(self) -> "DecodeBatch":
        """(Part of the captured work: the fields are copied out of the packed rows.)"""
        p = self.packed
        head = p[:, :self.HEAD].t().contiguous()
        self.tokens, self.positions, self.slots, self.lens, self.state_slots = head.unbind(0)
        self.tables = p[:, self.HEAD:]
        self.seq_of = torch.arange(self.rows, device=p.device, dtype=torch.int32)
        return self

    @staticmethod
    def fill(buf: np.ndarray, cache: HybridCache, seqs, tokens) -> None:
        n, bs = len(seqs), cache.block_size
        if n:
            slot = np.array([s.slot for s in seqs], dtype=np.int64)
            pos = np.array([s.length for s in seqs], dtype=np.int64)
            buf[:n, 0] = tokens
            buf[:n, 1] = pos
            buf[:n, 2] = cache.tables[slot, pos // bs] * bs + pos % bs
            buf[:n, 3] = pos + 1
            buf[:n, 4] = slot
            buf[:n, DecodeBatch.HEAD:] = cache.tables[slot]
        buf[n:] = 0
        buf[n:, 1] = buf[n:, 2] = buf[n:, 4] = -1
