"""Cache of decoders that mix attention over a paged cache with recurrent layers.

Two kinds of storage on one sequence table:

* *pages*: per layer that asks for them a pool ``[num_blocks + 1, 64, width]`` addressed through the block tables of
  ``PagedBlocks`` (rows of any width: the latent attention layers keep one row per token for all heads);
* *slots*: per recurrent layer named tensors ``[max_seqs + 1, ...]``; a sequence owns one slot index in all of them from
  ``add_sequence`` to ``free_sequence``. A slot is never cleared: the kernels start from zeros when a sequence's first
  token of a step is its position 0.

The last block and the last slot lie outside the pools; padding rows of captured decode steps write there. A recurrent
state has absorbed every token it saw, so a sequence with slots cannot be cut back (``can_truncate``); ``fork`` copies the
slot and shares the pages. When every layer with pages has a window, pages that lie wholly before the widest of them go back
to the pool while the sequence lives.

A layer that runs several times in a step (a looped stack) has a spec, pages and slots for every run; a model may add a spec of its own
behind them (the latest token of every sequence).

``split_groups`` divides a step's sequences into short and long portions, which run on different kernels; ``attention_runs`` joins
long portions into launches of an attention kernel whose keys are rows of one buffer."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .kv_cache import BLOCK, BatchMeta, PagedBlocks


@dataclass
class CacheSpec:
    """What one layer keeps per token (``page_width`` columns) and per sequence (``slots``: name -> (shape, dtype), a
    dtype of None is the model's). ``window`` > 0: no token looks back further than to the window - 1 tokens before it."""
    page_width: int = 0
    window: int = 0
    slots: Dict[str, Tuple[Tuple[int, ...], Optional[torch.dtype]]] = field(default_factory=dict)


class StateCache(PagedBlocks):
    def __init__(self, specs: Sequence[CacheSpec], num_blocks: int, max_seqs: int, dtype=torch.bfloat16, device="cuda",
                 max_length: int = 0):
        super().__init__(num_blocks, device)
        self.max_length = max_length
        self.max_seqs = max_seqs
        self.scratch_block, self.scratch_slot = num_blocks, max_seqs
        self.pages: Dict[int, torch.Tensor] = {}
        self.slots: Dict[int, Dict[str, torch.Tensor]] = {}
        for i, s in enumerate(specs):
            if s.page_width:
                self.pages[i] = torch.zeros(num_blocks + 1, BLOCK, s.page_width, dtype=dtype, device=device)
            if s.slots:
                self.slots[i] = {n: torch.zeros(max_seqs + 1, *shape, dtype=dt or dtype, device=device)
                                 for n, (shape, dt) in s.slots.items()}
        windows = [s.window for s in specs if s.page_width]
        self.window = max(windows) if windows and min(windows) > 0 else 0
        self.can_truncate = not self.slots and self.window == 0
        # without recurrent layers nothing is kept per sequence: every sequence names slot 0 and their number is not limited
        self.free_slots: List[int] = list(range(max_seqs - 1, -1, -1))
        self.slot_of: Dict[int, int] = {}

    def _copy_block(self, dst: int, src: int) -> None:
        for t in self.pages.values():
            t[dst].copy_(t[src])

    def nbytes(self) -> int:
        ts = list(self.pages.values()) + [t for d in self.slots.values() for t in d.values()]
        return sum(t.numel() * t.element_size() for t in ts)

    def bytes_per_token(self) -> int:
        return sum(t.shape[2] * t.element_size() for t in self.pages.values())

    # ------------------------------------------------------------------ sequences
    def can_admit(self) -> bool:
        return not self.slots or bool(self.free_slots)

    def _take_slot(self, seq_id: int) -> int:
        slot = self.free_slots.pop() if self.slots else 0
        self.slot_of[seq_id] = slot
        return slot

    def add_sequence(self, seq_id: int) -> None:
        if not self.can_admit():
            raise MemoryError(f"all {self.max_seqs} state slots are in use")
        super().add_sequence(seq_id)
        self._take_slot(seq_id)

    def free_sequence(self, seq_id: int) -> None:
        super().free_sequence(seq_id)
        slot = self.slot_of.pop(seq_id)
        if self.slots:
            self.free_slots.append(slot)

    def fork(self, src_id: int, dst_id: int) -> None:
        if not self.can_admit():
            raise MemoryError(f"all {self.max_seqs} state slots are in use")
        super().fork(src_id, dst_id)
        a, b = self.slot_of[src_id], self._take_slot(dst_id)
        for d in self.slots.values():
            for t in d.values():
                t[b].copy_(t[a])

    def truncate(self, seq_id: int, new_len: int) -> None:
        if new_len not in (0, self.seqs[seq_id].length) and not self.can_truncate:
            raise ValueError("tokens that a recurrent state has absorbed or a window has left behind cannot be dropped")
        super().truncate(seq_id, new_len)

    # ------------------------------------------------------------------ batch metadata
    def prepare(self, seq_ids: Sequence[int], new_tokens: Sequence[int]) -> BatchMeta:
        meta = super().prepare(seq_ids, new_tokens)
        dev = self.device
        meta.state_slots = torch.tensor([self.slot_of[s] for s in seq_ids], dtype=torch.int32).to(dev, non_blocking=True)
        meta.seq_of = torch.repeat_interleave(torch.arange(len(seq_ids), dtype=torch.int32),
                                              torch.tensor(list(new_tokens))).to(dev, non_blocking=True)
        return meta


@dataclass
class SeqGroup:
    """Some sequences of a step, as the kernels take them. ``q_start`` points into the step's token rows, ``c_start`` into
    tokens counted over the group alone; ``tok_rows`` is the step's row of each of those tokens."""
    n: int
    n_tok: int
    max_q: int
    max_kv: int
    block_table: torch.Tensor
    seq_lens: torch.Tensor
    q_start: torch.Tensor
    q_lens: torch.Tensor
    c_start: torch.Tensor
    state_slots: Optional[torch.Tensor]
    tok_rows: torch.Tensor
    host: List[Tuple[int, int, int, int]] = field(default_factory=list)     # (batch index, q_start, q_len, seq_len)


def split_groups(meta: BatchMeta, limit: int) -> Tuple[Optional[SeqGroup], Optional[SeqGroup]]:
    """(sequences with at most ``limit`` new tokens, the others); None for an empty side. A step whose lengths are not
    known on the host (a captured one) has one token per sequence."""
    if meta.host is None:
        if meta.max_q != 1:
            raise ValueError("a step without host metadata must bring one token per sequence")
        n = meta.q_lens.shape[0]
        return SeqGroup(n, n, 1, meta.max_kv, meta.block_table, meta.seq_lens, meta.q_start, meta.q_lens, meta.q_start,
                        meta.state_slots, meta.q_start), None
    _, _, seq_lens, q_start, q_lens, _ = meta.host
    sides = ([i for i, q in enumerate(q_lens) if q <= limit], [i for i, q in enumerate(q_lens) if q > limit])
    out = []
    for ix in sides:
        if not ix:
            out.append(None)
            continue
        c, c_start = 0, []
        for i in ix:
            c_start.append(c)
            c += q_lens[i]
        host = [(i, q_start[i], q_lens[i], seq_lens[i]) for i in ix]
        mq, mk = max(q_lens[i] for i in ix), max(seq_lens[i] for i in ix)
        if len(ix) == len(q_lens):
            out.append(SeqGroup(len(ix), c, mq, mk, meta.block_table, meta.seq_lens, meta.q_start, meta.q_lens,
                                meta.q_start, meta.state_slots,
                                torch.arange(c, dtype=torch.int32, device=meta.q_lens.device), host))
            continue
        dev = meta.q_lens.device
        rows = torch.tensor([q_start[i] + k for i in ix for k in range(q_lens[i])], dtype=torch.int32).to(dev, non_blocking=True)
        sel = torch.tensor(ix, dtype=torch.int64).to(dev, non_blocking=True)
        cs = torch.tensor(c_start, dtype=torch.int32).to(dev, non_blocking=True)
        out.append(SeqGroup(len(ix), c, mq, mk, meta.block_table[sel], meta.seq_lens[sel], meta.q_start[sel],
                            meta.q_lens[sel], cs, meta.state_slots[sel] if meta.state_slots is not None else None, rows, host))
    return out[0], out[1]


@dataclass
class AttnRun:
    """Consecutive sequences of a step whose attention is one launch: query rows ``rows`` of the step, key rows gathered from the
    cache rows ``slots``. Query i (from the first of ``rows`` on) sees key rows ``seq_start[i]`` .. i + ``shift``."""
    rows: slice
    n: int
    slots: torch.Tensor
    seq_start: torch.Tensor
    shift: int


def attention_runs(meta: BatchMeta, group: SeqGroup, chunk: int = 0) -> List[AttnRun]:
    """A run begins with any sequence and takes in the next ones as long as their rows follow and they have no earlier tokens: then
    every query row lies ``shift`` before its own key row, the earlier tokens of the first sequence (``chunk`` > 0: those of its
    chunk, as every query then sees the keys of its own chunk of positions alone)."""
    runs: List[List[Tuple[int, int, int, int]]] = []
    for s in group.host:
        i, q0, n, total = s
        if runs and total == n and q0 == runs[-1][-1][1] + runs[-1][-1][2]:
            runs[-1].append(s)
        else:
            runs.append([s])
    out, dev = [], meta.slots.device
    for run in runs:
        i, q0, n0, total = run[0]
        first, n = total - n0, sum(s[2] for s in run)
        key0 = first - first % chunk if chunk else 0          # position of the first key row
        prior = first - key0
        slots = meta.slots[q0:q0 + n]
        if prior:
            b0 = key0 // BLOCK
            pages = meta.block_table[i, b0:-(-first // BLOCK)].long()
            old = (pages[:, None] * BLOCK + torch.arange(BLOCK, device=dev)).view(-1)[key0 - b0 * BLOCK:first - b0 * BLOCK]
            slots = torch.cat([old, slots])
        base = torch.tensor([0] + [s[1] - q0 + prior for s in run[1:]], dtype=torch.int32)
        start = torch.repeat_interleave(base, torch.tensor([s[2] for s in run]))
        if chunk:
            pos = torch.cat([torch.arange(t - m, t, dtype=torch.int32) for _, _, m, t in run])
            at = torch.where(torch.arange(n) < n0, key0, 0)
            start = start + (pos - pos % chunk - at).to(torch.int32)
        out.append(AttnRun(slice(q0, q0 + n), n, slots.contiguous(), start.to(dev, non_blocking=True), prior))
    return out
