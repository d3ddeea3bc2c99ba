"""Slots, cache pages and the step function shared by the paged-cache runtimes.

``PagedSequences`` is the host side of a paged cache: request slots, a free list of pages with reference counts, and the
block table the attention kernels read (block 0 is never handed out: unused table entries point at it).

``PagedRuntime`` adds the passes over a model that supplies ``_forward``: ``step`` runs any mix of prompt portions and
single tokens of several requests as ONE batch, ``prefill`` is a run of such steps for one request, ``decode`` advances
a batch of requests by one token each, replayed from a CUDA graph per (batch size, context bucket).

(Role of the slot / paged-KV / batch interface in cpp_engine/include/inference_engine.hpp:126-181.)
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops.scan import Segments
from ..utils import canary


@dataclass
class SeqState:
    slot: int
    blocks: list[int] = field(default_factory=list)     # page of every block of positions; 0 once given back
    length: int = 0
    retired: int = 0                                     # leading blocks given back (never looked at again)


class NoComm:
    """Single-rank stand-in for the tensor-parallel communicator."""
    world, rank = 1, 0

    def all_reduce(self, t: torch.Tensor) -> torch.Tensor:
        return t

    def argmax_merge(self, idx: torch.Tensor, val: torch.Tensor) -> torch.Tensor:
        return idx

    def all_gather(self, t: torch.Tensor) -> torch.Tensor:
        return t.unsqueeze(0)


class PagedSequences:
    def __init__(self, device, max_slots: int, max_context: int, block_size: int = 64, num_blocks: int | None = None):
        self.device = torch.device(device)
        self.block_size, self.max_slots, self.max_context = block_size, max_slots, max_context
        self.max_blocks_per_seq = (max_context + block_size - 1) // block_size
        self.num_blocks = num_blocks or (self.max_blocks_per_seq * max_slots + 1)
        self.free_blocks = list(range(self.num_blocks - 1, 0, -1))
        self.block_refs = [0] * self.num_blocks          # sequences + prefix-cache entries holding each block
        self.free_slots = list(range(max_slots - 1, -1, -1))
        self.seqs: dict[int, SeqState] = {}
        self.block_table = torch.zeros(max_slots, self.max_blocks_per_seq, dtype=torch.int32, device=self.device)
        self._bt_host = torch.zeros(max_slots, self.max_blocks_per_seq, dtype=torch.int32)

    def allocate(self) -> int:
        if not self.free_slots:
            raise RuntimeError("no free slot")
        slot = self.free_slots.pop()
        self.seqs[slot] = SeqState(slot)
        return slot

    def free(self, slot: int) -> None:
        st = self.seqs.pop(slot)
        self._release_blocks([b for b in st.blocks if b])
        self.free_slots.append(slot)

    def _release_blocks(self, blocks: list[int]) -> None:
        for b in reversed(blocks):
            self.block_refs[b] -= 1
            if self.block_refs[b] == 0:
                self.free_blocks.append(b)

    def history_floor(self, length: int) -> int:
        """First position that a token at position ``length`` or later can still look at."""
        return 0

    def blocks_needed(self, tokens: int) -> int:
        return (tokens + self.block_size - 1) // self.block_size

    def history_span(self) -> int | None:
        """Largest distance between a position and the first one it can look at (None: unbounded)."""
        return None

    def pages_held(self, tokens: int, portion: int) -> int:
        """Upper bound on the pages a sequence of ``tokens`` tokens holds at any time when no step brings more than
        ``portion`` of them: with a bounded history a step needs the pages from the history's start to its own end."""
        total, span = self.blocks_needed(tokens), self.history_span()
        return total if span is None else min(total, self.blocks_needed(span + portion) + 1)

    def _ensure_blocks(self, st: SeqState, new_len: int) -> None:
        """Pages for positions up to ``new_len`` of a sequence; pages no later token can see go back first."""
        need = self.blocks_needed(new_len)
        if need > self.max_blocks_per_seq:
            raise RuntimeError("sequence exceeds max_context")
        changed = False
        dead = min(self.history_floor(st.length) // self.block_size, len(st.blocks))
        if dead > st.retired:
            self._release_blocks(st.blocks[st.retired:dead])
            for i in range(st.retired, dead):
                st.blocks[i] = 0
            self._bt_host[st.slot, st.retired:dead] = 0
            st.retired, changed = dead, True
        if need - len(st.blocks) > len(self.free_blocks):
            if changed:
                self.block_table[st.slot].copy_(self._bt_host[st.slot], non_blocking=True)
            raise RuntimeError("KV cache exhausted")
        while len(st.blocks) < need:
            b = self.free_blocks.pop()
            self.block_refs[b] = 1
            self._bt_host[st.slot, len(st.blocks)] = b
            st.blocks.append(b)
            changed = True
        if changed:
            self.block_table[st.slot].copy_(self._bt_host[st.slot], non_blocking=True)

    def cache_rows(self, st: SeqState, lo: int, hi: int) -> torch.Tensor:
        """int32 (host): flat cache row of positions [lo, hi)."""
        pos = torch.arange(lo, hi)
        return (self._bt_host[st.slot][pos // self.block_size] * self.block_size + pos % self.block_size).to(torch.int32)


class PagedRuntime(PagedSequences):
    """A model over a paged cache.  The model supplies

    ``_forward(ids, positions, kv_slots, meta, rows)``: fp32 logits of ``rows`` (int64 / int32 row numbers, or None for
    every row) after appending the batch to the cache, and ``_next(logits)``: greedy tokens.

    ``meta["mode"]``: ``"decode"`` - one row per sequence, static buffers (``block_table`` row i belongs to row i,
    ``kv_len``, ``max_kv_len``); ``"mixed"`` - the first ``tile_rows`` rows are portions of several sequences
    (``q_start``, ``q_len``, ``kv_len``, ``max_q_len``, ``tile_seq``; ``kv_start`` / ``kv_total``: where their contexts begin
    when they are laid out one after the other), the rest single rows (``row_seq``, ``max_kv_len``).  In both modes
    ``segments`` says which neighbouring rows form one sequence's portion and which state slot it has, for mixers that carry
    a recurrent state.

    Recurrent state is held per request slot in tensors from ``slot_state``; a slot's content is meaningless until its
    sequence's first token, whose position 0 the kernels take as "start from zero".  The slot after the last one is scratch:
    the pass that warms up a decode graph runs on it, because running a recurrent step twice would advance the state twice.
    """
    tile_min_rows = 2            # portions with fewer tokens run as single rows

    def __init__(self, device, max_slots: int, max_context: int, block_size: int = 64, num_blocks: int | None = None, comm=None):
        super().__init__(device, max_slots, max_context, block_size, num_blocks)
        self.comm = comm or NoComm()
        self._graphs: dict[tuple, dict] = {}
        self.launches = 0
        self.last_logits: torch.Tensor | None = None

    def slot_state(self, *shape: int, dtype: torch.dtype, name: str) -> torch.Tensor:
        """[request slots + scratch, ...] of recurrent state."""
        return canary.zeros(self.max_slots + 1, *shape, dtype=dtype, device=self.device, name=name)

    @property
    def scratch_slot(self) -> int:
        return self.max_slots

    @property
    def max_blocks(self) -> int:
        return self.max_blocks_per_seq

    def _ensure(self, st: SeqState, new_len: int) -> None:
        self._ensure_blocks(st, new_len)

    def _forward(self, ids, positions, kv_slots, meta, rows):
        raise NotImplementedError

    def _next(self, logits: torch.Tensor) -> torch.Tensor:
        from ..ops import basic
        return basic.argmax(logits)

    def greedy(self, logits: torch.Tensor) -> list[int]:
        """Arg-max tokens of ``step``'s logits."""
        return [int(t) for t in self._next(logits.contiguous()).tolist()]

    # ---- one batch of portions and single tokens
    @torch.no_grad()
    def step(self, entries) -> torch.Tensor | None:
        """``entries``: (slot, token ids, wanted places) per request, slots distinct.  Appends every entry's tokens to
        its sequence in one pass over the model; returns the fp32 logits at the wanted places in the given order
        ([wanted, vocab]; None when nothing is wanted)."""
        from ..ops import _lib
        l0 = _lib.LAUNCHES
        dev = self.device
        assert len({e[0] for e in entries}) == len(entries), "one entry per request and step"
        lens = [len(e[1]) for e in entries]
        assert entries and all(n > 0 for n in lens), "every entry brings at least one token"
        if all(n == 1 for n in lens):                    # a decode batch: the captured pass, one row per entry
            self.decode([e[0] for e in entries], torch.tensor([int(e[1][0]) for e in entries], dtype=torch.int32))
            want = [i for i, e in enumerate(entries) for _ in e[2]]
            return self.last_logits[torch.tensor(want, device=dev)] if want else None
        for (slot, _, _), n in zip(entries, lens):
            self._ensure(self.seqs[slot], self.seqs[slot].length + n)
        tiles = [i for i, n in enumerate(lens) if n >= self.tile_min_rows]
        singles = [i for i, n in enumerate(lens) if n < self.tile_min_rows]
        order = tiles + singles
        first: dict[int, int] = {}                       # entry -> its first row
        n_rows = 0
        for i in order:
            first[i] = n_rows
            n_rows += lens[i]
        tile_rows = sum(lens[i] for i in tiles)
        sts = [self.seqs[e[0]] for e in entries]
        cat = lambda parts: torch.cat(parts) if len(parts) > 1 else parts[0]
        tok = cat([torch.as_tensor(entries[i][1], dtype=torch.int32).reshape(-1).cpu() for i in order])
        pos = cat([torch.arange(sts[i].length, sts[i].length + lens[i], dtype=torch.int32) for i in order])
        rows = cat([self.cache_rows(sts[i], sts[i].length, sts[i].length + lens[i]) for i in order])
        seq = cat([torch.full((lens[i],), sts[i].slot, dtype=torch.int32) for i in order])
        want = torch.tensor([first[i] + w for i, e in enumerate(entries) for w in e[2]], dtype=torch.int32)
        start = cat([torch.full((lens[i],), first[i], dtype=torch.int32) for i in order])
        kv_start, kv_total = [], 0                       # the contexts of the tile entries, laid out one after the other
        for i in order:
            kv_start.append(kv_total)
            kv_total += sts[i].length + lens[i] if i in tiles else 0
        desc = torch.tensor([[first[i], lens[i], sts[i].length + lens[i], sts[i].slot, k] for i, k in zip(order, kv_start)],
                            dtype=torch.int32).t().reshape(-1)
        # one upload: [ids | positions | cache rows | table rows | entry starts | entry descriptors | wanted rows]
        up = cat([tok, pos, rows, seq, start, desc, want])
        up = up.pin_memory().to(dev, non_blocking=True) if dev.type == "cuda" else up
        ids, pos_d, slots_d, seq_d, start_d = (up[k * n_rows:(k + 1) * n_rows] for k in range(5))
        e_first, e_len, e_kv, e_slot, e_start = up[5 * n_rows:5 * n_rows + desc.numel()].view(5, -1)
        meta = {"mode": "mixed", "tile_rows": tile_rows, "row_seq": seq_d, "max_q_len": max([lens[i] for i in tiles], default=0),
                "max_kv_len": max(sts[i].length + lens[i] for i in range(len(entries))),
                "segments": Segments(start_d, seq_d, e_first, e_len, e_slot, max(lens), min(lens))}
        if tiles:
            n = len(tiles)
            meta.update(q_start=e_first[:n], q_len=e_len[:n], kv_len=e_kv[:n], tile_seq=e_slot[:n],
                        kv_start=e_start[:n], kv_total=kv_total)
        # a pass has to run even when no logits are asked for: it fills the cache
        wanted = up[5 * n_rows + desc.numel():]
        logits = self._forward(ids, pos_d, slots_d, meta, wanted)
        for st, n in zip(sts, lens):
            st.length += n
        self.launches = _lib.LAUNCHES - l0
        if want.numel() == 0:
            return None
        self.last_logits = logits
        return logits

    @torch.no_grad()
    def prefill(self, slot: int, token_ids: torch.Tensor, chunk: int = 4096) -> torch.Tensor:
        """Append a prompt in portions of ``chunk`` tokens; returns the greedy next token [1] (device)."""
        ids = torch.as_tensor(token_ids).to(torch.int32).reshape(-1).cpu()
        total, launches, logits = ids.numel(), 0, None
        for s in range(0, total, chunk):
            part = ids[s:s + chunk]
            logits = self.step([(slot, part, [part.numel() - 1] if s + chunk >= total else [])])
            launches += self.launches
        self.launches = launches
        return self._next(logits)

    # ---- one token for each of several requests
    def _decode_body(self, buf, bucket: int) -> torch.Tensor:
        row = buf["row"]
        meta = {"mode": "decode", "block_table": buf["bt"], "kv_len": buf["kv_len"], "max_kv_len": bucket,
                "segments": Segments(row, buf["slots"], row, buf["one"], buf["slots"], 1, 1)}
        buf["logits"] = self._forward(buf["ids"], buf["pos"], buf["kv_slots"], meta, None)
        return self._next(buf["logits"])

    @torch.no_grad()
    def decode(self, slots: list[int], token_ids: torch.Tensor, use_graph: bool = True) -> torch.Tensor:
        from ..ops import _lib
        b, dev = len(slots), self.device
        sts = [self.seqs[s] for s in slots]
        for st in sts:
            self._ensure(st, st.length + 1)
        bucket = 1 << max(10, max(st.length for st in sts).bit_length())
        entry = self._graphs.setdefault((b, bucket), {"buf": None, "graph": None})
        if entry["buf"] is None:
            z = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)
            entry["buf"] = {"ids": z(b), "pos": z(b), "kv_slots": z(b), "kv_len": z(b) + 1, "bt": z(b, self.max_blocks),
                            "slots": z(b) + self.scratch_slot, "one": z(b) + 1,
                            "row": torch.arange(b, dtype=torch.int32, device=dev)}
        buf = entry["buf"]
        host = torch.tensor([[st.length, st.length + 1, st.slot,
                              st.blocks[st.length // self.block_size] * self.block_size + st.length % self.block_size]
                             for st in sts], dtype=torch.int32).to(dev, non_blocking=True)
        buf["ids"].copy_(token_ids)
        buf["pos"].copy_(host[:, 0])
        buf["kv_len"].copy_(host[:, 1])
        buf["kv_slots"].copy_(host[:, 3])
        buf["bt"].copy_(self.block_table[host[:, 2].long()])
        graphed = use_graph and dev.type == "cuda"
        if graphed and entry["graph"] is None:
            buf["slots"].fill_(self.scratch_slot)       # the K/V rows the warm-up writes are rewritten by the replay
            self._decode_body(buf, bucket)
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            l0 = _lib.LAUNCHES
            with torch.cuda.graph(g):
                entry["out"] = self._decode_body(buf, bucket)
            entry["graph"], entry["launches"] = g, _lib.LAUNCHES - l0
        buf["slots"].copy_(host[:, 2])
        if not graphed:
            l0 = _lib.LAUNCHES
            out = self._decode_body(buf, bucket)
            self.launches = _lib.LAUNCHES - l0
        else:
            entry["graph"].replay()
            self.launches = entry["launches"]
            out = entry["out"]
        for st in sts:
            st.length += 1
        self.last_logits = buf["logits"]
        return out

    @torch.no_grad()
    def generate(self, prompt: torch.Tensor, max_new_tokens: int, chunk: int = 4096, use_graph: bool = True) -> list[int]:
        slot = self.allocate()
        try:
            tok = self.prefill(slot, prompt, chunk)
            out = [int(tok.item())]
            while len(out) < max_new_tokens:
                tok = self.decode([slot], tok.to(torch.int32), use_graph)
                out.append(int(tok.item()))
            return out
        finally:
            self.free(slot)

    def stats(self) -> dict:
        return {"kv_blocks_free": len(self.free_blocks), "kv_blocks_total": self.num_blocks - 1}
