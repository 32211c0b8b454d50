"""Teacher-forced stepping of a rollout engine: the caller brings the tokens, nothing is sampled.

:class:`TokenFeed` drives the engine's own prompt forward, decode step, scheduler, slots and pages, and returns logits
at chosen places.  It is what ``bin/trace_run`` replays traces with, and the way to compare cached decoding with whole
prompts."""
from __future__ import annotations

import torch


class TokenFeed:
    def __init__(self, engine):
        self.e = engine
        self.slot: dict = {}     # request -> slot
        self.length: dict = {}   # request -> tokens consumed
        self._rid: dict = {}     # request -> scheduler id
        self._next_rid = 0
        engine.seq_lens.fill_(-1)
        engine._reset_sums()

    @torch.no_grad()
    def step(self, entries, end=()) -> list[torch.Tensor]:
        """``entries``: [(request, tokens, want)].  A request seen for the first time starts with these tokens, another
        one goes on with them.  Returns, per entry, logits [len(want), V] (fp32) at the places ``want`` among its
        tokens.  ``end``: requests to release afterwards."""
        fresh = [i for i, (r, _, _) in enumerate(entries) if r not in self.slot]
        out: list = [None] * len(entries)
        if fresh:
            self._start([entries[i] for i in fresh], fresh, out)
        going = [i for i, (r, _, _) in enumerate(entries) if i not in set(fresh)]
        rows: dict[int, list] = {i: [] for i in going}
        for k in range(max((len(entries[i][1]) for i in going), default=0)):
            active = [i for i in going if k < len(entries[i][1])]
            logits = self._advance([(entries[i][0], entries[i][1][k]) for i in active])
            for i in active:
                if k in entries[i][2]:
                    rows[i].append((k, logits[self.slot[entries[i][0]]].float().clone()))
        for i in going:
            by_place = dict(rows[i])
            out[i] = torch.stack([by_place[k] for k in entries[i][2]]) if entries[i][2] else self._none()
        for r in end:
            self.release(r)
        return out

    def _none(self):
        return torch.empty(0, self.e.cfg.vocab_size, device=self.e.dev)

    def _start(self, entries, index, out):
        e = self.e
        for r, toks, _ in entries:
            if not toks:
                raise ValueError(f"request {r!r} starts without tokens")
            self._rid[r] = self._next_rid
            self._next_rid += 1
            e.sched.add(self._rid[r], len(toks), 0, self._rid[r])
        by_rid = {self._rid[r]: r for r, _, _ in entries}
        admitted = e.sched.admit(e.block_table_host.numpy())
        if len(admitted) != len(entries):
            raise RuntimeError(f"{len(entries)} requests do not fit the engine ({e.max_seqs} slots of at most {e.max_len} "
                               f"tokens, {e.sched.num_free_blocks} free pages)")
        for rid, slot, _, _ in admitted:
            self.slot[by_rid[rid]] = slot
        e.block_table.copy_(e.block_table_host)
        hidden, ctx = e._prefill_all([(self.slot[r], list(toks)) for r, toks, _ in entries])
        at = 0
        for i, (r, toks, want) in zip(index, entries):
            self.length[r] = len(toks)
            rows = torch.tensor([at + w for w in want], dtype=torch.long, device=e.dev)
            out[i] = e._head(hidden[rows]).float() if want else self._none()
            at += len(toks)

    def _advance(self, pairs):
        e = self.e
        grown = 0
        for r, _ in pairs:
            grown += e.sched.grow(self.slot[r], self.length[r] + 1, e.block_table_host.numpy())
        if grown:
            e.block_table.copy_(e.block_table_host)
        slots = torch.tensor([self.slot[r] for r, _ in pairs], device=e.dev)
        e.seq_lens.fill_(-1)
        e.seq_lens[slots] = torch.tensor([self.length[r] for r, _ in pairs], dtype=torch.int32, device=e.dev)
        e.next_input[slots] = torch.tensor([t for _, t in pairs], dtype=torch.int64, device=e.dev)
        logits = e._decode_logits()
        for r, _ in pairs:
            self.length[r] += 1
        return logits

    def release(self, r):
        slot = self.slot.pop(r)
        self.length.pop(r)
        rid = self._rid.pop(r)
        self.e.sched.retire(slot, rid)
        self.e.seq_lens[slot] = -1

    @property
    def live(self) -> int:
        return len(self.slot)
