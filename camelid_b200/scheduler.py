"""Requests onto the slots of an engine: who holds which slot, prompt portions, batched decode steps, sampling.

Works with any ``TokenEngine``.  A request takes a slot when one is free, its prompt goes in by portions, then it decodes
together with the others, one row per request, until it has its tokens; the slot goes to the next request as it is (an
engine starts a sequence from nothing at position 0)."""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field


class SlotTable:
    """Sequence slots by request id, and how many tokens each request has fed."""

    def __init__(self, n_slots: int):
        self._free = deque(range(n_slots))
        self._slot: dict = {}
        self._length: dict = {}

    def __contains__(self, rid) -> bool:
        return rid in self._slot

    def __len__(self) -> int:
        return len(self._slot)

    @property
    def free(self) -> int:
        return len(self._free)

    def acquire(self, rid) -> int:
        if rid in self._slot:
            raise ValueError(f"request {rid!r} already holds a slot")
        if not self._free:
            raise RuntimeError(f"no free slot for request {rid!r}: {len(self._slot)} requests are live")
        self._slot[rid] = self._free.popleft()
        self._length[rid] = 0
        return self._slot[rid]

    def slot(self, rid) -> int:
        return self._slot[rid]

    def length(self, rid) -> int:
        return self._length[rid]

    def advance(self, rid, n: int):
        self._length[rid] += n

    def release(self, rid):
        self._free.append(self._slot.pop(rid))
        del self._length[rid]


@dataclass
class Request:
    rid: object
    prompt: list
    max_new: int
    temperature: float = 0.0  # 0: greedy
    min_p: float = 0.0
    seed: int = 0
    stop: frozenset = frozenset()
    out: list = field(default_factory=list)

    def done(self) -> bool:
        return len(self.out) >= self.max_new or (bool(self.out) and self.out[-1] in self.stop)


class Scheduler:
    def __init__(self, engine, portion: int = 0, greedy_run: int = 32):
        """portion: most prompt tokens of one request per turn (0: the whole prompt).  greedy_run: most decode steps handed
        to the engine at once while every live request is greedy and nobody waits for a slot."""
        self.engine, self.portion, self.greedy_run = engine, portion, greedy_run
        self.slots = SlotTable(engine.cfg.max_seqs)
        self.waiting: deque = deque()
        self.filling: list = []   # hold a slot, prompt not yet complete
        self.live: list = []      # decoding
        self.finished: dict = {}

    def submit(self, rid, prompt, max_new: int, temperature: float = 0.0, min_p: float = 0.0, seed: int = 0, stop=()):
        prompt = [int(t) for t in prompt]
        if not prompt or max_new < 1:
            raise ValueError("a request needs a prompt and at least one new token")
        if len(prompt) + max_new - 1 > self.engine.cfg.max_pos:
            raise ValueError(f"{len(prompt)} + {max_new} tokens exceed the engine's {self.engine.cfg.max_pos} positions")
        self.waiting.append(Request(rid, prompt, max_new, temperature, min_p, seed, frozenset(stop)))

    def _draw(self, r: Request, row: int, greedy: int) -> int:
        if r.temperature <= 0:
            return greedy
        tok = self.engine.sample(r.temperature, r.seed + len(r.out), r.min_p, row)
        return greedy if tok is None else tok  # the filter left it undecided: take the best token

    def _retire(self, r: Request):
        self.slots.release(r.rid)
        self.finished[r.rid] = r.out

    def turn(self) -> bool:
        """One turn: admissions, a portion of every unfinished prompt, one batched decode step (or several, all greedy).
        False when there is nothing left to do."""
        while self.waiting and self.slots.free:
            r = self.waiting.popleft()
            self.slots.acquire(r.rid)
            self.filling.append(r)
        for r in list(self.filling):
            at = self.slots.length(r.rid)
            part = r.prompt[at:at + self.portion] if self.portion else r.prompt[at:]
            nxt, _ = self.engine.extend(self.slots.slot(r.rid), part, at)
            self.slots.advance(r.rid, len(part))
            if at + len(part) == len(r.prompt):
                r.out.append(self._draw(r, -1, nxt))
                self.filling.remove(r)
                if r.done():
                    self._retire(r)
                else:
                    self.live.append(r)
        if self.live:
            seqs = [self.slots.slot(r.rid) for r in self.live]
            toks = [r.out[-1] for r in self.live]
            pos = [self.slots.length(r.rid) for r in self.live]
            steps = min(self.greedy_run, min(r.max_new - len(r.out) for r in self.live))
            if steps > 1 and not self.waiting and not self.filling and all(r.temperature <= 0 for r in self.live):
                got = self.engine.decode_greedy(seqs, toks, pos, steps)
                for i, r in enumerate(self.live):
                    for t in got[:, i]:
                        if not r.done():
                            r.out.append(int(t))
                    self.slots.advance(r.rid, steps)
            else:
                got, _, _ = self.engine.step_batch(seqs, toks, pos)
                for i, r in enumerate(self.live):
                    r.out.append(self._draw(r, i, int(got[i])))
                    self.slots.advance(r.rid, 1)
            for r in [r for r in self.live if r.done()]:
                self.live.remove(r)
                self._retire(r)
        return bool(self.waiting or self.filling or self.live)

    def run(self) -> dict:
        """Until every request is finished: id -> generated tokens."""
        while self.turn():
            pass
        return self.finished
