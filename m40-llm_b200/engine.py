"""Request scheduler over a host.Model: admits requests to free sequence slots, runs prompts in portions mixed with the
decode rows of requests already running, and switches to graph-replayed bursts when every running request decodes.

The decode rows of a step come from the host library's batch plan (src/decode_batch.rs:143-230); sampling is greedy on the
device (src/sampling.rs:95-108).
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field

from . import host


@dataclass
class Request:
    id: int
    prompt: list[int]
    max_new: int
    stop: int | None = None
    slot: int = -1
    fed: int = 0                              # prompt tokens already run
    out: list[int] = field(default_factory=list)

    @property
    def done(self) -> bool:
        return len(self.out) >= self.max_new or (self.stop is not None and bool(self.out) and self.out[-1] == self.stop)


class Engine:
    def __init__(self, model: host.Model, portion: int = 512, burst: int = 32):
        self.model, self.portion, self.burst = model, portion, burst
        self.waiting: deque[Request] = deque()
        self.running: list[Request] = []
        self.finished: dict[int, list[int]] = {}
        self._next_id = 0

    def submit(self, prompt, max_new: int, stop: int | None = None) -> int:
        prompt = [int(t) for t in prompt]
        if not prompt or max_new < 1:
            raise ValueError("a request needs a prompt and at least one new token")
        self._next_id += 1
        self.waiting.append(Request(self._next_id, prompt, max_new, stop))
        return self._next_id

    def _admit(self):
        while self.waiting and len(self.running) < self.model.sequences:
            r = self.waiting.popleft()
            r.slot = self.model.acquire()
            self.running.append(r)

    def _retire(self):
        for r in [r for r in self.running if r.done]:
            self.model.release(r.slot)
            self.running.remove(r)
            self.finished[r.id] = r.out

    def step(self) -> bool:
        """One scheduling step; False when nothing is left to do."""
        self._admit()
        if not self.running:
            return False
        by_id = {r.id: r for r in self.running}
        decoding = [r for r in self.running if r.fed == len(r.prompt)]
        rows = []
        if decoding:
            # a request's last token is not in the cache yet: its length including it is length + 1
            _, _, ids = host.plan_from_requests([(r.id, r.slot, self.model.length(r.slot) + 1, r in decoding)
                                                 for r in self.running])
            rows = [by_id[int(i)] for i in ids]
        prompts = [r for r in self.running if r.fed < len(r.prompt)]
        if not prompts and all(r.stop is None for r in rows):
            n = min([self.burst] + [r.max_new - len(r.out) for r in rows])
            self.model.begin_sequences([r.slot for r in rows], [r.out[-1] for r in rows])
            ids, _ = self.model.generate(n)
            for j, r in enumerate(rows):
                r.out += [int(t) for t in ids[:, j]]
        else:
            entries, want, owners, at, room = [], [], [], 0, self.portion
            for r in rows:
                entries.append((r.slot, [r.out[-1]]))
                want.append(at)
                owners.append(r)
                at += 1
            for r in prompts:
                n = min(room, len(r.prompt) - r.fed)
                if n == 0:
                    break
                entries.append((r.slot, r.prompt[r.fed:r.fed + n]))
                r.fed += n
                at += n
                room -= n
                if r.fed == len(r.prompt):
                    want.append(at - 1)
                    owners.append(r)
            got = self.model.step(entries, want, want_logits=False, want_next=True)["next"]
            for r, t in zip(owners, got):
                r.out.append(int(t))
        self._retire()
        return bool(self.running or self.waiting)

    def run(self) -> dict[int, list[int]]:
        """Runs everything submitted; returns {request id: generated ids}."""
        while self.step():
            pass
        out, self.finished = self.finished, {}
        return out
