"""Generation: sequences of a model in slots, prompts in portions, one token per step after that.

A model brings ``state_parts()``, ``capacity``, ``vocab``, ``stream``, ``lib`` and
``step(seq, tokens, want, logits)``, and ``portion`` if a step takes no more tokens than that; the engine is
the same for every family.  A step runs one sequence:
the next portion of its prompt or its last token.  Live requests take turns.
"""
from collections import deque
from dataclasses import dataclass, field

import numpy as np

from .sequences import SequenceSlots


@dataclass
class Request:
    prompt: list
    max_new_tokens: int
    stop: frozenset = frozenset()
    output: list = field(default_factory=list)
    fed: int = 0              # prompt tokens that have been run
    key: object = None


class Engine:
    def __init__(self, model, slots=1, portion=2048):
        if portion < 1:
            raise ValueError("a portion has at least one token")
        self.model, self.portion = model, min(portion, getattr(model, "portion", portion))
        self.slots = SequenceSlots(model.lib, model.state_parts(), model.capacity, slots, model.stream)
        self.live = {}        # key -> Sequence

    # ---- sequences by key
    def feed(self, key, tokens, want=(), logits=True):
        """Runs the next tokens of sequence `key` (a new key starts a sequence), in portions if there are many; returns
        (logits at the wanted places or None, greedy token ids there)."""
        seq = self.live.get(key)
        if seq is None:
            seq = self.slots.acquire()
            if seq is None:
                raise RuntimeError("every sequence slot is in use")
            self.live[key] = seq
        tokens, want = np.asarray(tokens, np.int32), np.asarray(want, np.int64)
        if want.size and (want.min() < 0 or want.max() >= tokens.size):
            raise ValueError(f"wanted places {want.min()} .. {want.max()} of {tokens.size} tokens")
        out = np.empty((want.size, self.model.vocab), np.float32) if logits else None
        picked = np.empty(want.size, np.int64)
        for at in range(0, tokens.size, self.portion):
            part = tokens[at:at + self.portion]
            idx = np.flatnonzero((want >= at) & (want < at + part.size))
            lg, ids = self.model.step(seq, part, want[idx] - at, logits)
            picked[idx] = ids
            if logits:
                out[idx] = lg
        return out, picked

    def end(self, key):
        """The sequence is finished; its slot is free again."""
        self.slots.release(self.live.pop(key))

    # ---- requests
    def _advance(self, r):
        """One step of a request; true when it is finished."""
        if r.fed < len(r.prompt):
            part = r.prompt[r.fed:r.fed + self.portion]
            last = r.fed + len(part) == len(r.prompt)
            _, ids = self.feed(r.key, part, [len(part) - 1] if last else [], logits=False)
            r.fed += len(part)
            if not last:
                return False
        else:
            _, ids = self.feed(r.key, r.output[-1:], [0], logits=False)
        r.output.append(int(ids[0]))
        return len(r.output) >= r.max_new_tokens or r.output[-1] in r.stop

    def run(self, requests):
        """Greedy generation of all requests, oldest first into free slots; fills their `output`."""
        for i, r in enumerate(requests):
            r.key = ("request", i)
            if not len(r.prompt) or r.max_new_tokens < 1:
                raise ValueError("a request needs a prompt and at least one new token")
            if len(r.prompt) + r.max_new_tokens - 1 > self.model.capacity:
                raise ValueError(f"{len(r.prompt)} + {r.max_new_tokens} tokens do not fit a sequence of {self.model.capacity}")
        waiting, running = deque(requests), deque()
        while waiting or running:
            while waiting and self.slots.free:
                running.append(waiting.popleft())
                self._start(running[-1])
            r = running.popleft()
            if self._advance(r):
                self.end(r.key)
            else:
                running.append(r)
        return requests

    def _start(self, r):
        self.live[r.key] = self.slots.acquire()

    def generate(self, prompts, max_new_tokens, stop=()):
        """Greedy continuation of every prompt: a list of token lists."""
        return [r.output for r in self.run([Request(list(p), max_new_tokens, frozenset(stop)) for p in prompts])]

    def close(self):
        self.slots.close()
