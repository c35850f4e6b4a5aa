"""Requests over the sequence slots of a session: a request takes a free slot with its first tokens and gives it back when it
ends; every step appends tokens to any of the live requests (a whole prompt, a portion of one, or the next token) in one call."""
from __future__ import annotations

import numpy as np


class RequestPool:
    def __init__(self, session):
        self.session = session
        self.slot = {}                                    # live request -> slot
        self.free = list(range(session.batch))[::-1]

    def _take(self, rid):
        if rid not in self.slot:
            if not self.free:
                raise RuntimeError(f"request {rid!r}: all {self.session.batch} slots are taken")
            self.slot[rid] = self.free.pop()
        return self.slot[rid]

    def step(self, entries):
        """entries: (request, tokens, places whose logits are wanted) in any order.  Returns one [places, vocab] array per entry."""
        tokens = [[] for _ in range(self.session.batch)]
        want = [[] for _ in range(self.session.batch)]
        slots = []
        for rid, toks, places in entries:
            s = self._take(rid)
            if tokens[s]:
                raise ValueError(f"request {rid!r} appears twice in one step")
            tokens[s], want[s] = list(toks), list(places)
            slots.append(s)
        logits = self.session.extend(tokens, want)
        first = np.concatenate([[0], np.cumsum([len(w) for w in want])])
        return [logits[first[s]:first[s + 1]] for s in slots]

    def end(self, rids):
        """The requests are finished: their slots go back to position 0 and are free."""
        rids = [r for r in rids if r in self.slot]
        if not rids:
            return
        pos = self.session.positions()
        for r in rids:
            s = self.slot.pop(r)
            pos[s] = 0
            self.free.append(s)
        self.session.set_positions(pos)

    def generate(self, prompts, max_new, eot=None):
        """Greedy generation of many requests over the slots there are: {request: prompt ids} -> {request: new ids}.  A request
        waits for a slot, its prompt and the other requests' next tokens share steps, and it ends after max_new tokens or `eot`."""
        waiting, nxt, out = list(prompts), {}, {r: [] for r in prompts}
        while waiting or nxt:
            entries = [(r, [t], [0]) for r, t in nxt.items()]
            while waiting and len(entries) < self.session.batch:
                r = waiting.pop(0)
                entries.append((r, prompts[r], [len(prompts[r]) - 1]))
            done = []
            for (r, _, _), logits in zip(entries, self.step(entries)):
                t = int(np.argmax(logits[0]))
                out[r].append(t)
                nxt[r] = t
                if len(out[r]) >= max_new or t == eot:
                    done.append(r)
                    del nxt[r]
            self.end(done)
        return out
