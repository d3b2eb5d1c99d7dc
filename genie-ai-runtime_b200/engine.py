"""Requests over a model of the registry: a pool of sessions (one per live request, each with its own cache, all on the same
weights) that are taken, fed or generated on, and given back."""
from __future__ import annotations

from .registry import open_model


class Engine:
    def __init__(self, folder, dtype=None, max_context=4096):
        self.config, self._open = open_model(folder, dtype)
        self.max_context = max_context
        self._free, self._live = [], {}          # sessions; request id -> [session, tokens it holds]

    def _take(self):
        if self._free:
            return self._free.pop()
        return self._open(self.max_context)

    def _give_back(self, session):
        session.reset()
        self._free.append(session)

    def feed(self, request, tokens, want=()):
        """The request's next tokens; returns the logits at the wanted places among them, float32 [len(want), vocab].  A
        request starts with its first tokens."""
        if request not in self._live:
            self._live[request] = [self._take(), 0]
        entry = self._live[request]
        order = sorted(set(want))
        logits = entry[0].feed(tokens, entry[1], order)
        entry[1] += len(tokens)
        return logits if list(want) == order else logits[[order.index(w) for w in want]]

    def end(self, request):
        """Gives back what the request holds."""
        self._give_back(self._live.pop(request)[0])

    def generate(self, prompts, n_new):
        """Greedy continuation of each prompt (token ids), one request after the other; lists of n_new ids."""
        out = []
        for p in prompts:
            s = self._take()
            try:
                out.append([int(t) for t in s.generate(p, n_new)])
            finally:
                self._give_back(s)
        return out

    def close(self):
        for s in self._free + [e[0] for e in self._live.values()]:
            s.close()
        self._free, self._live = [], {}
