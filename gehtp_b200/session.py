"""Serving a row-count runlist: one sequence at a time lives in the engine's states; tokens are fed in portions, the
states carry on from run to run, a finished request gives its states back before the next begins."""
from collections import deque
from dataclasses import dataclass, field

import numpy as np

from .wtop import Engine


class Session:
    def __init__(self, model, dtype="bfloat16", max_tokens=2048, max_rows=2048, max_sel=64, lib=None):
        if lib is None:
            from . import lib as load
            lib = load()
        blob, self.man = model.runlist(dtype, max_tokens, max_rows, max_sel)
        self.engine = Engine(lib, blob)
        self.vocab = self.man["vocab"]
        self._face = np.zeros(self.man["max_rows"] + self.man["max_sel"], np.int32)
        self.reset()

    def reset(self):
        """Gives the states back: the next token is at position 0."""
        self.engine.state_reset()
        self.position = 0

    def close(self):
        self.engine.shutdown()

    def _run(self, tokens, sel, out_temp, out):
        n = len(tokens)
        self._face[:n] = tokens
        self._face[self.man["max_rows"]:self.man["max_rows"] + len(sel)] = sel
        self.engine.set_rows(n, len(sel))
        self.engine.run_io(self._face, out_temp, out)
        self.position += n

    def _check(self, tokens):
        t = np.asarray(tokens, np.int64)
        if t.ndim != 1 or t.size == 0:
            raise ValueError("no tokens")
        if t.min() < 0 or t.max() >= self.vocab:
            raise ValueError("token id outside the vocabulary")
        if self.position + t.size > self.man["nslots"]:
            raise ValueError("%d positions, the cache holds %d" % (self.position + t.size, self.man["nslots"]))
        return t.astype(np.int32)

    def _portions(self, n, want):
        """Cuts n tokens into runs of at most max_rows rows and max_sel wanted rows: (first, end, wanted in it)."""
        lo, k = 0, 0
        while lo < n:
            hi = min(lo + self.man["max_rows"], n)
            j = k
            while j < len(want) and want[j] < hi:
                if j - k == self.man["max_sel"]:
                    hi = want[j]
                    break
                j += 1
            yield lo, hi, want[k:j]
            lo, k = hi, j

    def feed(self, tokens, want=()):
        """Runs the next tokens of the sequence; logits [len(want), vocab] (fp32) at the wanted places among them."""
        t = self._check(tokens)
        order = sorted(set(int(w) for w in want))
        if order and not (0 <= order[0] and order[-1] < len(t)):
            raise ValueError("a wanted place lies outside the tokens")
        got = {}
        for lo, hi, sel in self._portions(len(t), order):
            out = np.empty((len(sel), self.vocab), np.float32) if sel else None
            self._run(t[lo:hi], [w - lo for w in sel], self.man["logits_temp"], out)
            got.update(zip(sel, out if sel else ()))
        return np.stack([got[int(w)] for w in want]) if len(want) else np.empty((0, self.vocab), np.float32)

    def choose(self, tokens):
        """Runs the next tokens; the greedy continuation of the last one, chosen on the device."""
        t = self._check(tokens)
        out = np.empty(1, np.int32)
        for lo, hi, sel in self._portions(len(t), [len(t) - 1]):
            self._run(t[lo:hi], [w - lo for w in sel], self.man["token_temp"], out if sel else None)
        return int(out[0])

    def generate(self, prompt, max_new, stop=()):
        """Greedy continuation of a prompt, from position 0."""
        self.reset()
        out, nxt = [], prompt
        while len(out) < max_new:
            tok = self.choose(nxt)
            out.append(tok)
            if tok in stop or self.position >= self.man["nslots"]:
                break
            nxt = [tok]
        return out


@dataclass
class Request:
    id: object
    prompt: list
    max_new: int
    stop: tuple = ()
    tokens: list = field(default_factory=list)
    error: str = None


class Scheduler:
    """First come, first served: the engine's states hold one sequence, so requests run to their end in order."""

    def __init__(self, session):
        self.session, self.queue = session, deque()

    def submit(self, request):
        self.queue.append(request)

    def run(self):
        """Serves every queued request and returns them in the order they were submitted; a request the session
        refuses (ids outside the vocabulary, prompt longer than the cache) carries its error and holds up no other."""
        done = []
        while self.queue:
            r = self.queue.popleft()
            try:
                r.tokens = self.session.generate(r.prompt, r.max_new, r.stop)
            except ValueError as e:
                r.error = str(e)
            finally:
                self.session.reset()
            done.append(r)
        return done
