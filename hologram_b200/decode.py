"""Serving a decoder model: the step function over its `.holo` archives, the cache, sampling and the request queue.

A model's archives are fixed step shapes; `StepRunner` keeps one session per row count in use (powers of two, the
portion is padded up) and one per logit count. All of them share the first session's device copies of the weights
and its cache, state, residual stream and position buffers, and replay as CUDA graphs after their first walk. Padding rows
lie after the portion's last token: no real row sees them. What they leave in a plain cache is dropped past its end or
overwritten by a later step before any row can see it; ring caches and recurrent states take the real rows only, by the
row count every step carries, and a state starts from zero where the step's position is 0.
"""
from collections import deque

import numpy as np

from .session import InferenceSession


class CacheFull(RuntimeError):
    """A step or a request needs more positions than the cache has, or the cache belongs to another sequence."""


def bucket(n):
    """The step shape for n rows: the next power of two."""
    b = 1
    while b < n:
        b *= 2
    return b


class SequenceCache:
    """The positions one sequence at a time holds in the sessions' shared cache and state buffers."""

    def __init__(self, capacity):
        self.capacity = capacity
        self.owner, self.length = None, 0

    def acquire(self, owner):
        if self.owner is not None and self.owner != owner:
            raise CacheFull(f"the cache is held by sequence {self.owner!r}")
        if self.owner is None:
            self.owner, self.length = owner, 0

    def check(self, n):
        if self.length + n > self.capacity:
            raise CacheFull(f"{self.length} + {n} positions exceed the cache's {self.capacity}")

    def release(self, owner):
        if self.owner == owner:
            self.owner, self.length = None, 0


class StepRunner:
    """Runs portions of a sequence: `step(id, tokens, want)` appends the tokens and returns the logits at the wanted places."""

    LOGIT_ROWS = 256

    def __init__(self, backend, model, capacity, max_rows=2048, graphs=True):
        self.backend, self.model, self.graphs = backend, model, graphs
        self.cache = SequenceCache(capacity)
        self.max_rows = 1
        while self.max_rows < min(max_rows, capacity):
            self.max_rows *= 2
        self._steps, self._heads = {}, {}
        # the single-token step holds every weight: the other shapes borrow from it
        self._root = InferenceSession(backend, model.build_step(1, capacity, self.max_rows, True), verify=False)
        self._steps[1] = [self._root, False]

    def close(self):
        for table in (self._heads, self._steps):
            for n, (s, _) in list(table.items()):
                if s is not self._root:
                    s.close()
        self._root.close()
        self._steps, self._heads = {}, {}

    def _session(self, table, rows, build):
        if rows not in table:
            table[rows] = [InferenceSession(self.backend, build(), verify=False, donor=self._root), False]
        return table[rows]

    def _execute(self, entry):
        session, captured = entry
        session.execute()
        if self.graphs and not captured:       # the first walk allocated what it needs: later ones replay it
            session.capture()
            entry[1] = True
        return session

    def _run_rows(self, tokens, base, want):
        """One portion of at most max_rows tokens; logits of the wanted rows."""
        m = self.model
        rows = bucket(len(tokens))
        entry = self._session(self._steps, rows, lambda: m.build_step(rows, self.cache.capacity, self.max_rows, False, weightless=True))
        step_in = np.zeros(4 + rows, dtype=np.int32)
        step_in[0], step_in[1] = base, len(tokens)
        step_in[4:4 + len(tokens)] = tokens
        entry[0].write("step_in", step_in)
        session = self._execute(entry)
        vocab = m.config.vocab
        if rows == 1:
            return session.read("logits", np.float32).reshape(1, vocab)[:len(want)]
        out = np.empty((len(want), vocab), dtype=np.float32)
        for lo in range(0, len(want), self.LOGIT_ROWS):
            part = want[lo:lo + self.LOGIT_ROWS]
            n = bucket(len(part))
            head = self._session(self._heads, n, lambda: m.build_head(n, self.max_rows, weightless=True))
            index = np.zeros(n, dtype=np.int32)
            index[:len(part)] = part
            head[0].write("want", index)
            out[lo:lo + len(part)] = self._execute(head).read("logits", np.float32).reshape(n, vocab)[:len(part)]
        if not len(want):
            self.backend.synchronize()
        return out

    def step(self, seq, tokens, want=None):
        """Append `tokens` to sequence `seq` (it takes the cache if nobody holds it) and return f32 logits [wanted, vocab];
        `want` lists places among the tokens, the last one by default."""
        tokens = np.asarray(tokens, dtype=np.int32)
        if tokens.ndim != 1 or tokens.size == 0:
            raise ValueError("a step brings at least one token")
        if tokens.min() < 0 or tokens.max() >= self.model.config.vocab:
            raise ValueError("token id outside the vocabulary")
        want = [tokens.size - 1] if want is None else [int(i) for i in want]
        if any(not 0 <= i < tokens.size for i in want):
            raise ValueError("a wanted place lies outside the step's tokens")
        self.cache.acquire(seq)
        self.cache.check(tokens.size)
        out = np.empty((len(want), self.model.config.vocab), dtype=np.float32)
        for lo in range(0, tokens.size, self.max_rows):
            part = tokens[lo:lo + self.max_rows]
            mine = [k for k, i in enumerate(want) if lo <= i < lo + part.size]
            out[mine] = self._run_rows(part, self.cache.length, [want[k] - lo for k in mine])
            self.cache.length += part.size
        return out

    def end(self, seq):
        """Give back what the sequence holds."""
        self.cache.release(seq)


class Sampler:
    """Greedy at temperature 0, otherwise a seeded draw from the `top_k` (0 = all) most likely tokens."""

    def __init__(self, temperature=0.0, top_k=0, seed=0):
        self.temperature, self.top_k = temperature, top_k
        self.rng = np.random.default_rng(seed)

    def __call__(self, logits):
        if self.temperature <= 0.0:
            return int(np.argmax(logits))
        z = logits.astype(np.float64) / self.temperature
        if 0 < self.top_k < z.size:
            z[z < np.partition(z, -self.top_k)[-self.top_k]] = -np.inf
        p = np.exp(z - z.max())
        return int(self.rng.choice(z.size, p=p / p.sum()))


class Request:
    def __init__(self, prompt, max_new_tokens, sampler=None, stop=()):
        self.prompt, self.max_new_tokens, self.sampler, self.stop = list(prompt), max_new_tokens, sampler or Sampler(), frozenset(stop)
        self.tokens = []           # generated so far


class Scheduler:
    """Runs requests one after another over one StepRunner: the prompt in portions, then one token per step."""

    def __init__(self, runner, portion=None):
        self.runner, self.portion = runner, portion or runner.max_rows
        self.queue, self._next = deque(), 0

    def submit(self, request):
        if not request.prompt:
            raise ValueError("an empty prompt")
        if len(request.prompt) + request.max_new_tokens > self.runner.cache.capacity:
            raise CacheFull("the request does not fit the cache")
        self.queue.append((self._next, request))
        self._next += 1
        return self._next - 1

    def run(self):
        """Work the queue off; yields (request number, token) as tokens come."""
        while self.queue:
            seq, r = self.queue.popleft()
            try:
                for lo in range(0, len(r.prompt), self.portion):
                    part = r.prompt[lo:lo + self.portion]
                    logits = self.runner.step(seq, part, None if lo + len(part) == len(r.prompt) else [])
                while len(r.tokens) < r.max_new_tokens:
                    token = r.sampler(logits[0])
                    r.tokens.append(token)
                    yield seq, token
                    if token in r.stop or len(r.tokens) == r.max_new_tokens:
                        break
                    logits = self.runner.step(seq, [token])
            finally:
                self.runner.end(seq)


def generate(runner, prompt, max_new_tokens, sampler=None, stop=(), portion=None):
    """The continuation of one prompt."""
    scheduler = Scheduler(runner, portion)
    request = Request(prompt, max_new_tokens, sampler, stop)
    scheduler.submit(request)
    for _ in scheduler.run():
        pass
    return request.tokens
