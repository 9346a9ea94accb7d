"""Which tokens the next step runs: admission, prompt portions and decoding of many requests over one page pool."""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field

from .paging import PagePool, Sequence


@dataclass
class Request:
    id: object
    prompt: list[int]
    max_new: int
    stop: frozenset = frozenset()
    output: list[int] = field(default_factory=list)
    seq: Sequence = field(default_factory=Sequence)

    @property
    def tokens(self) -> list[int]:
        return self.prompt + self.output

    @property
    def pending(self) -> int:
        """Tokens that are known and not yet in the cache: one while decoding, more while (re)reading a prompt."""
        return len(self.prompt) + len(self.output) - self.seq.length

    @property
    def finished(self) -> bool:
        return len(self.output) >= self.max_new or bool(self.output and self.output[-1] in self.stop)


class Scheduler:
    """Every step first continues the running requests, oldest first: one token of those that decode, the next portion of
    those whose prompt is not all in; then admits waiting ones while rows, sequences and pages are left.  When a running
    request cannot get a page, the youngest one gives its pages back and waits to be read again."""

    def __init__(self, pool: PagePool, *, block_size: int, max_tokens: int, max_sequences: int, window: int | None = None, keep_first: int = 0):
        self.pool, self.block_size, self.window, self.keep_first = pool, block_size, window, keep_first
        self.max_tokens, self.max_sequences = max_tokens, max_sequences
        self.waiting: deque[Request] = deque()
        self.running: list[Request] = []

    def add(self, request: Request) -> None:
        if not request.prompt:
            raise ValueError(f"request {request.id!r} has no tokens")
        self.waiting.append(request)

    @property
    def idle(self) -> bool:
        return not self.waiting and not self.running

    def plan(self) -> list[tuple[Request, list[int]]]:
        """[(request, tokens)] of the next step, pages reserved."""
        work, rows = [], self.max_tokens
        # decoding rows first, so that a long prompt never holds them up
        for r in sorted(self.running, key=lambda r: r.pending > 1):
            if rows == 0:
                break
            if r not in self.running:
                continue  # preempted for an older request of this very step
            while (n := self._fitting(r, rows)) < 1:
                victim = next((v for v in reversed(self.running) if v is not r and all(v is not w for w, _ in work)), None)
                if victim is None:
                    break
                self._preempt(victim)
            if n > 0:
                r.seq.reserve(self.pool, n, self.block_size)
                work.append((r, r.tokens[r.seq.length:r.seq.length + n]))
                rows -= n
        while self.waiting and rows > 0 and len(self.running) < self.max_sequences:
            r = self.waiting[0]
            n = self._fitting(r, rows)
            if n < 1 or (self.running and self._room(r) < r.pending):
                break  # beside running requests one is admitted only if all of its tokens fit: it would soon be sent back
            r.seq.reserve(self.pool, n, self.block_size)
            self.waiting.popleft()
            self.running.append(r)
            work.append((r, r.tokens[:n]))
            rows -= n
        if not work and not self.idle:
            raise RuntimeError("no request fits the page pool: it is too small for a single sequence of this length")
        return work

    def _fitting(self, r: Request, rows: int) -> int:
        """How many of the request's pending tokens the rows and the free pages take."""
        return min(r.pending, rows, self._room(r))

    def _room(self, r: Request) -> int:
        if r.seq.length == 0 and not r.seq.pages and not self.pool.has_state:
            return 0
        return (len(r.seq.pages) + self.pool.free_count) * self.block_size - r.seq.length

    def _preempt(self, r: Request) -> None:
        r.seq.release(self.pool)
        self.running.remove(r)
        self.waiting.appendleft(r)

    def advance(self, seq: Sequence, n: int) -> None:
        """The cache now holds n more tokens; pages no window reaches any more go back (those of the kept first tokens stay)."""
        seq.length += n
        if self.window is not None:
            seq.drop_before(self.pool, seq.length - self.window + 1, self.block_size, self.keep_first)

    def finish(self, r: Request) -> None:
        r.seq.release(self.pool)
        self.running.remove(r)
