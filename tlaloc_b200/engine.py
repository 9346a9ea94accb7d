"""Serving over one model: sequences that are fed tokens step by step, and greedy generation of many requests.

Both run the model's one step function over the same paged cache: `Engine.feed` for a caller that brings the tokens, `Engine.generate` with
the scheduler choosing them.
"""
from __future__ import annotations

import torch

from .paging import PagePool, Sequence, stage_ragged
from .scheduler import Request, Scheduler
from .step_model import StepModel


class Engine:
    def __init__(self, model: StepModel):
        self.model = model
        self.pool = PagePool(model.num_blocks, model.num_states)
        self.scheduler = Scheduler(self.pool, block_size=model.block_size, max_tokens=model.max_tokens, max_sequences=model.max_sequences,
                                   window=model.window, keep_first=model.keep_first)
        self.sequences: dict[object, Sequence] = {}

    # ------------------------------------------------------------------ token by token

    def _run(self, work, want) -> torch.Tensor:
        """work [(sequence, tokens)] with pages reserved; want: flat token rows.  Logits of those rows."""
        logits = self.model.run(stage_ragged(work, max_blocks=self.model.max_blocks, block_size=self.model.block_size), want)
        for seq, tokens in work:
            self.scheduler.advance(seq, len(tokens))
        return logits

    def feed(self, entries) -> list[torch.Tensor]:
        """entries [(id, tokens, want)]: the next tokens of each sequence (a new id opens one) and the places among them whose
        logits are asked for.  Returns one f32 tensor [len(want), vocab] on the host per entry.  More tokens than a step takes run in
        several steps."""
        out = []  # (reading the logits waits for the step, so the status read below costs no wait of its own)
        for key, tokens, want in entries:
            seq = self.sequences.setdefault(key, Sequence())
            rows = []
            for lo in range(0, len(tokens), self.model.max_tokens):
                part = tokens[lo:lo + self.model.max_tokens]
                if not seq.reserve(self.pool, len(part), self.model.block_size):
                    raise RuntimeError(f"sequence {key!r}: no pages (or no state slot) left for {len(part)} more tokens")
                rows.append(self._run([(seq, part)], [w - lo for w in want if lo <= w < lo + len(part)]).cpu())
            out.append(torch.cat(rows) if rows else torch.empty((0, self.model.vocab)))
        self._check()
        return out

    def _check(self) -> None:
        if self.model.device_status() != 0:
            raise RuntimeError("a wait inside a kernel ran out: the results of this step are not valid")

    def close(self, key) -> None:
        """The sequence is finished; its pages and its state slot go back."""
        self.sequences.pop(key).release(self.pool)

    # ------------------------------------------------------------------ generation

    def step(self) -> list[Request]:
        """One scheduled step; returns the requests it finished."""
        work = self.scheduler.plan()
        if not work:
            return []
        want, rows, ends = [], 0, []
        for r, tokens in work:
            rows += len(tokens)
            if r.pending == len(tokens):  # its last known token runs now: the next one comes out
                want.append(rows - 1)
                ends.append(r)
        logits = self._run([(r.seq, tokens) for r, tokens in work], want)
        done = []
        if want:
            for r, token in zip(ends, self.model.greedy(logits).tolist()):
                r.output.append(int(token))
                if r.finished:
                    self.scheduler.finish(r)
                    done.append(r)
        return done

    def generate(self, prompts, max_new: int, stop=()) -> list[list[int]]:
        """Greedy continuations of `prompts` (lists of token ids), `max_new` tokens each or up to a stop token."""
        requests = [Request(i, list(p), max_new, frozenset(stop)) for i, p in enumerate(prompts)]
        for r in requests:
            if not r.prompt or len(r.prompt) + max_new > self.model.max_blocks * self.model.block_size:
                raise ValueError(f"prompt {r.id}: {len(r.prompt)} + {max_new} tokens; this engine takes 1 to "
                                 f"{self.model.max_blocks * self.model.block_size}")
            if max_new > 0:
                self.scheduler.add(r)
        while not self.scheduler.idle:
            self.step()
        self._check()
        return [r.output for r in requests]
