"""What every model of the framework is to the engine: static device inputs, one step over a ragged set of tokens, CUDA
graphs of the steps that repeat, greedy next tokens.

A step is a flat list of token rows.  Each row has its own position, cache slot, visible length and block table; rows of one
sequence are consecutive and in order, and every row's cache entry is written before any row of the same layer attends, so a
prompt portion of any length, a decode batch and a mix of the two are the same call (`run`).
"""
from __future__ import annotations

import numpy as np
import torch

from . import _native as N
from . import ops
from .paging import PADDING_LENGTH, PADDING_PAGE, PADDING_SLOT, RaggedStep


class StepModel:
    """Base of the models.  A subclass computes a step over the input buffers in `_run_step(rows)`, leaving `logits[:rows]`
    and `next_ids[:rows]`."""

    window: int | None = None  # no row attends further back than this many positions (itself included); None: unbounded

    def __init__(self, rows: int, tables: int, num_blocks: int, max_blocks_per_seq: int, block_size: int, vocab: int, device):
        self.rows, self.device, self.vocab = rows, torch.device(device), vocab
        self.num_blocks, self.max_blocks, self.block_size = num_blocks, max_blocks_per_seq, block_size
        self.max_tokens = rows       # the most token rows of one step
        self.max_sequences = tables  # the most sequences of one step
        i32 = dict(dtype=torch.int32, device=self.device)
        # step inputs (static addresses: the CUDA graphs read them)
        self.token_ids = torch.zeros((rows,), **i32)
        self.positions = torch.zeros((rows,), **i32)
        self.block_tables = torch.zeros((tables, max_blocks_per_seq), **i32)
        self.seq_lens = torch.ones((rows,), **i32)
        self.slot_mapping = torch.full((rows,), PADDING_SLOT, **i32)
        self._graphs: dict[int, torch.cuda.CUDAGraph] = {}

    def _run_step(self, rows: int) -> None:
        raise NotImplementedError

    def set_inputs(self, token_ids, positions, block_tables, seq_lens, slot_mapping) -> None:
        """Host (NumPy or pinned torch) step inputs -> the device buffers the graph reads."""
        for dst, src in ((self.token_ids, token_ids), (self.positions, positions), (self.block_tables, block_tables),
                         (self.seq_lens, seq_lens), (self.slot_mapping, slot_mapping)):
            self._put(dst, src)

    @staticmethod
    def _put(dst: torch.Tensor, src) -> None:
        if src is None:
            return
        if isinstance(src, np.ndarray):
            src = torch.from_numpy(np.ascontiguousarray(src, dtype=np.int32))
        dst.copy_(src.reshape(dst.shape), non_blocking=True)

    def capture(self, rows: int | None = None) -> None:
        """Capture the step over `rows` rows into a CUDA graph (after one eager warm-up step on a side stream)."""
        rows = self.rows if rows is None else rows
        s = torch.cuda.Stream(device=self.device)
        s.wait_stream(torch.cuda.current_stream(self.device))
        with torch.cuda.stream(s):
            self._run_step(rows)
        torch.cuda.current_stream(self.device).wait_stream(s)
        torch.cuda.synchronize(self.device)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            self._run_step(rows)
        self._graphs[rows] = graph

    def step(self, rows: int | None = None) -> torch.Tensor:
        """One step over the current inputs; returns the device tensor of next token ids [rows]."""
        rows = self.rows if rows is None else rows
        graph = self._graphs.get(rows)
        if graph is not None:
            graph.replay()
        else:
            self._run_step(rows)
        return self.next_ids[:rows]

    def run(self, step: RaggedStep, want) -> torch.Tensor:
        """Runs the step's tokens; returns the f32 logits [len(want), vocab] of the rows named in `want` (device tensor,
        valid until the next step)."""
        raise NotImplementedError

    def device_status(self) -> int:
        """Nonzero if a bounded wait inside a kernel ran out since the last read: results since then are not valid."""
        return N.lib().tlaloc_b200_device_status()

    def greedy(self, logits: torch.Tensor) -> torch.Tensor:
        """First maximum of every row of logits, int32 on the device."""
        return ops.argmax(logits)

    def _padded(self, step: RaggedStep, rows: int):
        """The step's inputs with every row carrying its own block table, padded to `rows` rows: slot -1, length 1, page 0."""
        n = step.token_ids.shape[0]
        if n > rows:
            raise ValueError(f"{n} tokens do not fit a step of {rows} rows")

        def pad(a, fill):
            out = np.full((rows,), fill, np.int32)
            out[:n] = a
            return out

        tables = np.full((rows, self.max_blocks), PADDING_PAGE, np.int32)
        tables[:n] = step.block_tables[step.row_tables]
        return (pad(step.token_ids, 0), pad(step.positions, 0), tables, pad(step.seq_lens, PADDING_LENGTH),
                pad(step.slot_mapping, PADDING_SLOT))
