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
from .paging import PADDING_LENGTH, PADDING_PAGE, PADDING_SLOT, PADDING_STATE, RaggedStep


class StepModel:
    """Base of the models.  A subclass computes a step over the input buffers in `_run_step(rows)`, leaving `logits[:rows]`
    and `next_ids[:rows]`."""

    window: int | None = None  # no row attends further back than this many positions (itself included); None: unbounded
    keep_first: int = 0        # ... except to this many first positions
    num_states: int = 0        # state slots of a model with recurrent layers: sequences it can hold at a time

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


class RaggedModel(StepModel):
    """A model whose step takes ragged rows: every row names its block table and its state slot.  A subclass computes the residual
    stream of rows [0, n) in `x` (`_hidden`) and the logits of rows of it (`_head`, into `logits`)."""

    def __init__(self, *, width: int, dtype: torch.dtype, max_tokens: int, max_sequences: int, num_blocks: int, max_len: int,
                 block_size: int, vocab: int, device):
        if not torch.cuda.is_available():
            raise RuntimeError(f"tlaloc_b200.{type(self).__name__} needs a CUDA device: there is no CPU path")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"{type(self).__name__} runs in bfloat16 or float32, not {dtype}")
        max_blocks = -(-max_len // block_size)
        super().__init__(max(max_tokens, max_sequences), max_sequences, num_blocks, max_blocks, block_size, vocab, device)
        self.dtype, self.max_positions = dtype, max_blocks * block_size
        ops.init()
        dev, i32 = self.device, dict(dtype=torch.int32, device=self.device)
        self.row_tables = torch.zeros((self.rows,), **i32)
        self.row_states = torch.zeros((self.rows,), **i32)
        self.x = torch.empty((self.rows, width), dtype=torch.float32, device=dev)
        self.hn = torch.empty((self.rows, width), dtype=dtype, device=dev)
        self.logits = torch.empty((max_sequences, vocab), dtype=torch.float32, device=dev)
        self.next_ids = torch.zeros((max_sequences,), **i32)
        self._decode_uses: dict[int, int] = {}

    def _hidden(self, n: int, spans=None, trace: list | None = None) -> None:
        """Embedding and layers over rows [0, n) of the step inputs; the residual stream stays in x.  spans: [(first row, end row,
        table row, position of the first)], the rows of each sequence; None: one row per sequence.  trace: receives a copy of
        the residual stream after every layer."""
        raise NotImplementedError

    def _head(self, x: torch.Tensor) -> torch.Tensor:
        """Logits of rows of the residual stream: a view of `logits`."""
        raise NotImplementedError

    def _run_step(self, rows: int) -> None:
        """One token of `rows` sequences: row r uses block table r."""
        self._hidden(rows)
        ops.argmax(self._head(self.x[:rows]), out=self.next_ids[:rows])

    def run(self, step: RaggedStep, want, trace: list | None = None) -> torch.Tensor:
        n, s = step.token_ids.shape[0], step.block_tables.shape[0]
        if n > self.max_tokens or s > self.max_sequences:
            raise ValueError(f"a step of {n} tokens of {s} sequences; this model takes {self.max_tokens} of {self.max_sequences}")
        if n == s and trace is None:
            return self._run_decode(step, want)
        self._inputs(step)
        self._hidden(n, [(int(a), int(b), r, int(step.positions[a])) for r, (a, b) in enumerate(zip(step.starts[:-1], step.starts[1:]))], trace)
        out = []
        for k in range(0, len(want), self.max_sequences):
            rows = torch.as_tensor(np.asarray(want[k:k + self.max_sequences], np.int32), device=self.device)
            out.append(self._head(ops.embedding(self.x[:n], rows)))
            if len(want) > self.max_sequences:
                out[-1] = out[-1].clone()
        return torch.cat(out) if len(out) > 1 else out[0] if out else self.logits[:0]

    def _inputs(self, step: RaggedStep) -> None:
        for dst, src in ((self.token_ids, step.token_ids), (self.positions, step.positions), (self.seq_lens, step.seq_lens),
                         (self.slot_mapping, step.slot_mapping), (self.row_tables, step.row_tables), (self.row_states, step.row_states),
                         (self.block_tables, step.block_tables)):
            self._put(dst[:src.shape[0]], src)

    def _run_decode(self, step: RaggedStep, want) -> torch.Tensor:
        """One token of every sequence: the batch is padded to a power of two, and a size that comes up again is captured into a
        CUDA graph (padding rows write nothing a sequence reads and attend over the padding page)."""
        n = step.token_ids.shape[0]
        rows = min(1 << (n - 1).bit_length(), self.max_sequences)
        self._decode_uses[rows] = self._decode_uses.get(rows, 0) + 1
        if self._decode_uses[rows] == 3 and rows not in self._graphs:
            zeros = np.zeros((rows,), np.int32)  # the warm-up step of a capture must not touch any sequence's state: padding rows alone
            self.set_decode_inputs(zeros, zeros, np.full((rows, self.max_blocks), PADDING_PAGE, np.int32), zeros + PADDING_LENGTH,
                                   zeros + PADDING_SLOT, zeros + PADDING_STATE)
            self.capture(rows)
        states = np.full((rows,), PADDING_STATE, np.int32)
        states[:n] = step.row_states
        self.set_decode_inputs(*self._padded(step, rows), states)
        self.step(rows)
        if list(want) == list(range(n)):
            return self.logits[:n]
        return self.logits[torch.as_tensor(want, dtype=torch.long, device=self.device)]

    def set_decode_inputs(self, token_ids, positions, block_tables, seq_lens, slot_mapping, row_states=None) -> None:
        """Inputs of a step of one token per sequence, as many as there are ids; row r uses block table r."""
        rows = token_ids.shape[0]
        for dst, src in ((self.token_ids, token_ids), (self.positions, positions), (self.block_tables, block_tables),
                         (self.seq_lens, seq_lens), (self.slot_mapping, slot_mapping), (self.row_tables, np.arange(rows, dtype=np.int32)),
                         (self.row_states, row_states)):
            self._put(dst[:rows], src)
