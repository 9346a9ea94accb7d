"""Decoders whose layers choose their mixer and their feed-forward, on one B200, weights in bf16 (or f32).

A layer is x <- x + scale1 * norm(mixer(norm(x))), then the same around its feed-forward (if it has one): a norm on both sides of each
branch, the branch's output scaled element by element.  Mixers:
  differential attention   two softmax maps per head over the same values, subtracted with one learned factor per layer; grouped
                           key/value heads, rotate-half positions, a sliding window that keeps the first tokens, a gate per head.  A
                           layer may attend over the keys and values of an earlier one.
  retention                a linear recurrence with a fixed decay per head and an f32 state per sequence, rotate-half positions, a norm
                           per head and a SiLU gate.
Feed-forwards: dense (gated, tanh GELU) or a mixture of experts (gated, SiLU; softmax over the chosen logits; an optional shared
expert behind a sigmoid gate).

What a sequence holds: one row [keys | values] per position and attention layer with keys of its own, in the paged cache, and one state per
retention layer in the sequence's state slot.  A step launches per layer one projection of everything the mixer reads (queries, keys,
values, gate), the mixer (csrc/grouped_attention.cu, latent_prefill.cu, retention.cu), the output projection, one kernel that ends the
branch and begins the next (norm, scale, residual sum, norm), and the feed-forward's projections with the activation in the epilogue;
experts run as one grouped projection over tokens sorted by expert.  Norms, rotation, scores, softmax, routing, recurrence and the
residual stream are f32 throughout.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import numpy as np
import torch

from . import _native as N
from . import ops
from .rotary import Rotation, pair_tables
from .step_model import RaggedModel

PORTION_FROM = 16  # tokens of a portion from which the prompt kernels pay


# ---------------------------------------------------------------------------------------------- configuration

@dataclass(frozen=True)
class DifferentialAttention:
    heads: int
    kv_heads: int
    dim: int        # query/key dimensions of one map of a head
    vdim: int
    scale: float
    diff: float     # the layer's constant part of the subtracted map's factor
    rot: Rotation
    window: int | None = None  # a position sees itself and the window - 1 before it ...
    keep_first: int = 0        # ... and this many first positions
    kv_from: int | None = None  # the layer whose keys and values this one uses

    @property
    def kdim(self) -> int:
        """Elements of a key head in the cache: whole tensor-core steps, zeros past dim."""
        return -(-self.dim // 16) * 16

    @property
    def vpad(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def v_first(self) -> int:
        return self.kv_heads * 2 * self.kdim

    @property
    def row(self) -> int:
        return self.v_first + self.kv_heads * self.vpad

    @property
    def parts(self) -> tuple:
        """Columns of the layer's projection: (name, rows)."""
        kv = (("k", self.kv_heads * 2 * self.dim), ("v", self.kv_heads * self.vdim)) if self.kv_from is None else ()
        return (("q", self.heads * 2 * self.dim), *kv, ("g", self.heads))


@dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: Rotation

    @property
    def kdim(self) -> int:
        return -(-self.dim // 16) * 16

    @property
    def vpad(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def parts(self) -> tuple:
        return (("q", self.heads * self.dim), ("k", self.heads * self.dim), ("v", self.heads * self.vdim), ("g", self.heads * self.vdim))


@dataclass(frozen=True)
class Dense:
    ff: int


@dataclass(frozen=True)
class Experts:
    ff: int
    experts: int
    top: int
    shared_ff: int | None = None


@dataclass(frozen=True)
class Layer:
    mixer: DifferentialAttention | Retention
    mlp: Dense | Experts | None


def _attention(i: int, m: dict, layers: list) -> DifferentialAttention:
    mask = m.get("mask")
    heads, kv_heads, rot = int(m["heads"]), int(m["kv_heads"]), _rotation(i, m)
    source = m.get("kv_from")
    if heads < 1 or kv_heads < 1 or heads % kv_heads:
        raise ValueError(f"layer {i}: {heads} query heads over {kv_heads} key/value heads")
    out = DifferentialAttention(heads=heads, kv_heads=kv_heads, dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), diff=float(m["diff"]), rot=rot,
                                window=int(mask["size"]) if mask else None, keep_first=int(mask.get("keep_first", 0)) if mask else 0,
                                kv_from=int(source) if source is not None else None)
    if out.kv_from is not None:
        src = layers[out.kv_from].mixer if 0 <= out.kv_from < i else None
        if not isinstance(src, DifferentialAttention) or src.kv_from is not None or (src.kv_heads, src.dim, src.vdim) != (kv_heads, out.dim, out.vdim):
            raise ValueError(f"layer {i}: kv_from {out.kv_from} is not an earlier attention layer with keys and values of this shape")
    return out


def _rotation(i: int, m: dict) -> Rotation:
    rot = m.get("rot")
    if rot is None:
        return Rotation(0, 1.0)
    if rot.get("scaling") or int(rot["dims"]) > int(m["dim"]):
        raise ValueError(f"layer {i}: rotation {rot} is not built")
    return Rotation(int(rot["dims"]), float(rot["base"]))


@dataclass(frozen=True)
class MixedDecoderConfig:
    width: int
    vocab: int
    eps: float
    layers: tuple
    block_size: int = 64

    @property
    def window(self) -> int | None:
        """The longest window, None if some layer attends over everything (1 if none attends at all)."""
        sizes = [l.mixer.window for l in self.layers if isinstance(l.mixer, DifferentialAttention)]
        return None if any(s is None for s in sizes) else max(sizes, default=1)

    @property
    def keep_first(self) -> int:
        return max((l.mixer.keep_first for l in self.layers if isinstance(l.mixer, DifferentialAttention)), default=0)

    @property
    def recurrent(self) -> bool:
        return any(isinstance(l.mixer, Retention) for l in self.layers)

    @classmethod
    def from_config(cls, c: dict) -> "MixedDecoderConfig":
        """The design's config.json; what it names and this class does not know is refused."""
        layers: list[Layer] = []
        for i, e in enumerate(c["layers"]):
            m = e["mixer"]
            if e["type"] == "attention":
                mixer = _attention(i, m, layers)
            elif e["type"] == "retention":
                mixer = Retention(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(d) for d in m["decay"]), _rotation(i, m))
                if len(mixer.decay) != mixer.heads:
                    raise ValueError(f"layer {i}: {len(mixer.decay)} decays for {mixer.heads} heads")
            else:
                raise ValueError(f"layer {i}: mixer type {e['type']!r} is not built")
            f = e.get("mlp")
            if f is None:
                mlp = None
            elif f["kind"] == "dense":
                mlp = Dense(int(f["ff"]))
            elif f["kind"] == "moe":
                shared, router = f.get("shared"), f["router"]
                mlp = Experts(int(f["expert"]["ff"]), int(router["experts"]), int(router["top"]), int(shared["ff"]) if shared else None)
                if not 1 <= mlp.top <= mlp.experts:
                    raise ValueError(f"layer {i}: {mlp.top} of {mlp.experts} experts")
            else:
                raise ValueError(f"layer {i}: feed-forward kind {f['kind']!r} is not built")
            layers.append(Layer(mixer, mlp))
        return cls(width=int(c["width"]), vocab=int(c["vocab"]), eps=float(c["norm"]["eps"]), layers=tuple(layers))

    def tensor_shapes(self) -> dict:
        """Name -> shape of every tensor a checkpoint of this configuration holds."""
        w = self.width
        out = {"embed": (self.vocab, w), "head": (self.vocab, w), "final.norm": (w,)}

        def gated(p, ff):
            out[p + "gate"], out[p + "up"], out[p + "down"] = (ff, w), (ff, w), (w, ff)

        for i, l in enumerate(self.layers):
            m, p = l.mixer, f"l{i}."
            for name in ("norm1", "norm1b", "ls1") + (("norm2", "norm2b", "ls2") if l.mlp is not None else ()):
                out[p + name] = (w,)
            for name, rows in m.parts:
                out[p + "mix." + name] = (rows, w)
            out[p + "mix.o"] = (w, m.heads * m.vdim)
            if isinstance(m, DifferentialAttention):
                for name in ("lq1", "lk1", "lq2", "lk2"):
                    out[p + "mix." + name] = (m.dim,)
            if isinstance(l.mlp, Dense):
                gated(p + "mlp.", l.mlp.ff)
            elif l.mlp is not None:
                out[p + "mlp.router"] = (l.mlp.experts, w)
                for e in range(l.mlp.experts):
                    gated(f"{p}mlp.e{e}.", l.mlp.ff)
                if l.mlp.shared_ff is not None:
                    gated(p + "mlp.shared.", l.mlp.shared_ff)
                    out[p + "mlp.shared.sg"] = (1, w)
        return out


# ---------------------------------------------------------------------------------------------- the model

class MixedDecoder(RaggedModel):
    """Weights, pools, states and step buffers; `run` takes a ragged step, `step(rows)` one token of `rows` sequences."""

    def __init__(self, cfg: MixedDecoderConfig, *, num_blocks: int, max_len: int, max_tokens: int = 2048, max_sequences: int = 64,
                 dtype: torch.dtype = torch.bfloat16, device="cuda:0"):
        super().__init__(width=cfg.width, dtype=dtype, max_tokens=max_tokens, max_sequences=max_sequences, num_blocks=num_blocks, max_len=max_len,
                         block_size=cfg.block_size, vocab=cfg.vocab, device=device)
        self.cfg, self.window, self.keep_first = cfg, cfg.window, cfg.keep_first
        self.num_states = max_sequences if cfg.recurrent else 0
        dev, R = self.device, self.rows
        ty, f32, i32 = dict(dtype=dtype, device=dev), dict(dtype=torch.float32, device=dev), dict(dtype=torch.int32, device=dev)
        mixers, mlps = [l.mixer for l in cfg.layers], [l.mlp for l in cfg.layers]
        att = [m for m in mixers if isinstance(m, DifferentialAttention)]
        ret = [m for m in mixers if isinstance(m, Retention)]
        moe = [f for f in mlps if isinstance(f, Experts)]
        # what sequences hold
        self.pools = [torch.zeros((num_blocks, cfg.block_size, m.row), **ty) if isinstance(m, DifferentialAttention) and m.kv_from is None else None for m in mixers]
        for i, m in enumerate(mixers):
            if isinstance(m, DifferentialAttention) and m.kv_from is not None:
                self.pools[i] = self.pools[m.kv_from]
        self.states = [torch.zeros((self.num_states + 1, m.heads, m.dim, -(-m.vdim // 4) * 4), **f32) if isinstance(m, Retention) else None for m in mixers]
        tables: dict[Rotation, tuple] = {}
        for m in mixers:
            if m.rot not in tables:
                tables[m.rot] = tuple(torch.from_numpy(np.ascontiguousarray(t)).to(dev) for t in pair_tables(m.rot, self.max_positions))
        self._rot = [tables[m.rot] for m in mixers]
        self._decay = [torch.tensor(m.decay, **f32) if isinstance(m, Retention) else None for m in mixers]
        self.layers: list[dict] = []
        self.embed = self.head = self.final_norm = None
        # step buffers, shared by the layers: flat, viewed in each layer's own shape
        big = lambda xs, f: max((f(x) for x in xs), default=0)
        flat = lambda rows, cols, kind: torch.empty((rows * cols,), **kind)
        self.h = torch.empty((R, cfg.width), **ty)
        self._proj = flat(R, big(mixers, lambda m: sum(n for _, n in m.parts)), f32)
        self._q = flat(R, max(big(att, lambda m: m.heads * 2 * m.kdim), big(ret, lambda m: m.heads * m.kdim)), ty)
        self._k = flat(R, big(ret, lambda m: m.heads * m.kdim), ty)
        self._v = flat(R, big(ret, lambda m: m.heads * m.vpad), ty)
        self._maps = torch.empty((max([self._map_values(m, R) for m in att] + [R * m.heads * m.vdim for m in ret]),), **f32)
        sums = max((ops.retention_chunks_scratch_bytes(n, m.heads, m.dim, m.vdim) for m in ret for n in range(64, R + 64, 64)), default=0)
        self._state_sums = torch.empty((sums // 4,), **f32) if dtype == torch.bfloat16 else None
        self._mixed = flat(R, big(mixers, lambda m: m.heads * m.vdim), ty)
        self.y = torch.empty((R, cfg.width), **f32)
        pad = lambda ff: -(-ff // 16) * 16
        self._act = flat(R, max(big([f for f in mlps if isinstance(f, Dense)], lambda f: pad(f.ff)), big(moe, lambda f: pad(f.shared_ff or 0))), ty)
        entries = big(moe, lambda f: f.top)
        self._route = flat(R, big(moe, lambda f: f.experts + 1), f32)
        self._ids, self._rows_of, self._tokens_of = (torch.zeros((R * entries,), **i32) for _ in range(3))
        self._weights = flat(R, entries, f32)
        self._offsets = torch.zeros((big(moe, lambda f: f.experts) + 1,), **i32)
        self._sorted = flat(R * entries, cfg.width, ty)
        self._act_sorted = flat(R * entries, big(moe, lambda f: pad(f.ff)), ty)
        self._out_sorted = flat(R * entries, cfg.width, ty)
        self._portion_space: dict[str, torch.Tensor] = {}  # gathered keys and values of a portion's window; grown on demand

    def _max_live(self, m: DifferentialAttention) -> int:
        return self.max_positions if m.window is None else min(self.max_positions, m.window + m.keep_first)

    def _slices(self, m: DifferentialAttention, rows: int) -> int:
        return ops.grouped_attention_slices(rows, m.heads * 2, m.kv_heads, 2, m.kdim, m.vpad, self.block_size, self.dtype, self._max_live(m))

    def _map_values(self, m: DifferentialAttention, rows: int) -> int:
        """f32 values of the most records a step of up to `rows` rows leaves (few rows have several slices each)."""
        sizes = {1 << i for i in range(rows.bit_length())} | {rows}
        return max(max(n, 2 * n * (self._slices(m, n) > 1)) * self._slices(m, n) for n in sizes if n <= rows) * m.heads * 2 * (m.vpad + 2)

    # ------------------------------------------------------------------ weights

    def load_tensors(self, t: dict) -> None:
        """A checkpoint's tensors (name -> f32 array, linear weights [out, in]) in the layout the step wants: what reads the mixer's input
        stacked, gate and up projections interleaved, experts stacked, each branch's output norm multiplied by its scale."""
        shapes = self.cfg.tensor_shapes()
        unused = {f"l{i}.{n}" for i, l in enumerate(self.cfg.layers) if l.mlp is None for n in ("norm2", "norm2b", "ls2")}  # of a branch that is absent
        missing, extra = sorted(set(shapes) - set(t)), sorted(set(t) - set(shapes) - unused)
        if missing or extra:
            raise ValueError(f"the checkpoint does not fit its configuration: missing {missing[:5]}, unknown {extra[:5]}")
        for name, shape in shapes.items():
            if tuple(t[name].shape) != shape:
                raise ValueError(f"tensor {name!r} is {tuple(t[name].shape)}, the configuration says {shape}")
        dev = self.device
        put = lambda a: torch.as_tensor(np.ascontiguousarray(a) if isinstance(a, np.ndarray) else a, device=dev)
        w = lambda name: put(t[name]).to(self.dtype).contiguous()
        g = lambda name: put(t[name]).float().contiguous()
        self.embed, self.head, self.final_norm = w("embed"), w("head"), g("final.norm")
        self.layers = []

        def gated(p):
            """Gate and up interleaved, and the down projection with its columns padded like them."""
            down = w(p + "down")
            return ops.interleave_gate(w(p + "gate"), w(p + "up")), torch.nn.functional.pad(down, (0, -down.shape[1] % 16)).contiguous()

        for i, l in enumerate(self.cfg.layers):
            m, p = l.mixer, f"l{i}."
            lw = {"norm1": g(p + "norm1"), "post1": g(p + "norm1b") * g(p + "ls1"), "proj": torch.cat([w(p + "mix." + n) for n, _ in m.parts]), "o": w(p + "mix.o")}
            if isinstance(m, DifferentialAttention):
                dot = lambda a, b: math.exp(float((put(t[p + "mix." + a]).double() * put(t[p + "mix." + b]).double()).sum()))
                lw["lambda"] = dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff
            if l.mlp is not None:
                lw.update(norm2=g(p + "norm2"), post2=g(p + "norm2b") * g(p + "ls2"))
            if isinstance(l.mlp, Dense):
                lw["up"], lw["down"] = gated(p + "mlp.")
            elif l.mlp is not None:
                both = [gated(f"{p}mlp.e{e}.") for e in range(l.mlp.experts)]
                lw["e_up"], lw["e_down"] = torch.stack([a for a, _ in both]), torch.stack([b for _, b in both])
                del both
                lw["router"] = w(p + "mlp.router")
                if l.mlp.shared_ff is not None:
                    lw["router"] = torch.cat([lw["router"], w(p + "mlp.shared.sg")])
                    lw["up"], lw["down"] = gated(p + "mlp.shared.")
            self.layers.append(lw)

    def init_random_weights(self, seed: int = 0) -> None:
        """Random weights on the device, sized so that activations stay O(1) through the layers (throughput runs)."""
        gen = torch.Generator(device=self.device)
        gen.manual_seed(seed)
        t = {}
        for name, shape in self.cfg.tensor_shapes().items():
            r = torch.randn(shape, device=self.device, generator=gen, dtype=torch.bfloat16)
            t[name] = 1.0 + 0.1 * r if "norm" in name or ".ls" in name else 0.1 * r if len(shape) == 1 else r * shape[1] ** -0.5
        self.load_tensors(t)

    # ------------------------------------------------------------------ the step

    @staticmethod
    def _view(flat: torch.Tensor, *shape) -> torch.Tensor:
        return flat[:math.prod(shape)].view(*shape)

    def _attention(self, i: int, n: int, spans, proj: torch.Tensor, out: torch.Tensor) -> None:
        m, lw, pool, (cos, sin) = self.cfg.layers[i].mixer, self.layers[i], self.pools[i], self._rot[i]
        q = self._view(self._q, n, m.heads * 2, m.kdim)
        parts = [ops.rotate_part(q, 0, m.heads * 2, m.dim, padded=m.kdim, row_ld=m.heads * 2 * m.kdim)]
        if m.kv_from is None:
            k_first = m.heads * 2 * m.dim
            parts.append(ops.rotate_part(pool, k_first, m.kv_heads * 2, m.dim, padded=m.kdim, row_ld=m.row, by_slot=True))
            parts.append(ops.rotate_part(pool[0, 0, m.v_first:], k_first + m.kv_heads * 2 * m.dim, m.kv_heads, m.vdim, padded=m.vpad, row_ld=m.row,
                                         rotate=False, by_slot=True))
        ops.rotate_rows(proj, parts, self.positions, cos, sin, rot_dims=m.rot.dims, slots=self.slot_mapping, num_slots=self.num_blocks * self.block_size)
        gate = proj[:, proj.shape[1] - m.heads:]
        end = lambda lo, hi, maps, slices: ops.map_difference(maps, out[lo:hi], rows=hi - lo, heads=m.heads, vdim=m.vdim, in_ld=m.vpad, lam=lw["lambda"],
                                                              keep=1.0 - m.diff, eps=self.cfg.eps, slices=slices, gate=gate[lo:hi])

        def tokens(lo, hi):
            slices = self._slices(m, hi - lo)
            ops.grouped_attention(q[lo:hi], pool, self.block_tables, self.seq_lens[lo:hi], self._maps, v_heads=m.kv_heads, maps=2, vdim=m.vpad, v_first=m.v_first,
                                  scale=m.scale, slices=slices, window=m.window or 0, keep_first=m.keep_first, row_tables=self.row_tables[lo:hi])
            end(lo, hi, self._maps, slices)

        prompt_kernel = self.dtype == torch.bfloat16 and m.scale > 0 and ops.window_attention_applies(m.kdim, 0, m.vpad)
        lo = 0  # rows [lo, first) are waiting for one call
        for first, stop, table, pos in spans or ():
            if not prompt_kernel or stop - first < PORTION_FROM:
                continue
            if first > lo:
                tokens(lo, first)
            self._portion(i, first, stop, table, pos, q)
            end(first, stop, self._maps, 0)
            lo = stop
        if lo < n:
            tokens(lo, n)

    def _portion(self, i: int, lo: int, hi: int, table: int, pos: int, q: torch.Tensor) -> None:
        """Rows [lo, hi) of one sequence, positions pos ..: the maps' outputs over the kept tokens and the window, into the first of _maps."""
        m, n = self.cfg.layers[i].mixer, hi - lo
        first = max(0, pos - m.window + 1) if m.window else 0
        keep = m.keep_first if m.window else 0
        held = keep if first > keep else 0  # the window has left the kept tokens: their rows, then the window's
        first = first if held or not keep else 0
        keys = held + pos + n - first
        rows = self._portion_space.get("rows")
        if rows is None or rows.numel() < keys * m.row:
            rows = self._portion_space["rows"] = torch.empty((keys * m.row,), dtype=self.dtype, device=self.device)
        rows = rows[:keys * m.row].view(keys, m.row)
        ops.latent_gather(self.pools[i], self.block_tables[table], rows, first=first, keep=held)
        ops.window_attention(q[lo:hi], rows[:, :m.v_first].view(keys, m.kv_heads * 2, m.kdim), None, rows[:, m.v_first:].view(keys, m.kv_heads, m.vpad),
                             self._view(self._maps, n, m.heads * 2 * m.vpad), first_query=keys - n, scale=m.scale, window=m.window or 0, keep_first=keep, maps=2)

    def _retention(self, i: int, n: int, spans, proj: torch.Tensor, out: torch.Tensor) -> None:
        m, state, decay, (cos, sin) = self.cfg.layers[i].mixer, self.states[i], self._decay[i], self._rot[i]
        k_scale = m.dim ** -0.5

        def tokens(lo, hi):
            """Rows of different sequences, one token each."""
            ops.retention_step(proj[lo:hi], self.positions[lo:hi], cos, sin, decay, self.row_states[lo:hi], state, out[lo:hi], heads=m.heads, dim=m.dim,
                               vdim=m.vdim, rot_dims=m.rot.dims, k_scale=k_scale, eps=self.cfg.eps)

        lo = 0
        for first, stop, _, _ in spans or ():
            if stop - first < 2:
                continue
            if first > lo:
                tokens(lo, first)
            rows, vcol = stop - first, 2 * m.heads * m.dim
            q, k, v = self._view(self._q, rows, m.heads, m.kdim), self._view(self._k, rows, m.heads, m.kdim), self._view(self._v, rows, m.heads, m.vpad)
            ops.rotate_rows(proj[first:stop], [ops.rotate_part(q, 0, m.heads, m.dim, padded=m.kdim, row_ld=m.heads * m.kdim),
                                               ops.rotate_part(k, m.heads * m.dim, m.heads, m.dim, padded=m.kdim, row_ld=m.heads * m.kdim, scale=k_scale),
                                               ops.rotate_part(v, vcol, m.heads, m.vdim, padded=m.vpad, row_ld=m.heads * m.vpad, rotate=False)],
                            self.positions[first:stop], cos, sin, rot_dims=m.rot.dims)
            o = self._view(self._maps, rows, m.heads, m.vdim)
            operands = (q, k, v, self.positions[first:stop], decay, self.row_states[first:stop], state, o)
            if self.dtype == torch.bfloat16 and ops.retention_chunks_applies(m.dim, m.vdim):
                ops.retention_chunks(*operands, self._state_sums)
            else:
                ops.retention_scan(*operands)
            ops.head_norm_gate(o, proj[first:stop, vcol + m.heads * m.vdim:], out[first:stop], self.cfg.eps)
            lo = stop
        if lo < n:
            tokens(lo, n)

    def _experts(self, f: Experts, lw: dict, h: torch.Tensor, n: int) -> dict:
        """The experts' outputs of rows [0, n): what `residual_norm` sums."""
        logits = self._view(self._route, n, lw["router"].shape[0])
        route = ops.dense(h, lw["router"], logits)
        y = gate = None
        if f.shared_ff is not None:
            act = self._view(self._act, n, lw["down"].shape[1])
            ops.dense_gemm(ops.dense(h, lw["up"], act, act=N.ACT_SILU_MUL), route, weights_const=True)
            y, gate = self.y[:n], logits[:, f.experts]
        else:
            ops.dense_gemm(route, weights_const=True)
        ids, weights, rows_of = (self._view(b, n, f.top) for b in (self._ids, self._weights, self._rows_of))
        tokens_of, offsets = self._tokens_of[:n * f.top], self._offsets[:f.experts + 1]
        ops.moe_route(logits, ids, weights, offsets, rows_of, tokens_of, experts=f.experts)
        xs = self._view(self._sorted, n * f.top, self.cfg.width)
        ops.gather_rows(h, tokens_of, xs)
        acts = self._view(self._act_sorted, n * f.top, lw["e_down"].shape[2])
        outs = self._view(self._out_sorted, n * f.top, self.cfg.width)
        ops.dense_gemm(ops.grouped_dense(xs, lw["e_up"], acts, offsets, act=N.ACT_SILU_MUL))
        down = [ops.grouped_dense(acts, lw["e_down"], outs, offsets)]
        if f.shared_ff is not None:
            if n <= 64:
                down.insert(0, ops.dense(act, lw["down"], y))
            else:
                ops.dense_gemm(ops.dense(act, lw["down"], y), weights_const=True)
        ops.dense_gemm(*down)
        return dict(y=y, gate=gate, parts=outs, part_rows=rows_of, part_weights=weights)

    def _hidden(self, n: int, spans=None, trace: list | None = None) -> None:
        cfg, x, h = self.cfg, self.x[:n], self.h[:n]
        ops.embedding(self.embed, self.token_ids[:n], out=x)
        ops.rmsnorm_pair(x, self.layers[0]["norm1"], h, cfg.eps)
        for i, (l, lw) in enumerate(zip(cfg.layers, self.layers)):
            m = l.mixer
            proj, mixed = self._view(self._proj, n, lw["proj"].shape[0]), self._view(self._mixed, n, m.heads * m.vdim)
            ops.dense_gemm(ops.dense(h, lw["proj"], proj), weights_const=True)
            (self._attention if isinstance(m, DifferentialAttention) else self._retention)(i, n, spans, proj, mixed)
            ops.dense_gemm(ops.dense(mixed, lw["o"], self.y[:n]), weights_const=True)
            following = self.layers[i + 1]["norm1"] if i + 1 < len(self.layers) else None
            if l.mlp is None:
                ops.residual_norm(self.y[:n], x, lw["post1"], cfg.eps, gain_next=following, out=h if following is not None else None)
            else:
                ops.residual_norm(self.y[:n], x, lw["post1"], cfg.eps, gain_next=lw["norm2"], out=h)
                if isinstance(l.mlp, Dense):
                    act = self._view(self._act, n, lw["down"].shape[1])
                    ops.dense_gemm(ops.dense(h, lw["up"], act, act=N.ACT_GELU_TANH_MUL), weights_const=True)
                    ops.dense_gemm(ops.dense(act, lw["down"], self.y[:n]), weights_const=True)
                    branch = dict(y=self.y[:n])
                else:
                    branch = self._experts(l.mlp, lw, h, n)
                ops.residual_norm(x=x, gain_post=lw["post2"], eps=cfg.eps, gain_next=following, out=h if following is not None else None, **branch)
            if trace is not None:
                trace.append(x.clone())

    def _head(self, x: torch.Tensor) -> torch.Tensor:
        k = x.shape[0]
        ops.rmsnorm_pair(x, self.final_norm, self.hn[:k], self.cfg.eps)
        ops.dense_gemm(ops.dense(self.hn[:k], self.head, self.logits[:k]), weights_const=True)
        return self.logits[:k]
