"""Decoders of latent-attention layers on one B200: parallel attention and feed-forward branches, weights in bf16 (or f32).

A layer adds mixer(norm1(x)) + feed_forward(norm2(x)) to the residual stream x.  Latent attention keeps one row per position
and layer in the paged cache, shared by all heads: the RMS-normed key/value latent and the rotated key part.  Two ways to
attend, equal up to rounding:
  absorbed   the key up-projection is folded into the query (query -> latent space), the scores and the weighted sum run on
             cached rows as they are, and the value up-projection follows: what decoding does;
  expanded   the window's latents are gathered and up-projected to per-head keys and values once per prompt portion, and
             the portion attends over those: fewer operations per score once a portion has enough rows to share the
             up-projection.

A step launches per layer (csrc/dense_gemm*.cu, csrc/latent_*.cu): the pair of norms; one launch for the query|key/value
down-projection and the feed-forward's up-projection (bias and squared ReLU in its epilogue); norms, rotation and cache write; query
up-projection; attention; and one projection over [attention output | feed-forward activations] that adds both branches and
the residual.  Norms, rotation, scores, softmax and the residual stream are f32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np
import torch

from . import _native as N
from . import ops
from .rotary import Rotation, YarnScaling, pair_tables
from .step_model import RaggedModel


EXPAND_FROM = 32  # tokens of a portion from which the expanded way of attending pays


# ---------------------------------------------------------------------------------------------- configuration

@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int        # unrotated query/key dimensions per head
    rot_dim: int    # rotated ones; the key part is shared by the heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotation
    window: int | None = None  # a position sees itself and the window - 1 before it

    @property
    def row(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def q_dim(self) -> int:
        return self.dim + self.rot_dim


@dataclass(frozen=True)
class FeedForward:
    ff: int


@dataclass(frozen=True)
class Layer:
    mixer: LatentAttention
    mlp: FeedForward | None
    weights: int  # the layer whose tensors this one uses


@dataclass(frozen=True)
class LatentDecoderConfig:
    width: int
    vocab: int
    eps: float
    layers: tuple
    block_size: int = 64

    @property
    def window(self) -> int | None:
        """The longest window, or None if some layer attends over everything."""
        sizes = [l.mixer.window for l in self.layers]
        return None if any(s is None for s in sizes) else max(sizes)

    @classmethod
    def from_config(cls, c: dict) -> "LatentDecoderConfig":
        """The design's config.json; what it names and this class does not know is refused."""
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: mixer type {e['type']!r} is not built")
            m = e["mixer"]
            rot = m["rot"]
            scaling = rot.get("scaling")
            if rot["dims"] > m["rot_dim"]:
                raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions in a part of {m['rot_dim']}")
            mask = m.get("mask")
            mixer = LatentAttention(
                heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]),
                kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), window=int(mask["size"]) if mask else None,
                rot=Rotation(int(rot["dims"]), float(rot["base"]),
                             YarnScaling(*(float(scaling[k]) for k in ("factor", "original", "fast", "slow"))) if scaling else None))
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not built")
            source, passed = i, {i}
            while c["layers"][source].get("weights_of") is not None:
                nxt = int(c["layers"][source]["weights_of"])
                if not 0 <= nxt < len(c["layers"]) or nxt in passed:
                    raise ValueError(f"layer {source}: weights_of {nxt} leads to no layer with weights")
                passed.add(nxt)
                source = nxt
            layers.append(Layer(mixer, FeedForward(int(mlp["ff"])) if mlp is not None else None, source))
        return cls(width=int(c["width"]), vocab=int(c["vocab"]), eps=float(c["norm"]["eps"]), layers=tuple(layers))

    def tensor_shapes(self) -> dict:
        """Name -> shape of every tensor a checkpoint of this configuration holds."""
        out = {"embed": (self.vocab, self.width), "final.norm": (self.width,)}
        for i, l in enumerate(self.layers):
            if l.weights != i:
                continue
            m, p = l.mixer, f"l{i}."
            out[p + "norm1"] = (self.width,)
            out[p + "mix.dq"] = (m.q_rank, self.width)
            out[p + "mix.dq.norm"] = (m.q_rank,)
            out[p + "mix.uq"] = (m.heads * m.q_dim, m.q_rank)
            out[p + "mix.dkv"] = (m.row, self.width)
            out[p + "mix.dkv.norm"] = (m.kv_rank,)
            out[p + "mix.uk"] = (m.heads * m.dim, m.kv_rank)
            out[p + "mix.uv"] = (m.heads * m.vdim, m.kv_rank)
            out[p + "mix.o"] = (self.width, m.heads * m.vdim)
            if l.mlp is not None:
                out[p + "norm2"] = (self.width,)
                out[p + "mlp.up"], out[p + "mlp.up.b"] = (l.mlp.ff, self.width), (l.mlp.ff,)
                out[p + "mlp.down"], out[p + "mlp.down.b"] = (self.width, l.mlp.ff), (self.width,)
        return out


# ---------------------------------------------------------------------------------------------- the model

class LatentDecoder(RaggedModel):
    """Weights, latent pools and step buffers; `run` takes a ragged step, `step(rows)` one token of `rows` sequences."""

    def __init__(self, cfg: LatentDecoderConfig, *, num_blocks: int, max_len: int, max_tokens: int = 2048, max_sequences: int = 64,
                 dtype: torch.dtype = torch.bfloat16, device="cuda:0"):
        super().__init__(width=cfg.width, dtype=dtype, max_tokens=max_tokens, max_sequences=max_sequences, num_blocks=num_blocks, max_len=max_len,
                         block_size=cfg.block_size, vocab=cfg.vocab, device=device)
        self.cfg, self.window = cfg, cfg.window
        dev, R = self.device, self.rows
        ty, f32 = dict(dtype=dtype, device=dev), dict(dtype=torch.float32, device=dev)
        mixers = [l.mixer for l in cfg.layers]
        self.pools = [torch.zeros((num_blocks, cfg.block_size, -(-m.row // 8) * 8), **ty) for m in mixers]
        tables: dict[Rotation, tuple] = {}
        for m in mixers:
            if m.rot not in tables:
                tables[m.rot] = tuple(torch.from_numpy(t).to(dev) for t in pair_tables(m.rot, self.max_positions))
        self._rot = [tables[m.rot] for m in mixers]
        self.layers: list[dict] = []
        self.embed = self.final_norm = None
        # step buffers, shared by the layers: flat, viewed in each layer's own shape
        big = lambda f: max(f(l) for l in cfg.layers)
        self.h1, self.h2 = torch.empty((R, cfg.width), **ty), torch.empty((R, cfg.width), **ty)
        self._low = torch.empty((R * big(lambda l: l.mixer.q_rank + l.mixer.row),), **f32)
        self._cq = torch.empty((R * big(lambda l: l.mixer.q_rank),), **ty)
        self._q = torch.empty((R * big(lambda l: l.mixer.heads * l.mixer.q_dim),), **ty)
        self._cat = torch.empty((R * big(lambda l: self._o_width(l) + (l.mlp.ff if l.mlp else 0)),), **ty)
        self._qlat = torch.empty((R * big(lambda l: l.mixer.heads * l.mixer.row),), **ty)
        self._olat = torch.empty((R * big(lambda l: l.mixer.heads * l.mixer.kv_rank),), **ty)
        max_live = min(self.max_positions, cfg.window or self.max_positions)
        self._att_scratch = torch.empty((max(ops.latent_attention_scratch_bytes(R, m.heads, m.kv_rank, m.rot_dim, max_live) for m in mixers)
                                         // 4 + 4,), **f32)
        self._expanded = [dtype == torch.bfloat16 and ops.window_attention_applies(m.dim, m.rot_dim, m.vdim) and m.row % 8 == 0
                          and (m.heads * m.vdim) % 8 == 0 and m.scale > 0 for m in mixers]
        self._expand_space: dict[str, torch.Tensor] = {}  # gathered latents, keys and values of a portion's window; grown on demand

    @staticmethod
    def _o_width(l: Layer) -> int:
        """Columns of the attention output in front of the feed-forward's activations, kept to 16 bytes for both halves."""
        return -(-l.mixer.heads * l.mixer.vdim // 8) * 8 if l.mlp is not None else l.mixer.heads * l.mixer.vdim

    # ------------------------------------------------------------------ weights

    def load_tensors(self, t: dict) -> None:
        """A checkpoint's tensors (name -> f32 array, linear weights [out, in]; norms in front of the branches stored around
        zero) in the layout the step wants: query and key/value down-projection stacked, the two output projections side by side, the
        key up-projection also transposed per head."""
        shapes = self.cfg.tensor_shapes()
        unused = {f"l{i}.norm2" for i, l in enumerate(self.cfg.layers) if l.mlp is None}  # the norm of a branch that is absent
        missing, extra = sorted(set(shapes) - set(t)), sorted(set(t) - set(shapes) - unused)
        if missing or extra:
            raise ValueError(f"the checkpoint does not fit its configuration: missing {missing[:5]}, unknown {extra[:5]}")
        for name, shape in shapes.items():
            if tuple(t[name].shape) != shape:
                raise ValueError(f"tensor {name!r} is {tuple(t[name].shape)}, the configuration says {shape}")
        dev = self.device
        put = lambda a: torch.as_tensor(np.ascontiguousarray(a) if isinstance(a, np.ndarray) else a, device=dev)
        w = lambda a: put(a).to(self.dtype).contiguous()
        g = lambda a: put(a).float().contiguous()
        self.embed, self.final_norm = w(t["embed"]), g(t["final.norm"]) + 1.0
        built: dict[int, dict] = {}
        for i, l in enumerate(self.cfg.layers):
            if l.weights != i:
                continue
            m, p = l.mixer, f"l{i}."
            uk = w(t[p + "mix.uk"]).view(m.heads, m.dim, m.kv_rank)
            uv = w(t[p + "mix.uv"]).view(m.heads, m.vdim, m.kv_rank)
            lw = {"norm1": g(t[p + "norm1"]) + 1.0, "low": torch.cat([w(t[p + "mix.dq"]), w(t[p + "mix.dkv"])]),
                  "q_gain": g(t[p + "mix.dq.norm"]), "kv_gain": g(t[p + "mix.dkv.norm"]), "uq": w(t[p + "mix.uq"]),
                  "uk_t": uk.transpose(1, 2).contiguous(), "uv": uv}
            if self._expanded[i]:
                lw["ukv"] = torch.cat([uk, uv], dim=1).reshape(m.heads * (m.dim + m.vdim), m.kv_rank)
            out = w(t[p + "mix.o"])
            if l.mlp is not None:
                pad = torch.zeros((self.cfg.width, self._o_width(l) - m.heads * m.vdim), dtype=self.dtype, device=dev)
                out = torch.cat([out, pad, w(t[p + "mlp.down"])], dim=1)
                lw.update(norm2=g(t[p + "norm2"]) + 1.0, up=w(t[p + "mlp.up"]), up_b=g(t[p + "mlp.up.b"]), down_b=g(t[p + "mlp.down.b"]))
            lw["out"] = out.contiguous()
            built[i] = lw
        self.layers = [built[l.weights] for l in self.cfg.layers]

    def init_random_weights(self, seed: int = 0) -> None:
        """Random weights on the device, sized so that activations stay O(1) through the layers (throughput runs)."""
        gen = torch.Generator(device=self.device)
        gen.manual_seed(seed)
        t = {}
        for name, shape in self.cfg.tensor_shapes().items():
            r = torch.randn(shape, device=self.device, generator=gen, dtype=torch.bfloat16)
            if name.endswith((".dq.norm", ".dkv.norm")):
                r = 1.0 + 0.1 * r
            elif len(shape) == 1:
                r = 0.1 * r
            else:
                r *= 0.02 if name == "embed" else shape[1] ** -0.5
            t[name] = r
        self.load_tensors(t)

    def weight_bytes(self) -> int:
        """Bytes of weights one step reads (a shared layer is read each time it runs)."""
        n = sum(v.numel() * v.element_size() for lw in self.layers for k, v in lw.items() if k != "ukv")
        return n + self.embed.numel() * self.embed.element_size() + 4 * self.final_norm.numel()

    # ------------------------------------------------------------------ the step

    def _layer(self, i: int, n: int, spans) -> None:
        """One layer over rows [0, n): normed inputs h1 (and h2) -> residual stream x.  spans: [(first row, end row, table row,
        position of the first)], the rows of each sequence; None: one row per sequence."""
        l, lw, eps = self.cfg.layers[i], self.layers[i], self.cfg.eps
        m, pool, (cos, sin) = l.mixer, self.pools[i], self._rot[i]
        x, h1, h2 = self.x[:n], self.h1[:n], self.h2[:n]
        ow = self._o_width(l)
        low = self._low[:n * (m.q_rank + m.row)].view(n, m.q_rank + m.row)
        cat = self._cat[:n * (ow + (l.mlp.ff if l.mlp else 0))].view(n, -1)
        if ow != m.heads * m.vdim:
            cat[:, m.heads * m.vdim:ow].zero_()
        down = [ops.dense(h1, lw["low"], low)]
        if l.mlp is not None:
            down.append(ops.dense(h2, lw["up"], cat[:, ow:], bias=lw["up_b"], act=N.ACT_RELU2))
        ops.dense_gemm(*down, weights_const=True)
        cq = self._cq[:n * m.q_rank].view(n, m.q_rank)
        ops.latent_kv_write(low, lw["q_gain"], lw["kv_gain"], eps, self.positions, cos, sin, self.slot_mapping, cq, pool,
                            q_rank=m.q_rank, kv_rank=m.kv_rank, rot_dim=m.rot_dim, rot_dims=m.rot.dims)
        q = self._q[:n * m.heads * m.q_dim].view(n, m.heads, m.q_dim)
        ops.dense_gemm(ops.dense(cq, lw["uq"], q.view(n, -1)), weights_const=True)
        lo = 0  # rows [lo, first) are waiting for one absorbed call
        for first, end, table, pos in spans or ():
            if self._expanded[i] and end - first >= EXPAND_FROM:
                if first > lo:
                    self._attend_absorbed(i, lo, first, q, cat)
                self._attend_expanded(i, first, end, table, pos, q, cat)
                lo = end
        if lo < n:
            self._attend_absorbed(i, lo, n, q, cat)
        ops.dense_gemm(ops.dense(cat, lw["out"], x, bias=lw.get("down_b"), residual=x), weights_const=True)

    def _attend_absorbed(self, i: int, lo: int, hi: int, q: torch.Tensor, cat: torch.Tensor) -> None:
        """Rows [lo, hi): q [rows, heads, dim | rot_dim] -> attention output into the first columns of cat."""
        m, lw, (cos, sin), n = self.cfg.layers[i].mixer, self.layers[i], self._rot[i], hi - lo
        pool = self.pools[i]
        qlat = self._qlat[:n * m.heads * m.row].view(n, m.heads, m.row)
        olat = self._olat[:n * m.heads * m.kv_rank].view(n, m.heads, m.kv_rank)
        ops.dense_gemm(ops.dense(q[lo:hi, :, :m.dim].transpose(0, 1), lw["uk_t"], qlat[:, :, :m.kv_rank].transpose(0, 1)), weights_const=True)
        if m.rot_dim:
            ops.rope_interleaved(q[lo:hi, :, m.dim:], qlat[:, :, m.kv_rank:], self.positions[lo:hi], cos, sin, rot_dims=m.rot.dims)
        ops.latent_attention(qlat, pool, self.block_tables, self.seq_lens[lo:hi], olat, kv_rank=m.kv_rank, scale=m.scale,
                             window=m.window or 0, row_tables=self.row_tables[lo:hi], scratch=self._att_scratch)
        o = cat[lo:hi, :m.heads * m.vdim].view(n, m.heads, m.vdim)
        ops.dense_gemm(ops.dense(olat.transpose(0, 1), lw["uv"], o.transpose(0, 1)), weights_const=True)

    def _space(self, name: str, rows: int, cols: int) -> torch.Tensor:
        flat = self._expand_space.get(name)
        if flat is None or flat.numel() < rows * cols:
            flat = self._expand_space[name] = torch.empty((rows * cols,), dtype=self.dtype, device=self.device)
        return flat[:rows * cols].view(rows, cols)

    def _attend_expanded(self, i: int, lo: int, hi: int, table: int, pos: int, q: torch.Tensor, cat: torch.Tensor) -> None:
        """Rows [lo, hi) of one sequence, positions pos .., over the per-head keys and values of its window."""
        m, lw, (cos, sin) = self.cfg.layers[i].mixer, self.layers[i], self._rot[i]
        first = max(0, pos - m.window + 1) if m.window else 0
        keys = pos + hi - lo - first
        lat = self._space("latents", keys, m.row)
        ops.latent_gather(self.pools[i], self.block_tables[table], lat, first=first)
        kv = self._space("keys and values", keys, m.heads * (m.dim + m.vdim))
        ops.dense_gemm(ops.dense(lat[:, :m.kv_rank], lw["ukv"], kv), weights_const=True)
        if m.rot_dim:
            rotated = q[lo:hi, :, m.dim:]
            ops.rope_interleaved(rotated, rotated, self.positions[lo:hi], cos, sin, rot_dims=m.rot.dims)
        kv = kv.view(keys, m.heads, m.dim + m.vdim)
        ops.window_attention(q[lo:hi], kv[:, :, :m.dim], lat[:, m.kv_rank:], kv[:, :, m.dim:], cat[lo:hi, :m.heads * m.vdim],
                             first_query=pos - first, scale=m.scale, window=m.window or 0)

    def _norms(self, i: int, n: int) -> None:
        """The norms in front of layer i's branches."""
        lw = self.layers[i]
        ops.rmsnorm_pair(self.x[:n], lw["norm1"], self.h1[:n], self.cfg.eps, lw.get("norm2"), self.h2[:n] if "norm2" in lw else None)

    def _hidden(self, n: int, spans=None, trace: list | None = None) -> None:
        ops.embedding(self.embed, self.token_ids[:n], out=self.x[:n])
        for i in range(len(self.layers)):
            self._norms(i, n)
            self._layer(i, n, spans)
            if trace is not None:
                trace.append(self.x[:n].clone())

    def _head(self, x: torch.Tensor) -> torch.Tensor:
        k = x.shape[0]
        ops.rmsnorm_pair(x, self.final_norm, self.hn[:k], self.cfg.eps)
        ops.dense_gemm(ops.dense(self.hn[:k], self.embed, self.logits[:k]), weights_const=True)
        return self.logits[:k]
