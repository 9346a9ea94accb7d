"""Models by the architecture their config.json names: configuration, weights, and a model ready to run.

    model = registry.load(model_dir, dtype=torch.bfloat16, max_len=4096, cache_tokens=65536)
"""
from __future__ import annotations

import glob
import json
import os
from dataclasses import dataclass
from typing import Callable

import torch

from . import _native, weights
from .step_model import StepModel


@dataclass(frozen=True)
class Sizes:
    """What a caller decides about a model it loads."""

    max_len: int          # longest sequence
    cache_tokens: int     # tokens that live sequences hold at any time
    max_tokens: int       # token rows of one step
    max_sequences: int    # sequences of one step


@dataclass(frozen=True)
class Architecture:
    build: Callable[[dict, str, Sizes, torch.dtype, str], StepModel]
    dtypes: tuple
    kernels: str | None = None  # the subset of the library that the model needs; None: all of it


ARCHITECTURES: dict[str, Architecture] = {}


def register(name: str, **kw):
    def wrap(build):
        ARCHITECTURES[name] = Architecture(build, **kw)
        return build
    return wrap


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def architecture_of(config: dict) -> str:
    """`architecture`, or the first of a Hugging Face config's `architectures`."""
    name = config.get("architecture") or next(iter(config.get("architectures", [])), None)
    if name not in ARCHITECTURES:
        raise ValueError(f"architecture {name!r} is not one of {sorted(ARCHITECTURES)}")
    return name


def read_tensors(model_dir: str) -> dict:
    files = sorted(glob.glob(os.path.join(model_dir, "*.safetensors")))
    if not files:
        raise FileNotFoundError(f"{model_dir} holds no .safetensors file")
    out = {}
    for f in files:
        out.update(weights.read_safetensors(f))
    return out


def num_blocks(sizes: Sizes, block_size: int) -> int:
    """Pages for cache_tokens tokens: a part-filled page per sequence and the padding page on top."""
    return -(-sizes.cache_tokens // block_size) + sizes.max_sequences + 1


def load(model_dir: str, *, dtype: torch.dtype = torch.bfloat16, max_len: int = 4096, cache_tokens: int | None = None,
         max_tokens: int = 2048, max_sequences: int = 64, device: str = "cuda:0") -> StepModel:
    config = read_config(model_dir)
    arch = ARCHITECTURES[architecture_of(config)]
    if dtype not in arch.dtypes:
        raise ValueError(f"{architecture_of(config)} does not run in {dtype}")
    _native.select(arch.kernels)
    sizes = Sizes(max_len, cache_tokens if cache_tokens is not None else max_len * 4, max_tokens, max_sequences)
    return arch.build(config, model_dir, sizes, dtype, device)


@register("LlamaForCausalLM", dtypes=(torch.bfloat16,))
def _llama(config: dict, model_dir: str, sizes: Sizes, dtype: torch.dtype, device: str) -> StepModel:
    """int8 per-channel projections quantized from the checkpoint, bf16 pools."""
    from .decoder import Decoder, DecoderConfig

    if config.get("rope_scaling") or config.get("rope_parameters", {}).get("rope_type", "default") != "default":
        raise ValueError("LlamaForCausalLM: scaled rotary positions are not built")
    heads = config["num_attention_heads"]
    cfg = DecoderConfig(num_layers=config["num_hidden_layers"], d_model=config["hidden_size"], num_heads=heads,
                        num_kv_heads=config.get("num_key_value_heads", heads), head_dim=config.get("head_dim") or config["hidden_size"] // heads,
                        ffn=config["intermediate_size"], vocab=config["vocab_size"], rms_eps=config.get("rms_norm_eps", 1e-5),
                        rope_theta=config.get("rope_theta", config.get("rope_parameters", {}).get("rope_theta", 10000.0)), head_quant=True, max_positions=sizes.max_len)
    model = Decoder(cfg, min(sizes.max_sequences, 128), num_blocks(sizes, cfg.block_size), -(-sizes.max_len // cfg.block_size), device=device)
    model.load_host_weights(weights.quantize_checkpoint(read_tensors(model_dir), cfg.num_layers, head_quant=True,
                                                        tie_word_embeddings=bool(config.get("tie_word_embeddings"))))
    return model


@register("Marotar", dtypes=(torch.bfloat16, torch.float32), kernels="latent")
def _marotar(config: dict, model_dir: str, sizes: Sizes, dtype: torch.dtype, device: str) -> StepModel:
    """Latent attention through sliding windows beside a squared-ReLU feed-forward, tied embeddings."""
    from .latent_decoder import LatentDecoder, LatentDecoderConfig

    cfg = LatentDecoderConfig.from_config(config)
    model = LatentDecoder(cfg, num_blocks=num_blocks(sizes, cfg.block_size), max_len=sizes.max_len, max_tokens=sizes.max_tokens,
                          max_sequences=sizes.max_sequences, dtype=dtype, device=device)
    model.load_tensors(read_tensors(model_dir))
    return model


@register("Videdra", dtypes=(torch.bfloat16, torch.float32), kernels="mixed")
def _videdra(config: dict, model_dir: str, sizes: Sizes, dtype: torch.dtype, device: str) -> StepModel:
    """Differential attention and retention in any order, dense and expert feed-forwards, norms on both sides of every branch."""
    from .mixed_decoder import MixedDecoder, MixedDecoderConfig

    cfg = MixedDecoderConfig.from_config(config)
    model = MixedDecoder(cfg, num_blocks=num_blocks(sizes, cfg.block_size), max_len=sizes.max_len, max_tokens=sizes.max_tokens,
                         max_sequences=sizes.max_sequences, dtype=dtype, device=device)
    model.load_tensors(read_tensors(model_dir))
    return model
