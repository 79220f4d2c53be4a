"""Decoder families by the architecture name of config.json, and the loader that turns a model folder (config.json +
model.safetensors) into a running decoder."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Mapping, Optional, Tuple

import torch

from ..capi import InferenceSession, SessionOptions
from ..safetensors_lite import load_file
from . import fegilix, llama, rovurax
from .generation import PagedDecoderRunner


@dataclass(frozen=True)
class DecoderFamily:
    """``config(json, dtype, max_seq_len)`` parses config.json; ``build(config, tensors, device)`` returns the packed serving
    graph and its initializers; ``tensors`` None means random weights.  The config object declares what the model keeps per sequence (``cache_tensors()``)."""
    config: Callable[[Mapping[str, Any], str, int], Any]
    build: Callable[[Any, Optional[Mapping[str, torch.Tensor]], str], Tuple[bytes, Dict[str, torch.Tensor]]]


FAMILIES: Dict[str, DecoderFamily] = {}


def register_family(name: str, family: DecoderFamily) -> None:
    FAMILIES[name] = family


register_family("Fegilix", DecoderFamily(fegilix.FegilixConfig.from_json, lambda cfg, w, dev: fegilix.build_fegilix(
    cfg, w if w is not None else fegilix.random_weights(cfg, device=dev, low_rank=fegilix.default_rank(cfg)), device=dev)))
register_family("Rovurax", DecoderFamily(rovurax.RovuraxConfig.from_json, lambda cfg, w, dev: rovurax.build_rovurax(
    cfg, w if w is not None else rovurax.random_weights(cfg, device=dev), device=dev)))
register_family("LlamaForCausalLM", DecoderFamily(
    llama.LlamaConfig.from_json, lambda cfg, w, dev: llama.build_llama(cfg, external_weights=True, device=dev, paged=True, state=w)))

DTYPES = {"bfloat16": "bf16", "float16": "fp16", "float32": "fp32"}


def family_of(config: Mapping[str, Any]) -> DecoderFamily:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in FAMILIES:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(FAMILIES))}")
    return FAMILIES[name]


def create_decoder(config: Mapping[str, Any], tensors: Optional[Mapping[str, torch.Tensor]], dtype: str = "bfloat16", *, batch: int = 1,
                   max_len: int = 2048, max_tokens: Optional[int] = None, block_size: int = 256, provider: str = "CUDAExecutionProvider",
                   cuda_graph: bool = True, session_entries: Optional[Mapping[str, str]] = None) -> PagedDecoderRunner:
    """A decoder with room for ``batch`` sequences of at most ``max_len`` tokens; ``max_tokens`` bounds the tokens that all
    of them hold together (default: no further bound).  float32 runs every product in true 32-bit."""
    family = family_of(config)
    per_seq = (max_len + block_size - 1) // block_size
    cfg = family.config(config, DTYPES[dtype], per_seq * block_size)
    gpu = provider == "CUDAExecutionProvider"
    model, weights = family.build(cfg, tensors, "cuda" if gpu else "cpu")
    so = SessionOptions()
    so.add_external_initializers(list(weights.keys()), list(weights.values()))
    for k, v in {"ortb200.pdl": "1", **(session_entries or {})}.items():
        so.add_session_config_entry(k, v)
    options = {"use_tf32": "0", "enable_cuda_graph": "1" if cuda_graph else "0"} if gpu else {}
    sess = InferenceSession(model, so, providers=[(provider, options)], enable_fallback=False)
    num_blocks = batch * per_seq
    if max_tokens is not None:   # every sequence may leave its last block partly filled
        num_blocks = min(num_blocks, (max_tokens + block_size - 1) // block_size + batch)
    return PagedDecoderRunner(sess, cfg, batch, max_len, block_size=block_size, num_blocks=num_blocks)


def load_decoder(path: str, dtype: str = "bfloat16", **kw) -> PagedDecoderRunner:
    """``create_decoder`` from a folder with config.json and model.safetensors."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    return create_decoder(config, load_file(os.path.join(path, "model.safetensors")), dtype, **kw)
