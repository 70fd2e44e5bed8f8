"""Model designs by name: which class packs a checkpoint, in which precisions it runs.

A configuration names its design in ``architecture`` (or a list ``architectures``); one without either is a Llama, as in
the reference (``tvm/llama_auto_batcher/llama_for_causal_lm.py:10-21``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable

import torch

from . import checkpoint
from .model import PackedLlama
from .relidra import PackedRelidra
from .tevudra import PackedTevudra


@dataclass(frozen=True)
class Design:
    name: str
    pack: Callable     # (config, weights, adapters, scales, device, dtype) -> packed model with new_cache / new_engine
    dtypes: tuple
    adapters: bool     # takes LoRA adapters


def _pack_llama(cfg, weights, adapters, scales, device, dtype):
    return PackedLlama(cfg, weights, adapters, scales, device=device)


def _pack_tevudra(cfg, weights, adapters, scales, device, dtype):
    return PackedTevudra(cfg, weights, device=device, dtype=dtype)


def _pack_relidra(cfg, weights, adapters, scales, device, dtype):
    return PackedRelidra(cfg, weights, device=device, dtype=dtype)


DESIGNS = {d.name: d for d in (
    Design("LlamaForCausalLM", _pack_llama, (torch.bfloat16,), True),
    Design("Tevudra", _pack_tevudra, PackedTevudra.dtypes, False),
    Design("Relidra", _pack_relidra, PackedRelidra.dtypes, False),
)}


class UnsupportedPrecision(ValueError):
    """The design does not run in the precision asked for."""


def design_of(cfg: dict) -> Design:
    name = cfg.get("architecture") or (cfg.get("architectures") or ["LlamaForCausalLM"])[0]
    if name not in DESIGNS:
        raise ValueError(f"unknown model design {name!r} (known: {', '.join(sorted(DESIGNS))})")
    return DESIGNS[name]


def build_model(cfg: dict, weights: dict, adapters=(), scales=(), device="cuda", dtype=torch.bfloat16):
    """Packs ``weights`` on the device for the design ``cfg`` names."""
    d = design_of(cfg)
    if dtype not in d.dtypes:
        raise UnsupportedPrecision(f"{d.name} does not run in {dtype}")
    if len(adapters) and not d.adapters:
        raise ValueError(f"{d.name} takes no adapters")
    return d.pack(cfg, weights, adapters, scales, device, dtype)


def load_model(model_dir: str, device="cuda", dtype=torch.bfloat16):
    """A packed model from a folder with ``config.json`` and ``model.safetensors``."""
    cfg = checkpoint.read_config(model_dir)
    if dtype not in design_of(cfg).dtypes:
        raise UnsupportedPrecision(f"{design_of(cfg).name} does not run in {dtype}")
    return build_model(cfg, checkpoint.read_tensors(model_dir), device=device, dtype=dtype)
