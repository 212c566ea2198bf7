"""The model designs this package serves, chosen by a checkpoint directory's ``config.json`` or by the
checkpoint object itself: how each is read, which library its kernels are in, what holds a request's
history and what advances it."""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable

import torch

from .state import DecodeState, HybridState
from .weights import Checkpoint, DokulixCheckpoint, DokulixConfig, FezopelCheckpoint, FezopelConfig


@dataclass(frozen=True)
class Design:
    name: str
    libraries: tuple[str, ...]                    # build targets of its kernels
    checkpoint: type
    matches: Callable[[dict], bool]               # on the parsed config.json
    load: Callable                                # (directory, device) -> checkpoint
    allocate: Callable                            # (config, max_context, device, chunk, dtype) -> state
    dtypes: tuple[torch.dtype, ...]               # activation types it runs in
    chunk_logits: bool                            # whether a chunk returns the logits of its tokens
    model: Callable | None = None                 # (checkpoint, dtype) -> what advances a state by one token and by a chunk


def _load_qwen(path, device):
    from .loader import load_checkpoint, merge_fp8_scales
    ckpt = load_checkpoint(path, device=device)
    merge_fp8_scales(ckpt)            # projections that share an activation share a static FP8 scale
    return ckpt


def _load_hybrid(path, device):
    from .loader import load_hybrid_checkpoint
    return load_hybrid_checkpoint(path, device=device)


def _fezopel(ckpt, dtype):
    from .hybrid import FezopelModel
    return FezopelModel(ckpt, dtype)


def _dokulix(ckpt, dtype):
    from .hybrid import DokulixModel
    return DokulixModel(ckpt, dtype)


def _hybrid(name: str, libraries, checkpoint: type, config: type, model) -> Design:
    return Design(name, libraries, checkpoint, lambda data: data.get("architecture") == config.ARCHITECTURE, _load_hybrid,
                  lambda cfg, max_context, device, chunk, dtype: HybridState(cfg, max_context, device, chunk, dtype),
                  (torch.bfloat16, torch.float32), True, model)


DESIGNS = (
    Design("qwen3-next", ("nvfp4",), Checkpoint, lambda data: "text_config" in data, _load_qwen,
           lambda config, max_context, device, chunk, dtype: DecodeState.allocate(config, max_context, device), (torch.bfloat16,), False),
    _hybrid("fezopel", ("hybrid", "recurrent"), FezopelCheckpoint, FezopelConfig, _fezopel),
    _hybrid("dokulix", ("hybrid", "latent"), DokulixCheckpoint, DokulixConfig, _dokulix),
)


def design_of(ckpt) -> Design:
    for design in DESIGNS:
        if isinstance(ckpt, design.checkpoint):
            return design
    raise ValueError(f"no design for {type(ckpt).__name__}")


def design_of_directory(path: str | Path) -> Design:
    data = json.loads((Path(path) / "config.json").read_text())
    for design in DESIGNS:
        if design.matches(data):
            return design
    raise ValueError(f"{path}: config.json names no design this package serves")
