"""Builds an engine from a model directory or preset name: what the generation command line and the trace runner share."""
from __future__ import annotations

import os
from typing import Any, Optional

import torch

from . import checkpoint as ckpt
from .models.registry import architecture_of, build_engine, make_layout, resolve_model_config

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedDtype(ValueError):
    """The architecture's engine does not run this parameter type."""


def load_engine(model: str, dtype: str = "bfloat16", device: str = "cuda:0", seed: int = 0, max_model_len: Optional[int] = None,
                **engine_kw: Any) -> Any:
    """Engine over the weights in ``model`` (a directory with config.json and safetensors, or a preset name with random
    weights from ``seed``)."""
    cfg = resolve_model_config(model)
    if dtype not in architecture_of(cfg).dtypes:
        raise UnsupportedDtype(f"{architecture_of(cfg).name} models do not run in {dtype} (supported: {architecture_of(cfg).dtypes})")
    if not torch.cuda.is_available():
        raise RuntimeError("the native engine needs a CUDA device")
    dev = torch.device(device)
    torch.cuda.set_device(dev)
    layout = make_layout(cfg)
    if os.path.isdir(model) and any(f.endswith(".safetensors") for f in os.listdir(model)):
        params = ckpt.load_hf_model(model, layout).to(DTYPES[dtype]).to(dev)
    else:
        params = torch.empty(layout.total, dtype=DTYPES[dtype], device=dev)
        layout.init_random_device_(params, seed)
    return build_engine(cfg, layout, params, max_model_len=min(max_model_len or cfg.max_position_embeddings, cfg.max_position_embeddings),
                        **engine_kw)
