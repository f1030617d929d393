"""Which classes implement which architecture.

``config.json`` (or an inline dict) selects the entry: the key ``architecture`` names a listed design, anything else is
the dense Qwen2 / Llama family. The engine, the checkpoint reader, the command line and the launchers go through here,
so a new design needs one entry and no change in any of them.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Optional

from . import dezelorn, vazatar
from .config import PRESETS as DENSE_PRESETS
from .config import ModelConfig
from .layout import ParamLayout


def _dense_engine() -> Any:
    from ..engine.engine import RolloutEngine

    return RolloutEngine


def _listed_engine() -> Any:
    from ..engine.listed import ListedEngine

    return ListedEngine


def _dense_decoder() -> Any:
    from .decoder import NativeDecoder

    return NativeDecoder


def _dezelorn_decoder() -> Any:
    from .dezelorn_decoder import DezelornDecoder

    return DezelornDecoder


def _vazatar_decoder() -> Any:
    from .vazatar_decoder import VazatarDecoder

    return VazatarDecoder


@dataclass(frozen=True)
class Architecture:
    name: str
    config_from_dict: Callable[[Dict[str, Any]], Any]
    layout: Callable[..., ParamLayout]
    engine: Callable[[], Any]         # returns the engine class (imported on demand: it needs the extension)
    decoder: Callable[[], Any]        # returns the executor class, likewise
    trainable: bool                   # has a backward pass (trainer role) and a dense logprob forward
    dtypes: tuple                     # parameter types that the native engine runs


ARCHITECTURES: Dict[str, Architecture] = {
    "dense": Architecture("dense", ModelConfig.from_dict, ParamLayout, _dense_engine, _dense_decoder, True, ("bfloat16",)),
    "Dezelorn": Architecture("Dezelorn", dezelorn.DezelornConfig.from_dict, dezelorn.DezelornLayout, _listed_engine, _dezelorn_decoder, False,
                             ("bfloat16", "float32")),
    "Vazatar": Architecture("Vazatar", vazatar.VazatarConfig.from_dict, vazatar.VazatarLayout, _listed_engine, _vazatar_decoder, False,
                            ("bfloat16", "float32")),
}

LISTED_PRESETS: Dict[str, Any] = {**dezelorn.PRESETS, **vazatar.PRESETS}
PRESETS: Dict[str, Any] = {**DENSE_PRESETS, **LISTED_PRESETS}


def architecture_of(cfg: Any) -> Architecture:
    return ARCHITECTURES[getattr(cfg, "architecture", "dense")]


def config_from_dict(d: Dict[str, Any]) -> Any:
    if "preset" in d and d["preset"] in LISTED_PRESETS:
        base = LISTED_PRESETS[d["preset"]].to_hf_dict()
        base.update({k: v for k, v in d.items() if k != "preset"})
        d = base
    name = d.get("architecture")
    if name is None:
        return ModelConfig.from_dict(d)
    if name not in ARCHITECTURES or name == "dense":
        raise ValueError(f"unknown architecture {name!r} (known: {sorted(set(ARCHITECTURES) - {'dense'})})")
    return ARCHITECTURES[name].config_from_dict(d)


def resolve_model_config(model_name_or_path: Optional[str], inline: Optional[Dict[str, Any]] = None) -> Any:
    """Inline dict wins; otherwise a preset name or a directory holding ``config.json``."""
    if inline:
        return config_from_dict(inline)
    if model_name_or_path in PRESETS:
        return PRESETS[model_name_or_path]
    if model_name_or_path and os.path.isdir(model_name_or_path):
        with open(os.path.join(model_name_or_path, "config.json"), "r", encoding="utf-8") as f:
            return config_from_dict(json.load(f))
    raise FileNotFoundError(f"cannot resolve model config from {model_name_or_path!r}")


def make_layout(cfg: Any, shard_world: int = 1) -> ParamLayout:
    return architecture_of(cfg).layout(cfg, shard_world)


def require_trainable(cfg: Any) -> None:
    a = architecture_of(cfg)
    if not a.trainable:
        raise NotImplementedError(f"{a.name} has no backward pass here: it is served (generation command line, trace runner, "
                                  "rollout engine), not trained")


def build_engine(cfg: Any, layout: ParamLayout, params: Any, **kw: Any) -> Any:
    """The architecture's engine over a flat parameter buffer on the GPU."""
    return architecture_of(cfg).engine()(cfg, layout, params, **kw)
