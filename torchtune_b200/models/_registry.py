"""Models by the ``architecture`` their ``config.json`` names.

YAML configs name a builder; a checkpoint folder names only its architecture.  This table leads from the one to the other: builder, weight
conversion rules, and :func:`load_pretrained`, which does what the recipes do with the same parts (checkpointer, builder, default dtype)."""
from __future__ import annotations

import importlib
import json
import tempfile
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Dict, Mapping, Optional, Union

import torch
from torch import nn


@dataclass(frozen=True)
class Architecture:
    builder: str  # dotted path of builder(config, max_seq_len=...)
    model_type: str  # name of the ModelType whose rules convert the weights


ARCHITECTURES: Dict[str, Architecture] = {
    "Begapel": Architecture("torchtune_b200.models.begapel.begapel", "BEGAPEL"),
    "Ragenex": Architecture("torchtune_b200.models.ragenex.ragenex", "RAGENEX"),
}


def read_config(folder: Union[str, Path]) -> Dict[str, Any]:
    return as_mapping(Path(folder) / "config.json")


def as_mapping(config: Union[str, Path, Mapping[str, Any]]) -> Dict[str, Any]:
    """A model configuration given as a mapping, a ``config.json`` or the folder that holds one."""
    if isinstance(config, (str, Path)):
        path = Path(config)
        return json.loads((path / "config.json" if path.is_dir() else path).read_text())
    if hasattr(config, "to_dict"):
        return config.to_dict()
    from ..config import DictConfig, OmegaConf

    return OmegaConf.to_container(config) if isinstance(config, DictConfig) else dict(config)


def architecture_of(config: Dict[str, Any]) -> Architecture:
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"no model of this package has the architecture {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name]


def build_from_config(config: Dict[str, Any], **kwargs: Any) -> nn.Module:
    module, _, name = architecture_of(config).builder.rpartition(".")
    return getattr(importlib.import_module(module), name)(config, **kwargs)


def load_pretrained(folder: Union[str, Path], *, dtype: torch.dtype, device: torch.device, max_seq_len: Optional[int] = None) -> nn.Module:
    """Model of a checkpoint folder (``config.json`` and ``*.safetensors``) in evaluation mode on ``device``."""
    from ..training import FullModelHFCheckpointer, set_default_dtype

    folder = Path(folder)
    config = read_config(folder)
    files = sorted(p.name for p in folder.glob("*.safetensors"))
    if not files:
        raise FileNotFoundError(f"no *.safetensors file in {folder}")
    with tempfile.TemporaryDirectory() as scratch:  # the checkpointer wants a place to write to; nothing is written when loading
        state = FullModelHFCheckpointer(str(folder), files, architecture_of(config).model_type, output_dir=scratch).load_checkpoint()["model"]
    with set_default_dtype(dtype), device:
        model = build_from_config(config, **({} if max_seq_len is None else {"max_seq_len": max_seq_len}))
    model.load_state_dict(state)
    return model.eval()
