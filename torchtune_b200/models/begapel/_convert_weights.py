"""Tensor names of Begapel checkpoints ↔ this package's state-dict keys.  Layouts are the same on both sides (interleaved rotation,
``[out, in]`` matrices, heads stacked along the rows)."""
from __future__ import annotations

import re
from typing import Dict

import torch

_LAYER = {
    "norm1": "sa_norm.scale",
    "norm1b": "sa_scale.scale",
    "norm2": "mlp_norm.scale",
    "norm2b": "mlp_scale.scale",
    "mix.q": "attn.q_proj.weight",
    "mix.dkv": "attn.kv_down.weight",
    "mix.dkv.norm": "attn.kv_norm.scale",
    "mix.uk": "attn.k_up.weight",
    "mix.uv": "attn.v_up.weight",
    "mix.g": "attn.gate_proj.weight",
    "mix.o": "attn.output_proj.weight",
    "mlp.gate": "mlp.w1.weight",
    "mlp.up": "mlp.w3.weight",
    "mlp.down": "mlp.w2.weight",
}
_TOP = {"embed": "tok_embeddings.weight", "final.norm": "norm.scale", "head": "output.weight"}
_LAYER_BACK = {v: k for k, v in _LAYER.items()}
_TOP_BACK = {v: k for k, v in _TOP.items()}


def begapel_hf_to_tune(state_dict: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    out = {}
    for key, value in state_dict.items():
        m = re.fullmatch(r"l(\d+)\.(.+)", key)
        if m and m.group(2) in _LAYER:
            out[f"layers.{m.group(1)}.{_LAYER[m.group(2)]}"] = value
        elif key in _TOP:
            out[_TOP[key]] = value
        else:
            raise ValueError(f"unexpected tensor {key!r} in a Begapel checkpoint")
    return out


def begapel_tune_to_hf(state_dict: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    out = {}
    for key, value in state_dict.items():
        m = re.fullmatch(r"layers\.(\d+)\.(.+)", key)
        if m and m.group(2) in _LAYER_BACK:
            out[f"l{m.group(1)}.{_LAYER_BACK[m.group(2)]}"] = value
        elif key in _TOP_BACK:
            out[_TOP_BACK[key]] = value
        else:
            raise ValueError(f"{key!r} has no place in a Begapel checkpoint")
    return out


def _register() -> None:
    from ...training.checkpointing._codecs import register_hf_codec
    from ...training.checkpointing._utils import ModelType

    register_hf_codec(ModelType.BEGAPEL, lambda sd, cfg: begapel_hf_to_tune(sd), lambda sd, cfg: begapel_tune_to_hf(sd))


_register()
