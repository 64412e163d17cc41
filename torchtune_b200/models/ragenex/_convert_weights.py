"""Tensor names of Ragenex checkpoints ↔ this package's state-dict keys.  Layouts are the same on both sides (``[out, in]`` matrices, heads
stacked along the rows, mixing weights ``[from, to]``)."""
from __future__ import annotations

import re
from typing import Any, Dict, Mapping, Optional

import torch

_LAYER = {
    "norm1": "sa_norm.scale",
    "ls1": "sa_scale.scale",
    "hc1.in": "sa_streams.read",
    "hc1.out": "sa_streams.write",
    "hc1.mix": "sa_streams.mix",
    "norm2": "mlp_norm.scale",
    "ls2": "mlp_scale.scale",
    "hc2.in": "mlp_streams.read",
    "hc2.out": "mlp_streams.write",
    "hc2.mix": "mlp_streams.mix",
    "mix.q": "attn.q_proj.weight",
    "mix.k": "attn.k_proj.weight",
    "mix.v": "attn.v_proj.weight",
    "mix.g": "attn.gate_proj.weight",
    "mix.o": "attn.output_proj.weight",
    "mix.q.norm": "attn.q_norm.scale",
    "mix.k.norm": "attn.k_norm.scale",
    "mix.norm": "attn.norm.scale",
    "mlp.gate": "mlp.w1.weight",
    "mlp.up": "mlp.w3.weight",
    "mlp.down": "mlp.w2.weight",
}
_TOP = {"embed": "tok_embeddings.weight", "pos": "pos_embeddings.weight", "final.norm": "norm.scale", "head": "output.weight"}
_LAYER_BACK = {v: k for k, v in _LAYER.items()}
_TOP_BACK = {v: k for k, v in _TOP.items()}


_FEED_FORWARD = ("norm2", "ls2", "hc2.", "mlp.")


def ragenex_hf_to_tune(state_dict: Dict[str, torch.Tensor], config: Optional[Mapping[str, Any]] = None) -> Dict[str, torch.Tensor]:
    """With the model's ``config``, tensors around a feed-forward block that a layer does not have are left out."""
    layers = (config or {}).get("layers") or []
    bare = {i for i, layer in enumerate(layers) if layer.get("mlp") is None}
    out = {}
    for key, value in state_dict.items():
        m = re.fullmatch(r"l(\d+)\.(.+)", key)
        if m and int(m.group(1)) in bare and m.group(2).startswith(_FEED_FORWARD):
            continue
        if m and m.group(2) in _LAYER:
            out[f"layers.{m.group(1)}.{_LAYER[m.group(2)]}"] = value
        elif key in _TOP:
            out[_TOP[key]] = value
        else:
            raise ValueError(f"unexpected tensor {key!r} in a Ragenex checkpoint")
    return out


def ragenex_tune_to_hf(state_dict: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    out = {}
    for key, value in state_dict.items():
        m = re.fullmatch(r"layers\.(\d+)\.(.+)", key)
        if m and m.group(2) in _LAYER_BACK:
            out[f"l{m.group(1)}.{_LAYER_BACK[m.group(2)]}"] = value
        elif key in _TOP_BACK:
            out[_TOP_BACK[key]] = value
        else:
            raise ValueError(f"{key!r} has no place in a Ragenex checkpoint")
    return out


def _register() -> None:
    from ...training.checkpointing._codecs import register_hf_codec
    from ...training.checkpointing._utils import ModelType

    register_hf_codec(ModelType.RAGENEX, lambda sd, cfg: ragenex_hf_to_tune(sd, cfg), lambda sd, cfg: ragenex_tune_to_hf(sd))


_register()
