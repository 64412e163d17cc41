"""``begapel(config)`` / ``lora_begapel(..., config=...)`` from a ``config.json`` (a mapping or the path of the file)."""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Tuple, Union

from torch import nn

from ...modules import LatentAttention, RMSNorm, StreamRMSNorm
from ...modules.latent_attention import PreciseRotaryPositionalEmbeddings
from .._factory import AdapterSpec, DecoderArch, build_mlp
from .._generic import component_builders
from .._registry import as_mapping

_MIXER = "latent_attention"
_ATTN_MODULES = {"q_proj", "kv_down", "k_up", "v_up", "gate_proj", "output_proj"}


def _check_layers(layers: List[Dict[str, Any]]) -> None:
    for i, layer in enumerate(layers):
        if layer["type"] != _MIXER:
            raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        mix = layer["mixer"]
        if mix["rot"]["dims"] > mix["rot_dim"] or mix["rot"]["dims"] % 2:
            raise ValueError(f"layer {i}: {mix['rot']['dims']} rotated dimensions do not fit a rotated part of {mix['rot_dim']}")
        source = mix.get("kv_from")
        if source is None:
            continue
        if not 0 <= source < i:
            raise ValueError(f"layer {i} takes its latents from layer {source}, which does not come before it")
        other = layers[source]["mixer"]
        if other.get("kv_from") is not None:
            raise ValueError(f"layer {i} takes its latents from layer {source}, which has none of its own")
        for key in ("kv_rank", "rot_dim", "rot"):
            if other[key] != mix[key]:
                raise ValueError(f"layers {i} and {source} share latents but differ in {key}")


def _arch(config: Union[str, Mapping[str, Any]], max_seq_len: int = 32768) -> DecoderArch:
    cfg = as_mapping(config)
    layers, dim, eps = cfg["layers"], int(cfg["width"]), float(cfg["norm"]["eps"])
    _check_layers(layers)
    ropes: Dict[Tuple[int, float], nn.Module] = {}

    def rope(rot: Mapping[str, Any]) -> nn.Module:
        key = (int(rot["dims"]), float(rot["base"]))
        if key not in ropes:
            ropes[key] = PreciseRotaryPositionalEmbeddings(dim=key[0], max_seq_len=max_seq_len, base=key[1])
        return ropes[key]

    def attention(idx: int, ad: AdapterSpec) -> nn.Module:
        mix, mods = layers[idx]["mixer"], set(ad.attn_modules)
        if mods - _ATTN_MODULES:
            raise ValueError(f"unknown attention modules for LoRA: {sorted(mods - _ATTN_MODULES)}")
        H, d, r, dv, rank = (int(mix[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        own = mix.get("kv_from") is None
        return LatentAttention(
            embed_dim=dim, num_heads=H, head_dim=d, rot_dim=r, value_dim=dv, kv_rank=rank,
            q_proj=ad.make(dim, H * (d + r), "q_proj" in mods),
            kv_down=ad.make(dim, rank + r, "kv_down" in mods) if own else None,
            kv_norm=RMSNorm(rank, eps=eps) if own else None,
            k_up=ad.make(rank, H * d, "k_up" in mods),
            v_up=ad.make(rank, H * dv, "v_up" in mods),
            gate_proj=ad.make(dim, H * dv, "gate_proj" in mods),
            output_proj=ad.make(H * dv, dim, "output_proj" in mods),
            pos_embeddings=rope(mix["rot"]), scale=float(mix["scale"]), layer_index=idx, latent_from=None if own else int(mix["kv_from"]),
        )

    def feed_forward(idx: int, ad: AdapterSpec):
        mlp = layers[idx].get("mlp")
        return None if mlp is None else build_mlp(dim, int(mlp["ff"]), ad)

    first = layers[0]["mixer"]
    return DecoderArch(
        vocab_size=int(cfg["vocab"]), num_layers=len(layers), num_heads=int(first["heads"]), num_kv_heads=int(first["heads"]), embed_dim=dim, max_seq_len=max_seq_len,
        head_dim=int(first["dim"]) + int(first["rot_dim"]), norm_eps=eps, norm=lambda d, e: StreamRMSNorm(d, eps=e, zero_centered=True),
        attn_factory=attention, mlp_factory=feed_forward, post_norms=True, residual_stream=True, residual_mult=float(cfg["residual_mult"]),
        logit_softcap=float(cfg.get("logit_softcap") or 0.0), wide_logits=True,
    )


begapel, lora_begapel = component_builders("begapel", _arch, "Begapel decoder described by a ``config.json`` (mapping, file or folder).")
