"""``ragenex(config)`` / ``lora_ragenex(..., config=...)`` from a ``config.json`` (a mapping or the path of the file)."""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Union

from torch import nn

from ...modules import ClampedGLU, LightningAttention, QueryTemperature, RMSNorm, SpanAttention, StreamLayerNorm
from .._factory import AdapterSpec, DecoderArch, build_mlp
from .._generic import component_builders
from .._registry import as_mapping

_MIXERS = ("attention", "lightning")
_PROJECTIONS = {"q_proj", "k_proj", "v_proj", "gate_proj", "output_proj"}
_GLU_ALPHA = 1.702


def _check(cfg: Mapping[str, Any], layers: List[Dict[str, Any]]) -> None:
    for i, layer in enumerate(layers):
        if layer["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        mix = layer["mixer"]
        if layer["type"] == "attention" and int(mix["heads"]) % int(mix["kv_heads"]):
            raise ValueError(f"layer {i}: {mix['heads']} query heads do not share {mix['kv_heads']} key heads evenly")
        if layer["type"] == "lightning" and len(mix["decay"]) != int(mix["heads"]):
            raise ValueError(f"layer {i}: {len(mix['decay'])} decays for {mix['heads']} heads")
    if int(cfg.get("streams") or 1) < 1:
        raise ValueError(f"{cfg['streams']} residual streams")
    loop = cfg.get("loop")
    if loop is not None and not 0 <= int(loop["start"]) < int(loop["stop"]) <= len(layers):
        raise ValueError(f"the repeated layers {loop['start']} … {loop['stop']} are outside the {len(layers)} layers of the model")


def _arch(config: Union[str, Mapping[str, Any]], max_seq_len: Optional[int] = None) -> DecoderArch:
    cfg = as_mapping(config)
    layers, dim, eps, table = cfg["layers"], int(cfg["width"]), float(cfg["norm"]["eps"]), int(cfg["max_positions"])
    _check(cfg, layers)

    def mixer(idx: int, ad: AdapterSpec) -> nn.Module:
        kind, mix, mods = layers[idx]["type"], layers[idx]["mixer"], set(ad.attn_modules)
        if mods - _PROJECTIONS:
            raise ValueError(f"unknown attention modules for LoRA: {sorted(mods - _PROJECTIONS)}")
        H, d, dv = (int(mix[k]) for k in ("heads", "dim", "vdim"))
        G = int(mix["kv_heads"]) if kind == "attention" else H
        shared = dict(
            embed_dim=dim, num_heads=H, key_dim=d, value_dim=dv,
            q_proj=ad.make(dim, H * d, "q_proj" in mods), k_proj=ad.make(dim, G * d, "k_proj" in mods), v_proj=ad.make(dim, G * dv, "v_proj" in mods),
            output_proj=ad.make(H * dv, dim, "output_proj" in mods),
        )
        if kind == "lightning":
            return LightningAttention(**shared, decay=[float(z) for z in mix["decay"]], gate_proj=ad.make(dim, H * dv, "gate_proj" in mods), norm=RMSNorm(H * dv, eps=eps))
        temp = mix.get("q_temp")
        return SpanAttention(**shared, num_kv_heads=G, scale=float(mix["scale"]), q_norm=RMSNorm(H * d, eps=eps), k_norm=RMSNorm(G * d, eps=eps),
                             temperature=None if temp is None else QueryTemperature(temp["coef"], temp["every"]))

    def feed_forward(idx: int, ad: AdapterSpec) -> Optional[nn.Module]:
        mlp = layers[idx].get("mlp")
        return None if mlp is None else build_mlp(dim, int(mlp["ff"]), ad, ClampedGLU(mlp["limit"], _GLU_ALPHA))

    first, loop = layers[0]["mixer"], cfg.get("loop")
    return DecoderArch(
        vocab_size=int(cfg["vocab"]), num_layers=len(layers), num_heads=int(first["heads"]), num_kv_heads=int(first.get("kv_heads", first["heads"])), embed_dim=dim,
        max_seq_len=table if max_seq_len is None else min(max_seq_len, table), head_dim=int(first["dim"]), norm_eps=eps, norm=lambda d, e: StreamLayerNorm(d, eps=e),
        attn_factory=mixer, mlp_factory=feed_forward, streams=int(cfg.get("streams") or 1), learned_positions=table,
        loop=None if loop is None else (int(loop["start"]), int(loop["stop"]), int(loop["times"])), wide_logits=True,
    )


ragenex, lora_ragenex = component_builders("ragenex", _arch, "Ragenex decoder described by a ``config.json`` (mapping, file or folder).")
