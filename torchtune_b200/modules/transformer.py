"""Decoder layers and the decoder stack (parity: torchtune/modules/transformer.py:17-689)."""
from __future__ import annotations

import copy
from typing import Callable, List, Optional, Tuple, Union

import torch
from torch import nn

from .. import ops
from ..ops.mask import AttentionMask
from .attention import MaskLike, MultiHeadAttention
from .cached_mixer import CachedMixer
from .hyper_connections import HyperConnection, LayerScale, StreamEntry
from .rms_norm import StreamLayerNorm, StreamRMSNorm


class TransformerSelfAttentionLayer(nn.Module):
    """Pre-norm block: ``h = x + sa_scale(attn(sa_norm(x)))``, ``out = h + mlp_scale(mlp(mlp_norm(h)))``.

    ``mask_mod(mask, bsz, seq_len)`` may rewrite the mask for this layer only (Llama-4
    local attention layers)."""

    def __init__(
        self,
        attn: MultiHeadAttention,
        mlp: nn.Module,
        *,
        sa_norm: Optional[nn.Module] = None,
        mlp_norm: Optional[nn.Module] = None,
        sa_scale: Optional[nn.Module] = None,
        mlp_scale: Optional[nn.Module] = None,
        mask_mod: Optional[Callable[[MaskLike, int, int], MaskLike]] = None,
    ) -> None:
        super().__init__()
        self.attn = attn
        self.mlp = mlp
        self.sa_norm = sa_norm or nn.Identity()
        self.mlp_norm = mlp_norm or nn.Identity()
        self.sa_scale = sa_scale or nn.Identity()
        self.mlp_scale = mlp_scale or nn.Identity()
        self.mask_mod = mask_mod

    def setup_caches(self, batch_size: int, dtype: torch.dtype, *, encoder_max_seq_len: int, decoder_max_seq_len: int) -> None:
        self.attn.setup_cache(batch_size, dtype, max_seq_len=decoder_max_seq_len)

    def caches_are_setup(self) -> bool:
        return self.attn.kv_cache is not None

    def caches_are_enabled(self) -> bool:
        return self.attn.cache_enabled

    def reset_cache(self) -> None:
        self.attn.reset_cache()

    @property
    def _fuse_residual_attn(self) -> bool:
        # exact types only: converted or derived modules (tensor-parallel attention, adapters on the whole block) keep the plain path
        return type(self.sa_scale) is nn.Identity and type(self.attn) is MultiHeadAttention

    @property
    def _fuse_residual_mlp(self) -> bool:
        from .feed_forward import FeedForward

        return type(self.mlp_scale) is nn.Identity and type(self.mlp) is FeedForward

    def forward(self, x: torch.Tensor, *, mask: MaskLike = None, input_pos: Optional[torch.Tensor] = None, **kwargs) -> torch.Tensor:
        if self.mask_mod is not None:
            mask = self.mask_mod(mask, x.shape[0], x.shape[1])
        normed = self.sa_norm(x)
        # Without layer scales the two residual additions ride in the epilogues of the attention output projection and of the MLP down
        # projection (modules that take a ``residual`` argument); otherwise they are separate additions.
        if self._fuse_residual_attn:
            h = self.attn(normed, normed, mask=mask, input_pos=input_pos, residual=x)
        else:
            h = self.sa_scale(self.attn(normed, normed, mask=mask, input_pos=input_pos)) + x
        if self._fuse_residual_mlp:
            return self.mlp(self.mlp_norm(h), residual=h)
        return h + self.mlp_scale(self.mlp(self.mlp_norm(h)))


class ResidualStreamLayer(TransformerSelfAttentionLayer):
    """Decoder layer on a 32-bit residual stream with a norm on both sides of each sublayer:
    ``x = x + m · sa_scale(attn(sa_norm(x)))``, then ``x = x + m · mlp_scale(mlp(mlp_norm(x)))`` (left out with ``mlp=None``).

    All four norms are :class:`~torchtune_b200.modules.StreamRMSNorm`, so the end of one sublayer and the norm in front of the next run
    as one pass over the stream.  A decoder that chains layers passes ``(x, sa_norm(x))`` and the norm that follows this layer, and
    receives the same kind of pair for the next one."""

    def __init__(self, attn: nn.Module, mlp: Optional[nn.Module], *, sa_norm: nn.Module, sa_scale: nn.Module, mlp_norm: Optional[nn.Module] = None, mlp_scale: Optional[nn.Module] = None,
                 residual_mult: float = 1.0) -> None:
        nn.Module.__init__(self)
        if (mlp is None) != (mlp_norm is None) or (mlp is None) != (mlp_scale is None):
            raise ValueError("the feed-forward block and its two norms come together")
        self.attn, self.mlp = attn, mlp
        self.sa_norm, self.sa_scale, self.mlp_norm, self.mlp_scale = sa_norm, sa_scale, mlp_norm, mlp_scale
        self.mask_mod = None
        self.residual_mult = float(residual_mult)

    def forward(self, x, *, mask: MaskLike = None, input_pos: Optional[torch.Tensor] = None, layer_state: Optional[dict] = None, next_norm: Optional[nn.Module] = None, **kwargs):
        x, normed = x if isinstance(x, tuple) else (x.float(), None)
        if normed is None:
            normed = self.sa_norm(x)
        chain, m = StreamRMSNorm.chain, self.residual_mult
        x, normed = chain(x, self.attn(normed, mask=mask, input_pos=input_pos, layer_state=layer_state), self.sa_scale, m, next_norm if self.mlp is None else self.mlp_norm)
        if self.mlp is not None:
            x, normed = chain(x, self.mlp(normed), self.mlp_scale, m, next_norm)
        return x if next_norm is None else (x, normed)


class HyperConnectionLayer(TransformerSelfAttentionLayer):
    """Pre-norm decoder layer on several 32-bit residual streams (:class:`~torchtune_b200.modules.HyperConnection`) with layer scales; the
    feed-forward block is left out with ``mlp=None``.

    The end of one sublayer and the norm in front of the next run as one pass over the streams.  A decoder that chains layers passes
    ``(streams, normed input)`` and the :class:`~torchtune_b200.modules.hyper_connections.StreamEntry` of what follows this layer, and
    receives the same kind of pair for it.  A plain ``[b, s, dim]`` input stands for streams that are all equal."""

    def __init__(self, attn: nn.Module, mlp: Optional[nn.Module], *, streams: int, sa_norm: StreamLayerNorm, sa_scale: LayerScale, mlp_norm: Optional[StreamLayerNorm] = None,
                 mlp_scale: Optional[LayerScale] = None) -> None:
        nn.Module.__init__(self)
        if (mlp is None) != (mlp_norm is None) or (mlp is None) != (mlp_scale is None):
            raise ValueError("the feed-forward block, its norm and its scale come together")
        self.attn, self.mlp = attn, mlp
        self.sa_norm, self.sa_scale, self.mlp_norm, self.mlp_scale = sa_norm, sa_scale, mlp_norm, mlp_scale
        self.sa_streams = HyperConnection(streams)
        self.mlp_streams = HyperConnection(streams) if mlp is not None else None
        self.mask_mod = None

    @property
    def entry(self) -> StreamEntry:
        return StreamEntry(self.sa_streams.read, self.sa_norm)

    def forward(self, x, *, mask: MaskLike = None, input_pos: Optional[torch.Tensor] = None, layer_state: Optional[dict] = None, following: Optional[StreamEntry] = None, **kwargs):
        x, normed = x if isinstance(x, tuple) else (x, None)
        if x.dim() == 3:
            x = x.float().unsqueeze(2)
        if normed is None:
            normed = HyperConnection.enter(x, self.entry)
        y = self.attn(normed, mask=mask, input_pos=input_pos, layer_state=layer_state)
        x, normed = self.sa_streams.step(x, y, self.sa_scale, following if self.mlp is None else StreamEntry(self.mlp_streams.read, self.mlp_norm))
        if self.mlp is not None:
            x, normed = self.mlp_streams.step(x, self.mlp(normed), self.mlp_scale, following)
        return x if following is None else (x, normed)


class TransformerCrossAttentionLayer(nn.Module):
    """Cross-attention block over encoder tokens.  Query rows whose encoder mask is
    empty contribute nothing (attention and MLP outputs are zeroed for them)."""

    def __init__(
        self,
        attn: MultiHeadAttention,
        mlp: nn.Module,
        *,
        ca_norm: Optional[nn.Module] = None,
        mlp_norm: Optional[nn.Module] = None,
        ca_scale: Optional[nn.Module] = None,
        mlp_scale: Optional[nn.Module] = None,
    ) -> None:
        super().__init__()
        if attn.pos_embeddings is not None:
            raise AssertionError("Doesn't support positional embeddings for cross attention, because q and k are different sequences.")
        self.attn = attn
        self.mlp = mlp
        self.ca_norm = ca_norm or nn.Identity()
        self.mlp_norm = mlp_norm or nn.Identity()
        self.ca_scale = ca_scale or nn.Identity()
        self.mlp_scale = mlp_scale or nn.Identity()

    def setup_caches(self, batch_size: int, dtype: torch.dtype, *, encoder_max_seq_len: int, decoder_max_seq_len: int) -> None:
        self.attn.setup_cache(batch_size, dtype, encoder_max_seq_len)

    def caches_are_setup(self) -> bool:
        return self.attn.kv_cache is not None

    def caches_are_enabled(self) -> bool:
        return self.attn.cache_enabled

    def reset_cache(self) -> None:
        self.attn.reset_cache()

    @staticmethod
    def _skip_mask(mask: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """``[b, s_q, 1]`` True where a query row may attend to nothing; such rows are
        un-masked inside attention (avoids NaN) and zeroed afterwards."""
        if mask is None:
            return None
        if mask.dtype == torch.bool:
            m = ~mask
        else:
            m = torch.isneginf(mask)
        return torch.all(m, dim=-1, keepdim=True)

    def forward(
        self,
        x: torch.Tensor,
        *,
        encoder_input: Optional[torch.Tensor] = None,
        encoder_mask: Optional[torch.Tensor] = None,
        **kwargs,
    ) -> torch.Tensor:
        empty_cache = not self.caches_are_enabled() or self.attn.kv_cache.size == 0
        if encoder_input is None and empty_cache:
            return x
        skip = self._skip_mask(encoder_mask)
        if encoder_mask is not None:
            encoder_mask = encoder_mask.masked_fill(skip, True)
        attn_out = self.attn(self.ca_norm(x), encoder_input, mask=encoder_mask)
        if skip is not None:
            attn_out = attn_out.masked_fill(skip, 0)
        h = self.ca_scale(attn_out) + x
        mlp_out = self.mlp(self.mlp_norm(h))
        if skip is not None:
            mlp_out = mlp_out.masked_fill(skip, 0)
        return h + self.mlp_scale(mlp_out)


def _collapsed(h) -> torch.Tensor:
    """The hidden state a layer leaves: the sum of its streams where it has several."""
    h = h[0] if isinstance(h, tuple) else h
    return h.sum(2) if h.dim() == 4 else h


def _get_clones(module: nn.Module, n: int) -> nn.ModuleList:
    return nn.ModuleList([copy.deepcopy(module) for _ in range(n)])


class TransformerDecoder(nn.Module):
    """``tok_embeddings → layers → norm → output``.

    * ``skip_output_layer=True`` returns the normalised hidden states so a fused
      linear+loss operator can apply ``output`` itself.
    * ``num_output_chunks > 0`` returns the logits as a list of sequence chunks.
    * Materialised logits are fp32.
    """

    def __init__(
        self,
        *,
        tok_embeddings: nn.Embedding,
        layers: Union[nn.Module, List[nn.Module], nn.ModuleList],
        max_seq_len: int,
        num_heads: int,
        head_dim: int,
        norm: nn.Module,
        output: Union[nn.Linear, Callable],
        num_layers: Optional[int] = None,
        output_hidden_states: Optional[List[int]] = None,
    ) -> None:
        super().__init__()
        if isinstance(layers, nn.ModuleList):
            pass
        elif isinstance(layers, list):
            layers = nn.ModuleList(layers)
        else:
            if not isinstance(layers, nn.Module):
                raise AssertionError("num_layers is defined, layers must be a module")
            if num_layers is None:
                raise AssertionError("num_layers must be defined if layers is not a list")
            layers = _get_clones(layers, num_layers)
        self.tok_embeddings = tok_embeddings
        self.layers = layers
        self.norm = norm
        self.output = output
        self.output_hidden_states = output_hidden_states or []
        self.max_seq_len = max_seq_len
        self.num_heads = num_heads
        self.head_dim = head_dim
        self.causal_mask = None
        self.num_output_chunks = 0
        self.skip_output_layer = False
        # cap·tanh(logits/cap) applied to the logits (Gemma-2); 0 = none.  A loss that takes the hidden states instead
        # (``skip_output_layer``) reads this attribute and applies the cap itself.
        self.logit_softcap = 0.0
        # Vocabulary logits leave the output projection in fp32 instead of being widened from its rounded result.
        self.wide_logits = False
        # Prompts of unequal length may be described to the layers by the first key of every row instead of a boolean mask.
        self.span_masks = False
        # Learned embeddings of the positions, added to the token embeddings (fp32 sum).
        self.pos_embeddings: Optional[nn.Embedding] = None
        # Layers ``start … stop - 1`` run ``times`` times in a row before the rest follows.
        self.loop: Optional[Tuple[int, int, int]] = None
        self.encoder_max_cache_seq_len = None
        self.decoder_max_cache_seq_len = None

    # -- order of the layers ---------------------------------------------------
    def set_loop(self, start: int, stop: int, times: int) -> None:
        """Runs the layers ``start … stop - 1`` ``times`` times in a row, each time with a cache of its own."""
        if not 0 <= start < stop <= len(self.layers) or times < 1:
            raise ValueError(f"layers {start} … {stop} cannot run {times} times in a decoder of {len(self.layers)} layers")
        if self.caches_are_setup():
            raise RuntimeError("the order of the layers is fixed once caches exist")
        for layer in self.layers[start:stop]:
            if times > 1 and not isinstance(layer.attn, CachedMixer):
                raise ValueError(f"{type(layer.attn).__name__} keeps one cache and cannot run several times")
            layer.attn.num_passes = times
        self.loop = (start, stop, times)

    def run_order(self) -> List[Tuple[int, int]]:
        """``(layer, pass)`` in the order of execution."""
        start, stop, times = self.loop or (0, 0, 0)
        order = [(i, 0) for i in range(start)]
        order += [(i, n) for n in range(times) for i in range(start, stop)]
        return order + [(i, 0) for i in range(stop, len(self.layers))]

    # -- output chunking (deprecated path kept for API parity) -------------
    def set_num_output_chunks(self, num_output_chunks: int) -> None:
        self.num_output_chunks = num_output_chunks

    # -- KV caches -----------------------------------------------------------
    def setup_caches(
        self,
        batch_size: int,
        dtype: torch.dtype,
        *,
        encoder_max_seq_len: Optional[int] = None,
        decoder_max_seq_len: Optional[int] = None,
    ) -> None:
        kinds = [getattr(m, "inner_cls", type(m)) for m in self.modules()]  # sees through checkpoint wrappers
        has_enc = any(issubclass(k, TransformerCrossAttentionLayer) for k in kinds)
        has_dec = any(issubclass(k, TransformerSelfAttentionLayer) for k in kinds)
        if has_enc:
            self.encoder_max_cache_seq_len = encoder_max_seq_len if encoder_max_seq_len is not None else self.max_seq_len
        if has_dec:
            self.decoder_max_cache_seq_len = decoder_max_seq_len if decoder_max_seq_len is not None else self.max_seq_len
        for layer in self.layers:
            layer.setup_caches(
                batch_size,
                dtype,
                encoder_max_seq_len=self.encoder_max_cache_seq_len,
                decoder_max_seq_len=self.decoder_max_cache_seq_len,
            )

    def caches_are_setup(self) -> bool:
        return self.layers[0].caches_are_setup()

    def caches_are_enabled(self) -> bool:
        return self.layers[0].caches_are_enabled()

    def reset_caches(self) -> None:
        if not self.caches_are_enabled():
            raise RuntimeError("Key value caches are not setup. Call model.setup_caches first.")
        for layer in self.layers:
            layer.reset_cache()

    # -- forward ---------------------------------------------------------------
    def _cap(self, logits: torch.Tensor) -> torch.Tensor:
        cap = float(self.logit_softcap)
        return logits if cap <= 0.0 else ops.softcap(logits, cap)

    def chunked_output(self, last_hidden_state: torch.Tensor) -> List[torch.Tensor]:
        return [self._cap(self.output(chunk)) for chunk in last_hidden_state.tensor_split(self.num_output_chunks, dim=1)]

    def _validate_inputs(self, seq_len, mask=None, encoder_input=None, encoder_mask=None, input_pos=None) -> None:
        if seq_len > self.max_seq_len:
            raise ValueError(f"seq_len ({seq_len}) of input tensor should be smaller than max_seq_len ({self.max_seq_len})")
        if self.caches_are_enabled():
            if mask is None:
                raise ValueError("KV-caches for self-attention layers are setup for inference mode, causal masks must be provided! Use the `mask` arg to provide a causal mask.")
            if encoder_input is not None and encoder_mask is None:
                raise ValueError("KV-caches for cross-attention/fusion layers are setup for inference mode and you seem to be using encoder_input, causal masks must be provided! Use the `encoder_mask` arg to provide a causal mask.")
            if input_pos is None:
                raise ValueError("KV-caches are setup for inference mode, input positions must be provided!")

    def forward(
        self,
        tokens: Optional[torch.Tensor] = None,
        *,
        mask: MaskLike = None,
        encoder_input: Optional[torch.Tensor] = None,
        encoder_mask: Optional[torch.Tensor] = None,
        input_pos: Optional[torch.Tensor] = None,
        input_embeds: Optional[torch.Tensor] = None,
    ) -> Union[torch.Tensor, List[torch.Tensor]]:
        if (tokens is None) == (input_embeds is None):
            raise ValueError("Exactly one of `tokens` or `input_embeds` must be provided.")
        seq_len = tokens.shape[1] if input_embeds is None else input_embeds.shape[1]
        self._validate_inputs(seq_len, mask=mask, encoder_input=encoder_input, encoder_mask=encoder_mask, input_pos=input_pos)
        h = self._embed(tokens, input_embeds, input_pos)
        hidden = []
        layer_state: dict = {}
        order = self.run_order()
        for i, (idx, run) in enumerate(order):
            layer = self.layers[idx]
            if i in self.output_hidden_states:
                hidden.append(_collapsed(h))
            extra = {}
            kind = getattr(layer, "inner_cls", type(layer))
            after = self.layers[order[i + 1][0]] if i + 1 < len(order) else None
            if kind is ResidualStreamLayer:
                following = getattr(after, "sa_norm", None) if after is not None else self.norm
                extra = {"layer_state": layer_state, "next_norm": following if isinstance(following, StreamRMSNorm) else None}
            elif kind is HyperConnectionLayer:
                layer_state["pass"] = run
                last = StreamEntry(None, self.norm, keep=len(order) in self.output_hidden_states)
                extra = {"layer_state": layer_state, "following": last if after is None else after.entry}
            h = layer(h, mask=mask, encoder_input=encoder_input, encoder_mask=encoder_mask, input_pos=input_pos, **extra)
        if len(order) in self.output_hidden_states:
            hidden.append(_collapsed(h))
        h, normed = h if isinstance(h, tuple) else (h, None)
        h = self.norm(h) if normed is None else normed
        if self.skip_output_layer:
            output = h
        elif self.num_output_chunks > 0:
            output = self.chunked_output(h)
        else:
            output = self.unembed_normed(h)
        return output if not hidden else [*hidden, output]

    def _embed(self, tokens: Optional[torch.Tensor], input_embeds: Optional[torch.Tensor], input_pos: Optional[torch.Tensor]) -> torch.Tensor:
        if self.pos_embeddings is None:
            return ops.embed_tokens(self.tok_embeddings, tokens) if input_embeds is None else input_embeds
        b, s = (tokens if input_embeds is None else input_embeds).shape[:2]
        pos = torch.arange(s, device=self.pos_embeddings.weight.device) if input_pos is None else input_pos
        pos = pos.reshape(-1, s).expand(b, s)
        if input_embeds is not None:
            return input_embeds.float() + self.pos_embeddings(pos).float()
        return ops.embed_positions(tokens, pos, self.tok_embeddings.weight, self.pos_embeddings.weight)

    @property
    def position_limit(self) -> Optional[int]:
        """Longest sequence the position embeddings reach; ``None`` without a table."""
        return None if self.pos_embeddings is None else self.pos_embeddings.num_embeddings

    def unembed_normed(self, h: torch.Tensor) -> torch.Tensor:
        if self.wide_logits and type(self.output).__name__ == "Linear" and self.output.bias is None:
            return self._cap(ops.linear_wide(h, self.output.weight))
        return self._cap(self.output(h).float())

    def unembed(self, h: torch.Tensor) -> torch.Tensor:
        """Final norm + output projection of a hidden state (fp32 logits)."""
        h = self.norm(h)
        if self.num_output_chunks > 0:
            return self.chunked_output(h)
        return self.unembed_normed(h)
