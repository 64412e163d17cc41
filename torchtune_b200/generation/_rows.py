"""Batches of rows that start together and go on one token at a time.

Prompts of unequal length are padded on the left, so all rows append at the same cache slot.  :class:`RowLayout` knows where each row
begins and gives the positions and the visible keys of any range of slots; :class:`BatchDecoder` runs a model on its KV caches with it,
returning hidden states, and gives up rows that are finished."""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ..modules import TransformerDecoder
from ..modules.attention import MaskLike
from ..modules.common_utils import delete_kv_caches
from ..ops.mask import AttentionMask


def hidden_states(model: TransformerDecoder, x: torch.Tensor, *, input_pos: torch.Tensor, mask: MaskLike) -> torch.Tensor:
    """Normalised hidden states ``[b, s, d]`` in front of the output projection."""
    before = model.skip_output_layer
    model.skip_output_layer = True
    try:
        return model(x, input_pos=input_pos, mask=mask)
    finally:
        model.skip_output_layer = before


class RowLayout:
    """Cache slots of left-padded rows: ``real`` ``[b, s]`` is True on prompt tokens, every later slot is a real token of its row."""

    def __init__(self, real: torch.Tensor) -> None:
        n = real.shape[1]
        padded = not bool(real.all())
        slots = torch.arange(n, device=real.device)
        if padded and not bool((real == (slots[None, :] >= n - real.sum(1, keepdim=True))).all()):
            # a pad id inside a prompt: the row starts at its first real token and what follows counts as tokens
            first = torch.where(real.any(1), real.to(torch.int8).argmax(1), n)
        else:
            first = n - real.sum(1)
        self.start = first.to(torch.int32)
        self.padded = padded
        self.batch = real.shape[0]

    def positions(self, first: int, count: int) -> torch.Tensor:
        """``[b, count]`` int32 positions of the slots ``first …``, counted from each row's own first token (0 on padding)."""
        slots = torch.arange(first, first + count, dtype=torch.int32, device=self.start.device)
        return (slots[None, :] - self.start[:, None]).clamp_min_(0)

    def mask(self, first: int, count: int) -> AttentionMask:
        return AttentionMask(causal=True, key_start=self.start, query_start=first)

    def keep(self, rows: Sequence[int]) -> None:
        self.start = self.start[list(rows)].contiguous()
        self.batch = len(rows)


class DecodeGraph:
    """The one-token step of a batch as a CUDA graph: embedding to final norm with every launch recorded once, the cache slot held on the
    device and moved on by the graph itself.  Calling it with ``[b, 1]`` tokens replays the step on the model's caches; the result lives
    in a buffer that the next call overwrites."""

    def __init__(self, model: TransformerDecoder, layout: RowLayout) -> None:
        self.caches = [layer.attn.kv_cache for layer in model.layers if layer.attn.kv_cache is not None]
        used = self.caches[0].size
        dev = layout.start.device
        self.batch = layout.batch
        self.tokens = torch.zeros(self.batch, 1, dtype=torch.int64, device=dev)
        self.start = layout.start
        self.slot = torch.tensor([used], dtype=torch.int32, device=dev)
        mask = layout.mask(used, 1)

        def body() -> torch.Tensor:
            return hidden_states(model, self.tokens, input_pos=(self.slot - self.start).clamp_min_(0)[:, None], mask=mask)

        saved = [c.snapshot() for c in self.caches]  # the first launches are a step of their own, undone before the recording

        def undo() -> None:
            for c, before in zip(self.caches, saved):
                c.restore(before)

        for c in self.caches:
            c.slot = self.slot
        try:
            side = torch.cuda.Stream(device=dev)
            side.wait_stream(torch.cuda.current_stream(dev))
            with torch.cuda.stream(side):  # first launches and their one-time set-up stay out of the recording
                body()
            torch.cuda.current_stream(dev).wait_stream(side)
            undo()
            self.graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(self.graph):
                self.hidden = body()
                self.slot.add_(1)
        finally:
            for c in self.caches:
                c.slot = None
            undo()
        self._next = used

    def __call__(self, tokens: torch.Tensor) -> torch.Tensor:
        at = self.caches[0].reserve(self.batch, 1)
        if at != self._next:
            self.slot.fill_(at)
        self.tokens.copy_(tokens.view(self.batch, 1))
        self.graph.replay()
        for c in self.caches:
            c.advance(1)
        self._next = at + 1
        return self.hidden


class BatchDecoder:
    """One batch at a time on a model's KV caches: :meth:`begin`, then :meth:`advance` until every row has been ended.

    ``max_tokens`` is the most tokens that live rows hold together; the caches of a batch are sized from it (padding included)."""

    def __init__(self, model: TransformerDecoder, device: torch.device, dtype: torch.dtype, max_tokens: int, graphs: bool = True) -> None:
        if not getattr(model, "span_masks", False):
            raise ValueError("this decoder needs a model that takes its key ranges from row starts")
        self.model, self.device, self.dtype, self.max_tokens = model, device, dtype, int(max_tokens)
        self.layout: Optional[RowLayout] = None
        self.used = 0
        self.lengths: List[int] = []  # tokens of each live row
        self._capacity = (0, 0)
        self._graphs = graphs and device.type == "cuda"
        self._graph: Optional[DecodeGraph] = None

    @property
    def rows(self) -> int:
        return 0 if self.layout is None else self.layout.batch

    def _reserve(self, batch: int, slots: int) -> None:
        if batch > self._capacity[0] or slots > self._capacity[1]:
            if self.model.caches_are_setup():
                delete_kv_caches(self.model)
            with self.device:
                self.model.setup_caches(batch, self.dtype, decoder_max_seq_len=slots)
            self._capacity = (batch, slots)
        else:
            self.model.reset_caches()

    def begin(self, prompts: List[List[int]]) -> torch.Tensor:
        """Hidden states ``[b, longest, d]`` of new rows; row ``i`` occupies the last ``len(prompts[i])`` places."""
        if self.rows:
            raise RuntimeError("the batch before has unfinished rows")
        lengths = [len(p) for p in prompts]
        longest, shortest = max(lengths), min(lengths)
        if shortest < 1:
            raise ValueError("a row starts with at least one token")
        self._check_positions(longest)
        # a row may go on alone until it holds every token of the budget: that many slots behind the padding of the shortest one
        self._reserve(len(prompts), longest + max(self.max_tokens - shortest, 0))
        tokens = torch.tensor([[0] * (longest - n) + p for p, n in zip(prompts, lengths)], device=self.device)
        real = torch.arange(longest)[None, :] >= torch.tensor([longest - n for n in lengths])[:, None]
        self.layout, self.used, self.lengths = RowLayout(real.to(self.device)), 0, lengths
        return self._run(tokens)

    def _check_positions(self, length: int) -> None:
        limit = getattr(self.model, "position_limit", None)
        if limit is not None and length > limit:
            raise ValueError(f"a row of {length} tokens is longer than the model's {limit} positions")

    def advance(self, tokens: List[int]) -> torch.Tensor:
        """Hidden states ``[b, 1, d]`` of one more token per live row."""
        if len(tokens) != self.rows or not tokens:
            raise ValueError(f"{len(tokens)} tokens for {self.rows} rows")
        self._check_positions(max(self.lengths) + 1)
        self.lengths = [n + 1 for n in self.lengths]
        step = torch.tensor(tokens, device=self.device)[:, None]
        if not self._graphs:
            return self._run(step)
        if self._graph is None:
            self._graph = DecodeGraph(self.model, self.layout)
        self.used += 1
        return self._graph(step).clone()

    def _run(self, tokens: torch.Tensor) -> torch.Tensor:
        first, count = self.used, tokens.shape[1]
        h = hidden_states(self.model, tokens, input_pos=self.layout.positions(first, count), mask=self.layout.mask(first, count))
        self.used += count
        return h

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of hidden states ``[..., d]``."""
        return self.model.unembed_normed(hidden)

    def end(self, rows: Sequence[int]) -> None:
        """Gives up rows (indices into the live ones); the others close ranks, so later :meth:`advance` calls name only them."""
        gone = set(rows)
        kept = [i for i in range(self.rows) if i not in gone]
        if not kept:
            self.layout, self.used, self.lengths, self._graph = None, 0, [], None
            self.model.reset_caches()
            return
        if len(kept) == self.rows:
            return
        self._graph = None
        self.lengths = [self.lengths[i] for i in kept]
        for layer in self.model.layers:
            cache = layer.attn.kv_cache
            if cache is not None:
                cache.keep_rows(kept)
        self.layout.keep(kept)
