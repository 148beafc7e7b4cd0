"""Input and output ends of the decoder.

``TokenEmbedding``: a table lookup (times a constant where the model has one, plus a row for the pair of this token and the one
before it and a learned row for its position where the model has those), or rows of caller-given embeddings
(edgerag/core/model.py:106-110: exactly one of ids and embeddings per token); the result is
written to the float32 residual stream.  ``LMHead``: bias-free projection to float32 logits over
the rows that were asked for (edgerag/core/model.py:150-152); where the plan names a tensor to
tie the head to, a checkpoint without a head of its own shares that tensor.
"""

from __future__ import annotations

import torch

from ..cache.manager import StateSpec
from ..ops import kernels
from .base import Part, PartSpec, WeightSpec, build_part, register_part


@register_part("embedding", "table")
class TokenEmbedding(Part):
    graph_safe = True

    def __init__(self, vocab: int, hidden: int, dtype: torch.dtype, device: torch.device, scale: float = 1.0,
                 tensor: str = "weight", norm: PartSpec | None = None, pairs: tuple[str, int, int, int] | None = None,
                 positions: tuple[str, int] | None = None) -> None:
        """``pairs = (tensor, buckets, mul_prev, mul_cur)``: the row ``(token before * mul_prev + token * mul_cur) mod buckets`` of the
        tensor ``[buckets + 1, hidden]`` is added, its last row for a sequence's first token (the token before a portion is a
        state record of its sequence); ``positions = (tensor, count)``: the row of the token's position is added, and no sequence
        may be longer than ``count``.  ``scale`` multiplies every row as it enters the float32 stream; ``tensor`` names the table; ``norm``: a norm
        that acts on the stream right after the lookup (its tensors' names are relative to this part's prefix)."""
        self.vocab, self.hidden = vocab, hidden
        self.dtype, self.device = dtype, device
        self.scale, self.tensor = float(scale), tensor
        self.weight: torch.Tensor | None = None
        self.pairs, self.positions = pairs, positions
        self.pair_table = self.pos_table = None
        self.needs_token_ids = pairs is not None
        self.max_positions = int(positions[1]) if positions is not None else None
        if pairs is not None and (int(pairs[1]) < 1 or int(pairs[2]) < 0 or int(pairs[3]) < 0):
            raise ValueError(f"embedding of token pairs: bad buckets or multipliers {pairs[1:]}")
        self._norm_prefix = norm.prefix if norm is not None else ""
        self.norm = build_part("norm", norm, dtype, device) if norm is not None else None
        if self.norm is not None and not hasattr(self.norm, "norm_stream"):
            raise ValueError(f"norm {norm.kind!r} cannot act on the stream in place")
        self.graph_safe = self.norm is None or bool(getattr(self.norm, "graph_safe", False))

    def weight_specs(self) -> list[WeightSpec]:
        specs = [WeightSpec(self.tensor, (self.vocab, self.hidden))]
        if self.pairs is not None:
            specs.append(WeightSpec(self.pairs[0], (int(self.pairs[1]) + 1, self.hidden)))
        if self.positions is not None:
            specs.append(WeightSpec(self.positions[0], (self.max_positions, self.hidden)))
        if self.norm is not None:
            specs += [WeightSpec(self._norm_prefix + s.name, s.shape, s.kind, s.fallback) for s in self.norm.weight_specs()]
        return specs

    def state_specs(self) -> list[StateSpec]:
        """The last token of every sequence, where the next one's row depends on it."""
        return [StateSpec("last_id", (1,), "int32", fillers=True)] if self.pairs is not None else []

    def load_weights(self, tensors: dict[str, torch.Tensor]) -> None:
        cast = lambda name: tensors[name].to(device=self.device, dtype=self.dtype).contiguous()  # noqa: E731
        self.weight = cast(self.tensor)
        self.pair_table = cast(self.pairs[0]) if self.pairs is not None else None
        self.pos_table = cast(self.positions[0]) if self.positions is not None else None
        if self.norm is not None:
            self.norm.load_weights({s.name: tensors[self._norm_prefix + s.name] for s in self.norm.weight_specs()})

    def forward(self, ctx, hidden: torch.Tensor) -> None:
        embed_row = ctx.embed_row if ctx.embeds is not None else None
        if self.pairs is None and self.positions is None:
            kernels.embed_rows(hidden, self.weight, ctx.token_ids, ctx.status, embeds=ctx.embeds, embed_row=embed_row, scale=self.scale)
        else:
            paired = {} if self.pairs is None else {
                "pairs": self.pair_table, "pair_hash": self.pairs[1:], "last_id": ctx.state("last_id", "embedding"),
                "seq_of_token": ctx.seq_of_token, "seq_starts": ctx.seq_starts, "state_slots": ctx.state_slots}
            kernels.embed_sum(hidden, self.weight, ctx.token_ids, ctx.status, ctx.positions, scale=self.scale, embeds=ctx.embeds,
                              embed_row=embed_row, pos_table=self.pos_table, **paired)
        if self.norm is not None:
            self.norm.norm_stream(hidden)


@register_part("head", "linear")
class LMHead(Part):
    graph_safe = True

    def __init__(self, vocab: int, hidden: int, dtype: torch.dtype, device: torch.device,
                 tied_to: str | None = None, softcap: float = 0.0, tensor: str = "weight", scale: float = 1.0) -> None:
        """``tied_to``: model-relative name of the tensor to share when the checkpoint has no head of
        its own (the plan names it; this part does not know what the model calls its embedding).
        ``softcap`` c > 0: logits <- c * tanh(logits / c), in float; ``scale``: a constant that multiplies the
        float logits (after the cap)."""
        self.scale = float(scale)
        self.vocab, self.hidden, self.tied_to = vocab, hidden, tied_to
        self.dtype, self.device = dtype, device
        self.softcap, self.tensor = float(softcap or 0.0), tensor
        self.weight: torch.Tensor | None = None

    def weight_specs(self) -> list[WeightSpec]:
        return [WeightSpec(self.tensor, (self.vocab, self.hidden), fallback=self.tied_to)]

    def load_weights(self, tensors: dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.tensor].to(device=self.device, dtype=self.dtype).contiguous()

    def forward(self, x: torch.Tensor, logits: torch.Tensor) -> None:
        kernels.linear(x, self.weight, logits)
        if self.softcap > 0.0:
            kernels.softcap(logits, self.softcap, self.dtype)
        if self.scale != 1.0:
            kernels.scale_rows(logits, self.scale, self.dtype)
