"""Operations on the residual stream after a layer: an input of its own per token and layer, and an average over depth.

``TokenSide``, the per-layer token input: every layer has a piece ``e`` (``dim`` entries) of one table's row of the token,

    x <- x + RMSnorm(W_proj (gelu_tanh(W_gate x) * e)) * w            (the norm's eps inside the root)

``DepthAverage``: with ``X_0`` the embedding's output and ``X_(i+1)`` the result of layer ``i``, what goes on after layer
``i`` is ``x <- sum over j <= i + 1 of a_ij X_j``, with the layer's weights ``a_i``.  The results of a step's tokens are kept
in float32 for the step; tokens do not mix, so nothing of them outlives it.

Both are stream operations of the run order, called after their layer with its number as the index.  The sum that the layer
leaves pending and the rounded copy for ``W_gate`` are one kernel; the norm of the side input, its add, the new entry of the
history, the average and the norm that opens the next layer are one kernel (``DepthUpdate``).
"""

from __future__ import annotations

import torch

from ..ops import kernels
from .base import DepthUpdate, NormedUpdate, PartSpec, StreamCall, StreamOp, SumUpdate, WeightSpec, build_part, register_part, settle_update
from .rmsnorm import RMSNorm


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


@register_part("stream", "token_side")
class TokenSide(StreamOp):
    graph_safe = True
    needs_token_ids = True

    def __init__(self, hidden: int, vocab: int, dim: int, n_layers: int, eps: float, dtype: torch.dtype, device: torch.device,
                 table: str = "side.embed", layer: str = "l{}.side.", names: tuple[str, str, str] = ("gate", "proj", "norm")) -> None:
        """``table``: the tensor ``[vocab, n_layers * dim]``; ``layer``: the prefix of layer ``i``'s tensors, ``names``
        those of its gate ``[dim, hidden]``, projection ``[hidden, dim]`` and norm weight ``[hidden]`` below it."""
        self.hidden, self.vocab, self.dim, self.n_layers = hidden, vocab, int(dim), int(n_layers)
        self.padded = _pad8(self.dim)              # rows of the small products start 16-byte aligned
        self.dtype, self.device = dtype, device
        self.table_name, self.layer_fmt, self.names = table, layer, tuple(names)
        self.norms = [build_part("norm", PartSpec("rmsnorm", {"size": hidden, "eps": eps, "exact": True, "tensor": names[2]}), dtype, device)
                      for _ in range(self.n_layers)]
        self.table: torch.Tensor | None = None
        self.gate: list[torch.Tensor] = []
        self.proj: list[torch.Tensor] = []

    def weight_specs(self) -> list[WeightSpec]:
        gate, proj, norm = self.names
        specs = [WeightSpec(self.table_name, (self.vocab, self.n_layers * self.dim))]
        for i in range(self.n_layers):
            pre = self.layer_fmt.format(i)
            specs += [WeightSpec(pre + gate, (self.dim, self.hidden)), WeightSpec(pre + proj, (self.hidden, self.dim)),
                      WeightSpec(pre + norm, (self.hidden,), "vector32")]
        return specs

    def load_weights(self, tensors: dict[str, torch.Tensor]) -> None:
        gate, proj, norm = self.names
        cast = lambda t: t.to(device=self.device, dtype=self.dtype)          # noqa: E731
        extra = self.padded - self.dim
        self.table = cast(tensors[self.table_name]).contiguous()
        self.gate, self.proj = [], []
        for i in range(self.n_layers):
            pre = self.layer_fmt.format(i)
            self.gate.append(torch.nn.functional.pad(cast(tensors[pre + gate]), (0, 0, 0, extra)).contiguous())
            self.proj.append(torch.nn.functional.pad(cast(tensors[pre + proj]), (0, extra)).contiguous())
            self.norms[i].load_weights({norm: tensors[pre + norm]})

    def forward(self, hidden, delta, ctx, call: StreamCall):
        i, n = call.index, hidden.shape[0]
        x = ctx.buf("side.x", (n, self.hidden), self.dtype)
        if isinstance(delta, SumUpdate):
            kernels.sum_updates(hidden, delta.a, delta.b, self.dtype, out=x)
        elif isinstance(delta, torch.Tensor):
            kernels.sum_updates(hidden, delta, None, self.dtype, out=x)
        else:
            settle_update(hidden, delta, self.dtype)
            kernels.cast_rows(hidden, x)
        g = ctx.buf("side.g", (n, self.padded), self.dtype)
        kernels.linear(x, self.gate[i], g)
        act = ctx.buf("side.act", (n, self.padded), self.dtype)
        kernels.side_gate(g, self.table, ctx.token_ids, i * self.dim, self.dim, act)
        y = ctx.buf("side.y", (n, self.hidden), self.dtype)
        kernels.linear(act, self.proj[i], y)
        return NormedUpdate(y, self.norms[i])


@register_part("stream", "depth_average")
class DepthAverage(StreamOp):
    graph_safe = True

    def __init__(self, hidden: int, n_layers: int, dtype: torch.dtype, device: torch.device, tensor: str = "l{}.dwa") -> None:
        """``tensor``: the name of layer ``i``'s weights ``[i + 2]``, the embedding's output first."""
        self.hidden, self.n_layers = hidden, int(n_layers)
        self.dtype, self.device, self.fmt = dtype, device, tensor
        self.mix: list[torch.Tensor] = []

    def weight_specs(self) -> list[WeightSpec]:
        return [WeightSpec(self.fmt.format(i), (i + 2,), "vector32") for i in range(self.n_layers)]

    def load_weights(self, tensors: dict[str, torch.Tensor]) -> None:
        self.mix = [tensors[self.fmt.format(i)].to(device=self.device, dtype=torch.float32).contiguous() for i in range(self.n_layers)]

    def _history(self, ctx, n: int) -> torch.Tensor:
        return ctx.buf("depth.history", (self.n_layers + 1, n, self.hidden), torch.float32)

    def begin(self, ctx, hidden: torch.Tensor) -> None:
        self._history(ctx, hidden.shape[0])[0].copy_(hidden)

    def forward(self, hidden, delta, ctx, call: StreamCall):
        history = self._history(ctx, hidden.shape[0])
        post = None
        if isinstance(delta, NormedUpdate) and isinstance(delta.norm, RMSNorm) and delta.bias is None:
            delta, post = delta.tensor, (delta.norm.weight, delta.norm.eps)
        elif delta is not None and not isinstance(delta, torch.Tensor):
            settle_update(hidden, delta, self.dtype)
            delta = None
        return DepthUpdate(history, call.index, self.mix[call.index], delta, post)
