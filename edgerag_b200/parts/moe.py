"""A feed-forward of routed experts: every token is sent to the ``top`` experts its router scores highest, and
optionally through a shared expert that every token uses.

    z = W_router x (float32),   s = sigmoid(z),   chosen = the ``top`` largest s (the lower index wins a tie)
    y = sum over chosen e of expert_e(w_e x) + shared(x),      expert(r) = W_down (silu(W_gate r) * (W_up r))

``weights`` says what ``w_e`` is: ``"score"`` (the score itself) or ``"score_normed"`` (the chosen scores divided by their
sum + 1e-20).  With ``scale_input`` the weight multiplies the expert's input (rounded once to the element type),
otherwise its output: ``y = sum_e w_e expert_e(x)``, the weight applied in float to the down product's sums.  Experts
have no biases.  The experts' tensors are ``e<i>.{gate, up, down}`` below the part's prefix, the router ``router``, the
shared expert a feed-forward part of its own under ``shared.``.

Further options: ``scores = "softmax"`` (the scores are the softmax of the logits over all experts; the choice still
goes by the largest); ``groups = (count, keep)``: the experts form ``count`` equal groups of neighbours, a group's score
is its best expert's, and only experts of the ``keep`` best groups can be chosen; ``gated = False`` with ``act =
"relu_squared"``: experts without a gate branch, ``W_down relu(W_up r)^2`` (tensors ``e<i>.{up, down}``); ``correction`` (a tensor's name, sigmoid scores): the choice goes
by ``s + correction``, the weights by ``s``; ``group_score = "top2_sum"``: a group counts as much as the sum of its two best
experts; ``weight_scale``: a constant that multiplies every weight at last; ``shared_gate`` (a tensor's name, ``[1, hidden]``): the
shared expert's output is multiplied by ``sigmoid(w . x)``, one number per token.  That row is stored below the router's: its logit
is made with the experts' and the shared expert's activation kernel takes the sigmoid per row (a constant per row commutes with
the down product).

Nothing here goes through the host: the router's kernel leaves, on the device, every expert's list of (token, choice)
pairs, and the two product kernels walk row tiles of those lists, so the launches of a step depend on its number of
tokens only and the step can be replayed from a CUDA graph.  The update leaves as float32 partial sums, one per choice
plus one for the shared expert, which whoever adds the update sums in that order.
"""

from __future__ import annotations

import torch

from ..ops import kernels
from .base import FeedForward, PartSpec, WeightSpec, build_part, register_part


@register_part("ffn", "routed_experts")
class RoutedExperts(FeedForward):
    graph_safe = True

    def __init__(self, hidden: int, intermediate: int, n_experts: int, top: int, dtype: torch.dtype, device: torch.device,
                 shared: PartSpec | None = None, weights: str = "score", scale_input: bool = True,
                 names: tuple[str, str, str] = ("gate", "up", "down"), router: str = "router", expert: str = "e{}.",
                 scores: str = "sigmoid", groups: tuple[int, int] | None = None, gated: bool = True,
                 act: str = "silu", correction: str | None = None, group_score: str = "best", weight_scale: float = 1.0,
                 shared_gate: str | None = None) -> None:
        if not 0 < top <= n_experts:
            raise ValueError(f"routed_experts: top {top} of {n_experts} experts")
        if weights not in ("score", "score_normed"):
            raise ValueError(f"routed_experts: weights {weights!r}; known: score, score_normed")
        if group_score not in kernels.MOE_GROUP_SCORES or (scores != "sigmoid" and (correction or group_score != "best")):
            raise ValueError("routed_experts: a correction and groups that count their two best go with sigmoid scores")
        self.normalise, self.correction_name, self.group_score = weights == "score_normed", correction, group_score
        self.correction: torch.Tensor | None = None
        self.weight_scale, self.shared_gate = float(weight_scale), shared_gate
        if shared_gate is not None and shared is None:
            raise ValueError("routed_experts: a gate of the shared expert without a shared expert")
        if scores not in kernels.MOE_SCORES:
            raise ValueError(f"routed_experts: scores {scores!r}; known: {sorted(kernels.MOE_SCORES)}")
        if (gated and act != "silu") or (not gated and act != "relu_squared"):
            raise ValueError("routed_experts: gated experts use silu, experts without a gate branch relu_squared")
        if groups is not None:
            count, keep = (int(v) for v in groups)
            if count < 1 or n_experts % count or not 1 <= keep <= count or top > keep * (n_experts // count):
                raise ValueError(f"routed_experts: {count} groups of which {keep} are kept cannot give {top} of {n_experts} experts")
            groups = (count, keep)
        self.scores, self.groups, self.gated, self.scale_input = scores, groups, bool(gated), bool(scale_input)
        self.hidden, self.intermediate, self.n_experts, self.top = hidden, intermediate, n_experts, top
        self.dtype, self.device = dtype, device
        self.names, self.router_name, self.expert_fmt = tuple(names), router, expert
        self._shared_prefix = shared.prefix if shared is not None else ""
        self.shared = build_part("ffn", shared, dtype, device) if shared is not None else None
        self.graph_safe = self.shared is None or bool(getattr(self.shared, "graph_safe", False))
        self.w_router = self.w_gate_up = self.w_down = None

    def weight_specs(self) -> list[WeightSpec]:
        gate, up, down = self.names
        specs = [WeightSpec(self.router_name, (self.n_experts, self.hidden), "vector32")]
        if self.correction_name is not None:
            specs.append(WeightSpec(self.correction_name, (self.n_experts,), "vector32"))
        for e in range(self.n_experts):
            pre = self.expert_fmt.format(e)
            if self.gated:
                specs.append(WeightSpec(pre + gate, (self.intermediate, self.hidden)))
            specs += [WeightSpec(pre + up, (self.intermediate, self.hidden)), WeightSpec(pre + down, (self.hidden, self.intermediate))]
        if self.shared_gate is not None:
            specs.append(WeightSpec(self.shared_gate, (1, self.hidden), "vector32"))
        if self.shared is not None:
            specs += [WeightSpec(self._shared_prefix + s.name, s.shape, s.kind, s.fallback) for s in self.shared.weight_specs()]
        return specs

    def load_weights(self, tensors: dict[str, torch.Tensor]) -> None:
        gate, up, down = self.names
        cast = lambda t: t.to(device=self.device, dtype=self.dtype)  # noqa: E731
        self.w_router = tensors[self.router_name].to(device=self.device, dtype=torch.float32).contiguous()
        if self.shared_gate is not None:
            side = tensors[self.shared_gate].to(device=self.device, dtype=torch.float32)
            self.w_router = torch.cat([self.w_router, side], 0).contiguous()
        if self.correction_name is not None:
            self.correction = tensors[self.correction_name].to(device=self.device, dtype=torch.float32).contiguous()
        pres = [self.expert_fmt.format(e) for e in range(self.n_experts)]
        if self.gated:
            self.w_gate_up = torch.stack([torch.cat([cast(tensors[p + gate]), cast(tensors[p + up])], 0) for p in pres]).contiguous()
        else:       # (the one matrix of an expert without a gate branch, under the same attribute)
            self.w_gate_up = torch.stack([cast(tensors[p + up]) for p in pres]).contiguous()
        self.w_down = torch.stack([cast(tensors[p + down]) for p in pres]).contiguous()
        if self.shared is not None:
            self.shared.load_weights({s.name: tensors[self._shared_prefix + s.name] for s in self.shared.weight_specs()})

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        n, top = x.shape[0], self.top
        lists = ctx.buf("moe.lists", (kernels.moe_lists_ints(n, self.n_experts, top),), torch.int32)
        score = ctx.buf("moe.score", (n * top,), torch.float32)
        act = ctx.buf("moe.act", (n * top, self.intermediate), self.dtype)
        parts = ctx.buf("ffn.out_parts", (top + (self.shared is not None), n, self.hidden), torch.float32)
        route = dict(scores=self.scores, groups=self.groups, correction=self.correction, group_score=self.group_score,
                     normalise=self.normalise, weight=self.weight_scale)
        row_scale = None
        if self.shared_gate is not None:
            row_scale = route["side_gate"] = ctx.buf("moe.side_gate", (n,), torch.float32)
        if kernels.moe_route_few(n, self.n_experts, top, self.dtype):
            route["logits"] = ctx.buf("moe.logits", (n, self.w_router.shape[0]), torch.float32)
        in_score, out_score = (score, None) if self.scale_input else (None, score)
        if kernels.moe_tc_supported(self.dtype, self.hidden, self.intermediate):
            # tensor cores: row tiles sized by the step's tokens, the (scaled) rows gathered once in list order
            tile_rows = kernels.moe_tc_tile_rows(n, self.n_experts, top)
            kernels.moe_route(x, self.w_router, top, lists, score, tile_rows, **route)
            xs = ctx.buf("moe.rows", (n * top, self.hidden), self.dtype)
            kernels.moe_tc_gather(x, lists, in_score, self.n_experts, top, xs)
            if self.gated:
                kernels.moe_tc_gate_up(xs, self.w_gate_up, lists, top, tile_rows, act)
            else:
                kernels.moe_tc_up_act(xs, self.w_gate_up, lists, top, tile_rows, act)
            kernels.moe_tc_down(act, self.w_down, lists, top, tile_rows, parts, out_score=out_score)
        else:
            kernels.moe_route(x, self.w_router, top, lists, score, **route)
            if self.gated:
                kernels.moe_gate_up(x, self.w_gate_up, lists, in_score, top, act)
            else:
                if in_score is not None:
                    raise ValueError("routed_experts: experts without a gate branch take their weight on the output")
                kernels.moe_up_act(x, self.w_gate_up, lists, top, act)
            kernels.moe_down(act, self.w_down, lists, top, parts, out_score=out_score)
        if self.shared is not None:
            if row_scale is None:
                self.shared.forward_into(x, ctx, parts[top])
            else:
                self.shared.forward_into(x, ctx, parts[top], row_scale=row_scale)
        return parts
