"""Kikarax: a pre-norm decoder whose layers are listed one by one in config.json, all of them chunked attention with capped
scores, gated outputs and values blended with the first layer's, over an embedding of tokens, token pairs and positions.

config.json keys read: ``architecture``, ``width``, ``vocab``, ``embedding.{scale, bigram.{buckets, mul_prev, mul_cur}}``,
``max_positions``, ``norm.eps``, ``logit_scale`` and ``layers``: per layer ``type`` (``attention``), ``mixer`` (the mixer's sizes)
and ``mlp`` (or null).

* the input: ``scale * embed[token] + bigram[(token before * mul_prev + token * mul_cur) mod buckets] + pos[position]``; a sequence's
  first token has the bigram table's last row (``parts/embedding.py``).
* ``attention``: ``heads, kv_heads, dim, vdim, scale``, optional ``softcap``, ``mask.size`` and ``v_mix``: grouped-query attention
  without biases or rotation, a unit-RMS norm over a token's whole query and whole key projection, scores ``c tanh(s / c)``, a mask of
  chunks, and a gate per entry of the concatenated heads.  Layers with ``v_mix`` blend their values with those of the first such
  layer (``parts/attention.py``).
* ``mlp.kind = dense``: ``ff, limit``: ``down(g sigmoid(1.702 g) (u + 1))``, ``g`` and ``u`` bounded by ``limit`` (``parts/glu.py``).
* ``mlp.kind = moe``: ``expert.ff``, ``router.{experts, top, scale}``, optional ``shared.ff``: gated silu experts chosen and weighted by
  their softmax scores times ``scale``, beside a shared expert that one sigmoid per token multiplies (``parts/moe.py``).

The head is the embedding table without its scale, the logits are multiplied by ``logit_scale``.  Tensor names: ``embed``,
``bigram``, ``pos``, ``final.norm``, ``l<i>.{norm1, norm2}``, ``l<i>.mix.{q, k, v, g, o, q.norm, k.norm, vmix}``,
``l<i>.mlp.{gate, up, down}`` or ``l<i>.mlp.{router, e<j>.{gate, up, down}, shared.{gate, up, down, sg}}``.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from ..config.model_config import ConfigError
from ..parts.base import LayerCall, LayerSpec, ModelPlan, PartSpec

MLP_KINDS = ("dense", "moe")
GATE_ALPHA, GATE_SHIFT = 1.702, 1.0      # of the dense feed-forward's gated unit


def _need(d: Any, key: str, where: str) -> Any:
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"{where}: no '{key}'")
    return d[key]


def _positive(d: Any, keys: tuple[str, ...], where: str) -> None:
    for key in keys:
        if not float(_need(d, key, where)) > 0:
            raise ConfigError(f"{where}: '{key}' must be positive")


def _or(value: Any, default: float) -> float:
    return default if value is None else float(value)


def _check_mixer(m: dict[str, Any], at: str) -> None:
    where = at + ".mixer"
    _positive(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{at}: kv_heads must divide heads")
    if m.get("softcap") is not None:
        _positive(m, ("softcap",), where)
    if m.get("mask") is not None:
        _positive(m["mask"], ("size",), where + ".mask")


def _check_mlp(mlp: dict[str, Any], at: str) -> None:
    where = at + ".mlp"
    if mlp.get("kind") not in MLP_KINDS:
        raise ConfigError(f"{at}: mlp.kind {mlp.get('kind')!r} is not supported; known: {MLP_KINDS}")
    if mlp["kind"] == "dense":
        _positive(mlp, ("ff", "limit"), where)
        return
    _positive(_need(mlp, "expert", where), ("ff",), where + ".expert")
    router = _need(mlp, "router", where)
    _positive(router, ("experts", "top"), where + ".router")
    if router["top"] > router["experts"]:
        raise ConfigError(f"{at}: router.top must lie in 1..experts")
    if mlp.get("shared") is not None:
        _positive(mlp["shared"], ("ff",), where + ".shared")


@dataclass
class KikaraxConfig:
    hidden_size: int
    vocab_size: int
    embedding_scale: float
    norm_eps: float
    logit_scale: float
    #: (buckets, mul_prev, mul_cur) of the table of token pairs, or None
    bigram: tuple[int, int, int] | None = None
    max_position_embeddings: int | None = None
    layers: list[dict[str, Any]] = field(default_factory=list)
    architectures: list[str] = field(default_factory=lambda: ["Kikarax"])

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str = "config") -> "KikaraxConfig":
        layers = _need(raw, "layers", where)
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        out: list[dict[str, Any]] = []
        blended: dict[str, Any] | None = None        # the first mixer with v_mix
        for i, layer in enumerate(layers):
            at = f"{where}: layers[{i}]"
            kind = _need(layer, "type", at)
            if kind != "attention":
                raise ConfigError(f"{at}: unknown layer type {kind!r}; known: attention")
            m = dict(_need(layer, "mixer", at))
            _check_mixer(m, at)
            if m.get("v_mix"):
                blended = blended or m
                if any(blended[k] != m[k] for k in ("kv_heads", "vdim")):
                    raise ConfigError(f"{at}: v_mix blends values of equal kv_heads and vdim")
            mlp = layer.get("mlp")
            if mlp is not None:
                _check_mlp(mlp, at)
            out.append({"type": kind, "mixer": m, "mlp": dict(mlp) if mlp is not None else None})
        embedding = raw.get("embedding") or {}
        bigram = embedding.get("bigram")
        if bigram is not None:
            _positive(bigram, ("buckets",), where + ": embedding.bigram")
            if min(int(_need(bigram, k, where + ": embedding.bigram")) for k in ("mul_prev", "mul_cur")) < 0:
                raise ConfigError(f"{where}: embedding.bigram: multipliers must not be negative")
            bigram = tuple(int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur"))
        if raw.get("max_positions") is not None:
            _positive(raw, ("max_positions",), where)
        return cls(hidden_size=int(_need(raw, "width", where)), vocab_size=int(_need(raw, "vocab", where)),
                   embedding_scale=_or(embedding.get("scale"), 1.0),
                   norm_eps=float(_need(_need(raw, "norm", where), "eps", where + ": norm")),
                   logit_scale=_or(raw.get("logit_scale"), 1.0), bigram=bigram,
                   max_position_embeddings=int(raw["max_positions"]) if raw.get("max_positions") is not None else None, layers=out)


def _ffn(mlp: dict[str, Any] | None, h: int) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("glu_bounded", {"hidden": h, "intermediate": mlp["ff"], "limit": mlp["limit"], "alpha": GATE_ALPHA,
                                        "shift": GATE_SHIFT}, "mlp.")
    router, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", {
        "hidden": h, "intermediate": mlp["expert"]["ff"], "n_experts": router["experts"], "top": router["top"],
        "scores": "softmax", "weights": "score", "scale_input": False, "weight_scale": _or(router.get("scale"), 1.0),
        "shared": None if shared is None else PartSpec("glu_bounded", {"hidden": h, "intermediate": shared["ff"]}, "shared."),
        "shared_gate": None if shared is None else "shared.sg"}, "mlp.")


def kikarax_plan(cfg: KikaraxConfig) -> ModelPlan:
    h, eps = cfg.hidden_size, cfg.norm_eps
    norm = lambda tensor, prefix="": PartSpec("rmsnorm", {"size": h, "eps": eps, "exact": True, "tensor": tensor}, prefix)   # noqa: E731
    layers, mixed = [], False
    for i, layer in enumerate(cfg.layers):
        m = layer["mixer"]
        value_mix = None
        if m.get("v_mix"):
            value_mix, mixed = "blend" if mixed else "first", True
        mixer = PartSpec("attention", {
            "hidden": h, "n_q_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"],
            "scale": m["scale"], "softcap": _or(m.get("softcap"), 0.0), "chunk": int((m.get("mask") or {}).get("size") or 0),
            "whole_norm_eps": eps, "gate": "g", "value_mix": value_mix, "position": PartSpec("none"),
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}}, "mix.")
        ffn = _ffn(layer["mlp"], h)
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("prenorm"), norm1=norm("norm1"), mixer=mixer,
                                norm2=None if ffn is None else norm("norm2"), ffn=ffn))
    return ModelPlan(
        hidden_size=h, vocab_size=cfg.vocab_size,
        embedding=PartSpec("table", {"vocab": cfg.vocab_size, "hidden": h, "scale": cfg.embedding_scale, "tensor": "embed",
                                     "pairs": ("bigram", *cfg.bigram) if cfg.bigram else None,
                                     "positions": ("pos", cfg.max_position_embeddings) if cfg.max_position_embeddings else None}),
        layers=layers, schedule=[LayerCall(i, i) for i in range(len(layers))], final_norm=norm("norm", "final."),
        head=PartSpec("linear", {"vocab": cfg.vocab_size, "hidden": h, "scale": cfg.logit_scale, "tensor": "head", "tied_to": "embed"}),
        name_prefixes=("",),
    )
