"""Sabolorn: a decoder whose layers are listed one by one in config.json, each with one norm that its mixer and its
feed-forward both read (``x += mixer(norm1(x)) + ff(norm1(x))``), an input of its own per token after the feed-forward, and an
average over the results of all layers so far before the next one.

config.json keys read: ``architecture``, ``width``, ``vocab``, ``embedding.scale``, ``norm.eps``, ``token_side.dim``,
``logit_softcap`` and ``layers``: per layer ``type`` (``mamba2`` | ``attention`` | ``latent_attention``), ``mixer`` (the
mixer's sizes) and ``mlp`` (or null).

* ``mamba2``: ``heads, vdim, state, groups, conv, norm_groups`` (``parts/ssd.py``).
* ``attention``: ``heads, kv_heads, dim, vdim, scale, conv``: grouped-query attention with biases on q, k and v, a causal
  convolution on each of their channels, no rotation, and a penalty that grows with the logarithm of the distance
  (``parts/attention.py``).
* ``latent_attention``: ``heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot.{base, dims, scaling.{factor, original,
  fast, slow}}``, optional ``kv_from: j`` (no down-projection of its own: it reads the cache rows of layer ``j``): attention
  through a normed latent, queries through another, a gate per entry of the concatenated heads
  (``parts/latent_attention.py``).
* ``mlp.kind = dense``: ``ff``; ``down(relu(up x)^2)``.
* ``mlp.kind = moe``: ``expert.ff``, ``router.{experts, top, groups.{count, keep}}``: gated silu experts, sigmoid scores,
  chosen by score + correction among the best groups (a group counts as much as its two best), the chosen scores divided by
  their sum (``parts/moe.py``).

The layers' norms and the final norm are layer norms without bias; the head is the embedding table without its scale, and
the logits pass ``c * tanh(x / c)``.  Tensor names: ``embed``, ``side.embed``, ``final.norm``, ``l<i>.norm1``,
``l<i>.mix.*``, ``l<i>.mlp.{up, down}`` or ``l<i>.mlp.{router, correction, e<j>.{gate, up, down}}``,
``l<i>.side.{gate, proj, norm}``, ``l<i>.dwa``.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from ..config.model_config import ConfigError
from ..parts.base import LayerCall, LayerSpec, ModelPlan, PartSpec, StreamCall

LAYER_TYPES = ("mamba2", "attention", "latent_attention")
MLP_KINDS = ("dense", "moe")


def _need(d: Any, key: str, where: str) -> Any:
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"{where}: no '{key}'")
    return d[key]


def _positive(d: Any, keys: tuple[str, ...], where: str) -> None:
    for key in keys:
        if int(_need(d, key, where)) <= 0:
            raise ConfigError(f"{where}: '{key}' must be positive")


def _check_mixer(kind: str, m: dict[str, Any], i: int, layers: list[dict[str, Any]], at: str) -> None:
    where = at + ".mixer"
    if kind == "mamba2":
        _positive(m, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), where)
        if m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"]:
            raise ConfigError(f"{at}: groups must divide heads, norm_groups the inner width")
    elif kind == "attention":
        _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
        _need(m, "scale", where)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{at}: kv_heads must divide heads")
        if int(m.get("conv") or 0) < 0:
            raise ConfigError(f"{at}: conv must not be negative")
    else:
        _positive(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"), where)
        _need(m, "scale", where)
        rot = _need(m, "rot", where)
        _need(rot, "base", where + ".rot")
        dims = int(_need(rot, "dims", where + ".rot"))
        if dims % 2 or dims > m["rot_dim"] or m["rot_dim"] % 2 or m["kv_rank"] % 2:
            raise ConfigError(f"{at}: kv_rank, rot_dim and rot.dims must be even, rot.dims at most rot_dim")
        scaling = rot.get("scaling")
        if scaling is not None:
            for key in ("factor", "original", "fast", "slow"):
                if not float(_need(scaling, key, where + ".rot.scaling")) > 0:
                    raise ConfigError(f"{at}: rot.scaling.{key} must be positive")
        src = m.get("kv_from")
        if src is not None:
            if not (isinstance(src, int) and 0 <= src < i) or layers[src].get("type") != "latent_attention" \
                    or layers[src]["mixer"].get("kv_from") is not None:
                raise ConfigError(f"{at}: kv_from must name an earlier latent attention layer with a down-projection of its own")
            theirs = layers[src]["mixer"]
            if any(theirs.get(k) != m.get(k) for k in ("kv_rank", "rot_dim", "rot")):
                raise ConfigError(f"{at}: kv_from layer {src} has another latent size or rotation")


def _check_mlp(mlp: dict[str, Any], at: str) -> None:
    if mlp.get("kind") not in MLP_KINDS:
        raise ConfigError(f"{at}: mlp.kind {mlp.get('kind')!r} is not supported; known: {MLP_KINDS}")
    if mlp["kind"] == "dense":
        _positive(mlp, ("ff",), at + ".mlp")
        return
    _positive(_need(mlp, "expert", at + ".mlp"), ("ff",), at + ".mlp.expert")
    router = _need(mlp, "router", at + ".mlp")
    _positive(router, ("experts", "top"), at + ".mlp.router")
    if router["top"] > router["experts"]:
        raise ConfigError(f"{at}: router.top must lie in 1..experts")
    groups = router.get("groups")
    if groups is not None:
        _positive(groups, ("count", "keep"), at + ".mlp.router.groups")
        count, keep = groups["count"], groups["keep"]
        if router["experts"] % count or keep > count or router["top"] > keep * (router["experts"] // count):
            raise ConfigError(f"{at}: router.groups must split the experts evenly and leave at least 'top' to choose from")


@dataclass
class SabolornConfig:
    hidden_size: int
    vocab_size: int
    embedding_scale: float
    norm_eps: float
    logit_softcap: float
    side_dim: int
    layers: list[dict[str, Any]] = field(default_factory=list)
    architectures: list[str] = field(default_factory=lambda: ["Sabolorn"])

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str = "config") -> "SabolornConfig":
        layers = _need(raw, "layers", where)
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        out = []
        for i, layer in enumerate(layers):
            at = f"{where}: layers[{i}]"
            kind = _need(layer, "type", at)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"{at}: unknown layer type {kind!r}; known: {LAYER_TYPES}")
            m = dict(_need(layer, "mixer", at))
            _check_mixer(kind, m, i, layers, at)
            mlp = layer.get("mlp")
            if mlp is not None:
                _check_mlp(mlp, at)
            out.append({"type": kind, "mixer": m, "mlp": dict(mlp) if mlp is not None else None})
        embedding = raw.get("embedding") or {}
        side = raw.get("token_side")
        if side is not None:
            _positive(side, ("dim",), where + ": token_side")
        scale = embedding.get("scale")
        return cls(hidden_size=int(_need(raw, "width", where)), vocab_size=int(_need(raw, "vocab", where)),
                   embedding_scale=1.0 if scale is None else float(scale),
                   norm_eps=float(_need(_need(raw, "norm", where), "eps", where + ": norm")),
                   logit_softcap=float(raw.get("logit_softcap") or 0.0), side_dim=int(side["dim"]) if side else 0, layers=out)


def sabolorn_plan(cfg: SabolornConfig) -> ModelPlan:
    h, eps = cfg.hidden_size, cfg.norm_eps
    norm = lambda tensor, prefix="": PartSpec("layernorm", {"size": h, "eps": eps, "tensor": tensor, "bias": False}, prefix)   # noqa: E731
    stream_ops, after = [], []
    if cfg.side_dim:
        after.append(len(stream_ops))
        stream_ops.append(PartSpec("token_side", {"hidden": h, "vocab": cfg.vocab_size, "dim": cfg.side_dim,
                                                  "n_layers": cfg.n_layers, "eps": eps}))
    after.append(len(stream_ops))
    stream_ops.append(PartSpec("depth_average", {"hidden": h, "n_layers": cfg.n_layers}))
    layers, schedule = [], []
    cache_layer_of: dict[int, int] = {}
    for i, layer in enumerate(cfg.layers):
        m = layer["mixer"]
        if layer["type"] == "mamba2":
            mixer = PartSpec("ssd", {"hidden": h, "n_heads": m["heads"], "head_dim": m["vdim"], "state": m["state"],
                                     "groups": m["groups"], "conv": m["conv"], "norm_groups": m["norm_groups"], "eps": eps}, "mix.")
        elif layer["type"] == "attention":
            mixer = PartSpec("attention", {
                "hidden": h, "n_q_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"],
                "scale": m["scale"], "conv": int(m.get("conv") or 0), "qkv_bias": True, "penalty": ("r1", "r2"),
                "position": PartSpec("none"),
                "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b"}}, "mix.")
        else:
            mixer = PartSpec("latent_attention", {
                "hidden": h, "n_heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "v_dim": m["vdim"],
                "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": m["scale"], "rot_base": m["rot"]["base"],
                "rot_dims": m["rot"]["dims"], "rot_scaling": m["rot"].get("scaling"), "eps": eps,
                "own_kv": m.get("kv_from") is None, "gate_entries": True}, "mix.")
        mlp = layer["mlp"]
        if mlp is None:
            ffn = None
        elif mlp["kind"] == "dense":
            ffn = PartSpec("dense_act", {"hidden": h, "intermediate": mlp["ff"], "act": "relu_squared"}, "mlp.")
        else:
            router = mlp["router"]
            groups = router.get("groups")
            ffn = PartSpec("routed_experts", {
                "hidden": h, "intermediate": mlp["expert"]["ff"], "n_experts": router["experts"], "top": router["top"],
                "weights": "score_normed", "scale_input": False, "correction": "correction", "group_score": "top2_sum",
                "groups": (groups["count"], groups["keep"]) if groups else None}, "mlp.")
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("parallel"), norm1=norm("norm1"), mixer=mixer, norm2=None, ffn=ffn))
        src = m.get("kv_from") if layer["type"] == "latent_attention" else None
        if src is None:
            cache_layer_of[i] = len(cache_layer_of)
        schedule.append(LayerCall(i, cache_layer_of[i if src is None else src], writes_cache=src is None))
        schedule += [StreamCall(op, i) for op in after]
    return ModelPlan(
        hidden_size=h, vocab_size=cfg.vocab_size,
        embedding=PartSpec("table", {"vocab": cfg.vocab_size, "hidden": h, "scale": cfg.embedding_scale, "tensor": "embed"}),
        layers=layers, schedule=schedule, final_norm=norm("norm", "final."),
        head=PartSpec("linear", {"vocab": cfg.vocab_size, "hidden": h, "softcap": cfg.logit_softcap, "tensor": "head", "tied_to": "embed"}),
        stream_ops=stream_ops, name_prefixes=("",),
    )
