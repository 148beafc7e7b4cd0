"""A plain, slow implementation of the Kikarax decoder in float64, one function per mechanism.

It shares no code with the package: it works on whole sequences with ordinary torch arithmetic on the CPU
and exists to be compared against.  ``config`` is the dictionary of a config.json, ``tensors`` maps the
checkpoint's names to tensors.

The design, in this file's notation.  The stream starts as

    x_p = scale * E[t_p] + B[row(t_{p-1}, t_p)] + P[p],     row(a, b) = (a * mul_prev + b * mul_cur) mod buckets

with ``row = buckets`` (the last row of B) at p = 0.  A layer adds ``mixer(rms(x) * w1)`` and, where it has a
feed-forward, ``ff(rms(x) * w2)``.  The logits are ``logit_scale * E (rms(x) * w_final)``.

* mixer ``attention``: grouped-query attention without biases or positions.  Queries and keys pass a unit-RMS norm over
  a token's whole projection (a weight per entry); a score ``c`` becomes ``cap * tanh(scale * q.k / cap)``; a query sees
  the keys of its own run of ``size`` positions up to itself.  From the second layer with ``v_mix`` on the values are a
  blend ``(1 - l) v + l v'`` with the values ``v'`` that the first such layer made of the same token.  The heads' outputs
  are multiplied by ``sigmoid(W_g h)`` entry by entry before the output projection.
* feed-forward ``dense``: ``W_down (g * sigmoid(1.702 g) * (u + 1))`` with ``g`` cut from above and ``u`` from both sides
  at ``limit``.
* feed-forward ``moe``: the ``top`` experts with the largest softmax scores, each a gated silu feed-forward whose output is
  multiplied by its score times a constant; beside them a shared expert times one sigmoid per token.
"""

from __future__ import annotations

import copy
import math

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    x = x.to(F64)
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight.to(F64)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# --- the input ------------------------------------------------------------------------------------

def bigram_rows(ids: torch.Tensor, bigram: dict) -> torch.Tensor:
    """The row of the bigram table for every token of a sequence (Python integers: no overflow)."""
    rows = [int(bigram["buckets"])]
    for before, now in zip(ids.tolist()[:-1], ids.tolist()[1:]):
        rows.append((before * int(bigram["mul_prev"]) + now * int(bigram["mul_cur"])) % int(bigram["buckets"]))
    return torch.tensor(rows, dtype=torch.long)


def embed(config: dict, t: dict, ids: torch.Tensor) -> torch.Tensor:
    e = config.get("embedding") or {}
    x = t["embed"].to(F64)[ids] * float(e.get("scale", 1.0))
    if e.get("bigram") is not None:
        x = x + t["bigram"].to(F64)[bigram_rows(ids, e["bigram"])]
    if config.get("max_positions") is not None:
        x = x + t["pos"].to(F64)[: len(ids)]
    return x


# --- attention ------------------------------------------------------------------------------------

def chunk_mask(n: int, size: int) -> torch.Tensor:
    """[n, n] of booleans: the query at ``i`` sees the key at ``j`` (``size`` 0: all keys up to itself)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen & (i // size == j // size) if size else seen


def soft_cap(score: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(score / cap) if cap else score


def blend_values(v: torch.Tensor, first: torch.Tensor, amount: torch.Tensor) -> torch.Tensor:
    a = amount.to(F64)
    return (1.0 - a) * v + a * first


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: float, size: int) -> torch.Tensor:
    """q: [n, H, d], k: [n, G, d], v: [n, G, dv] -> [n, H, dv]."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = chunk_mask(n, size)
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for head in range(H):
        g = head // (H // G)
        score = soft_cap(q[:, head] @ k[:, g].T * scale, cap).masked_fill(~seen, -math.inf)
        out[:, head] = torch.softmax(score, dim=-1) @ v[:, g]
    return out


def attention_mixer(h: torch.Tensor, m: dict, t: dict, pre: str, eps: float, first_values: torch.Tensor | None):
    """(the update, the layer's own values [n, G * dv]); ``first_values``: those to blend with, or None."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda name: h @ t[pre + name].to(F64).T                                   # noqa: E731
    q = rms_norm(lin("q"), t[pre + "q.norm"], eps).view(n, H, d)
    k = rms_norm(lin("k"), t[pre + "k.norm"], eps).view(n, G, d)
    own = lin("v")
    v = own if first_values is None else blend_values(own, first_values, t[pre + "vmix"])
    out = attend(q, k, v.view(n, G, dv), float(m["scale"]), float(m.get("softcap") or 0.0), int((m.get("mask") or {}).get("size", 0)))
    out = out.reshape(n, H * dv) * torch.sigmoid(lin("g"))
    return out @ t[pre + "o"].to(F64).T, own


# --- feed-forward ---------------------------------------------------------------------------------

def dense_ff(h: torch.Tensor, mlp: dict, t: dict, pre: str) -> torch.Tensor:
    limit = float(mlp["limit"])
    g = torch.clamp(h @ t[pre + "gate"].to(F64).T, max=limit)
    u = torch.clamp(h @ t[pre + "up"].to(F64).T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ t[pre + "down"].to(F64).T


def expert(h: torch.Tensor, t: dict, pre: str) -> torch.Tensor:
    return (silu(h @ t[pre + "gate"].to(F64).T) * (h @ t[pre + "up"].to(F64).T)) @ t[pre + "down"].to(F64).T


def routed_choice(h: torch.Tensor, t: dict, pre: str, router: dict, chosen: torch.Tensor | None = None):
    """(indices [n, top], weights [n, top]): the largest softmax scores, times the router's constant."""
    s = torch.softmax(h @ t[pre + "router"].to(F64).T, dim=-1)
    idx = torch.topk(s, int(router["top"]), dim=-1).indices if chosen is None else chosen.long()
    return idx, torch.gather(s, 1, idx) * float(router.get("scale", 1.0))


def moe_ff(h: torch.Tensor, mlp: dict, t: dict, pre: str, chosen: torch.Tensor | None = None) -> torch.Tensor:
    """``chosen`` [n, top]: experts to use instead of the router's own choice (their scores stay the router's)."""
    idx, w = routed_choice(h, t, pre, mlp["router"], chosen)
    out = torch.zeros(h.shape[0], t[pre + "e0.down"].shape[0], dtype=F64)
    for e in range(int(mlp["router"]["experts"])):
        for slot in range(idx.shape[1]):
            rows = (idx[:, slot] == e).nonzero().flatten()
            if rows.numel():
                out[rows] += w[rows, slot][:, None] * expert(h[rows], t, f"{pre}e{e}.")
    if mlp.get("shared") is not None:
        out += torch.sigmoid(h @ t[pre + "shared.sg"].to(F64).T) * expert(h, t, pre + "shared.")
    return out


# --- the model ------------------------------------------------------------------------------------

def forward(config: dict, tensors: dict, tokens, return_layers: bool = False, chosen: dict | None = None, _gaps=None):
    """Logits [tokens, vocab] of one whole sequence (float64); with ``return_layers`` also the stream after every layer.
    ``chosen``: layer -> [tokens, top] experts that the layer's feed-forward is to use whatever its router says."""
    eps = float(config["norm"]["eps"])
    x = embed(config, tensors, torch.as_tensor(tokens, dtype=torch.long))
    first, after = None, []
    for i, layer in enumerate(config["layers"]):
        m, pre = layer["mixer"], f"l{i}."
        mixes = bool(m.get("v_mix"))
        y, own = attention_mixer(rms_norm(x, tensors[pre + "norm1"], eps), m, tensors, pre + "mix.", eps, first if mixes else None)
        if mixes and first is None:
            first = own
        x = x + y
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(x, tensors[pre + "norm2"], eps)
            if mlp["kind"] == "dense":
                x = x + dense_ff(h, mlp, tensors, pre + "mlp.")
            else:
                if _gaps is not None:
                    z = torch.sort(h @ tensors[pre + "mlp.router"].to(F64).T, dim=-1, descending=True).values
                    top = int(mlp["router"]["top"])
                    _gaps.append(z[:, top - 1] - z[:, top] if top < z.shape[1] else torch.full_like(z[:, 0], math.inf))
                x = x + moe_ff(h, mlp, tensors, pre + "mlp.", None if chosen is None else chosen.get(i))
        after.append(x.clone())
    logits = rms_norm(x, tensors["final.norm"], eps) @ tensors["embed"].to(F64).T * float(config.get("logit_scale", 1.0))
    return (logits, torch.stack(after)) if return_layers else logits


def router_margins(config: dict, tensors: dict, tokens) -> torch.Tensor:
    """Per layer with experts and token: the gap between the last chosen and the first not chosen router logit."""
    gaps: list[torch.Tensor] = []
    forward(config, tensors, tokens, _gaps=gaps)
    return torch.stack(gaps) if gaps else torch.zeros(0, len(tokens), dtype=F64)


# --- small configurations and random weights for tests ------------------------------------------------

def dense_mlp(ff=48, limit=1.5) -> dict:
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe_mlp(ff=24, experts=6, top=2, scale=1.7, shared=40) -> dict:
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def attention_layer(heads=4, kv_heads=2, dim=32, vdim=None, size=24, scale=0.2, softcap=7.0, v_mix=True, mlp=None) -> dict:
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim, "scale": scale, "v_mix": v_mix}
    if size is not None:
        mixer["mask"] = {"size": size}
    if softcap is not None:
        mixer["softcap"] = softcap
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def make_config(layers: list[dict], width=64, vocab=160, eps=1e-5, scale=5.0, buckets=97, mul_prev=13, mul_cur=7, positions=4096,
                logit_scale=0.7) -> dict:
    embedding: dict = {"scale": scale}
    if buckets:
        embedding["bigram"] = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    out = {"architecture": "Kikarax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": embedding,
           "logit_scale": logit_scale, "layers": copy.deepcopy(layers)}
    if positions:
        out["max_positions"] = positions
    return out


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    w = config["width"]
    shapes: dict[str, tuple[int, ...]] = {"embed": (config["vocab"], w)}
    bigram = (config.get("embedding") or {}).get("bigram")
    if bigram is not None:
        shapes["bigram"] = (bigram["buckets"] + 1, w)
    if config.get("max_positions") is not None:
        shapes["pos"] = (config["max_positions"], w)
    for i, layer in enumerate(config["layers"]):
        m, pre = layer["mixer"], f"l{i}.mix."
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes.update({f"l{i}.norm1": (w,), pre + "q": (H * d, w), pre + "k": (G * d, w), pre + "v": (G * dv, w),
                       pre + "q.norm": (H * d,), pre + "k.norm": (G * d,), pre + "g": (H * dv, w), pre + "o": (w, H * dv)})
        if m.get("v_mix"):
            shapes[pre + "vmix"] = ()
        mlp, f = layer.get("mlp"), f"l{i}.mlp."
        if mlp is None:
            continue
        shapes[f"l{i}.norm2"] = (w,)
        glu = lambda at, ff: {at + "gate": (ff, w), at + "up": (ff, w), at + "down": (w, ff)}     # noqa: E731
        if mlp["kind"] == "dense":
            shapes.update(glu(f, mlp["ff"]))
            continue
        shapes[f + "router"] = (mlp["router"]["experts"], w)
        for e in range(mlp["router"]["experts"]):
            shapes.update(glu(f"{f}e{e}.", mlp["expert"]["ff"]))
        if mlp.get("shared") is not None:
            shapes.update(glu(f + "shared.", mlp["shared"]["ff"]))
            shapes[f + "shared.sg"] = (1, w)
    shapes["final.norm"] = (w,)
    return shapes


def random_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Seeded weights, rounded to bfloat16 (so that both number formats of the engine see the same values)."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        noise = torch.randn(shape, generator=gen)
        if last == "vmix":
            t = 0.35 + 0.2 * noise
        elif "norm" in last:
            t = 1.0 + 0.2 * noise
            if last == "norm" and ".mix." in name:
                t = t * 1.5                                   # sharper scores: a wrong key shows
        elif name in ("embed", "bigram", "pos"):
            t = noise * {"embed": 0.4, "bigram": 0.8, "pos": 0.5}[name]
        elif last == "router":
            t = noise * 2.5 / math.sqrt(shape[1])
        else:
            t = noise / math.sqrt(shape[1])
            if last == "gate":
                t = t * 1.5                                   # so that both sides of the bound occur
        out[name] = t.to(torch.bfloat16)
    return out
