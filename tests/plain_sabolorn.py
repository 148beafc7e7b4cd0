"""A plain, slow Sabolorn in float64 on the CPU: one function per mechanism, written from the design's equations.

It shares no code with the package: it reads the same config.json keys and tensor names and computes every token of
a sequence at once with dense masks.  Notation: ``x`` rows are tokens, ``W`` is stored ``[out, in]`` and applied as
``x @ W.T``; positions count from 0.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The layers' norm: mean taken off, unit variance, a weight and no bias."""
    dev = x - x.mean(-1, keepdim=True)
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor | None = None) -> torch.Tensor:
    """y_t = b + sum_j w[:, j] * u_(t - taps + 1 + j), zeros before the start.  ``u``: [T, C], ``w``: [C, taps]."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j: j + u.shape[0]] * w[:, j]
    return y if b is None else y + b


# --- mixers -------------------------------------------------------------------------------------------------------

def ssd_recurrence(x, B, C, dt, A_log, D):
    """One head: x [T, P], B and C [T, N], dt [T] (after softplus).  S <- exp(-exp(A_log) dt) S + dt B x^T; y = S^T C + D x."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=F64)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(A_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        y[t] = S.T @ C[t] + D * x[t]
    return y


def gated_group_rms(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """(y * silu(z)), each of ``parts`` equal pieces of the row brought to unit RMS by itself, times ``w``."""
    g = y * silu(z)
    return rms_unit(g.view(g.shape[0], parts, -1), eps).reshape(g.shape) * w


def mamba2_mixer(h, w, pre, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = h @ w[pre + "in"].to(F64).T
    z, xbc, dt = proj[:, :inner], proj[:, inner: 2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[pre + "conv"].to(F64), w[pre + "conv.b"].to(F64)))
    dt = softplus(dt + w[pre + "dt_bias"].to(F64))
    x, B, C = xbc[:, :inner], xbc[:, inner: inner + G * N], xbc[:, inner + G * N:]
    A, D = w[pre + "A_log"].to(F64), w[pre + "D"].to(F64)
    ys = []
    for i in range(H):
        g = i // (H // G)
        ys.append(ssd_recurrence(x[:, i * P: (i + 1) * P], B[:, g * N: (g + 1) * N], C[:, g * N: (g + 1) * N], dt[:, i], A[i], D[i]))
    y = gated_group_rms(torch.cat(ys, -1), z, w[pre + "norm"].to(F64), m["norm_groups"], eps)
    return y @ w[pre + "o"].to(F64).T


def causal_softmax(scores: torch.Tensor) -> torch.Tensor:
    """Softmax of [query, key] scores over the keys j <= i."""
    n = scores.shape[0]
    seen = torch.arange(n)[None, :] <= torch.arange(n)[:, None]
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), -1)


def distance_bias(n: int, r1: float, r2: float) -> torch.Tensor:
    """[query, key]: r1 * ln(1 + r2 * (i - j)) where j <= i, 0 elsewhere."""
    d = (torch.arange(n, dtype=F64)[:, None] - torch.arange(n, dtype=F64)[None, :]).clamp(min=0.0)
    return r1 * torch.log1p(r2 * d)


def attention_mixer(h, w, pre, m, eps=None):
    """Grouped-query attention: biases, a short convolution on q, k and v, a penalty that grows with the log of the distance."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ w[pre + n].to(F64).T + w[pre + n + ".b"].to(F64), w[pre + n + ".conv"].to(F64)) for n in "qkv")
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    heads = []
    for i in range(H):
        g = i // (H // G)
        score = (q[:, i] @ k[:, g].T) * m["scale"]
        score = score - distance_bias(T, float(w[pre + "r1"][i]), float(w[pre + "r2"][i]))
        heads.append(causal_softmax(score) @ v[:, g])
    return torch.cat(heads, -1) @ w[pre + "o"].to(F64).T


def yarn(base: float, dims: int, scaling: dict | None) -> tuple[torch.Tensor, float]:
    """(frequencies, what multiplies cosines and sines): fast pairs keep theirs, slow ones are divided by the factor, with
    a ramp between the pairs that make ``fast`` and ``slow`` turns within ``original`` positions."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    if not scaling:
        return f, 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])
    pair = lambda turns: dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))    # noqa: E731
    lo = max(math.floor(pair(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f.tolist()):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x: torch.Tensor, pos: torch.Tensor, freq: torch.Tensor, mult: float = 1.0) -> torch.Tensor:
    """Entry 2i is paired with entry 2i + 1 among the first ``2 len(freq)`` of the last axis; cos and sin times ``mult``."""
    half = freq.numel()
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    a = (pos.to(F64)[:, None] * freq[None, :]).reshape(shape)
    c, s = mult * a.cos(), mult * a.sin()
    out = x.clone()
    u, v = x[..., 0: 2 * half: 2], x[..., 1: 2 * half: 2]
    out[..., 0: 2 * half: 2] = u * c - v * s
    out[..., 1: 2 * half: 2] = v * c + u * s
    return out


def latent_rows(h, w, pre, m, eps):
    """What a layer's cache holds: the normed latent [T, kv_rank] and the rotated key part [T, rot_dim]."""
    r = m["kv_rank"]
    freq, mult = yarn(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    down = h @ w[pre + "dkv"].to(F64).T
    c = rms_unit(down[:, :r], eps) * w[pre + "dkv.norm"].to(F64)
    return c, rotate_pairs(down[:, r:], torch.arange(h.shape[0]), freq, mult)


def latent_attention_mixer(h, w, pre, m, eps, rows):
    """``rows``: the (latent, rotated key part) to attend over, this layer's own or another layer's."""
    T, H, d, dr, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    freq, mult = yarn(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    cq = rms_unit(h @ w[pre + "dq"].to(F64).T, eps) * w[pre + "dq.norm"].to(F64)
    q = (cq @ w[pre + "uq"].to(F64).T).view(T, H, d + dr)
    q_plain, q_rot = q[..., :d], rotate_pairs(q[..., d:], torch.arange(T), freq, mult)
    c, k_rot = rows
    k_plain = (c @ w[pre + "uk"].to(F64).T).view(T, H, d)
    v = (c @ w[pre + "uv"].to(F64).T).view(T, H, dv)
    heads = []
    for i in range(H):
        score = (q_plain[:, i] @ k_plain[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        heads.append(causal_softmax(score) @ v[:, i])
    out = torch.cat(heads, -1) * torch.sigmoid(h @ w[pre + "g"].to(F64).T)
    return out @ w[pre + "o"].to(F64).T


# --- feed-forward -------------------------------------------------------------------------------------------------

def dense_ff(h, w, pre):
    return (torch.relu(h @ w[pre + "up"].to(F64).T) ** 2) @ w[pre + "down"].to(F64).T


def expert_ff(h, w, pre):
    return (silu(h @ w[pre + "gate"].to(F64).T) * (h @ w[pre + "up"].to(F64).T)) @ w[pre + "down"].to(F64).T


def routed_choice(h, w_router, correction, router) -> torch.Tensor:
    """Chosen experts [T, top]: the largest of sigmoid scores plus correction, among the best groups only (a group's
    score: the sum of its two largest corrected scores)."""
    s = torch.sigmoid(h @ w_router.to(F64).T) + correction.to(F64)
    T, E = s.shape
    groups = router.get("groups")
    if groups:
        count, keep = groups["count"], groups["keep"]
        by_group = s.view(T, count, E // count)
        score = by_group.sort(-1, descending=True).values[..., :2].sum(-1)
        kept = score.topk(keep, -1).indices
        for t in range(T):
            for g in range(count):
                if g not in kept[t].tolist():
                    s.view(T, count, E // count)[t, g] = float("-inf")
    return s.topk(router["top"], -1).indices


def moe_ff(h, w, pre, mlp, chosen=None):
    """``chosen`` [T, top]: experts handed in (their weights are still this router's scores), else the router's own."""
    if chosen is None:
        chosen = routed_choice(h, w[pre + "router"], w[pre + "correction"], mlp["router"])
    s = torch.sigmoid(h @ w[pre + "router"].to(F64).T).gather(1, chosen.long())
    weight = s / (s.sum(-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(chosen[t].tolist(), weight[t].tolist()):
            out[t] += p * expert_ff(h[t: t + 1], w, f"{pre}e{e}.")[0]
    return out


# --- the stack ----------------------------------------------------------------------------------------------------

def token_side(x, e, w, pre, eps):
    """x + RMSnorm(proj(gelu(gate x) * e)): the layer's own embedding ``e`` of the tokens, gated by the stream."""
    g = gelu_tanh(x @ w[pre + "side.gate"].to(F64).T) * e
    return x + rms_unit(g @ w[pre + "side.proj"].to(F64).T, eps) * w[pre + "side.norm"].to(F64)


def depth_average(history: list, weights: torch.Tensor) -> torch.Tensor:
    out = torch.zeros_like(history[0])
    for X, a in zip(history, weights.to(F64).tolist()):
        out = out + a * X
    return out


def forward(w: dict, cfg: dict, tokens: list[int], layers_out: list | None = None, chosen: dict | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` receives every layer's result (before the averaging over depth);
    ``chosen``: layer -> the experts [T, top] to use there instead of the router's choice."""
    eps = cfg["norm"]["eps"]
    ids = torch.tensor(tokens)
    x = w["embed"].to(F64)[ids] * cfg["embedding"]["scale"]
    history, rows = [x], {}
    side = cfg.get("token_side")
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        h = layer_norm(x, w[pre + "norm1"].to(F64), eps)
        if layer["type"] == "mamba2":
            y = mamba2_mixer(h, w, pre + "mix.", m, eps)
        elif layer["type"] == "attention":
            y = attention_mixer(h, w, pre + "mix.", m)
        else:
            src = m.get("kv_from")
            if src is None:
                rows[i] = latent_rows(h, w, pre + "mix.", m, eps)
            y = latent_attention_mixer(h, w, pre + "mix.", m, eps, rows[i if src is None else src])
        mlp = layer.get("mlp")
        if mlp:
            y = y + (dense_ff(h, w, pre + "mlp.") if mlp["kind"] == "dense" else
                     moe_ff(h, w, pre + "mlp.", mlp, None if chosen is None else chosen.get(i)))
        x = x + y
        if side:
            x = token_side(x, w["side.embed"].to(F64)[ids][:, i * side["dim"]: (i + 1) * side["dim"]], w, pre, eps)
        history.append(x)
        if layers_out is not None:
            layers_out.append(x.clone())
        x = depth_average(history, w[pre + "dwa"])
    logits = layer_norm(x, w["final.norm"].to(F64), eps) @ w["embed"].to(F64).T
    cap = float(cfg.get("logit_softcap") or 0.0)
    return cap * torch.tanh(logits / cap) if cap else logits


def greedy(w: dict, cfg: dict, prompt: list[int], n_new: int) -> list[int]:
    seq, out = list(prompt), []
    for _ in range(n_new):
        out.append(int(forward(w, cfg, seq)[-1].argmax()))
        seq.append(out[-1])
    return out


# --- configurations and random weights for the tests --------------------------------------------------------------

def mamba_layer(heads=4, vdim=8, state=12, groups=2, conv=4, norm_groups=2, mlp=None) -> dict:
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": mlp}


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, scale=None, mlp=None) -> dict:
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                           "scale": scale or dim ** -0.5}, "mlp": mlp}


def latent_layer(heads=3, dim=8, rot_dim=8, vdim=16, kv_rank=24, q_rank=20, scale=None, base=500.0, scaling=None, kv_from=None,
                 mlp=None) -> dict:
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
             "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}
    if scaling:
        mixer["rot"]["scaling"] = scaling
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def dense_mlp(ff=48) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_mlp(ff=16, experts=6, top=2, groups=(3, 2)) -> dict:
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def make_config(layers: list[dict], width=32, vocab=97, eps=1e-5, scale=3.0, side=8, softcap=9.0) -> dict:
    out = {"architecture": "Sabolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "logit_softcap": softcap, "layers": layers}
    return {**out, "token_side": {"dim": side}} if side else out


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    W, S, n = cfg["width"], (cfg.get("token_side") or {}).get("dim", 0), len(cfg["layers"])
    shapes: dict[str, tuple[int, ...]] = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    if S:
        shapes["side.embed"] = (cfg["vocab"], n * S)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        shapes.update({p + "norm1": (W,), p + "dwa": (i + 2,)})
        if S:
            shapes.update({p + "side.gate": (S, W), p + "side.proj": (W, S), p + "side.norm": (W,)})
        if layer["type"] == "mamba2":
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            ch = H * P + 2 * G * N
            shapes.update({x + "in": (H * P + ch + H, W), x + "conv": (ch, m["conv"]), x + "conv.b": (ch,), x + "dt_bias": (H,),
                           x + "A_log": (H,), x + "D": (H,), x + "norm": (H * P,), x + "o": (W, H * P)})
        elif layer["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                shapes.update({x + name: (rows, W), x + name + ".b": (rows,), x + name + ".conv": (rows, m["conv"])})
            shapes.update({x + "r1": (H,), x + "r2": (H,), x + "o": (W, H * dv)})
        else:
            H, d, dr, dv, r, rq = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            shapes.update({x + "dq": (rq, W), x + "dq.norm": (rq,), x + "uq": (H * (d + dr), rq)})
            if m.get("kv_from") is None:
                shapes.update({x + "dkv": (r + dr, W), x + "dkv.norm": (r,)})
            shapes.update({x + "uk": (H * d, r), x + "uv": (H * dv, r), x + "g": (H * dv, W), x + "o": (W, H * dv)})
        mlp = layer.get("mlp")
        if not mlp:
            continue
        if mlp["kind"] == "dense":
            shapes.update({p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
        else:
            ff, experts = mlp["expert"]["ff"], mlp["router"]["experts"]
            for e in range(experts):
                shapes.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
            shapes.update({p + "mlp.router": (experts, W), p + "mlp.correction": (experts,)})
    return shapes


def random_weights(cfg: dict, seed: int = 0, dtype: torch.dtype = torch.bfloat16) -> dict[str, torch.Tensor]:
    """Weights of a size that keeps every sublayer's update comparable with the stream."""
    gen = torch.Generator().manual_seed(seed)
    normal = lambda shape, std=1.0, mean=0.0: mean + std * torch.randn(shape, generator=gen)                # noqa: E731
    between = lambda shape, lo, hi: lo + (hi - lo) * torch.rand(shape, generator=gen)                       # noqa: E731
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if name in ("embed", "side.embed"):
            t = normal(shape)
        elif leaf == "norm" and ".side." in name:
            t = normal(shape, 0.1, 0.7)
        elif leaf in ("norm1", "norm"):
            t = normal(shape, 0.1, 1.0)
        elif leaf == "dwa":
            t = normal(shape, 0.3)
            t[-1] += 1.0
        elif leaf == "conv":
            t = normal(shape, shape[1] ** -0.5)
        elif leaf == "b":
            t = normal(shape, 0.3)
        elif leaf == "dt_bias":
            t = between(shape, -3.5, -0.5)
        elif leaf == "A_log":
            t = between(shape, -4.0, 0.5)
        elif leaf == "D":
            t = normal(shape, 0.5, 1.0)
        elif leaf == "r1":
            t = between(shape, 0.0, 2.0)
        elif leaf == "r2":
            t = between(shape, 0.05, 0.6)
        elif leaf == "router":
            t = normal(shape, 2.0 * shape[1] ** -0.5)
        elif leaf == "correction":
            t = normal(shape, 0.4, -0.5)
        else:
            t = normal(shape, 1.2 * shape[-1] ** -0.5)
        out[name] = t.to(dtype)
    return out
