"""Sabolorn through the engine against the plain implementation of ``plain_sabolorn``.

Small configurations with random weights of their own: head counts, state, key and value sizes, convolution lengths, groups,
expert counts and choices, side widths that differ from layer to layer and from test to test (also the degenerate ones: one
kv head, as many as heads, one tap, one group, all groups kept, groups of one expert, one expert chosen, no groups, no
scaling of the rotation, a scaling whose factor is 1, a layer without a feed-forward, constants of 1).  Every mechanism
alone; whole prompts against token-by-token decoding and portions down to two tokens; unequal requests in one batch with
pages and slots that are freed, poisoned and used again; keys made dominant far away, at page borders, at position 0 and at
their own, under a penalty that would otherwise hide them; a state and convolution records cut anywhere; the first tokens;
long decoding; greedy generation through ``Engine.generate`` and the scheduler; the trace replay program.

In bfloat16 a router's close call may fall the other way than in the plain float64 implementation, which changes a
token's experts, not the arithmetic under test.  So the bfloat16 comparisons hand the plain implementation the experts
that the engine chose (read from the device lists of the feed-forward); float32 comparisons use the plain router.
"""

from __future__ import annotations

import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_sabolorn as plain

ROOT = Path(__file__).resolve().parent.parent

YARN = {"factor": 6.0, "original": 64, "fast": 8.0, "slow": 1.0}
MAM = plain.mamba_layer(heads=4, vdim=8, state=12, groups=2, conv=4, norm_groups=2, mlp=plain.moe_mlp(ff=16, experts=6, top=2, groups=(3, 2)))
MAM_B = plain.mamba_layer(heads=3, vdim=16, state=16, groups=1, conv=2, norm_groups=1, mlp=plain.dense_mlp(40))
MAM_C = plain.mamba_layer(heads=6, vdim=5, state=7, groups=3, conv=1, norm_groups=5, mlp=None)
ATT = plain.attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, mlp=plain.dense_mlp(48))
ATT_B = plain.attention_layer(heads=3, kv_heads=3, dim=20, vdim=12, conv=2, scale=0.3, mlp=plain.moe_mlp(ff=24, experts=8, top=3, groups=(2, 1)))
ATT_C = plain.attention_layer(heads=6, kv_heads=1, dim=8, vdim=8, conv=1, mlp=None)
ATT_D = plain.attention_layer(heads=2, kv_heads=1, dim=64, vdim=64, conv=3, mlp=plain.moe_mlp(ff=8, experts=5, top=1, groups=None))
LAT = plain.latent_layer(heads=3, dim=8, rot_dim=8, vdim=16, kv_rank=24, q_rank=20, scaling=YARN, mlp=plain.moe_mlp(ff=16, experts=4, top=2, groups=(4, 3)))
LAT_B = plain.latent_layer(heads=5, dim=16, rot_dim=4, vdim=8, kv_rank=40, q_rank=12, base=20000.0, mlp=plain.dense_mlp(40))
LAT_C = plain.latent_layer(heads=2, dim=24, rot_dim=16, vdim=24, kv_rank=16, q_rank=32, scaling={**YARN, "factor": 1.0}, mlp=None)


def _reading(layer: dict, source: int, **over) -> dict:
    """A latent layer that reads layer ``source``'s cache rows: the latent's size and rotation are those of ``layer``."""
    out = copy.deepcopy(layer)
    out["mixer"].update(kv_from=source, **over)
    return out


FULL = plain.make_config([ATT, MAM, LAT, ATT_B, _reading(LAT, 2, heads=4, dim=12, vdim=8, q_rank=16), MAM_B, LAT_B, MAM_C, ATT_C,
                          _reading(LAT, 2, heads=2), ATT_D], width=80, vocab=203, eps=1e-5, scale=2.5, side=12, softcap=11.0)

ALONE = {
    "mamba_grouped_experts": plain.make_config([MAM]),
    "mamba_one_group_two_taps_dense": plain.make_config([MAM_B], width=72, scale=1.0),
    "mamba_one_tap_odd_sizes_no_ffn": plain.make_config([MAM_C], width=40, side=5),
    "attention_dense": plain.make_config([ATT]),
    "attention_all_kv_heads_two_taps_one_group_kept": plain.make_config([ATT_B], width=56, side=3),
    "attention_one_kv_head_one_tap_no_ffn": plain.make_config([ATT_C], width=48, softcap=30.0),
    "attention_heads_of_64_one_expert": plain.make_config([ATT_D], width=64),
    "latent_stretched_rotation_groups_of_one": plain.make_config([LAT]),
    "latent_plain_rotation_dense": plain.make_config([LAT_B], width=88),
    "latent_factor_one_no_ffn": plain.make_config([LAT_C], width=40),
    "rows_of_50_entries": plain.make_config([MAM_B, ATT, LAT], width=50, vocab=61, side=7),
    "no_side_input_no_cap": plain.make_config([ATT, MAM_C, LAT], width=64, side=0, softcap=0.0),
    "latent_reading_another_layers_rows": plain.make_config([LAT, _reading(LAT, 0, heads=5, dim=4, vdim=12, q_rank=8)], side=1),
}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from edgerag_b200.weights.safetensors_io import write_safetensors

    base = tmp_path_factory.mktemp("sabolorn")
    made = {}

    def get(name: str, raw: dict, seed: int = 0, edit=None):
        if name not in made:
            folder = base / name
            folder.mkdir()
            tensors = plain.random_weights(raw, seed)
            if edit is not None:
                edit(tensors)
            (folder / "config.json").write_text(json.dumps(raw))
            write_safetensors(folder / "model.safetensors", tensors)
            made[name] = (folder, raw, tensors)
        return made[name]

    return get


class ChoiceLog:
    """Records, for every layer with routed experts, the experts the engine chose for the rows of every step."""

    def __init__(self, model) -> None:
        self.steps: list[dict[int, torch.Tensor]] = []
        for i, block in enumerate(model.blocks):
            if block.ffn is not None and hasattr(block.ffn, "n_experts"):
                block.ffn.forward = self._wrap(i, block.ffn)

    def _wrap(self, layer, ffn):
        inner = ffn.forward

        def forward(x, ctx):
            from edgerag_b200.ops import kernels

            out = inner(x, ctx)
            n = x.shape[0]
            lists = ctx.buf("moe.lists", (kernels.moe_lists_ints(n, ffn.n_experts, ffn.top),), torch.int32)
            if self.steps:
                self.steps[-1][layer] = lists[: n * ffn.top].reshape(n, ffn.top).cpu().clone()
            return out

        return forward

    def new_step(self) -> None:
        self.steps.append({})

    def of_rows(self, picks: list[tuple[int, int, int]]) -> dict[int, torch.Tensor]:
        layers = self.steps[picks[0][0]].keys()
        return {layer: torch.cat([self.steps[s][layer][first: first + n] for s, first, n in picks]) for layer in layers}


def make_engine(folder, dtype, **over):
    from edgerag_b200.engine.engine import Engine, EngineOptions

    opts = dict(dtype=dtype, block_size=16, num_blocks=64, max_batch_size=4, max_step_tokens=512, max_model_len=1 << 20,
                cuda_graphs=False, poison_freed_pages=True)
    opts.update(over)
    eng = Engine.from_pretrained(folder, EngineOptions(**opts))
    eng.log = ChoiceLog(eng.model)
    return eng


def feed(runner, rid, tokens, cuts, log: ChoiceLog | None = None):
    from edgerag_b200.engine.step import StepEntry

    rows, pos, picks = [], 0, []
    for c in cuts:
        c = min(c, len(tokens) - pos)
        if c <= 0:
            break
        if log is not None:
            log.new_step()
            picks.append((len(log.steps) - 1, 0, c))
        out = runner.step([StepEntry(rid, tokens=tokens[pos: pos + c], want=list(range(c)))])
        rows.append(out.float().cpu().clone())
        pos += c
    assert pos == len(tokens), "the cuts do not cover the tokens"
    return torch.cat(rows), (log.of_rows(picks) if log is not None and log.steps and log.steps[picks[0][0]] else None)


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)


#: float32 (worst row, mean over rows): only the order of sums differs from the plain implementation.
#: bfloat16 (mean over rows, worst row): activations are rounded to 8 bits between the products.
BANDS = {"float32": (2e-4, 4e-5), "bfloat16": (2.5e-2, 0.12)}


def assert_close(got, want, dtype, what=""):
    assert torch.isfinite(got).all(), f"{what} {dtype}: non-finite logits"
    e = row_errors(got, want)
    where = f"{what} {dtype}: worst {e.max():.2e} (row {int(e.argmax())}), mean {e.mean():.2e}"
    worst, mean = (BANDS[dtype][0], BANDS[dtype][1]) if dtype == "float32" else (BANDS[dtype][1], BANDS[dtype][0])
    assert e.max() <= worst and e.mean() <= mean, where


def tokens_for(raw, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, raw["vocab"], (n,), generator=g).tolist()


def check_request(eng, raw, tensors, toks, cuts, dtype, what):
    eng.runner.admit(what)
    got, chosen = feed(eng.runner, what, toks, cuts, eng.log if dtype == "bfloat16" else None)
    eng.runner.release(what)
    want = plain.forward(tensors, raw, toks, chosen=chosen)
    assert_close(got, want, dtype, what)
    eng.cache.check_invariants()


# --- configuration, plan, plain mechanisms (CPU) ---------------------------------------------------

def test_plan_names_every_tensor_and_declares_pages_and_records():
    from edgerag_b200.config.registry import architecture_of
    from edgerag_b200.models.decoder import DecoderModel

    arch = architecture_of(FULL)
    cfg = arch.read_config(FULL, "test")
    model = DecoderModel(arch.make_plan(cfg), torch.float32, torch.device("cpu"))
    specs = {s.name: tuple(s.shape) for s in model.weight_specs()}
    assert specs.pop("head") == (FULL["vocab"], FULL["width"])            # tied to the embedding where absent
    assert specs == plain.tensor_shapes(FULL)
    groups = {(g.n_kv_heads, g.head_dim, g.v_head_dim): g.n_layers for g in model.cache_layout.groups}
    # (attention heads padded to one size; the two layers that read layer 2's rows have none of their own)
    assert groups == {(2, 24, None): 1, (1, 32, 0): 1, (3, 24, None): 1, (1, 44, 0): 1, (1, 8, None): 1, (1, 64, None): 1}
    states = {s.name.split("@")[0]: 0 for s in model.cache_layout.states}
    assert set(states) == {"attn_conv", "conv", "ssm"}
    shapes = [tuple(s.shape) for s in model.cache_layout.states if s.name.startswith("attn_conv")]
    assert shapes == [(3, (4 + 2 + 2) * 24), (1, 9 * 24), (2, (2 + 1 + 1) * 64)]                    # one tap: no record
    assert model.graph_safe and model.needs_token_ids
    assert model.head.softcap == 11.0 and model.embedding.scale == 2.5
    reads = [(c.layer, c.cache_layer, c.writes_cache) for c in model.schedule if hasattr(c, "layer")]
    assert reads[4] == (4, reads[2][1], False) and reads[9] == (9, reads[2][1], False) and all(w for i, (_, _, w) in enumerate(reads) if i not in (4, 9))


def test_configuration_errors_name_the_key():
    from edgerag_b200.config.model_config import ConfigError
    from edgerag_b200.models.sabolorn import SabolornConfig

    def broken(change):
        raw = copy.deepcopy(plain.make_config([ATT, LAT, MAM, _reading(LAT, 1)]))
        change(raw)
        return raw

    SabolornConfig.from_dict(broken(lambda r: None), "t")
    cases = [
        (lambda r: r["layers"][0].update(type="delta"), "unknown layer type"),
        (lambda r: r["layers"][0]["mixer"].pop("kv_heads"), "kv_heads"),
        (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "kv_heads must divide"),
        (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
        (lambda r: r["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
        (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
        (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
        (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
        (lambda r: r["layers"][1]["mlp"].update(kind="glu"), "mlp.kind"),
        (lambda r: r["layers"][1]["mlp"]["router"].update(top=9), "router.top"),
        (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(count=3), "router.groups"),
        (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(keep=1), "router.groups"),
        (lambda r: r["layers"][2]["mlp"]["expert"].pop("ff"), "ff"),
        (lambda r: r["layers"][2]["mixer"].update(groups=3), "groups must divide"),
        (lambda r: r["layers"][3]["mixer"].update(kv_from=0), "kv_from"),
        (lambda r: r["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
        (lambda r: r["layers"][3]["mixer"].update(kv_rank=8), "kv_from"),
        (lambda r: r["token_side"].pop("dim"), "dim"),
        (lambda r: r.pop("norm"), "norm"),
        (lambda r: r.pop("width"), "width"),
    ]
    for change, word in cases:
        with pytest.raises(ConfigError, match=word):
            SabolornConfig.from_dict(broken(change), "t")


def test_stretched_frequencies_and_their_multiplier():
    from edgerag_b200.parts.rope import rotary_frequencies, rotary_multiplier

    for base, dims, sc in ((1000.0, 16, YARN), (10000.0, 64, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                           (500.0, 8, {"factor": 40.0, "original": 20, "fast": 32.0, "slow": 0.5}),
                           (700.0, 4, {"factor": 1.0, "original": 100, "fast": 8.0, "slow": 2.0})):
        f, mult = plain.yarn(base, dims, sc)
        assert torch.allclose(rotary_frequencies(base, dims, sc), f, rtol=1e-14, atol=0) and rotary_multiplier(sc) == pytest.approx(mult, rel=1e-15)
        plain_f, one = plain.yarn(base, dims, None)
        assert one == 1.0 and torch.equal(rotary_frequencies(base, dims), plain_f) and rotary_multiplier(None) == 1.0
        assert ((f <= plain_f * (1 + 1e-15)) & (f >= plain_f / sc["factor"] * (1 - 1e-15))).all()
    # by hand: dims 16, base 1000: pair(8) = 16 ln(64 / (16 pi)) / (2 ln 1000) = 0.28 -> 0, pair(1) = 2.69 -> 3
    f, mult = plain.yarn(1000.0, 16, YARN)
    g = [1000.0 ** (-i / 8) for i in range(8)]
    want = [g[0], g[1] * (2 / 3 + 1 / 18), g[2] * (1 / 3 + 1 / 9), g[3] / 6, g[4] / 6, g[5] / 6, g[6] / 6, g[7] / 6]
    assert torch.allclose(f, torch.tensor(want, dtype=torch.float64)) and mult == pytest.approx(1 + 0.1 * math.log(6.0))


def test_plain_router_by_hand():
    """The correction decides the choice and not the weights; a group counts its two best; ruled-out groups lose even to
    negative choice scores."""
    z = torch.tensor([[0.0, 4.0, 1.0, 1.0, -2.0, 3.0]], dtype=torch.float64)
    eye = torch.eye(6, dtype=torch.float64)
    s = torch.sigmoid(z)[0]
    none = torch.zeros(6, dtype=torch.float64)
    pick = lambda corr, **router: sorted(plain.routed_choice(z, eye, corr, {"experts": 6, **router})[0].tolist())   # noqa: E731
    assert pick(none, top=2) == [1, 5]
    # groups (0,1) 0.5+0.98, (2,3) 0.73+0.73, (4,5) 0.12+0.95: the best single expert but one is in the worst group
    assert pick(none, top=2, groups={"count": 3, "keep": 2}) == [1, 2] or pick(none, top=2, groups={"count": 3, "keep": 2}) == [1, 3]
    corr = torch.tensor([-3.0, -3.0, -3.0, -3.0, -1.0, -9.0], dtype=torch.float64)
    assert pick(corr, top=2, groups={"count": 3, "keep": 2}) == [1, 2] or pick(corr, top=2, groups={"count": 3, "keep": 2}) == [1, 3]
    assert pick(corr, top=1) == [4]
    w = {"p.router": eye, "p.correction": corr}
    h = z
    for e in range(6):
        w.update({f"p.e{e}.gate": torch.full((1, 6), 0.1, dtype=torch.float64), f"p.e{e}.up": torch.ones(1, 6, dtype=torch.float64),
                  f"p.e{e}.down": torch.full((6, 1), float(e), dtype=torch.float64)})
    out = plain.moe_ff(h, w, "p.", {"router": {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}}, torch.tensor([[1, 2]]))
    base = plain.silu((0.1 * z.sum())) * z.sum()
    assert torch.allclose(out[0], base * (s[1] * 1 + s[2] * 2) / (s[1] + s[2]) * torch.ones(6, dtype=torch.float64))


def test_plain_penalty_convolution_and_recurrence_by_hand():
    b = plain.distance_bias(4, 1.5, 0.5)
    assert b[3, 0] == pytest.approx(1.5 * math.log(2.5)) and b[2, 2] == 0.0 and b[1, 3] == 0.0
    x = torch.arange(1.0, 6.0, dtype=torch.float64)[:, None]
    y = plain.causal_conv(x, torch.tensor([[2.0, 0.0, 1.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64))
    assert torch.allclose(y[:, 0], torch.tensor([1.5, 2.5, 5.5, 8.5, 11.5], dtype=torch.float64))
    one = torch.ones(3, 1, dtype=torch.float64)
    dt = torch.tensor([1.0, 2.0, 0.5], dtype=torch.float64)
    y = plain.ssd_recurrence(one, one, one, dt, torch.tensor(0.0, dtype=torch.float64), torch.tensor(10.0, dtype=torch.float64))
    s1 = 1.0
    s2 = math.exp(-2.0) * s1 + 2.0
    s3 = math.exp(-0.5) * s2 + 0.5
    assert torch.allclose(y[:, 0], torch.tensor([s1, s2, s3], dtype=torch.float64) + 10.0)
    hist = [torch.full((2, 3), float(k), dtype=torch.float64) for k in (1, 10, 100)]
    assert torch.allclose(plain.depth_average(hist, torch.tensor([2.0, -1.0, 0.5])), torch.full((2, 3), 42.0, dtype=torch.float64))


# --- every mechanism alone ------------------------------------------------------------------------

@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_alone(name, dtype, folders):
    folder, raw, tensors = folders(name, ALONE[name], seed=11)
    toks = tokens_for(raw, 75, 5)
    eng = make_engine(folder, dtype)
    check_request(eng, raw, tensors, toks, [75], dtype, f"{name} whole")
    check_request(eng, raw, tensors, toks, [17, 2, 1, 1, 16, 3, 1, 1, 1, 2, 20, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1], dtype, f"{name} in portions")


@pytest.mark.gpu
def test_layers_agree_with_plain_one_by_one(folders):
    """Every layer's result (float32), before and after the average over depth."""
    from edgerag_b200.engine.step import StepEntry
    from edgerag_b200.parts.base import DepthUpdate, settle_update

    folder, raw, tensors = folders("full", FULL, seed=1)
    toks = tokens_for(raw, 50, 2)
    want: list = []
    plain.forward(tensors, raw, toks, layers_out=want)
    eng = make_engine(folder, "float32")
    r, model = eng.runner, eng.model
    r.admit("x")
    r.pools.zero_slots(r.cache.drain_new_slots())
    ctx, ordered = r.prepare([StepEntry("x", tokens=toks, want=[])])
    hidden = ctx.buf("model.hidden", (len(toks), model.hidden_size), torch.float32)
    model.embedding.forward(ctx, hidden)
    for op in model.stream_ops:
        op.begin(ctx, hidden)
    delta, done = None, [tensors["embed"].double()[torch.tensor(toks)] * raw["embedding"]["scale"]]
    for call in model.schedule:
        if hasattr(call, "layer"):
            delta = model.blocks[call.layer].forward(hidden, delta, ctx, call)
            continue
        delta = model.stream_ops[call.op].forward(hidden, delta, ctx, call)
        if not isinstance(delta, DepthUpdate):
            continue
        layer = call.index
        settle_update(hidden, delta, model.dtype)
        err = (delta.history[layer + 1].cpu().double() - want[layer]).abs().max() / want[layer].abs().max()
        assert err < 2e-5, f"layer {layer}: {err:.2e}"
        done.append(want[layer])
        mean = plain.depth_average(done, tensors[f"l{layer}.dwa"])
        assert (hidden.cpu().double() - mean).abs().max() / mean.abs().max() < 2e-5, f"average after layer {layer}"
        delta = None
    r.finish(ordered)


# --- the whole model: prompts, decoding, portions, batches ------------------------------------------

@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_decoding_and_portions_agree_with_plain(dtype, folders):
    folder, raw, tensors = folders("full", FULL, seed=1)
    toks = tokens_for(raw, 150, 6)
    eng = make_engine(folder, dtype)
    for rid, cuts in (("whole", [150]), ("decode", [40] + [1] * 110), ("portions", [2, 31, 2, 16, 15, 1, 2, 33, 3, 2, 2, 17] + [1] * 30),
                      ("pairs", [2] * 75), ("from the first token", [1] * 60 + [90])):
        check_request(eng, raw, tensors, toks, cuts, dtype, rid)


@pytest.mark.gpu
@pytest.mark.parametrize("page", [4, 64])
def test_other_page_sizes(page, folders):
    folder, raw, tensors = folders("full", FULL, seed=1)
    toks = tokens_for(raw, 90, 8)
    eng = make_engine(folder, "float32", block_size=page, num_blocks=256 // page)
    check_request(eng, raw, tensors, toks, [33, 2, 1, 1, 19] + [1] * 34, "float32", f"pages of {page}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_equal_each_alone(dtype, folders):
    """Portions of some requests beside single tokens of others; a request pauses for a step; requests end and their
    pages and state slots go to new ones (four slots, six requests, freed pages poisoned).  A slot that is used again
    must start from zeros: a state or a convolution's record left behind by the request before shows in the first rows."""
    from edgerag_b200.engine.step import StepEntry

    folder, raw, tensors = folders("full", FULL, seed=1)
    lens = {"a": 70, "b": 33, "c": 1, "d": 90, "e": 18, "f": 47}
    toks = {k: tokens_for(raw, n, 20 + i) for i, (k, n) in enumerate(lens.items())}
    eng = make_engine(folder, dtype, num_blocks=14)       # 224 tokens of pages: never room for all at once
    r = eng.runner
    plan = [
        [("a", 30), ("b", 2)], [("a", 1), ("b", 16), ("c", 1)], [("a", 17), ("b", 1)], [("b", 14), ("d", 40), ("a", 1)],
        [("a", 21), ("d", 1)], [("d", 33), ("e", 2)], [("d", 16), ("e", 1), ("f", 3)], [("e", 15), ("f", 1)], [("f", 43)],
    ]
    fed = {k: 0 for k in lens}
    got = {k: [] for k in lens}
    picks = {k: [] for k in lens}
    slots_seen = {}
    for step in plan:
        entries = []
        for rid, n in step:
            if fed[rid] == 0:
                r.admit(rid)
                slots_seen[rid] = eng.cache.requests[rid].slot
            entries.append(StepEntry(rid, tokens=toks[rid][fed[rid]: fed[rid] + n], want=list(range(n))))
        eng.log.new_step()
        first_row, row = {}, 0                               # the runner puts single tokens first: every entry's rows in the step
        for rid, n in sorted(step, key=lambda e: e[1] != 1):
            first_row[rid] = row
            row += n
        out = r.step(entries).float().cpu()
        row = 0
        for rid, n in step:
            got[rid].append(out[row: row + n].clone())
            picks[rid].append((len(eng.log.steps) - 1, first_row[rid], n))
            row += n
            fed[rid] += n
            if fed[rid] == lens[rid]:
                r.release(rid)
        eng.cache.check_invariants()
    assert fed == lens
    assert len(set(slots_seen.values())) < len(lens), "no state slot was used twice"
    for rid in lens:
        chosen = eng.log.of_rows(picks[rid]) if dtype == "bfloat16" else None
        assert_close(torch.cat(got[rid]), plain.forward(tensors, raw, toks[rid], chosen=chosen), dtype, f"request {rid}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, folders):
    folder, raw, tensors = folders("full", FULL, seed=1)
    toks = tokens_for(raw, 260, 9)
    eng = make_engine(folder, dtype)
    check_request(eng, raw, tensors, toks, [3] + [1] * 257, dtype, "260 tokens, 257 of them one by one")


LARGER = [
    plain.mamba_layer(heads=8, vdim=32, state=64, groups=2, conv=4, norm_groups=2, mlp=plain.moe_mlp(ff=64, experts=8, top=2, groups=(4, 3))),
    plain.attention_layer(heads=8, kv_heads=2, dim=64, vdim=64, conv=4, mlp=plain.dense_mlp(256)),
    plain.latent_layer(heads=16, dim=32, rot_dim=32, vdim=32, kv_rank=64, q_rank=96, base=10000.0,
                       scaling={"factor": 4.0, "original": 256, "fast": 32.0, "slow": 1.0}, mlp=plain.moe_mlp(ff=128, experts=8, top=3, groups=(2, 2))),
    plain.attention_layer(heads=2, kv_heads=2, dim=128, vdim=96, conv=2, mlp=None),
    plain.attention_layer(heads=4, kv_heads=4, dim=32, vdim=32, conv=3, mlp=None),
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_sizes_of_a_larger_model(dtype, folders):
    """Heads of 64 (the tensor-core kernels for portions and for grouped heads), of 32 and 128 (the bulk-copy kernel), a
    prompt of several key tiles and splits, more experts' rows than a tile."""
    raw = plain.make_config(LARGER, width=128, vocab=96, side=32)
    folder, raw, tensors = folders("larger", raw, seed=3)
    toks = tokens_for(raw, 1300, 9)
    eng = make_engine(folder, dtype, num_blocks=256, max_step_tokens=2048)
    check_request(eng, raw, tensors, toks, [1300], dtype, "whole")
    check_request(eng, raw, tensors, toks, [590, 2, 9, 257, 400, 30] + [1] * 12, dtype, "portions")
    check_request(eng, raw, tensors, toks[:640], [598] + [1] * 42, dtype, "decoding")


# --- kernels with inputs made so that a fault shows ---------------------------------------------------

def _paged(rows, page_size, dtype, shuffle_seed=0):
    """Scatter each sequence's rows [len, G, d] over shuffled pages; unused slots hold NaN.  (pages [P, G, page, d], tables)."""
    G, d = rows[0].shape[1:]
    need = [-(-r.shape[0] // page_size) for r in rows]
    order = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(shuffle_seed)).tolist()
    pages = torch.full((sum(need) + 3, G, page_size, d), float("nan"), dtype=torch.float64)
    tables = torch.zeros(len(rows), max(need), dtype=torch.int32)
    for s, r in enumerate(rows):
        for i in range(need[s]):
            page = order.pop()
            tables[s, i] = page
            part = r[i * page_size: (i + 1) * page_size]
            pages[page, :, : part.shape[0]] = part.transpose(0, 1)
    return pages.to(dtype).cuda(), tables.cuda()


def _penalised(q, keys, values, where, scale, r1, r2, rep):
    """q [n, H, d]; keys[seq], values[seq] [len, G, d]; where[t] = (sequence, position)."""
    out = torch.zeros(q.shape[0], q.shape[1], values[0].shape[-1], dtype=torch.float64)
    for t, (seq, pos) in enumerate(where):
        dist = torch.arange(pos, -1, -1, dtype=torch.float64)
        for h in range(q.shape[1]):
            s = keys[seq][: pos + 1, h // rep] @ q[t, h] * scale - r1[h] * torch.log1p(r2[h] * dist)
            out[t, h] = torch.softmax(s, 0) @ values[seq][: pos + 1, h // rep]
    return out


PENALTY_CASES = [  # (heads, kv heads, head size, page)
    (4, 2, 64, 16), (8, 1, 64, 16), (2, 2, 64, 32), (6, 1, 32, 16), (4, 4, 128, 16), (3, 3, 24, 16), (2, 1, 40, 8), (4, 2, 80, 4), (12, 1, 64, 16),
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", PENALTY_CASES)
def test_distance_penalty_in_every_attention_kernel(case, dtype):
    """Each query looks for one key (far away, at a page's or a tile's border, position 0, its own), strongly enough that
    it and a rival near the query share the weight: a penalty that is left out, taken off another head's score or counted
    from another distance moves the result.  Portions and single tokens, every kernel that takes the sizes."""
    from edgerag_b200.ops import kernels as k

    H, G, d, page = case
    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(H * 100 + d)
    lens, new, scale = [150, 77, 700, 300], [40, 1, 260, 129], 0.5
    r1 = (0.2 + 2.0 * torch.rand(H, generator=g)).double()
    r2 = (0.05 + 0.5 * torch.rand(H, generator=g)).double()
    keys = [(torch.randn(n, G, d, generator=g, dtype=torch.float64) * 0.3).to(tdt).double() for n in lens]
    values = [torch.randn(n, G, d, generator=g, dtype=torch.float64).to(tdt).double() for n in lens]
    qs, where = [], []
    for s, n in enumerate(lens):
        for i, pos in enumerate(range(n - new[s], n)):
            target = max(0, min(pos, [0, pos, (pos // page) * page - 1, (pos // page) * page, pos - 128, 1, pos // 2, (pos // 128) * 128 - 1][i % 8]))
            rival = max(0, pos - 1 - i % 5)
            q = torch.randn(H, d, generator=g, dtype=torch.float64) * 0.2
            for h in range(H):
                far, near = keys[s][target, h // (H // G)], keys[s][rival, h // (H // G)]
                lift = float(r1[h] * math.log1p(float(r2[h]) * (pos - target)) - r1[h] * math.log1p(float(r2[h]) * (pos - rival)))
                q[h] += (8.0 + lift) / scale * far / far.norm() ** 2 + 8.0 / scale * near / near.norm() ** 2
            qs.append(q.to(tdt).double())
            where.append((s, pos))
    q = torch.stack(qs)
    want = _penalised(q, keys, values, where, scale, r1, r2, H // G)
    assert (want - _penalised(q, keys, values, where, scale, 0 * r1, r2, H // G)).abs().max() > 0.3, "the inputs do not show the penalty"
    assert (want - _penalised(q, keys, values, where, scale, r1.flip(0), r2, H // G)).abs().max() > 0.1 or H == 1
    k_pages, tables = _paged(keys, page, tdt, 1)
    v_pages, _ = _paged(values, page, tdt, 1)
    pen = torch.stack([r1, r2]).float().cuda()
    n = len(where)
    seq = torch.tensor([s for s, _ in where], dtype=torch.int32).cuda()
    pos = torch.tensor([p for _, p in where], dtype=torch.int32).cuda()
    starts = torch.tensor([0] + list(np.cumsum(new)), dtype=torch.int32).cuda()
    qd = q.reshape(n, H * d).to(tdt).cuda().contiguous()
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    tol = 3e-5 if dtype == "float32" else 4e-2
    out = torch.full((n, H * d), float("nan"), dtype=tdt, device="cuda")
    err = lambda o, w: float((o.double().cpu().view(w.shape) - w).abs().max())      # noqa: E731
    k.attention_rows(qd, k_pages, v_pages, tables, seq, pos, out, H, scale, penalty=pen)
    assert err(out, want) < tol, "rows"
    if k.prefill_tc_supported(tdt, d, 0, page):
        for ranges in (1, 3):
            out.fill_(float("nan"))
            need_o, need_ml = k.prefill_tc_scratch_floats(n, H, ranges)
            po = torch.empty(need_o, dtype=torch.float32, device="cuda")
            pm = torch.empty(need_ml, dtype=torch.float32, device="cuda")
            k.attention_prefill_tc(qd, k_pages, v_pages, tables, starts, pos, out, k.prefill_tc_blocks(new), H, scale, status,
                                   key_splits=ranges, part_o=po, part_ml=pm, penalty=pen)
            assert int(status) == 0 and err(out, want) < tol, f"portions on tensor cores, {ranges} ranges"
    # single tokens: every sequence's last token as a step of its own, keys in splits
    last = [int(starts[s + 1]) - 1 for s in range(len(lens))]
    q1, pos1 = qd[last].contiguous(), pos[last].contiguous()
    tok = torch.arange(len(lens), dtype=torch.int32).cuda()
    for split in (128, 512):
        n_splits = -(-max(lens) // split)
        acc, ml = k.decode_scratch_floats(len(lens), H, d, n_splits)
        acc = torch.full((acc,), float("nan"), dtype=torch.float32, device="cuda")
        ml = torch.full((ml,), float("nan"), dtype=torch.float32, device="cuda")
        o1 = torch.full((len(lens), H * d), float("nan"), dtype=tdt, device="cuda")
        k.attention_decode(q1, k_pages, v_pages, tables, tok, pos1, o1, H, scale, acc, ml, n_splits, split_keys=split, penalty=pen)
        assert err(o1, want[last]) < tol, f"single tokens, splits of {split}"
        if k.decode_bulk_supported(tdt, d, 0, H, G, n_splits):
            o1.fill_(float("nan"))
            k.attention_decode_bulk(q1, k_pages, v_pages, tables, tok, pos1, o1, H, scale, acc, ml, n_splits, status, split_keys=split, penalty=pen)
            assert int(status) == 0 and err(o1, want[last]) < tol, f"bulk copies, splits of {split}"
        if k.decode_gqa_supported(tdt, d, 0, H, G, page, split, n_splits):
            o1.fill_(float("nan"))
            k.attention_decode_gqa(q1, k_pages, v_pages, tables, tok, pos1, o1, H, scale, acc, ml, n_splits, status, split_keys=split, penalty=pen)
            assert int(status) == 0 and err(o1, want[last]) < tol, f"grouped heads, splits of {split}"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 1, 8, 3, 16), (3, 3, 16, 4, 8), (4, 2, 24, 2, 16), (2, 2, 8, 1, 4), (5, 1, 64, 5, 16), (2, 1, 8, 0, 16)])
def test_convolution_of_queries_keys_and_values_from_the_record(sizes, dtype):
    """Two requests in portions: the inputs before a portion come from the request's record (biased; zeros, not the bias,
    before the sequence's start), single tokens and portions move the record on, keys and values land in their slots."""
    from edgerag_b200.ops import kernels as k

    H, G, D, taps, page = sizes
    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(sum(sizes))
    C, qw, kw = (H + 2 * G) * D, H * D, G * D
    lens = {0: 23, 1: 9}
    proj = {s: torch.randn(n, C, generator=g, dtype=torch.float64).to(tdt).double() for s, n in lens.items()}
    bias = torch.randn(C, generator=g).float()
    weight = torch.randn(max(taps, 1), C, generator=g).float()
    want = {}
    for s in lens:
        u = proj[s] + bias.double()
        want[s] = plain.causal_conv(u, weight.double().T.contiguous()) if taps else u
    k_pages = torch.full((16, G, page, D), float("nan"), dtype=tdt, device="cuda")
    v_pages = torch.full((16, G, page, D), float("nan"), dtype=tdt, device="cuda")
    state = torch.zeros(4, taps - 1, C, dtype=torch.float32, device="cuda") if taps > 1 else None
    if state is not None:
        state[1].fill_(float("nan"))            # a slot nobody uses
    slot_of, page_of = {0: 3, 1: 0}, {0: [5, 1, 6, 2, 7, 0], 1: [4, 3, 9]}
    fed = {0: 0, 1: 0}
    tol = 1e-5 if dtype == "float32" else 6e-2
    # (single tokens come first in a step, as the runner orders them)
    for step in ([(0, 5), (1, 2)], [(1, 1), (0, 1)], [(0, 1), (1, 2)], [(1, 4), (0, 2)], [(0, 14)]):
        rows = torch.cat([proj[s][fed[s]: fed[s] + n] for s, n in step]).to(tdt).cuda().contiguous()
        total = rows.shape[0]
        seq_of = torch.tensor([i for i, (_, n) in enumerate(step) for _ in range(n)], dtype=torch.int32).cuda()
        starts = torch.tensor([0] + list(np.cumsum([n for _, n in step])), dtype=torch.int32).cuda()
        st_slots = torch.tensor([slot_of[s] for s, _ in step], dtype=torch.int32).cuda()
        slots = torch.tensor([page_of[s][p // page] * page + p % page for s, n in step for p in range(fed[s], fed[s] + n)],
                             dtype=torch.int32).cuda()
        q_out = torch.full((total, qw), float("nan"), dtype=tdt, device="cuda")
        k.qkv_conv(rows, q_out, H, G, D, taps=taps, bias=bias.cuda(), weight=weight.cuda() if taps else None, conv_state=state,
                   seq_of_token=seq_of, seq_starts=starts, state_slots=st_slots, n_seqs=len(step),
                   first_portion=sum(1 for _, n in step if n == 1), slots=slots, k_pages=k_pages, v_pages=v_pages, page_size=page)
        row = 0
        for s, n in step:
            assert (q_out[row: row + n].double().cpu() - want[s][fed[s]: fed[s] + n, :qw]).abs().max() < tol, (step, s)
            row += n
            fed[s] += n
            if state is not None:               # the record: the last taps - 1 biased inputs, zeros before the start
                u = torch.cat([torch.zeros(taps - 1, C, dtype=torch.float64), proj[s][: fed[s]] + bias.double()])[-(taps - 1):]
                assert torch.allclose(state[slot_of[s]].double().cpu(), u, atol=1e-6), (step, s)
    assert fed == lens
    for s, n in lens.items():
        for p in range(n):
            pg, off = page_of[s][p // page], p % page
            assert (k_pages[pg, :, off].double().cpu().flatten() - want[s][p, qw: qw + kw]).abs().max() < tol
            assert (v_pages[pg, :, off].double().cpu().flatten() - want[s][p, qw + kw:]).abs().max() < tol
    if state is not None:
        assert torch.isnan(state[1]).all(), "a record of another slot was written"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(12, 4, (4, 3), 64), (6, 2, (3, 2), 40), (8, 3, None, 96), (16, 1, (8, 1), 128), (5, 5, (5, 5), 24),
                                   (64, 6, (8, 4), 256), (9, 2, (3, 1), 33)])
def test_router_with_correction_and_gated_experts_on_both_product_paths(sizes, dtype):
    """Choices and weights against the plain router (rows without close calls), with corrections that make choice scores
    negative; gated experts with their weight on the output, on the general kernels and (bfloat16) the tensor cores."""
    from edgerag_b200.ops import kernels as k

    E, top, groups, width = sizes
    ff = 24
    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(E * 7 + top)
    router = {"experts": E, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    w_router = (torch.randn(E, width, generator=g) * 2.0 / math.sqrt(width)).float()
    corr = torch.where(torch.rand(E, generator=g) < 0.5, -2.0, -1.0) + 0.3 * torch.randn(E, generator=g)
    w_gu = (torch.randn(E, 2 * ff, width, generator=g) / math.sqrt(width)).to(tdt)
    w_down = (torch.randn(E, width, ff, generator=g) / math.sqrt(ff)).to(tdt)
    for n in (5, 16, 200):
        x = torch.randn(n, width, generator=g).to(tdt)
        s = torch.sigmoid(x.double() @ w_router.double().T)
        chosen = plain.routed_choice(x.double(), w_router, corr, router)
        picked = s.gather(1, chosen)
        weight = picked / (picked.sum(-1, keepdim=True) + 1e-20)
        c = s + corr.double()
        gap = lambda v: float((v.sort(descending=True).values[:-1] - v.sort(descending=True).values[1:]).min()) if v.numel() > 1 else 1.0   # noqa: E731
        clear = torch.ones(n, dtype=torch.bool)
        for t in range(n):
            clear[t] = gap(c[t]) > 1e-4
            if groups and clear[t]:
                clear[t] = gap(c[t].view(groups[0], -1).sort(-1, descending=True).values[:, :2].sum(-1)) > 1e-4
        assert int(clear.sum()) > n // 4
        lists = torch.zeros(k.moe_lists_ints(n, E, top), dtype=torch.int32, device="cuda")
        score = torch.zeros(n * top, dtype=torch.float32, device="cuda")
        tc = k.moe_tc_supported(tdt, width, ff)
        tile_rows = k.moe_tc_tile_rows(n, E, top) if tc else 0
        how = dict(groups=groups, correction=corr.float().cuda(), group_score="top2_sum", normalise=True)
        k.moe_route(x.cuda(), w_router.cuda(), top, lists, score, tile_rows, **how)
        got_c, got_s = lists[: n * top].reshape(n, top).cpu(), score.reshape(n, top).cpu()
        if k.moe_route_few(n, E, top, tdt):           # the kernels for few tokens: the same choices, weights and lists to the bit
            lists2, score2 = torch.zeros_like(lists), torch.zeros_like(score)
            k.moe_route(x.cuda(), w_router.cuda(), top, lists2, score2, tile_rows, logits=torch.empty(n, E, device="cuda"), **how)
            assert torch.equal(lists, lists2) and torch.equal(score, score2)
            for scores, gr in (("sigmoid", groups), ("softmax", groups)):
                k.moe_route(x.cuda(), w_router.cuda(), top, lists2, score2, tile_rows, scores=scores, groups=gr)
                l3, s3 = torch.zeros_like(lists), torch.zeros_like(score)
                k.moe_route(x.cuda(), w_router.cuda(), top, l3, s3, tile_rows, scores=scores, groups=gr, logits=torch.empty(n, E, device="cuda"))
                assert torch.equal(l3, lists2) and torch.equal(s3, score2), scores
        assert torch.equal(got_c[clear].long(), chosen[clear]), "choices"
        assert torch.allclose(got_s[clear].double(), weight[clear], rtol=2e-5, atol=1e-7), "weights: the scores without correction, over their sum"
        want = torch.zeros(n, width, dtype=torch.float64)          # the update from the engine's own choices
        for t in range(n):
            for j in range(top):
                e = int(got_c[t, j])
                both = x[t].double() @ w_gu[e].double().T
                a = plain.silu(both[:ff]) * both[ff:]
                if dtype == "bfloat16":
                    a = a.to(tdt).double()
                want[t] += float(got_s[t, j]) * (a @ w_down[e].double().T)
        act = torch.empty(n * top, ff, dtype=tdt, device="cuda")
        parts = torch.full((top, n, width), float("nan"), dtype=torch.float32, device="cuda")
        tol = (1e-5 if dtype == "float32" else 2e-2) * float(want.abs().max())
        if tc:
            xs = torch.empty(n * top, width, dtype=tdt, device="cuda")
            k.moe_tc_gather(x.cuda(), lists, None, E, top, xs)
            k.moe_tc_gate_up(xs, w_gu.cuda(), lists, top, tile_rows, act)
            k.moe_tc_down(act, w_down.cuda(), lists, top, tile_rows, parts, out_score=score)
            assert (parts.sum(0).double().cpu() - want).abs().max() < tol, "tensor cores"
            k.moe_route(x.cuda(), w_router.cuda(), top, lists, score, **how)
            parts.fill_(float("nan"))
        k.moe_gate_up(x.cuda(), w_gu.cuda(), lists, None, top, act)
        k.moe_down(act, w_down.cuda(), lists, top, parts, out_score=score)
        assert (parts.sum(0).double().cpu() - want).abs().max() < tol, "general kernels"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [32, 70, 512, 2048, 3000, 5000, 9000])
def test_stream_kernels_between_layers(width, dtype):
    """The sum of two updates, the side input's gate, and the average over depth with the norms on either side of it: every
    form of update, layer norm without and with bias, RMS norm, plain cast, a selection of rows."""
    from edgerag_b200.ops import kernels as k

    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(width)
    n, tol = 7, 2e-5 if dtype == "float32" else 2e-2
    rnd = lambda *s: torch.randn(*s, generator=g)                                   # noqa: E731
    hidden, a, parts = rnd(n, width), rnd(n, width).to(tdt), rnd(3, n, width)
    for b in (None, a, parts):
        for first in (a, parts):
            h, out = hidden.clone().cuda(), torch.empty(n, width, dtype=tdt, device="cuda")
            k.sum_updates(h, first.cuda(), None if b is None else b.cuda(), tdt, out=out)
            total = lambda u: u.double().sum(0) if u.dim() == 3 else u.double()      # noqa: E731
            want = hidden.double() + total(first) + (0 if b is None else total(b))
            assert (h.double().cpu() - want).abs().max() < 1e-5 and (out.double().cpu() - want).abs().max() < tol * want.abs().max()
    dim, vocab, pad = 5, 11, 8
    table, gate = rnd(vocab, 4 * dim).to(tdt), rnd(n, pad).to(tdt)
    ids = torch.tensor([3, 10, 0, 3, 7, 1, 9], dtype=torch.int32)
    act = torch.full((n, pad), float("nan"), dtype=tdt, device="cuda")
    k.side_gate(gate.cuda(), table.cuda(), ids.cuda(), 2 * dim, dim, act)
    want = plain.gelu_tanh(gate.double()[:, :dim]) * table.double()[ids.long(), 2 * dim: 3 * dim]
    assert (act[:, :dim].double().cpu() - want).abs().max() < tol * 3 and bool((act[:, dim:] == 0).all())
    w, bias, pw = 1 + 0.1 * rnd(width), 0.2 * rnd(width), 0.5 + 0.1 * rnd(width)
    for layer in (0, 4):
        hist = rnd(8, n, width)
        mix = rnd(layer + 2)
        for delta, post in ((None, None), (a, None), (a, (pw, 1e-5)), (parts, (pw, 1e-5))):
            d = 0.0 if delta is None else (delta.double().sum(0) if delta.dim() == 3 else delta.double())
            x = hidden.double() + (plain.rms_unit(d, 1e-5) * pw.double() if post else d)
            done = [hist[j].double() for j in range(layer + 1)] + [x]
            mean = plain.depth_average(done, mix)
            outs = {"layernorm": plain.layer_norm(mean, w.double(), 1e-5) + bias.double(), "rmsnorm": plain.rms_unit(mean, 1e-5) * w.double(), "cast": mean}
            for kind, norm_want in outs.items():
                if kind == "layernorm" and layer == 0:
                    norm_want = norm_want - bias.double()
                h, hs = hidden.clone().cuda(), hist.clone().cuda()
                out = torch.empty(n, width, dtype=tdt, device="cuda")
                how = dict(delta=None if delta is None else delta.cuda(), post=(pw.cuda(), 1e-5) if post else None, out_kind=kind,
                           weight=w.cuda() if kind != "cast" else None, bias=bias.cuda() if kind == "layernorm" and layer else None, eps=1e-5)
                k.depth_mix(h, hs, layer, mix.cuda(), tdt, out=out, **how)
                assert (h.double().cpu() - mean).abs().max() < 2e-5 and (hs[layer + 1].double().cpu() - x).abs().max() < 2e-5
                assert (out.double().cpu() - norm_want).abs().max() < tol * norm_want.abs().max(), (kind, layer)
                assert torch.equal(hs[: layer + 1].cpu(), hist[: layer + 1]) and torch.equal(hs[layer + 2:].cpu(), hist[layer + 2:])
                rows = torch.tensor([5, 0, 6], dtype=torch.int32).cuda()
                h, hs, few = hidden.clone().cuda(), hist.clone().cuda(), torch.empty(3, width, dtype=tdt, device="cuda")
                k.depth_mix(h, hs, layer, mix.cuda(), tdt, out=few, rows=rows, **how)
                assert torch.equal(few.cpu(), out[[5, 0, 6]].cpu()) and torch.equal(h.cpu(), hidden) and torch.equal(hs.cpu(), hist)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_norm_without_bias_and_entrywise_gate(dtype):
    from edgerag_b200.ops import kernels as k

    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    tol = 2e-5 if dtype == "float32" else 2e-2
    g = torch.Generator().manual_seed(4)
    for width in (24, 70, 1024):
        x, w = 3.0 + torch.randn(5, width, generator=g), 1 + 0.1 * torch.randn(width, generator=g)
        out = torch.empty(5, width, dtype=tdt, device="cuda")
        k.add_layernorm(x.cuda(), w.cuda(), None, out, 1e-5)
        assert (out.double().cpu() - plain.layer_norm(x.double(), w.double(), 1e-5)).abs().max() < tol * 4
        y, z = torch.randn(5, width, generator=g).to(tdt), torch.randn(5, 2 * width, generator=g).to(tdt)
        got = y.clone().cuda()
        k.sigmoid_gate(got, z.cuda()[:, width:])
        assert (got.double().cpu() - y.double() * torch.sigmoid(z.double()[:, width:])).abs().max() < tol * 3
        got = y.clone().cuda()
        k.sigmoid_gate(got, z.cuda()[:, 2: width + 2])                  # (a view that is not 16-byte aligned)
        assert (got.double().cpu() - y.double() * torch.sigmoid(z.double()[:, 2: width + 2])).abs().max() < tol * 3


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_rows_and_queries_turned_with_a_multiplier(dtype):
    """The cached row's rotated part and the queries' turned by stretched frequencies, cosines and sines times a constant."""
    from edgerag_b200.ops import kernels as k

    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(8)
    H, d, dr, R, n, page = 3, 4, 8, 24, 6, 4
    freq, mult = plain.yarn(300.0, dr, YARN)
    proj = torch.randn(n, R + dr, generator=g).to(tdt)
    q = torch.randn(n, H * (d + dr), generator=g).to(tdt)
    pos = torch.tensor([0, 1, 5, 63, 64, 1200], dtype=torch.int32)
    w = 1 + 0.1 * torch.randn(R, generator=g)
    pages = torch.zeros(2, 1, page, R + dr, dtype=tdt, device="cuda")
    slots = torch.arange(n, dtype=torch.int32).cuda()
    k.latent_store(proj.cuda(), pos.cuda(), 1e-5, off_kv=0, rank=R, rot_dim=dr, kv_weight=w.cuda(), inv_freq=freq.float().cuda(), rot_dims=dr,
                   slots=slots, pages=pages, rot_mult=mult)
    rows = pages.view(-1, R + dr)[:n].double().cpu()
    tol = 3e-4 if dtype == "float32" else 3e-2               # (position 1,200 times a float32 frequency)
    assert (rows[:, :R] - plain.rms_unit(proj.double()[:, :R], 1e-5) * w.double()).abs().max() < (1e-5 if dtype == "float32" else 3e-2)
    assert (rows[:, R:] - plain.rotate_pairs(proj.double()[:, R:], pos, freq, mult)).abs().max() < tol
    ql = torch.zeros(n, H, R + dr, dtype=torch.float32, device="cuda")
    k.latent_q_rotate(q.cuda(), pos.cuda(), freq.float().cuda(), H, d, dr, R, dr, ql, rot_mult=mult)
    want = plain.rotate_pairs(q.double().view(n, H, d + dr)[..., d:], pos, freq, mult)
    assert (ql[..., R:].double().cpu() - want).abs().max() < 3e-4


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_that_asks_for_far_keys_and_keeps_its_state(dtype, folders):
    """Weights made so that a lost or late key, state or record shows in the logits: queries scaled up and the penalty of
    one head turned down (it looks at the whole past), states that hardly decay, a strong last tap behind the current one."""
    def edit(t):
        for name in t:
            if name.endswith((".q", ".uq")):
                t[name] = (t[name].float() * 2.0).to(t[name].dtype)
            if name.endswith(".r1"):
                t[name][0] = 0.02
            if name.endswith(".A_log"):
                t[name] = torch.full_like(t[name], -6.0)
            if name.endswith(".conv") and t[name].shape[1] > 1:
                t[name][:, 0] = 1.5

    raw = plain.make_config([MAM, ATT, LAT, _reading(LAT, 2)], width=64, vocab=90)
    folder, raw, tensors = folders("far", raw, seed=5, edit=edit)
    toks = tokens_for(raw, 200, 3)
    other = list(toks)
    other[0] = (other[0] + 1) % raw["vocab"]
    a, b = plain.forward(tensors, raw, toks), plain.forward(tensors, raw, other)
    assert row_errors(b[-20:], a[-20:]).min() > 10 * BANDS["float32"][0], "the first token does not show at the end"
    eng = make_engine(folder, dtype)
    for rid, cuts in (("whole", [200]), ("decoded", [100] + [1] * 100), ("portions", [16, 16, 2, 30, 64, 1, 1, 2, 60, 8])):
        check_request(eng, raw, tensors, toks, cuts, dtype, rid)


@pytest.mark.gpu
def test_a_step_of_embeddings_is_refused(folders):
    from edgerag_b200.engine.step import StepEntry, StepError

    folder, raw, _ = folders("attention_dense", ALONE["attention_dense"], seed=11)
    eng = make_engine(folder, "float32")
    eng.runner.admit("x")
    with pytest.raises(StepError, match="ids"):
        eng.runner.step([StepEntry("x", embeds=torch.zeros(3, raw["width"]), want=[2])])


@pytest.mark.gpu
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(graphs, folders):
    from edgerag_b200 import SamplingParams
    from edgerag_b200.engine.engine import Engine, EngineOptions

    # (a small embedding: with the head tied to a large one, random weights would repeat the prompt's last token for ever)
    folder, raw, tensors = folders("small embedding", {**FULL, "embedding": {"scale": 0.1}}, seed=1)
    prompts = [tokens_for(raw, n, 40 + i) for i, n in enumerate((37, 5, 21))]
    eng = Engine.from_pretrained(folder, EngineOptions(dtype="float32", block_size=16, num_blocks=24, max_batch_size=2,
                                                       max_step_tokens=64, chunk_size=8, cuda_graphs=graphs))
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=12))
    for prompt, out in zip(prompts, outs):
        seq = list(prompt)
        for tok in out:                     # the engine's token is the plain argmax wherever the plain margin is clear
            logits = plain.forward(tensors, raw, seq)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) > 1e-3 * float(logits.abs().max()):
                assert tok == int(logits.argmax())
            seq.append(tok)
        assert len(out) == 12
    assert len({t for out in outs for t in out}) > 12


@pytest.mark.gpu
def test_trace_replay_program(folders, tmp_path):
    import helpers

    folder, raw, tensors = folders("full", FULL, seed=1)
    trace = helpers.Trace()
    for i, n in enumerate((70, 33, 90, 18, 47)):
        trace.sequences[f"r{i}"] = tokens_for(raw, n, 60 + i)
    helpers.cut_mixed(trace, list(trace.sequences), seed=3)
    cmd = [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path / "out"),
           "--max-tokens", str(trace.max_tokens), "--poison-freed-pages"]
    text = "".join(json.dumps(s) + "\n" for s in trace.steps)
    proc = subprocess.run(cmd, input=text, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [int(l.split()[1]) for l in proc.stdout.splitlines() if l.startswith("done ")] == [s["step"] for s in trace.steps]
    want = {rid: plain.forward(tensors, raw, seq) for rid, seq in trace.sequences.items()}
    got_rows, want_rows = [], []
    files = {}
    for step, row, rid, pos in trace.expect:
        if step not in files:
            files[step] = np.fromfile(tmp_path / "out" / f"{step}.f32", dtype="<f4").reshape(-1, raw["vocab"])
        got_rows.append(torch.from_numpy(files[step][row].copy()))
        want_rows.append(want[rid][pos])
    assert_close(torch.stack(got_rows), torch.stack(want_rows), "float32", "trace")


@pytest.mark.gpu
def test_serving_from_a_saved_model_in_bfloat16(folders):
    folder, raw, tensors = folders("full", FULL, seed=1)
    from edgerag_b200 import Engine, SamplingParams

    eng = Engine.from_pretrained(folder, dtype="bfloat16", block_size=16, num_blocks=16)
    out = eng.generate([tokens_for(raw, 9, 77)], SamplingParams(max_new_tokens=5))[0]
    assert len(out) == 5 and all(0 <= t < raw["vocab"] for t in out)
