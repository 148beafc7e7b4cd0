"""Kikarax through the engine against the plain implementation of ``plain_kikarax``.

Small configurations with random weights of their own: head counts, key and value sizes, chunk sizes, caps, bounds, expert counts and
choices, buckets and multipliers that differ from layer to layer and from test to test (also the degenerate ones: one kv head, as
many as heads, one expert chosen, all experts chosen, one bucket, no cap, no mask, no blended values, no shared expert, no
positions, a layer without a feed-forward, constants of 1).  Every mechanism alone; whole prompts against token-by-token decoding
and portions down to two tokens; unequal requests in one batch with pages and slots that are freed, poisoned and used again; keys
made dominant just inside and just outside a chunk, at page borders, at position 0 and at their own, with scores below and far
above the cap; pairs of tokens across a portion's edge; the first tokens; long decoding; greedy generation through
``Engine.generate`` and the scheduler; the trace replay program; the command line.

In bfloat16 a router's close call may fall the other way than in the plain float64 implementation, which changes a token's experts,
not the arithmetic under test.  So the bfloat16 comparisons hand the plain implementation the experts that the engine chose;
float32 comparisons use the plain router.
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

import plain_kikarax as plain
from test_sabolorn import ChoiceLog, _paged, assert_close, feed, row_errors, tokens_for

ROOT = Path(__file__).resolve().parent.parent

DENSE = plain.attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, size=20, scale=0.3, softcap=5.0, mlp=plain.dense_mlp(48, 0.9))
EXPERTS = plain.attention_layer(heads=6, kv_heads=2, dim=24, vdim=24, size=13, scale=0.17, softcap=9.0, mlp=plain.moe_mlp(ff=24, experts=7, top=3, scale=1.3, shared=40))
ODD = plain.attention_layer(heads=5, kv_heads=1, dim=12, vdim=20, size=33, scale=0.4, softcap=3.0, v_mix=False, mlp=plain.moe_mlp(ff=16, experts=4, top=1, scale=2.5, shared=24))
BARE = plain.attention_layer(heads=3, kv_heads=3, dim=20, vdim=12, size=None, scale=0.25, softcap=None, v_mix=False, mlp=None)


def _sized(layer: dict, **mixer) -> dict:
    out = copy.deepcopy(layer)
    out["mixer"].update(mixer)
    return out


FULL = plain.make_config([_sized(ODD), DENSE, _sized(EXPERTS, vdim=24), BARE, _sized(DENSE, heads=2, dim=40, mask={"size": 32}),
                          _sized(EXPERTS, heads=4, dim=8, mask={"size": 7}, softcap=2.0)],
                         width=80, vocab=203, eps=1e-5, scale=3.5, buckets=89, mul_prev=17, mul_cur=5, positions=700, logit_scale=0.6)

ALONE = {
    "dense_bounded": plain.make_config([DENSE]),
    "experts_with_shared": plain.make_config([EXPERTS], width=72),
    "one_expert_of_four_one_kv_head": plain.make_config([ODD], width=56, logit_scale=1.0),
    "no_mask_no_cap_no_ffn_all_kv_heads": plain.make_config([BARE], width=40, scale=1.0),
    "all_experts_chosen_no_shared_weight_one": plain.make_config([_sized(EXPERTS) | {"mlp": plain.moe_mlp(ff=16, experts=3, top=3, scale=1.0, shared=None)}]),
    "values_blended_over_three_layers": plain.make_config([_sized(DENSE), _sized(DENSE, heads=2, dim=32), _sized(DENSE, v_mix=False), _sized(DENSE, softcap=1.0)]),
    "heads_of_64": plain.make_config([plain.attention_layer(heads=4, kv_heads=1, dim=64, size=48, softcap=4.0, mlp=None)], width=64),
    "one_bucket": plain.make_config([DENSE], buckets=1),
    "no_pairs": plain.make_config([DENSE], buckets=0),
    "no_positions": plain.make_config([DENSE], positions=0),
    "table_alone": plain.make_config([DENSE], buckets=0, positions=0, scale=1.0),
    "large_multipliers": plain.make_config([DENSE], buckets=1009, mul_prev=2_000_000_011, mul_cur=1_999_999_973),
    "rows_of_50_entries": plain.make_config([DENSE, ODD], width=50, vocab=61),
    "chunks_of_one_key": plain.make_config([_sized(DENSE, mask={"size": 1})]),
}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from edgerag_b200.weights.safetensors_io import write_safetensors

    base = tmp_path_factory.mktemp("kikarax")
    made = {}

    def get(name: str, raw: dict, seed: int = 0, edit=None):
        if name not in made:
            folder = base / name.replace(" ", "_")
            folder.mkdir()
            tensors = plain.random_weights(raw, seed)
            if edit is not None:
                edit(tensors)
            (folder / "config.json").write_text(json.dumps(raw))
            write_safetensors(folder / "model.safetensors", tensors)
            made[name] = (folder, raw, tensors)
        return made[name]

    return get


def make_engine(folder, dtype, **over):
    from edgerag_b200.engine.engine import Engine, EngineOptions

    opts = dict(dtype=dtype, block_size=16, num_blocks=64, max_batch_size=4, max_step_tokens=512, max_model_len=1 << 20,
                cuda_graphs=False, poison_freed_pages=True)
    opts.update(over)
    eng = Engine.from_pretrained(folder, EngineOptions(**opts))
    eng.log = ChoiceLog(eng.model)
    return eng


def check_request(eng, raw, tensors, toks, cuts, dtype, what):
    eng.runner.admit(what)
    got, chosen = feed(eng.runner, what, toks, cuts, eng.log if dtype == "bfloat16" else None)
    eng.runner.release(what)
    assert_close(got, plain.forward(raw, tensors, toks, chosen=chosen), dtype, what)
    eng.cache.check_invariants()


# --- configuration, plan, plain mechanisms (CPU) ---------------------------------------------------

def _model(raw, dtype=torch.float32):
    from edgerag_b200.config.registry import architecture_of
    from edgerag_b200.models.decoder import DecoderModel

    arch = architecture_of(raw)
    return DecoderModel(arch.make_plan(arch.read_config(raw, "test")), dtype, torch.device("cpu"))


@pytest.mark.parametrize("name", ["full", *sorted(ALONE)])
def test_plan_names_every_tensor(name):
    raw = FULL if name == "full" else ALONE[name]
    model = _model(raw)
    specs = {s.name: tuple(s.shape) for s in model.weight_specs()}
    assert specs.pop("head") == (raw["vocab"], raw["width"])              # tied to the embedding where absent
    assert specs == plain.tensor_shapes(raw)
    assert model.graph_safe and model.max_positions == raw.get("max_positions")
    assert model.needs_token_ids == bool(raw["embedding"].get("bigram"))


def test_plan_declares_pages_by_chunk_and_the_record_of_the_last_token():
    model = _model(FULL)
    groups = {(g.n_kv_heads, g.head_dim, g.chunk): g.n_layers for g in model.cache_layout.groups}
    # (heads padded to one size for keys and values; layers of one geometry and chunk share pages)
    assert groups == {(1, 24, 33): 1, (2, 24, 20): 1, (2, 24, 13): 1, (3, 24, 0): 1, (2, 40, 32): 1, (2, 24, 7): 1}
    assert [(s.name, tuple(s.shape), s.dtype, s.fillers) for s in model.cache_layout.states] == [("last_id@embedding", (1,), "int32", True)]
    assert [b.mixer.value_mix for b in model.blocks] == [None, "first", "blend", None, "blend", "blend"]
    assert [b.mixer.softcap for b in model.blocks] == [3.0, 5.0, 9.0, 0.0, 5.0, 2.0]
    assert model.head.scale == 0.6 and model.embedding.scale == 3.5


def test_configuration_errors_name_the_key():
    from edgerag_b200.config.model_config import ConfigError
    from edgerag_b200.models.kikarax import KikaraxConfig

    def broken(change):
        raw = copy.deepcopy(plain.make_config([DENSE, _sized(EXPERTS)]))
        change(raw)
        return raw

    KikaraxConfig.from_dict(broken(lambda r: None), "t")
    cases = [
        (lambda r: r["layers"][0].update(type="delta"), "unknown layer type"),
        (lambda r: r["layers"][0]["mixer"].pop("kv_heads"), "kv_heads"),
        (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "kv_heads must divide"),
        (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
        (lambda r: r["layers"][0]["mixer"].update(softcap=0), "softcap"),
        (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "size"),
        (lambda r: r["layers"][1]["mixer"].update(vdim=8), "v_mix"),
        (lambda r: r["layers"][1]["mixer"].update(kv_heads=1), "v_mix"),
        (lambda r: r["layers"][0]["mlp"].update(kind="glu"), "mlp.kind"),
        (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
        (lambda r: r["layers"][1]["mlp"]["router"].update(top=9), "router.top"),
        (lambda r: r["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
        (lambda r: r["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
        (lambda r: r["embedding"]["bigram"].pop("mul_prev"), "mul_prev"),
        (lambda r: r["embedding"]["bigram"].update(mul_cur=-1), "multipliers"),
        (lambda r: r["embedding"]["bigram"].update(buckets=0), "buckets"),
        (lambda r: r.update(max_positions=0), "max_positions"),
        (lambda r: r.pop("norm"), "norm"),
        (lambda r: r.pop("width"), "width"),
    ]
    for change, word in cases:
        with pytest.raises(ConfigError, match=word):
            KikaraxConfig.from_dict(broken(change), "t")


def test_attention_refuses_options_that_do_not_go_together():
    from edgerag_b200.parts.base import PartSpec, build_part

    def build(**over):
        params = dict(hidden=32, n_q_heads=2, n_kv_heads=1, head_dim=16, position=PartSpec("none"))
        return build_part("mixer", PartSpec("attention", {**params, **over}), torch.float32, torch.device("cpu"))

    build(softcap=3.0, gate="g", value_mix="blend")
    for bad in (dict(softcap=3.0, penalty=("a", "b")), dict(softcap=-1.0), dict(value_mix="last"), dict(value_mix="blend", own_kv=False),
                dict(gate="g", qkv_bias=True), dict(value_mix="first", conv=3)):
        with pytest.raises(ValueError, match="attention"):
            build(**bad)


def test_plain_mechanisms_by_hand():
    ids = torch.tensor([4, 2, 9, 9])
    assert plain.bigram_rows(ids, {"buckets": 10, "mul_prev": 3, "mul_cur": 1}).tolist() == [10, 4, 5, 6]
    assert plain.soft_cap(torch.tensor([2.0], dtype=torch.float64), 4.0).item() == pytest.approx(4.0 * math.tanh(0.5))
    assert plain.soft_cap(torch.tensor([2.0]), 0.0).item() == 2.0
    m = plain.chunk_mask(7, 3)
    assert m.int().tolist() == [[1, 0, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0, 0], [0, 0, 0, 1, 0, 0, 0],
                                [0, 0, 0, 1, 1, 0, 0], [0, 0, 0, 1, 1, 1, 0], [0, 0, 0, 0, 0, 0, 1]]
    assert plain.blend_values(torch.tensor(1.0), torch.tensor(5.0), torch.tensor(0.25)).item() == 2.0
    # one token, width 1: the gate branch is cut at 2 from above only, the up branch at -2 as well
    one = lambda v: torch.tensor([[v]], dtype=torch.float64)      # noqa: E731
    t = {"gate": one(1.0), "up": one(-1.0), "down": one(1.0)}
    f = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)     # noqa: E731
    assert plain.dense_ff(one(5.0), {"limit": 2.0}, t, "").item() == pytest.approx(f(2.0, -2.0))
    assert plain.dense_ff(one(-3.0), {"limit": 2.0}, t, "").item() == pytest.approx(f(-3.0, 2.0))
    eye = torch.eye(3, dtype=torch.float64)
    idx, w = plain.routed_choice(torch.tensor([[0.0, 2.0, 1.0]], dtype=torch.float64), {"router": eye}, "", {"top": 2, "scale": 3.0})
    z = 1 + math.e + math.e ** 2
    assert idx.tolist() == [[1, 2]] and w[0].tolist() == pytest.approx([3 * math.e ** 2 / z, 3 * math.e / z])


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
    """The embedding and the stream after every layer (float32)."""
    from edgerag_b200.engine.step import StepEntry
    from edgerag_b200.parts.base import settle_update

    folder, raw, tensors = folders("full", FULL, seed=1)
    toks = tokens_for(raw, 50, 2)
    _, want = plain.forward(raw, tensors, toks, return_layers=True)
    eng = make_engine(folder, "float32")
    r, model = eng.runner, eng.model
    r.admit("x")
    r.pools.zero_slots(r.cache.drain_new_slots())
    ctx, ordered = r.prepare([StepEntry("x", tokens=toks, want=[])])
    hidden = ctx.buf("model.hidden", (len(toks), model.hidden_size), torch.float32)
    model.embedding.forward(ctx, hidden)
    x0 = plain.embed(raw, tensors, torch.tensor(toks))
    assert (hidden.cpu().double() - x0).abs().max() < 1e-5
    assert int(r.pools.states["last_id@embedding"][eng.cache.requests["x"].slot]) == toks[-1]
    delta = None
    for i, call in enumerate(model.schedule):
        delta = model.blocks[call.layer].forward(hidden, delta, ctx, call)
        settle_update(hidden, delta, model.dtype)
        delta = None
        err = (hidden.cpu().double() - want[i]).abs().max() / want[i].abs().max()
        assert err < 2e-5, f"layer {i}: {err:.2e}"
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
    """Portions of some requests beside single tokens of others; a request pauses for a step; requests end and their pages and
    state slots go to new ones (four slots, six requests, freed pages poisoned; a chunk's pages go back while its request
    lives).  Steps with three single tokens also run filler rows, which must leave the records of live slots alone."""
    from edgerag_b200.engine.step import StepEntry, _fill_to

    folder, raw, tensors = folders("full", FULL, seed=1)
    lens = {"a": 71, "b": 35, "c": 1, "d": 91, "e": 19, "f": 47}
    toks = {k: tokens_for(raw, n, 20 + i) for i, (k, n) in enumerate(lens.items())}
    eng = make_engine(folder, dtype, num_blocks=14)       # 224 tokens of pages: never room for all at once
    r = eng.runner
    plan = [
        [("a", 30), ("b", 2)], [("a", 1), ("b", 16), ("c", 1)], [("a", 17), ("b", 1)], [("b", 14), ("d", 40), ("a", 1)],
        [("a", 1), ("b", 1), ("d", 1)], [("a", 21), ("b", 1), ("d", 1)], [("d", 33), ("e", 2)], [("d", 15), ("e", 1), ("f", 2)],
        [("d", 1), ("e", 1), ("f", 1)], [("e", 15), ("f", 1)], [("f", 43)],
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
        singles = sum(1 for _, n in step if n == 1)
        first_row, row = {}, 0                      # the runner puts single tokens first, then fillers: every entry's rows in the step
        for i, (rid, n) in enumerate(sorted(step, key=lambda e: e[1] != 1)):
            if i == singles and singles:
                row += _fill_to(singles) - singles
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
        assert_close(torch.cat(got[rid]), plain.forward(raw, tensors, toks[rid], chosen=chosen), dtype, f"request {rid}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_in_the_pages_of_a_chunk(dtype, folders):
    """260 tokens one by one where the pool could not hold them all: the pages of earlier chunks are used again."""
    raw = plain.make_config([DENSE, _sized(EXPERTS, vdim=24, mask={"size": 20}), _sized(DENSE, heads=8, softcap=1.5)], width=64)
    folder, raw, tensors = folders("chunked only", raw, seed=2)
    toks = tokens_for(raw, 260, 9)
    eng = make_engine(folder, dtype, num_blocks=4)
    assert len(eng.cache.layout.groups) == 1
    check_request(eng, raw, tensors, toks, [3] + [1] * 257, dtype, "260 tokens, 257 of them one by one")
    check_request(eng, raw, tensors, toks, [19, 21, 20, 2, 18, 40] + [20] * 7, dtype, "portions that end at, before and behind a chunk's end")


LARGER = [
    plain.attention_layer(heads=8, kv_heads=2, dim=64, size=300, scale=0.125, softcap=6.0, mlp=plain.dense_mlp(256, 2.5)),
    plain.attention_layer(heads=8, kv_heads=2, dim=64, size=520, scale=0.2, softcap=2.5, mlp=plain.moe_mlp(ff=64, experts=8, top=2, scale=1.5, shared=128)),
    plain.attention_layer(heads=2, kv_heads=2, dim=128, vdim=96, size=700, scale=0.1, v_mix=False, mlp=plain.dense_mlp(96)),
    plain.attention_layer(heads=4, kv_heads=4, dim=32, size=64, scale=0.2, v_mix=False, mlp=None),
    plain.attention_layer(heads=2, kv_heads=2, dim=32, vdim=64, size=128, scale=0.2, softcap=30.0, mlp=plain.moe_mlp(ff=128, experts=16, top=5, scale=0.8)),
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_sizes_of_a_larger_model(dtype, folders):
    """Heads of 64 (the tensor-core kernels for portions and for grouped heads), of 32 and 128 (the bulk-copy kernel), a
    prompt of several key tiles and splits, more experts' rows than a tile."""
    folder, raw, tensors = folders("larger", plain.make_config(LARGER, width=128, vocab=96), seed=3)
    toks = tokens_for(raw, 1300, 9)
    eng = make_engine(folder, dtype, num_blocks=256, max_step_tokens=2048)
    check_request(eng, raw, tensors, toks, [1300], dtype, "whole")
    check_request(eng, raw, tensors, toks, [590, 2, 9, 257, 400, 30] + [1] * 12, dtype, "portions")
    check_request(eng, raw, tensors, toks[:640], [588] + [1] * 52, dtype, "decoding over two chunks' ends")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_that_asks_for_far_keys(dtype, folders):
    """Queries and keys scaled up: single keys decide rows, also just inside a chunk's first position.  The test's own sharpness:
    with chunks one longer or one shorter the plain model differs clearly, and the first token shows in its whole chunk."""
    raw = plain.make_config([_sized(DENSE, softcap=40.0, mask={"size": 37}), _sized(DENSE, softcap=60.0, mask={"size": 37}, heads=2)], width=64, vocab=90)

    def edit(t):
        for name in t:
            if name.endswith(("q.norm", "k.norm")):
                t[name] = (t[name].float() * 3.0).to(t[name].dtype)

    folder, raw, tensors = folders("far", raw, seed=5, edit=edit)
    toks = tokens_for(raw, 200, 3)
    want = plain.forward(raw, tensors, toks)
    for other in (36, 38):
        blind = copy.deepcopy(raw)
        for layer in blind["layers"]:
            layer["mixer"]["mask"]["size"] = other
        assert row_errors(plain.forward(blind, tensors, toks)[40:], want[40:]).max() > 0.3
    eng = make_engine(folder, dtype)
    for rid, cuts in (("whole", [200]), ("decoded", [100] + [1] * 100), ("portions", [16, 16, 2, 30, 10, 1, 1, 35, 37, 2, 50])):
        check_request(eng, raw, tensors, toks, cuts, dtype, rid)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_token_before_a_portion_decides_its_first_row(dtype, folders):
    """A bigram table that outweighs the rest; the sequence's very first token, a slot that another request has used, and a request
    that waits while others use the batch."""
    from edgerag_b200.engine.step import StepEntry

    raw = plain.make_config([DENSE], width=48, vocab=70, scale=0.2)

    def edit(t):
        t["bigram"] = (t["bigram"].float() * 6.0).to(torch.bfloat16)

    folder, raw, tensors = folders("bigram", raw, seed=8, edit=edit)
    a, b, c = (tokens_for(raw, n, 70 + n) for n in (21, 17, 12))
    wrong = [(a[0] + 1) % 70] + a[1:]
    assert row_errors(plain.forward(raw, tensors, wrong)[1:2], plain.forward(raw, tensors, a)[1:2]).max() > 0.5
    eng = make_engine(folder, dtype, max_batch_size=2, pad_decodes=True)
    r = eng.runner
    rows = {"a": [], "b": [], "c": []}
    seqs, fed = {"a": a, "b": b, "c": c}, {"a": 0, "b": 0, "c": 0}
    for step in ([("a", 4)], [("b", 1), ("a", 2)], [("b", 1)], [("b", 3), ("a", 1)], [("a", 1), ("b", 1)], [("b", 11), ("a", 13)],
                 [("c", 1)], [("c", 1)], [("c", 2)], [("c", 8)]):
        for rid, _ in step:
            if fed[rid] == 0:
                r.admit(rid)
        out = r.step([StepEntry(rid, tokens=seqs[rid][fed[rid]: fed[rid] + n], want=list(range(n))) for rid, n in step]).float().cpu()
        at = 0
        for rid, n in step:
            rows[rid].append(out[at: at + n].clone())
            at, fed[rid] = at + n, fed[rid] + n
            if fed[rid] == len(seqs[rid]):
                r.release(rid)
    for rid in rows:
        assert_close(torch.cat(rows[rid]), plain.forward(raw, tensors, seqs[rid]), dtype, rid)


@pytest.mark.gpu
def test_steps_that_the_model_cannot_run_are_refused(folders):
    from edgerag_b200.engine.step import StepEntry, StepError

    folder, raw, tensors = folders("short", plain.make_config([DENSE], positions=20), seed=11)
    eng = make_engine(folder, "float32")
    assert eng.max_model_len == 20
    r = eng.runner
    r.admit("x")
    with pytest.raises(StepError, match="ids"):
        r.step([StepEntry("x", embeds=torch.zeros(3, raw["width"]), want=[2])])
    toks = tokens_for(raw, 21, 4)
    with pytest.raises(StepError, match="position"):
        r.step([StepEntry("x", tokens=toks, want=[2])])
    got = torch.cat([r.step([StepEntry("x", tokens=toks[:19], want=list(range(19)))]).cpu().clone(),
                     r.step([StepEntry("x", tokens=toks[19:20], want=[0])]).cpu()])
    assert_close(got, plain.forward(raw, tensors, toks[:20]), "float32", "up to the last position")
    with pytest.raises(StepError, match="position"):
        r.step([StepEntry("x", tokens=toks[20:], want=[0])])
    eng.cache.check_invariants()


@pytest.mark.gpu
def test_rows_of_embeddings_beside_positions(folders):
    """Without pairs of tokens, rows of embeddings may stand in for the table's: scaled as they are, the position's row added."""
    from edgerag_b200.engine.step import StepEntry

    folder, raw, tensors = folders("no_pairs", ALONE["no_pairs"], seed=11)
    toks = tokens_for(raw, 30, 4)
    eng = make_engine(folder, "float32")
    eng.runner.admit("x")
    rows = tensors["embed"][torch.tensor(toks)].float().cuda()
    got = torch.cat([eng.runner.step([StepEntry("x", embeds=rows[:13], want=list(range(13)))]).cpu().clone(),
                     eng.runner.step([StepEntry("x", tokens=toks[13:], want=list(range(17)))]).cpu()])
    assert_close(got, plain.forward(raw, tensors, toks), "float32", "embeddings, then ids")


# --- kernels with inputs made so that a fault shows ---------------------------------------------------

def _capped(q, keys, values, where, scale, cap, chunk, rep, gate):
    """q, gate [n, H, d]; keys[seq], values[seq] [len, G, d]; where[t] = (sequence, position)."""
    out = torch.zeros(q.shape[0], q.shape[1], values[0].shape[-1], dtype=torch.float64)
    for t, (seq, pos) in enumerate(where):
        lo = pos - pos % chunk if chunk else 0
        for h in range(q.shape[1]):
            s = plain.soft_cap(keys[seq][lo: pos + 1, h // rep] @ q[t, h] * scale, cap)
            out[t, h] = torch.softmax(s, 0) @ values[seq][lo: pos + 1, h // rep]
    return out if gate is None else out * torch.sigmoid(gate)


CAP_CASES = [  # (heads, kv heads, head size, page, chunk)
    (4, 2, 64, 16, 96), (8, 1, 64, 16, 0), (2, 2, 64, 32, 130), (6, 1, 32, 16, 50), (4, 4, 128, 16, 64), (3, 3, 24, 16, 0),
    (2, 1, 40, 8, 33), (4, 2, 80, 4, 0), (12, 1, 64, 16, 257),
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("strong", [False, True], ids=["below the cap", "above the cap"])
@pytest.mark.parametrize("case", CAP_CASES)
def test_capped_scores_and_output_gate_in_every_attention_kernel(case, strong, dtype):
    """Each query looks for one key: its chunk's first position, a page's or a tile's border, position 0, its own.  Weak scores
    stay below the cap; strong ones lie several caps out, where the cap decides how much of the weight the one key gets."""
    from edgerag_b200.ops import kernels as k

    H, G, d, page, chunk = case
    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(H * 100 + d + strong)
    lens, new, scale = [150, 77, 700, 300], [40, 1, 260, 129], 0.5
    cap, want_score = (4.0, 14.0) if strong else (12.0, 7.0)
    keys = [(torch.randn(n, G, d, generator=g, dtype=torch.float64) * 0.3).to(tdt).double() for n in lens]
    values = [torch.randn(n, G, d, generator=g, dtype=torch.float64).to(tdt).double() for n in lens]
    qs, where = [], []
    for s, n in enumerate(lens):
        for i, pos in enumerate(range(n - new[s], n)):
            lo = pos - pos % chunk if chunk else 0
            target = [lo, pos, (pos // page) * page - 1, (pos // page) * page, pos - 128, lo + 1, (lo + pos) // 2, (pos // 128) * 128 - 1][i % 8]
            target = max(lo, min(pos, target))
            q = torch.randn(H, d, generator=g, dtype=torch.float64) * 0.2
            for h in range(H):
                key = keys[s][target, h // (H // G)]
                q[h] += want_score / scale * key / key.norm() ** 2
            qs.append(q.to(tdt).double())
            where.append((s, pos))
    q, n = torch.stack(qs), len(where)
    gate_all = torch.randn(n, H * d + 24, generator=g).to(tdt)          # the gate's columns lie inside wider rows
    gate = gate_all[:, 16: 16 + H * d].double().view(n, H, d)
    want = _capped(q, keys, values, where, scale, cap, chunk, H // G, gate)
    assert (want - _capped(q, keys, values, where, scale, 0.0, chunk, H // G, gate)).abs().max() > 0.1, "the inputs do not show the cap"
    if chunk:
        assert (want - _capped(q, keys, values, where, scale, cap, chunk + 1, H // G, gate)).abs().max() > 0.2, "nor the chunk"
    k_pages, tables = _paged(keys, page, tdt, 1)
    v_pages, _ = _paged(values, page, tdt, 1)
    seq = torch.tensor([s for s, _ in where], dtype=torch.int32).cuda()
    pos = torch.tensor([p for _, p in where], dtype=torch.int32).cuda()
    starts = torch.tensor([0] + list(np.cumsum(new)), dtype=torch.int32).cuda()
    qd = q.reshape(n, H * d).to(tdt).cuda().contiguous()
    gates = gate_all.cuda()[:, 16: 16 + H * d]
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    tol = 3e-5 if dtype == "float32" else 4e-2
    out = torch.full((n, H * d), float("nan"), dtype=tdt, device="cuda")
    err = lambda o, w: float((o.double().cpu().view(w.shape) - w).abs().max())      # noqa: E731
    how = dict(softcap=cap, chunk=chunk, gate=gates)
    k.attention_rows(qd, k_pages, v_pages, tables, seq, pos, out, H, scale, **how)
    assert err(out, want) < tol, "rows"
    ungated = _capped(q, keys, values, where, scale, cap, chunk, H // G, None)
    k.attention_rows(qd, k_pages, v_pages, tables, seq, pos, out, H, scale, softcap=cap, chunk=chunk)
    assert err(out, ungated) < tol, "rows without a gate"
    if k.prefill_tc_supported(tdt, d, 0, page):
        for ranges in (1, 3):
            need_o, need_ml = k.prefill_tc_scratch_floats(n, H, ranges)
            po = torch.empty(need_o, dtype=torch.float32, device="cuda")
            pm = torch.empty(need_ml, dtype=torch.float32, device="cuda")
            for gt, ref in ((gates, want), (None, ungated)):
                out.fill_(float("nan"))
                k.attention_prefill_tc(qd, k_pages, v_pages, tables, starts, pos, out, k.prefill_tc_blocks(new), H, scale, status,
                                       key_splits=ranges, part_o=po, part_ml=pm, softcap=cap, chunk=chunk, gate=gt)
                assert int(status) == 0 and err(out, ref) < tol, f"portions on tensor cores, {ranges} ranges"
    # single tokens: every sequence's last token as a step of its own, keys in splits
    last = [int(starts[s + 1]) - 1 for s in range(len(lens))]
    q1, pos1, g1 = qd[last].contiguous(), pos[last].contiguous(), gate_all.cuda()[last][:, 16: 16 + H * d]
    tok = torch.arange(len(lens), dtype=torch.int32).cuda()
    for split in (128, 512):
        n_splits = min(-(-max(lens) // split), (chunk or 10 ** 9) // split + 2)
        acc, ml = k.decode_scratch_floats(len(lens), H, d, n_splits)
        acc = torch.full((acc,), float("nan"), dtype=torch.float32, device="cuda")
        ml = torch.full((ml,), float("nan"), dtype=torch.float32, device="cuda")
        o1 = torch.full((len(lens), H * d), float("nan"), dtype=tdt, device="cuda")
        how = dict(split_keys=split, softcap=cap, chunk=chunk, gate=g1)
        k.attention_decode(q1, k_pages, v_pages, tables, tok, pos1, o1, H, scale, acc, ml, n_splits, **how)
        assert err(o1, want[last]) < tol, f"single tokens, splits of {split}"
        if k.decode_bulk_supported(tdt, d, 0, H, G, n_splits):
            o1.fill_(float("nan"))
            k.attention_decode_bulk(q1, k_pages, v_pages, tables, tok, pos1, o1, H, scale, acc, ml, n_splits, status, **how)
            assert int(status) == 0 and err(o1, want[last]) < tol, f"bulk copies, splits of {split}"
        if k.decode_gqa_supported(tdt, d, 0, H, G, page, split, n_splits):
            o1.fill_(float("nan"))
            k.attention_decode_gqa(q1, k_pages, v_pages, tables, tok, pos1, o1, H, scale, acc, ml, n_splits, status, **how)
            assert int(status) == 0 and err(o1, want[last]) < tol, f"grouped heads, splits of {split}"


@pytest.mark.gpu
def test_a_cap_and_a_penalty_exclude_each_other():
    from edgerag_b200.ops import kernels as k

    q = torch.zeros(1, 64, device="cuda")
    pages = torch.zeros(1, 1, 16, 64, device="cuda")
    zero = torch.zeros(1, dtype=torch.int32, device="cuda")
    with pytest.raises(k.KernelError, match="exclude"):
        k.attention_rows(q, pages, pages, zero.view(1, 1), zero, zero, torch.empty_like(q), 1, 0.5, softcap=2.0, penalty=torch.ones(2, 1, device="cuda"))


@pytest.mark.gpu
def test_polynomial_and_exact_cap_meet():
    """One tile of keys whose scores run through the place where the tensor-core kernel changes from the polynomial to the exact form:
    the weights on either side agree with the plain ones to 16-bit rounding."""
    from edgerag_b200.ops import kernels as k

    d, n = 64, 128
    cap = 3.0
    keys = torch.zeros(n, 1, d, dtype=torch.float64)
    for top in (0.98, 1.0, 1.02, 4.0):
        keys[:, 0, 0] = torch.linspace(-top * cap, top * cap, n, dtype=torch.float64)
        keys = keys.bfloat16().double()
        values = torch.eye(n, d, dtype=torch.float64)[:, None] * 8 + torch.linspace(-1, 1, n, dtype=torch.float64)[:, None, None]
        values = values.bfloat16().double()
        q = torch.zeros(2, 1, d, dtype=torch.float64)
        q[:, 0, 0] = 1.0
        want = _capped(q, [keys], [values], [(0, n - 2), (0, n - 1)], 1.0, cap, 0, 1, None)
        kp, tables = _paged([keys], 16, torch.bfloat16)
        vp, _ = _paged([values], 16, torch.bfloat16)
        out = torch.empty(2, d, dtype=torch.bfloat16, device="cuda")
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        k.attention_prefill_tc(q.view(2, d).bfloat16().cuda(), kp, vp, tables, torch.tensor([0, 2], dtype=torch.int32).cuda(),
                               torch.tensor([n - 2, n - 1], dtype=torch.int32).cuda(), out, 1, 1, 1.0, status, softcap=cap)
        assert int(status) == 0 and (out.double().cpu().view(2, 1, d) - want).abs().max() < 1e-2, top


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 1, 8, 8, 8), (4, 2, 16, 12, 16), (3, 3, 24, 20, 24), (5, 1, 40, 40, 8)])
def test_blended_values_and_norms_over_the_projection(sizes, dtype):
    """The first layer leaves its values, later layers cache blends with them; rows without a cache slot leave theirs too."""
    from edgerag_b200.ops import kernels as k

    H, G, D, dv, page = sizes[0], sizes[1], sizes[2], sizes[3], sizes[4]
    dq = D - 4 if D > 8 else D                      # true size of queries and keys
    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(sum(sizes))
    n, eps = 7, 1e-5
    pad = lambda t, heads, true: torch.nn.functional.pad(t.view(n, heads, true), (0, D - true)).reshape(n, heads * D)     # noqa: E731
    slots = torch.tensor([page * 2 + 1, 0, -1, page - 1, page, 3, page * 3], dtype=torch.int32)
    first = torch.full((n, G * dv), float("nan"), dtype=tdt, device="cuda")
    v0 = None
    for blend in (None, 0.3, 1.0, -0.5):
        q, kk, v = (torch.randn(n, h * true, generator=g).to(tdt) for h, true in ((H, dq), (G, dq), (G, dv)))
        qn, kn = 1 + 0.3 * torch.randn(H * dq, generator=g), 1 + 0.3 * torch.randn(G * dq, generator=g)
        row = torch.cat([pad(q, H, dq), pad(kk, G, dq), pad(v, G, dv), torch.full((n, 8), 7.0).to(tdt)], 1).cuda().contiguous()
        kp = torch.zeros(4, G, page, D, dtype=tdt, device="cuda")
        vp = torch.zeros(4, G, page, D, dtype=tdt, device="cuda")
        wpad = lambda w, heads: torch.nn.functional.pad(w.view(heads, dq), (0, D - dq)).reshape(-1).cuda().contiguous()    # noqa: E731
        k.qkv_whole_norm(row, torch.zeros(n, dtype=torch.int32, device="cuda"), H, G, D, q_count=H * dq, k_count=G * dq, eps=eps, q_norm=wpad(qn, H),
                         k_norm=wpad(kn, G), slots=slots.cuda(), k_pages=kp, v_pages=vp, page_size=page, first_values=first,
                         blend=None if blend is None else torch.tensor([blend], device="cuda"))
        if blend is None:
            v0 = v.double()
            assert torch.equal(first.cpu(), v), "the first layer's values as they were projected"
        mixed = v.double() if blend is None else plain.blend_values(v.double(), v0, torch.tensor(blend))
        wq, wk = plain.rms_norm(q.double(), qn, eps), plain.rms_norm(kk.double(), kn, eps)
        tol = 2e-5 if dtype == "float32" else 4e-2
        assert (row[:, : H * D].double().cpu().view(n, H, D)[..., :dq] - wq.view(n, H, dq)).abs().max() < tol
        assert bool((row[:, -8:] == 7.0).all()), "columns behind the values were touched"
        for t, s in enumerate(slots.tolist()):
            if s >= 0:
                assert (kp[s // page, :, s % page, :dq].double().cpu() - wk[t].view(G, dq)).abs().max() < tol
                assert (vp[s // page, :, s % page, :dv].double().cpu() - mixed[t].view(G, dv)).abs().max() < tol
        assert int((vp.abs().sum(-1) > 0).sum()) == 6 * G


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [30, 64, 1024])
def test_embedding_of_pairs_and_positions(width, dtype):
    """Single tokens and portions of several sequences in one launch: the record before a portion, the record after it, a
    sequence's first token, a row without a record, ids and positions out of range."""
    from edgerag_b200.ops import kernels as k

    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(width)
    vocab, buckets, mp, mc, n_pos, scale = 40, 23, 3_000_000_019, 7, 50, 2.25
    table, pairs, pos_table = (torch.randn(r, width, generator=g).to(tdt) for r in (vocab, buckets + 1, n_pos))
    # sequences of the step: (slot, first position, ids); the records hold the ids before
    seqs = [(2, 9, [5]), (0, 0, [6]), (-1, 0, [0]), (3, 17, [7, 8, 9, 10]), (1, 0, [11, 12, 11])]
    before = torch.tensor([31, 32, 33, 34], dtype=torch.int32)
    ids = torch.tensor([t for _, _, s in seqs for t in s], dtype=torch.int32)
    pos = torch.tensor([p + i for _, p, s in seqs for i in range(len(s))], dtype=torch.int32)
    seq_of = torch.tensor([i for i, (_, _, s) in enumerate(seqs) for _ in s], dtype=torch.int32)
    starts = torch.tensor([0] + list(np.cumsum([len(s) for _, _, s in seqs])), dtype=torch.int32)
    want, rows = [], []
    for slot, p, s in seqs:
        prev = int(before[slot])
        for i, t in enumerate(s):
            row = buckets if p + i == 0 else (prev * mp + t * mc) % buckets
            rows.append(row)
            want.append(table[t].double() * scale + pairs[row].double() + pos_table[p + i].double())
            prev = t
    assert len(set(rows)) > 5
    hidden = torch.full((len(ids), width), float("nan"), device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    last = before.clone().view(4, 1).cuda()
    how = dict(pair_hash=(buckets, mp, mc), seq_of_token=seq_of.cuda(), seq_starts=starts.cuda(),
               state_slots=torch.tensor([s for s, _, _ in seqs], dtype=torch.int32).cuda(), last_id=last)
    dev = [t.cuda() for t in (table, pairs, pos_table)]
    k.embed_sum(hidden, dev[0], ids.cuda(), status, pos.cuda(), scale=scale, pairs=dev[1], pos_table=dev[2], **how)
    assert (hidden.double().cpu() - torch.stack(want)).abs().max() < 2e-6 * 10 and int(status) == 0
    assert last.flatten().tolist() == [6, 11, 5, 10]
    only = torch.stack([table[t].double() * scale + pos_table[p].double() for t, p in zip(ids.tolist(), pos.tolist())])
    k.embed_sum(hidden, dev[0], ids.cuda(), status, pos.cuda(), scale=scale, pos_table=dev[2])
    assert (hidden.double().cpu() - only).abs().max() < 2e-5
    far = pos.clone()
    far[4] = n_pos
    k.embed_sum(hidden, dev[0], ids.cuda(), status, far.cuda(), scale=scale, pos_table=dev[2])
    assert int(status) == 5 and bool((hidden[4] == 0).all()) and (hidden[3].double().cpu() - only[3]).abs().max() < 2e-5
    status.zero_()
    bad = ids.clone()
    bad[1] = vocab
    k.embed_sum(hidden, dev[0], bad.cuda(), status, pos.cuda(), scale=scale, pairs=dev[1], pos_table=dev[2], **how)
    assert int(status) == 2 and bool((hidden[1] == 0).all())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(12, 4, 64), (5, 1, 40), (8, 8, 96), (64, 6, 256), (33, 2, 33)])
def test_router_with_a_scaled_weight_and_the_shared_experts_gate(sizes, dtype):
    """Softmax scores times a constant, and one more row of the router whose sigmoid is left per token; it is no expert, however
    large its logit.  The kernels for few tokens give the same bits."""
    from edgerag_b200.ops import kernels as k

    E, top, width = sizes
    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(E + top)
    router = (torch.randn(E, width, generator=g) * 2.0 / math.sqrt(width)).float()
    side = (torch.randn(1, width, generator=g) * 6.0 / math.sqrt(width)).float()
    for n in (5, 16, 200):
        x = torch.randn(n, width, generator=g).to(tdt)
        idx, w = plain.routed_choice(x.double(), {"router": router.double()}, "", {"top": top, "scale": 1.75})
        z = (x.double() @ router.double().T).sort(-1, descending=True).values
        clear = (z[:, :-1] - z[:, 1:]).min(-1).values > 1e-4
        assert int(clear.sum()) > n // 4
        lists = torch.zeros(k.moe_lists_ints(n, E, top), dtype=torch.int32, device="cuda")
        score = torch.zeros(n * top, device="cuda")
        gate = torch.full((n,), float("nan"), device="cuda")
        how = dict(scores="softmax", weight=1.75)
        both = torch.cat([router, side]).cuda()
        k.moe_route(x.cuda(), both, top, lists, score, side_gate=gate, **how)
        assert torch.equal(lists[: n * top].view(n, top).cpu()[clear].long(), idx[clear])
        assert torch.allclose(score.view(n, top).cpu().double()[clear], w[clear], rtol=2e-5, atol=1e-7)
        assert (gate.double().cpu() - torch.sigmoid(x.double() @ side.double().T)[:, 0]).abs().max() < 1e-5
        assert int(lists[: n * top].max()) < E
        plain_lists, plain_score = torch.zeros_like(lists), torch.zeros_like(score)
        k.moe_route(x.cuda(), router.cuda(), top, plain_lists, plain_score, scores="softmax")
        assert torch.equal(plain_lists, lists) and torch.allclose(plain_score * 1.75, score, rtol=1e-6)
        if k.moe_route_few(n, E, top, tdt):
            l2, s2, g2 = torch.zeros_like(lists), torch.zeros_like(score), torch.zeros_like(gate)
            k.moe_route(x.cuda(), both, top, l2, s2, side_gate=g2, logits=torch.empty(n, E + 1, device="cuda"), **how)
            assert torch.equal(l2, lists) and torch.equal(s2, score) and torch.equal(g2, gate)
        k.moe_route(x.cuda(), router.cuda(), top, lists, score, scores="softmax", normalise=True, weight=2.0)
        assert torch.allclose(score.view(n, top).sum(-1).cpu(), torch.full((n,), 2.0), atol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inter", [24, 30, 128])
def test_gated_unit_with_a_factor_per_row(inter, dtype):
    from edgerag_b200.ops import kernels as k

    tdt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(inter)
    n, tol = 9, 2e-5 if dtype == "float32" else 2e-2
    gu, f = (torch.randn(n, 2 * inter, generator=g) * 2).to(tdt), torch.rand(n, generator=g)
    for limit, alpha, shift in ((0.0, 1.0, 0.0), (1.5, 1.702, 1.0)):
        a, b = gu[:, :inter].double(), gu[:, inter:].double()
        if limit:
            a, b = a.clamp(max=limit), b.clamp(-limit, limit)
        want = a * torch.sigmoid(alpha * a) * (b + shift) * f.double()[:, None]
        out = torch.empty(n, inter, dtype=tdt, device="cuda")
        k.glu_bounded(gu.cuda(), out, limit, alpha, shift, row_scale=f.cuda())
        assert (out.double().cpu() - want).abs().max() < tol * want.abs().max()
    if dtype == "bfloat16":            # the product and the gated unit in one kernel: the same bits as the two
        x, w = torch.randn(n, 64, generator=g).to(tdt).cuda(), (torch.randn(2 * inter, 64, generator=g) / 8).to(tdt).cuda()
        both, one, two = (torch.empty(n, c, dtype=tdt, device="cuda") for c in (2 * inter, inter, inter))
        for bounded in ((0.0, 1.0, 0.0), (0.8, 1.702, 1.0)):
            k.linear(x, w, both)
            k.glu_bounded(both, two, *bounded, row_scale=f.cuda())
            k.linear_glu(x, w, one, bounded=bounded, row_scale=f.cuda())
            assert torch.equal(one, two)


# --- through the framework's entry points -----------------------------------------------------------

def _greedy_holds(raw, tensors, prompt, out):
    """The engine's token is the plain argmax wherever the plain margin is clear."""
    seq = list(prompt)
    for tok in out:
        logits = plain.forward(raw, tensors, seq)[-1]
        top = torch.topk(logits, 2).values
        if float(top[0] - top[1]) > 1e-3 * float(logits.abs().max()):
            assert tok == int(logits.argmax())
        seq.append(tok)


@pytest.mark.gpu
@pytest.mark.parametrize("lookahead", [False, True])
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(graphs, lookahead, folders):
    """Five prompts of unequal length, three at a time: portions beside single tokens, steps of three single tokens (filled up to
    four), tokens fed back on the device (their predecessors then are known there only), replayed graphs."""
    from edgerag_b200 import SamplingParams
    from edgerag_b200.engine.engine import Engine, EngineOptions

    # (a small embedding: with the head tied to a large one, random weights would repeat the prompt's last token for ever)
    small = copy.deepcopy(FULL)
    small["embedding"]["scale"] = 0.1
    folder, raw, tensors = folders("small embedding", small, seed=1)
    prompts = [tokens_for(raw, n, 40 + i) for i, n in enumerate((37, 5, 21, 1, 12))]
    eng = Engine.from_pretrained(folder, EngineOptions(dtype="float32", block_size=16, num_blocks=24, max_batch_size=3, lookahead=lookahead,
                                                       max_step_tokens=64, chunk_size=8, cuda_graphs=graphs))
    outs = eng.generate(prompts, [SamplingParams(max_new_tokens=n) for n in (14, 18, 12, 16, 15)])
    assert [len(o) for o in outs] == [14, 18, 12, 16, 15]
    for prompt, out in zip(prompts, outs):
        _greedy_holds(raw, tensors, prompt, out)
    assert len({t for out in outs for t in out}) > 12
    assert (eng.runner.graph_replays > 0) == graphs and (eng.lookahead_steps > 0) == lookahead
    eng.cache.check_invariants()
    assert eng.cache.free_pages() == [24] * len(eng.cache.layout.groups)


@pytest.mark.gpu
def test_generation_stops_at_the_last_position(folders):
    from edgerag_b200 import SamplingParams
    from edgerag_b200.engine.engine import Engine, EngineOptions

    folder, raw, tensors = folders("short", plain.make_config([DENSE], positions=20), seed=11)
    eng = Engine.from_pretrained(folder, EngineOptions(dtype="float32", block_size=16, num_blocks=8, chunk_size=8))
    eng.generate([tokens_for(raw, 12, 3)], SamplingParams(max_new_tokens=8))
    with pytest.raises(RuntimeError, match="rejected"):
        eng.generate([tokens_for(raw, 12, 3)], SamplingParams(max_new_tokens=30))
    out = eng.generate([tokens_for(raw, 15, 4)], SamplingParams(max_new_tokens=5))[0]
    assert len(out) == 5


@pytest.mark.gpu
@pytest.mark.parametrize("extra", [(), ("--cuda-graphs",)])
def test_trace_replay_program(extra, folders, tmp_path):
    import helpers

    folder, raw, tensors = folders("full", FULL, seed=1)
    trace = helpers.Trace()
    for i, n in enumerate((70, 33, 90, 18, 47)):
        trace.sequences[f"r{i}"] = tokens_for(raw, n, 60 + i)
    helpers.cut_mixed(trace, list(trace.sequences), seed=3)
    cmd = [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path / "out"),
           "--max-tokens", str(trace.max_tokens), "--poison-freed-pages", *extra]
    text = "".join(json.dumps(s) + "\n" for s in trace.steps)
    proc = subprocess.run(cmd, input=text, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [int(l.split()[1]) for l in proc.stdout.splitlines() if l.startswith("done ")] == [s["step"] for s in trace.steps]
    want = {rid: plain.forward(raw, tensors, seq) for rid, seq in trace.sequences.items()}
    files = {s: torch.from_numpy(np.fromfile(tmp_path / "out" / f"{s}.f32", dtype="<f4").reshape(-1, raw["vocab"])) for s in {e[0] for e in trace.expect}}
    got = torch.stack([files[step][row] for step, row, _, _ in trace.expect])
    assert_close(got, torch.stack([want[rid][pos] for _, _, rid, pos in trace.expect]), "float32", "trace")


@pytest.mark.gpu
def test_serving_from_a_saved_model_in_bfloat16(folders):
    from edgerag_b200 import Engine, SamplingParams

    folder, raw, tensors = folders("full", FULL, seed=1)
    eng = Engine.from_pretrained(folder, dtype="bfloat16", block_size=16, num_blocks=16)
    out = eng.generate([tokens_for(raw, 9, 77)], SamplingParams(max_new_tokens=5))[0]
    assert len(out) == 5 and all(0 <= t < raw["vocab"] for t in out)


@pytest.mark.gpu
def test_command_line_with_random_weights(tmp_path):
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(FULL))
    base = [sys.executable, "-m", "edgerag_b200", "--dtype", "fp32", "--num-blocks", "16", "--max-batch-size", "2", "--chunk-size", "16",
            "--max-new-tokens", "5", "--prompt-ids", "3,1,4,1,5,9,2,6", "--prompt-ids", "7", "--json"]
    first = subprocess.run(base + ["--random-weights", "3", "--config", str(cfg), "--save-model", str(tmp_path / "m"), "--weights-std", "0.1"],
                           capture_output=True, text=True, timeout=900, cwd=ROOT)
    assert first.returncode == 0, first.stderr[-2000:]
    again = subprocess.run(base + ["--model", str(tmp_path / "m")], capture_output=True, text=True, timeout=900, cwd=ROOT)
    assert again.returncode == 0, again.stderr[-2000:]
    a, b = (json.loads(p.stdout.strip().splitlines()[-1])["outputs"] for p in (first, again))
    assert [len(o["token_ids"]) for o in a] == [5, 5] and a == b
