"""Zabusun on the GPU against the plain implementation (``plain_zabusun``): each mechanism alone, then whole models of
several made-up shapes stepped through the engine under every cutting, and generation through the scheduler.

The models' weights are drawn here, larger than a trained model's, so that a key that is wrongly seen or missed, a number per head
or a gate that is left out, a state that is lost, a wrong expert or a share that weighs the wrong side all move the logits by much
more than the tolerance."""
from __future__ import annotations

import json
import math

import numpy as np
import pytest
import torch
from safetensors.torch import save_file

import plain_zabusun as plain
import trace_tools
from test_parts_gpu import step_view
from test_zemavik_gpu import assert_logits, engine_for, fresh_cache, make_requests, on, run_part

pytestmark = pytest.mark.gpu

DEVICE = "cuda"


# ---------------------------------------------------------------------------------------
# made-up models
# ---------------------------------------------------------------------------------------
def dense(ff, limit=2.0):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top, limit=2.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def layer(left, rot, right, scales, mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale); rot: (dims, base, scaling or None) or None; right: width."""
    attention = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left))
    if rot is not None:
        attention["rot"] = {"dims": rot[0], "base": rot[1], "scaling": rot[2]}
    return {"type": "parallel", "mixer": {"left": attention, "left_scale": scales[0], "right": {"width": right}, "right_scale": scales[1]}, "mlp": mlp}


def model(vocab, width, layers, eps=1e-5, logit_scale=0.5):
    return {"architecture": "Zabusun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "logit_scale": logit_scale}


YARN = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}
CONFIGS = {
    # values wider and narrower than keys, grouped heads, a head per kv head and one head; rotation of part of a head with YaRN, of all of it
    # without, and none; a recurrence wider and narrower than the model and of an odd width; experts, dense, no feed-forward
    "mix": model(97, 72, [
        layer((6, 2, 16, 24, 0.3), (12, 500.0, YARN), 88, (0.7, 1.2), moe(24, 5, 2)),
        layer((3, 3, 24, 8, 0.2), (24, 10000.0, None), 33, (1.1, 0.6)),
        layer((1, 1, 8, 8, 0.5), None, 16, (0.5, 1.0), dense(40, 1.5)),
    ], logit_scale=0.7),
    # heads of sizes that are no multiples of 8, one expert a token, experts and a stream of an odd width; pages of 4
    "odd": model(61, 45, [
        layer((4, 1, 10, 6, 0.4), (6, 50.0, YARN), 7, (1.3, 0.9), moe(9, 3, 1, 1.0)),
        layer((2, 2, 12, 20, 0.3), (4, 300.0, {"factor": 2.0, "original": 64, "fast": 16.0, "slow": 2.0}), 20, (0.8, -0.5), dense(12, 3.0)),
    ], eps=1e-4, logit_scale=1.0),
    # the sizes at which prompts run on the tcgen05 kernels and decoded tokens on the TMA-fed ones: heads of 64 and (values of 96 kept
    # wider) 128, pages of 64; enough tokens an expert for the grouped product in the longest prompt
    "cores": model(130, 128, [
        layer((4, 2, 64, 64, 0.12), (32, 10000.0, YARN), 96, (1.1, 0.5), moe(32, 3, 1)),
        layer((6, 1, 128, 96, 0.09), (64, 5000.0, YARN), 160, (0.6, 0.9), moe(48, 4, 2, 1.2)),
    ], logit_scale=0.4),
    # a width at which decode products come as partial sums over slices of k, a last product over both mixers' outputs side by side
    "wide": model(112, 1024, [layer((8, 2, 64, 64, 0.1), (64, 10000.0, YARN), 520, (0.9, 0.7), moe(256, 4, 2)), layer((4, 4, 128, 128, 0.08), (32, 900.0, YARN), 512, (1.0, 1.0), dense(1024))],
                  logit_scale=0.1),
}
PAGE_SIZES = {"mix": 8, "odd": 4, "cores": 64, "wide": 64}
LENGTHS = {"mix": (61, 23, 5, 38, 1, 44, 17), "odd": (70, 9, 35, 2, 41), "cores": (330, 70, 3, 129), "wide": (150, 66, 9)}


def draw_weights(config, seed):
    """Weights of a made-up model: matrices N(0, 1/in) times a gain, norm weights around one, numbers per head that keep most weights
    well below one, gates of the recurrence from quick to nearly shut."""
    g = torch.Generator().manual_seed(seed)
    rand = lambda *shape: torch.randn(*shape, generator=g)
    matrix = lambda out, inner, gain=1.0: rand(out, inner) * gain / math.sqrt(inner)
    width = config["width"]
    w = {"embed": rand(config["vocab"], width), "embed.norm": 1 + 0.2 * rand(width), "final.norm": 1 + 0.2 * rand(width)}
    for index, one in enumerate(config["layers"]):
        name, left, channels, mlp = f"l{index}.", one["mixer"]["left"], one["mixer"]["right"]["width"], one["mlp"]
        heads, groups, dim, vdim = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
        w[name + "norm1"] = 1 + 0.2 * rand(width)
        mix = name + "mix.left."
        w[mix + "q"], w[mix + "k"], w[mix + "v"] = matrix(heads * dim, width), matrix(groups * dim, width), matrix(groups * vdim, width)
        w[mix + "o"], w[mix + "g"] = matrix(width, heads * vdim, 2.0), matrix(heads, width, 2.0)
        w[mix + "q.norm"], w[mix + "k.norm"], w[mix + "pb"] = 1.5 + 0.4 * rand(dim), 1.5 + 0.4 * rand(dim), -3.0 + rand(heads)
        mix = name + "mix.right."
        w[mix + "z"], w[mix + "x"], w[mix + "g"], w[mix + "o"] = matrix(channels, width), matrix(channels, width, 1.5), matrix(channels, width, 1.5), matrix(width, channels)
        w[mix + "z.b"], w[mix + "x.b"] = -3.0 + 2.5 * rand(channels), 0.5 * rand(channels)
        if mlp is None:
            continue
        w[name + "norm2"] = 1 + 0.2 * rand(width)
        if mlp["kind"] == "dense":
            w[name + "mlp.gate"], w[name + "mlp.up"], w[name + "mlp.down"] = matrix(mlp["ff"], width, 1.5), matrix(mlp["ff"], width, 1.5), matrix(width, mlp["ff"])
            continue
        ff = mlp["expert"]["ff"]
        w[name + "mlp.router"] = matrix(mlp["router"]["experts"], width, 1.0)     # scores all over (0, 1)
        for e in range(mlp["router"]["experts"]):
            p = f"{name}mlp.e{e}."
            w[p + "gate"], w[p + "up"], w[p + "down"] = matrix(ff, width, 2.5), matrix(ff, width, 2.5), matrix(width, ff)
    return {key: value.to(torch.bfloat16).contiguous() for key, value in w.items()}


def every_expert(config):
    """The same model with every token going through all of a layer's experts: no choice is left that rounding could turn."""
    out = json.loads(json.dumps(config))
    for one in out["layers"]:
        if one["mlp"] is not None and one["mlp"]["kind"] == "moe":
            one["mlp"]["router"]["top"] = one["mlp"]["router"]["experts"]
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (folder, config, weights as stored); under ``name + "/all"`` the same weights with a configuration in which
    every expert is used: a 16-bit run is compared on the latter, since a rounded input turns a close choice now and then."""
    made = {}
    for seed, (name, config) in enumerate(CONFIGS.items()):
        weights = draw_weights(config, 900 + seed)
        for key, stored in ((name, config), (name + "/all", every_expert(config))):
            folder = tmp_path_factory.mktemp("zabusun_" + name)
            save_file(weights, str(folder / "model.safetensors"), metadata={"format": "pt"})
            (folder / "config.json").write_text(json.dumps(stored))
            made[key] = (folder, stored, weights)
    return made


def plain_logits(config, weights, requests):
    logits = {name: plain.forward(config, weights, tokens).numpy() for name, tokens in requests.items()}
    return logits, {name: len(tokens) for name, tokens in requests.items()}


# ---------------------------------------------------------------------------------------
# whole models under every cutting
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cutting_gives_the_plain_logits(models, name, dtype):
    folder, config, weights = models[name if dtype == "float32" else name + "/all"]
    requests = make_requests(config, LENGTHS[name], seed=7)
    want, sure = plain_logits(config, weights, requests)
    page = PAGE_SIZES[name]
    cuttings = {
        "whole": trace_tools.whole(requests),
        "tail one by one": trace_tools.tail_one_by_one(requests, tail=30),
        "changing portions": trace_tools.changing_portions(requests),
        "mixed": trace_tools.mixed(requests, seed=3, max_live=3, decode_tail=9, max_portion=19),
    }
    for what, steps in cuttings.items():
        pool = trace_tools.pool_tokens(steps, round_to=page)     # no page to spare: pages and slots are used again
        engine = engine_for(folder, dtype, page, pool, slots=3, prefill_chunk_size=pool)
        got = trace_tools.run_in_process(engine, steps)
        assert_logits(got, want, sure, dtype, f"{name}, {what}, {dtype}")
        assert engine.cache.free_slots() == 3 and all(group.pool.free_count == group.pool.num_pages for group in engine.cache.groups)
        del engine


def test_layer_by_layer_in_32_bit(models):
    from pylon_b200.engine import StepEntry

    folder, config, weights = models["mix"]
    tokens = make_requests(config, (37,), seed=5)["r0"]
    want: list = []
    plain.forward(config, weights, tokens, layers_out=want)
    engine = engine_for(folder, "float32", 8, 64)
    taps: list = []
    forward = engine.model.forward
    engine.model.forward = lambda step, caches: forward(step, caches, taps)
    request = engine.open("a", len(tokens))
    engine.step([StepEntry(request, tokens, [0])])
    assert len(taps) == len(want) == 3
    for index, (got, expected) in enumerate(zip(taps, want)):
        torch.testing.assert_close(got.double().cpu(), expected, rtol=1e-4, atol=1e-4 * float(expected.abs().max()), msg=lambda m: f"layer {index}: {m}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_over_many_pages(models, dtype):
    """A short prompt, then 200 tokens one by one: every token reads all keys before it, the state is carried 200 times."""
    folder, config, weights = models["mix" if dtype == "float32" else "mix/all"]
    requests = make_requests(config, (212,), seed=11)
    want, sure = plain_logits(config, weights, requests)
    engine = engine_for(folder, dtype, 8, 216)
    got = trace_tools.run_in_process(engine, trace_tools.tail_one_by_one(requests, tail=200))
    assert_logits(got, want, sure, dtype, "long decoding")


def test_the_replay_program_runs_the_model(models, tmp_path):
    folder, config, weights = models["odd"]
    requests = make_requests(config, (33, 12, 20), seed=2)
    want, sure = plain_logits(config, weights, requests)
    steps = trace_tools.mixed(requests, seed=1, max_live=2, decode_tail=5, max_portion=9)
    got = trace_tools.run_program(folder, "float32", steps, tmp_path / "out", extra_args=("--page-size", "4"))
    assert_logits(got, want, sure, "float32", "bin/trace_run")


@pytest.mark.parametrize("name,graphs", [("mix", False), ("mix", True), ("cores", True)])
def test_greedy_generation_through_the_scheduler(models, name, graphs):
    """Several prompts through ``Engine.generate`` with a small prompt budget and few slots: every generated token is the
    arg-max of the plain logits of its own prefix."""
    from pylon_b200.sampling.params import SamplingParams

    folder, config, weights = models[name]
    prompts = list(make_requests(config, (19, 3, 40, 11, 27, 8), seed=13).values())
    new_tokens = 12
    engine = engine_for(folder, "float32", PAGE_SIZES[name], 4 * 64, slots=3, prefill_chunk_size=16, cuda_graphs=graphs)
    results = engine.generate(prompts, SamplingParams(max_new_tokens=new_tokens, temperature=0.0, ignore_eos=True))
    for prompt, result in zip(prompts, results):
        assert len(result.output_ids) == new_tokens
        sequence = list(prompt) + list(result.output_ids)
        logits = plain.forward(config, weights, sequence[:-1])
        for place in range(len(prompt) - 1, len(sequence) - 1):
            row = logits[place]
            best = int(row.argmax())
            if sequence[place + 1] != best:   # a tie within rounding may go either way
                assert float(row[best] - row[sequence[place + 1]]) < 1e-3 * float(row.std()), f"token {place + 1} of a request is not the plain arg-max"
    engine.cache.check()
    assert engine.cache.free_slots() == 3


def test_bfloat16_generation_from_graphs_follows_the_plain_logits(models):
    """The 16-bit decode steps from CUDA graphs and the padded graphs of steps with portions: a generated token's plain logit lies
    within what rounding moves of the plain arg-max's."""
    from pylon_b200.sampling.params import SamplingParams

    folder, config, weights = models["cores/all"]
    prompts = list(make_requests(config, (70, 3, 130, 65), seed=17).values())
    engine = engine_for(folder, "bfloat16", 64, 3 * 192, slots=3, prefill_chunk_size=48, cuda_graphs=True)
    results = engine.generate(prompts, SamplingParams(max_new_tokens=20, temperature=0.0, ignore_eos=True))
    for prompt, result in zip(prompts, results):
        sequence = list(prompt) + list(result.output_ids)
        logits = plain.forward(config, weights, sequence[:-1])
        for place in range(len(prompt) - 1, len(sequence) - 1):
            row = logits[place]
            assert float(row.max() - row[sequence[place + 1]]) < 0.25 * float(row.std())
    engine.cache.check()


# ---------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------
def attention_spec(width, m, eps):
    from pylon_b200.parts import PartSpec

    rot = m.get("rot")
    position = None if rot is None else PartSpec("rope", {
        "head_dim": m["dim"], "theta": rot["base"], "max_positions": 256, "rotary_dim": rot["dims"],
        "scaling": None if rot["scaling"] is None else {"kind": "yarn", **rot["scaling"]}, "layout": "halves"})
    return PartSpec("gqa_attention", {
        "width": width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "scale": m["scale"],
        "position": position, "qk_norm_eps": eps, "weighting": "sigmoid", "score_bias": True, "head_gate": True,
        "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "score_bias": "pb", "head_gate": "g"}})


def mixer_case(name, rand, matrix, width, eps):
    """(the mixer's tensors, its part's description, the plain function) of a small made-up mixer."""
    from pylon_b200.parts import PartSpec

    bf = lambda t: t.to(torch.bfloat16)
    sizes = {"narrow": (4, 2, 20, 12), "equal": (6, 2, 32, 32), "wider": (3, 1, 8, 24), "cores": (8, 2, 64, 64)}.get(name, (4, 2, 20, 12))
    heads, groups, dim, vdim = sizes
    left = {"heads": heads, "kv_heads": groups, "dim": dim, "vdim": vdim, "scale": 0.35, "rot": {"dims": 8, "base": 300.0, "scaling": YARN}}
    w_left = {"q": matrix(heads * dim, width, 1.5), "k": matrix(groups * dim, width, 1.5), "v": matrix(groups * vdim, width), "o": matrix(width, heads * vdim),
              "g": matrix(heads, width, 2.0), "q.norm": bf(1.5 + 0.4 * rand(dim)), "k.norm": bf(1.5 + 0.4 * rand(dim)), "pb": bf(-3 + rand(heads))}
    channels = 37 if name == "recurrence_odd" else 36
    w_right = {"z": matrix(channels, width, 1.5), "x": matrix(channels, width, 1.5), "g": matrix(channels, width, 1.5), "o": matrix(width, channels),
               "z.b": bf(-2 + 2 * rand(channels)), "x.b": bf(0.5 * rand(channels))}
    recurrent = PartSpec("min_gru", {"width": width, "channels": channels})
    if name.startswith("recurrence"):
        return w_right, recurrent, lambda h, w: plain.min_gru(h, w, "")
    if name == "side_by_side":
        w = {**{"left." + k: v for k, v in w_left.items()}, **{"right." + k: v for k, v in w_right.items()}}
        spec = PartSpec("weighted_mixers", {"mixers": (attention_spec(width, left, eps), recurrent), "prefixes": ("left.", "right."), "scales": (1.3, 0.4)})
        return w, spec, lambda h, w: plain.mixer(h, w, "", {"left": left, "right": {"width": channels}, "left_scale": 1.3, "right_scale": 0.4}, eps)
    return w_left, attention_spec(width, left, eps), lambda h, w: plain.sigmoid_attention(h, w, "", left, eps)


def built(name, dtype, seed=21, width=56, eps=1e-5):
    from pylon_b200.parts import MIXERS

    g = torch.Generator().manual_seed(seed)
    rand = lambda *shape: torch.randn(*shape, generator=g)
    matrix = lambda out, inner, gain=1.0: (rand(out, inner) * gain / math.sqrt(inner)).to(torch.bfloat16)
    w, spec, oracle = mixer_case(name, rand, matrix, width, eps)
    part = MIXERS.build(spec)
    declared = {d.name: d for d in part.tensors()}
    assert set(declared) == set(w) and all(tuple(w[k].shape) == tuple(declared[k].shape) for k in w)
    part.load({k: on(v, torch.float32 if declared[k].role == "vector" else dtype) for k, v in w.items()}, dtype, torch.device(DEVICE))
    return part, w, oracle, rand


MIXER_NAMES = ["narrow", "equal", "wider", "cores", "recurrence", "recurrence_odd", "side_by_side"]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", MIXER_NAMES)
def test_each_mixer_alone_against_its_plain_statement(name, dtype):
    """A mixer part from its input to its output: a prompt in one step, then the same in portions down to single tokens, and token
    by token from the start."""
    part, w, oracle, rand = built(name, dtype)
    count, page = 60, 64 if name == "cores" else 8
    h = rand(count, 56).to(dtype)
    want = oracle(h.double(), {k: v.double() for k, v in w.items()})
    spread = float(want.std())
    limit = 0.06 * spread if dtype == torch.bfloat16 else 1e-4 * spread
    for cutting in ((count,), (20, 2, 1, 1, 28, 8), (1,) * 12 + (2, 2, 44), (9, 9, 9, 33), (8, 1, 9, 42), (2,) * 30, (1,) * count):
        got = run_part(part, h, cutting, page, dtype)
        assert float((got - want).abs().max()) <= limit, f"{name}, {cutting}: off by {float((got - want).abs().max()):.3g} of {spread:.3g}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", MIXER_NAMES)
def test_unequal_requests_in_one_step_against_each_alone(name, dtype):
    """Three requests of 1, 17 and 6 new tokens at different places of their sequences in one step, in state slots and pages
    that another request used before: every request's result is the one it has alone."""
    part, w, oracle, rand = built(name, dtype, seed=8)
    page = 64 if name == "cores" else 8
    before, new = (12, 0, 30), (1, 17, 6)
    inputs = [rand(b + n, 56).to(dtype) for b, n in zip(before, new)]
    want = [oracle(h.double(), {k: v.double() for k, v in w.items()}) for h in inputs]
    need = part.cache_need()
    cache = fresh_cache(need, page, dtype, table=tuple(range(15)), slots=4)
    slots = (2, 0, 3)
    if need.kv is not None:
        cache.block_table = torch.tensor([[9, 3, 12, 0, 7], [1, 14, 5, 10, 2], [6, 11, 4, 13, 8]], device=DEVICE, dtype=torch.int32)
        cache.k_pages.fill_(3.0)                               # what an earlier request left in the pages
        cache.v_pages.fill_(-2.0)

    def run(rows, sizes, starts):
        step = step_view(sizes, starts, dtype)
        step.slots = torch.tensor([slots[r] for r in rows], device=DEVICE, dtype=torch.int32)
        saved = cache.block_table
        if need.kv is not None:
            cache.block_table = saved[list(rows)].contiguous()
        out = part.forward(on(torch.cat([inputs[r][s : s + n] for r, n, s in zip(rows, sizes, starts)])), step, cache)
        cache.block_table = saved
        return (out.sum(dim=0) if out.dim() == 3 else out).double().cpu()

    if need.state is not None:
        cache.state.normal_()                                  # what an earlier request left in the slots ...
        cache.state[list(slots)] = 0.0                         # ... and a slot is handed out cleared
    for r in (0, 2):                                           # what the requests hold already, each alone
        run((r,), (before[r],), (0,))
    got = run((0, 1, 2), new, before)
    spread = float(torch.cat(want).std())
    limit = 0.06 * spread if dtype == torch.bfloat16 else 1e-4 * spread
    cursor = 0
    for r in range(3):
        mine = got[cursor : cursor + new[r]]
        cursor += new[r]
        worst = float((mine - want[r][before[r] :]).abs().max())
        assert worst <= limit, f"{name}: request {r} in the batch is off by {worst:.3g} of {spread:.3g}"


@pytest.mark.parametrize("dtype,dim,group,page", [(torch.float32, 24, 2, 16), (torch.bfloat16, 24, 2, 16), (torch.bfloat16, 48, 4, 16), (torch.bfloat16, 64, 1, 64),
                                                  (torch.bfloat16, 64, 5, 64), (torch.bfloat16, 128, 4, 64), (torch.bfloat16, 256, 2, 64)])
def test_keys_that_stand_out_far_away_and_at_page_borders(dtype, dim, group, page):
    """Hundreds of keys whose weights are next to nothing (the number per head is -9) and four that weigh almost one, each with a value of
    its own: the first key, the last of a page, the first of the next and one in the middle.  A token sees each from its own position
    on and never before.  As one prompt, with a tail token by token, in portions that end at the keys, in portions of two; into a slice of wider
    rows whose edges stay as they are, with gated heads and a factor."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(5)
    count, kv_heads = 300, 2
    heads = kv_heads * group
    places = (0, 2 * page - 1, 2 * page, 201)
    keys = torch.randn(count, kv_heads, dim, generator=g) * 0.1
    values = torch.randn(count, kv_heads, dim, generator=g) * 0.5
    direction = torch.ones(dim)
    for n, place in enumerate(places):
        keys[place] = direction
        values[place] = torch.linspace(-4.0, 4.0, dim) * (1 if n % 2 else -1) + n
    queries = direction + torch.randn(count, heads, dim, generator=g) * 0.1
    scale = 18.0 / dim                                    # a key that stands out scores about 18
    bias = torch.full((heads,), -9.0) + 0.3 * torch.randn(heads, generator=g)
    gate, factor = torch.randn(count, heads, generator=g), 0.6
    q, k, v, gates = (t.to(dtype).double() for t in (queries, keys, values, gate))
    index = torch.arange(count)
    seen = index[:, None] >= index[None, :]
    scores = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(group, dim=1)) * scale + bias.double()[:, None, None]
    weights = plain.sigmoid(scores) * seen
    assert float(weights[:, -1, list(places)].min()) > 0.95 and float(weights[:, -1].sum(dim=-1).max()) < 4.6    # the four, and little besides
    want = (torch.einsum("hij,jhd->ihd", weights, v.repeat_interleave(group, dim=1)) * plain.sigmoid(gates)[..., None] * factor).reshape(count, heads * dim)
    pages_needed = -(-count // page)
    order = torch.randperm(pages_needed + 3, generator=g)[:pages_needed]
    k_pages, v_pages = (torch.full((pages_needed + 3, kv_heads, page, dim), 5.0) for _ in range(2))
    for logical, physical in enumerate(order.tolist()):
        for rows, pages in ((keys, k_pages), (values, v_pages)):
            part = rows[logical * page : (logical + 1) * page]
            pages[physical, :, : part.shape[0]] = part.transpose(0, 1)
    k_pages, v_pages, table = on(k_pages, dtype), on(v_pages, dtype), on(order[None].to(torch.int32))

    def run(cutting):
        outs, cursor = [], 0
        for size in cutting:
            step = step_view((size,), (cursor,), dtype)
            wide = torch.full((size, heads * dim + 24), 9.0, device=DEVICE, dtype=dtype)
            mine = slice(cursor, cursor + size)
            ops.paged_attention(on(queries[mine].to(dtype)).view(size, heads * dim), k_pages, v_pages, step.positions, step.token_row, step.q_start, step.kv_len, table,
                                heads, step.max_q, step.max_kv, scale=scale, weighting="sigmoid", score_bias=on(bias), head_gate=on(gate[mine].to(dtype)), out_factor=factor,
                                out=wide[:, 8 : 8 + heads * dim])
            assert float(wide[:, :8].min()) == 9.0 == float(wide[:, 8 + heads * dim :].max())
            outs.append(wide[:, 8 : 8 + heads * dim])
            cursor += size
        return torch.cat(outs).double().cpu()

    tolerance = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-4)
    for cutting in ((count,), (count - 40,) + (1,) * 40, (1, 2 * page - 2, 1, 1, count - 2 * page - 1), (2 * page, 201 - 2 * page, 1, 98), (2,) * 150, (190, 20, 20, 70)):
        assert sum(cutting) == count
        torch.testing.assert_close(run(cutting), want, **tolerance)


def test_many_small_weights_add_up_with_more_than_eight_bits():
    """2,000 keys of one value and equal scores: the output is the sum of the weights.  Each weight rounded to bfloat16 would be off
    the same way, and with it the sum; in 16 bits it is not."""
    from pylon_b200.kernels import ops

    count, dim, page = 2000, 64, 64
    for bias in (-7.31, -6.2, -5.013):
        pages_needed = -(-count // page)
        k_pages, v_pages = torch.zeros(pages_needed, 1, page, dim, device=DEVICE, dtype=torch.bfloat16), torch.ones(pages_needed, 1, page, dim, device=DEVICE, dtype=torch.bfloat16)
        table = torch.arange(pages_needed, device=DEVICE, dtype=torch.int32)[None]
        score_bias = torch.full((4,), bias, device=DEVICE)
        want = float(torch.sigmoid(score_bias[0].double().cpu()))
        for size in (200, 1):     # a prompt's portion on the tcgen05 kernel, a decoded token on the TMA-fed one
            step = step_view((size,), (count - size,), torch.bfloat16)
            q = torch.zeros(size, 4 * dim, device=DEVICE, dtype=torch.bfloat16)
            out = ops.paged_attention(q, k_pages, v_pages, step.positions, step.token_row, step.q_start, step.kv_len, table, 4, step.max_q, step.max_kv,
                                      scale=1.0, weighting="sigmoid", score_bias=score_bias, out_factor=256.0 / (want * count))
            exact = 256.0 * torch.arange(count - size + 1, count + 1, dtype=torch.float64)[:, None] / count
            assert float((out.double().cpu() / exact - 1.0).abs().max()) < 2.0 ** -8 + 1e-4, (bias, size)   # the output's own rounding and no more


def gru_identity(channels):
    eye = torch.eye(3 * channels)
    return {"z": eye[:channels], "x": eye[channels : 2 * channels], "g": eye[2 * channels :], "o": torch.eye(channels), "z.b": torch.zeros(channels), "x.b": torch.zeros(channels)}


def test_the_recurrence_reads_back_what_was_written_long_ago():
    """A channel whose gate is shut but for one token keeps what that token wrote for more than 2,000 tokens, through several rounds of the
    clusters' walk; the channel beside it is overwritten at every token.  The projections are unit matrices, so the layer's input is
    the product's columns themselves.  In one step, with single tokens around the write and the end, and in portions."""
    from pylon_b200.parts import MIXERS, PartSpec

    count, write, channels = 2300, 3, 6
    g = torch.Generator().manual_seed(3)
    h = torch.zeros(count, 3 * channels)
    h[:, :3] = -18.0                                        # the first three channels' gates are shut ...
    h[write, :3] = 18.0                                     # ... but for one token
    h[:, 3:channels] = 2.0 * torch.randn(count, 3, generator=g)
    h[:, channels : 2 * channels] = torch.randn(count, channels, generator=g)
    h[write, channels : channels + 3] = torch.tensor([5.0, -3.0, 0.0])      # candidates of both branches, and where they meet
    h[:, 2 * channels :] = 2.0 + torch.rand(count, channels, generator=g)
    w = gru_identity(channels)
    want = plain.min_gru(h.double(), {k: v.double() for k, v in w.items()}, "")
    silu = h[-1, 2 * channels : 2 * channels + 3].double()
    kept = (want[-1, :3] / (silu * torch.sigmoid(silu)))
    torch.testing.assert_close(kept, torch.tensor([5.5, 1 / (1 + math.exp(3.0)), 0.5], dtype=torch.float64), rtol=1e-3, atol=1e-3)
    assert float(want[write - 1, :3].abs().max()) < 1e-6
    part = MIXERS.build(PartSpec("min_gru", {"width": 3 * channels, "channels": channels}))
    part.load({k: on(v) for k, v in w.items()}, torch.float32, torch.device(DEVICE))
    for cutting in ((count,), (write, 1, 1, count - write - 19) + (1,) * 17, (2, 2, 9, 17, 600, 1100, count - 1730), (1024, 1024, 252), (8,) * 10 + (2220,)):
        assert sum(cutting) == count
        torch.testing.assert_close(run_part(part, h, cutting, 8, torch.float32), want, rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("channels", [1, 5, 64, 130])
def test_rows_of_many_lengths_in_one_call_of_the_recurrence(channels, dtype):
    """Rows of one token to more than a cluster's round, a row without tokens, slots in another order than rows, factors, slices of wider
    rows: every row against the plain walk from the state its slot holds."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(channels)
    lengths = (1, 130, 0, 9, 1100, 8, 17)
    slots = (3, 9, 1, 0, 7, 2, 5)
    total = sum(lengths)
    stored = torch.randn(total, 3 * channels + 16, generator=g).to(dtype)
    proj = stored[:, 8 : 8 + 3 * channels]
    bias, state = torch.randn(2, channels, generator=g) - 1.0, torch.rand(10, channels, generator=g)
    out = torch.full((total, channels + 16), 7.0, device=DEVICE, dtype=dtype)
    held = on(state.clone())
    q_start = torch.tensor([0, *np.cumsum(lengths)], dtype=torch.int32, device=DEVICE)
    ops.min_gru(on(stored)[:, 8 : 8 + 3 * channels], on(bias), held, q_start, torch.tensor(slots, dtype=torch.int32, device=DEVICE), len(lengths), max(lengths),
                out[:, 8 : 8 + channels], factor=-0.7)
    want_state, want, cursor = state.double().clone(), [], 0
    for length, slot in zip(lengths, slots):
        s = want_state[slot]
        for t in range(cursor, cursor + length):
            z, u, gate = (proj[t].double()[i * channels : (i + 1) * channels] for i in range(3))
            z, u = plain.sigmoid(z + bias[0].double()), u + bias[1].double()
            s = (1 - z) * s + z * torch.where(u >= 0, u + 0.5, plain.sigmoid(u))
            want.append(-0.7 * s * gate * plain.sigmoid(gate))
        want_state[slot] = s
        cursor += length
    torch.testing.assert_close(held.double().cpu(), want_state, rtol=1e-4, atol=1e-5)
    tolerance = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-5)
    torch.testing.assert_close(out[:, 8 : 8 + channels].double().cpu(), torch.stack(want), **tolerance)
    assert float(out[:, :8].min()) == 7.0 == float(out[:, 8 + channels :].max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [1, 30, 72, 200, 2048, 5000])
def test_the_norm_on_an_output_and_on_the_embedding(width, dtype):
    from pylon_b200.parts import NORMS, PartSpec, ResidualStream

    g = torch.Generator().manual_seed(width)
    norm = NORMS.build(PartSpec("rmsnorm", {"width": width, "eps": 1e-3, "weight_name": ""}))
    weight = torch.rand(width, generator=g) + 0.5
    norm.load({"": on(weight)}, dtype, torch.device(DEVICE))
    tol = dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=1e-5, atol=1e-5)
    table = (0.03 * torch.randn(11, width, generator=g)).to(dtype)
    ids = torch.tensor([3, 0, 10, 3, 7], dtype=torch.int32)
    stream = norm.enter(on(ids), on(table), 1.5)
    want = plain.rms_unit(table.double()[ids.long()] * 1.5, 1e-3) * weight.double()
    torch.testing.assert_close(stream.residual.double().cpu(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(stream.read(dtype).double().cpu(), want, **tol)
    for output in (torch.randn(5, width, generator=g).to(dtype), torch.randn(3, 5, width, generator=g)):    # a block, partial sums
        norm.join(stream, on(output))
        whole = output.double() if output.dim() == 2 else output.double().sum(dim=0)
        want = plain.add_normed(want, whole, weight.double(), 1e-3)
        torch.testing.assert_close(stream.residual.double().cpu(), want, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(stream.read(dtype).double().cpu(), want, **tol)
    delta = torch.randn(5, width, generator=g).to(dtype)     # something pending joins the sum first, and the copy is made anew
    stream.add(on(delta))
    torch.testing.assert_close(stream.read(dtype).double().cpu(), want + delta.double(), **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,top,parts,shared", [(30, 1, 0, False), (72, 3, 0, True), (200, 2, 2, False), (2048, 2, 5, True)])
def test_the_norm_on_rows_that_lie_in_slots(width, top, parts, shared, dtype):
    """An output that is still scattered: the sum of ``top`` rows a token, each times its share, as they lie or as partial sums."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(width)
    tokens, slots, eps = 7, 40, 1e-4
    rows = torch.randn(parts, slots, width, generator=g) if parts else torch.randn(slots, width, generator=g).to(dtype)
    slot_of = torch.randperm(slots, generator=g)[: tokens * top].to(torch.int32)
    share = torch.rand(tokens, top, generator=g) if shared else None
    weight, residual = torch.rand(width, generator=g) + 0.5, torch.randn(tokens, width, generator=g)
    whole = (rows.double().sum(dim=0) if parts else rows.double())[slot_of.long()].view(tokens, top, width)
    whole = (whole * share.double()[..., None] if shared else whole).sum(dim=1)
    want = plain.add_normed(residual.double(), whole, weight.double(), eps)
    held = on(residual.clone())
    copy = ops.output_norm(held, ops.ScatteredRows(on(rows), on(slot_of), top, None if share is None else on(share)), on(weight), eps, dtype)
    torch.testing.assert_close(held.double().cpu(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(copy.double().cpu(), want, **(dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=1e-5, atol=1e-5)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,experts,top,tokens", [(40, 12, 3, 1, 1), (56, 20, 6, 6, 7), (48, 24, 12, 4, 150), (128, 64, 33, 3, 70), (64, 40, 2, 1, 40),
                                                         (256, 136, 4, 2, 700), (384, 256, 3, 1, 600), (72, 9, 5, 2, 90), (64, 1024, 3, 2, 20)])
def test_the_mixture_whose_scores_weigh_the_experts_input(width, ff, experts, top, tokens, dtype):
    """Sigmoid scores in 32-bit as they are, the clamped unit on both sides of its limits, an expert's input times its score: one token, few and
    many, tiles that are partly filled, an inner width that is no whole piece; two shapes have enough tokens an expert for the grouped
    tensor-core product.  Tokens whose choice hangs on a margin that 16-bit rounding of the input can turn are left out there."""
    from pylon_b200.parts import FEED_FORWARDS, PartSpec

    g = torch.Generator().manual_seed(17)
    rand = lambda *shape: torch.randn(*shape, generator=g)
    matrix = lambda out, inner, gain=1.0: (rand(out, inner) * gain / math.sqrt(inner)).to(torch.bfloat16)
    w = {"router": matrix(experts, width, 1.5)}
    for e in range(experts):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = matrix(ff, width, 2.5), matrix(ff, width, 2.5), matrix(width, ff, 1.5)
    limit = 1.3
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    part = FEED_FORWARDS.build(PartSpec("expert_mixture", {
        "width": width, "intermediate": ff, "experts": experts, "top": top, "activation": "clamped", "limit": limit, "routing": "sigmoid", "share_normalized": False,
        "weigh": "input"}))
    declared = {d.name: d for d in part.tensors()}
    assert set(declared) == set(w) and all(tuple(w[k].shape) == tuple(declared[k].shape) for k in w)
    part.load({k: on(v, torch.float32 if declared[k].role == "vector" else dtype) for k, v in w.items()}, dtype, torch.device(DEVICE))
    h = rand(tokens, width).to(dtype)
    doubles = {k: v.double() for k, v in w.items()}
    want = plain.experts(h.double(), doubles, "", mlp)
    logits = (h.double() @ doubles["router"].T).sort(dim=1, descending=True).values
    sure = logits[:, top - 1] - logits[:, top] > (1e-4 if dtype == torch.float32 else 0.02) if top < experts else torch.ones(tokens, dtype=torch.bool)
    assert int(sure.sum()) >= 0.7 * tokens
    out = part.forward(on(h), step_view((tokens,), (0,), dtype))
    got = (out.sum(dim=0) if out.dim() == 3 else out).double().cpu()
    spread = float(want.std())
    tolerance = 0.06 * spread if dtype == torch.bfloat16 else 1e-4 * spread
    assert float((got - want)[sure].abs().max()) <= tolerance
    # the rows where the experts left them, for a reader that adds them up itself
    loose = part.forward_scattered(on(h), step_view((tokens,), (0,), dtype))
    rows = (loose.rows.sum(dim=0) if loose.rows.dim() == 3 else loose.rows).double().cpu()[loose.slot_of.long().cpu()].view(tokens, top, width).sum(dim=1)
    torch.testing.assert_close(rows, got, rtol=1e-5, atol=1e-5)
    # the same tokens in another order and among others: a token's result does not depend on its place in the step
    order = torch.randperm(tokens, generator=g)
    both = torch.cat([h[order], rand(5, width).to(dtype)])
    again = part.forward(on(both), step_view((tokens + 5,), (0,), dtype))
    again = (again.sum(dim=0) if again.dim() == 3 else again).double().cpu()[:tokens]
    if tokens + 5 < 512 or tokens >= 512:      # (the same kernels either way)
        assert torch.equal(again, got[order])


@pytest.mark.parametrize("nq,nkv,dim,vdim,rot,own", [(3, 1, 16, 24, 16, 16), (4, 2, 64, 64, 32, 64), (6, 2, 48, 48, 16, 40), (2, 2, 128, 96, 128, 128), (8, 8, 8, 8, 0, 8), (2, 1, 256, 256, 64, 200)])
def test_norm_rotation_and_cache_write_in_16_byte_pieces(nq, nkv, dim, vdim, rot, own):
    """The vector form of the kernel between projections and attention against plain arithmetic: heads whose own elements are fewer than the
    ones kept, values of another width, a slice of wider rows, a token of no request, rotation of none, part and all of a head."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(dim)
    tokens, page = 9, 4
    columns = (nq + nkv) * dim + nkv * vdim
    stored = torch.randn(tokens, columns + 8, generator=g).to(torch.bfloat16)
    heads = stored[:, : (nq + nkv) * dim].view(tokens, nq + nkv, dim)
    heads[..., own:] = 0.0
    positions = torch.tensor([5, 6, 7, 8, 9, 0, 0, 1, 2], dtype=torch.int32)
    row = torch.tensor([0, 0, 0, 0, 0, -1, 1, 1, 1], dtype=torch.int32)
    table = torch.tensor([[4, 2, 0], [3, 1, 5]], dtype=torch.int32)
    angle = torch.rand(16, max(rot // 2, 1), generator=g) * 6
    cos, sin = angle.cos() * 1.1, angle.sin() * 1.1
    q_weight, k_weight = torch.rand(dim, generator=g) + 0.5, torch.rand(dim, generator=g) + 0.5
    q_weight[own:] = k_weight[own:] = 0.0
    k_pages, v_pages = (torch.full((6, nkv, page, size), 7.0, device=DEVICE, dtype=torch.bfloat16) for size in (dim, vdim))
    work = on(stored.clone())
    ops.qkv_rotate_write(work[:, :columns], None, on(cos) if rot else None, on(sin) if rot else None, rot, "halves", "before", on(q_weight), on(k_weight), 1e-5, on(positions), on(row),
                         on(table), page, k_pages, v_pages, nq, nkv, dim, vdim, norm_size=own)
    x = heads.double()
    x = x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) / own + 1e-5) * torch.cat((q_weight.expand(nq, dim), k_weight.expand(nkv, dim))).double()
    if rot:
        c, s = cos.double()[positions.long()][:, None], sin.double()[positions.long()][:, None]
        u, v = x[..., : rot // 2].clone(), x[..., rot // 2 : rot].clone()
        x[..., : rot // 2], x[..., rot // 2 : rot] = u * c - v * s, v * c + u * s
    values = stored[:, (nq + nkv) * dim : columns].view(tokens, nkv, vdim).double()
    for t in range(tokens):
        if row[t] < 0:
            assert torch.equal(work[t].cpu(), stored[t])
            continue
        torch.testing.assert_close(work[t, : nq * dim].double().cpu().view(nq, dim), x[t, :nq], rtol=1e-2, atol=1e-2)
        physical, place = int(table[row[t], positions[t] // page]), int(positions[t]) % page
        torch.testing.assert_close(k_pages[physical, :, place].double().cpu(), x[t, nq:], rtol=1e-2, atol=1e-2)
        assert torch.equal(v_pages[physical, :, place].double().cpu(), values[t])
    assert torch.equal(work[:, columns:].cpu(), stored[:, columns:])
    ops.raise_on_kernel_errors(torch.device(DEVICE))
