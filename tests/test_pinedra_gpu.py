"""Pinedra on the GPU against the plain implementation (``plain_pinedra``): each mechanism alone, then whole models of several made-up
shapes stepped through the engine under every cutting, and generation through the scheduler.

The models' weights are drawn here, larger than a trained model's, so that a key that is wrongly seen or missed, a slope, a sink, a gate,
a bias or a factor that is left out, or a wrong expert moves the logits by much more than the tolerance."""
from __future__ import annotations

import json
import math

import numpy as np
import pytest
import torch
from safetensors.torch import save_file

import plain_pinedra as plain
import trace_tools
from test_parts_gpu import step_view
from test_zemavik_gpu import assert_logits, engine_for, fresh_cache, make_requests, on, run_part

pytestmark = pytest.mark.gpu

DEVICE = "cuda"


# ---------------------------------------------------------------------------------------
# made-up models
# ---------------------------------------------------------------------------------------
def moe(ff, experts, top, identity=0, groups=None, scale=1.0, shared=None):
    router = {"experts": experts, "top": top, "identity": identity, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def mixer(heads, kv_heads, dim, vdim, scale, **more):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, **more}


def first(sizes, mlp=None):
    return {"type": "attention", "mixer": mixer(*sizes), "mlp": mlp}


def second(sizes, temperature=None, mlp=None):
    more = {} if temperature is None else {"q_temp": {"coef": temperature[0], "every": temperature[1]}}
    return {"type": "attention_2", "mixer": mixer(*sizes, **more), "mlp": mlp}


def third(sizes, rot=None, cap=None, chunk=None, mlp=None):
    more = {}
    if rot is not None:
        more["rot"] = {"dims": rot[0], "base": rot[1]}
    if cap is not None:
        more["softcap"] = cap
    if chunk is not None:
        more["mask"] = {"size": chunk}
    return {"type": "attention_3", "mixer": mixer(*sizes, **more), "mlp": mlp}


def model(vocab, width, layers, loop=None, eps=1e-5, embedding=1.0):
    config = {"architecture": "Pinedra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": embedding}}
    if loop is not None:
        config["loop"] = dict(zip(("start", "stop", "times"), loop))
    return config


CONFIGS = {
    # values wider and narrower than keys, grouped heads, a loop in the middle; experts in groups with some that hand their input back, a shared
    # expert of more than one piece, of less than one, none, no feed-forward
    "mix": model(97, 72, [
        second((6, 2, 16, 24, 0.4), (0.7, 5), moe(24, 5, 3, identity=1, groups=(3, 2), scale=1.4, shared=40)),
        first((4, 2, 20, 20, 0.3), moe(16, 6, 2, identity=2, groups=(4, 2), scale=0.8, shared=8)),
        third((3, 1, 24, 8, 0.4), (12, 300.0), 3.0, 11, moe(32, 4, 2)),
        first((2, 1, 8, 8, 0.5)),
    ], loop=(1, 3, 2), embedding=1.5),
    # nothing a multiple of 8: heads, experts and the stream; one expert a token, one group, one value to a head, no cap, no chunk, no rotation;
    # the whole model three times; pages of 4
    "odd": model(61, 45, [
        third((4, 2, 10, 6, 0.5), (6, 50.0), None, 7, moe(9, 3, 1, identity=1, groups=(2, 1), scale=2.0, shared=13)),
        second((3, 3, 6, 1, 0.6), None, moe(11, 5, 1, groups=(1, 1), shared=11)),
        third((2, 2, 12, 20, 0.4), None, 5.0, None),
        first((3, 1, 14, 14, 0.3), moe(7, 2, 2, identity=3)),
        third((1, 1, 9, 9, 0.4), (8, 20.0), None, None),
    ], loop=(0, 5, 3), eps=1e-4),
    # the sizes at which prompts run on the tcgen05 kernels and decoded tokens on the TMA-fed ones: heads of 64 and (values of 96 kept wider)
    # 128, pages of 64, groups of one and of five heads; enough tokens an expert for the grouped product in the longest prompt
    "cores": model(130, 128, [
        second((4, 4, 64, 64, 0.15), (0.4, 50), moe(32, 3, 1, identity=1, groups=(2, 1), scale=1.3, shared=48)),
        first((10, 2, 64, 64, 0.12), moe(48, 4, 2, identity=1, shared=48)),
        third((6, 1, 128, 96, 0.12), (64, 5000.0), 6.0, 96, moe(40, 2, 1, shared=16)),
        second((6, 2, 128, 128, 0.1), (0.2, 30)),
    ], loop=(0, 2, 2), embedding=2.0),
    # a width at which decode products come as partial sums over slices of k and the stacked products run on the TMA-fed kernel
    "wide": model(112, 1024, [
        second((16, 4, 128, 128, 0.1), (0.3, 20), moe(256, 4, 2, identity=2, groups=(3, 2), scale=1.2, shared=256)),
        first((8, 2, 128, 128, 0.1), moe(1024, 3, 2, shared=512)),
        third((16, 2, 64, 64, 0.14), (32, 900.0), 8.0, 70),
    ]),
}
PAGE_SIZES = {"mix": 8, "odd": 4, "cores": 64, "wide": 64}
LENGTHS = {"mix": (61, 23, 5, 38, 1, 44, 17), "odd": (50, 9, 35, 2, 41), "cores": (330, 70, 3, 129), "wide": (150, 66, 9)}


def draw_mixer(rand, matrix, kind, m, width):
    """The tensors of a mixer, names below ``mix.``."""
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {"q": matrix(heads * dim, width, 1.5), "k": matrix(groups * dim, width, 1.5), "o": matrix(width, heads * vdim, 2.0),
         "g": matrix(heads if kind == "attention_3" else heads * vdim, width, 2.0)}
    if kind != "attention":
        w["v"] = matrix(groups * vdim, width)
    if kind == "attention":
        w.update({"q.b": 0.5 * rand(heads * dim), "k.b": 0.7 * rand(groups * dim), "o.b": 0.5 * rand(width), "q.norm": 1.5 + 0.5 * rand(heads * dim), "k.norm": 1.5 + 0.5 * rand(groups * dim)})
    elif kind == "attention_2":
        w.update({"q.norm": 1.5 + 0.5 * rand(dim), "k.norm": 1.5 + 0.5 * rand(dim)})
    else:
        w.update({"q.b": 0.5 * rand(heads * dim), "k.b": 0.5 * rand(groups * dim), "v.b": 0.7 * rand(groups * vdim)})
    return w


def draw_mixture(rand, matrix, mlp, width):
    router, ff = mlp["router"], mlp["expert"]["ff"]
    choices = router["experts"] + router.get("identity", 0)
    w = {"router": matrix(choices, width, 1.2), "correction": rand(choices) / choices - 0.2}
    for name, inner in [(f"e{e}.", ff) for e in range(router["experts"])] + ([] if mlp.get("shared") is None else [("shared.", mlp["shared"]["ff"])]):
        w[name + "gate"], w[name + "up"], w[name + "down"] = matrix(inner, width, 1.6), matrix(inner, width, 1.6), matrix(width, inner)
    return w


def drawing(seed):
    g = torch.Generator().manual_seed(seed)
    rand = lambda *shape: torch.randn(*shape, generator=g)
    return rand, lambda out, inner, gain=1.0: rand(out, inner) * gain / math.sqrt(inner)


def draw_weights(config, seed):
    rand, matrix = drawing(seed)
    width = config["width"]
    w = {"embed": rand(config["vocab"], width), "head": matrix(config["vocab"], width), "final.norm": 1 + 0.3 * rand(1)[0]}
    for index, one in enumerate(config["layers"]):
        w[f"l{index}.norm1"] = 0.8 + 0.2 * torch.rand((), generator=torch.Generator().manual_seed(seed + index))
        w.update({f"l{index}.mix.{key}": value for key, value in draw_mixer(rand, matrix, one["type"], one["mixer"], width).items()})
        if one["mlp"] is not None:
            w.update({f"l{index}.mlp.{key}": value for key, value in draw_mixture(rand, matrix, one["mlp"], width).items()})
    return {key: value.to(torch.bfloat16).contiguous() for key, value in w.items()}


def every_expert(config):
    """The same model with every token going through all of a layer's choices: no choice is left that rounding could turn."""
    out = json.loads(json.dumps(config))
    for one in out["layers"]:
        if one["mlp"] is not None:
            router = one["mlp"]["router"]
            router["top"] = router["experts"] + router["identity"]
            router.pop("groups", None)
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (folder, config, weights as stored); under ``name + "/all"`` the same weights with a configuration in which every choice is
    used: a 16-bit run is compared on the latter, since a rounded input turns a close choice now and then."""
    made = {}
    for seed, (name, config) in enumerate(CONFIGS.items()):
        weights = draw_weights(config, 700 + seed)
        for key, stored in ((name, config), (name + "/all", every_expert(config))):
            folder = tmp_path_factory.mktemp("pinedra_" + name)
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


def test_layer_run_by_layer_run_in_32_bit(models):
    from pylon_b200.engine import StepEntry

    folder, config, weights = models["mix"]
    tokens = make_requests(config, (37,), seed=5)["r0"]
    want: list = []
    plain.forward(config, weights, tokens, taps=want)
    engine = engine_for(folder, "float32", 8, 64)
    taps: list = []
    forward = engine.model.forward
    engine.model.forward = lambda step, caches: forward(step, caches, taps)
    request = engine.open("a", len(tokens))
    engine.step([StepEntry(request, tokens, [0])])
    assert len(taps) == len(want) == 6
    for index, (got, expected) in enumerate(zip(taps, want)):
        torch.testing.assert_close(got.double().cpu(), expected, rtol=1e-4, atol=1e-4 * float(expected.abs().max()), msg=lambda m: f"layer run {index}: {m}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_over_many_pages_chunks_and_steps_of_the_factor(models, dtype):
    """A short prompt, then 200 tokens one by one."""
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
# mixers alone
# ---------------------------------------------------------------------------------------
SIZES = {"narrow": (4, 2, 20, 12, 0.35), "equal": (6, 2, 32, 32, 0.3), "wider": (3, 1, 8, 24, 0.5), "cores": (8, 2, 64, 64, 0.15), "odd": (2, 2, 5, 3, 0.35)}
MIXER_NAMES = ["attention-equal", "attention-odd", "attention-cores", "attention_2-narrow", "attention_2-wider", "attention_2-cores", "attention_2-odd",
               "attention_3-narrow", "attention_3-wider", "attention_3-cores", "attention_3-odd"]


def built(name, dtype, seed=21, width=56, eps=1e-5):
    """(the mixer part of a small made-up model, its tensors, the plain function, the source of random numbers)."""
    from pylon_b200.config.model_config import PinedraConfig
    from pylon_b200.models.pinedra import pinedra_spec
    from pylon_b200.parts import MIXERS

    kind, sizes = name.split("-")
    sizes = SIZES[sizes]
    if kind == "attention":
        sizes = (*sizes[:3], sizes[2], sizes[4])
    dim = sizes[2]
    one = {"attention": first(sizes), "attention_2": second(sizes, (0.6, 9)), "attention_3": third(sizes, (dim // 4 * 2, 300.0), 2.5, 9)}[kind]
    rand, matrix = drawing(seed)
    w = {key: value.to(torch.bfloat16) for key, value in draw_mixer(rand, matrix, kind, one["mixer"], width).items()}
    spec = pinedra_spec(PinedraConfig.from_dict(model(11, width, [one], eps=eps)), 256)
    part = MIXERS.build(spec.layers[0].block.params["mixer"])
    declared = {d.name: d for d in part.tensors()}
    assert set(declared) == set(w) and all(tuple(w[k].shape) == tuple(declared[k].shape) for k in w)
    part.load({k: on(v, torch.float32 if declared[k].role == "vector" else dtype) for k, v in w.items()}, dtype, torch.device(DEVICE))
    return part, w, lambda h: plain.MIXERS[kind](h.double(), {k: v.double() for k, v in w.items()}, "", one["mixer"], eps), rand


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", MIXER_NAMES)
def test_each_mixer_alone_against_its_plain_statement(name, dtype):
    """A mixer part from its input to its output: a prompt in one step, then the same in portions that end at, before and behind the edges of
    chunks and pages, and token by token from the start."""
    part, w, oracle, rand = built(name, dtype)
    count, page = 60, 64 if "cores" in name else 8
    h = rand(count, 56).to(dtype)
    want = oracle(h)
    spread = float(want.std())
    limit = 0.06 * spread if dtype == torch.bfloat16 else 1e-4 * spread
    for cutting in ((count,), (20, 2, 1, 1, 28, 8), (1,) * 12 + (2, 2, 44), (9, 9, 9, 33), (8, 1, 9, 42), (2,) * 30, (1,) * count):
        got = run_part(part, h, cutting, page, dtype)
        assert float((got - want).abs().max()) <= limit, f"{name}, {cutting}: off by {float((got - want).abs().max()):.3g} of {spread:.3g}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", MIXER_NAMES)
def test_unequal_requests_in_one_step_against_each_alone(name, dtype):
    """Three requests of 1, 17 and 6 new tokens at different places of their sequences in one step, in pages that another request used
    before, with a padding token behind them: every request's result is the one it has alone."""
    part, w, oracle, rand = built(name, dtype, seed=8)
    page = 64 if "cores" in name else 8
    before, new = (12, 0, 30), (1, 17, 6)
    inputs = [rand(b + n, 56).to(dtype) for b, n in zip(before, new)]
    want = [oracle(h) for h in inputs]
    cache = fresh_cache(part.cache_need(), page, dtype, table=tuple(range(15)))
    cache.block_table = torch.tensor([[9, 3, 12, 0, 7], [1, 14, 5, 10, 2], [6, 11, 4, 13, 8]], device=DEVICE, dtype=torch.int32)
    cache.k_pages.fill_(3.0)                               # what an earlier request left in the pages
    cache.v_pages.fill_(-2.0)

    def run(rows, sizes, starts, padding=0):
        step = step_view(sizes, starts, dtype)
        h = torch.cat([inputs[r][s : s + n] for r, n, s in zip(rows, sizes, starts)] + [torch.full((padding, 56), 4.0, dtype=dtype)])
        step.positions = torch.nn.functional.pad(step.positions, (0, padding))
        step.token_row = torch.nn.functional.pad(step.token_row, (0, padding), value=-1)
        step.num_tokens += padding
        saved = cache.block_table
        cache.block_table = saved[list(rows)].contiguous()
        out = part.forward(on(h), step, cache)
        cache.block_table = saved
        return (out.sum(dim=0) if out.dim() == 3 else out).double().cpu()

    for r in (0, 2):                                           # what the requests hold already, each alone
        run((r,), (before[r],), (0,))
    got = run((0, 1, 2), new, before, padding=1)
    spread = float(torch.cat(want).std())
    limit = 0.06 * spread if dtype == torch.bfloat16 else 1e-4 * spread
    cursor = 0
    for r in range(3):
        mine = got[cursor : cursor + new[r]]
        cursor += new[r]
        worst = float((mine - want[r][before[r] :]).abs().max())
        assert worst <= limit, f"{name}: request {r} in the batch is off by {worst:.3g} of {spread:.3g}"


# ---------------------------------------------------------------------------------------
# attention: a softmax with slopes, a sink, gates
# ---------------------------------------------------------------------------------------
def in_pages(keys, values, page, dtype, seed=5, spare=3):
    """``[T, kv_heads, size]`` keys and values of one request in shuffled pages: (key pages, value pages, block table)."""
    needed = -(-keys.shape[0] // page)
    order = torch.randperm(needed + spare, generator=torch.Generator().manual_seed(seed))[:needed]
    k_pages, v_pages = (torch.full((needed + spare, rows.shape[1], page, rows.shape[2]), 5.0) for rows in (keys, values))
    for logical, physical in enumerate(order.tolist()):
        for rows, pages in ((keys, k_pages), (values, v_pages)):
            part = rows[logical * page : (logical + 1) * page]
            pages[physical, :, : part.shape[0]] = part.transpose(0, 1)
    return on(k_pages, dtype), on(v_pages, dtype), on(order[None].to(torch.int32))


def plain_attention(q, k, v, scale, slopes=None, sinks=None, chunk=None, cap=None):
    """All of it at once, in float64: ``q [T, H, d]``, ``k``/``v [T, G, *]`` -> ``[T, H, dv]``."""
    count, heads = q.shape[:2]
    k, v = (t.repeat_interleave(heads // t.shape[1], dim=1) for t in (k, v))
    index = torch.arange(count)
    seen = index[:, None] >= index[None, :]
    if chunk is not None:
        seen &= index[:, None] // chunk == index[None, :] // chunk
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s if cap is None else cap * torch.tanh(s / cap)
    if slopes is not None:
        s = s - slopes[:, None, None] * (index[:, None] - index[None, :])
    s = s.masked_fill(~seen, -math.inf)
    top = s.amax(dim=-1, keepdim=True)
    if sinks is not None:
        top = torch.maximum(top, sinks[:, None, None])
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True) + (torch.exp(sinks[:, None, None] - top) if sinks is not None else 0.0)
    return torch.einsum("hij,jhd->ihd", e / total, v)


FORMS = [(torch.float32, 24, 2, 16), (torch.bfloat16, 24, 2, 16), (torch.bfloat16, 48, 4, 16), (torch.bfloat16, 64, 1, 64), (torch.bfloat16, 64, 5, 64), (torch.bfloat16, 128, 4, 64),
         (torch.bfloat16, 256, 2, 64)]


@pytest.mark.parametrize("gated", ["heads", "elements"])
@pytest.mark.parametrize("dtype,dim,group,page", FORMS)
def test_keys_that_stand_out_against_slopes_a_sink_and_chunks(dtype, dim, group, page, gated):
    """Hundreds of keys of scores around -2, and four that stand out with values of their own: the first key, the last of a page, the first of
    the next, one in the middle (at the end of a chunk) and its neighbour behind the edge.  With slopes that a far key must overcome and a sink
    that takes a good part, with chunks and a cap, with neither; as one prompt, with a tail token by token, in portions that end at the keys and
    in portions of two; gated, times a factor, into a slice of wider rows whose edges stay as they are."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(5)
    count, kv_heads = 300, 2
    heads = kv_heads * group
    places = (0, 2 * page - 1, 2 * page, 199, 200)
    keys = torch.randn(count, kv_heads, dim, generator=g) * 0.1 - 0.1
    values = torch.randn(count, kv_heads, dim, generator=g) * 0.5
    for n, place in enumerate(places):
        keys[place] = 1.0
        values[place] = torch.linspace(-4.0, 4.0, dim) * (1 if n % 2 else -1) + n
    queries = 1.0 + torch.randn(count, heads, dim, generator=g) * 0.1
    scale, factor = 18.0 / dim, 0.6
    slopes = torch.tensor([0.02 + 0.05 * h / heads for h in range(heads)])
    sinks = torch.linspace(8.0, 19.0, heads)
    gate = torch.randn(count, heads if gated == "heads" else heads * dim, generator=g)
    q, k, v, gates = (t.to(dtype).double() for t in (queries, keys, values, gate))
    k_pages, v_pages, table = in_pages(keys, values, page, dtype)

    def run(cutting, options):
        outs, cursor = [], 0
        for size in cutting:
            step = step_view((size,), (cursor,), dtype)
            wide = torch.full((size, heads * dim + 24), 9.0, device=DEVICE, dtype=dtype)
            mine = slice(cursor, cursor + size)
            ops.paged_attention(on(queries[mine].to(dtype)).view(size, heads * dim), k_pages, v_pages, step.positions, step.token_row, step.q_start, step.kv_len, table,
                                heads, step.max_q, step.max_kv, scale=scale, head_gate=on(gate[mine].to(dtype)), out_factor=factor, out=wide[:, 8 : 8 + heads * dim],
                                rows_alike=cursor % 2 == 0, **options)
            assert float(wide[:, :8].min()) == 9.0 == float(wide[:, 8 + heads * dim :].max())
            outs.append(wide[:, 8 : 8 + heads * dim])
            cursor += size
        return torch.cat(outs).double().cpu()

    tolerance = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-4)
    for options in ({"slopes": slopes, "sinks": sinks}, {"chunk": 100, "cap": 25.0, "sinks": sinks}, {"slopes": slopes, "chunk": 40, "cap": 30.0}, {}):
        want = plain_attention(q, k, v, scale, **{key: value.double() if torch.is_tensor(value) else value for key, value in options.items()})
        opened = plain.sigmoid(gates)
        want = (want * (opened[..., None] if gated == "heads" else opened.view(count, heads, dim)) * factor).reshape(count, heads * dim)
        given = {"distance_slopes": on(options["slopes"]) if "slopes" in options else None, "sinks": on(options["sinks"]) if "sinks" in options else None,
                 "chunk": options.get("chunk"), "softcap": options.get("cap")}
        for cutting in ((count,), (count - 40,) + (1,) * 40, (1, 2 * page - 2, 1, 1, count - 2 * page - 1), (2 * page, 200 - 2 * page, 1, 99), (2,) * 150, (190, 20, 20, 70)):
            assert sum(cutting) == count
            torch.testing.assert_close(run(cutting, given), want, **tolerance, msg=lambda m: f"{options.keys()}, {cutting[:6]}: {m}")
    ops.raise_on_kernel_errors(torch.device(DEVICE))


@pytest.mark.parametrize("dtype,dim,group,page", FORMS)
def test_a_sink_is_met_once_however_the_keys_are_dealt_out(dtype, dim, group, page):
    """All scores equal c and all values one: the output is n / (n + exp(sink - c)), whatever n is - for rows of one tile and of many, requests of
    equal lengths (clusters of blocks) and of unequal ones (runs), prompts with their keys in splits, one decode block and all of them."""
    from pylon_b200.kernels import ops

    kv_heads, c = 2, -1.5
    heads = kv_heads * group
    sinks = torch.linspace(-3.0, 6.0, heads)
    q_row = torch.zeros(dim)
    q_row[0] = c
    for lengths in ((1,), (3,), (70,), (1000,), (1000, 990, 1000), (1, 640, 17, 64, 65, 2)):
        longest, rows = max(lengths), len(lengths)
        width = -(-longest // page)
        k_pages = torch.zeros(rows * width, kv_heads, page, dim, device=DEVICE, dtype=dtype)
        k_pages[..., 0] = 1.0
        v_pages = torch.ones_like(k_pages)
        table = torch.randperm(rows * width, generator=torch.Generator().manual_seed(1)).view(rows, width).to(torch.int32).to(DEVICE)
        for new in {1, min(3, min(lengths)), min(lengths)}:
            step = step_view((new,) * rows, tuple(n - new for n in lengths), dtype)
            q = q_row.repeat(new * rows, heads).to(dtype).to(DEVICE)
            seen = (step.positions.double().cpu() + 1.0)[:, None]
            want = (seen / (seen + torch.exp(sinks.double() - c))).repeat_interleave(dim, dim=1)
            for more in ({}, {"rows_alike": True}, {"num_splits": 3}, {"prefill_kernel": "mma"}, {"decode_blocks": 1}, {"decode_blocks": 7}):
                got = ops.paged_attention(q, k_pages, v_pages, step.positions, step.token_row, step.q_start, step.kv_len, table, heads, step.max_q, step.max_kv, scale=1.0,
                                          sinks=on(sinks), split_weights=True, **more)
                torch.testing.assert_close(got.double().cpu(), want, **(dict(rtol=6e-3, atol=1e-4) if dtype == torch.bfloat16 else dict(rtol=1e-5, atol=1e-6)), msg=lambda m: f"{lengths}, {new}, {more}: {m}")
    ops.raise_on_kernel_errors(torch.device(DEVICE))


@pytest.mark.parametrize("dim,page", [(64, 64), (128, 64), (48, 16)])
def test_weights_count_with_more_than_eight_bits(dim, page):
    """Half of the keys have the value 1 and a weight of one, half -1 and a weight just below it: what is left is the difference of the weights,
    which a rounding to eight bits would turn into another number or nothing."""
    from pylon_b200.kernels import ops

    count = 512
    for gap in (2.0 ** -9, 3.3e-3, 7e-3):
        keys, values = torch.zeros(count, 1, dim), torch.ones(count, 1, dim)
        keys[1::2, 0, 0] = -gap
        values[1::2] = -1.0
        k_pages, v_pages, table = in_pages(keys, values, page, torch.bfloat16)
        stored = float(keys[1, 0, 0].to(torch.bfloat16))
        w = math.exp(stored)
        q_row = torch.zeros(dim)
        q_row[0] = 1.0
        for size in (200, 2, 1):
            step = step_view((size,), (count - size,), torch.bfloat16)
            q = q_row.repeat(size, 4).to(torch.bfloat16).to(DEVICE)
            got = ops.paged_attention(q, k_pages, v_pages, step.positions, step.token_row, step.q_start, step.kv_len, table, 4, step.max_q, step.max_kv, scale=1.0, split_weights=True)
            assert abs(float(got[-1].double().mean()) - (1 - w) / (1 + w)) < 2e-5, (gap, size)      # eight bits would be off by up to 2e-3


# ---------------------------------------------------------------------------------------
# between projections and attention
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("norm,rot,from_keys", [("whole", 0, True), ("whole", 8, False), ("before", 0, False), (None, 16, True), ("after", 16, False)])
@pytest.mark.parametrize("nq,nkv,dim,vdim,own", [(3, 1, 16, 16, 16), (6, 2, 48, 48, 40), (16, 4, 128, 128, 128), (2, 2, 20, 20, 17), (5, 5, 64, 64, 64)])
def test_biases_norms_factors_and_values_from_the_keys(nq, nkv, dim, vdim, own, norm, rot, from_keys, dtype):
    """The kernel between projections and attention against plain arithmetic: biases, the norm per head or over whole rows (heads whose own
    elements are fewer than the ones kept), rotation, a factor by position on the queries, values that are the keys before all of that; a
    slice of wider rows, a token of no request, a page that others used."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(dim + nq)
    tokens, page = 9, 4
    columns = (nq + nkv) * dim + (0 if from_keys else nkv * vdim)
    stored = torch.randn(tokens, columns + 8, generator=g).to(dtype)
    bias = torch.randn(columns, generator=g)
    for rows in (stored[:, : (nq + nkv) * dim].view(tokens, nq + nkv, dim), bias[: (nq + nkv) * dim].view(nq + nkv, dim)):
        rows[..., own:] = 0.0
    positions = torch.tensor([5, 6, 7, 8, 9, 0, 0, 1, 2], dtype=torch.int32)
    row = torch.tensor([0, 0, 0, 0, 0, -1, 1, 1, 1], dtype=torch.int32)
    table = torch.tensor([[4, 2, 0], [3, 1, 5]], dtype=torch.int32)
    angle = torch.rand(16, max(rot // 2, 1), generator=g) * 6
    factors = 1.0 + torch.rand(16, generator=g)
    sizes = (nq, nkv) if norm == "whole" else (1, 1)
    weights = [(torch.rand(heads, dim, generator=g) + 0.5) * (torch.arange(dim) < own) for heads in sizes]
    k_pages, v_pages = (torch.full((6, nkv, page, size), 7.0, device=DEVICE, dtype=dtype) for size in (dim, vdim))
    work = on(stored.clone())
    ops.qkv_rotate_write(work[:, :columns], on(bias), on(angle.cos()) if rot else None, on(angle.sin()) if rot else None, rot, "halves", norm, on(weights[0].reshape(-1)), on(weights[1].reshape(-1)),
                         1e-3, on(positions), on(row), on(table), page, k_pages, v_pages, nq, nkv, dim, vdim, norm_size=own, values_from_keys=from_keys, q_factors=on(factors))
    whole = stored[:, :columns].double() + bias.double()
    q, k = whole[:, : nq * dim].view(tokens, nq, dim), whole[:, nq * dim : (nq + nkv) * dim].view(tokens, nkv, dim)
    values = k if from_keys else whole[:, (nq + nkv) * dim :].view(tokens, nkv, vdim)

    def normed(x, weight):
        over = (x * x).sum(dim=-1, keepdim=True) / own
        return x / torch.sqrt((over.mean(dim=1, keepdim=True) if norm == "whole" else over) + 1e-3) * weight.double()

    def turned(x):
        if not rot:
            return x
        c, s = angle.cos().double()[positions.long()][:, None], angle.sin().double()[positions.long()][:, None]
        u, v = x[..., : rot // 2], x[..., rot // 2 : rot]
        return torch.cat((u * c - v * s, v * c + u * s, x[..., rot:]), dim=-1)

    results = []
    for x, weight in ((q, weights[0]), (k, weights[1])):
        x = normed(x, weight) if norm in ("before", "whole") else x
        x = turned(x)
        results.append(normed(x, weight) if norm == "after" else x)
    results[0] = results[0] * factors.double()[positions.long()][:, None, None]
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=1e-5, atol=1e-5)
    for t in range(tokens):
        if row[t] < 0:
            assert torch.equal(work[t].cpu(), stored[t])
            continue
        torch.testing.assert_close(work[t, : nq * dim].double().cpu().view(nq, dim), results[0][t], **tol)
        physical, place = int(table[row[t], positions[t] // page]), int(positions[t]) % page
        torch.testing.assert_close(k_pages[physical, :, place].double().cpu(), results[1][t], **tol)
        torch.testing.assert_close(v_pages[physical, :, place].double().cpu(), values[t], **tol)
    assert torch.equal(work[:, columns:].cpu(), stored[:, columns:])
    ops.raise_on_kernel_errors(torch.device(DEVICE))


# ---------------------------------------------------------------------------------------
# feed-forward, and what joins the stream
# ---------------------------------------------------------------------------------------
def built_mixture(mlp, width, dtype, seed=17):
    from pylon_b200.config.model_config import PinedraConfig
    from pylon_b200.models.pinedra import pinedra_spec
    from pylon_b200.parts import FEED_FORWARDS

    rand, matrix = drawing(seed)
    w = {key: value.to(torch.bfloat16) for key, value in draw_mixture(rand, matrix, mlp, width).items()}
    spec = pinedra_spec(PinedraConfig.from_dict(model(11, width, [first((1, 1, 8, 8, 1.0), mlp)])), 8)
    part = FEED_FORWARDS.build(spec.layers[0].block.params["feed_forward"])
    declared = {d.name: d for d in part.tensors()}
    assert set(declared) == set(w) and all(tuple(w[k].shape) == tuple(declared[k].shape) for k in w)
    part.load({k: on(v, torch.float32 if declared[k].role == "vector" else dtype) for k, v in w.items()}, dtype, torch.device(DEVICE))
    return part, {k: v.double() for k, v in w.items()}, rand


def margin(scores, correction, top, groups):
    """By how much a token's choice scores would have to change to turn a choice: between experts, and between groups."""
    value = (scores + correction).sort(descending=True).values
    least = math.inf
    if groups is not None and groups["keep"] < groups["count"]:
        worth = (scores + correction).view(groups["count"], -1).amax(dim=1)
        order = worth.sort(descending=True)
        least = float(order.values[groups["keep"] - 1] - order.values[groups["keep"]])
        kept = set(order.indices[: groups["keep"]].tolist())
        size = scores.shape[0] // groups["count"]
        value = torch.stack([s for e, s in enumerate(scores + correction) if e // size in kept]).sort(descending=True).values
    return min(least, float(value[top - 1] - value[top])) if top < value.shape[0] else least


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,tokens,mlp", [
    (40, 1, moe(12, 3, 1, identity=1, groups=(2, 1), scale=1.7, shared=12)), (56, 7, moe(20, 6, 6)), (48, 150, moe(24, 10, 3, identity=2, groups=(4, 2), scale=0.5, shared=60)),
    (128, 70, moe(64, 30, 3, identity=6, groups=(36, 5), shared=8)), (64, 40, moe(40, 1, 3, identity=3, scale=2.0)), (256, 700, moe(136, 4, 2, identity=2, groups=(3, 2), scale=1.4, shared=200)),
    (384, 600, moe(256, 3, 1, identity=1, groups=(2, 1), shared=256)), (72, 90, moe(9, 5, 2, identity=1, shared=20)), (64, 20, moe(1024, 3, 2, shared=1024)), (64, 33, moe(16, 60, 4, identity=4, groups=(8, 3)))])
def test_the_mixture_against_token_by_token(width, tokens, mlp, dtype):
    """Softmax scores over all, a correction that turns choices and never weighs, groups worth their best, experts that hand their input back, a
    factor, a shared expert of less than one piece and of several: one token, few and many; two shapes have enough tokens an expert for the
    grouped tensor-core product.  Tokens whose choice hangs on a margin that 16-bit rounding of the input can turn are left out there."""
    part, w, rand = built_mixture(mlp, width, dtype)
    h = rand(tokens, width).to(dtype)
    want = plain.mixture(h.double(), w, "", mlp)
    router = mlp["router"]
    scores = torch.softmax(h.double() @ w["router"].T, dim=1)
    close = 1e-6 if dtype == torch.float32 else 2e-3 / scores.shape[1] ** 0.5
    sure = torch.tensor([margin(row, w["correction"], router["top"], router.get("groups")) > close for row in scores])
    assert int(sure.sum()) >= 0.7 * tokens
    chosen = [plain.choose(row, w["correction"], router["top"], router.get("groups")) for row in scores]
    if router["identity"] and tokens > 5:
        assert any(e >= router["experts"] for row in chosen for e in row)
    step = step_view((tokens,), (0,), dtype)
    out = part.forward(on(h), step)
    got = (out.sum(dim=0) if out.dim() == 3 else out).double().cpu()
    spread = float(want.std())
    assert float((got - want)[sure].abs().max()) <= (0.06 * spread if dtype == torch.bfloat16 else 1e-4 * spread)
    # the rows where the experts left them, for a reader that adds them up itself
    loose = part.forward_scattered(on(h), step)
    rows = (loose.rows.sum(dim=0) if loose.rows.dim() == 3 else loose.rows).double().cpu()
    slots = loose.slot_of.long().cpu().view(tokens, loose.top)
    together = (rows[slots.clamp(min=0)] * loose.share.double().cpu()[..., None] * (slots >= 0)[..., None]).sum(dim=1)
    if loose.same is not None:
        together += loose.same.double().cpu() * loose.same_share.double().cpu()[:, None]
    torch.testing.assert_close(together, got, rtol=1e-5, atol=1e-5)
    assert (slots < 0).any() == any(e >= router["experts"] for row in chosen for e in row) or not sure.all()
    # the same tokens in another order and among others: a token's result does not depend on its place in the step
    order = torch.randperm(tokens, generator=torch.Generator().manual_seed(1))
    again = part.forward(on(torch.cat([h[order], rand(5, width).to(dtype)])), step_view((tokens + 5,), (0,), dtype))
    again = (again.sum(dim=0) if again.dim() == 3 else again).double().cpu()[:tokens]
    if tokens + 5 < 512 or tokens >= 512:      # (the same kernels either way)
        assert torch.equal(again, got[order])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [1, 30, 72, 200, 2048, 4096, 8192, 9000, 16384])
def test_outputs_side_by_side_join_the_stream_in_one_pass(width, dtype):
    """Every form of the two outputs - a block, partial sums of one part to five, rows in slots with and without shares, some of them nowhere, rows
    handed back, nothing - with and without a bias, with the norm, without it, and with a selection of rows that leaves the stream as it is."""
    from pylon_b200.kernels import ops

    g = torch.Generator().manual_seed(width)
    rand = lambda *shape: torch.randn(*shape, generator=g)
    tokens, slots, top, eps = 5, 23, 3, 1e-3
    weight, bias = torch.rand(width, generator=g) + 0.5, rand(width)
    slot_of = torch.randperm(slots, generator=g)[: tokens * top].to(torch.int32)
    slot_of[[1, 7]] = -1
    share, same_share = torch.rand(tokens, top, generator=g), torch.rand(tokens, generator=g)
    same_share[2] = 0.0
    same = rand(tokens, width + 8).to(dtype)

    def added(rows):
        return (rows.double().sum(dim=0) if rows.dim() == 3 else rows.double())

    def scattered(rows, shares, back):
        mine = slot_of.long().view(tokens, top)
        total = (added(rows)[mine.clamp(min=0)] * (mine >= 0)[..., None] * (share.double()[..., None] if shares else 1.0)).sum(dim=1)
        if back:
            total = total + same[:, :width].double() * same_share.double()[:, None]
        return total, ops.ScatteredRows(on(rows), on(slot_of), top, on(share) if shares else None, on(same)[:, :width] if back else None, on(same_share) if back else None)

    block = lambda: rand(tokens, width).to(dtype)
    parts = lambda n, rows=tokens: rand(n, rows, width)
    seconds = [(0.0, None)]
    for rows in (block(), parts(1), parts(4)):
        seconds.append((added(rows), on(rows)))
    for rows, shares, back in ((rand(slots, width).to(dtype), True, True), (parts(2, slots), True, False), (parts(5, slots), False, True)):
        seconds.append(scattered(rows, shares, back))
    tol = dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)
    for index, (amount, second_output) in enumerate(seconds):
        output = (block(), parts(1), parts(3), parts(5))[index % 4]
        use_bias = index % 2 == 1
        residual = rand(tokens, width)
        want = residual.double() + added(output) + amount + (bias.double() if use_bias else 0.0)
        joined = ops.SideBySide(on(output), on(bias) if use_bias else None, second_output)
        normed = plain.rms_unit(want, eps) * weight.double()
        pick = torch.tensor([3, 0, 3], dtype=torch.int32)
        held = on(residual.clone())
        got = ops.join_norm(held, joined, on(weight), eps, dtype, rows=on(pick))
        assert torch.equal(held.cpu(), residual)
        torch.testing.assert_close(got.double().cpu(), normed[pick.long()], **tol)
        got = ops.join_norm(held, joined, on(weight), eps, dtype)
        torch.testing.assert_close(held.double().cpu(), want, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(got.double().cpu(), normed, **tol)
        held = on(residual.clone())
        assert ops.join_norm(held, joined) is None
        torch.testing.assert_close(held.double().cpu(), want, rtol=1e-5, atol=1e-5)


def test_what_was_left_side_by_side_joins_also_for_norms_without_such_a_kernel():
    from pylon_b200.kernels import ops
    from pylon_b200.parts import NORMS, PartSpec, ResidualStream

    g = torch.Generator().manual_seed(2)
    x, y, z, bias = (torch.randn(4, 24, generator=g) for _ in range(4))
    want = x.double() + y.double() + z.double() + bias[0].double()
    for kind in ("layernorm", "rmsnorm", "dynamic_tanh"):
        params = {"width": 24} if kind == "dynamic_tanh" else {"width": 24, "eps": 1e-5}
        norm = NORMS.build(PartSpec(kind, params))
        norm.load({d.name: on(torch.full(d.shape, 0.7)) for d in norm.tensors()}, torch.float32, torch.device(DEVICE))
        for then in ("norm", "total", "another"):
            stream = ResidualStream(on(x.clone()))
            stream.add_together(ops.SideBySide(on(y), on(bias[0]), on(z)))
            expected = want
            if then == "another":
                stream.add(on(z))
                expected = want + z.double()
            if then != "total":
                norm.apply(stream)
            torch.testing.assert_close(stream.total().double().cpu(), expected, rtol=1e-5, atol=1e-5)


def test_a_mixer_with_an_output_bias_in_a_block_that_adds_one_output_at_a_time():
    """``forward`` alone gives everything, the bias included, whatever form the product has."""
    for dtype, limit in ((torch.float32, 1e-4), (torch.bfloat16, 0.06)):
        part, w, oracle, rand = built("attention-equal", dtype, width=1024)
        h = rand(6, 1024).to(dtype)
        cache = fresh_cache(part.cache_need(), 8, dtype)
        step = step_view((6,), (0,), dtype)
        whole = part.forward(on(h), step, cache)
        output, bias = part.forward_unjoined(on(h), step, cache)
        assert bias is not None and torch.equal(bias.cpu(), w["o.b"].float())
        want = oracle(h)
        for got in (whole.sum(dim=0) if whole.dim() == 3 else whole, (output.sum(dim=0) if output.dim() == 3 else output).float() + bias):
            assert float((got.double().cpu() - want).abs().max()) <= limit * float(want.std())
