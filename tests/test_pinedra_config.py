"""Pinedra without a GPU: its configuration, the model description built from it (tensor names and shapes, what each run keeps between
steps), how a stacked mixer and a shared expert lie in their matrices, and what the parts refuse."""
from __future__ import annotations

import copy
import json
import math

import pytest
import torch

import plain_pinedra as plain
from pylon_b200.cache.manager import CacheManager
from pylon_b200.config.model_config import ConfigError, PinedraConfig
from pylon_b200.config.registry import ARCHITECTURES, architecture_of, read_config
from pylon_b200.models.decoder import DecoderModel
from pylon_b200.parts import FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, PartSpec
from pylon_b200.parts.base import KVNeed

CONFIG = {
    "architecture": "Pinedra", "vocab": 70, "width": 40, "embedding": {"scale": 2.5}, "norm": {"eps": 1e-4},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        {"type": "attention_3", "mixer": {"heads": 6, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.3, "rot": {"dims": 8, "base": 50.0}, "softcap": 4.0, "mask": {"size": 9}},
         "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2, "scale": 0.75, "identity": 1, "groups": {"count": 3, "keep": 2}}, "shared": {"ff": 30}}},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 10, "scale": 0.2}, "mlp": None},
        {"type": "attention_2", "mixer": {"heads": 3, "kv_heads": 3, "dim": 16, "vdim": 8, "scale": 0.25, "q_temp": {"coef": 0.3, "every": 7}},
         "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 4, "top": 4, "scale": 2.0, "identity": 0}}},
        {"type": "attention_3", "mixer": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0}, "mlp": None},
    ],
}


def built(data=CONFIG, max_positions=64):
    config = PinedraConfig.from_dict(data)
    return config, ARCHITECTURES["Pinedra"].build_spec(config, max_positions)


def draw(part, dtype, seed=1):
    g = torch.Generator().manual_seed(seed)
    return {d.name: torch.randn(*d.shape, generator=g).to(torch.float32 if d.role == "vector" else dtype) for d in part.tensors()}


def test_the_configuration_reads_every_key_and_writes_it_back():
    config = PinedraConfig.from_dict(CONFIG)
    assert (config.vocab, config.width, config.embedding_scale, config.norm_eps, config.loop) == (70, 40, 2.5, 1e-4, (1, 3, 3))
    third, first, second, bare = config.layers
    assert (third.mixer.kind, third.mixer.heads, third.mixer.kv_heads, third.mixer.dim, third.mixer.vdim, third.mixer.scale) == ("attention_3", 6, 2, 12, 20, 0.3)
    assert (third.mixer.rot.dims, third.mixer.rot.base, third.mixer.softcap, third.mixer.chunk) == (8, 50.0, 4.0, 9)
    assert (third.mlp.ff, third.mlp.experts, third.mlp.top, third.mlp.scale, third.mlp.identity, third.mlp.groups, third.mlp.groups_keep, third.mlp.shared_ff) == (24, 5, 2, 0.75, 1, 3, 2, 30)
    assert first.mlp is None and first.mixer.kind == "attention"
    assert second.mixer.temperature == (0.3, 7.0) and (second.mlp.groups, second.mlp.shared_ff, second.mlp.identity) == (None, None, 0)
    assert (bare.mixer.rot, bare.mixer.softcap, bare.mixer.chunk) == (None, None, None)
    assert config.to_dict() == CONFIG
    assert PinedraConfig.from_dict(json.loads(json.dumps(config.to_dict()))) == config


def test_the_registry_finds_the_architecture(tmp_path):
    assert architecture_of(CONFIG) is ARCHITECTURES["Pinedra"]
    (tmp_path / "config.json").write_text(json.dumps(CONFIG))
    architecture, config = read_config(tmp_path)
    assert architecture.name == "Pinedra" and isinstance(config, PinedraConfig)


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="other"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "cannot be grouped"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0.0), "scale must be positive"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "exceeds"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 2.0}), "not scaled"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "must be positive"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=12), "vdim must be dim"),
    (lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=0), "every must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=2), "7 experts in 3 groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "negative"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "cannot use 5"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "are kept"),
    (lambda c: c["layers"][0].update(mlp=3), "an object or null"),
    (lambda c: c.update(loop={"start": 2, "stop": 9, "times": 1}), "does not fit"),
    (lambda c: c["norm"].update(eps=0.0), "norm.eps"),
    (lambda c: c.update(layers=[]), "at least one layer"),
])
def test_what_the_configuration_refuses(change, text):
    data = copy.deepcopy(CONFIG)
    change(data)
    with pytest.raises(ConfigError, match=text):
        PinedraConfig.from_dict(data)


def test_the_run_order_repeats_the_loop_and_adds_the_embedding_before_every_pass_but_the_first():
    config, spec = built()
    order = [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert config.run_order() == order == plain.run_order(CONFIG)
    assert [(run.layer, run.add_embedding) for run in spec.order] == order
    assert spec.embedding_scale == 2.5 and spec.lm_head_name == "head"
    for change in (None, {"start": 1, "stop": 1, "times": 4}, {"start": 0, "stop": 4, "times": 1}):
        data = copy.deepcopy(CONFIG)
        data["loop"] = change
        assert PinedraConfig.from_dict(data).run_order() == plain.run_order(data) == [(i, False) for i in range(4)]


def test_tensor_names_and_shapes():
    _, spec = built()
    shapes = {name: tuple(decl.shape) for name, decl in DecoderModel(spec).tensor_decls().items()}
    expected = {"embed": (70, 40), "head": (70, 40), "final.norm": ()}
    expected.update({f"l{i}.norm1": () for i in range(4)})
    expected.update({"l0.mix.q": (72, 40), "l0.mix.q.b": (72,), "l0.mix.k": (24, 40), "l0.mix.k.b": (24,), "l0.mix.v": (40, 40), "l0.mix.v.b": (40,), "l0.mix.g": (6, 40), "l0.mix.o": (40, 120)})
    expected.update({"l1.mix.q": (40, 40), "l1.mix.q.b": (40,), "l1.mix.k": (20, 40), "l1.mix.k.b": (20,), "l1.mix.q.norm": (40,), "l1.mix.k.norm": (20,), "l1.mix.g": (40, 40),
                     "l1.mix.o": (40, 40), "l1.mix.o.b": (40,)})
    expected.update({"l2.mix.q": (48, 40), "l2.mix.k": (48, 40), "l2.mix.v": (24, 40), "l2.mix.q.norm": (16,), "l2.mix.k.norm": (16,), "l2.mix.g": (24, 40), "l2.mix.o": (40, 24)})
    expected.update({"l3.mix.q": (8, 40), "l3.mix.q.b": (8,), "l3.mix.k": (8, 40), "l3.mix.k.b": (8,), "l3.mix.v": (8, 40), "l3.mix.v.b": (8,), "l3.mix.g": (1, 40), "l3.mix.o": (40, 8)})
    for layer, experts, ff, choices in ((0, 5, 24, 6), (2, 4, 16, 4)):
        for e in range(experts):
            expected.update({f"l{layer}.mlp.e{e}.gate": (ff, 40), f"l{layer}.mlp.e{e}.up": (ff, 40), f"l{layer}.mlp.e{e}.down": (40, ff)})
        expected.update({f"l{layer}.mlp.router": (choices, 40), f"l{layer}.mlp.correction": (choices,)})
    expected.update({"l0.mlp.shared.gate": (30, 40), "l0.mlp.shared.up": (30, 40), "l0.mlp.shared.down": (40, 30)})
    assert shapes == expected


def test_what_every_run_keeps_and_that_passed_chunks_give_their_pages_back():
    _, spec = built()
    needs = DecoderModel(spec).cache_needs()
    assert [need.kv for need in needs] == [KVNeed(2, 12, None, 20, 9), KVNeed(2, 10), KVNeed(3, 16, None, 8)] + [KVNeed(2, 10), KVNeed(3, 16, None, 8)] * 2 + [KVNeed(1, 8)]
    manager = CacheManager(needs, [run.cache_of for run in spec.order], page_size=4, num_pages=32, max_requests=2)
    assert [len(group.runs) for group in manager.groups] == [1, 3, 3, 1]      # every pass of the loop has pages of its own
    request = manager.open("a", 40)
    for count in (7, 2, 1, 8, 1, 9):
        manager.prepare([(request, count)])
        manager.commit(request)
        first = request.length - request.length % 9               # the chunk of the next token: what lies before it is read no more
        assert [page >= 0 for page in request.tables[0]] == [(index + 1) * 4 > first for index in range(len(request.tables[0]))]
        assert all(page >= 0 for g in (1, 2, 3) for page in request.tables[g])
    manager.close(request)
    manager.check()


@pytest.mark.parametrize("dtype,kept", [(torch.float32, 10), (torch.bfloat16, 16)])
def test_a_stacked_mixer_lies_in_one_product_in_and_one_out(dtype, kept):
    """Rows: q, k (no values: they are the keys), the gate of every element; in bfloat16 heads are kept at whole 16s, filled up with zeros everywhere."""
    _, spec = built()
    mixer = MIXERS.build(spec.layers[1].block.params["mixer"])
    t = draw(mixer, dtype)
    mixer.load(t, dtype, torch.device("cpu"))
    assert (mixer.kept_head_dim, mixer.kept_value_dim) == (kept, kept) and mixer.stacked and not mixer.splits_products
    filled = (4 + 2 + 4) * kept
    rows = mixer.input_rows[:filled].view(10, kept, 40)
    assert mixer.input_rows.shape == (-(-filled // 8) * 8, 40) and float(mixer.input_rows[filled:].abs().sum()) == 0.0 == float(rows[:, 10:].abs().sum())
    assert torch.equal(rows[:, :10].reshape(100, 40), torch.cat((t["q"], t["k"], t["g"])))
    for mine, name, heads in ((mixer.q_norm, "q.norm", 4), (mixer.k_norm, "k.norm", 2)):
        assert torch.equal(mine.view(heads, kept)[:, :10].reshape(-1), t[name]) and float(mine.view(heads, kept)[:, 10:].abs().sum()) == 0.0
    bias = mixer.b_in.view(6, kept)
    assert torch.equal(bias[:, :10].reshape(-1), torch.cat((t["q.b"], t["k.b"]))) and float(bias[:, 10:].abs().sum()) == 0.0
    assert torch.equal(mixer.b_out, t["o.b"])
    assert torch.equal(mixer.output_columns.view(40, 4, kept)[..., :10].reshape(40, 40), t["o"]) and float(mixer.output_columns.view(40, 4, kept)[..., 10:].abs().sum()) == 0.0
    assert mixer.cache_need().kv == KVNeed(2, kept)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,shared", [(24, 30), (24, 24), (24, 7), (10, 35), (8, 16)])
def test_the_shared_expert_in_pieces_is_the_shared_expert(ff, shared, dtype):
    """The pieces behind the experts, each a gated unit over its part of the inner width, add up to the whole one."""
    part = FEED_FORWARDS.build(PartSpec("expert_mixture", {"width": 16, "intermediate": ff, "experts": 3, "top": 2, "routing": "softmax_all", "share_normalized": False, "always_intermediate": shared}))
    t = draw(part, dtype)
    part.load(t, dtype, torch.device("cpu"))
    assert part.always == math.ceil(shared / ff) and part.w_gate_up.shape == (3 + part.always, 2 * ff, 16) and part.w_down.shape == (3 + part.always, 16, ff)
    h = torch.randn(5, 16, generator=torch.Generator().manual_seed(2)).to(dtype).double()
    total = torch.zeros(5, 16, dtype=torch.float64)
    for piece in range(3, 3 + part.always):
        rows = part.w_gate_up[piece].double()
        gate, up = (rows.view(ff // 8, 2, 8, 16)[:, half].reshape(ff, 16) for half in (0, 1)) if part.interleaved else (rows[:ff], rows[ff:])
        total += (plain.silu(h @ gate.T) * (h @ up.T)) @ part.w_down[piece].double().T
    want = plain.unit(h, {k: v.double() for k, v in t.items()}, "shared.")
    torch.testing.assert_close(total, want, rtol=1e-12, atol=1e-12)


def test_the_choice_of_the_plain_statement():
    """A group is worth its best choice score; what is not kept counts as nothing although choice scores may be negative; the weights know no correction."""
    scores, correction = torch.tensor([0.1, 0.2, 0.3, 0.05, 0.25, 0.1]), torch.tensor([-1.0, -1.0, -1.1, -1.3, -0.9, -2.0])
    assert plain.choose(scores, correction, 2, {"count": 3, "keep": 1}) == [4, 5]      # -0.65 and -1.9: the others are better than the last, but not in the group
    assert plain.choose(scores, correction, 2, {"count": 3, "keep": 2}) == [4, 2 - 1]  # groups worth -0.8, -0.8 (a tie: the first), -0.65
    assert plain.choose(scores, correction, 3, None) == [4, 1, 2] or plain.choose(scores, correction, 3, None) == [4, 2, 1]


def test_the_factor_on_queries_and_the_slopes():
    table = POSITION_ENCODINGS.build(PartSpec("log_steps", {"coef": 0.3, "every": 7, "max_positions": 60})).query_factors(torch.device("cpu"))
    want = torch.tensor([plain.query_factor(p, 0.3, 7) for p in range(60)], dtype=torch.float64)
    torch.testing.assert_close(table.double(), want, rtol=1e-6, atol=0)
    assert float(table[5]) == 1.0 < float(table[6])               # the first step is taken at the 7th position
    _, spec = built()
    slopes = spec.layers[2].block.params["mixer"].params["distance_slopes"]
    assert slopes == tuple(plain.slope(h, 3) for h in range(3)) and slopes[-1] == 2.0 ** -8


def test_a_norm_of_one_number_spreads_it_over_the_row():
    norm = NORMS.build(PartSpec("rmsnorm", {"width": 6, "eps": 1e-5, "weight_name": "", "one_number": True}))
    assert [(d.name, d.shape) for d in norm.tensors()] == [("", ())]
    norm.load({"": torch.tensor(1.5)}, torch.float32, torch.device("cpu"))
    assert norm.weight.tolist() == [1.5] * 6 and norm.weight.is_contiguous()


@pytest.mark.parametrize("error,options", [
    (ValueError, {"output_gate": "rows"}), (ValueError, {"values_from_keys": True, "value_dim": 4}), (ValueError, {"distance_slopes": (0.5,)}),
    (NotImplementedError, {"output_gate": "heads", "sink": True}), (NotImplementedError, {"fixed_sink": 0.0, "window": 4, "keep_first": 1}),
    (NotImplementedError, {"out_bias": True, "value_mix": "source"}), (NotImplementedError, {"weighting": "sigmoid", "fixed_sink": 0.0}),
    (NotImplementedError, {"weighting": "sigmoid", "distance_slopes": (0.5, 0.25)}), (ValueError, {"weighting": "sigmoid", "head_gate": True, "output_gate": "heads"})])
def test_what_a_stacked_mixer_refuses(error, options):
    with pytest.raises(error):
        MIXERS.build(PartSpec("gqa_attention", {"width": 16, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, **options}))


@pytest.mark.parametrize("error,options", [
    (ValueError, {"identity": 2}), (ValueError, {"share_scale": 2.0}), (ValueError, {"routing": "softmax_all", "group_score": "worst"}),
    (ValueError, {"routing": "softmax_all", "identity": 1, "groups": 4, "groups_keep": 1}), (ValueError, {"routing": "softmax_all", "top": 5}),
    (NotImplementedError, {"routing": "softmax_all", "identity": 1, "weigh": "input"}), (NotImplementedError, {"routing": "sigmoid", "always_intermediate": 8, "shared_intermediate": 8}),
    (NotImplementedError, {"routing": "sigmoid", "always_intermediate": 8, "gated": False})])
def test_what_a_mixture_with_experts_that_hand_their_input_back_refuses(error, options):
    with pytest.raises(error):
        FEED_FORWARDS.build(PartSpec("expert_mixture", {"width": 16, "intermediate": 8, "experts": 4, "top": 2, **options}))
