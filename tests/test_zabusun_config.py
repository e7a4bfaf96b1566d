"""Zabusun without a GPU: its configuration, the model description built from it (tensor names and shapes, what each run keeps between
steps), how mixers that split off their products are stacked, and what the parts refuse."""
from __future__ import annotations

import copy
import json

import pytest
import torch

from pylon_b200.config.model_config import ConfigError, ZabusunConfig
from pylon_b200.config.registry import ARCHITECTURES, architecture_of, read_config
from pylon_b200.models.decoder import DecoderModel
from pylon_b200.parts import FEED_FORWARDS, MIXERS, PartSpec
from pylon_b200.parts.base import KVNeed, StateNeed

YARN = {"factor": 4.0, "original": 16, "fast": 8.0, "slow": 1.0}
CONFIG = {
    "architecture": "Zabusun", "vocab": 50, "width": 24, "norm": {"eps": 1e-6}, "logit_scale": 1.25,
    "layers": [
        {"type": "parallel", "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 4, "scale": 0.5, "rot": {"dims": 6, "base": 100.0, "scaling": YARN}},
                                       "left_scale": 0.7, "right": {"width": 12}, "right_scale": 1.5},
         "mlp": {"kind": "moe", "expert": {"ff": 16, "limit": 2.0}, "router": {"experts": 6, "top": 2}}},
        {"type": "parallel", "mixer": {"left": {"heads": 2, "kv_heads": 2, "dim": 8, "vdim": 20, "scale": 0.25, "rot": {"dims": 8, "base": 10.0, "scaling": None}},
                                       "left_scale": 1.0, "right": {"width": 9}, "right_scale": 2.0},
         "mlp": {"kind": "dense", "ff": 32, "limit": 7.0}},
        {"type": "parallel", "mixer": {"left": {"heads": 3, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 0.1}, "left_scale": 1.0, "right": {"width": 5}, "right_scale": 1.0}, "mlp": None},
    ],
}


def built(data=CONFIG, max_positions=64):
    config = ZabusunConfig.from_dict(data)
    return config, ARCHITECTURES["Zabusun"].build_spec(config, max_positions)


def test_the_configuration_reads_every_key_and_writes_it_back():
    config = ZabusunConfig.from_dict(CONFIG)
    assert (config.vocab, config.width, config.norm_eps, config.logit_scale) == (50, 24, 1e-6, 1.25)
    first, second, third = config.layers
    left = first.left
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.rot.dims, left.rot.base, dict(left.rot.scaling)) == (4, 2, 8, 4, 0.5, 6, 100.0, YARN)
    assert (first.right_width, first.left_scale, first.right_scale) == (12, 0.7, 1.5)
    assert (first.mlp.kind, first.mlp.ff, first.mlp.limit, first.mlp.experts, first.mlp.top) == ("moe", 16, 2.0, 6, 2)
    assert (second.mlp.kind, second.mlp.ff, second.mlp.limit, second.mlp.experts) == ("dense", 32, 7.0, None) and second.left.rot.scaling is None
    assert third.mlp is None and third.left.rot is None
    assert config.to_dict() == CONFIG
    assert ZabusunConfig.from_dict(json.loads(json.dumps(config.to_dict()))) == config


def test_the_registry_finds_the_architecture(tmp_path):
    assert architecture_of(CONFIG) is ARCHITECTURES["Zabusun"]
    (tmp_path / "config.json").write_text(json.dumps(CONFIG))
    architecture, config = read_config(tmp_path)
    assert architecture.name == "Zabusun" and isinstance(config, ZabusunConfig)


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="other"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "cannot be grouped"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=10), "exceeds the head's dim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=5), "must be even"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "cannot use"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][1]["mlp"].update(kind="other"), "unknown feed-forward"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("width"), "width"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.update(layers=[]), "at least one layer"),
])
def test_what_the_configuration_refuses(change, text):
    data = copy.deepcopy(CONFIG)
    change(data)
    with pytest.raises(ConfigError, match=text):
        ZabusunConfig.from_dict(data)


def test_the_model_description():
    config, spec = built()
    assert [run.layer for run in spec.order] == [0, 1, 2] and spec.logit_scale == 1.25 and spec.lm_head_name is None
    model = DecoderModel(spec)
    decls = model.tensor_decls()
    expected = {
        "embed": (50, 24), "embed.norm": (24,), "final.norm": (24,), "l0.norm1": (24,), "l0.norm2": (24,),
        "l0.mix.left.q": (32, 24), "l0.mix.left.k": (16, 24), "l0.mix.left.v": (8, 24), "l0.mix.left.o": (24, 16), "l0.mix.left.g": (4, 24), "l0.mix.left.pb": (4,),
        "l0.mix.left.q.norm": (8,), "l0.mix.left.k.norm": (8,),
        "l0.mix.right.z": (12, 24), "l0.mix.right.z.b": (12,), "l0.mix.right.x": (12, 24), "l0.mix.right.x.b": (12,), "l0.mix.right.g": (12, 24), "l0.mix.right.o": (24, 12),
        "l0.mlp.router": (6, 24), "l0.mlp.e5.gate": (16, 24), "l0.mlp.e0.up": (16, 24), "l0.mlp.e3.down": (24, 16),
        "l1.mlp.gate": (32, 24), "l1.mlp.up": (32, 24), "l1.mlp.down": (24, 32), "l1.mix.left.v": (40, 24), "l2.mix.left.q": (12, 24),
    }
    for name, shape in expected.items():
        assert tuple(decls[name].shape) == shape, name
    assert len(decls) == 3 + 3 * 15 + 2 + (1 + 6 * 3) + 3 and not any(name.startswith("l2.mlp.") or name == "l2.norm2" for name in decls)
    needs = model.cache_needs()
    assert needs[0].kv == KVNeed(2, 8, None, 4) and needs[0].state == StateNeed((12,))
    assert needs[1].kv == KVNeed(2, 8, None, 20) and needs[1].state == StateNeed((9,))
    assert model.takes_padding()


def draw(part, dtype):
    g = torch.Generator().manual_seed(1)
    return {d.name: torch.randn(*d.shape, generator=g).to(torch.float32 if d.role == "vector" else dtype) for d in part.tensors()}


def test_mixers_that_split_off_their_products_are_stacked():
    """One matrix in, rows of every mixer from a multiple of 8 on, and one out, columns likewise; what fills the gaps is zeros.  In bfloat16
    keys and values are kept at one width of whole 16s."""
    config, spec = built()
    for dtype, kept in ((torch.float32, (8, 20)), (torch.bfloat16, (32, 32))):
        mixer = MIXERS.build(spec.layers[1].block.params["mixer"])
        tensors = draw(mixer, dtype)
        mixer.load(tensors, dtype, torch.device("cpu"))
        attention = mixer.mixers[0]
        assert (attention.kept_head_dim, attention.kept_value_dim) == kept
        rows = 4 * kept[0] + 2 * kept[1] + 2             # q of 2 heads, k of 2, v of 2, a gate row per head
        assert mixer.in_slices[0] == slice(0, -(-rows // 8) * 8) and mixer.in_slices[1].start == mixer.in_slices[0].stop
        assert mixer.w_in.shape == (mixer.in_slices[1].start + 32, 24) and mixer.w_out.shape == (24, mixer.out_slices[1].start + 16)     # 27 and 9, filled up
        assert torch.equal(mixer.w_in[mixer.in_slices[1]], torch.cat([tensors["right." + key] for key in ("z", "x", "g")]))
        assert torch.equal(mixer.w_in[rows - 2 : rows], tensors["left.g"]) and float(mixer.w_in[rows : mixer.in_slices[1].start].abs().sum()) == 0.0
        q = mixer.w_in[: 2 * kept[0]].view(2, kept[0], 24)
        assert torch.equal(q[:, :8].reshape(16, 24), tensors["left.q"]) and float(q[:, 8:].abs().sum()) == 0.0
        o = mixer.w_out[:, : 2 * kept[1]].view(24, 2, kept[1])
        assert torch.equal(o[..., :20].reshape(24, 40), tensors["left.o"]) and float(o[..., 20:].abs().sum()) == 0.0
        assert torch.equal(mixer.w_out[:, mixer.out_slices[1]], tensors["right.o"]) and float(mixer.w_out[:, mixer.out_slices[1].stop :].abs().sum()) == 0.0
        assert attention.input_rows.data_ptr() == mixer.w_in.data_ptr()      # no second copy
        need = mixer.cache_need()
        assert need.kv == KVNeed(2, kept[0], None, None if kept[0] == kept[1] else kept[1]) and need.state == StateNeed((9,))


@pytest.mark.parametrize("options", [
    {"sink": True}, {"qk_norm": "whole", "qk_norm_eps": 1e-5}, {"bias": True}, {"value_mix": "source"}, {"window": 4, "keep_first": 1}, {"distance_bias": {"rows": 4, "far": 9}}])
def test_what_sigmoid_weights_do_not_go_with(options):
    with pytest.raises(NotImplementedError):
        MIXERS.build(PartSpec("gqa_attention", {"width": 16, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "weighting": "sigmoid", **options}))


def test_what_goes_with_sigmoid_weights_only():
    for options in ({"score_bias": True}, {"head_gate": True}):
        with pytest.raises(NotImplementedError):
            MIXERS.build(PartSpec("gqa_attention", {"width": 16, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, **options}))
    with pytest.raises(ValueError):
        MIXERS.build(PartSpec("gqa_attention", {"width": 16, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "weighting": "other"}))


@pytest.mark.parametrize("options", [
    {"activation": "clamped"}, {"limit": 2.0}, {"activation": "clamped", "limit": -1.0}, {"weigh": "other"}, {"share_normalized": False}, {"weigh": "input", "gated": False, "routing": "sigmoid"}])
def test_what_a_mixture_of_experts_refuses(options):
    with pytest.raises(ValueError):
        FEED_FORWARDS.build(PartSpec("expert_mixture", {"width": 16, "intermediate": 8, "experts": 4, "top": 2, **options}))
