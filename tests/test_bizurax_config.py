"""The Bizurax configuration without a GPU: reading config.json, what may be absent, what is refused, the schedule of looped
layers, the tensors it expects, and hand-made numbers for the plain implementation's mechanisms."""
import copy
import json
import math

import pytest
import torch

import plain_bizurax as plain
from qwen_triton_b200 import config_from_dict, load_preset
from qwen_triton_b200.config import BizuraxConfig, ConfigError, PartSpec
from qwen_triton_b200.engine.model import expected_tensors
from qwen_triton_b200.parts.base import Runtime, Workspace, part_class

RAW = {
    "architecture": "Bizurax", "vocab": 40, "width": 24, "norm": {"eps": 1e-5}, "streams": 2, "residual_mult": 0.7, "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        {"type": "attention", "mlp": {"kind": "dense", "ff": 10},
         "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.2, "softcap": 9.0, "rot": {"base": 50.0, "dims": 4, "scaling": {"factor": 3.0}}}},
        {"type": "retention", "mlp": None, "mixer": {"heads": 3, "dim": 8, "vdim": 4, "decay": [0.9, 0.5, 1.0], "rot": {"base": 60.0, "dims": 8}}},
        {"type": "latent_attention", "mlp": {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 7}},
         "mixer": {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 5, "kv_rank": 7, "scale": 0.3, "rot": {"base": 100.0, "dims": 4}}},
        {"type": "retention", "mlp": {"kind": "moe", "expert": {"ff": 3}, "router": {"experts": 2, "top": 2}}, "mixer": {"heads": 1, "dim": 4, "vdim": 4, "decay": [0.3]}},
    ],
}


def test_it_is_chosen_by_its_name_and_round_trips():
    config = config_from_dict(RAW)
    assert isinstance(config, BizuraxConfig) and config.vocab_size == 40 and config.hidden_size == 24 and config.num_hidden_layers == 4
    assert config_from_dict(json.loads(json.dumps(config.to_hf_dict()))) == config
    for name in ("bizurax-tiny-a", "bizurax-tiny-b"):
        preset = load_preset(name)
        assert config_from_dict(preset.to_hf_dict()) == preset


def test_looped_layers_run_again_with_caches_of_their_own():
    spec = config_from_dict(RAW).model_spec()
    assert [call.layer for call in spec.schedule] == [0, 1, 2, 1, 2, 3] and all(call.cache_of is None and call.entry is None for call in spec.schedule)
    assert plain.schedule(RAW) == [0, 1, 2, 1, 2, 3] and spec.streams == 2
    raw = copy.deepcopy(RAW)
    del raw["loop"]
    assert [call.layer for call in config_from_dict(raw).model_spec().schedule] == [0, 1, 2, 3] == plain.schedule(raw)


def test_the_tensors_it_expects():
    names = expected_tensors(config_from_dict(RAW).model_spec())
    wanted = {"embed": (40, 24), "final.norm": (24,), "head": (40, 24), "l0.norm1": (24,), "l0.norm2": (24,), "l0.hc1.in": (2,), "l0.hc1.out": (2,), "l0.hc1.mix": (2, 2),
              "l0.hc2.mix": (2, 2), "l0.mix.q": (24, 24), "l0.mix.q.b": (24,), "l0.mix.k": (12, 24), "l0.mix.k.b": (12,), "l0.mix.v": (10, 24), "l0.mix.v.b": (10,),
              "l0.mix.sink": (4,), "l0.mix.o": (24, 20), "l0.mlp.up": (10, 24), "l0.mlp.down": (24, 10), "l1.mix.q": (24, 24), "l1.mix.k": (24, 24), "l1.mix.v": (12, 24),
              "l1.mix.g": (12, 24), "l1.mix.o": (24, 12), "l1.hc1.in": (2,), "l2.mix.q": (20, 24), "l2.mix.dkv": (11, 24), "l2.mix.dkv.norm": (7,), "l2.mix.uk": (12, 7),
              "l2.mix.uv": (10, 7), "l2.mix.o": (24, 10), "l2.mlp.router": (6, 24), "l2.mlp.router.b": (6,), "l2.mlp.e5.gate": (9, 24), "l2.mlp.e0.up": (9, 24),
              "l2.mlp.e0.down": (24, 9), "l2.mlp.shared.gate": (7, 24), "l2.mlp.shared.down": (24, 7), "l3.mlp.e1.up": (3, 24)}
    for name, shape in wanted.items():
        assert tuple(names[name].shape) == shape and not names[name].optional, name
    for name in ("l0.mix.o.b", "l2.mix.g", "l2.mix.dq", "l0.mlp.gate", "l3.mlp.shared.gate", "l1.mix.norm"):
        assert name not in names, name
    for name in ("l1.norm2", "l1.hc2.in", "l1.hc2.mix"):         # of the feed-forward that layer 1 lacks
        assert name not in names or names[name].optional, name


def test_what_may_be_absent():
    raw = copy.deepcopy(RAW)
    for key in ("streams", "residual_mult", "loop"):
        del raw[key]
    del raw["layers"][0]["mixer"]["softcap"], raw["layers"][0]["mixer"]["rot"]["scaling"], raw["layers"][1]["mixer"]["rot"], raw["layers"][1]["mixer"]["vdim"]
    config = config_from_dict(raw)
    assert config.layers[0].mixer.softcap is None and config.layers[0].mixer.rot.factor == 1.0 and config.layers[1].mixer.rot.dims == 0
    assert config.layers[1].mixer.vdim == 8 and config.streams is None and config.residual_mult == 1.0
    assert config_from_dict(config.to_hf_dict()) == config
    spec = config.model_spec()
    assert spec.streams == 1 and not any(".hc" in name for name in expected_tensors(spec))


@pytest.mark.parametrize("change, words", [
    (lambda r: r["layers"][0].update(type="conv"), "no mixer"),
    (lambda r: r["layers"][0]["mlp"].update(kind="plain"), "no feed-forward"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "divide"),
    (lambda r: r["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=3), "even"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=8), "at most 6"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(scaling={"factor": 0.0}), "factor"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5, 0.5]), "decays"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5, 0.5, 0.0]), "decays"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=6), "at most 4"),
    (lambda r: r["layers"][2]["mlp"]["router"].update(top=7), "of experts=6"),
    (lambda r: r["layers"][2]["mlp"]["shared"].pop("ff"), "shared"),
    (lambda r: r.update(streams=0), "streams"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r["loop"].update(times=0), "loop"),
    (lambda r: r["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda r: r.pop("vocab"), "vocab"),
])
def test_refusals_in_words(change, words):
    raw = copy.deepcopy(RAW)
    change(raw)
    with pytest.raises(ConfigError, match=words):
        config_from_dict(raw)


def cpu_runtime():
    device = torch.device("cpu")
    return Runtime(device=device, dtype=torch.float32, max_step_tokens=8, max_positions=16, workspace=Workspace(device), sm_count=148)


def test_the_rotation_table_with_stretched_angles():
    spec = PartSpec("rope", {"theta": 100.0, "rotary_dim": 4, "head_dim": 6, "angles": "float64", "factor": 5.0})
    part = part_class("position", spec)(spec.params, cpu_runtime())
    table = part.table(16)
    for pos in (0, 1, 15):
        angles = [pos / 5.0, pos * 0.1 / 5.0]
        want = [math.cos(a) for a in angles] + [math.sin(a) for a in angles]
        torch.testing.assert_close(table[pos].double(), torch.tensor(want, dtype=torch.float64), atol=1e-6, rtol=1e-6)
    plainly = part_class("position", spec)({**spec.params, "factor": 1.0}, cpu_runtime())
    assert part.key() != plainly.key()


def test_neighbouring_pairs_become_halves_when_the_weights_are_loaded():
    """The latent attention's rows are reordered so that the kernels' rotation of halves turns the stored neighbours: the dot product
    of a rotated query and a rotated key is that of the plain implementation's interleaved rotation."""
    layer = config_from_dict(RAW).model_spec().layers[2]
    part = part_class("mixer", layer.mixer)(layer.mixer.params, "p", cpu_runtime())
    assert part.interleaved
    torch.manual_seed(0)
    weight = torch.randn(2 * (6 + 4), 24)
    moved = part._halves_order(weight, 2, 6).view(2, 10, 24)
    stored = weight.view(2, 10, 24)
    assert torch.equal(moved[:, :6], stored[:, :6]) and torch.equal(moved[:, 6:], stored[:, [6, 8, 7, 9]])
    x, y, at = torch.randn(3, 2, 4, dtype=torch.float64), torch.randn(3, 2, 4, dtype=torch.float64), torch.tensor([0, 3, 11])
    order = [0, 2, 1, 3]
    want = (plain.rotate(x, at, 4, 100.0, interleaved=True) * plain.rotate(y, at + 2, 4, 100.0, interleaved=True)).sum(-1)
    got = (plain.rotate(x[..., order], at, 4, 100.0) * plain.rotate(y[..., order], at + 2, 4, 100.0)).sum(-1)
    torch.testing.assert_close(got, want)


def test_the_plain_mechanisms_on_numbers_made_by_hand():
    D = torch.float64
    # two streams: u = 1 x_1 + 2 x_2; x_1 <- 3 x_1 + 5 x_2 + m out_1 y, x_2 <- 4 x_1 + 6 x_2 + m out_2 y
    t = {"c.in": torch.tensor([1.0, 2.0], dtype=D), "c.mix": torch.tensor([[3.0, 4.0], [5.0, 6.0]], dtype=D), "c.out": torch.tensor([10.0, 20.0], dtype=D)}
    x = torch.tensor([[[1.0]], [[7.0]]], dtype=D)
    assert float(plain.read_streams(x, t, "c")) == 15.0
    new = plain.write_streams(x, torch.tensor([[2.0]], dtype=D), t, "c", 0.5)
    assert new[:, 0, 0].tolist() == [3 + 35 + 10, 4 + 42 + 20]
    # a sink of score ln 2 beside keys of score 0: 1/3 for the first query's key, 1/4 each for the second's two
    weights = plain.causal_softmax(torch.zeros(2, 2, dtype=D), torch.tensor(math.log(2.0), dtype=D))
    torch.testing.assert_close(weights, torch.tensor([[1 / 3, 0.0], [0.25, 0.25]], dtype=D))
    torch.testing.assert_close(plain.cap(torch.tensor([0.1, 100.0], dtype=D), 2.0), torch.tensor([2 * math.tanh(0.05), 2.0], dtype=D))
    # a quarter turn of neighbours, of halves, and a stretched one
    one = torch.tensor([[[1.0, 0.0, 7.0, 0.0]]], dtype=D)
    c, s, c2, s2 = math.cos(1.0), math.sin(1.0), math.cos(0.2), math.sin(0.2)
    torch.testing.assert_close(plain.rotate(one, torch.tensor([1]), 4, 25.0, interleaved=True), torch.tensor([[[c, s, 7 * c2, 7 * s2]]], dtype=D))
    torch.testing.assert_close(plain.rotate(one, torch.tensor([1]), 4, 25.0), torch.tensor([[[c - 7 * s, 0.0, 7 * c + s, 0.0]]], dtype=D))
    torch.testing.assert_close(plain.rotate(one, torch.tensor([2]), 2, 25.0, 2.0), torch.tensor([[[c, s, 7.0, 0.0]]], dtype=D))
    # decay 0.5: S_1 = k_1 v_1 = 10, o_2 = (0.5 * 10 + 1 * 7) q_2
    q, k = torch.tensor([[[1.0]], [[3.0]]], dtype=D), torch.tensor([[[2.0]], [[1.0]]], dtype=D)
    v = torch.tensor([[[5.0]], [[7.0]]], dtype=D)
    assert plain.fixed_decay_recurrence(q, k, v, torch.tensor([0.5], dtype=D))[:, 0, 0].tolist() == [10.0, 36.0]
    # the two largest logits, weighted by a softmax over the two alone
    chosen, weights = plain.route(torch.log(torch.tensor([[0.1, 3.0, 0.4, 1.0]], dtype=D)), 2)
    assert chosen[0].tolist() == [1, 3]
    torch.testing.assert_close(weights, torch.tensor([[0.75, 0.25]], dtype=D))
    assert plain.dense(torch.tensor([[2.0]], dtype=D), {"p.up": torch.tensor([[3.0], [-1.0]], dtype=D), "p.down": torch.tensor([[1.0, 100.0]], dtype=D)}, "p").item() == 36.0
