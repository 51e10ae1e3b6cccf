"""The Misudra configuration without a GPU: reading config.json, what may be absent, what is refused, the schedule of looped
layers, the tensors it expects, and hand-made numbers for the plain implementation's mechanisms."""
import copy
import json
import math

import pytest
import torch

import plain_misudra as plain
from qwen_triton_b200 import config_from_dict, load_preset
from qwen_triton_b200.config import ConfigError, MisudraConfig
from qwen_triton_b200.engine.model import expected_tensors
from qwen_triton_b200.ops import kernels

RAW = {
    "architecture": "Misudra", "vocab": 40, "width": 24, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        {"type": "mamba2", "mlp": {"kind": "dense", "ff": 10}, "mixer": {"heads": 4, "vdim": 6, "state": 5, "groups": 2, "conv": 3, "norm_groups": 2}},
        {"type": "gla", "mlp": None, "mixer": {"heads": 3, "dim": 8, "vdim": 4, "tau": 2.0, "ranks": {"decay": 7}}},
        {"type": "latent_attention", "mlp": {"kind": "moe", "expert": {"ff": 9, "limit": 2.0}, "router": {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}},
         "mixer": {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 5, "q_rank": 11, "kv_rank": 7, "scale": 0.3, "mask": {"size": 9}, "rot": {"base": 100.0, "dims": 4}}},
        {"type": "gla", "mlp": None, "mixer": {"heads": 1, "dim": 4, "vdim": 4, "tau": 1.0, "ranks": {"decay": 2}}},
    ],
}


def test_it_is_chosen_by_its_name_and_round_trips():
    config = config_from_dict(RAW)
    assert isinstance(config, MisudraConfig) and config.vocab_size == 40 and config.hidden_size == 24 and config.num_hidden_layers == 4
    assert config_from_dict(json.loads(json.dumps(config.to_hf_dict()))) == config
    for name in ("misudra-tiny-a", "misudra-tiny-b"):
        preset = load_preset(name)
        assert config_from_dict(preset.to_hf_dict()) == preset


def test_looped_layers_run_again_with_caches_of_their_own_behind_a_map_of_the_stream():
    spec = config_from_dict(RAW).model_spec()
    assert [call.layer for call in spec.schedule] == [0, 1, 2, 1, 2, 3] and all(call.cache_of is None for call in spec.schedule)
    assert [call.entry for call in spec.schedule] == [None, 0, None, 0, None, None]
    assert plain.schedule(RAW) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    names = expected_tensors(spec)
    wanted = {"embed": (40, 24), "embed.norm": (24,), "loop.in": (24, 48), "final.norm": (24,), "head": (40, 24), "l0.norm1": (24,), "l0.norm2": (24,),
              "l0.mix.in": (24 + 24 + 20 + 4, 24), "l0.mix.conv": (44, 3), "l0.mix.conv.b": (44,), "l0.mix.dt_bias": (4,), "l0.mix.A_log": (4,),
              "l0.mix.D": (4,), "l0.mix.norm": (24,), "l0.mix.o": (24, 24), "l0.mlp.gate": (10, 24), "l0.mlp.gate.b": (10,), "l0.mlp.up.b": (10,),
              "l0.mlp.down": (24, 10), "l0.mlp.down.b": (24,), "l1.mix.q": (24, 24), "l1.mix.v": (12, 24), "l1.mix.g": (12, 24), "l1.mix.a1": (7, 24),
              "l1.mix.a2": (24, 7), "l1.mix.a2.b": (24,), "l1.mix.norm": (4,), "l1.mix.o": (24, 12), "l2.mix.dq": (11, 24), "l2.mix.dq.norm": (11,),
              "l2.mix.uq": (20, 11), "l2.mix.dkv": (11, 24), "l2.mix.dkv.norm": (7,), "l2.mix.uk": (12, 7), "l2.mix.uv": (10, 7), "l2.mix.g": (2, 24),
              "l2.mix.o": (24, 10), "l2.mlp.router": (6, 24), "l2.mlp.e5.gate": (9, 24), "l2.mlp.e0.down": (24, 9)}
    for name, shape in wanted.items():
        assert tuple(names[name].shape) == shape, name
    assert "l1.norm2" not in names or names["l1.norm2"].optional
    raw = copy.deepcopy(RAW)
    del raw["loop"]
    spec = config_from_dict(raw).model_spec()
    assert [call.layer for call in spec.schedule] == [0, 1, 2, 3] and not spec.entries and "loop.in" not in expected_tensors(spec)


def test_the_narrow_projections_columns_come_from_the_tensors():
    raw = copy.deepcopy(RAW)
    del raw["layers"][1]["mixer"]["ranks"]
    config = config_from_dict(raw)
    with pytest.raises(ConfigError, match="l1.mix.a1"):
        config.model_spec()
    full = config.with_tensor_shapes({"l1.mix.a1": (5, 24), "l3.mix.a1": (2, 24)})
    assert tuple(expected_tensors(full.model_spec())["l1.mix.a2"].shape) == (24, 5)


def test_what_may_be_absent():
    raw = copy.deepcopy(RAW)
    del raw["layers"][2]["mixer"]["mask"], raw["layers"][2]["mlp"]["router"]["groups"]
    config = config_from_dict(raw)
    assert config.layers[2].mixer.window is None and config.layers[2].mlp.group_count == 1
    assert config_from_dict(config.to_hf_dict()) == config


@pytest.mark.parametrize("change, words", [
    (lambda r: r["layers"][0].update(type="conv"), "no mixer"),
    (lambda r: r["layers"][0]["mlp"].update(kind="plain"), "no feed-forward"),
    (lambda r: r["layers"][0]["mixer"].update(groups=3), "divide"),
    (lambda r: r["layers"][0]["mixer"].update(norm_groups=5), "divide"),
    (lambda r: r["layers"][0]["mixer"].update(conv=17), "taps"),
    (lambda r: r["layers"][1]["mixer"].update(tau=0.0), "tau"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=3), "even"),
    (lambda r: r["layers"][2]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda r: r["layers"][2]["mlp"]["router"].update(top=7), "of experts=6"),
    (lambda r: r["layers"][2]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda r: r["layers"][2]["mlp"]["router"].update(top=3, groups={"count": 6, "keep": 2}), "out of 2 groups"),
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


def test_scratch_of_the_chunked_recurrence_holds_every_chunk():
    """A sequence's chunks are numbered from seq_start // 64 + its place on: distinct, and below tokens // 64 + sequences."""
    generator = torch.Generator().manual_seed(0)
    for _ in range(200):
        lengths = torch.randint(1, 200, (int(torch.randint(1, 9, (1,), generator=generator)),), generator=generator).tolist()
        seen, begin = set(), 0
        for place, length in enumerate(lengths):
            for chunk in range(-(-length // kernels.DECAY_CHUNK)):
                number = begin // kernels.DECAY_CHUNK + place + chunk
                assert number not in seen and number < sum(lengths) // kernels.DECAY_CHUNK + len(lengths)
                seen.add(number)
            begin += length


def test_the_plain_mechanisms_on_numbers_made_by_hand():
    D = torch.float64
    # window 2: query 2 sees keys 1 and 2 with equal scores
    weights = plain.windowed_softmax(torch.zeros(3, 3, dtype=D), 2)
    torch.testing.assert_close(weights, torch.tensor([[1.0, 0, 0], [0.5, 0.5, 0], [0, 0.5, 0.5]], dtype=D))
    # two key channels with decays 0.5 and 0.1: S_1 = k_1 v_1, S_2 = diag(decay) S_1 + k_2 v_2
    q = torch.tensor([[[1.0, 1.0]], [[1.0, 10.0]]], dtype=D)
    k = torch.tensor([[[2.0, 3.0]], [[1.0, 0.0]]], dtype=D)
    v, decay = torch.tensor([[[5.0]], [[7.0]]], dtype=D), torch.tensor([[[0.9, 0.9]], [[0.5, 0.1]]], dtype=D)
    torch.testing.assert_close(plain.decayed_recurrence(q, k, v, decay)[:, 0, 0], torch.tensor([25.0, 0.5 * 10 + 7 + 10 * 0.1 * 15], dtype=D))
    # taps (1, 10), bias 0.5, zeros before the start
    out = plain.causal_convolution(torch.tensor([[1.0], [2.0]], dtype=D), torch.tensor([[1.0, 10.0]], dtype=D), torch.tensor([0.5], dtype=D))
    torch.testing.assert_close(out[:, 0], torch.tensor([10.5, 21.5], dtype=D))
    # each half by its own root mean square
    torch.testing.assert_close(plain.grouped_rms(torch.tensor([[3.0, 3.0, 0.1, -0.1]], dtype=D), 2, 0.0), torch.tensor([[1.0, 1.0, 1.0, -1.0]], dtype=D))
    # groups of two: the second-best expert (1) is in the dropped group's shadow: keep 1 group chooses experts 0 and 1 only
    logits = torch.log(torch.tensor([[0.4, 0.1, 0.3, 0.2]], dtype=D))
    chosen, weights = plain.route(logits, 2, {"count": 2, "keep": 1})
    assert chosen[0].tolist() == [0, 1]
    torch.testing.assert_close(weights, torch.tensor([[0.8, 0.2]], dtype=D))
    chosen, weights = plain.route(logits, 2)
    assert chosen[0].tolist() == [0, 2]
    torch.testing.assert_close(plain.choice_margin(logits, 2, {"count": 2, "keep": 1}), torch.log(torch.tensor([4.0 / 3.0], dtype=D)))
    # capped gate at 1: g = min(3, 1) = 1, u = clamp(-5) = -1, y = 1 sigmoid(1.702) (-1 + 1) = 0; and with u = 0.5
    one = torch.ones(1, 1, dtype=D)
    assert float(plain.capped_expert(one, 3 * one, -5 * one, one, 1.0)) == 0.0
    torch.testing.assert_close(plain.capped_expert(one, 3 * one, 0.5 * one, one, 1.0)[0, 0], torch.tensor(1.5 / (1.0 + math.exp(-1.702)), dtype=D))
    # a quarter turn
    turned = plain.rotate(torch.tensor([[[1.0, 0.0, 7.0]]], dtype=D), torch.tensor([1]), 2, 5.0)
    torch.testing.assert_close(turned, torch.tensor([[[math.cos(1.0), math.sin(1.0), 7.0]]], dtype=D))
