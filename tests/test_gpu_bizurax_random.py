"""Bizurax models drawn at random from what config.json allows (widths, head counts, ranks and sizes off 8 and off 16 among them,
values narrower and wider than keys, partial, stretched and no rotation, caps narrow, wide and none, 1 to 6 streams and none, the
order and number of layers, loops of any range and count and none, 1 to 12 experts with and without a shared one, dense layers and
layers without a feed-forward), each run whole, token by token, in portions and as an unequal batch in both types against the
plain implementation."""
import random
import tempfile
from pathlib import Path

import pytest
import torch

import plain_bizurax as plain
from qwen_triton_b200 import Engine, StepEntry, config_from_dict, write_random_model
from qwen_triton_b200.weights import Checkpoint, write_safetensors
from test_gpu_vunepel import STORE, close as close_all

CLOSE_CALL = 0.15      # a router's gap, over the scale of its logits, below which bfloat16 may choose otherwise

pytestmark = pytest.mark.gpu


def draw_rotation(rng, most: int) -> dict | None:
    most = most // 2 * 2
    if most == 0 or rng.random() < 0.1:
        return None
    rot = {"dims": most if rng.random() < 0.6 else rng.randrange(2, most + 1, 2), "base": rng.choice([100.0, 10000.0, 300000.0])}
    if rng.random() < 0.4:
        rot["scaling"] = {"factor": rng.choice([1.5, 2.0, 8.0])}
    return rot


def draw_mixer(rng, kind: str) -> dict:
    heads = rng.choice([1, 2, 3, 4, 6, 8])
    vdim = rng.choice([4, 8, 20, 32, 33, 64, 72])
    if kind == "retention":
        dim = rng.choice([3, 8, 16, 20, 64, 100, 128])
        mixer = {"heads": heads, "dim": dim, "vdim": vdim, "decay": [rng.choice([0.3, 0.9, 0.99, 1.0 - 2.0 ** -9, 1.0]) for _ in range(heads)]}
        rot = draw_rotation(rng, dim)
    elif kind == "attention":
        dim = rng.choice([10, 16, 32, 48, 64, 64, 128])
        mixer = {"heads": heads, "kv_heads": rng.choice([g for g in (1, 2, 3, heads) if heads % g == 0]), "dim": dim, "vdim": dim if rng.random() < 0.7 else vdim,
                 "scale": round(rng.uniform(0.3, 1.5) * 8.0 / dim, 4)}
        if rng.random() < 0.8:
            mixer["softcap"] = rng.choice([1.0, 4.0, 15.0, 60.0])
        rot = draw_rotation(rng, dim)
    else:
        rot_dim = rng.choice([0, 2, 6, 8, 16, 32])
        mixer = {"heads": rng.choice([heads, 20, 34]) if rng.random() < 0.3 else heads, "dim": rng.choice([4, 10, 16, 32, 64]), "rot_dim": rot_dim, "vdim": vdim,
                 "kv_rank": rng.choice([6, 8, 16, 40, 64, 136]), "scale": round(rng.uniform(0.05, 0.4), 3)}
        rot = draw_rotation(rng, rot_dim)
    if rot is not None:
        mixer["rot"] = rot
    return mixer


def draw(seed: int) -> dict:
    rng = random.Random(9000 + seed)
    layers = []
    for _ in range(rng.randint(1, 6)):
        kind = rng.choice(["retention", "attention", "latent_attention"])
        mlp, roll = None, rng.random()
        if roll < 0.35:
            mlp = {"kind": "dense", "ff": rng.choice([8, 9, 20, 48, 100, 128])}
        elif roll < 0.85:
            count = rng.randint(1, 12)
            mlp = {"kind": "moe", "expert": {"ff": rng.choice([8, 9, 20, 48, 100])}, "router": {"experts": count, "top": rng.randint(1, min(count, 4))}}
            if rng.random() < 0.6:
                mlp["shared"] = {"ff": rng.choice([8, 11, 48, 64])}
        layers.append({"type": kind, "mixer": draw_mixer(rng, kind), "mlp": mlp})
    raw = {"architecture": "Bizurax", "vocab": rng.randint(30, 300), "width": rng.choice([36, 40, 64, 72, 96, 100, 128, 200]),
           "norm": {"eps": rng.choice([1e-6, 1e-5, 1e-3])}, "layers": layers, "residual_mult": rng.choice([0.2, 0.5, 1.0])}
    if rng.random() < 0.9:
        raw["streams"] = rng.randint(1, 6)
    if rng.random() < 0.75:
        start = rng.randrange(len(layers))
        raw["loop"] = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.randint(1, 3)}
    return raw


@pytest.mark.parametrize("dtype", ("fp32", "bf16"))
@pytest.mark.parametrize("seed", range(14))
def test_a_model_drawn_at_random(seed, dtype):
    config = config_from_dict(draw(seed))
    raw = config.to_hf_dict()
    with tempfile.TemporaryDirectory() as holder:
        folder = write_random_model(holder, config, seed=seed, dtype=STORE[dtype])
        checkpoint = Checkpoint(folder)
        tensors = {n: checkpoint.read(n) for n in checkpoint.names()}
        for index, layer in enumerate(config.layers):                   # sharper attention than the draw gives
            if layer.type == "latent_attention":
                tensors[f"l{index}.mix.q"] = (tensors[f"l{index}.mix.q"].float() * 3.0).to(STORE[dtype])
        write_safetensors(Path(folder) / "model.safetensors", tensors)
        weights = {n: t.float() for n, t in tensors.items()}
        engine = Engine.from_pretrained(folder, dtype=dtype, max_tokens=2048, max_step_tokens=random.Random(seed).choice([96, 512, 4096]))
    if "streams" not in raw:                       # the plain residual sum, in the plain implementation's terms
        for index in range(len(config.layers)):
            for q in ("hc1", "hc2"):
                weights |= {f"l{index}.{q}.in": torch.ones(1), f"l{index}.{q}.out": torch.ones(1), f"l{index}.{q}.mix": torch.ones(1, 1)}
        raw["streams"] = 1
    generator = torch.Generator().manual_seed(seed)
    lengths = (200, 1, 70)
    requests = [torch.randint(0, config.vocab_size, (n + 8,), generator=generator).tolist() for n in lengths]
    wants, clear = [], []
    for r in requests:
        margins = []
        wants.append(plain.forward(raw, weights, r, margins=margins).float())
        clear.append(torch.stack(margins).min(dim=0).values >= CLOSE_CALL if margins and dtype == "bf16" else torch.ones(len(r), dtype=torch.bool))
    what = f"seed {seed}: {raw}"

    def close(actual, request, rows, text):
        actual = actual.float().cpu()
        assert bool(torch.isfinite(actual).all()), text
        keep = clear[request][rows]
        if bool(keep.any()):
            close_all(actual[keep], wants[request][rows][keep], dtype, text, model_rows=True)

    # whole, then the same request with its last 40 tokens one by one, then in portions of 19
    slot = engine.new_sequence()
    close(engine.step([StepEntry(slot, requests[0], list(range(len(requests[0]))))]), 0, slice(None), "whole, " + what)
    engine.release(slot)
    slot = engine.new_sequence()
    head = len(requests[0]) - 40
    rows = [engine.step([StepEntry(slot, requests[0][:head], [head - 1])])]
    rows += [engine.step([StepEntry(slot, [t], [0])]) for t in requests[0][head:]]
    engine.release(slot)
    close(torch.cat(rows), 0, slice(head - 1, None), "token by token, " + what)
    slot = engine.new_sequence()
    rows = []
    for begin in range(0, len(requests[0]), 19):
        piece = requests[0][begin:begin + 19]
        rows.append(engine.step([StepEntry(slot, piece, list(range(len(piece))))]))
    engine.release(slot)
    close(torch.cat(rows), 0, slice(None), "in portions, " + what)
    # an unequal batch, then eight tokens each
    slots = [engine.new_sequence() for _ in requests]
    rows = [[] for _ in requests]
    out = engine.step([StepEntry(s, r[:n], [n - 1]) for s, r, n in zip(slots, requests, lengths)])
    for i in range(len(requests)):
        rows[i].append(out[i:i + 1])
    for t in range(8):
        out = engine.step([StepEntry(s, [r[n + t]], [0]) for s, r, n in zip(slots, requests, lengths)])
        for i in range(len(requests)):
            rows[i].append(out[i:i + 1])
    for i, n in enumerate(lengths):
        close(torch.cat(rows[i]), i, slice(n - 1, None), f"batch row {i}, " + what)
    for s in slots:
        engine.release(s)
    engine.cache.book.check()
    engine.check_kernels()
