"""The Bizurax design on the GPU against the plain implementation (tests/plain_bizurax.py): every mechanism alone at the
kernels, with inputs made so that a fault shows (streams mixed the wrong way round, scores far beyond their cap, a sink that
outweighs every key, a far key, a rotation of the wrong pairs, a state written once and read hundreds of tokens later), single
layers of every kind, then whole models through the engine: whole prompts, token by token, portions down to two tokens, unequal
batches, slots, state rows and pages used again, long decoding, greedy generation through the entry point, the command line and
the trace replay."""
import functools
import json
import math
import subprocess
import sys
import tempfile
from pathlib import Path

import pytest
import torch

import plain_bizurax as plain
from qwen_triton_b200 import Engine, QwenB200ForCausalLM, StepEntry, config_from_dict, load_preset, write_random_model
from qwen_triton_b200.ops import kernels
from qwen_triton_b200.ops.kernels import GemmOut
from qwen_triton_b200.weights import Checkpoint, write_safetensors
from test_gpu_vunepel import STORE, _Step, close, paged

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = Path(__file__).resolve().parent.parent
DTYPES = ("fp32", "bf16")
PAGE = 64
_KEEP = []

# a third configuration beside the two presets: a width off 8 (no tensor-core products), one stream, no loop, sizes off 8 and off
# 2, values wider than keys, layers that turn nothing, one key channel, one expert, all experts chosen, layers without a feed-forward
ODD = {
    "architecture": "Bizurax", "vocab": 61, "width": 36, "norm": {"eps": 1e-4}, "streams": 1, "residual_mult": 1.3,
    "layers": [
        {"type": "attention", "mlp": {"kind": "dense", "ff": 21},
         "mixer": {"heads": 3, "kv_heads": 1, "dim": 10, "vdim": 14, "scale": 0.5, "softcap": 1.5, "rot": {"base": 70.0, "dims": 2}}},
        {"type": "retention", "mlp": {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 1, "top": 1}, "shared": {"ff": 5}},
         "mixer": {"heads": 2, "dim": 1, "vdim": 9, "decay": [0.99, 0.2]}},
        {"type": "latent_attention", "mlp": None, "mixer": {"heads": 2, "dim": 10, "rot_dim": 6, "vdim": 12, "kv_rank": 11, "scale": 0.4, "rot": {"base": 100.0, "dims": 6}}},
        {"type": "latent_attention", "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 3, "top": 3}},
         "mixer": {"heads": 1, "dim": 7, "rot_dim": 0, "vdim": 5, "kv_rank": 8, "scale": 0.9}},
        {"type": "retention", "mlp": None, "mixer": {"heads": 1, "dim": 100, "vdim": 3, "decay": [1.0], "rot": {"base": 5000.0, "dims": 6, "scaling": {"factor": 4.0}}}},
        {"type": "attention", "mlp": None, "mixer": {"heads": 5, "kv_heads": 5, "dim": 13, "vdim": 13, "scale": 0.7}},
    ],
}
MODELS = ("bizurax-tiny-a", "bizurax-tiny-b", "odd")
CASES = [(name, dtype) for name in MODELS for dtype in DTYPES]


def config_of(name):
    return config_from_dict(ODD) if name == "odd" else load_preset(name)


@functools.lru_cache(maxsize=None)
def model(name: str, dtype: str, peaky: bool = False):
    """(folder, raw config, float weights for the plain implementation).  ``peaky``: the latent layers' queries are four times as
    large, so that few keys, far ones among them, carry each softmax (the other attention's scores are set by its scale)."""
    config = config_of(name)
    holder = tempfile.TemporaryDirectory(prefix=f"qt_{name}_{dtype}_")
    _KEEP.append(holder)
    folder = write_random_model(holder.name, config, seed=23 + len(name), dtype=STORE[dtype])
    if peaky:
        checkpoint = Checkpoint(folder)
        tensors = {n: checkpoint.read(n) for n in checkpoint.names()}
        for index, layer in enumerate(config.layers):
            if layer.type == "latent_attention":
                n = f"l{index}.mix.q"
                tensors[n] = (tensors[n].float() * 4.0).to(tensors[n].dtype)
        write_safetensors(Path(folder) / "model.safetensors", tensors)
    checkpoint = Checkpoint(folder)
    weights = {n: checkpoint.read(n).float() for n in checkpoint.names()}
    return folder, config.to_hf_dict(), weights


@functools.lru_cache(maxsize=None)
def oracle_and_margins(name: str, dtype: str, peaky: bool, tokens: tuple):
    _, raw, weights = model(name, dtype, peaky)
    margins = []
    logits = plain.forward(raw, weights, list(tokens), margins=margins).float()
    return logits, (torch.stack(margins).min(dim=0).values if margins else torch.full((len(tokens),), math.inf, dtype=torch.float64))


def oracle(name: str, dtype: str, peaky: bool, tokens: tuple) -> torch.Tensor:
    return oracle_and_margins(name, dtype, peaky, tokens)[0]


CLOSE_CALL = 0.15      # a router's gap, over the scale of its logits, below which bfloat16 may choose otherwise


def close_rows(actual, name, dtype, peaky, tokens, rows, what):
    """The engine's logits for the positions ``rows`` (a slice) of a request against the plain implementation's.  float32:
    every element.  bfloat16: per position relative to the logits' scale (the bar of ``close``); positions at which some
    router's choice is nearly a tie in the plain implementation may fall the other way and are only asked to be finite."""
    want, margins = oracle_and_margins(name, dtype, peaky, tuple(tokens))
    want, margins = want[rows], margins[rows]
    if dtype != "bf16":
        return close(actual, want, dtype, what, model_rows=True)
    actual = actual.float().cpu()
    assert actual.shape == want.shape and bool(torch.isfinite(actual).all()), what
    clear = margins >= CLOSE_CALL
    if bool(clear.any()):
        close(actual[clear], want[clear], dtype, what, model_rows=True)


def tokens_of(name: str, length: int, seed: int) -> list[int]:
    generator = torch.Generator().manual_seed(733 + seed)
    return torch.randint(0, config_of(name).vocab_size, (length,), generator=generator).tolist()


def engine_of(name, dtype, peaky=False, **kwargs) -> Engine:
    kwargs.setdefault("max_tokens", 2048)
    return Engine.from_pretrained(model(name, dtype, peaky)[0], dtype=dtype, **kwargs)


def as_int(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


# ============================================================================= mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, streams, width, splits", [(5, 1, 7, 1), (3, 2, 96, 3), (300, 3, 96, 1), (2, 4, 1000, 2), (17, 5, 1024, 16), (1, 8, 4100, 4),
                                                            (260, 4, 2048, 1), (9, 3, 1030, 2), (4, 9, 40, 2), (2, 3, 17000, 1), (257, 7, 1024, 2), (3, 6, 64, 1)])
def test_what_is_between_two_sublayers(dtype, tokens, streams, width, splits):
    """The update of the streams, the read and its norm; the mix is far from symmetric, so [to, from] in its place would show."""
    torch.manual_seed(width + streams)
    x = torch.randn(tokens, streams, width)
    y = torch.randn(splits, tokens, width)
    t = {"c.in": torch.randn(streams), "c.mix": torch.randn(streams, streams), "c.out": torch.randn(streams)}
    nxt = torch.randn(streams)
    weight = torch.randn(width) * 0.2 + 1.0
    d = {n: v.double() for n, v in t.items()}
    new = plain.write_streams(x.double().transpose(0, 1), y.double().sum(0), d, "c", 0.3)                 # [S, T, W]
    on = {n: v.to(DEV) for n, v in t.items()}
    out_weight = (t["c.out"] * 0.3).to(DEV)
    for read in (nxt, None):
        factor = read.double() if read is not None else torch.ones(streams, dtype=torch.float64)
        want = plain.rms_norm(plain.read_streams(new, {"n.in": factor}, "n"), 1e-3, weight.double())
        have = x.to(DEV)
        out = torch.empty(tokens, width, dtype=STORE[dtype], device=DEV)
        dev_read = read.to(DEV) if read is not None else None
        kernels.streams_norm(have, GemmOut(y.to(DEV)), on["c.mix"], out_weight, dev_read, weight.to(DEV), 1e-3, out)
        close(out, want, dtype, "normed read")
        torch.testing.assert_close(have.cpu().double(), new.transpose(0, 1), atol=2e-5 * streams, rtol=1e-4)
        # listed rows only: the streams stay as they are
        have = x.to(DEV)
        rows = [tokens - 1, 0, tokens // 2]
        out = torch.empty(3, width, dtype=STORE[dtype], device=DEV)
        kernels.streams_norm(have, GemmOut(y.to(DEV)), on["c.mix"], out_weight, dev_read, weight.to(DEV), 1e-3, out, as_int(rows))
        close(out, want[rows], dtype, "listed rows")
        assert torch.equal(have.cpu(), x)
        # nothing to add
        kernels.streams_norm(have, None, None, None, dev_read, weight.to(DEV), 1e-3, out, as_int(rows))
        still = plain.rms_norm(plain.read_streams(x.double().transpose(0, 1), {"n.in": factor}, "n"), 1e-3, weight.double())
        close(out, still[rows], dtype, "nothing added")
        assert torch.equal(have.cpu(), x)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_embedding_starts_every_stream(dtype):
    table = torch.randn(20, 70).to(STORE[dtype])
    ids = torch.tensor([3, 19, 0, 3], dtype=torch.int32)
    streams = torch.full((4, 3, 70), 9.0, device=DEV)
    kernels.embedding(streams, table.to(DEV), ids.to(DEV))
    assert torch.equal(streams.cpu(), table.float()[ids.long()][:, None].expand(4, 3, 70))


def attention_oracle(q, k, v, scale, softcap, sinks):
    total, heads, _ = q.shape
    group = heads // k.shape[1]
    out = torch.zeros(total, heads, v.shape[-1], dtype=torch.float64)
    for h in range(heads):
        score = plain.cap(q[:, h].double() @ k[:, h // group].double().T * scale, softcap)
        out[:, h] = plain.causal_softmax(score, None if sinks is None else sinks[h].double()) @ v[:, h // group].double()
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, d, dv, scale, softcap, unit, sink", [
    (4, 2, 64, 64, 0.11, 41.0, True, True), (4, 1, 128, 128, 0.25, 7.0, False, True), (6, 2, 128, 128, 0.0884, 15.0, True, True),
    (3, 3, 64, 64, 0.5, 2.0, False, False), (8, 2, 32, 32, 0.3, 12.0, True, True), (20, 1, 48, 48, 0.2, 3.0, False, True),
    (2, 1, 40, 24, 0.4, 5.0, True, True), (4, 4, 10, 30, 0.7, 1.0, False, True), (4, 2, 64, 64, 0.2, None, False, True), (2, 2, 128, 128, 0.1, None, False, True), (4, 1, 96, 96, 0.15, 20.0, True, True),
    (6, 3, 80, 80, 0.3, 4.0, False, True), (2, 1, 256, 256, 0.06, 9.0, False, True)])
def test_attention_with_capped_scores_and_a_sink(dtype, heads, kv_heads, d, dv, scale, softcap, unit, sink):
    """300 positions over pages in no order: a prompt, a late portion of it, single tokens with several counts of key ranges.  Key
    5 is seen by every later query with a score far above all others (beyond the cap where queries and keys are not unit), and
    key 130 with one far below; the sinks range from nothing to more than every key."""
    torch.manual_seed(heads + d)
    store, total = STORE[dtype], 300
    q, k, v = torch.randn(total, heads, d), torch.randn(total, kv_heads, d), torch.randn(total, kv_heads, dv)
    q[:, :, 0] = 3.0
    k[5] = torch.nn.functional.one_hot(torch.tensor(0), d) * (25.0 if not unit else 4.0)
    k[130] = -k[5]
    if unit:
        q, k = plain.rms_norm(q, 1e-6), plain.rms_norm(k, 1e-6)
    q, k, v = (x.to(store).float() for x in (q, k, v))
    sinks = torch.linspace(-6.0, 12.0, heads) if sink else None
    want = attention_oracle(q, k, v, scale, softcap, sinks)
    order = [3, 1, 4, 0, 2]
    k_pool, v_pool, table = paged(k, PAGE, order, store), paged(v, PAGE, order, store), as_int([order])
    on = dict(sinks=sinks.to(DEV) if sink else None, softcap=softcap)
    bound = d * scale if unit else None
    tc = dtype == "bf16" and d == dv and d <= 128                # what the tensor-core kernels take, in steps of 16
    for begin in (0, 190, 298):
        for impl in [None, "generic"] + (["mma"] if tc and d % 16 == 0 else []) + (["tc"] if tc and d in (64, 128) else []):
            for known in {None, bound}:
                out = torch.full((total - begin, heads, dv), float("nan"), dtype=store, device=DEV)
                kernels.attention_prefill(q[begin:].to(DEV, store), k_pool, v_pool, out, table, as_int([0, total - begin]), as_int([begin]), total - begin, kv_heads,
                                          PAGE, 0, None, scale, impl=impl, score_bound=known, **on)
                close(out, want[begin:], dtype, f"{impl}: portion from {begin}, bound {known}")
    for t in (0, 5, 63, 64, 128, 130, 256, 299):
        for impl in [None, "generic"] + (["ws"] if tc and d % 16 == 0 else []):
            for splits, warps in ((1, 1), (3, 4), (9, 2)):
                out = torch.full((1, heads, dv), float("nan"), dtype=store, device=DEV)
                kernels.attention_decode(q[t:t + 1].to(DEV, store), k_pool, v_pool, out, table, as_int([t + 1]), kv_heads, PAGE, 0, None, scale, splits,
                                         torch.empty(9 * heads * dv, device=DEV), torch.empty(18 * heads, device=DEV), impl=impl, warps=warps, score_bound=bound, **on)
                close(out, want[t:t + 1], dtype, f"{impl}: token {t}, {splits} ranges")
    kernels.check_status(DEV)


def test_the_two_forms_of_the_cap_agree_with_tanh():
    """Queries and keys of one element in many sizes: one visible key's score against a second key of score 0, read back as the ratio
    of their softmax weights, for scores from tiny to many times the cap."""
    scale, softcap, d = 0.5, 6.0, 64
    sizes = torch.cat((torch.linspace(-12.0, 12.0, 63), torch.tensor([400.0, -400.0])))
    n = sizes.numel()
    q = torch.zeros(n, 1, d)
    q[:, 0, 0] = sizes
    k, v = torch.zeros(2, 1, d), torch.zeros(2, 1, d)
    k[0, 0, 0] = 1.0
    v[0, 0, 0], v[1, 0, 1] = 1.0, 1.0
    k_pool, v_pool = paged(k, PAGE, [1], torch.bfloat16), paged(v, PAGE, [1], torch.bfloat16)
    q16 = q.to(torch.bfloat16)
    score = plain.cap(q16[:, 0, 0].double() * scale, softcap)
    for bound, keep in ((None, slice(None)), (softcap / 1.02, q16[:, 0, 0].float().abs() * scale <= softcap)):
        for impl in ("ws", "generic"):
            out = torch.empty(n, 1, d, dtype=torch.bfloat16, device=DEV)
            kernels.attention_decode(q16.to(DEV), k_pool, v_pool, out, as_int([[1]] * n), as_int([2] * n), 1, PAGE, 0, None, scale, 1, None, None, impl=impl,
                                     softcap=softcap, score_bound=bound)
            got = out.float().cpu()[keep, 0].double()
            want = torch.stack((torch.sigmoid(score), torch.sigmoid(-score)), dim=-1)[keep]
            torch.testing.assert_close(got[:, :2], want, atol=4e-3, rtol=1e-2)


@pytest.mark.parametrize("heads, dim, rd, v_cols, splits", [(4, 24, 24, 40, 1), (6, 16, 8, 12, 3), (2, 10, 6, 7, 2), (8, 64, 64, 256, 1), (2, 1 + 1, 2, 1, 1), (6, 20, 12, 4, 4)])
def test_rotated_rows_of_a_recurrence(heads, dim, rd, v_cols, splits):
    torch.manual_seed(dim)
    tokens, cols, extra = 37, heads * dim + v_cols, 5
    parts = torch.randn(splits, tokens, cols + extra)
    positions = torch.randperm(500)[:tokens]
    from qwen_triton_b200.config import PartSpec
    from qwen_triton_b200.parts.base import Runtime, Workspace, part_class
    runtime = Runtime(device=torch.device(DEV), dtype=torch.float32, max_step_tokens=64, max_positions=512, workspace=Workspace(torch.device(DEV)))
    spec = PartSpec("rope", {"theta": 300.0, "rotary_dim": rd, "head_dim": dim, "angles": "float64", "factor": 2.5})
    table = part_class("position", spec)(spec.params, runtime).table(512)
    out = torch.full((tokens, cols), float("nan"), device=DEV)
    kernels.linear_attention_rotate(GemmOut(parts.to(DEV)), cols, out, heads, dim, table, positions.int().to(DEV))
    sums = parts.double().sum(0)
    want = plain.rotate(sums[:, :heads * dim].view(tokens, heads, dim), positions, rd, 300.0, 2.5).reshape(tokens, -1)
    torch.testing.assert_close(out.cpu().double(), torch.cat((want, sums[:, heads * dim:cols]), dim=-1), atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, width", [(3, 40), (200, 72), (5, 7)])
def test_squared_relu(dtype, rows, width):
    x = torch.randn(2, rows, width) * 2.0
    out = torch.empty(rows, width, dtype=STORE[dtype], device=DEV)
    kernels.activation(GemmOut(x.to(DEV)), out, "relu2")
    close(out, torch.relu(x.double().sum(0)).square(), dtype, "relu2")


@pytest.mark.parametrize("activation, function", [("relu2", lambda z: torch.relu(z).square()), ("gelu", lambda z: 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0))))])
@pytest.mark.parametrize("rows", [1, 3, 16, 40, 300, 700])
def test_an_activation_in_the_products_epilogues(rows, activation, function):
    """Without a gate, in each tensor-core kernel; sizes whose last tiles are partial."""
    torch.manual_seed(rows)
    width, inter = 192, 172
    x, w, b = torch.randn(rows, width).to(torch.bfloat16), (torch.randn(inter, width) * 0.1).to(torch.bfloat16), torch.randn(inter)
    want = function(x.double() @ w.double().T + b.double())
    out = torch.empty(rows, inter, dtype=torch.bfloat16, device=DEV)
    for product in (kernels.gemm_tc, kernels.gemm_tc_pair):
        out.fill_(float("nan"))
        product(x.to(DEV), w.to(DEV), GemmOut(out.view(1, rows, inter)), activate=True, activation=activation, bias=b.to(DEV))
        close(out, want, "bf16", product.__name__)
    if rows <= 16:
        out.fill_(float("nan"))
        kernels.gemm_fused_store(x.to(DEV), w.to(DEV), out, splits=3, bias=b.to(DEV), activation=activation)
        close(out, want, "bf16", "fused")
    kernels.check_status(DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [3, 90, 400])
def test_the_feed_forwards_alone(dtype, tokens):
    """The dense feed-forward and the routed ones, with and without a shared expert, as parts, few and many tokens.  The router's
    bias outweighs its logits for one expert, which a router without it would hardly choose."""
    from qwen_triton_b200.parts.base import Runtime, Workspace, part_class
    torch.manual_seed(tokens)
    store, width, device = STORE[dtype], 96, torch.device(DEV)
    mixer = ODD["layers"][1]["mixer"]
    mlps = [{"kind": "dense", "ff": 112}, {"kind": "moe", "expert": {"ff": 40}, "router": {"experts": 8, "top": 2}, "shared": {"ff": 48}},
            {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 1}}]
    raw = {**ODD, "width": width, "layers": [{"type": "retention", "mixer": mixer, "mlp": mlp} for mlp in mlps]}
    for mlp, layer in zip(mlps, config_from_dict(raw).model_spec().layers):
        runtime = Runtime(device=device, dtype=store, max_step_tokens=512, max_positions=64, workspace=Workspace(device))
        cls = part_class("feed_forward", layer.feed_forward)
        part = cls(layer.feed_forward.params, "p", runtime)
        tensors = {n: (torch.randn(*s.shape) * (1.0 if n.endswith("router") else 0.2)).to(store)
                   for n, s in cls.expected_tensors(layer.feed_forward.params, "p").items()}
        if "p.router.b" in tensors:
            tensors["p.router.b"][3] = 25.0
        part.load(lambda name: tensors[name])
        runtime.workspace.allocate()
        x = torch.randn(tokens, width).to(store)
        result = part.forward(x.to(DEV), None)
        got = result.value().cpu().double()
        t = {n: v.double() for n, v in tensors.items()}
        margins = []
        want = plain.dense(x.double(), t, "p") if mlp["kind"] == "dense" else plain.experts(x.double(), t, "p", mlp, margins)
        if dtype == "fp32":
            torch.testing.assert_close(got, want, atol=5e-4, rtol=5e-4)
        else:
            off = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
            if margins:
                off = off[margins[0] > 0.02]
            assert float(off.mean()) < 0.02 and float(off.max()) < 0.1, f"{mlp}: mean {float(off.mean()):.4f}, worst {float(off.max()):.4f}"
    kernels.check_status(DEV)


@pytest.mark.parametrize("impl", ["steps", "chunks"])
def test_a_state_with_fixed_decays_in_portions(impl):
    """Three unequal sequences, states in rows that are not in order, decays of 1, of 0.9995 and of 0.02 side by side; the first
    token's key alone meets the last token's query hundreds of tokens later."""
    heads, dim, vdim = 3, 40, 24
    decay = torch.tensor([1.0, 0.9995, 0.02], dtype=torch.float64)
    lengths, slots = (400, 1, 85), (3, 0, 1)
    torch.manual_seed(1)
    rows = [torch.randn(n, 2 * heads * dim + heads * vdim) for n in lengths]
    rows[0][0, heads * dim:heads * dim + dim] = 50.0
    want = []
    for r in rows:
        q, k = (r[:, i * heads * dim:(i + 1) * heads * dim].double().view(-1, heads, dim) for i in (0, 1))
        want.append(plain.fixed_decay_recurrence(q, k * dim ** -0.5, r[:, 2 * heads * dim:].double().view(-1, heads, vdim), decay))
    logs = decay.log().float().to(DEV)
    for portions in ((1000, 1, 1000), (64, 1, 20), (33, 1, 64), (131, 1, 2)):
        states = torch.full((6, heads, vdim, dim), 55.0, device=DEV)
        states[list(slots)] = 0.0
        scratch = {n: torch.full((numel,), float("nan"), device=DEV) for n, numel in kernels.decay_scratch(1024, heads, dim, vdim, False).items()}
        done, got = [0, 0, 0], [[], [], []]
        while any(d < n for d, n in zip(done, lengths)):
            count = [min(p, n - d) for p, n, d in zip(portions, lengths, done)]
            live = [s for s in range(3) if count[s] > 0]
            step = _Step([count[s] for s in live], [done[s] for s in live], [slots[s] for s in live])
            piece = torch.cat([rows[s][done[s]:done[s] + count[s]] for s in live]).to(DEV).contiguous()
            out = torch.full((piece.shape[0], heads, vdim), float("nan"), device=DEV)
            kernels.decayed_attention(GemmOut(piece[None]), 0, heads * dim, 2 * heads * dim, logs.expand(piece.shape[0], heads).contiguous(), states, out, step, dim,
                                      scratch, out_scale=dim ** -0.5, impl=impl)
            at = 0
            for s in live:
                got[s].append(out[at:at + count[s]].cpu())
                at += count[s]
                done[s] += count[s]
        for s in range(3):
            error = float((torch.cat(got[s]).double() - want[s]).abs().max())
            assert error < 1e-4 * float(want[s].abs().max()), f"sequence {s} in portions of {portions}: {error}"
        assert float((states[[2, 4, 5]] - 55.0).abs().max()) == 0.0


def run_whole(engine, tokens):
    slot = engine.new_sequence()
    try:
        return engine.step([StepEntry(slot, list(tokens), list(range(len(tokens))))])
    finally:
        engine.release(slot)


# ============================================================================= one layer of each kind
LAYERS = {
    # unit-norm queries and keys: a score is scale * dim * cosine, so a large scale makes far keys stand out beneath a wide and a narrow cap
    "capped": {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.5, "softcap": 40.0, "rot": {"base": 900.0, "dims": 64}}},
    "narrow cap": {"type": "attention", "mixer": {"heads": 4, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": 0.5, "softcap": 5.0, "rot": {"base": 900.0, "dims": 40}}},
    "stretched": {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 1.0, "rot": {"base": 60.0, "dims": 32, "scaling": {"factor": 7.0}}}},
    "other values": {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 24, "vdim": 56, "scale": 0.8, "softcap": 11.0, "rot": {"base": 400.0, "dims": 8}}},
    "latent": {"type": "latent_attention", "mixer": {"heads": 4, "dim": 32, "rot_dim": 16, "vdim": 40, "kv_rank": 64, "scale": 1.5, "rot": {"base": 700.0, "dims": 16}}},
    "latent, many heads": {"type": "latent_attention", "mixer": {"heads": 33, "dim": 16, "rot_dim": 24, "vdim": 8, "kv_rank": 136, "scale": 1.0,
                                                                 "rot": {"base": 50.0, "dims": 24, "scaling": {"factor": 3.0}}}},
    "retention": {"type": "retention", "mixer": {"heads": 3, "dim": 48, "vdim": 32, "decay": [0.99999, 0.98, 0.6], "rot": {"base": 800.0, "dims": 48}}},
    "retention, few turn": {"type": "retention", "mixer": {"heads": 2, "dim": 130, "vdim": 72, "decay": [1.0, 0.999], "rot": {"base": 30.0, "dims": 6}}},
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", LAYERS)
def test_one_layer_whole_and_token_by_token(kind, dtype):
    """A model of one mixer and nothing else, over 200 tokens: the prompt whole, in portions of 2 and 50, and token by token from
    token 120 on."""
    config = config_from_dict({"architecture": "Bizurax", "vocab": 50, "width": 64, "norm": {"eps": 1e-5}, "streams": 2, "residual_mult": 0.9,
                               "layers": [{**LAYERS[kind], "mlp": None}]})
    tokens = torch.randint(0, 50, (200,), generator=torch.Generator().manual_seed(8)).tolist()
    with tempfile.TemporaryDirectory() as holder:
        folder = write_random_model(holder, config, seed=3, dtype=STORE[dtype])
        checkpoint = Checkpoint(folder)
        want = plain.forward(config.to_hf_dict(), {n: checkpoint.read(n).float() for n in checkpoint.names()}, tokens).float()
        engine = Engine.from_pretrained(folder, dtype=dtype, max_tokens=1024)
    close(run_whole(engine, tokens), want, dtype, f"{kind}, whole", model_rows=True)
    for portion in (2, 50):
        slot = engine.new_sequence()
        rows = []
        for begin in range(0, 200, portion):
            rows.append(engine.step([StepEntry(slot, tokens[begin:begin + portion], list(range(portion)))]))
        engine.release(slot)
        close(torch.cat(rows), want, dtype, f"{kind}, portions of {portion}", model_rows=True)
    slot = engine.new_sequence()
    rows = [engine.step([StepEntry(slot, tokens[:120], [119])])] + [engine.step([StepEntry(slot, [t], [0])]) for t in tokens[120:]]
    close(torch.cat(rows), want[119:], dtype, f"{kind}, token by token", model_rows=True)
    engine.check_kernels()


# ============================================================================= whole models through the engine
@pytest.mark.parametrize("name, dtype", CASES)
def test_each_request_alone_and_whole(name, dtype):
    engine = engine_of(name, dtype, peaky=True)
    for length, seed in ((1, 0), (7, 1), (150, 2)):
        tokens = tokens_of(name, length, seed)
        close_rows(run_whole(engine, tokens), name, dtype, True, tokens, slice(None), f"{name} {length} tokens")
    engine.check_kernels()


@pytest.mark.parametrize("name, dtype", CASES)
def test_prompt_then_token_by_token_across_page_edges(name, dtype):
    """A prompt of 20 tokens, then 130 one by one: positions 63 to 65, 127 and 128 among them."""
    engine = engine_of(name, dtype, peaky=True)
    tokens = tokens_of(name, 150, 3)
    slot = engine.new_sequence()
    rows = [engine.step([StepEntry(slot, tokens[:20], [19])])]
    rows += [engine.step([StepEntry(slot, [t], [0])]) for t in tokens[20:]]
    engine.release(slot)
    close_rows(torch.cat(rows), name, dtype, True, tokens, slice(19, None), name)
    engine.check_kernels()


@pytest.mark.parametrize("name, dtype", CASES)
def test_token_by_token_from_the_first_token(name, dtype):
    engine = engine_of(name, dtype)
    tokens = tokens_of(name, 24, 4)
    slot = engine.new_sequence()
    rows = [engine.step([StepEntry(slot, [t], [0])]) for t in tokens]
    engine.release(slot)
    close_rows(torch.cat(rows), name, dtype, False, tokens, slice(None), name)


@pytest.mark.parametrize("name, dtype", CASES)
@pytest.mark.parametrize("portion", [2, 3, 17, 64, 100])
def test_portions_of_a_prompt(name, dtype, portion):
    engine = engine_of(name, dtype, peaky=True)
    tokens = tokens_of(name, 140, 5)
    slot = engine.new_sequence()
    rows = []
    for begin in range(0, len(tokens), portion):
        piece = tokens[begin:begin + portion]
        rows.append(engine.step([StepEntry(slot, piece, list(range(len(piece))))]))
    engine.release(slot)
    close_rows(torch.cat(rows), name, dtype, True, tokens, slice(None), f"{name} in portions of {portion}")
    engine.check_kernels()


@pytest.mark.parametrize("name, dtype", CASES)
def test_passes_smaller_than_a_prompt(name, dtype):
    """Passes of 96 tokens cut the prompt; 300 tokens take the products' many-row forms."""
    tokens = tokens_of(name, 300, 6)
    for options in ({"max_step_tokens": 96}, {"max_step_tokens": 4096}):
        engine = engine_of(name, dtype, peaky=True, **options)
        close_rows(run_whole(engine, tokens), name, dtype, True, tokens, slice(None), f"{name}, {options}")
        engine.check_kernels()


@pytest.mark.parametrize("name, dtype", CASES)
def test_unequal_batches_with_slots_states_and_pages_used_again(name, dtype):
    """Three unequal requests start together and are decoded together; one ends early; a fourth takes the slot, state rows and
    pages that were given back, and must find states of zero there."""
    engine = engine_of(name, dtype, peaky=True, max_tokens=640)
    lengths, more = (70, 1, 129), (6, 3, 9)
    requests = [tokens_of(name, n + m, 10 + i) for i, (n, m) in enumerate(zip(lengths, more))]
    slots = [engine.new_sequence() for _ in requests]
    got = [[] for _ in requests]
    out = engine.step([StepEntry(s, r[:n], [n - 1]) for s, r, n in zip(slots, requests, lengths)])
    for i in range(3):
        got[i].append(out[i:i + 1])
    live = [0, 1, 2]
    for t in range(max(more)):
        for i in list(live):
            if t >= more[i]:
                engine.release(slots[i])
                live.remove(i)
        out = engine.step([StepEntry(slots[i], [requests[i][lengths[i] + t]], [0]) for i in live])
        for row, i in enumerate(live):
            got[i].append(out[row:row + 1])
    late = tokens_of(name, 90, 20)
    slot = engine.new_sequence()
    assert slot in slots[:2]
    rows = engine.step([StepEntry(slot, late, list(range(90))), StepEntry(slots[2], [requests[2][-1]], [])])
    close_rows(rows, name, dtype, True, late, slice(None), f"{name}: a request in a slot used again")
    for i, (n, req) in enumerate(zip(lengths, requests)):
        close_rows(torch.cat(got[i]), name, dtype, True, req, slice(n - 1, n + more[i]), f"{name} batch row {i}")
    engine.release(slot)
    engine.release(slots[2])
    engine.cache.book.check()
    engine.check_kernels()


@pytest.mark.parametrize("name, dtype", [("bizurax-tiny-a", "fp32"), ("bizurax-tiny-a", "bf16"), ("bizurax-tiny-b", "bf16"), ("odd", "fp32")])
def test_many_short_requests_at_once(name, dtype):
    """Twenty-one requests of 2 to 24 tokens, then a batch of 70 (more ends of chunks than the scratch of short steps holds)."""
    engine = engine_of(name, dtype, peaky=True, max_tokens=8192, max_step_tokens=2048)
    for count, step in ((21, 5), (70, 7)):
        requests = [tokens_of(name, 2 + (step * i) % 23, 30 + i) for i in range(count)]
        slots = [engine.new_sequence() for _ in requests]
        out = engine.step([StepEntry(s, r[:-1], list(range(len(r) - 1))) for s, r in zip(slots, requests)])
        last = engine.step([StepEntry(s, r[-1:], [0]) for s, r in zip(slots, requests)])
        at = 0
        for i, req in enumerate(requests):
            rows = torch.cat([out[at:at + len(req) - 1], last[i:i + 1]])
            at += len(req) - 1
            if i % (count // 10) == 0:
                close_rows(rows, name, dtype, True, req, slice(None), f"{name} request {i} of {count}")
        for slot in slots:
            engine.release(slot)
    engine.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_of_several_rows(dtype):
    """Five rows decoded for 150 steps from short prompts: the states carry 150 updates."""
    name = "bizurax-tiny-a"
    engine = engine_of(name, dtype, peaky=True)
    requests = [tokens_of(name, 1 + 2 * i + 150, 40 + i) for i in range(5)]
    slots = [engine.new_sequence() for _ in requests]
    engine.step([StepEntry(slot, req[:1 + 2 * i], []) for i, (slot, req) in enumerate(zip(slots, requests))])
    last = None
    for step in range(150):
        last = engine.step([StepEntry(slot, [req[1 + 2 * i + step]], [0]) for i, (slot, req) in enumerate(zip(slots, requests))]).cpu()
    for i, req in enumerate(requests):
        close_rows(last[i:i + 1], name, dtype, True, req, slice(len(req) - 1, None), f"row {i} after 150 steps")
    engine.check_kernels()


@pytest.mark.parametrize("name", MODELS)
def test_greedy_generation_through_the_entry_point(name):
    folder, _, _ = model(name, "fp32")
    lm = QwenB200ForCausalLM.from_pretrained_hf(folder, dtype="fp32", max_tokens=1024)
    prompts = [tokens_of(name, n, 60 + n) for n in (5, 1, 40)]
    results = lm.generate(prompts, max_new_tokens=12, ignore_eos=True)
    for prompt, result in zip(prompts, results):
        assert len(result.tokens) == 12
        sequence = list(prompt)
        for token in result.tokens:
            logits = oracle(name, "fp32", False, tuple(sequence))[-1]
            best = logits.topk(2).values
            if float(best[0] - best[1]) > 1e-3:          # a clear choice: the library must have made it
                assert int(logits.argmax()) == token, f"{name}: after {len(sequence)} tokens"
            sequence.append(token)
    lm16 = QwenB200ForCausalLM.from_pretrained_hf(model(name, "bf16")[0], dtype="bf16", max_tokens=1024)
    for result in lm16.generate(prompts, max_new_tokens=12, ignore_eos=True, temperature=0.7, seed=3):
        assert len(result.tokens) == 12 and all(0 <= t < config_of(name).vocab_size for t in result.tokens)


def test_the_plain_residual_sum_where_streams_are_absent():
    """Without ``streams`` a layer adds its sublayers times the constant: the same logits as one stream read, kept and written with 1."""
    raw = {k: v for k, v in load_preset("bizurax-tiny-a").to_hf_dict().items() if k != "streams"}
    config = config_from_dict(raw)
    tokens = tokens_of("bizurax-tiny-a", 60, 80)
    with tempfile.TemporaryDirectory() as holder:
        folder = write_random_model(holder, config, seed=5, dtype=torch.float32)
        checkpoint = Checkpoint(folder)
        weights = {n: checkpoint.read(n).float() for n in checkpoint.names()}
        engine = Engine.from_pretrained(folder, dtype="fp32", max_tokens=512)
    assert not any(".hc" in n for n in weights)
    for index in range(len(config.layers)):
        for q in ("hc1", "hc2"):
            weights |= {f"l{index}.{q}.in": torch.ones(1), f"l{index}.{q}.out": torch.ones(1), f"l{index}.{q}.mix": torch.ones(1, 1)}
    close(run_whole(engine, tokens), plain.forward({**raw, "streams": 1}, weights, tokens).float(), "fp32", "no streams", model_rows=True)


def test_random_weights_on_the_device_equal_the_written_folder():
    name = "bizurax-tiny-b"
    folder, _, _ = model(name, "bf16")
    tokens = tokens_of(name, 50, 70)
    written = run_whole(Engine.from_pretrained(folder, dtype="bf16", max_tokens=512), tokens)
    drawn = run_whole(Engine.from_config(config_of(name), seed=23 + len(name), dtype="bf16", max_tokens=512), tokens)
    assert torch.equal(written, drawn)


def test_command_line_with_a_preset_and_random_weights():
    result = subprocess.run([sys.executable, "-m", "qwen_triton_b200.scripts.smoke", "--preset", "bizurax-tiny-a", "--random-weights",
                             "--random-prompts", "9,2", "--max-new-tokens", "5", "--dtype", "bf16"], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert result.returncode == 0, result.stderr[-2000:]


@pytest.mark.parametrize("dtype, name", [("float32", "fp32"), ("bfloat16", "bf16")])
def test_trace_replay_of_a_folder(tmp_path, dtype, name):
    """bin/trace_run as a child process: two requests start together, decode together, one ends earlier; a third comes alone
    afterwards and finds their slots and state rows."""
    import numpy as np
    model_name = "bizurax-tiny-b"
    folder, _, _ = model(model_name, name)
    requests = {"a": tokens_of(model_name, 90, 90), "b": tokens_of(model_name, 31, 91), "c": tokens_of(model_name, 70, 92)}
    a, b, c = requests.values()
    steps = [{"entries": [{"id": "a", "tokens": a[:80], "want": [0, 63, 64, 79]}, {"id": "b", "tokens": b[:30], "want": [29]}], "end": []},
             {"entries": [{"id": "a", "tokens": [a[80]], "want": [0]}, {"id": "b", "tokens": [b[30]], "want": [0]}], "end": ["b"]}]
    steps += [{"entries": [{"id": "a", "tokens": [a[i]], "want": [0] if i % 2 else []}], "end": ["a"] if i == 89 else []} for i in range(81, 90)]
    steps.append({"entries": [{"id": "c", "tokens": c, "want": [69]}], "end": ["c"]})
    steps = [{"step": i, **record} for i, record in enumerate(steps)]
    out = tmp_path / "out"
    result = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "160"],
                            input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900, cwd=ROOT)
    assert result.returncode == 0, result.stderr[-2000:]
    assert [line for line in result.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    at = dict.fromkeys(requests, 0)
    for record in steps:
        wanted = [(entry["id"], at[entry["id"]] + w) for entry in record["entries"] for w in entry["want"]]
        for entry in record["entries"]:
            at[entry["id"]] += len(entry["tokens"])
        path = out / f"{record['step']}.f32"
        assert path.exists() == bool(wanted)
        if wanted:
            got = torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(len(wanted), -1).copy())
            for row, (key, place) in zip(got, wanted):
                close_rows(row[None], model_name, name, False, requests[key], slice(place, place + 1), f"step {record['step']}, {key} at {place}")
