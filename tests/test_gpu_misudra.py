"""The Misudra design on the GPU against the plain implementation (tests/plain_misudra.py): every mechanism alone at the
kernels, with inputs made so that a fault shows (a key just outside a window, a far key, a state written once and read
hundreds of tokens later, decays of e^-60 beside decays of 1, a group whose second expert would win), then whole models
through the engine: whole prompts, token by token, portions down to two tokens, unequal batches, slots, state rows and pages
used again, long decoding, greedy generation through the entry point, the command line and the trace replay."""
import functools
import json
import math
import subprocess
import sys
import tempfile
from pathlib import Path

import pytest
import torch

import plain_misudra as plain
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

# a third configuration beside the two presets: a width off 8 (no tensor-core products), a loop over everything that starts
# with the first layer and runs once, latents and ranks off 8, a window of one position and none at all, an unrotated key part
# longer than the rotation, one key channel, a state of 136 rows, a convolution of one tap, one expert, as many chosen as a
# group holds, layers without a feed-forward
ODD = {
    "architecture": "Misudra", "vocab": 61, "width": 36, "norm": {"eps": 1e-4}, "loop": {"start": 0, "stop": 6, "times": 1},
    "layers": [
        {"type": "gla", "mlp": {"kind": "dense", "ff": 21}, "mixer": {"heads": 3, "dim": 1, "vdim": 20, "tau": 0.5, "ranks": {"decay": 1}}},
        {"type": "latent_attention", "mlp": {"kind": "moe", "expert": {"ff": 9, "limit": 3.0}, "router": {"experts": 1, "top": 1}},
         "mixer": {"heads": 2, "dim": 10, "rot_dim": 6, "vdim": 12, "q_rank": 13, "kv_rank": 11, "scale": 0.4, "rot": {"base": 100.0, "dims": 4}}},
        {"type": "mamba2", "mlp": None, "mixer": {"heads": 5, "vdim": 7, "state": 136, "groups": 5, "conv": 1, "norm_groups": 7}},
        {"type": "latent_attention", "mlp": None,
         "mixer": {"heads": 3, "dim": 4, "rot_dim": 2, "vdim": 4, "q_rank": 5, "kv_rank": 6, "scale": 0.6, "mask": {"size": 1}, "rot": {"base": 50.0, "dims": 2}}},
        {"type": "mamba2", "mlp": {"kind": "moe", "expert": {"ff": 12, "limit": 0.5}, "router": {"experts": 6, "top": 3, "groups": {"count": 2, "keep": 1}}},
         "mixer": {"heads": 2, "vdim": 33, "state": 10, "groups": 1, "conv": 7, "norm_groups": 2}},
        {"type": "gla", "mlp": None, "mixer": {"heads": 1, "dim": 100, "vdim": 9, "tau": 16.0, "ranks": {"decay": 3}}},
    ],
}
MODELS = ("misudra-tiny-a", "misudra-tiny-b", "odd")
CASES = [(name, dtype) for name in MODELS for dtype in DTYPES]


def config_of(name):
    return config_from_dict(ODD) if name == "odd" else load_preset(name)


@functools.lru_cache(maxsize=None)
def model(name: str, dtype: str, peaky: bool = False):
    """(folder, raw config, float weights for the plain implementation).  ``peaky``: the query latents' norm weights are four
    times as large, so that few keys, far ones among them, carry each softmax."""
    config = config_of(name)
    holder = tempfile.TemporaryDirectory(prefix=f"qt_{name}_{dtype}_")
    _KEEP.append(holder)
    folder = write_random_model(holder.name, config, seed=17 + len(name), dtype=STORE[dtype])
    if peaky:
        checkpoint = Checkpoint(folder)
        tensors = {n: checkpoint.read(n) for n in checkpoint.names()}
        for n in list(tensors):
            if n.endswith(".dq.norm"):
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
    generator = torch.Generator().manual_seed(377 + seed)
    return torch.randint(0, config_of(name).vocab_size, (length,), generator=generator).tolist()


def engine_of(name, dtype, peaky=False, **kwargs) -> Engine:
    kwargs.setdefault("max_tokens", 2048)
    return Engine.from_pretrained(model(name, dtype, peaky)[0], dtype=dtype, **kwargs)


def as_int(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


# ============================================================================= mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [7, 96, 1000])
def test_normed_embedding_and_the_stream_beside_it(dtype, width):
    """The gather with a norm behind it, its copy, and the rows [stream + what is pending | copy] with the stream zeroed."""
    torch.manual_seed(width)
    store = STORE[dtype]
    table = torch.randn(20, width).to(store)
    ids = torch.tensor([3, 19, 0, 3], dtype=torch.int32)
    weight = torch.randn(width) * 0.2 + 1.0
    stream = torch.empty(4, width, device=DEV)
    start = torch.empty(4, width, dtype=store, device=DEV)
    kernels.embedding(stream, table.to(DEV), ids.to(DEV), 1.0, weight.to(DEV), 1e-3, start)
    want = plain.rms_norm(table.double()[ids.long()], 1e-3, weight.double())
    close(stream, want, "fp32", "normed embedding")
    close(start, want, dtype, "its copy")
    parts = torch.randn(3, 4, width)
    rows = torch.empty(4, 2 * width, dtype=store, device=DEV)
    kernels.stream_concat(stream, GemmOut(parts.to(DEV)), start, rows)
    close(rows, torch.cat((want + parts.double().sum(0), start.double().cpu()), dim=-1), dtype, "stream beside its start")
    assert float(stream.abs().max()) == 0.0


@pytest.mark.parametrize("rows", [3, 16, 40, 100, 300, 700])
def test_biases_in_the_products_epilogues(rows):
    """A bias ahead of the tanh-GELU gate and one on float sums (whole and split over K) in each tensor-core kernel, and on the
    sums added to the stream by the cluster-fused product."""
    torch.manual_seed(rows)
    width, inter, out_width = 192, 160, 132
    x = torch.randn(rows, width).to(torch.bfloat16)
    gate, up = (torch.randn(inter, width) * 0.1).to(torch.bfloat16), (torch.randn(inter, width) * 0.1).to(torch.bfloat16)
    gb, ub = torch.randn(inter), torch.randn(inter) * 2.0
    want = plain.gelu_tanh(x.double() @ gate.double().T + gb.double()) * (x.double() @ up.double().T + ub.double())
    weight = kernels.interleave_gate_up(gate, up, kernels.SWIGLU_GROUP).to(DEV).contiguous()
    bias = kernels.interleave_gate_up(gb[:, None], ub[:, None], kernels.SWIGLU_GROUP).reshape(-1).to(DEV).contiguous()
    out = torch.empty(rows, inter, dtype=torch.bfloat16, device=DEV)
    options = dict(activation="gelu_pytorch_tanh", bias=bias)
    for product in (kernels.gemm_tc, kernels.gemm_tc_pair):
        out.zero_()
        product(x.to(DEV), weight, GemmOut(out.view(1, rows, inter)), swiglu=True, **options)
        close(out, want, "bf16", f"gate, {product.__name__}")
    sums = torch.empty(1, rows, 2 * inter, device=DEV)
    kernels.gemm_tc(x.to(DEV), weight, GemmOut(sums))
    kernels.swiglu(GemmOut(sums), out, kernels.SWIGLU_GROUP, **options)
    close(out, want, "bf16", "gate kernel")
    w = (torch.randn(out_width, width) * 0.1).to(torch.bfloat16)
    b = torch.randn(out_width)
    want = x.double() @ w.double().T + b.double()
    for product in (kernels.gemm_tc, kernels.gemm_tc_pair):
        for splits in (1, 3):
            got = torch.empty(splits, rows, out_width, device=DEV)
            product(x.to(DEV), w.to(DEV), GemmOut(got), bias=b.to(DEV))
            torch.testing.assert_close(got.sum(0).cpu().double(), want, atol=2e-4, rtol=2e-4)
    if rows <= 16:
        out.zero_()
        kernels.gemm_fused_swiglu(x.to(DEV), weight, out, splits=2, **options)
        close(out, plain.gelu_tanh(x.double() @ gate.double().T + gb.double()) * (x.double() @ up.double().T + ub.double()), "bf16", "gate, fused")
        stream = torch.randn(rows, out_width)
        got = stream.to(DEV)
        kernels.gemm_fused_residual(x.to(DEV), w.to(DEV), got, splits=2, bias=b.to(DEV))
        torch.testing.assert_close(got.cpu().double(), stream.double() + want, atol=2e-4, rtol=2e-4)
        plainly = torch.empty(rows, out_width, device=DEV)
        kernels.gemm_fused_store(x.to(DEV), w.to(DEV), plainly, splits=3, bias=b.to(DEV))
        torch.testing.assert_close(plainly.cpu().double(), want, atol=2e-4, rtol=2e-4)
    kernels.check_status(DEV)


def latent_oracle(q, rows, rank, scale, window):
    total, heads, _ = q.shape
    out = torch.zeros(total, heads, rank, dtype=torch.float64)
    for h in range(heads):
        out[:, h] = plain.windowed_softmax(q[:, h].double() @ rows.double().T * scale, window) @ rows[:, :rank].double()
    return out


def ring_pool(rows, upto, ring_pages, order, store):
    """The pages of a ring that has taken ``rows`` up to position ``upto`` (exclusive): position p at element p % ring."""
    pool = torch.full((len(order) + 1, 1, PAGE, rows.shape[1]), 40.0, dtype=store, device=DEV)
    for p in range(upto):
        at = p % (ring_pages * PAGE)
        pool[order[at // PAGE], 0, at % PAGE] = rows[p].to(store)
    return pool


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, rank, rot, window", [(3, 40, 16, 37), (20, 64, 32, 64), (40, 72, 24, 65), (1, 11, 6, 1), (70, 16, 8, 130), (5, 264, 8, 100),
                                                      (8, 32, 8, None)])
def test_attention_over_latent_rows_under_a_window(dtype, heads, rank, rot, window):
    """300 positions, the cache plain or a ring that has wrapped: a prompt, a late portion of it, single tokens with several
    counts of key ranges.  For every query the key just outside its window scores far above everything (it must not be
    seen) and the key just inside it carries the softmax."""
    torch.manual_seed(heads + rank)
    store, total, row = STORE[dtype], 300, rank + rot
    rows = (torch.randn(total, row) * 0.3).to(store).float()
    q = (torch.randn(total, heads, row) * 0.5).to(store).float()
    if window is not None:                                     # key t - window speaks to query t alone, in directions made for it
        for t in range(max(window, 200), total, 7):
            rows[t - window + 1] = torch.nn.functional.one_hot(torch.tensor(t % row), row) * 6.0
            rows[t - window] = torch.nn.functional.one_hot(torch.tensor((t + 1) % row), row) * 6.0
            q[t] = 0.0
            q[t, :, t % row] = 4.0
            q[t, :, (t + 1) % row] += 9.0
        rows, q = rows.to(store).float(), q.to(store).float()
    want = latent_oracle(q, rows, rank, 0.5, window)
    order = [3, 1, 4, 0, 2]
    pool, table = ring_pool(rows, total, 5, order, store), as_int([order + [5]])
    impls = ["generic"] + (["latent"] if kernels.attention_latent_shape(store, row, rank, PAGE) else [])
    for impl in impls:
        for begin in (0, 190, 298):
            out = torch.full((total - begin, heads, rank), float("nan"), dtype=store, device=DEV)
            kernels.attention_prefill(q[begin:].to(DEV, store), pool, pool, out, table, as_int([0, total - begin]), as_int([begin]), total - begin, 1, PAGE, 0,
                                      window, 0.5, impl=impl, v_dim=rank)
            close(out, want[begin:], dtype, f"{impl}: portion from {begin}")
        for t in (0, 63, 64, 127, 128, 207, 256, 291, 299):
            for splits in (1, 4, 12):
                out = torch.full((1, heads, rank), float("nan"), dtype=store, device=DEV)
                kernels.attention_decode(q[t:t + 1].to(DEV, store), pool, pool, out, table, as_int([t + 1]), 1, PAGE, 0, window, 0.5, splits,
                                         torch.empty(12 * heads * rank, device=DEV), torch.empty(24 * heads, device=DEV), impl=impl, v_dim=rank)
                close(out, want[t:t + 1], dtype, f"{impl}: token {t}, {splits} ranges")
        if window is not None and window <= 65:                # a ring of 192 positions: a portion of 100 behind 200, then single tokens
            ring = ring_pool(rows, total, 3, order, store)
            out = torch.full((100, heads, rank), float("nan"), dtype=store, device=DEV)
            kernels.attention_prefill(q[200:].to(DEV, store), ring, ring, out, table, as_int([0, 100]), as_int([200]), 100, 1, PAGE, 3 * PAGE, window, 0.5,
                                      impl=impl, v_dim=rank)
            close(out, want[200:], dtype, f"{impl}: a portion in a ring")
            for splits in (1, 4):
                out = torch.full((1, heads, rank), float("nan"), dtype=store, device=DEV)
                kernels.attention_decode(q[-1:].to(DEV, store), ring, ring, out, table, as_int([total]), 1, PAGE, 3 * PAGE, window, 0.5, splits,
                                         torch.empty(12 * heads * rank, device=DEV), torch.empty(24 * heads, device=DEV), impl=impl, v_dim=rank)
                close(out, want[-1:], dtype, f"{impl}: one token in a ring, {splits} ranges")
    kernels.check_status(DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, n, k", [(3, 40, 24), (5, 17, 9), (2, 128, 64)])
def test_one_gate_per_head_on_a_product_per_head(dtype, heads, n, k):
    torch.manual_seed(n)
    store, tokens = STORE[dtype], 77
    x = torch.randn(tokens, heads, k).to(store)
    w = (torch.randn(heads, n, k) * 0.3).to(store)
    gate = torch.randn(2, tokens, heads + 5) * 2.0
    out = torch.empty(tokens, heads, n, dtype=store, device=DEV)
    kernels.head_product(x.to(DEV), w.to(DEV), out, x_row=heads * k, x_head=k, gate=GemmOut(gate.to(DEV)), gate_offset=3, gate_per_head=True)
    want = torch.einsum("thk,hnk->thn", x.double(), w.double()) * torch.sigmoid(gate.double().sum(0)[:, 3:3 + heads])[:, :, None]
    close(out, want, dtype, "gate per head")


@pytest.mark.parametrize("tokens, rank, n, tau", [(5, 16, 70, 16.0), (300, 7, 200, 1.0), (40, 1, 3, 0.5)])
def test_the_logarithm_of_a_decay_that_is_a_power_of_a_sigmoid(tokens, rank, n, tau):
    torch.manual_seed(n)
    rows = torch.randn(2, tokens, rank + 6) * 3.0
    w, b = torch.randn(n, rank), torch.randn(n) * 8.0
    out = torch.empty(tokens, n, device=DEV)
    kernels.lowrank(GemmOut(rows.to(DEV)), 4, w.t().contiguous().to(DEV), out, b.to(DEV), power=1.0 / tau)
    z = rows.double().sum(0)[:, 4:4 + rank] @ w.double().T + b.double()
    want = torch.sigmoid(z).pow(1.0 / tau)
    torch.testing.assert_close(torch.exp(out.cpu().double()), want, atol=1e-5, rtol=1e-4)
    torch.testing.assert_close(out.cpu().double(), -plain.softplus(-z) / tau, atol=1e-4, rtol=1e-4)


def run_recurrence(rows, at, log_decay, v_scale, out_scale, group, states, slots, lengths, portions, dim, vdim, impl):
    """Sequences of ``lengths`` tokens, their rows one after the other in ``rows`` (a list), run in portions; returns o per sequence."""
    heads = states.shape[1]
    scratch = {name: torch.full((numel,), float("nan"), device=DEV)
               for name, numel in kernels.decay_scratch(1024, heads, dim, vdim, log_decay[0].dim() == 3).items()}
    got, done = [[] for _ in lengths], [0] * len(lengths)
    while any(d < n for d, n in zip(done, lengths)):
        count = [min(portions[s], n - done[s]) for s, n in enumerate(lengths)]
        live = [s for s, c in enumerate(count) if c > 0]
        step = _Step([count[s] for s in live], [done[s] for s in live], [slots[s] for s in live])
        piece = torch.cat([rows[s][done[s]:done[s] + count[s]] for s in live]).to(DEV).contiguous()
        decay = torch.cat([log_decay[s][done[s]:done[s] + count[s]] for s in live]).to(DEV).contiguous()
        scale = torch.cat([v_scale[s][done[s]:done[s] + count[s]] for s in live]).to(DEV).contiguous() if v_scale else None
        out = torch.full((piece.shape[0], heads, vdim), float("nan"), device=DEV)
        kernels.decayed_attention(GemmOut(piece[None]), *at, decay, states, out, step, dim, scratch, heads_per_key=group, v_scale=scale, out_scale=out_scale,
                                  impl=impl)
        at_row = 0
        for s in live:
            got[s].append(out[at_row:at_row + count[s]].cpu())
            at_row += count[s]
            done[s] += count[s]
    return [torch.cat(g) for g in got]


@pytest.mark.parametrize("impl", ["steps", "chunks"])
@pytest.mark.parametrize("per_channel, heads, group, dim, vdim", [(True, 2, 1, 16, 24), (True, 3, 1, 72, 40), (True, 1, 1, 1, 5), (True, 2, 1, 200, 70),
                                                                  (True, 4, 2, 64, 64), (False, 4, 2, 16, 24), (False, 6, 6, 48, 48), (False, 2, 1, 130, 9),
                                                                  (False, 8, 4, 128, 64), (False, 1, 1, 256, 130)])
def test_the_recurrence_with_decays_of_the_token(impl, per_channel, heads, group, dim, vdim):
    """Three unequal sequences in portions that end inside, at and behind chunks of 64 tokens (and of one and two tokens), the
    states in rows that are not in order; decays near 1, of e^-3 and of e^-60 side by side, so that a product of decays that
    is formed by a difference of large sums, or a quotient, would show.  Rows of no sequence are left alone."""
    torch.manual_seed(dim + vdim)
    lengths, slots = (150, 1, 85), (3, 0, 1)
    keys = heads // group
    cols = 2 * keys * dim + heads * vdim + 3
    at = (2, 2 + keys * dim, 2 + 2 * keys * dim)
    rows = [torch.randn(n, cols) for n in lengths]
    shape = (heads, dim) if per_channel else (heads,)
    kinds = torch.tensor([-0.001, -0.02, -0.3, -3.0, -60.0])
    log_decay = [kinds[torch.randint(0, 5, (n, *shape)) * (torch.rand(n, *shape) < 0.4)] * torch.rand(n, *shape) for n in lengths]
    v_scale = None if per_channel else [torch.rand(n, heads) + 0.2 for n in lengths]
    out_scale = 0.37
    want = []
    for n, r, g, s in zip(lengths, rows, log_decay, v_scale or [None] * 3):
        q, k = (r[:, a:a + keys * dim].double().view(n, keys, dim)[:, torch.arange(heads) // group] for a in at[:2])
        v = r[:, at[2]:at[2] + heads * vdim].double().view(n, heads, vdim) * (s.double()[..., None] if s is not None else 1.0)
        decay = torch.exp(g.double()) if per_channel else torch.exp(g.double())[..., None].expand(n, heads, dim)
        want.append(plain.decayed_recurrence(q * out_scale, k, v, decay))
    for portions in ((1000, 1000, 1000), (64, 1, 20), (33, 1, 64), (2, 1, 3)):
        if impl == "chunks" and portions[0] == 2 and dim > 100:
            continue
        states = torch.full((6, heads, vdim, dim), 55.0, device=DEV)
        states[list(slots)] = 0.0
        got = run_recurrence(rows, at, log_decay, v_scale, out_scale, group, states, slots, lengths, portions, dim, vdim, impl)
        for s, n in enumerate(lengths):
            bound = 1e-4 * float(want[s].abs().max())
            assert float((got[s].double() - want[s]).abs().max()) < bound, f"sequence {s} in portions of {portions}"
        assert float((states[[2, 4, 5]] - 55.0).abs().max()) == 0.0


@pytest.mark.parametrize("impl", ["steps", "chunks"])
@pytest.mark.parametrize("per_channel", [True, False])
def test_a_write_to_the_state_survives_hundreds_of_tokens(impl, per_channel):
    """With decays of 1 the first token's key and value come back 600 tokens later; with 0.99 a token times 0.99^600."""
    heads, dim, vdim, tokens = 2, 16, 8, 601
    rows = torch.zeros(tokens, 2 * heads * dim + heads * vdim)
    rows[0, heads * dim:2 * heads * dim] = 1.0
    rows[0, 2 * heads * dim:] = torch.arange(1, heads * vdim + 1).float()
    rows[-1, :heads * dim] = 1.0 / dim
    decay = torch.log(torch.tensor([1.0, 0.99]))
    log_decay = decay[None, :, None].expand(tokens, heads, dim) if per_channel else decay[None].expand(tokens, heads)
    states = torch.zeros(2, heads, vdim, dim, device=DEV)
    got = run_recurrence([rows], (0, heads * dim, 2 * heads * dim), [log_decay], None, 1.0, 1, states, [1], [tokens], [170], dim, vdim, impl)[0]
    want = torch.arange(1, heads * vdim + 1).double().view(heads, vdim) * torch.tensor([1.0, 0.99], dtype=torch.float64)[:, None] ** 600
    torch.testing.assert_close(got[-1].double(), want, atol=1e-4, rtol=1e-4)
    assert float(got[1:-1].abs().max()) == 0.0


@pytest.mark.parametrize("channels, heads, taps", [(72, 6, 4), (33, 0, 1), (200, 3, 2), (130, 2, 7), (16, 1, 16), (40, 5, 3)])
def test_short_convolution_with_bias_and_silu_in_portions(channels, heads, taps):
    """Two sequences in unequal portions (shorter than the taps reach back among them, and steps of one token each), their last
    inputs kept in slots that are not in order; beside it the step sizes and the logarithms of the decays."""
    torch.manual_seed(channels + taps)
    lengths, slots, at = (60, 25), [3, 1], 5
    cols = at + channels + heads + 2
    inputs = [torch.randn(n, cols, dtype=torch.float64) for n in lengths]
    w, b = torch.randn(channels, taps) * 0.5, torch.randn(channels)
    step_b, rate = torch.randn(max(heads, 1)), torch.randn(max(heads, 1))
    want = [plain.silu(plain.causal_convolution(u[:, at:at + channels], w.double(), b.double())) for u in inputs]
    kept = torch.zeros(5, max(taps - 1, 1), channels, device=DEV)
    got, sizes, decays, done = [[], []], [[], []], [[], []], [0, 0]
    for portion in ((33, 1), (1, 2), (1, 1), (2, 20), (23, 0), (0, 1)):
        live = [s for s in (0, 1) if portion[s]]
        count = [portion[s] for s in live]
        step = _Step(count, [done[s] for s in live], [slots[s] for s in live])
        step.is_decode = all(c == 1 for c in count)
        rows = torch.cat([inputs[s][done[s]:done[s] + portion[s]] for s in live], dim=0)
        proj = GemmOut(torch.stack((rows * 0.25, rows * 0.75)).float().to(DEV).contiguous())
        out = torch.empty(rows.shape[0], channels, device=DEV)
        extra = {}
        if heads:
            extra = dict(at_step=at + channels, step_bias=step_b.to(DEV), rate_log=rate.to(DEV), step=torch.empty(rows.shape[0], heads, device=DEV),
                         log_decay=torch.empty(rows.shape[0], heads, device=DEV))
        kernels.conv_act(proj, at, w.to(DEV), b.to(DEV), kept, step, out, **extra)
        at_row = 0
        for s in live:
            got[s].append(out[at_row:at_row + portion[s]].cpu())
            if heads:
                sizes[s].append(extra["step"][at_row:at_row + portion[s]].cpu())
                decays[s].append(extra["log_decay"][at_row:at_row + portion[s]].cpu())
            at_row += portion[s]
            done[s] += portion[s]
    assert float(kept[[0, 2, 4]].abs().max()) == 0.0
    for s in (0, 1):
        torch.testing.assert_close(torch.cat(got[s]).double(), want[s], atol=1e-4, rtol=1e-4)
        if heads:
            dt = plain.softplus(inputs[s][:, at + channels:at + channels + heads] + step_b.double())
            torch.testing.assert_close(torch.cat(sizes[s]).double(), dt, atol=1e-5, rtol=1e-4)
            torch.testing.assert_close(torch.cat(decays[s]).double(), -torch.exp(rate.double()) * dt, atol=1e-5, rtol=1e-4)
        if taps > 1:
            torch.testing.assert_close(kept[slots[s]].cpu(), inputs[s][-(taps - 1):, at:at + channels].float(), atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, width, groups, shared, first, skips", [(5, 96, 4, True, False, 0), (300, 96, 1, False, True, 6), (7, 60, 5, False, True, 12),
                                                                         (2, 3000, 2, False, True, 3), (400, 2600, 1, False, False, 0), (3, 12, 12, True, False, 0),
                                                                         (33, 600, 2, True, True, 4)])
def test_skip_gate_and_norm_in_groups(dtype, tokens, width, groups, shared, first, skips):
    torch.manual_seed(width)
    o, proj = torch.randn(tokens, width) * 2.0, torch.randn(2, tokens, width + 9)
    weight = torch.randn(width // groups if shared else width) * 0.2 + 1.0
    x, skip = torch.randn(tokens, width + 4), torch.randn(max(skips, 1))
    out = torch.empty(tokens, width, dtype=STORE[dtype], device=DEV)
    kernels.group_gate_norm(o.to(DEV), weight.to(DEV), 1e-3, out, groups=groups, proj=GemmOut(proj.to(DEV)), at_gate=7, gate="silu", gate_first=first,
                            x=x.to(DEV) if skips else None, at_x=4, skip=skip.to(DEV) if skips else None)
    y = o.double()
    if skips:
        y = y + x.double()[:, 4:] * skip.double().repeat_interleave(width // skips)
    gate = plain.silu(proj.double().sum(0)[:, 7:7 + width])
    y = plain.grouped_rms(y * gate if first else y, groups, 1e-3) * (weight.double().repeat(groups) if shared else weight.double())
    close(out, y if first else y * gate, dtype, "skip, gate and norm")


@pytest.mark.parametrize("tokens, experts, top, groups, keep", [(50, 12, 3, 3, 2), (7, 64, 8, 8, 3), (100, 10, 2, 5, 1), (5, 1, 1, 1, 1), (33, 40, 5, 1, 1), (9, 6, 6, 2, 2)])
def test_softmax_router_among_the_best_groups(tokens, experts, top, groups, keep):
    """Logits spread widely; in every fourth token the runner-up of all experts sits in a group whose best is just below the
    last kept group's: it must not be chosen."""
    torch.manual_seed(experts)
    logits = torch.randn(tokens, experts) * 4.0
    if groups > keep:
        size = experts // groups
        logits[::4] = torch.arange(experts, 0, -1).float() * 0.01
        for g in range(groups):
            logits[::4, g * size] = 10.0 - g                            # groups in order, the first `keep` are kept
            if size > 1:
                logits[::4, g * size + 1] = 10.0 - g - 0.5 if g >= keep else -3.0
    parts = torch.stack((logits * 0.5, logits * 0.25, logits * 0.25))
    chosen = torch.empty(tokens, top, dtype=torch.int32, device=DEV)
    weights = torch.empty(tokens, top, device=DEV)
    kernels.route_top(GemmOut(parts.to(DEV)), chosen, weights, None, experts, 1.0, True, True, groups, keep)
    want, shares = plain.route(logits.double(), top, {"count": groups, "keep": keep} if groups > 1 else None)
    assert torch.equal(chosen.cpu().long(), want)
    torch.testing.assert_close(weights.cpu().double(), shares, atol=1e-6, rtol=1e-4)
    kernels.route_top(GemmOut(parts.to(DEV)), chosen, weights, None, experts, 2.0, False, True, groups, keep)      # the scores as they are
    torch.testing.assert_close(weights.cpu().double(), 2.0 * torch.softmax(logits.double(), -1).gather(1, want), atol=1e-6, rtol=1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [3, 90, 400])
def test_the_feed_forwards_alone(dtype, tokens):
    """The dense feed-forward with biases and the routed one with capped experts, as parts, few and many tokens."""
    from qwen_triton_b200.parts.base import Runtime, Workspace, part_class
    torch.manual_seed(tokens)
    store, width, device = STORE[dtype], 96, torch.device(DEV)
    raw = {**ODD, "width": width, "loop": None, "layers": [
        {"type": "gla", "mixer": ODD["layers"][0]["mixer"], "mlp": {"kind": "dense", "ff": 112}},
        {"type": "gla", "mixer": ODD["layers"][0]["mixer"], "mlp": {"kind": "moe", "expert": {"ff": 40, "limit": 0.8},
                                                                    "router": {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}}}]}
    for index, layer in enumerate(config_from_dict(raw).model_spec().layers):
        runtime = Runtime(device=device, dtype=store, max_step_tokens=512, max_positions=64, workspace=Workspace(device))
        cls = part_class("feed_forward", layer.feed_forward)
        part = cls(layer.feed_forward.params, "p", runtime)
        tensors = {n: (torch.randn(*s.shape) * (1.0 if n.endswith(("router", ".b")) else 0.2)).to(store)
                   for n, s in cls.expected_tensors(layer.feed_forward.params, "p").items()}
        part.load(lambda name: tensors[name])
        runtime.workspace.allocate()
        x = torch.randn(tokens, width).to(store)
        got = part.forward(x.to(DEV), None).value().cpu().double()
        t = {n: v.double() for n, v in tensors.items()}
        margins = []
        mlp = raw["layers"][index]["mlp"]
        want = plain.dense(x.double(), t, "p") if index == 0 else plain.experts(x.double(), t, "p", mlp, margins)
        if dtype == "fp32":
            torch.testing.assert_close(got, want, atol=3e-4, rtol=3e-4)
        else:
            off = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
            if margins:
                off = off[margins[0] > 0.02]
            assert float(off.mean()) < 0.02 and float(off.max()) < 0.1, f"{mlp['kind']}: mean {float(off.mean()):.4f}, worst {float(off.max()):.4f}"
    kernels.check_status(DEV)


# ============================================================================= whole models through the engine
def run_whole(engine, tokens):
    slot = engine.new_sequence()
    try:
        return engine.step([StepEntry(slot, list(tokens), list(range(len(tokens))))])
    finally:
        engine.release(slot)


@pytest.mark.parametrize("name, dtype", CASES)
def test_each_request_alone_and_whole(name, dtype):
    engine = engine_of(name, dtype, peaky=True)
    for length, seed in ((1, 0), (7, 1), (150, 2)):
        tokens = tokens_of(name, length, seed)
        close_rows(run_whole(engine, tokens), name, dtype, True, tokens, slice(None), f"{name} {length} tokens")
    engine.check_kernels()


@pytest.mark.parametrize("name, dtype", CASES)
def test_prompt_then_token_by_token_across_window_and_page_edges(name, dtype):
    """A prompt of 20 tokens, then 130 one by one: every window passes over decoded tokens, positions 63 to 65, 127 and 128 too."""
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
def test_passes_smaller_than_a_prompt_and_prompts_longer_than_a_ring(name, dtype):
    """Passes of 96 tokens cut the prompt; 300 tokens take the products' many-row forms; chunks of 64 tokens make the windowed
    layers' rings wrap inside the prompt."""
    tokens = tokens_of(name, 300, 6)
    for options in ({"max_step_tokens": 96}, {"max_step_tokens": 4096}, {"chunk_tokens": 64}):
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


@pytest.mark.parametrize("name, dtype", [("misudra-tiny-a", "fp32"), ("misudra-tiny-a", "bf16"), ("misudra-tiny-b", "bf16"), ("odd", "fp32")])
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
    """Five rows decoded for 150 steps from short prompts: every window passes over decoded tokens several times over, and the
    states carry 150 updates."""
    name = "misudra-tiny-a"
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


def test_random_weights_on_the_device_equal_the_written_folder():
    name = "misudra-tiny-b"
    folder, _, _ = model(name, "bf16")
    tokens = tokens_of(name, 50, 70)
    written = run_whole(Engine.from_pretrained(folder, dtype="bf16", max_tokens=512), tokens)
    drawn = run_whole(Engine.from_config(config_of(name), seed=17 + len(name), dtype="bf16", max_tokens=512), tokens)
    assert torch.equal(written, drawn)


def test_command_line_with_a_preset_and_random_weights():
    result = subprocess.run([sys.executable, "-m", "qwen_triton_b200.scripts.smoke", "--preset", "misudra-tiny-a", "--random-weights",
                             "--random-prompts", "9,2", "--max-new-tokens", "5", "--dtype", "bf16"], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert result.returncode == 0, result.stderr[-2000:]


@pytest.mark.parametrize("dtype, name", [("float32", "fp32"), ("bfloat16", "bf16")])
def test_trace_replay_of_a_folder(tmp_path, dtype, name):
    """bin/trace_run as a child process: two requests start together, decode together, one ends earlier; a third comes alone
    afterwards and finds their slots and state rows."""
    import numpy as np
    model_name = "misudra-tiny-b"
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
