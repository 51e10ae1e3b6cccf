"""A plain, slow statement of the Bizurax design, one function per mechanism, in float64 on the CPU.

It shares no code with the package: tensors come in as a dict name -> tensor, the configuration as the dict that
config.json holds.  Every sequence is run by itself, token after token where a mechanism is recurrent.

The design: the stream is S parallel copies of the embedding's row; a sublayer reads a weighted sum of them, and its result
(times a constant and a weight per stream) is added to a linear mix of them; the head reads the normed sum of all.  Mixers:
softmax attention with biased projections, unit-norm rotated queries and keys, capped scores and a learned sink; attention
through a latent with interleaved rotation pairs; linear attention with a fixed decay per head ("retention").  Feed-forward:
two matrices with the squared ReLU, or SiLU-gated experts chosen by a biased router beside a shared one.  A range of layers
may run several times with the same weights.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(x):
    return x * torch.sigmoid(x)


def rotate(x, positions, dims, base, factor=1.0, interleaved=False):
    """x [T, heads, n], its first ``dims`` elements in pairs (i, i + dims/2), or (2i, 2i + 1), each turned by
    position * base^(-2i/dims) / factor."""
    half = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) / factor for i in range(half)], dtype=F)
    angle = positions.to(F)[:, None] * freq[None, :]
    cos, sin = angle.cos()[:, None, :], angle.sin()[:, None, :]
    out = x.clone()
    first = slice(0, dims, 2) if interleaved else slice(0, half)
    second = slice(1, dims, 2) if interleaved else slice(half, dims)
    u, v = x[..., first], x[..., second]
    out[..., first] = u * cos - v * sin
    out[..., second] = v * cos + u * sin
    return out


def cap(score, softcap):
    return score if softcap is None else softcap * torch.tanh(score / softcap)


def causal_softmax(score, sink=None):
    """score [T, T] of one head over the keys up to each query; ``sink``: one more term of the denominator."""
    tokens = score.shape[0]
    gap = torch.arange(tokens)[:, None] - torch.arange(tokens)[None, :]
    score = score.masked_fill(gap < 0, -math.inf)
    top = score.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    weight = torch.exp(score - top)
    total = weight.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return weight / total


def rotation(m):
    rot = m.get("rot") or {}
    return int(rot.get("dims") or 0), float(rot.get("base", 1.0)), float((rot.get("scaling") or {}).get("factor", 1.0))


# ----------------------------------------------------------------------------- mixers
def attention(h, t, prefix, m, eps):
    tokens = h.shape[0]
    heads, groups, dim = m["heads"], m["kv_heads"], m["dim"]
    vdim = m.get("vdim") or dim
    q = (h @ t[prefix + ".q"].T + t[prefix + ".q.b"]).view(tokens, heads, dim)
    k = (h @ t[prefix + ".k"].T + t[prefix + ".k.b"]).view(tokens, groups, dim)
    v = (h @ t[prefix + ".v"].T + t[prefix + ".v.b"]).view(tokens, groups, vdim)
    dims, base, factor = rotation(m)
    if dims:
        q, k = (rotate(x, torch.arange(tokens), dims, base, factor) for x in (q, k))
    q, k = rms_norm(q, eps), rms_norm(k, eps)
    out = torch.zeros(tokens, heads, vdim, dtype=F)
    for n in range(heads):
        g = n // (heads // groups)
        score = cap(q[:, n] @ k[:, g].T * float(m["scale"]), m.get("softcap"))
        out[:, n] = causal_softmax(score, t[prefix + ".sink"][n]) @ v[:, g]
    return out.reshape(tokens, heads * vdim) @ t[prefix + ".o"].T


def latent_attention(h, t, prefix, m, eps):
    tokens = h.shape[0]
    heads, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m.get("vdim") or m["dim"], m["kv_rank"]
    q = (h @ t[prefix + ".q"].T).view(tokens, heads, dim + rot)
    down = h @ t[prefix + ".dkv"].T
    c = rms_norm(down[:, :rank], eps, t[prefix + ".dkv.norm"])
    dims, base, factor = rotation(m)
    q_rot, k_rot = q[..., dim:], down[:, None, rank:]
    if dims:
        q_rot, k_rot = (rotate(x, torch.arange(tokens), dims, base, factor, interleaved=True) for x in (q_rot, k_rot))
    k = (c @ t[prefix + ".uk"].T).view(tokens, heads, dim)
    v = (c @ t[prefix + ".uv"].T).view(tokens, heads, vdim)
    out = torch.zeros(tokens, heads, vdim, dtype=F)
    for n in range(heads):
        score = (q[:, n, :dim] @ k[:, n].T + q_rot[:, n] @ k_rot[:, 0].T) * float(m["scale"])
        out[:, n] = causal_softmax(score) @ v[:, n]
    return out.reshape(tokens, heads * vdim) @ t[prefix + ".o"].T


def fixed_decay_recurrence(q, k, v, decay):
    """S <- decay_h S + k_t v_t^T; o_t = S^T q_t, from a zero state.  q, k [T, H, n], v [T, H, m], decay [H]."""
    tokens, heads, n = q.shape
    state = torch.zeros(heads, n, v.shape[-1], dtype=F)
    out = []
    for i in range(tokens):
        state = decay[:, None, None] * state + k[i][:, :, None] * v[i][:, None, :]
        out.append((state * q[i][:, :, None]).sum(1))
    return torch.stack(out)


def retention(h, t, prefix, m, eps):
    tokens = h.shape[0]
    heads, dim = m["heads"], m["dim"]
    vdim = m.get("vdim") or dim
    q = (h @ t[prefix + ".q"].T).view(tokens, heads, dim)
    k = (h @ t[prefix + ".k"].T).view(tokens, heads, dim)
    v = (h @ t[prefix + ".v"].T).view(tokens, heads, vdim)
    dims, base, factor = rotation(m)
    if dims:
        q, k = (rotate(x, torch.arange(tokens), dims, base, factor) for x in (q, k))
    o = fixed_decay_recurrence(q, k * dim ** -0.5, v, torch.tensor(m["decay"], dtype=F))
    o = rms_norm(o, eps).reshape(tokens, heads * vdim)
    return (o * silu(h @ t[prefix + ".g"].T)) @ t[prefix + ".o"].T


# ----------------------------------------------------------------------------- feed-forward
def dense(h, t, prefix):
    return torch.relu(h @ t[prefix + ".up"].T).square() @ t[prefix + ".down"].T


def gated_expert(h, t, prefix):
    return (silu(h @ t[prefix + ".gate"].T) * (h @ t[prefix + ".up"].T)) @ t[prefix + ".down"].T


def route(logits, top):
    """logits [T, E] -> (chosen [T, top], weights [T, top]): the largest logits, weighted by a softmax over them alone."""
    values, chosen = logits.topk(top, dim=-1)
    return chosen, torch.softmax(values, dim=-1)


def choice_margin(logits, top):
    """How far, in logits, each token's router is from choosing otherwise."""
    if top >= logits.shape[-1]:
        return torch.full((logits.shape[0],), math.inf, dtype=F)
    ranked = logits.sort(-1, descending=True).values
    return ranked[:, top - 1] - ranked[:, top]


def experts(h, t, prefix, m, margins=None):
    router = m["router"]
    logits = h @ t[prefix + ".router"].T + t[prefix + ".router.b"]
    chosen, weights = route(logits, router["top"])
    if margins is not None:
        margins.append(choice_margin(logits, router["top"]) / logits.std(unbiased=False).clamp(min=1e-9))
    out = torch.zeros_like(h)
    for e in range(router["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out.index_add_(0, rows, gated_expert(h[rows], t, f"{prefix}.e{e}") * weights[rows, place][:, None])
    if m.get("shared") is not None:
        out = out + gated_expert(h, t, prefix + ".shared")
    return out


# ----------------------------------------------------------------------------- the streams
def read_streams(x, t, prefix):
    """x [S, T, W] -> [T, W], what a sublayer sees of the streams."""
    return torch.einsum("s,stw->tw", t[prefix + ".in"], x)


def write_streams(x, y, t, prefix, mult):
    """The streams after a sublayer returned y: the mix [from, to] of the old ones plus a share of y for each."""
    return torch.einsum("su,stw->utw", t[prefix + ".mix"], x) + mult * t[prefix + ".out"][:, None, None] * y[None]


# ----------------------------------------------------------------------------- the model
MIXERS = {"attention": attention, "latent_attention": latent_attention, "retention": retention}


def schedule(config):
    """Layer numbers in the order in which they run."""
    loop, count = config.get("loop"), len(config["layers"])
    if not loop:
        return list(range(count))
    return (list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], count)))


def forward(config, weights, tokens, streams=None, margins=None):
    """Logits [T, vocab] of one sequence; ``streams`` collects the sum of the streams behind every layer run, ``margins`` the
    routers' distances from another choice."""
    t = {name: tensor.to(F) for name, tensor in weights.items()}
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    x = t["embed"][torch.tensor(tokens)].expand(config["streams"], -1, -1)
    for index in schedule(config):
        layer, prefix = config["layers"][index], f"l{index}"
        h = rms_norm(read_streams(x, t, prefix + ".hc1"), eps, t[prefix + ".norm1"])
        x = write_streams(x, MIXERS[layer["type"]](h, t, prefix + ".mix", layer["mixer"], eps), t, prefix + ".hc1", mult)
        if layer.get("mlp") is not None:
            h = rms_norm(read_streams(x, t, prefix + ".hc2"), eps, t[prefix + ".norm2"])
            y = dense(h, t, prefix + ".mlp") if layer["mlp"]["kind"] == "dense" else experts(h, t, prefix + ".mlp", layer["mlp"], margins)
            x = write_streams(x, y, t, prefix + ".hc2", mult)
        if streams is not None:
            streams.append(x.sum(0))
    return rms_norm(x.sum(0), eps, t["final.norm"]) @ t["head"].T
