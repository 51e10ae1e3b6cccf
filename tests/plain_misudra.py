"""A plain, slow statement of the Misudra design, one function per mechanism, in float64 on the CPU.

It shares no code with the package: tensors come in as a dict name -> tensor, the configuration as the dict that
config.json holds.  Every sequence is run by itself, token after token where a mechanism is recurrent.

The design: x = RMS(embed[token]) w; layers x += mixer(norm1(x)), x += ff(norm2(x)) with RMS norms; a range of layers runs
several times with the same weights, each pass starting from x <- W_in [x; x0] with x0 the normed embedding; the logits are
head RMS(x).  Mixers: attention through a latent (a rotated key part shared by the heads, a sliding window, one sigmoid
gate per head); linear attention with a decay per key channel and token (``gla``); a state-space recurrence with a decay
per head and token behind a short convolution (``mamba2``).  Feed-forward: dense, tanh-GELU gate with biases, or experts
with a capped gate chosen by a softmax router among the best groups.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rotate(x, positions, dims, base):
    """x [T, heads, n]: element i < dims/2 turns together with element i + dims/2 by position * base^(-2i/dims)."""
    half = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    angle = positions.to(F)[:, None] * freq[None, :]
    cos, sin = angle.cos()[:, None, :], angle.sin()[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, x[..., dims:]), dim=-1)


# ----------------------------------------------------------------------------- attention through a latent
def windowed_softmax(score, window):
    """score [T, T] of one head; query i sees key j with 0 <= i - j < window (None: every j <= i)."""
    tokens = score.shape[0]
    gap = torch.arange(tokens)[:, None] - torch.arange(tokens)[None, :]
    seen = gap >= 0
    if window is not None:
        seen = seen & (gap < window)
    score = score.masked_fill(~seen, -math.inf)
    weight = torch.exp(score - score.max(-1, keepdim=True).values)
    return weight / weight.sum(-1, keepdim=True)


def latent_attention(h, t, prefix, m, eps):
    tokens = h.shape[0]
    heads, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(tokens)
    cq = rms_norm(h @ t[prefix + ".dq"].T, eps, t[prefix + ".dq.norm"])
    q = (cq @ t[prefix + ".uq"].T).view(tokens, heads, dim + rot)
    down = h @ t[prefix + ".dkv"].T
    c = rms_norm(down[:, :rank], eps, t[prefix + ".dkv.norm"])
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    k_rot = rotate(down[:, None, rank:], positions, dims, base)[:, 0]
    q_rot = rotate(q[..., dim:], positions, dims, base)
    k = (c @ t[prefix + ".uk"].T).view(tokens, heads, dim)
    v = (c @ t[prefix + ".uv"].T).view(tokens, heads, vdim)
    window = (m.get("mask") or {}).get("size")
    gate = torch.sigmoid(h @ t[prefix + ".g"].T)                     # [T, heads]
    out = torch.zeros(tokens, heads, vdim, dtype=F)
    for n in range(heads):
        score = (q[:, n, :dim] @ k[:, n].T + q_rot[:, n] @ k_rot.T) * float(m["scale"])
        out[:, n] = windowed_softmax(score, window) @ v[:, n] * gate[:, n:n + 1]
    return out.reshape(tokens, heads * vdim) @ t[prefix + ".o"].T


# ----------------------------------------------------------------------------- the two recurrences
def decayed_recurrence(q, k, v, decay):
    """S <- diag(decay_t) S + k_t v_t^T; o_t = S^T q_t, from a zero state.  q, k, decay [T, H, n], v [T, H, m]."""
    tokens, heads, n = q.shape
    state = torch.zeros(heads, n, v.shape[-1], dtype=F)
    out = []
    for i in range(tokens):
        state = decay[i][:, :, None] * state + k[i][:, :, None] * v[i][:, None, :]
        out.append((state * q[i][:, :, None]).sum(1))
    return torch.stack(out)


def gla(h, t, prefix, m, eps):
    tokens = h.shape[0]
    heads, dim, vdim, tau = m["heads"], m["dim"], m["vdim"], float(m["tau"])
    q = (h @ t[prefix + ".q"].T).view(tokens, heads, dim) * dim ** -0.5
    k = (h @ t[prefix + ".k"].T).view(tokens, heads, dim)
    v = (h @ t[prefix + ".v"].T).view(tokens, heads, vdim)
    z = (h @ t[prefix + ".a1"].T) @ t[prefix + ".a2"].T + t[prefix + ".a2.b"]
    decay = torch.sigmoid(z).pow(1.0 / tau).view(tokens, heads, dim)
    o = rms_norm(decayed_recurrence(q, k, v, decay), eps, t[prefix + ".norm"])
    return (o.reshape(tokens, heads * vdim) * silu(h @ t[prefix + ".g"].T)) @ t[prefix + ".o"].T


def causal_convolution(x, taps, bias):
    """x [T, C], taps [C, K] (last column: the current token), zeros before the start."""
    count = taps.shape[1]
    padded = torch.cat((torch.zeros(count - 1, x.shape[1], dtype=F), x))
    return sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(count)) + bias


def grouped_rms(x, groups, eps):
    tokens, width = x.shape
    return rms_norm(x.view(tokens, groups, width // groups), eps).reshape(tokens, width)


def mamba2(h, t, prefix, m, eps):
    tokens = h.shape[0]
    heads, vdim, n, groups = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * vdim
    u = h @ t[prefix + ".in"].T
    z, mixed, dt = u[:, :inner], u[:, inner:2 * inner + 2 * groups * n], u[:, 2 * inner + 2 * groups * n:]
    mixed = silu(causal_convolution(mixed, t[prefix + ".conv"], t[prefix + ".conv.b"]))
    x = mixed[:, :inner].view(tokens, heads, vdim)
    b = mixed[:, inner:inner + groups * n].view(tokens, groups, n)
    c = mixed[:, inner + groups * n:].view(tokens, groups, n)
    of = torch.arange(heads) // (heads // groups)
    dt = softplus(dt + t[prefix + ".dt_bias"])                        # [T, heads]
    decay = torch.exp(-torch.exp(t[prefix + ".A_log"]) * dt)
    y = decayed_recurrence(c[:, of], b[:, of], x * dt[..., None], decay[..., None].expand(tokens, heads, n))
    y = (y + t[prefix + ".D"][None, :, None] * x).reshape(tokens, inner)
    return (grouped_rms(y * silu(z), m["norm_groups"], eps) * t[prefix + ".norm"]) @ t[prefix + ".o"].T


# ----------------------------------------------------------------------------- feed-forward
def dense(h, t, prefix):
    gate = h @ t[prefix + ".gate"].T + t[prefix + ".gate.b"]
    up = h @ t[prefix + ".up"].T + t[prefix + ".up.b"]
    return (gelu_tanh(gate) * up) @ t[prefix + ".down"].T + t[prefix + ".down.b"]


def capped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(logits, top, groups=None):
    """logits [T, E] -> (chosen [T, top], weights [T, top]): softmax scores, only the experts of the ``keep`` groups (of
    ``count`` equal runs of neighbours) with the largest best score, weights over their sum."""
    scores = torch.softmax(logits, dim=-1)
    allowed = torch.ones_like(scores, dtype=torch.bool)
    if groups is not None:
        tokens, experts = scores.shape
        best = scores.view(tokens, groups["count"], -1).max(-1).values
        kept = best.topk(groups["keep"], dim=-1).indices
        allowed = torch.zeros(tokens, groups["count"], dtype=torch.bool).scatter_(1, kept, True)
        allowed = allowed.repeat_interleave(experts // groups["count"], dim=1)
    chosen = scores.masked_fill(~allowed, -1.0).topk(top, dim=-1).indices
    picked = scores.gather(1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def choice_margin(logits, top, groups=None):
    """How far, in logits, the router of each token is from choosing otherwise: the gap between the last chosen and the
    first passed-over expert among the kept groups, and between the last kept and the first dropped group."""
    tokens, experts = logits.shape
    allowed = logits
    margin = torch.full((tokens,), math.inf, dtype=F)
    if groups is not None and groups["keep"] < groups["count"]:
        best = logits.view(tokens, groups["count"], -1).max(-1).values.sort(-1, descending=True)
        margin = best.values[:, groups["keep"] - 1] - best.values[:, groups["keep"]]
        mask = torch.zeros(tokens, groups["count"], dtype=torch.bool).scatter_(1, best.indices[:, :groups["keep"]], True)
        allowed = logits.masked_fill(~mask.repeat_interleave(experts // groups["count"], dim=1), -math.inf)
    ranked = allowed.sort(-1, descending=True).values
    if top < experts:
        margin = torch.minimum(margin, ranked[:, top - 1] - ranked[:, top])
    return margin


def experts(h, t, prefix, m, margins=None):
    router, limit = m["router"], float(m["expert"]["limit"])
    logits = h @ t[prefix + ".router"].T
    chosen, weights = route(logits, router["top"], router.get("groups"))
    if margins is not None:
        margins.append(choice_margin(logits, router["top"], router.get("groups")) / logits.std(unbiased=False).clamp(min=1e-9))
    out = torch.zeros_like(h)
    for e in range(router["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            y = capped_expert(h[rows], t[f"{prefix}.e{e}.gate"], t[f"{prefix}.e{e}.up"], t[f"{prefix}.e{e}.down"], limit)
            out.index_add_(0, rows, y * weights[rows, place][:, None])
    return out


# ----------------------------------------------------------------------------- the model
MIXERS = {"latent_attention": latent_attention, "gla": gla, "mamba2": mamba2}


def schedule(config):
    """(layer, starts a pass) in the order in which the layers run."""
    loop, count = config.get("loop"), len(config["layers"])
    if not loop:
        return [(i, False) for i in range(count)]
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], count)]


def forward(config, weights, tokens, streams=None, margins=None):
    """Logits [T, vocab] of one sequence; ``streams`` collects the stream behind every layer run, ``margins`` the routers'
    distances from another choice."""
    t = {name: tensor.to(F) for name, tensor in weights.items()}
    eps = float(config["norm"]["eps"])
    start = rms_norm(t["embed"][torch.tensor(tokens)], eps, t["embed.norm"])
    x = start
    for index, begins in schedule(config):
        layer, prefix = config["layers"][index], f"l{index}"
        if begins:
            x = torch.cat((x, start), dim=-1) @ t["loop.in"].T
        x = x + MIXERS[layer["type"]](rms_norm(x, eps, t[prefix + ".norm1"]), t, prefix + ".mix", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h = rms_norm(x, eps, t[prefix + ".norm2"])
            x = x + (dense(h, t, prefix + ".mlp") if layer["mlp"]["kind"] == "dense" else experts(h, t, prefix + ".mlp", layer["mlp"], margins))
        if streams is not None:
            streams.append(x)
    return rms_norm(x, eps, t["final.norm"]) @ t["head"].T
