"""A recurrent mixer: the gated delta rule with one decay per head and key channel.

Per head a float state S [dim, vdim] is carried from token to token of a sequence:

    S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t

where o_t is read after token t has been written.  Around it:

* q = W_q h and k = W_k h ([kv_heads, dim]; head h reads kv head h // (heads / kv_heads)), v = W_v h ([heads, vdim]);
  each passes a short causal convolution per channel (``conv`` taps, the last one the current token's, zeros before
  the sequence's start) and SiLU; q and k are then made unit vectors per head, x / sqrt(sum x^2 + 1e-6), q also
  times dim^-1/2;
* beta = sigmoid(W_b h), one per head;
* g = exp(-exp(A_log_h) softplus(W_a2 (W_a1 h) + dt_bias)), [heads, dim]: a projection through few columns (the
  kernels pass its logarithm on);
* every head's o is divided by its root mean square over vdim (``eps`` inside the root), times a weight [vdim] shared
  by the heads, times sigmoid(W_g2 (W_g1 h)) ([heads, vdim]); then W_o.

Per sequence the mixer keeps two things, both float, both in the cache's per-slot state (zero for a new sequence):
the states S [heads, dim, vdim] and the last ``conv`` - 1 inputs of the convolutions.  The six projections of h run as
one product with float sums; everything between it and the output projection is float (``csrc/delta_rule.cu``).

Parameters: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``v_head_dim``, ``conv``, ``eps``,
``decay_rank`` and ``gate_rank`` (columns of the two narrow projections; read from the tensors' shapes by the
configuration), ``float_out``, ``init_std``, and the tensor names (``q``, ``k``, ``v``, ``beta``, ``decay_in``,
``decay_out``, ``decay_bias``, ``decay_rate``, ``gate_in``, ``gate_out``, ``norm``, ``o``, ``conv_suffix``,
``weight_suffix``).
"""
from __future__ import annotations

import torch

from ..ops import kernels
from ..ops.kernels import GemmOut
from ..weights.tensors import TensorSpec
from .base import DeferredProduct, Runtime, StateRequest, part_class, register_mixer, to_device
from .linear import Linear

_UNIT_EPS = 1e-6      # inside the root of the unit norms of q and k
_FEW_TOKENS = 4       # steps in which no sequence brings more tokens run the recurrence token by token


@register_mixer("gated_delta_rule")
class GatedDeltaRule:
    graph_safe = True

    def __init__(self, params, prefix: str, runtime: Runtime) -> None:
        self.prefix = prefix
        self.runtime = runtime
        self.params = dict(params)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["num_heads"])
        self.kv_heads = int(params.get("num_kv_heads") or self.heads)
        self.dim = int(params["head_dim"])
        self.vdim = int(params.get("v_head_dim") or self.dim)
        self.taps = int(params.get("conv", 1))
        self.eps = float(params.get("eps", 1e-6))
        self.decay_rank = int(params["decay_rank"])
        self.gate_rank = int(params["gate_rank"])
        if self.heads % self.kv_heads:
            raise ValueError(f"{prefix}: {self.heads} heads are not a multiple of {self.kv_heads} kv heads")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"{prefix}: a convolution of {self.taps} taps (1..16)")
        if self.dim > 512:
            raise ValueError(f"{prefix}: {self.dim} key channels per head are beyond what the recurrence kernel holds (512)")
        self.channels = 2 * self.kv_heads * self.dim + self.heads * self.vdim
        # columns of the first product: q | k | v | beta | decay_in | gate_in, padded to a multiple of 8
        self.at_decay = self.channels + self.heads
        self.at_gate = self.at_decay + self.decay_rank
        used = self.at_gate + self.gate_rank
        self.proj_rows = -(-used // 8) * 8
        self.proj = Linear("delta.proj", self.proj_rows, self.hidden, runtime, float_out=True)
        float_out = bool(params.get("float_out", False))
        self.o = Linear("delta.o" + (".float" if float_out else ""), self.hidden, self.heads * self.vdim, runtime, float_out=float_out, role="attn_out")
        ws = runtime.workspace
        tokens = runtime.max_step_tokens
        for name, width in (("delta.q", self.kv_heads * self.dim), ("delta.k", self.kv_heads * self.dim), ("delta.v", self.heads * self.vdim),
                            ("delta.beta", self.heads), ("delta.decay", self.heads * self.dim), ("delta.gate", self.heads * self.vdim),
                            ("delta.read", self.heads * self.vdim)):
            ws.declare(name, tokens * width, torch.float32)
        ws.declare("delta.normed", tokens * self.heads * self.vdim, runtime.dtype)
        ws.declare("delta.chunks", tokens * self.heads * (4 * self.dim + 2 * kernels.DELTA_CHUNK + 4), torch.float32)
        self.conv = self.decay_out = self.decay_bias = self.decay_rate = self.gate_out = self.norm = None

    # ------------------------------------------------------------------ weights
    @staticmethod
    def _names(params, prefix: str) -> dict[str, str]:
        w = str(params.get("weight_suffix", ".weight"))
        conv = str(params.get("conv_suffix", ".conv"))
        defaults = {"q": "q", "k": "k", "v": "v", "beta": "beta", "decay_in": "decay_in", "decay_out": "decay_out", "gate_in": "gate_in",
                    "gate_out": "gate_out", "o": "o"}
        n = {key: f"{prefix}.{params.get(key, default)}{w}" for key, default in defaults.items()}
        for key in ("q", "k", "v"):
            n[key + "_conv"] = f"{prefix}.{params.get(key, key)}{conv}"
        for key, default in (("decay_bias", "decay_bias"), ("decay_rate", "decay_rate"), ("norm", "norm")):
            n[key] = f"{prefix}.{params.get(key, default)}"
        return n

    @classmethod
    def expected_tensors(cls, params, prefix: str) -> dict[str, TensorSpec]:
        hidden, heads, dim = int(params["hidden_size"]), int(params["num_heads"]), int(params["head_dim"])
        kv_heads, vdim, taps = int(params.get("num_kv_heads") or heads), int(params.get("v_head_dim") or dim), int(params.get("conv", 1))
        ra, rg = int(params["decay_rank"]), int(params["gate_rank"])
        n = cls._names(params, prefix)
        std = float(params.get("init_std", 0.02))
        narrow = float(params.get("narrow_init_std", 0.2))
        out = {n["q"]: TensorSpec((kv_heads * dim, hidden), init_std=std), n["k"]: TensorSpec((kv_heads * dim, hidden), init_std=std),
               n["v"]: TensorSpec((heads * vdim, hidden), init_std=std), n["beta"]: TensorSpec((heads, hidden), init_std=std),
               n["decay_in"]: TensorSpec((ra, hidden), init_std=std), n["decay_out"]: TensorSpec((heads * dim, ra), init_std=narrow),
               n["gate_in"]: TensorSpec((rg, hidden), init_std=std), n["gate_out"]: TensorSpec((heads * vdim, rg), init_std=narrow),
               n["o"]: TensorSpec((hidden, heads * vdim), init_std=std),
               n["decay_bias"]: TensorSpec((heads * dim,), role="vector", init_std=0.5, init_mean=-3.0),
               n["decay_rate"]: TensorSpec((heads,), role="vector", init_std=0.3, init_mean=0.0),
               n["norm"]: TensorSpec((vdim,), role="vector", init_std=0.1, init_mean=1.0)}
        # a convolution of one tap is a factor per channel; a model may leave such tensors out (all ones)
        for key, channels in (("q_conv", kv_heads * dim), ("k_conv", kv_heads * dim), ("v_conv", heads * vdim)):
            out[n[key]] = TensorSpec((channels, taps), role="vector", init_std=0.3, init_mean=0.3, optional=taps == 1)
        return out

    def load(self, source) -> None:
        n = self._names(self.params, self.prefix)
        dtype, device = self.runtime.dtype, self.runtime.device
        rows = [source(n[key]).to(dtype) for key in ("q", "k", "v", "beta", "decay_in", "gate_in")]
        used = sum(r.shape[0] for r in rows)
        if self.proj_rows > used:
            rows.append(torch.zeros(self.proj_rows - used, self.hidden, dtype=dtype, device=rows[0].device))
        self.proj.set_weight(torch.cat(rows, dim=0))
        self.o.set_weight(source(n["o"]))
        pieces = []
        for key, channels in (("q", self.kv_heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.heads * self.vdim)):
            stored = source(n[key + "_conv"])
            pieces.append(stored.float().cpu() if stored is not None else torch.ones(channels, self.taps))
        conv = torch.cat(pieces, dim=0)
        self.conv = to_device(conv, torch.float32, device)
        # the narrow projections' second matrices: float, transposed to [rank, N] so that neighbouring threads read neighbouring outputs
        self.decay_out = to_device(source(n["decay_out"]).float().t(), torch.float32, device)
        self.gate_out = to_device(source(n["gate_out"]).float().t(), torch.float32, device)
        self.decay_bias = to_device(source(n["decay_bias"]), torch.float32, device)
        self.decay_rate = to_device(source(n["decay_rate"]), torch.float32, device)
        self.norm = to_device(source(n["norm"]), torch.float32, device)

    # ------------------------------------------------------------------ what it keeps per sequence
    def cache_request(self):
        return [StateRequest((self.heads, self.dim, self.vdim), torch.float32),
                StateRequest((max(self.taps - 1, 1), self.channels), torch.float32)]

    # ------------------------------------------------------------------ run
    def forward(self, x, ctx, cache):
        states, kept = cache
        if not states.writable:
            raise ValueError(f"{self.prefix}: a recurrent mixer cannot read another layer's state")
        tokens = x.shape[0]
        ws = self.runtime.workspace
        proj = self.proj(x)
        q = ws.view("delta.q", tokens, self.kv_heads, self.dim)
        k = ws.view("delta.k", tokens, self.kv_heads, self.dim)
        v = ws.view("delta.v", tokens, self.heads, self.vdim)
        beta = ws.view("delta.beta", tokens, self.heads)
        decay = ws.view("delta.decay", tokens, self.heads, self.dim)
        gate = ws.view("delta.gate", tokens, self.heads, self.vdim)
        read = ws.view("delta.read", tokens, self.heads, self.vdim)
        kept_rows = kept.state if self.taps > 1 else kept.state[:, :0]
        kernels.delta_prepare(proj, self.conv, kept_rows, ctx, q, k, v, beta, self.heads, self.kv_heads, self.dim, self.vdim, _UNIT_EPS)
        kernels.lowrank(proj, self.at_decay, self.decay_out, decay.view(tokens, self.heads * self.dim), self.decay_bias, self.decay_rate, self.dim)
        kernels.lowrank(proj, self.at_gate, self.gate_out, gate.view(tokens, self.heads * self.vdim))
        if ctx.max_q_len > _FEW_TOKENS and self.dim <= kernels.DELTA_CHUNKED_MAX_DIM:
            kernels.delta_scan_chunked(q, k, v, beta, decay, states.state, read,
                                       ws.view("delta.chunks", tokens * self.heads * (4 * self.dim + 2 * kernels.DELTA_CHUNK + 4)), ctx)
        else:
            kernels.delta_scan(q, k, v, beta, decay, states.state, read, ctx)
        normed = ws.view("delta.normed", tokens, self.heads, self.vdim)
        kernels.gated_head_norm(read, gate, self.norm, self.eps, normed)
        normed = normed.view(tokens, self.heads * self.vdim)
        # few tokens: the product is left to the block, which launches it with the residual addition in its epilogue
        return DeferredProduct(self.o, normed) if self.o.fusable(tokens) else self.o(normed)


@register_mixer("linear_attention")
class LinearAttention:
    """Linear attention with a constant decay per head ("lightning attention"):

        S <- decay_h S + k_t v_t^T;   o_t = S^T q_t

    with q = act(W_q h), k = act(W_k h) ([heads, dim]) and v = act(W_v h) ([heads, vdim]), act = SiLU (``activation``: "silu"
    or "none"), no other scale.  The heads' outputs of a token are RMS-normed together (one mean over all heads x vdim
    elements, ``eps`` inside the root) with a weight of that size, multiplied by sigmoid(W_g h) (``gate``) and projected by
    W_o.  Per sequence the mixer keeps the states, float, zero for a new sequence, in the cache's per-slot state rows
    (stored transposed, [heads, vdim, dim]).  The four projections of h run as one product with float sums; SiLU, the
    recurrence, the norm and the gate are float (``csrc/linear_attention.cu``).

    Parameters: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_head_dim``, ``decay`` (one number per head), ``eps``,
    ``activation``, ``gate``, ``float_out``, ``init_std``, and the tensor-name pieces ``q``, ``k``, ``v``, ``g``, ``o``, ``norm``,
    ``weight_suffix``."""

    graph_safe = True

    def __init__(self, params, prefix: str, runtime: Runtime) -> None:
        self.prefix, self.runtime, self.params = prefix, runtime, dict(params)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["num_heads"])
        self.dim = int(params["head_dim"])
        self.vdim = int(params.get("v_head_dim") or self.dim)
        self.eps = float(params.get("eps", 1e-6))
        self.gated = bool(params.get("gate", True))
        activation = params.get("activation", "silu")
        if activation not in ("silu", "none"):
            raise ValueError(f"{prefix}: activation {activation!r} on q, k and v (silu or none)")
        self.act = activation == "silu"
        decay = [float(d) for d in params["decay"]]
        if len(decay) != self.heads:
            raise ValueError(f"{prefix}: {len(decay)} decays for {self.heads} heads")
        if self.dim > kernels.LINEAR_ATTENTION_MAX_DIM:
            raise ValueError(f"{prefix}: {self.dim} key channels per head are beyond what the recurrence kernel holds "
                             f"({kernels.LINEAR_ATTENTION_MAX_DIM})")
        self.decay_values = decay
        self.decay = None
        self.at_k = self.heads * self.dim
        self.at_v = 2 * self.heads * self.dim
        self.at_gate = self.at_v + self.heads * self.vdim
        used = self.at_gate + (self.heads * self.vdim if self.gated else 0)
        self.proj_rows = -(-used // 8) * 8
        self.proj = Linear("linattn.proj", self.proj_rows, self.hidden, runtime, float_out=True)
        float_out = bool(params.get("float_out", False))
        self.o = Linear("linattn.o" + (".float" if float_out else ""), self.hidden, self.heads * self.vdim, runtime, float_out=float_out, role="attn_out")
        ws = runtime.workspace
        ws.declare("linattn.read", runtime.max_step_tokens * self.heads * self.vdim, torch.float32)
        ws.declare("linattn.qkv", runtime.max_step_tokens * self.at_gate, torch.float32)
        ws.declare("linattn.normed", runtime.max_step_tokens * self.heads * self.vdim, runtime.dtype)
        self.norm = None

    @staticmethod
    def _names(params, prefix: str) -> dict[str, str]:
        w = str(params.get("weight_suffix", ".weight"))
        n = {key: f"{prefix}.{params.get(key, key)}{w}" for key in ("q", "k", "v", "g", "o")}
        n["norm"] = f"{prefix}.{params.get('norm', 'norm')}"
        return n

    @classmethod
    def expected_tensors(cls, params, prefix: str) -> dict[str, TensorSpec]:
        hidden, heads, dim = int(params["hidden_size"]), int(params["num_heads"]), int(params["head_dim"])
        vdim = int(params.get("v_head_dim") or dim)
        n = cls._names(params, prefix)
        std = float(params.get("init_std", 0.02))
        out = {n["q"]: TensorSpec((heads * dim, hidden), init_std=std), n["k"]: TensorSpec((heads * dim, hidden), init_std=std),
               n["v"]: TensorSpec((heads * vdim, hidden), init_std=std), n["o"]: TensorSpec((hidden, heads * vdim), init_std=std),
               n["norm"]: TensorSpec((heads * vdim,), role="vector", init_std=0.1, init_mean=1.0)}
        if params.get("gate", True):
            out[n["g"]] = TensorSpec((heads * vdim, hidden), init_std=std)
        return out

    def load(self, source) -> None:
        n = self._names(self.params, self.prefix)
        dtype, device = self.runtime.dtype, self.runtime.device
        rows = [source(n[key]).to(dtype) for key in (("q", "k", "v", "g") if self.gated else ("q", "k", "v"))]
        used = sum(r.shape[0] for r in rows)
        if self.proj_rows > used:
            rows.append(torch.zeros(self.proj_rows - used, self.hidden, dtype=dtype, device=rows[0].device))
        self.proj.set_weight(torch.cat(rows, dim=0))
        self.o.set_weight(source(n["o"]))
        self.norm = to_device(source(n["norm"]), torch.float32, device)
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=device)

    def cache_request(self):
        return StateRequest((self.heads, self.vdim, self.dim), torch.float32)

    def forward(self, x, ctx, cache):
        if not cache.writable:
            raise ValueError(f"{self.prefix}: a recurrent mixer cannot read another layer's state")
        tokens = x.shape[0]
        ws = self.runtime.workspace
        proj = self.proj(x)
        read = ws.view("linattn.read", tokens, self.heads, self.vdim)
        # q, k and v are summed and activated once, not by every block of the recurrence that reads them
        ready = kernels.linear_attention_prepare(proj, self.at_gate, ws.view("linattn.qkv", tokens, self.at_gate), self.act)
        kernels.linear_attention_scan(ready, 0, self.at_k, self.at_v, self.decay, cache.state, read, ctx, self.dim, False)
        normed = ws.view("linattn.normed", tokens, self.heads * self.vdim)
        kernels.group_gate_norm(read.view(tokens, self.heads * self.vdim), self.norm, self.eps, normed, proj=proj if self.gated else None, at_gate=self.at_gate)
        return self.o(normed)


class _DecayedMixer:
    """What the mixers around ``kernels.decayed_attention`` share: its scratch, their output product and their checks."""

    graph_safe = True

    def _declare_scratch(self, per_channel: bool) -> None:
        ws, tokens = self.runtime.workspace, self.runtime.max_step_tokens
        self._scratch = {f"decayed.{name}": numel for name, numel in kernels.decay_scratch(tokens, self.heads, self.dim, self.vdim, per_channel).items()}
        for name, numel in self._scratch.items():
            ws.declare(name, numel, torch.float32)
        ws.declare("decayed.read", tokens * self.heads * self.vdim, torch.float32)
        ws.declare("decayed.normed", tokens * self.heads * self.vdim, self.runtime.dtype)

    def _scratch_views(self) -> dict:
        return {name.split(".", 1)[1]: self.runtime.workspace.view(name, numel) for name, numel in self._scratch.items()}

    def _check(self, states) -> None:
        if not states.writable:
            raise ValueError(f"{self.prefix}: a recurrent mixer cannot read another layer's state")

    def _output(self, normed, tokens: int):
        # few tokens: the product is left to the block, whose next norm launches it with the residual addition in its epilogue
        return DeferredProduct(self.o, normed) if self.o.fusable(tokens) else self.o(normed)


@register_mixer("gated_linear_attention")
class GatedLinearAttention(_DecayedMixer):
    """Linear attention with a decay per key channel and token ("gated linear attention"):

        S <- diag(alpha_t) S + k_t v_t^T;   o_t = dim^-1/2 S^T q_t

    with q = W_q h, k = W_k h ([heads, dim]), v = W_v h ([heads, vdim]) and alpha = sigmoid(W_a2 (W_a1 h) + b)^(1/tau), [heads,
    dim], a projection through few columns (the kernels pass its logarithm on).  Every head's o is RMS-normed over vdim with
    a weight shared by the heads (``eps`` inside the root), the concatenated heads are multiplied by silu(W_g h) and projected
    by W_o.  Per sequence the mixer keeps the states, float, zero for a new sequence, in the cache's per-slot state rows
    (stored transposed, [heads, vdim, dim]).  The five projections of h run as one product with float sums; everything between
    it and the output projection is float (``csrc/linear_attention.cu``, ``csrc/linear_attention_chunk.cu``, the narrow
    projection in ``csrc/delta_rule.cu``).

    Parameters: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_head_dim``, ``tau``, ``decay_rank``, ``eps``, ``float_out``,
    ``init_std``, and the tensor-name pieces ``q``, ``k``, ``v``, ``g``, ``o``, ``norm``, ``decay_in``, ``decay_out``, ``weight_suffix``,
    ``bias_suffix``."""

    def __init__(self, params, prefix: str, runtime: Runtime) -> None:
        self.prefix, self.runtime, self.params = prefix, runtime, dict(params)
        self.hidden = int(params["hidden_size"])
        self.heads, self.dim = int(params["num_heads"]), int(params["head_dim"])
        self.vdim = int(params.get("v_head_dim") or self.dim)
        self.tau = float(params["tau"])
        self.rank = int(params["decay_rank"])
        self.eps = float(params.get("eps", 1e-6))
        if self.dim > kernels.LINEAR_ATTENTION_MAX_DIM:
            raise ValueError(f"{prefix}: {self.dim} key channels per head are beyond what the recurrence kernels hold "
                             f"({kernels.LINEAR_ATTENTION_MAX_DIM})")
        self.at_k = self.heads * self.dim
        self.at_v = 2 * self.heads * self.dim
        self.at_gate = self.at_v + self.heads * self.vdim
        self.at_decay = self.at_gate + self.heads * self.vdim
        self.proj_rows = -(-(self.at_decay + self.rank) // 8) * 8
        self.proj = Linear("gla.proj", self.proj_rows, self.hidden, runtime, float_out=True, role="qkv")
        self.takes_scaled_rows = self.proj.fused_capable
        float_out = bool(params.get("float_out", False))
        self.o = Linear("gla.o" + (".float" if float_out else ""), self.hidden, self.heads * self.vdim, runtime, float_out=float_out, role="attn_out")
        ws = runtime.workspace
        ws.declare("gla.decay", runtime.max_step_tokens * self.heads * self.dim, torch.float32)
        ws.declare("gla.qkv", runtime.max_step_tokens * self.at_gate, torch.float32)
        self._declare_scratch(per_channel=True)
        self.norm = self.decay_out = self.decay_bias = None

    @staticmethod
    def _names(params, prefix: str) -> dict[str, str]:
        w, b = str(params.get("weight_suffix", ".weight")), str(params.get("bias_suffix", ".bias"))
        n = {key: f"{prefix}.{params.get(key, key)}{w}" for key in ("q", "k", "v", "g", "o", "decay_in", "decay_out")}
        n["decay_bias"] = f"{prefix}.{params.get('decay_out', 'decay_out')}{b}"
        n["norm"] = f"{prefix}.{params.get('norm', 'norm')}"
        return n

    @classmethod
    def expected_tensors(cls, params, prefix: str) -> dict[str, TensorSpec]:
        hidden, heads, dim = int(params["hidden_size"]), int(params["num_heads"]), int(params["head_dim"])
        vdim, rank = int(params.get("v_head_dim") or dim), int(params["decay_rank"])
        n = cls._names(params, prefix)
        std, narrow = float(params.get("init_std", 0.02)), float(params.get("narrow_init_std", 0.2))
        return {n["q"]: TensorSpec((heads * dim, hidden), init_std=std), n["k"]: TensorSpec((heads * dim, hidden), init_std=std),
                n["v"]: TensorSpec((heads * vdim, hidden), init_std=std), n["g"]: TensorSpec((heads * vdim, hidden), init_std=std),
                n["o"]: TensorSpec((hidden, heads * vdim), init_std=std), n["norm"]: TensorSpec((vdim,), role="vector", init_std=0.1, init_mean=1.0),
                n["decay_in"]: TensorSpec((rank, hidden), init_std=std), n["decay_out"]: TensorSpec((heads * dim, rank), init_std=narrow),
                n["decay_bias"]: TensorSpec((heads * dim,), role="vector", init_std=0.5, init_mean=1.0)}

    def load(self, source) -> None:
        n = self._names(self.params, self.prefix)
        dtype, device = self.runtime.dtype, self.runtime.device
        rows = [source(n[key]).to(dtype) for key in ("q", "k", "v", "g", "decay_in")]
        used = sum(r.shape[0] for r in rows)
        if self.proj_rows > used:
            rows.append(torch.zeros(self.proj_rows - used, self.hidden, dtype=dtype, device=rows[0].device))
        self.proj.set_weight(torch.cat(rows, dim=0))
        self.o.set_weight(source(n["o"]))
        # the narrow projection's second matrix: float, transposed to [rank, N] so that neighbouring threads read neighbouring outputs
        self.decay_out = to_device(source(n["decay_out"]).float().t(), torch.float32, device)
        self.decay_bias = to_device(source(n["decay_bias"]), torch.float32, device)
        self.norm = to_device(source(n["norm"]), torch.float32, device)

    def cache_request(self):
        return StateRequest((self.heads, self.vdim, self.dim), torch.float32)

    def forward(self, x, ctx, cache):
        self._check(cache)
        tokens, width = x.shape[0], self.heads * self.vdim
        ws = self.runtime.workspace
        proj = self.proj.finished(x)
        decay = ws.view("gla.decay", tokens, self.heads, self.dim)
        kernels.lowrank(proj, self.at_decay, self.decay_out, decay.view(tokens, self.heads * self.dim), self.decay_bias, power=1.0 / self.tau)
        # split sums are added once, not by every block of the recurrence that reads them
        rows = proj if proj.n_splits == 1 else kernels.linear_attention_prepare(proj, self.at_gate, ws.view("gla.qkv", tokens, self.at_gate), False)
        read = ws.view("decayed.read", tokens, self.heads, self.vdim)
        kernels.decayed_attention(rows, 0, self.at_k, self.at_v, decay, cache.state, read, ctx, self.dim, self._scratch_views(),
                                  out_scale=self.dim ** -0.5)
        normed = ws.view("decayed.normed", tokens, width)
        kernels.group_gate_norm(read.view(tokens, width), self.norm, self.eps, normed, groups=self.heads, proj=proj, at_gate=self.at_gate, gate="silu")
        return self._output(normed, tokens)


@register_mixer("retention")
class Retention(_DecayedMixer):
    """Linear attention with a fixed decay per head and rotated queries and keys ("retention"):

        S <- decay_h S + k_t v_t^T;   o_t = dim^-1/2 S^T q_t

    with q = R(W_q h), k = R(W_k h) ([heads, dim]) and v = W_v h ([heads, vdim]), R the rotation of the part ``position`` by the token's
    position (pairs (i, i + dims / 2)).  Every head's o is divided by its root mean square over vdim (``eps`` inside the root, no
    weight), the concatenated heads are multiplied by silu(W_g h) and projected by W_o.  Per sequence the mixer keeps the states,
    float, zero for a new sequence, in the cache's per-slot state rows (stored transposed, [heads, vdim, dim]).  The four projections
    of h run as one product with float sums; everything between it and the output projection is float
    (``csrc/linear_attention.cu``, ``csrc/linear_attention_chunk.cu``: the kernels for decays that depend on the token, here given
    the same logarithm for every token).

    Parameters: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_head_dim``, ``decay`` (one number per head, above 0 and at most 1),
    ``position``, ``eps``, ``float_out``, ``init_std``, and the tensor-name pieces ``q``, ``k``, ``v``, ``g``, ``o``, ``weight_suffix``."""

    def __init__(self, params, prefix: str, runtime: Runtime) -> None:
        self.prefix, self.runtime, self.params = prefix, runtime, dict(params)
        self.hidden = int(params["hidden_size"])
        self.heads, self.dim = int(params["num_heads"]), int(params["head_dim"])
        self.vdim = int(params.get("v_head_dim") or self.dim)
        self.eps = float(params.get("eps", 1e-6))
        self.decay_values = [float(d) for d in params["decay"]]
        if len(self.decay_values) != self.heads or not all(0.0 < d <= 1.0 for d in self.decay_values):
            raise ValueError(f"{prefix}: {self.heads} heads need as many decays above 0 and at most 1, not {self.decay_values}")
        if self.dim > kernels.LINEAR_ATTENTION_MAX_DIM:
            raise ValueError(f"{prefix}: {self.dim} key channels per head are beyond what the recurrence kernels hold "
                             f"({kernels.LINEAR_ATTENTION_MAX_DIM})")
        position_spec = params["position"]
        self.position = part_class("position", position_spec)(position_spec.params, runtime)
        if getattr(self.position, "interleaved", False):
            raise ValueError(f"{prefix}: the recurrence's rotation pairs element i with element i + dims / 2")
        self.cos_sin = None
        self.at_k = self.heads * self.dim
        self.at_v = 2 * self.heads * self.dim
        self.at_gate = self.at_v + self.heads * self.vdim
        self.proj_rows = -(-(self.at_gate + self.heads * self.vdim) // 8) * 8
        self.proj = Linear("retention.proj", self.proj_rows, self.hidden, runtime, float_out=True, role="qkv")
        self.takes_scaled_rows = self.proj.fused_capable
        float_out = bool(params.get("float_out", False))
        self.o = Linear("retention.o" + (".float" if float_out else ""), self.hidden, self.heads * self.vdim, runtime, float_out=float_out, role="attn_out")
        runtime.workspace.declare("retention.qkv", runtime.max_step_tokens * self.at_gate, torch.float32)
        self._declare_scratch(per_channel=False)
        self.norm = self.log_decay = None

    @staticmethod
    def _names(params, prefix: str) -> dict[str, str]:
        w = str(params.get("weight_suffix", ".weight"))
        return {key: f"{prefix}.{params.get(key, key)}{w}" for key in ("q", "k", "v", "g", "o")}

    @classmethod
    def expected_tensors(cls, params, prefix: str) -> dict[str, TensorSpec]:
        hidden, heads, dim = int(params["hidden_size"]), int(params["num_heads"]), int(params["head_dim"])
        vdim = int(params.get("v_head_dim") or dim)
        n = cls._names(params, prefix)
        std = float(params.get("init_std", 0.02))
        return {n["q"]: TensorSpec((heads * dim, hidden), init_std=std), n["k"]: TensorSpec((heads * dim, hidden), init_std=std),
                n["v"]: TensorSpec((heads * vdim, hidden), init_std=std), n["g"]: TensorSpec((heads * vdim, hidden), init_std=std),
                n["o"]: TensorSpec((hidden, heads * vdim), init_std=std)}

    def load(self, source) -> None:
        n = self._names(self.params, self.prefix)
        dtype, device = self.runtime.dtype, self.runtime.device
        rows = [source(n[key]).to(dtype) for key in ("q", "k", "v", "g")]
        used = sum(r.shape[0] for r in rows)
        if self.proj_rows > used:
            rows.append(torch.zeros(self.proj_rows - used, self.hidden, dtype=dtype, device=rows[0].device))
        self.proj.set_weight(torch.cat(rows, dim=0))
        self.o.set_weight(source(n["o"]))
        self.norm = torch.ones(self.vdim, dtype=torch.float32, device=device)
        # the logarithms, formed in double, for as many tokens as a step may have
        logs = torch.tensor(self.decay_values, dtype=torch.float64).log().to(torch.float32)
        self.log_decay = logs.to(device).expand(self.runtime.max_step_tokens, self.heads).contiguous()
        tables = self.runtime.options.setdefault("position_tables", {})
        key = self.position.key() + (self.runtime.max_positions,)
        if key not in tables:
            tables[key] = self.position.table(self.runtime.max_positions)
        self.cos_sin = tables[key]

    def cache_request(self):
        return StateRequest((self.heads, self.vdim, self.dim), torch.float32)

    def forward(self, x, ctx, cache):
        self._check(cache)
        tokens, width = x.shape[0], self.heads * self.vdim
        ws = self.runtime.workspace
        proj = self.proj.finished(x)
        if self.cos_sin is not None:
            rows = kernels.linear_attention_rotate(proj, self.at_gate, ws.view("retention.qkv", tokens, self.at_gate), 2 * self.heads, self.dim, self.cos_sin,
                                                   ctx.token_pos)
        else:
            rows = proj if proj.n_splits == 1 else kernels.linear_attention_prepare(proj, self.at_gate, ws.view("retention.qkv", tokens, self.at_gate), False)
        read = ws.view("decayed.read", tokens, self.heads, self.vdim)
        kernels.decayed_attention(rows, 0, self.at_k, self.at_v, self.log_decay[:tokens], cache.state, read, ctx, self.dim, self._scratch_views(),
                                  out_scale=self.dim ** -0.5)
        normed = ws.view("decayed.normed", tokens, width)
        kernels.group_gate_norm(read.view(tokens, width), self.norm, self.eps, normed, groups=self.heads, proj=proj, at_gate=self.at_gate, gate="silu")
        return self._output(normed, tokens)


@register_mixer("state_space")
class StateSpace(_DecayedMixer):
    """A state-space recurrence with a decay per head and token ("Mamba-2"):

        S <- exp(-exp(A_h) d_t) S + d_t B_t x_t^T;   y_t = S^T C_t + D_h x_t

    W_in h is laid out as [z | x | B | C | d]: z and x [heads, vdim], B and C [groups, state] (head h reads group
    h // (heads / groups)), d one number per head.  x, B and C together pass a causal convolution per channel (``conv`` taps,
    the last one the current token's, zeros before the sequence's start; with a bias) and SiLU; d is softplus(d + bias).  The
    heads' y are concatenated, multiplied by silu(z), divided by the root mean square of each of ``norm_groups`` equal parts
    (``eps`` inside the root), times a weight, and projected by W_o.  Per sequence the mixer keeps the states [heads, vdim,
    state] and the convolution's last ``conv`` - 1 inputs, both float, zero for a new sequence, in the cache's per-slot state
    rows.  The first product hands on float sums and everything between it and the output projection is float
    (``csrc/short_conv.cu``, ``csrc/linear_attention.cu``, ``csrc/linear_attention_chunk.cu``).

    Parameters: ``hidden_size``, ``num_heads``, ``v_head_dim``, ``state``, ``groups``, ``conv``, ``norm_groups``, ``eps``, ``float_out``,
    ``init_std``, and the tensor-name pieces ``in``, ``conv_name``, ``step_bias``, ``decay_rate``, ``skip``, ``norm``, ``o``,
    ``weight_suffix``, ``bias_suffix``."""

    def __init__(self, params, prefix: str, runtime: Runtime) -> None:
        self.prefix, self.runtime, self.params = prefix, runtime, dict(params)
        self.hidden = int(params["hidden_size"])
        self.heads, self.vdim, self.dim = int(params["num_heads"]), int(params["v_head_dim"]), int(params["state"])
        self.groups, self.taps = int(params.get("groups", 1)), int(params.get("conv", 1))
        self.norm_groups, self.eps = int(params.get("norm_groups", 1)), float(params.get("eps", 1e-6))
        self.inner = self.heads * self.vdim
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"{prefix}: {self.groups} groups for {self.heads} heads, {self.norm_groups} norm groups for {self.inner} columns")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"{prefix}: a convolution of {self.taps} taps (1..16)")
        if self.dim > kernels.LINEAR_ATTENTION_MAX_DIM:
            raise ValueError(f"{prefix}: states of {self.dim} rows per head are beyond what the recurrence kernels hold ({kernels.LINEAR_ATTENTION_MAX_DIM})")
        self.channels = self.inner + 2 * self.groups * self.dim
        self.at_step = self.inner + self.channels
        self.rows = self.at_step + self.heads
        self.proj_rows = -(-self.rows // 8) * 8
        self.proj = Linear("ssm.proj", self.proj_rows, self.hidden, runtime, float_out=True, role="qkv")
        self.takes_scaled_rows = self.proj.fused_capable
        float_out = bool(params.get("float_out", False))
        self.o = Linear("ssm.o" + (".float" if float_out else ""), self.hidden, self.inner, runtime, float_out=float_out, role="attn_out")
        ws, tokens = runtime.workspace, runtime.max_step_tokens
        ws.declare("ssm.mixed", tokens * self.channels, torch.float32)
        ws.declare("ssm.step", tokens * self.heads, torch.float32)
        ws.declare("ssm.decay", tokens * self.heads, torch.float32)
        self._declare_scratch(per_channel=False)
        self.conv = self.conv_bias = self.step_bias = self.rate_log = self.skip = self.norm = None

    @staticmethod
    def _names(params, prefix: str) -> dict[str, str]:
        w, b = str(params.get("weight_suffix", ".weight")), str(params.get("bias_suffix", ".bias"))
        conv = str(params.get("conv_name", "conv"))
        n = {key: f"{prefix}.{params.get(key, key)}{w}" for key in ("in", "o")}
        n.update({key: f"{prefix}.{params.get(key, key)}" for key in ("step_bias", "decay_rate", "skip", "norm")})
        n["conv"], n["conv_bias"] = f"{prefix}.{conv}{w}", f"{prefix}.{conv}{b}"
        return n

    @classmethod
    def expected_tensors(cls, params, prefix: str) -> dict[str, TensorSpec]:
        hidden, heads, vdim, state = (int(params[key]) for key in ("hidden_size", "num_heads", "v_head_dim", "state"))
        groups, taps = int(params.get("groups", 1)), int(params.get("conv", 1))
        inner = heads * vdim
        channels = inner + 2 * groups * state
        n = cls._names(params, prefix)
        std = float(params.get("init_std", 0.02))
        return {n["in"]: TensorSpec((inner + channels + heads, hidden), init_std=std), n["o"]: TensorSpec((hidden, inner), init_std=std),
                n["conv"]: TensorSpec((channels, taps), role="vector", init_std=0.3, init_mean=0.3),
                n["conv_bias"]: TensorSpec((channels,), role="vector", init_std=0.1), n["step_bias"]: TensorSpec((heads,), role="vector", init_std=0.5, init_mean=-1.0),
                n["decay_rate"]: TensorSpec((heads,), role="vector", init_std=0.5, init_mean=-1.0),
                n["skip"]: TensorSpec((heads,), role="vector", init_std=0.3, init_mean=1.0),
                n["norm"]: TensorSpec((inner,), role="vector", init_std=0.1, init_mean=1.0)}

    def load(self, source) -> None:
        n = self._names(self.params, self.prefix)
        dtype, device = self.runtime.dtype, self.runtime.device
        weight = source(n["in"]).to(dtype)
        if self.proj_rows > self.rows:
            weight = torch.cat((weight, torch.zeros(self.proj_rows - self.rows, self.hidden, dtype=dtype, device=weight.device)), dim=0)
        self.proj.set_weight(weight)
        self.o.set_weight(source(n["o"]))
        self.conv, self.conv_bias, self.step_bias, self.rate_log, self.skip, self.norm = (
            to_device(source(n[key]), torch.float32, device) for key in ("conv", "conv_bias", "step_bias", "decay_rate", "skip", "norm"))

    def cache_request(self):
        return [StateRequest((self.heads, self.vdim, self.dim), torch.float32), StateRequest((max(self.taps - 1, 1), self.channels), torch.float32)]

    def forward(self, x, ctx, cache):
        states, kept = cache
        self._check(states)
        tokens = x.shape[0]
        ws = self.runtime.workspace
        proj = self.proj.finished(x)
        mixed = ws.view("ssm.mixed", tokens, self.channels)
        step, decay = ws.view("ssm.step", tokens, self.heads), ws.view("ssm.decay", tokens, self.heads)
        kernels.conv_act(proj, self.inner, self.conv, self.conv_bias, kept.state, ctx, mixed, self.at_step, self.step_bias, self.rate_log, step, decay)
        read = ws.view("decayed.read", tokens, self.heads, self.vdim)
        at_b, at_c = self.inner, self.inner + self.groups * self.dim
        kernels.decayed_attention(GemmOut(mixed.view(1, tokens, self.channels)), at_c, at_b, 0, decay, states.state, read, ctx, self.dim,
                                  self._scratch_views(), heads_per_key=self.heads // self.groups, v_scale=step)
        normed = ws.view("decayed.normed", tokens, self.inner)
        kernels.group_gate_norm(read.view(tokens, self.inner), self.norm, self.eps, normed, groups=self.norm_groups, proj=proj, at_gate=0, gate="silu",
                                gate_first=True, x=mixed, at_x=0, skip=self.skip)
        return self._output(normed, tokens)
