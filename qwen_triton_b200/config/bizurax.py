"""Typed configuration of the Bizurax design, read from config.json.

The file names its design under ``architecture`` and gives ``vocab``, ``width``, ``norm.eps``, ``streams`` (parallel copies of the residual
stream; absent: the plain residual sum), ``residual_mult`` (a constant on everything that is added to the stream; absent: 1) and a list
``layers``.  An entry has ``type`` (its mixer), the mixer's sizes and constants under ``mixer`` and its feed-forward under ``mlp`` (null
for none).  Layers need not be alike.  ``loop`` (absent: none) makes the layers ``start`` .. ``stop`` - 1 run ``times`` times in a row
with the same weights, every pass with a cache and states of its own.

``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap`` (absent: scores are not capped), ``rot``.
``latent_attention``: ``heads``, ``dim`` and ``rot_dim`` (unrotated and rotated query/key elements per head), ``vdim``, ``kv_rank``,
``scale``, ``rot``.
``retention``: ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head), ``rot``.
``rot``: ``dims`` (absent or 0: no rotation), ``base`` and ``scaling.factor`` (every frequency is divided by it; absent: 1).
``mlp``: ``kind`` "dense" with ``ff``, or "moe" with ``expert.ff``, ``router.experts``, ``router.top`` and ``shared.ff`` (absent: no
shared expert).

What the design fixes, and ``model_spec`` therefore states as parameters of the parts: RMS norms with weights in front of every
sublayer and in front of the head; every sublayer reads and writes the streams with weights of its own; ``attention`` with biases on q,
k and v, rotation of halves, q and k divided by their root mean square, a learned sink; the latent attention without a query latent or
a gate, its rotation of neighbouring pairs; the ``retention``'s rotation of halves, its norm per head without a weight and its SiLU
gate; a dense feed-forward of two matrices with the squared ReLU; SiLU-gated experts chosen by a router with a bias, weighted by the
softmax over the chosen, the shared expert added as it is; tensor names without a ``.weight`` suffix.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .qwen3 import ConfigError
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec

MAX_POSITIONS = 1 << 20          # the design names no longest sequence; the rotation table is made for the cache's length
MAX_STREAMS = 32                 # of the kernel between two sublayers


@dataclass(frozen=True)
class BizuraxRotation:
    dims: int
    base: float = 10000.0
    factor: float = 1.0

    def part(self, head_dim: int, pairing: str = "half") -> PartSpec:
        if not self.dims:
            return PartSpec("none")
        return PartSpec("rope", {"theta": self.base, "rotary_dim": self.dims, "head_dim": head_dim, "pairing": pairing, "angles": "float64",
                                 "factor": self.factor})

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.factor != 1.0:
            out["scaling"] = {"factor": self.factor}
        return out


@dataclass(frozen=True)
class BizuraxAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None = None
    rot: BizuraxRotation = BizuraxRotation(0)


@dataclass(frozen=True)
class BizuraxLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: BizuraxRotation = BizuraxRotation(0)


@dataclass(frozen=True)
class BizuraxRetention:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: BizuraxRotation = BizuraxRotation(0)


@dataclass(frozen=True)
class BizuraxFeedForward:
    kind: str                          # "dense" or "moe"
    ff: int
    experts: int = 0
    top: int = 0
    shared_ff: int | None = None


@dataclass(frozen=True)
class BizuraxLayer:
    type: str
    mixer: BizuraxAttention | BizuraxLatent | BizuraxRetention
    mlp: BizuraxFeedForward | None = None


@dataclass(frozen=True)
class BizuraxLoop:
    start: int
    stop: int
    times: int


def _need(mapping: Mapping[str, Any], key: str, where: str):
    if not isinstance(mapping, Mapping) or mapping.get(key) is None:
        raise ConfigError(f"config.json lacks {where}.{key}" if where else f"config.json lacks the key {key!r}")
    return mapping[key]


def _rotation(m: Mapping[str, Any], at: str) -> BizuraxRotation:
    rot = m.get("rot")
    if not rot or not rot.get("dims"):
        return BizuraxRotation(0)
    scaling = rot.get("scaling")
    return BizuraxRotation(int(rot["dims"]), float(_need(rot, "base", f"{at}.rot")),
                           float(_need(scaling, "factor", f"{at}.rot.scaling")) if scaling else 1.0)


def _mixer(kind: str, m: Mapping[str, Any], at: str):
    def size(key: str) -> int:
        return int(_need(m, key, at))

    common = {"heads": size("heads"), "dim": size("dim"), "vdim": int(m.get("vdim") or size("dim")), "rot": _rotation(m, at)}
    if kind == "attention":
        cap = m.get("softcap")
        return BizuraxAttention(**common, kv_heads=int(m.get("kv_heads") or common["heads"]), scale=float(_need(m, "scale", at)),
                                softcap=None if cap is None else float(cap))
    if kind == "latent_attention":
        return BizuraxLatent(**common, rot_dim=int(m.get("rot_dim") or 0), kv_rank=size("kv_rank"), scale=float(_need(m, "scale", at)))
    if kind == "retention":
        return BizuraxRetention(**common, decay=tuple(float(d) for d in _need(m, "decay", at)))
    raise ConfigError(f"{at}: the Bizurax design has no mixer {kind!r}")


def _feed_forward(mlp, at: str) -> BizuraxFeedForward | None:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", at)
    if kind == "dense":
        return BizuraxFeedForward("dense", int(_need(mlp, "ff", at)))
    if kind != "moe":
        raise ConfigError(f"{at}: the Bizurax design has no feed-forward {kind!r}")
    router, shared = _need(mlp, "router", at), mlp.get("shared")
    return BizuraxFeedForward("moe", int(_need(_need(mlp, "expert", at), "ff", f"{at}.expert")), int(_need(router, "experts", f"{at}.router")),
                              int(_need(router, "top", f"{at}.router")), None if shared is None else int(_need(shared, "ff", f"{at}.shared")))


@dataclass(frozen=True)
class BizuraxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[BizuraxLayer, ...]
    streams: int | None = None
    residual_mult: float = 1.0
    loop: BizuraxLoop | None = None
    architecture: str = "Bizurax"
    raw: Mapping[str, Any] = field(default_factory=dict, repr=False, compare=False)

    family = "bizurax"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_hf_config(cls, raw: Mapping[str, Any]) -> "BizuraxConfig":
        if not isinstance(raw, Mapping):
            raise TypeError(f"unsupported config type: {type(raw)!r}")
        entries = _need(raw, "layers", "")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]"
            kind = _need(entry, "type", where)
            layers.append(BizuraxLayer(kind, _mixer(kind, _need(entry, "mixer", where), f"{where}.mixer"),
                                       _feed_forward(entry.get("mlp"), f"{where}.mlp")))
        loop = raw.get("loop")
        if loop is not None:
            loop = BizuraxLoop(*(int(_need(loop, key, "loop")) for key in ("start", "stop", "times")))
        mult = raw.get("residual_mult")
        config = cls(vocab=int(_need(raw, "vocab", "")), width=int(_need(raw, "width", "")),
                     norm_eps=float(_need(_need(raw, "norm", ""), "eps", "norm")), layers=tuple(layers),
                     streams=None if raw.get("streams") is None else int(raw["streams"]), residual_mult=1.0 if mult is None else float(mult),
                     loop=loop, architecture=str(raw.get("architecture", "Bizurax")), raw=dict(raw))
        config.validate()
        return config

    def validate(self) -> None:
        problems: list[str] = []
        if self.vocab <= 0 or self.width <= 0:
            problems.append("vocab and width must be positive")
        if self.norm_eps <= 0.0:
            problems.append("norm.eps must be positive")
        if self.streams is not None and not 1 <= self.streams <= MAX_STREAMS:
            problems.append(f"streams={self.streams} (1..{MAX_STREAMS})")
        for index, layer in enumerate(self.layers):
            where, m = f"layers[{index}]", layer.mixer
            if min(m.heads, m.dim, m.vdim) <= 0:
                problems.append(f"{where}: heads, dim and vdim must be positive")
            turning = m.rot_dim if isinstance(m, BizuraxLatent) else m.dim
            if m.rot.dims % 2 or not 0 <= m.rot.dims <= turning or (m.rot.dims and (m.rot.base <= 0 or m.rot.factor <= 0)):
                problems.append(f"{where}: rot.dims={m.rot.dims} must be even and at most {turning}, base and factor positive")
            if isinstance(m, BizuraxAttention):
                if m.kv_heads <= 0 or m.heads % m.kv_heads:
                    problems.append(f"{where}: kv_heads={m.kv_heads} must divide heads={m.heads}")
                if m.softcap is not None and m.softcap <= 0:
                    problems.append(f"{where}: softcap={m.softcap} must be positive")
            elif isinstance(m, BizuraxLatent):
                if m.kv_rank <= 0 or m.rot_dim < 0:
                    problems.append(f"{where}: kv_rank={m.kv_rank} must be positive, rot_dim={m.rot_dim} not negative")
            elif len(m.decay) != m.heads or not all(0.0 < d <= 1.0 for d in m.decay):
                problems.append(f"{where}: {m.heads} heads need as many decays above 0 and at most 1")
            f = layer.mlp
            if f is not None and (f.ff <= 0 or (f.kind == "moe" and not 0 < f.top <= f.experts) or (f.shared_ff is not None and f.shared_ff <= 0)):
                problems.append(f"{where}.mlp: ff={f.ff}, top={f.top} of experts={f.experts}, shared={f.shared_ff}")
        if self.loop is not None and not (0 <= self.loop.start < self.loop.stop <= len(self.layers) and self.loop.times >= 1):
            problems.append(f"loop: layers {self.loop.start} .. {self.loop.stop} - 1 of {len(self.layers)}, {self.loop.times} times")
        if problems:
            raise ConfigError("invalid Bizurax configuration: " + "; ".join(problems))

    # ------------------------------------------------------------------ export
    def to_hf_dict(self) -> dict[str, Any]:
        """The config.json that parses back into this configuration."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            mixer: dict[str, Any] = {"dim": m.dim, "heads": m.heads, "vdim": m.vdim}
            if m.rot.dims:
                mixer["rot"] = m.rot.to_dict()
            if isinstance(m, BizuraxAttention):
                mixer |= {"kv_heads": m.kv_heads, "scale": m.scale}
                if m.softcap is not None:
                    mixer["softcap"] = m.softcap
            elif isinstance(m, BizuraxLatent):
                mixer |= {"kv_rank": m.kv_rank, "rot_dim": m.rot_dim, "scale": m.scale}
            else:
                mixer["decay"] = list(m.decay)
            f, mlp = layer.mlp, None
            if f is not None and f.kind == "dense":
                mlp = {"ff": f.ff, "kind": "dense"}
            elif f is not None:
                mlp = {"expert": {"ff": f.ff}, "kind": "moe", "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff is not None:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"mixer": mixer, "mlp": mlp, "type": layer.type})
        out: dict[str, Any] = {"architecture": self.architecture, "layers": layers, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                               "vocab": self.vocab, "width": self.width}
        if self.streams is not None:
            out["streams"] = self.streams
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out

    # ------------------------------------------------------------------ parts
    def _mixer_part(self, m, init_std: float) -> PartSpec:
        common = {"hidden_size": self.width, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "float_out": True, "init_std": init_std,
                  "weight_suffix": ""}
        if isinstance(m, BizuraxAttention):
            return PartSpec("attention", {**common, "num_kv_heads": m.kv_heads, "scale": m.scale, "softcap": m.softcap, "position": m.rot.part(m.dim),
                                          "bias": True, "o_bias": False, "bias_suffix": ".b", "float_proj": True, "qk_norm": "unit",
                                          "qk_norm_eps": self.norm_eps, "sink": "learned"})
        if isinstance(m, BizuraxLatent):
            return PartSpec("latent_attention", {**common, "rot_dim": m.rot_dim, "kv_rank": m.kv_rank, "scale": m.scale, "eps": self.norm_eps,
                                                 "position": m.rot.part(m.rot_dim, "interleaved"), "gate": False, "norm_suffix": ".norm"})
        return PartSpec("retention", {**common, "decay": m.decay, "eps": self.norm_eps, "position": m.rot.part(m.dim)})

    def _feed_forward_part(self, f: BizuraxFeedForward, init_std: float) -> PartSpec:
        names = {"up": "up", "down": "down", "weight_suffix": "", "init_std": init_std}
        if f.kind == "dense":
            return PartSpec("plain_mlp", {"hidden_size": self.width, "intermediate_size": f.ff, "activation": "relu2", "float_out": True, **names})
        return PartSpec("routed_experts", {"hidden_size": self.width, "expert_size": f.ff, "experts": f.experts, "top": f.top, "score": "softmax",
                                           "activation": "silu", "router": "router", "router_bias": True, "bias_suffix": ".b", "expert": "e{}", "gate": "gate",
                                           "shared": None if f.shared_ff is None else {"intermediate_size": f.shared_ff}, "shared_gated": False,
                                           "router_init_std": 0.3, **names})

    def model_spec(self) -> ModelSpec:
        init_std = 0.06
        norm = PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "suffix": ""})
        # the plain residual sum times a constant is one stream that is read and kept as it is
        connection = {"streams": self.streams or 1, "mult": self.residual_mult, "learned": self.streams is not None, "in": "in", "mix": "mix", "out": "out"}
        block = PartSpec("hyper_connections", {"mixer": "mix", "feed_forward": "mlp", "mixer_norm": "norm1", "feed_forward_norm": "norm2",
                                               "mixer_connection": "hc1", "feed_forward_connection": "hc2", "connection": connection})
        layers = tuple(LayerSpec(prefix=f"l{index}", block=block, mixer=self._mixer_part(layer.mixer, init_std),
                                 feed_forward=None if layer.mlp is None else self._feed_forward_part(layer.mlp, init_std), norm=norm)
                       for index, layer in enumerate(self.layers))
        order = list(range(len(layers)))
        if self.loop is not None:
            start, stop = self.loop.start, self.loop.stop
            order = order[:start] + order[start:stop] * self.loop.times + order[stop:]
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, streams=self.streams or 1,
            embedding=PartSpec("token_embedding", {"name": "embed", "init_std": 0.5}),
            layers=layers, schedule=tuple(LayerCall(layer=index) for index in order),
            final_norm=PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "suffix": "", "name": "final.norm"}),
            head=PartSpec("linear_head", {"name": "head", "tied_to": None, "init_std": 0.25}),
            max_positions=MAX_POSITIONS, eos_token_ids=(),
        )
        spec.validate()
        return spec
