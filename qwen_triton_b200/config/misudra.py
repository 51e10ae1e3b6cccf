"""Typed configuration of the Misudra design, read from config.json.

The file names its design under ``architecture`` and gives ``vocab``, ``width``, ``norm.eps`` and a list ``layers``.  An entry
has ``type`` (its mixer), the mixer's sizes and constants under ``mixer`` and its feed-forward under ``mlp`` (null for none).
Layers need not be alike.  ``loop`` (absent: none) makes the layers ``start`` .. ``stop`` - 1 run ``times`` times in a row with the
same weights, every pass with a cache and states of its own.

``latent_attention``: ``heads``, ``dim`` and ``rot_dim`` (unrotated and rotated query/key elements per head), ``vdim``, ``q_rank``,
``kv_rank``, ``scale``, ``rot.dims`` / ``rot.base``, ``mask.size`` (absent: every earlier token is seen).
``gla``: ``heads``, ``dim``, ``vdim``, ``tau``.  The column count of the decay's narrow projection is no key of the file but the
shape of ``l<i>.mix.a1`` (a configuration that draws random weights names it under ``mixer.ranks.decay``).
``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` (taps), ``norm_groups``.
``mlp``: ``kind`` "dense" with ``ff``, or "moe" with ``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top`` and
``router.groups`` (``count``, ``keep``; absent: every expert may be chosen).

What the design fixes, and ``model_spec`` therefore states as parameters of the parts: RMS norms with weights in front of
every sublayer, behind the embedding and in front of the head; a pass of the loop starts with a matrix over the stream and
the embedding's output side by side; the latent attention's query latent, its window and one sigmoid gate per head; the
``gla`` decay sigmoid(.)^(1/tau) per key channel, its norm per head and its SiLU gate; the state-space mixer's biased
convolution with SiLU, its skip term, the gate ahead of its norm in groups; a dense feed-forward with biases and the
tanh-GELU gate; experts with the capped gate, chosen by a softmax router, their scores renormalised; tensor names without a
``.weight`` suffix.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Mapping

from .qwen3 import ConfigError
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec

MAX_POSITIONS = 1 << 20          # the design names no longest sequence; the rotation table is made for the cache's length


@dataclass(frozen=True)
class MisudraLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_dims: int = 0
    rot_base: float = 10000.0
    window: int | None = None          # mask.size


@dataclass(frozen=True)
class MisudraGla:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 0                # 0: not known yet (see with_tensor_shapes)


@dataclass(frozen=True)
class MisudraStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class MisudraFeedForward:
    kind: str                          # "dense" or "moe"
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    group_count: int = 1
    group_keep: int = 1


@dataclass(frozen=True)
class MisudraLayer:
    type: str
    mixer: MisudraLatent | MisudraGla | MisudraStateSpace
    mlp: MisudraFeedForward | None = None


@dataclass(frozen=True)
class MisudraLoop:
    start: int
    stop: int
    times: int


def _need(mapping: Mapping[str, Any], key: str, where: str):
    if not isinstance(mapping, Mapping) or mapping.get(key) is None:
        raise ConfigError(f"config.json lacks {where}.{key}" if where else f"config.json lacks the key {key!r}")
    return mapping[key]


def _mixer(kind: str, m: Mapping[str, Any], at: str):
    def size(key: str) -> int:
        return int(_need(m, key, at))

    if kind == "latent_attention":
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        return MisudraLatent(heads=size("heads"), dim=size("dim"), rot_dim=size("rot_dim"), vdim=int(m.get("vdim") or size("dim")),
                             q_rank=size("q_rank"), kv_rank=size("kv_rank"), scale=float(_need(m, "scale", at)),
                             rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base", 10000.0)),
                             window=int(mask["size"]) if mask.get("size") is not None else None)
    if kind == "gla":
        return MisudraGla(heads=size("heads"), dim=size("dim"), vdim=int(m.get("vdim") or size("dim")), tau=float(_need(m, "tau", at)),
                          decay_rank=int((m.get("ranks") or {}).get("decay") or 0))
    if kind == "mamba2":
        return MisudraStateSpace(heads=size("heads"), vdim=size("vdim"), state=size("state"), groups=int(m.get("groups") or 1),
                                 conv=int(m.get("conv") or 1), norm_groups=int(m.get("norm_groups") or 1))
    raise ConfigError(f"{at}: the Misudra design has no mixer {kind!r}")


def _feed_forward(mlp, at: str) -> MisudraFeedForward | None:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", at)
    if kind == "dense":
        return MisudraFeedForward("dense", int(_need(mlp, "ff", at)))
    if kind != "moe":
        raise ConfigError(f"{at}: the Misudra design has no feed-forward {kind!r}")
    expert, router = _need(mlp, "expert", at), _need(mlp, "router", at)
    groups = router.get("groups")
    count, keep = (1, 1) if groups is None else (int(_need(groups, key, f"{at}.router.groups")) for key in ("count", "keep"))
    return MisudraFeedForward("moe", int(_need(expert, "ff", f"{at}.expert")), float(_need(expert, "limit", f"{at}.expert")),
                              int(_need(router, "experts", f"{at}.router")), int(_need(router, "top", f"{at}.router")), count, keep)


@dataclass(frozen=True)
class MisudraConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[MisudraLayer, ...]
    loop: MisudraLoop | None = None
    architecture: str = "Misudra"
    raw: Mapping[str, Any] = field(default_factory=dict, repr=False, compare=False)

    family = "misudra"

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
    def from_hf_config(cls, raw: Mapping[str, Any]) -> "MisudraConfig":
        if not isinstance(raw, Mapping):
            raise TypeError(f"unsupported config type: {type(raw)!r}")
        entries = _need(raw, "layers", "")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]"
            kind = _need(entry, "type", where)
            layers.append(MisudraLayer(kind, _mixer(kind, _need(entry, "mixer", where), f"{where}.mixer"),
                                       _feed_forward(entry.get("mlp"), f"{where}.mlp")))
        loop = raw.get("loop")
        if loop is not None:
            loop = MisudraLoop(*(int(_need(loop, key, "loop")) for key in ("start", "stop", "times")))
        config = cls(vocab=int(_need(raw, "vocab", "")), width=int(_need(raw, "width", "")),
                     norm_eps=float(_need(_need(raw, "norm", ""), "eps", "norm")), layers=tuple(layers), loop=loop,
                     architecture=str(raw.get("architecture", "Misudra")), raw=dict(raw))
        config.validate()
        return config

    def with_tensor_shapes(self, shapes: Mapping[str, tuple[int, ...]]) -> "MisudraConfig":
        """The sizes that only the stored tensors give: ``l<i>.mix.a1`` of a ``gla`` layer is [decay columns, width]."""
        layers = []
        for index, layer in enumerate(self.layers):
            shape = shapes.get(f"l{index}.mix.a1")
            if isinstance(layer.mixer, MisudraGla) and shape is not None and len(shape) == 2:
                layer = replace(layer, mixer=replace(layer.mixer, decay_rank=int(shape[0])))
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def validate(self) -> None:
        problems: list[str] = []
        if self.vocab <= 0 or self.width <= 0:
            problems.append("vocab and width must be positive")
        if self.norm_eps <= 0.0:
            problems.append("norm.eps must be positive")
        for index, layer in enumerate(self.layers):
            where, m = f"layers[{index}]", layer.mixer
            if isinstance(m, MisudraLatent):
                if min(m.heads, m.dim, m.vdim, m.q_rank, m.kv_rank) <= 0 or m.rot_dim < 0:
                    problems.append(f"{where}: heads, dim, vdim, q_rank and kv_rank must be positive, rot_dim not negative")
                if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.rot_dim:
                    problems.append(f"{where}: rot.dims={m.rot_dims} must be even and at most rot_dim={m.rot_dim}")
                if m.window is not None and m.window <= 0:
                    problems.append(f"{where}: mask.size={m.window} must be positive")
            elif isinstance(m, MisudraGla):
                if min(m.heads, m.dim, m.vdim) <= 0 or m.tau <= 0.0 or m.decay_rank < 0:
                    problems.append(f"{where}: heads, dim, vdim and tau must be positive")
            else:
                if min(m.heads, m.vdim, m.state, m.groups, m.norm_groups) <= 0:
                    problems.append(f"{where}: heads, vdim, state, groups and norm_groups must be positive")
                elif m.heads % m.groups or (m.heads * m.vdim) % m.norm_groups:
                    problems.append(f"{where}: groups={m.groups} must divide heads={m.heads}, norm_groups={m.norm_groups} must divide {m.heads * m.vdim}")
                if not 1 <= m.conv <= 16:
                    problems.append(f"{where}: conv={m.conv} taps (1..16)")
            f = layer.mlp
            if f is None:
                continue
            if f.ff <= 0:
                problems.append(f"{where}.mlp: ff={f.ff}")
            if f.kind == "moe":
                if f.limit <= 0 or not 0 < f.top <= f.experts:
                    problems.append(f"{where}.mlp: limit={f.limit}, top={f.top} of experts={f.experts}")
                elif f.group_count <= 0 or f.experts % f.group_count or not 0 < f.group_keep <= f.group_count:
                    problems.append(f"{where}.mlp: keep={f.group_keep} of {f.group_count} groups for {f.experts} experts")
                elif f.top > f.group_keep * (f.experts // f.group_count):
                    problems.append(f"{where}.mlp: top={f.top} experts out of {f.group_keep} groups of {f.experts // f.group_count}")
        if self.loop is not None and not (0 <= self.loop.start < self.loop.stop <= len(self.layers) and self.loop.times >= 1):
            problems.append(f"loop: layers {self.loop.start} .. {self.loop.stop} - 1 of {len(self.layers)}, {self.loop.times} times")
        if problems:
            raise ConfigError("invalid Misudra configuration: " + "; ".join(problems))

    # ------------------------------------------------------------------ export
    def to_hf_dict(self) -> dict[str, Any]:
        """The config.json that parses back into this configuration."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if isinstance(m, MisudraLatent):
                mixer: dict[str, Any] = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "rot_dim": m.rot_dim,
                                         "scale": m.scale, "vdim": m.vdim}
                if m.rot_dims:
                    mixer["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
                if m.window is not None:
                    mixer["mask"] = {"size": m.window}
            elif isinstance(m, MisudraGla):
                mixer = {"dim": m.dim, "heads": m.heads, "tau": m.tau, "vdim": m.vdim}
                if m.decay_rank:
                    mixer["ranks"] = {"decay": m.decay_rank}
            else:
                mixer = {"conv": m.conv, "groups": m.groups, "heads": m.heads, "norm_groups": m.norm_groups, "state": m.state, "vdim": m.vdim}
            f, mlp = layer.mlp, None
            if f is not None and f.kind == "dense":
                mlp = {"ff": f.ff, "kind": "dense"}
            elif f is not None:
                router: dict[str, Any] = {"experts": f.experts, "top": f.top}
                if f.group_count > 1:
                    router["groups"] = {"count": f.group_count, "keep": f.group_keep}
                mlp = {"expert": {"ff": f.ff, "limit": f.limit}, "kind": "moe", "router": router}
            layers.append({"mixer": mixer, "mlp": mlp, "type": layer.type})
        out: dict[str, Any] = {"architecture": self.architecture, "layers": layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out

    # ------------------------------------------------------------------ parts
    def _mixer_part(self, index: int, m, init_std: float) -> PartSpec:
        common = {"hidden_size": self.width, "eps": self.norm_eps, "float_out": True, "init_std": init_std, "weight_suffix": ""}
        if isinstance(m, MisudraLatent):
            position = PartSpec("rope", {"theta": m.rot_base, "rotary_dim": m.rot_dims, "head_dim": m.rot_dim, "angles": "float64"}) \
                if m.rot_dims else PartSpec("none")
            return PartSpec("latent_attention", {**common, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim,
                                                 "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale, "window": m.window,
                                                 "position": position, "gate": "head", "norm_suffix": ".norm"})
        if isinstance(m, MisudraGla):
            if not m.decay_rank:
                raise ConfigError(f"layers[{index}]: the column count of the decay's narrow projection is unknown: it is the shape of "
                                  f"l{index}.mix.a1 in a model folder, or mixer.ranks.decay in the configuration")
            return PartSpec("gated_linear_attention", {**common, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "tau": m.tau,
                                                       "decay_rank": m.decay_rank, "decay_in": "a1", "decay_out": "a2", "bias_suffix": ".b"})
        return PartSpec("state_space", {**common, "num_heads": m.heads, "v_head_dim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv,
                                        "norm_groups": m.norm_groups, "bias_suffix": ".b", "decay_rate": "A_log", "skip": "D",
                                        "step_bias": "dt_bias"})

    def _feed_forward_part(self, f: MisudraFeedForward, init_std: float) -> PartSpec:
        names = {"gate": "gate", "up": "up", "down": "down", "weight_suffix": "", "init_std": init_std}
        if f.kind == "dense":
            return PartSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": f.ff, "activation": "gelu_pytorch_tanh", "bias": True,
                                          "bias_suffix": ".b", "float_out": True, **names})
        return PartSpec("routed_experts", {"hidden_size": self.width, "expert_size": f.ff, "experts": f.experts, "top": f.top, "score": "softmax",
                                           "groups": f.group_count, "keep_groups": f.group_keep, "activation": "capped_sigmoid", "limit": f.limit,
                                           "router": "router", "expert": "e{}", "router_init_std": 0.3, **names})

    def model_spec(self) -> ModelSpec:
        init_std = 0.06
        norm = PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "suffix": ""})
        block = PartSpec("pre_norm", {"mixer": "mix", "feed_forward": "mlp", "mixer_norm": "norm1", "feed_forward_norm": "norm2"})
        layers = tuple(LayerSpec(prefix=f"l{index}", block=block, mixer=self._mixer_part(index, layer.mixer, init_std),
                                 feed_forward=None if layer.mlp is None else self._feed_forward_part(layer.mlp, init_std), norm=norm)
                       for index, layer in enumerate(self.layers))
        order = [(index, None) for index in range(len(layers))]
        entries: tuple[PartSpec, ...] = ()
        if self.loop is not None:
            start, stop = self.loop.start, self.loop.stop
            one_pass = [(index, 0 if index == start else None) for index in range(start, stop)]
            order = order[:start] + one_pass * self.loop.times + order[stop:]
            entries = (PartSpec("linear_of_concat", {"hidden_size": self.width, "name": "loop.in", "init_std": init_std}),)
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            embedding=PartSpec("token_embedding", {"name": "embed", "init_std": 0.5, "norm": {"name": "embed.norm", "eps": self.norm_eps}}),
            layers=layers, schedule=tuple(LayerCall(layer=index, entry=entry) for index, entry in order), entries=entries,
            final_norm=PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "suffix": "", "name": "final.norm"}),
            head=PartSpec("linear_head", {"name": "head", "tied_to": None, "init_std": 0.25}),
            max_positions=MAX_POSITIONS, eos_token_ids=(),
        )
        spec.validate()
        return spec
