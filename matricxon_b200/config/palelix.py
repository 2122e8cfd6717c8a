"""Palelix configuration: a decoder whose mixer and feed-forward stand side by side on one norm, with lightning attention,
the gated delta rule, or softmax attention beside a delta rule that decays per channel, and a repeated run of layers.

``config.json`` holds ``architecture: "Palelix"``, ``vocab``, ``width``, ``norm.eps``, optionally ``loop`` (``start``, ``stop``,
``times``) and a list ``layers``; every entry gives ``type``, the mixer's sizes under ``mixer`` and its feed-forward under
``mlp`` (``kind: dense`` with ``ff``; ``kind: moe`` with ``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top`` and
optionally ``router.groups.count`` / ``router.groups.keep``; null for none).

Layer types:

* ``lightning`` (``heads``, ``dim``, ``vdim``, ``decay``): linear attention with a constant decay per head; q, k and v are the
  silu of their projections; one RMS norm over the concatenated heads, a sigmoid gate.
* ``delta`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``): the gated delta rule behind short convolutions with a decay
  per head, an RMS norm per head, a silu gate.
* ``parallel`` (``left``, ``left_scale``, ``right``, ``right_scale``): the sum of two scaled mixers of the same input. Left
  (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot``): causal grouped-query attention, q and k rotated. Right (the
  sizes of ``delta``): the delta rule with a decay per head and key channel, decay and sigmoid gate through low-rank maps.

A layer computes ``x += mixer(n(x)) + ff(n(x))``. The layers ``start .. stop - 1`` run ``times`` times with the same weights, a
cache and state per pass, ``loop.step[t]`` added to the stream before pass t.

Tensor names: ``embed``, ``head``, ``loop.step``, ``l<i>.norm1``, ``l<i>.mix.{q,k,v,g,o,norm}``, ``l<i>.mix.{q,k,v}.conv``,
``l<i>.mix.{a,b,A_log,dt_bias}``, ``l<i>.mix.left.{q,k,v,o}``, ``l<i>.mix.right.{q,k,v,b,A_log,dt_bias,a1,a2,g1,g2,norm,o}``,
``l<i>.mlp.{gate,up,down}``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.router``, ``final.norm`` (no ``.weight`` suffix). The
ranks of the low-rank maps are no keys of ``config.json``: they are read from the shapes of ``a1`` and ``g1``. This file is the
only place that knows those names and keys; the parts are generic.
"""

from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any

from matricxon_b200.config.base import ConfigError, ConfigReader
from matricxon_b200.parts.spec import (
    ClampedGluSpec,
    DeltaRuleSpec,
    GatedMlpSpec,
    LayerSpec,
    ModelSpec,
    NormedRotaryAttentionSpec,
    PairedRotarySpec,
    ParallelMixerSpec,
    RetentionSpec,
    RmsNormSpec,
    RoutedExpertsSpec,
    ScheduleEntry,
    StepVectorSpec,
)

# what the design fixes
DENSE_ACTIVATION = "silu"
EXPERT_SLOPE = 1.702
EXPERT_SHIFT = 1.0
UNIT_EPS = 1e-6
LAYER_TYPES = ("lightning", "delta", "parallel")
DEFAULT_RANK = 16            # of the low-rank maps where no tensors say otherwise (random weights)
# no key of config.json limits a sequence's length; this sizes the block tables of captured steps
# (longer sequences run uncaptured)
DEFAULT_MAX_POSITIONS = 32768


def _object(raw: Any, key: str, where: str) -> dict:
    value = raw.get(key) if isinstance(raw, dict) else None
    if not isinstance(value, dict):
        raise ConfigError(f"{where}: {key!r} must be an object")
    return value


def _heads(m: ConfigReader, where: str) -> tuple[int, int]:
    heads = m.integer("heads", minimum=1)
    kv_heads = m.integer("kv_heads", heads, minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    return heads, kv_heads


def _size(m: ConfigReader, key: str, where: str, what: str, default: int | None = None) -> int:
    size = m.integer(key, minimum=1) if default is None else m.integer(key, default, minimum=1)
    if size > 256:
        raise ConfigError(f"{where}: {key!r} of {size}: {what} above 256 have no kernel")
    return size


@dataclass(frozen=True)
class PalelixLightning:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "PalelixLightning":
        m = ConfigReader(mixer, where)
        heads, dim = m.integer("heads", minimum=1), _size(m, "dim", where, "key channels per head")
        decay = mixer.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or \
                any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
            raise ConfigError(f"{where}: 'decay' must list a number for each of the {heads} heads")
        return cls(heads=heads, dim=dim, vdim=m.integer("vdim", dim, minimum=1), decay=tuple(float(d) for d in decay))

    def to_dict(self) -> dict:
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}

    def spec(self, width: int, eps: float):
        return RetentionSpec(
            hidden_size=width, num_heads=self.heads, head_dim=self.dim, value_dim=self.vdim, decay=self.decay, key_scale=1.0,
            eps=eps, position=None, query_name="q", key_name="k", value_name="v", gate_name="g", output_name="o",
            activation="silu", norm="all", norm_name="norm", gate="sigmoid")


@dataclass(frozen=True)
class PalelixDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    per_channel: bool = False           # the decay's span; with it the low-rank maps and the sigmoid gate
    decay_rank: int = DEFAULT_RANK
    gate_rank: int = DEFAULT_RANK

    @classmethod
    def from_dict(cls, mixer: dict, where: str, per_channel: bool = False) -> "PalelixDelta":
        m = ConfigReader(mixer, where)
        heads, kv_heads = _heads(m, where)
        dim = _size(m, "dim", where, "key channels per head")
        conv = m.integer("conv", minimum=1)
        if conv > 16:
            raise ConfigError(f"{where}: 'conv' of {conv}: convolutions of more than 16 taps have no kernel")
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=m.integer("vdim", dim, minimum=1), conv=conv,
                   per_channel=per_channel)

    def to_dict(self) -> dict:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}

    def spec(self, width: int, eps: float):
        if self.per_channel:
            kind = {"decay": "channel", "gate": "sigmoid", "decay_names": ("a1", "a2"), "gate_names": ("g1", "g2"),
                    "decay_rank": self.decay_rank, "gate_rank": self.gate_rank}
        else:
            kind = {"decay": "head", "gate": "silu", "decay_names": ("a",), "gate_names": ("g",)}
        return DeltaRuleSpec(
            hidden_size=width, num_heads=self.heads, num_kv_heads=self.kv_heads, head_dim=self.dim, value_dim=self.vdim,
            taps=self.conv, eps=eps, query_scale=self.dim ** -0.5, query_name="q", key_name="k", value_name="v",
            beta_name="b", a_log_name="A_log", dt_bias_name="dt_bias", norm_name="norm", output_name="o",
            unit_eps=UNIT_EPS, **kind)


@dataclass(frozen=True)
class PalelixParallel:
    heads: int                    # left: softmax attention
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: tuple[int, float] | None           # dims, base
    left_scale: float
    right: PalelixDelta
    right_scale: float

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "PalelixParallel":
        m = ConfigReader(mixer, where)
        left, here = _object(mixer, "left", where), where + ".left"
        lr = ConfigReader(left, here)
        heads, kv_heads = _heads(lr, here)
        dim = _size(lr, "dim", here, "head sizes")
        vdim = _size(lr, "vdim", here, "head sizes", dim)
        rot = None
        if left.get("rot") is not None:
            r = ConfigReader(_object(left, "rot", here), here + ".rot")
            dims, base = r.integer("dims", minimum=0), r.number("base", positive=True)
            if dims % 2 or dims > dim:
                raise ConfigError(f"{here}.rot: 'dims' must be even and at most dim ({dim}), got {dims}")
            rot = (dims, base)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=lr.number("scale"), rot=rot,
                   left_scale=m.number("left_scale", 1.0), right_scale=m.number("right_scale", 1.0),
                   right=PalelixDelta.from_dict(_object(mixer, "right", where), where + ".right", per_channel=True))

    def to_dict(self) -> dict:
        left: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                                "vdim": self.vdim}
        if self.rot is not None:
            left["rot"] = {"base": self.rot[1], "dims": self.rot[0]}
        return {"left": left, "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}

    def spec(self, width: int, eps: float):
        position = PairedRotarySpec(rotary_dim=self.rot[0], theta=self.rot[1], pairing="half") if self.rot is not None else None
        left = NormedRotaryAttentionSpec(
            hidden_size=width, num_heads=self.heads, num_kv_heads=self.kv_heads, head_dim=self.dim, value_dim=self.vdim,
            scale=self.scale, eps=eps, position=position, query_name="q", key_name="k", value_name="v", output_name="o")
        return ParallelMixerSpec(hidden_size=width, branches=((left, self.left_scale, "left."),
                                                              (self.right.spec(width, eps), self.right_scale, "right.")))


@dataclass(frozen=True)
class PalelixFeedForward:
    kind: str                     # "dense" | "moe"
    ff: int                       # width of the dense feed-forward or of one expert
    limit: float | None = None
    experts: int = 0
    top: int = 0
    groups: tuple[int, int] | None = None       # count, keep

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "PalelixFeedForward":
        r = ConfigReader(raw, where)
        kind = r.string("kind")
        if kind == "dense":
            return cls(kind=kind, ff=r.integer("ff", minimum=1))
        if kind != "moe":
            raise ConfigError(f"{where}: unknown feed-forward kind {kind!r}; Palelix has 'dense' and 'moe'")
        raw_router, here = _object(raw, "router", where), where + ".router"
        router = ConfigReader(raw_router, here)
        experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
        if top > experts:
            raise ConfigError(f"{here}: 'top' ({top}) exceeds the {experts} experts")
        groups = None
        if raw_router.get("groups") is not None:
            g = ConfigReader(_object(raw_router, "groups", here), here + ".groups")
            count, keep = g.integer("count", minimum=1), g.integer("keep", minimum=1)
            if experts % count or keep > count or keep * (experts // count) < top:
                raise ConfigError(f"{here}.groups: {keep} of {count} equal groups of {experts} experts cannot supply {top}")
            groups = (count, keep)
        expert = ConfigReader(_object(raw, "expert", where), where + ".expert")
        limit = expert.number("limit", positive=True) if expert.raw.get("limit") is not None else None
        return cls(kind=kind, ff=expert.integer("ff", minimum=1), limit=limit, experts=experts, top=top, groups=groups)

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        expert: dict[str, Any] = {"ff": self.ff}
        if self.limit is not None:
            expert["limit"] = self.limit
        router: dict[str, Any] = {"experts": self.experts, "top": self.top}
        if self.groups is not None:
            router["groups"] = {"count": self.groups[0], "keep": self.groups[1]}
        return {"expert": expert, "kind": "moe", "router": router}

    def spec(self, width: int):
        if self.kind == "dense":
            return GatedMlpSpec(hidden_size=width, intermediate_size=self.ff, activation=DENSE_ACTIVATION, gate_name="gate",
                                up_name="up", down_name="down")
        expert = ClampedGluSpec(hidden_size=width, intermediate_size=self.ff, limit=self.limit, gate_name="gate",
                                up_name="up", down_name="down", slope=EXPERT_SLOPE, shift=EXPERT_SHIFT)
        count, keep = self.groups or (1, 1)
        return RoutedExpertsSpec(
            hidden_size=width, num_experts=self.experts, top=self.top, num_groups=count, groups_kept=keep, route_scale=1.0,
            expert=expert, router_name="router", expert_format="e{index}.", group_best=1, score="softmax")


@dataclass(frozen=True)
class PalelixLayer:
    type: str
    mixer: Any
    feed_forward: PalelixFeedForward | None = None

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "PalelixLayer":
        kind = ConfigReader(raw, where).string("type")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}: unknown layer type {kind!r}; Palelix has {list(LAYER_TYPES)}")
        mixer_class = {"lightning": PalelixLightning, "delta": PalelixDelta, "parallel": PalelixParallel}[kind]
        mixer = mixer_class.from_dict(_object(raw, "mixer", where), where + ".mixer")
        feed_forward = None
        if raw.get("mlp") is not None:
            feed_forward = PalelixFeedForward.from_dict(raw["mlp"], where + ".mlp")
        return cls(type=kind, mixer=mixer, feed_forward=feed_forward)

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": self.feed_forward.to_dict() if self.feed_forward else None,
                "type": self.type}


@dataclass(frozen=True)
class PalelixConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[PalelixLayer, ...]
    loop: tuple[int, int, int] | None = None        # start, stop, times
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Palelix"
    model_type = "palelix"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str = "config.json") -> "PalelixConfig":
        r = ConfigReader(raw, where)
        eps = ConfigReader(_object(raw, "norm", where), where + ".norm").number("eps", positive=True)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        parsed = tuple(PalelixLayer.from_dict(layer, f"{where}.layers[{i}]") for i, layer in enumerate(layers))
        loop = None
        if raw.get("loop") is not None:
            here = ConfigReader(_object(raw, "loop", where), where + ".loop")
            loop = (here.integer("start", minimum=0), here.integer("stop", minimum=1), here.integer("times", minimum=1))
            if not loop[0] < loop[1] <= len(parsed):
                raise ConfigError(f"{where}.loop: layers {loop[0]} .. {loop[1] - 1} of {len(parsed)} cannot be repeated")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), eps=eps, layers=parsed, loop=loop,
                   max_positions=r.integer("max_positions", DEFAULT_MAX_POSITIONS, minimum=1))

    def with_tensor_shapes(self, shape_of) -> "PalelixConfig":
        """Takes the ranks of the low-rank maps from the tensors: ``shape_of(name)`` gives a tensor's shape or None."""
        layers = []
        for index, layer in enumerate(self.layers):
            if layer.type == "parallel":
                ranks = {}
                for field, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
                    shape = shape_of(f"l{index}.mix.right.{name}")
                    if shape is not None:
                        ranks[field] = int(shape[0])
                layer = replace(layer, mixer=replace(layer.mixer, right=replace(layer.mixer.right, **ranks)))
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "layers": [layer.to_dict() for layer in self.layers],
                               "norm": {"eps": self.eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ------------------------------------------------------------------ description
    def schedule(self) -> tuple[ScheduleEntry, ...]:
        start, stop, times = self.loop or (0, 0, 0)
        entries = [ScheduleEntry(layer=i) for i in range(start)]
        for t in range(times):
            entries += [ScheduleEntry(layer=i, pass_index=t if i == start else None) for i in range(start, stop)]
        return tuple(entries + [ScheduleEntry(layer=i) for i in range(stop, len(self.layers))])

    def model_spec(self) -> ModelSpec:
        norm = RmsNormSpec(size=self.width, eps=self.eps, weight_name="")
        layers = []
        for layer in self.layers:
            feed_forward = layer.feed_forward.spec(self.width) if layer.feed_forward is not None else None
            layers.append(LayerSpec(
                mixer=layer.mixer.spec(self.width, self.eps), feed_forward=feed_forward, mixer_norm=norm, ffn_norm=None,
                mixer_name="mix.", feed_forward_name="mlp.", mixer_norm_name="norm1", ffn_norm_name="",
                block="pre_norm_parallel", part_separator=""))
        return ModelSpec(
            hidden_size=self.width, vocab_size=self.vocab, layers=tuple(layers), schedule=self.schedule(), final_norm=norm,
            tie_word_embeddings=False, max_position_embeddings=self.max_positions, embedding_name="embed",
            layer_prefix="l", final_norm_name="final.norm", head_name="head", weight_suffix="",
            layer_prefix_format="{prefix}{index}.", final_norm_prefix="final.norm",
            pass_input=StepVectorSpec(hidden_size=self.width, passes=self.loop[2], step_name="loop.step")
            if self.loop is not None else None)
