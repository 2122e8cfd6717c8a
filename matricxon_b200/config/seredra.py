"""Seredra configuration: a pre-norm decoder whose layers each pick attention behind short convolutions, capped attention
beside a selective recurrence, or retention, with dense or routed feed-forwards.

``config.json`` holds ``architecture: "Seredra"``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` and a list
``layers``; every entry gives ``type``, the mixer's sizes under ``mixer`` and its feed-forward under ``mlp`` (``kind: dense``
with ``ff``; ``kind: moe`` with ``expert.ff`` and ``router.experts`` / ``router.top``; null for a layer that has only the
mixer sublayer).

Layer types:

* ``attention`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``, ``scale``, ``q_temp.coef`` / ``q_temp.every``, optionally
  ``kv_from``): biased projections, each through a causal convolution of ``conv`` taps; q and k RMS-normalised over the whole
  projection; q times ``1 + coef ln(floor((p + 1) / every) + 1)``; scores ``q . k * scale - r1_h ln(1 + r2_h (i - j))``. A layer
  with ``kv_from: j`` has queries only and attends over layer j's keys and values.
* ``parallel`` (``left``, ``left_scale``, ``right``, ``right_scale``): the sum of two scaled mixers of the same input. Left
  (``heads``, ``kv_heads``, ``dim``, ``scale``, ``softcap``, ``rot``): grouped queries whose values are the keys as projected; q
  and k RMS-normalised per head with a weight, then rotated (``rot.scaling``: ``factor``, ``original``, ``fast``, ``slow``
  stretch the frequencies), scores capped. Right (``inner``, ``state``, ``dt_rank``, ``conv``): a selective recurrence.
* ``retention`` (``heads``, ``dim``, ``vdim``, ``decay``, ``rot``): linear attention with a constant decay per head, q and k
  rotated, k times ``dim^(-1/2)``, every head normalised without a weight and gated by ``silu``.

A layer computes ``x += mixer(norm1(x))``, ``x += ff(norm2(x))`` with RMS norms whose weight is one number. The dense
feed-forward is ``down(max(up h, 0)^2)``; an expert is ``down(silu(gate h) * up h)`` on its input times the router's sigmoid
score, which is not normalised over the chosen experts.

Tensor names: ``embed``, ``head``, ``l<i>.norm1|norm2``, ``l<i>.mix.{q,k,v}{,.b,.conv}``, ``l<i>.mix.{q,k}.norm``,
``l<i>.mix.{r1,r2,o,o.b}``, ``l<i>.mix.left.{q,k,q.norm,k.norm,o}``, ``l<i>.mix.right.{in,conv,conv.b,x,dt,dt.b,A_log,D,o}``,
``l<i>.mix.{q,k,v,g,o}``, ``l<i>.mlp.{up,down}``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.router``, ``final.norm`` (no
``.weight`` suffix). This file is the only place that knows those names and keys; the parts are generic.
"""

from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any

from matricxon_b200.config.base import ConfigError, ConfigReader
from matricxon_b200.parts.spec import (
    ConvAttentionSpec,
    GatedMlpSpec,
    InterpolatedRotarySpec,
    LayerSpec,
    MlpSpec,
    ModelSpec,
    NormedRotaryAttentionSpec,
    PairedRotarySpec,
    ParallelMixerSpec,
    RetentionSpec,
    RmsNormSpec,
    RoutedExpertsSpec,
    ScheduleEntry,
    SelectiveScanSpec,
)

# what the design fixes
DENSE_ACTIVATION = "relu_squared"
EXPERT_ACTIVATION = "silu"
LAYER_TYPES = ("attention", "parallel", "retention")
# no key of config.json limits a sequence's length; this sizes the block tables of captured steps
# (longer sequences run uncaptured)
DEFAULT_MAX_POSITIONS = 32768


def _object(raw: Any, key: str, where: str) -> dict:
    value = raw.get(key) if isinstance(raw, dict) else None
    if not isinstance(value, dict):
        raise ConfigError(f"{where}: {key!r} must be an object")
    return value


@dataclass(frozen=True)
class SeredraRotation:
    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None      # factor, original, fast, slow

    @classmethod
    def from_mixer(cls, mixer: dict, dim: int, where: str, scalable: bool) -> "SeredraRotation | None":
        """The mixer's ``rot``; None where it has none (nothing is rotated)."""
        if mixer.get("rot") is None:
            return None
        raw = _object(mixer, "rot", where)
        r = ConfigReader(raw, where + ".rot")
        dims, base = r.integer("dims", minimum=0), r.number("base", positive=True)
        if dims % 2 or dims > dim:
            raise ConfigError(f"{where}.rot: 'dims' must be even and at most dim ({dim}), got {dims}")
        scaling = None
        if raw.get("scaling") is not None:
            if not scalable:
                raise ConfigError(f"{where}.rot: 'scaling' belongs to the parallel mixer's left side")
            s = ConfigReader(_object(raw, "scaling", where + ".rot"), where + ".rot.scaling")
            scaling = tuple(s.number(key, positive=True) for key in ("factor", "original", "fast", "slow"))
        return cls(dims=dims, base=base, scaling=scaling)

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return out

    def spec(self):
        if self.scaling is None:
            return PairedRotarySpec(rotary_dim=self.dims, theta=self.base, pairing="half")
        factor, original, fast, slow = self.scaling
        return InterpolatedRotarySpec(rotary_dim=self.dims, theta=self.base, factor=factor, original=original, fast=fast,
                                      slow=slow)


def _heads(m: ConfigReader, where: str) -> tuple[int, int]:
    heads = m.integer("heads", minimum=1)
    kv_heads = m.integer("kv_heads", heads, minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    return heads, kv_heads


def _head_size(m: ConfigReader, key: str, where: str, default: Any = None) -> int:
    size = m.integer(key, minimum=1) if default is None else m.integer(key, default, minimum=1)
    if size > 256:
        raise ConfigError(f"{where}: {key!r} of {size}: head sizes above 256 have no attention kernel")
    return size


@dataclass(frozen=True)
class SeredraAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int | None
    scale: float
    temperature: tuple[float, float] | None
    kv_from: int | None = None

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "SeredraAttention":
        m = ConfigReader(mixer, where)
        heads, kv_heads = _heads(m, where)
        dim = _head_size(m, "dim", where)
        temperature = None
        if mixer.get("q_temp") is not None:
            t = ConfigReader(_object(mixer, "q_temp", where), where + ".q_temp")
            temperature = (t.number("coef"), t.number("every", positive=True))
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_head_size(m, "vdim", where, dim),
                   conv=m.optional_integer("conv", minimum=1), scale=m.number("scale", positive=True),
                   temperature=temperature, kv_from=m.optional_integer("kv_from", minimum=0))

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                               "vdim": self.vdim}
        if self.conv is not None:
            out["conv"] = self.conv
        if self.temperature is not None:
            out["q_temp"] = {"coef": self.temperature[0], "every": self.temperature[1]}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out

    def spec(self, width: int, eps: float):
        return ConvAttentionSpec(
            hidden_size=width, num_heads=self.heads, num_kv_heads=self.kv_heads, head_dim=self.dim, value_dim=self.vdim,
            taps=self.conv, scale=self.scale, eps=eps, temperature=self.temperature, bias=True, query_name="q",
            key_name="k", value_name="v", output_name="o", query_norm_name="q.norm", key_norm_name="k.norm",
            distance_names=("r1", "r2"), shares_kv=self.kv_from is not None)


@dataclass(frozen=True)
class SeredraParallel:
    heads: int                    # left: capped attention whose values are its keys
    kv_heads: int
    dim: int
    scale: float
    softcap: float | None
    rot: SeredraRotation | None
    left_scale: float
    inner: int                    # right: selective recurrence
    state: int
    dt_rank: int
    conv: int
    right_scale: float

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "SeredraParallel":
        m = ConfigReader(mixer, where)
        left = _object(mixer, "left", where)
        here = where + ".left"
        lr = ConfigReader(left, here)
        heads, kv_heads = _heads(lr, here)
        dim = _head_size(lr, "dim", here)
        if lr.integer("vdim", dim, minimum=1) != dim:
            raise ConfigError(f"{here}: the values are the keys, so 'vdim' must equal dim ({dim}), got {left['vdim']}")
        rr = ConfigReader(_object(mixer, "right", where), where + ".right")
        state = rr.integer("state", minimum=1)
        if state > 128:
            raise ConfigError(f"{where}.right: 'state' of {state}: more than 128 states per channel have no kernel")
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, scale=lr.number("scale", positive=True),
                   softcap=lr.number("softcap", positive=True) if left.get("softcap") is not None else None,
                   rot=SeredraRotation.from_mixer(left, dim, here, scalable=True), left_scale=m.number("left_scale", 1.0),
                   inner=rr.integer("inner", minimum=1), state=state, dt_rank=rr.integer("dt_rank", minimum=1),
                   conv=rr.integer("conv", minimum=1), right_scale=m.number("right_scale", 1.0))

    def to_dict(self) -> dict:
        left: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                                "vdim": self.dim}
        if self.softcap is not None:
            left["softcap"] = self.softcap
        if self.rot is not None:
            left["rot"] = self.rot.to_dict()
        right = {"conv": self.conv, "dt_rank": self.dt_rank, "inner": self.inner, "state": self.state}
        return {"left": left, "left_scale": self.left_scale, "right": right, "right_scale": self.right_scale}

    def spec(self, width: int, eps: float):
        left = NormedRotaryAttentionSpec(
            hidden_size=width, num_heads=self.heads, num_kv_heads=self.kv_heads, head_dim=self.dim, value_dim=self.dim,
            scale=self.scale, eps=eps, position=self.rot.spec() if self.rot is not None else None, query_name="q",
            key_name="k", value_name=None, output_name="o", softcap=self.softcap, query_norm_name="q.norm",
            key_norm_name="k.norm")
        right = SelectiveScanSpec(
            hidden_size=width, channels=self.inner, states=self.state, dt_rank=self.dt_rank, taps=self.conv,
            input_name="in", conv_name="conv", low_name="x", dt_name="dt", a_log_name="A_log", d_name="D",
            output_name="o")
        return ParallelMixerSpec(hidden_size=width, branches=((left, self.left_scale, "left."),
                                                              (right, self.right_scale, "right.")))


@dataclass(frozen=True)
class SeredraRetention:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: SeredraRotation | None

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "SeredraRetention":
        m = ConfigReader(mixer, where)
        heads, dim = m.integer("heads", minimum=1), m.integer("dim", minimum=1)
        if dim > 256:
            raise ConfigError(f"{where}: 'dim' of {dim}: more than 256 key channels per head have no kernel")
        decay = mixer.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or \
                any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
            raise ConfigError(f"{where}: 'decay' must list a number for each of the {heads} heads")
        return cls(heads=heads, dim=dim, vdim=m.integer("vdim", dim, minimum=1), decay=tuple(float(d) for d in decay),
                   rot=SeredraRotation.from_mixer(mixer, dim, where, scalable=False))

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        return out

    def spec(self, width: int, eps: float):
        return RetentionSpec(
            hidden_size=width, num_heads=self.heads, head_dim=self.dim, value_dim=self.vdim, decay=self.decay,
            key_scale=self.dim ** -0.5, eps=eps, position=self.rot.spec() if self.rot is not None else None,
            query_name="q", key_name="k", value_name="v", gate_name="g", output_name="o")


@dataclass(frozen=True)
class SeredraFeedForward:
    kind: str                     # "dense" | "moe"
    ff: int                       # width of the dense feed-forward or of one expert
    experts: int = 0
    top: int = 0

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "SeredraFeedForward":
        r = ConfigReader(raw, where)
        kind = r.string("kind")
        if kind == "dense":
            return cls(kind=kind, ff=r.integer("ff", minimum=1))
        if kind != "moe":
            raise ConfigError(f"{where}: unknown feed-forward kind {kind!r}; Seredra has 'dense' and 'moe'")
        router = ConfigReader(_object(raw, "router", where), where + ".router")
        experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
        if top > experts:
            raise ConfigError(f"{where}.router: 'top' ({top}) exceeds the {experts} experts")
        ff = ConfigReader(_object(raw, "expert", where), where + ".expert").integer("ff", minimum=1)
        return cls(kind=kind, ff=ff, experts=experts, top=top)

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        return {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}

    def spec(self, width: int):
        if self.kind == "dense":
            return MlpSpec(hidden_size=width, intermediate_size=self.ff, bias=False, activation=DENSE_ACTIVATION,
                           up_name="up", down_name="down", weight_suffix="")
        expert = GatedMlpSpec(hidden_size=width, intermediate_size=self.ff, activation=EXPERT_ACTIVATION,
                              gate_name="gate", up_name="up", down_name="down")
        return RoutedExpertsSpec(
            hidden_size=width, num_experts=self.experts, top=self.top, num_groups=1, groups_kept=1, route_scale=1.0,
            expert=expert, router_name="router", expert_format="e{index}.", score="sigmoid", normalize=False,
            weight_on="input")


_MIXERS = {"attention": SeredraAttention, "parallel": SeredraParallel, "retention": SeredraRetention}


@dataclass(frozen=True)
class SeredraLayer:
    type: str
    mixer: Any
    feed_forward: SeredraFeedForward | None = None

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "SeredraLayer":
        kind = ConfigReader(raw, where).string("type")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}: unknown layer type {kind!r}; Seredra has {list(LAYER_TYPES)}")
        mixer = _MIXERS[kind].from_dict(_object(raw, "mixer", where), where + ".mixer")
        feed_forward = None
        if raw.get("mlp") is not None:
            feed_forward = SeredraFeedForward.from_dict(raw["mlp"], where + ".mlp")
        return cls(type=kind, mixer=mixer, feed_forward=feed_forward)

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": self.feed_forward.to_dict() if self.feed_forward else None,
                "type": self.type}


@dataclass(frozen=True)
class SeredraConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple[SeredraLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    # tensors a model folder holds although the model does not use them (the second norm of a layer without a
    # feed-forward): (name, shape), found by ``with_tensor_shapes``; expected at the weight check and never fetched
    unused_tensors: tuple[tuple[str, tuple[int, ...]], ...] = ()

    architecture = "Seredra"
    model_type = "seredra"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str = "config.json") -> "SeredraConfig":
        r = ConfigReader(raw, where)
        eps = ConfigReader(_object(raw, "norm", where), where + ".norm").number("eps", positive=True)
        scale = 1.0                                        # no 'embedding': the table is taken as it is
        if raw.get("embedding") is not None:
            scale = ConfigReader(_object(raw, "embedding", where), where + ".embedding").number("scale", 1.0)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        parsed = tuple(SeredraLayer.from_dict(layer, f"{where}.layers[{i}]") for i, layer in enumerate(layers))
        for index, layer in enumerate(parsed):
            source = layer.mixer.kv_from if layer.type == "attention" else None
            if source is None:
                continue
            here = f"{where}.layers[{index}].mixer"
            if source >= index or parsed[source].type != "attention" or parsed[source].mixer.kv_from is not None:
                raise ConfigError(f"{here}: 'kv_from' must name an earlier attention layer with keys and values of its "
                                  f"own, got {source}")
            theirs = parsed[source].mixer
            if (theirs.kv_heads, theirs.dim, theirs.vdim) != (layer.mixer.kv_heads, layer.mixer.dim, layer.mixer.vdim):
                raise ConfigError(f"{here}: 'kv_from' names layer {source}, whose key and value heads differ in number or "
                                  "size")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), eps=eps, embedding_scale=scale,
                   layers=parsed, max_positions=r.integer("max_positions", DEFAULT_MAX_POSITIONS, minimum=1))

    def with_tensor_shapes(self, shape_of) -> "SeredraConfig":
        """Notes the tensors that a model folder holds unused: ``shape_of(name)`` gives a tensor's shape or None."""
        unused = []
        for index, layer in enumerate(self.layers):
            if layer.feed_forward is None:
                shape = shape_of(f"l{index}.norm2")
                if shape is not None:
                    unused.append((f"l{index}.norm2", tuple(int(extent) for extent in shape)))
        return replace(self, unused_tensors=tuple(unused))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
                               "layers": [layer.to_dict() for layer in self.layers], "norm": {"eps": self.eps},
                               "vocab": self.vocab, "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ------------------------------------------------------------------ description
    def schedule(self) -> tuple[ScheduleEntry, ...]:
        return tuple(ScheduleEntry(layer=i, cache_of=layer.mixer.kv_from if layer.type == "attention" else None)
                     for i, layer in enumerate(self.layers))

    def model_spec(self) -> ModelSpec:
        norm = RmsNormSpec(size=self.width, eps=self.eps, weight_name="", scalar=True)
        layers = []
        for layer in self.layers:
            feed_forward = layer.feed_forward.spec(self.width) if layer.feed_forward is not None else None
            layers.append(LayerSpec(
                mixer=layer.mixer.spec(self.width, self.eps), feed_forward=feed_forward, mixer_norm=norm,
                ffn_norm=norm if feed_forward is not None else None, mixer_name="mix.", feed_forward_name="mlp.",
                mixer_norm_name="norm1", ffn_norm_name="norm2", block="pre_norm_sequential", part_separator=""))
        return ModelSpec(
            hidden_size=self.width, vocab_size=self.vocab, layers=tuple(layers), schedule=self.schedule(), final_norm=norm,
            tie_word_embeddings=False, max_position_embeddings=self.max_positions, embedding_name="embed",
            layer_prefix="l", final_norm_name="final.norm", head_name="head", embedding_scale=self.embedding_scale,
            weight_suffix="", layer_prefix_format="{prefix}{index}.", final_norm_prefix="final.norm",
            extra={"unused_tensors": self.unused_tensors})
