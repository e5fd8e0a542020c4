"""Neburax as data: a decoder whose sub-layers read the residual stream itself and whose outputs are normed before they join
it; the mixers are the state-space recurrence with a scalar decay per head, and a weighted pair of chunked attention and a
gated linear recurrence; the feed-forwards square a ReLU or are a mixture with experts that give back their input beside
a shared expert.  A layer may run with an earlier layer's tensors.

``config.json`` (every size, and every constant that can differ between models of the design, is read from it):

* ``architecture``: "Neburax"; ``vocab``, ``width``; ``norm: {eps}``;
* ``layers``: a list; entry i has ``type`` (``mamba2`` or ``parallel``), ``mixer`` (its sizes and constants) and ``mlp``
  (``{kind: dense, ff}``, ``{kind: moe, router: {experts, top, identity}, expert: {ff}, shared: {ff}}``, or null); its tensors
  start with ``l<i>.``, or, with ``weights_of: j``, are those of layer j, whose entry is the same otherwise; caches and
  states are always the layer's own.

The network: ``x = embed[token]``; per layer ``x += rms(mixer(x)) * norm1`` and ``x += rms(ff(x)) * norm2``;
``logits = embed (rms(x) * final.norm)``.

* ``mamba2`` (``parts/recurrent.py``, ``state_space``): ``heads, vdim, state, groups, conv, norm_groups``.
* ``parallel`` (``parts/recurrent.py``, ``side_by_side``): ``left_scale * left + right_scale * right``; ``left`` — ``heads,
  kv_heads, dim, vdim, scale, mask: {size}`` — attention inside chunks, queries and keys normed as whole rows, no rotation;
  ``right`` — ``width, blocks, conv`` — ``gated_linear``.
* mixture (``parts/feed_forward.py``): choice by softmax score plus correction, weights the scores over their sum; the last
  ``identity`` of the router's experts + identity outputs have no matrices.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, take
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec

ARCHITECTURE = "Neburax"
# The design has no table of positions and hence no largest position of its own; this bounds what one request may hold.
MAX_POSITIONS = 1 << 17
MIXER_TYPES = ("mamba2", "parallel")


def _obj(raw: Mapping[str, Any], key: str, where: str, optional: bool = False) -> Optional[Mapping[str, Any]]:
    value = raw.get(key)
    if value is None:
        if optional:
            return None
        raise ConfigError(f"invalid model config: {where}'{key}' is missing")
    if not isinstance(value, dict):
        raise ConfigError(f"invalid model config: {where}'{key}' must be an object")
    return value


def _positive(raw: Mapping[str, Any], key: str, where: str) -> int:
    try:
        v = take(raw, key, int)
    except ConfigError as exc:
        raise ConfigError(f"{exc} (in {where})") from None
    if v <= 0:
        raise ConfigError(f"invalid model config: {where}'{key}' must be positive, got {v}")
    return v


def _number(raw: Mapping[str, Any], key: str, where: str) -> float:
    try:
        return float(take(raw, key, float))
    except ConfigError as exc:
        raise ConfigError(f"{exc} (in {where})") from None


def _multiple(what: str, value: int, of: str, divisor: int, where: str) -> None:
    if value % divisor:
        raise ConfigError(f"invalid model config: {where}{what}={value} is not a multiple of {of}={divisor}")


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "StateSpaceConfig":
        out = cls(*(_positive(raw, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        _multiple("heads", out.heads, "groups", out.groups, where)
        _multiple("heads * vdim", out.heads * out.vdim, "norm_groups", out.norm_groups, where)
        return out

    def to_dict(self) -> dict:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}

    def spec(self, eps: float) -> PartSpec:
        return PartSpec("state_space", name="mix", num_heads=self.heads, vdim=self.vdim, state_size=self.state, groups=self.groups,
                        taps=self.conv, norm_groups=self.norm_groups, eps=eps)


@dataclass(frozen=True)
class LeftConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]          # None: every earlier key is seen

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "LeftConfig":
        if raw.get("rot") is not None:
            raise ConfigError(f"unsupported option: {where}rot (this mixer rotates nothing)")
        mask = _obj(raw, "mask", where, optional=True)
        out = cls(*(_positive(raw, k, where) for k in ("heads", "kv_heads", "dim", "vdim")), scale=_number(raw, "scale", where),
                  chunk=_positive(mask, "size", where + "mask.") if mask else None)
        _multiple("heads", out.heads, "kv_heads", out.kv_heads, where)
        return out

    def to_dict(self) -> dict:
        out: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        return out

    def spec(self, eps: float) -> PartSpec:
        return PartSpec("window_attention", num_heads=self.heads, num_kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                        scale=self.scale, window=self.chunk, chunked=self.chunk is not None, qk_norm="row", eps=eps)


@dataclass(frozen=True)
class RightConfig:
    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "RightConfig":
        out = cls(*(_positive(raw, k, where) for k in ("width", "blocks", "conv")))
        _multiple("width", out.width, "blocks", out.blocks, where)
        return out

    def to_dict(self) -> dict:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}

    def spec(self) -> PartSpec:
        return PartSpec("gated_linear", width=self.width, blocks=self.blocks, taps=self.conv)


@dataclass(frozen=True)
class ParallelConfig:
    left: LeftConfig
    right: RightConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "ParallelConfig":
        return cls(LeftConfig.from_dict(_obj(raw, "left", where), where + "left."), RightConfig.from_dict(_obj(raw, "right", where), where + "right."),
                   _number(raw, "left_scale", where), _number(raw, "right_scale", where))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}

    def spec(self, eps: float) -> PartSpec:
        return PartSpec("side_by_side", name="mix", left=self.left.spec(eps), right=self.right.spec(), scales=(self.left_scale, self.right_scale))


_MIXER_CONFIGS = {"mamba2": StateSpaceConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                   # "dense" or "moe"
    ff: int                     # dense: its size; moe: an expert's size
    experts: int = 0
    top: int = 0
    identity: int = 0           # experts that give back their input
    shared: int = 0             # the shared expert's size; 0: none

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "FeedForwardConfig":
        kind = take(raw, "kind", str)
        if kind == "dense":
            return cls("dense", _positive(raw, "ff", where))
        if kind == "moe":
            router, expert = _obj(raw, "router", where), _obj(raw, "expert", where)
            shared = _obj(raw, "shared", where, optional=True)
            identity = take(router, "identity", int) if router.get("identity") is not None else 0
            out = cls("moe", _positive(expert, "ff", where + "expert."), _positive(router, "experts", where + "router."),
                      _positive(router, "top", where + "router."), identity, _positive(shared, "ff", where + "shared.") if shared else 0)
            if out.identity < 0:
                raise ConfigError(f"invalid model config: {where}router.identity must not be negative")
            if out.top > out.experts + out.identity:
                raise ConfigError(f"invalid model config: {where}router.top={out.top} exceeds the {out.experts + out.identity} experts")
            return out
        raise ConfigError(f"unsupported option: {where}kind={kind!r} (dense or moe)")

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        out: dict = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top, "identity": self.identity}}
        if self.shared:
            out["shared"] = {"ff": self.shared}
        return out

    def spec(self) -> PartSpec:
        if self.kind == "dense":
            return PartSpec("relu2", name="mlp", intermediate_size=self.ff, names=("up", "down"), bias=True)
        return PartSpec("moe_routed", name="mlp", experts=self.experts, top=self.top, intermediate_size=self.ff, activation="silu",
                        score="softmax", correction_name="correction", renorm=True, identity=self.identity, router_name="router",
                        expert_names=("e{}.gate", "e{}.up", "e{}.down"), shared_size=self.shared,
                        shared_names=("shared.gate", "shared.up", "shared.down"))


@dataclass(frozen=True)
class NeburaxLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[FeedForwardConfig]
    weights_of: Optional[int] = None


@dataclass(frozen=True)
class NeburaxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[NeburaxLayerConfig, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def max_model_len(self) -> int:
        return MAX_POSITIONS

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i runs with."""
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
        return i

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "NeburaxConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("invalid model config: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"invalid model config: layers[{i}] must be an object")
            kind = take(entry, "type", str)
            if kind not in _MIXER_CONFIGS:
                raise ConfigError(f"unsupported option: {where}type={kind!r} (one of {', '.join(MIXER_TYPES)})")
            source = entry.get("weights_of")
            if source is not None and (not isinstance(source, int) or isinstance(source, bool) or not 0 <= source < i):
                raise ConfigError(f"invalid model config: {where}weights_of must name an earlier layer, got {source!r}")
            mlp = _obj(entry, "mlp", where, optional=True)
            layer = NeburaxLayerConfig(kind, _MIXER_CONFIGS[kind].from_dict(_obj(entry, "mixer", where), where + "mixer."),
                                       FeedForwardConfig.from_dict(mlp, where + "mlp.") if mlp else None, source)
            if source is not None and (layers[source].type, layers[source].mixer, layers[source].mlp) != (kind, layer.mixer, layer.mlp):
                raise ConfigError(f"invalid model config: layers[{i}] differs from layer {source}, whose weights it uses")
            layers.append(layer)
        eps = _number(_obj(raw, "norm", ""), "eps", "norm.")
        if not eps > 0:
            raise ConfigError("invalid model config: norm.eps must be positive")
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else (eos,) if isinstance(eos, int) else tuple(eos)
        return cls(vocab=_positive(raw, "vocab", ""), width=_positive(raw, "width", ""), norm_eps=eps, layers=tuple(layers), eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        layers = []
        for layer in self.layers:
            entry: dict = {"type": layer.type, "mixer": layer.mixer.to_dict(), "mlp": layer.mlp.to_dict() if layer.mlp else None}
            if layer.weights_of is not None:
                entry["weights_of"] = layer.weights_of
            layers.append(entry)
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out


def neburax_spec(cfg: NeburaxConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", eps=cfg.norm_eps, weight_suffix="")
    block = PartSpec("postnorm", norm_names=("norm1", "norm2"))
    # a layer with another's tensors is that layer run again: the model's layers are those with tensors of their own, and
    # every run has a cache and a state of its own
    place: Dict[int, int] = {}
    layers = []
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is None:
            place[i] = len(layers)
            layers.append(LayerSpec(prefix=f"l{i}", block=block, mixer=layer.mixer.spec(cfg.norm_eps),
                                    feed_forward=layer.mlp.spec() if layer.mlp else PartSpec("none", name="mlp"), norm=norm))
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS, layers=tuple(layers), final_norm=norm,
                     embedding_name="embed", final_norm_prefix="final.norm", lm_head_name=None,
                     order=tuple(place[cfg.owner(i)] for i in range(len(cfg.layers))), eos_token_ids=tuple(cfg.eos_token_ids))


register_architecture(ARCHITECTURE, NeburaxConfig.from_dict, neburax_spec, replace=True)
