"""Nugolorn as data: a decoder whose layers have ONE norm, read by a mixer and a feed-forward whose outputs join the residual
together, times a constant; the mixers are attention with sigmoid weights behind short convolutions (some layers reading the
keys and values an earlier one cached), a pair of log-biased attention and a delta rule with a decay per channel, and
RWKV-style time mixing; the feed-forwards are gated or a mixture with experts that give back their input.

``config.json`` (every size, and every constant that can differ between models of the design, is read from it; the inner
sizes of the low-rank products are the checkpoint's):

* ``architecture``: "Nugolorn"; ``vocab``, ``width``; ``norm: {eps, groups}``; ``residual_mult``; ``logit_scale``;
* ``layers``: a list; entry i has ``type`` (``attention``, ``parallel`` or ``wkv``), ``mixer`` (its sizes and constants) and
  ``mlp`` (``{kind: dense, ff}``, ``{kind: moe, router: {experts, top, identity}, expert: {ff}}``, or null); its tensors start
  with ``l<i>.``.

The network: ``x = embed[token]``; per layer ``h = rms(x) * norm1`` and ``x += residual_mult * (mixer(h) + ff(h))``;
``logits = logit_scale * head(rms(x) * final.norm)``.  The model's ``rms`` divides each of ``norm.groups`` equal parts of the
row by its own root mean square.

* ``attention`` (``parts/window_attention.py``): ``heads, kv_heads, dim, vdim, scale, conv, rot: {base, dims}``, optionally
  ``kv_from: j``; q, k, v with biases, then the convolution, then the rotation in halves on q and k; weights
  ``sigmoid(score + pb_h)``, not normalised; a gate per head.
* ``parallel`` (``parts/recurrent.py``, ``side_by_side``): ``left`` — ``heads, kv_heads, dim, vdim, scale, q_temp: {coef,
  every}`` — attention without rotation, with the query temperature, the bias ``-r1_h ln(1 + r2_h (i - j))`` and a gate per
  value; ``right`` — ``heads, kv_heads, dim, vdim, conv`` — ``channel_delta``.
* ``wkv`` (``parts/recurrent.py``): ``heads, dim``.
* mixture (``parts/feed_forward.py``): choice by softmax score plus correction, weights the scores, not renormalised; the
  last ``identity`` of the router's experts + identity outputs have no matrices.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, take
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec

ARCHITECTURE = "Nugolorn"
# The design has no table of positions and hence no largest position of its own; this bounds what one request may hold.
MAX_POSITIONS = 1 << 17
MIXER_TYPES = ("attention", "parallel", "wkv")


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


def _heads(raw: Mapping[str, Any], where: str) -> Tuple[int, int]:
    heads, kv = _positive(raw, "heads", where), _positive(raw, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"invalid model config: {where}heads={heads} is not a multiple of kv_heads={kv}")
    return heads, kv


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int
    rot_base: float
    rot_dims: int                 # 0: nothing is rotated
    kv_from: Optional[int]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "AttentionConfig":
        rot = _obj(raw, "rot", where, optional=True)
        source = raw.get("kv_from")
        if source is not None and (not isinstance(source, int) or isinstance(source, bool) or source < 0):
            raise ConfigError(f"invalid model config: {where}kv_from must name a layer, got {source!r}")
        if raw.get("mask") is not None:
            raise ConfigError(f"unsupported option: {where}mask (this mixer sees every earlier token)")
        out = cls(*_heads(raw, where), dim=_positive(raw, "dim", where), vdim=_positive(raw, "vdim", where),
                  scale=_number(raw, "scale", where), conv=_positive(raw, "conv", where),
                  rot_base=_number(rot, "base", where + "rot.") if rot else 1.0, rot_dims=take(rot, "dims", int) if rot else 0,
                  kv_from=source)
        if out.rot_dims < 0 or out.rot_dims % 2 or out.rot_dims > out.dim:
            raise ConfigError(f"invalid model config: {where}rot.dims={out.rot_dims} must be even and at most dim={out.dim}")
        if not out.rot_base > 0:
            raise ConfigError(f"invalid model config: {where}rot.base must be positive")
        return out

    def to_dict(self) -> dict:
        out: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "conv": self.conv}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out

    def spec(self, eps: float, width: int) -> PartSpec:
        position = PartSpec("rope_half", theta=self.rot_base, rotary_dim=self.rot_dims) if self.rot_dims else PartSpec("none")
        return PartSpec("window_attention", name="mix", num_heads=self.heads, num_kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                        scale=self.scale, qk_norm="none", eps=eps, bias=True, conv=self.conv, own_kv=self.kv_from is None,
                        weights="sigmoid", gate="head", position=position)


@dataclass(frozen=True)
class LeftConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[Tuple[float, int]]       # coefficient, period

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "LeftConfig":
        temp = _obj(raw, "q_temp", where, optional=True)
        for option in ("mask", "rot"):
            if raw.get(option) is not None:
                raise ConfigError(f"unsupported option: {where}{option} (this mixer sees every earlier token and rotates nothing)")
        return cls(*_heads(raw, where), dim=_positive(raw, "dim", where), vdim=_positive(raw, "vdim", where),
                   scale=_number(raw, "scale", where),
                   q_temp=(_number(temp, "coef", where + "q_temp."), _positive(temp, "every", where + "q_temp.")) if temp else None)

    def to_dict(self) -> dict:
        out: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.q_temp:
            out["q_temp"] = {"coef": self.q_temp[0], "every": self.q_temp[1]}
        return out

    def spec(self, eps: float) -> PartSpec:
        return PartSpec("window_attention", num_heads=self.heads, num_kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                        scale=self.scale, qk_norm="none", eps=eps, q_temp=self.q_temp, log_bias=True, gate="value")


@dataclass(frozen=True)
class RightConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "RightConfig":
        return cls(*_heads(raw, where), *(_positive(raw, k, where) for k in ("dim", "vdim", "conv")))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}

    def spec(self, eps: float, rank: int) -> PartSpec:
        return PartSpec("channel_delta", num_heads=self.heads, num_kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, taps=self.conv,
                        eps=eps, rank=rank)


def _drawn_rank(width: int) -> int:
    """The inner size of the low-rank products where no checkpoint says it (random weights): a thirty-second of the width, in
    multiples of eight."""
    return max(8, width // 32 // 8 * 8)


@dataclass(frozen=True)
class ParallelConfig:
    left: LeftConfig
    right: RightConfig

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "ParallelConfig":
        return cls(LeftConfig.from_dict(_obj(raw, "left", where), where + "left."), RightConfig.from_dict(_obj(raw, "right", where), where + "right."))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}

    def spec(self, eps: float, width: int) -> PartSpec:
        return PartSpec("side_by_side", name="mix", left=self.left.spec(eps), right=self.right.spec(eps, _drawn_rank(width)), eps=eps)


@dataclass(frozen=True)
class TimeMixingConfig:
    heads: int
    dim: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "TimeMixingConfig":
        return cls(_positive(raw, "heads", where), _positive(raw, "dim", where))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim}

    def spec(self, eps: float, width: int) -> PartSpec:
        return PartSpec("wkv", name="mix", num_heads=self.heads, dim=self.dim, eps=eps, rank=_drawn_rank(width))


_MIXER_CONFIGS = {"attention": AttentionConfig, "parallel": ParallelConfig, "wkv": TimeMixingConfig}


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                   # "dense" or "moe"
    ff: int                     # dense: its size; moe: an expert's size
    experts: int = 0
    top: int = 0
    identity: int = 0           # experts that give back their input

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "FeedForwardConfig":
        kind = take(raw, "kind", str)
        if kind == "dense":
            return cls("dense", _positive(raw, "ff", where))
        if kind == "moe":
            router, expert = _obj(raw, "router", where), _obj(raw, "expert", where)
            identity = take(router, "identity", int) if router.get("identity") is not None else 0
            out = cls("moe", _positive(expert, "ff", where + "expert."), _positive(router, "experts", where + "router."),
                      _positive(router, "top", where + "router."), identity)
            if out.identity < 0:
                raise ConfigError(f"invalid model config: {where}router.identity must not be negative")
            if out.top > out.experts + out.identity:
                raise ConfigError(f"invalid model config: {where}router.top={out.top} exceeds the {out.experts + out.identity} experts")
            return out
        raise ConfigError(f"unsupported option: {where}kind={kind!r} (dense or moe)")

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top, "identity": self.identity}}

    def spec(self) -> PartSpec:
        if self.kind == "dense":
            return PartSpec("gated", name="mlp", intermediate_size=self.ff, activation="silu", names=("gate", "up", "down"))
        return PartSpec("moe_routed", name="mlp", experts=self.experts, top=self.top, intermediate_size=self.ff, activation="silu",
                        score="softmax", correction_name="correction", identity=self.identity, router_name="router",
                        expert_names=("e{}.gate", "e{}.up", "e{}.down"))


@dataclass(frozen=True)
class NugolornLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[FeedForwardConfig]


@dataclass(frozen=True)
class NugolornConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    residual_mult: float
    logit_scale: float
    layers: Tuple[NugolornLayerConfig, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def max_model_len(self) -> int:
        return MAX_POSITIONS

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "NugolornConfig":
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
            mlp = _obj(entry, "mlp", where, optional=True)
            layers.append(NugolornLayerConfig(kind, _MIXER_CONFIGS[kind].from_dict(_obj(entry, "mixer", where), where + "mixer."),
                                              FeedForwardConfig.from_dict(mlp, where + "mlp.") if mlp else None))
        for i, layer in enumerate(layers):
            m = layer.mixer
            if layer.type != "attention" or m.kv_from is None:
                continue
            where = f"layers[{i}].mixer."
            if m.kv_from >= i or layers[m.kv_from].type != "attention" or layers[m.kv_from].mixer.kv_from is not None:
                raise ConfigError(f"invalid model config: {where}kv_from={m.kv_from} must name an earlier attention layer with projections of its own")
            src = layers[m.kv_from].mixer
            if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                raise ConfigError(f"invalid model config: {where}kv_heads, dim and vdim must equal those of layer {m.kv_from}, whose cache it reads")
        norm = _obj(raw, "norm", "")
        eps = _number(norm, "eps", "norm.")
        if not eps > 0:
            raise ConfigError("invalid model config: norm.eps must be positive")
        width = _positive(raw, "width", "")
        groups = _positive(norm, "groups", "norm.") if norm.get("groups") is not None else 1
        if width % groups:
            raise ConfigError(f"invalid model config: width={width} does not split into norm.groups={groups}")
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else (eos,) if isinstance(eos, int) else tuple(eos)
        return cls(vocab=_positive(raw, "vocab", ""), width=width, norm_eps=eps, norm_groups=groups,
                   residual_mult=_number(raw, "residual_mult", "") if raw.get("residual_mult") is not None else 1.0,
                   logit_scale=_number(raw, "logit_scale", "") if raw.get("logit_scale") is not None else 1.0,
                   layers=tuple(layers), eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "residual_mult": self.residual_mult,
               "logit_scale": self.logit_scale,
               "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": l.mlp.to_dict() if l.mlp else None} for l in self.layers]}
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out


def nugolorn_spec(cfg: NugolornConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", eps=cfg.norm_eps, weight_suffix="", groups=cfg.norm_groups)
    block = PartSpec("parallel", norm_name="norm1", multiplier=cfg.residual_mult)
    layers = tuple(LayerSpec(prefix=f"l{i}", block=block, mixer=layer.mixer.spec(cfg.norm_eps, cfg.width),
                             feed_forward=layer.mlp.spec() if layer.mlp else PartSpec("none", name="mlp"), norm=norm)
                   for i, layer in enumerate(cfg.layers))
    # no layer runs twice: a layer's run has the layer's number
    sources = {i: layer.mixer.kv_from for i, layer in enumerate(cfg.layers) if layer.type == "attention" and layer.mixer.kv_from is not None}
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS, layers=layers,
                     final_norm=norm.replace(gain_scale=cfg.logit_scale), embedding_name="embed", final_norm_prefix="final.norm",
                     lm_head_name="head", cache_source=sources, eos_token_ids=tuple(cfg.eos_token_ids))


register_architecture(ARCHITECTURE, NugolornConfig.from_dict, nugolorn_spec, replace=True)
