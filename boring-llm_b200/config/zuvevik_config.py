"""Typed configuration of the Zuvevik decoder, read from its own config.json keys.

    {"architecture": "Zuvevik", "vocab": V, "width": d, "norm": {"eps": e}, "streams": n, "logit_scale": c,
     "embedding": {"bigram": {"buckets", "mul_prev", "mul_cur"}},
     "layers": [{"type": "attention", "mixer": {...}, "mlp": {...} | null}, ...]}

    attention mixer:  {"heads", "kv_heads", "dim", "vdim", "scale", "rot": {"base", "dims"}, "mask": {"size"}, "v_mix"}
    mlp:              {"kind": "dense", "ff"}
                      {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"}}

Every size and every constant that can differ between models of the design is a field.
"""
from __future__ import annotations

import warnings
from dataclasses import dataclass, field
from typing import List, Optional, Tuple, Union

from .model_config import ConfigError, _get, _positive, architecture_name


@dataclass(frozen=True)
class WindowedAttentionConfig:
    """'attention': q and k normed over the whole projection and rotated in halves, a window of `window` tokens (0: none), a
    sigmoid gate per channel; `v_mix`: the values are blended with those of the first layer that says so."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    window: int
    v_mix: bool = False

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "rot": {"base": self.rot_base, "dims": self.rot_dims}, "v_mix": self.v_mix}
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class DenseFFConfig:
    """down(silu(gate h) * up h) with hidden size `ff`."""
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertsConfig:
    """`experts` clamped-GLU experts of hidden size `ff`, `top` a token, the chosen sigmoid scores on what the experts read."""
    ff: int
    limit: float
    experts: int
    top: int

    def to_dict(self):
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class PairTableConfig:
    buckets: int
    mul_prev: int
    mul_cur: int

    def to_dict(self):
        return {"bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}}


@dataclass(frozen=True)
class ZuvevikLayerConfig:
    type: str
    mixer: WindowedAttentionConfig
    mlp: Union[DenseFFConfig, ExpertsConfig, None] = None

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}


def _sizes(m: dict, where: str, keys) -> dict:
    return {k: _positive(f"{where}.{k}", _get(m, k, int)) for k in keys}


def _mixer(kind: str, m: dict, where: str) -> WindowedAttentionConfig:
    if kind != "attention":
        raise ConfigError(f"config.json: {where}: unknown layer type {kind!r} (attention)")
    n = _sizes(m, where, ("heads", "kv_heads", "dim"))
    if n["heads"] % n["kv_heads"] != 0:
        raise ConfigError(f"config.json: {where}: {n['heads']} heads cannot share {n['kv_heads']} key/value heads")
    vdim = _positive(f"{where}.vdim", _get(m, "vdim", int, n["dim"]))
    rot = _get(m, "rot", dict)
    base = float(_get(rot, "base", float))
    if not base > 0:
        raise ConfigError(f"config.json: {where}.rot.base must be positive, got {base}")
    dims = _get(rot, "dims", int, n["dim"])
    if dims < 0 or dims % 2 != 0 or dims > n["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims ({dims}) must be even and at most dim ({n['dim']})")
    window = 0
    if m.get("mask") is not None:
        window = _positive(f"{where}.mask.size", _get(_get(m, "mask", dict), "size", int))
    return WindowedAttentionConfig(n["heads"], n["kv_heads"], n["dim"], vdim, float(_get(m, "scale", float)), base, dims, window,
                                   bool(_get(m, "v_mix", bool, False)))


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where} must be an object or null")
    kind = _get(mlp, "kind", str)
    if kind == "dense":
        return DenseFFConfig(_positive(f"{where}.ff", _get(mlp, "ff", int)))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not supported (dense, moe)")
    expert, router = _get(mlp, "expert", dict), _get(mlp, "router", dict)
    experts = _positive(f"{where}.router.experts", _get(router, "experts", int))
    top = _positive(f"{where}.router.top", _get(router, "top", int))
    if top > experts:
        raise ConfigError(f"config.json: {where}.router: {top} experts a token out of {experts}")
    limit = float(_get(expert, "limit", float))
    if not limit > 0:
        raise ConfigError(f"config.json: {where}.expert.limit must be positive, got {limit}")
    return ExpertsConfig(_positive(f"{where}.expert.ff", _get(expert, "ff", int)), limit, experts, top)


def _check_blends(layers) -> None:
    """The layers that blend their values do so channel by channel with those of the first one."""
    widths = [(i, l.mixer.kv_heads * l.mixer.vdim) for i, l in enumerate(layers) if l.mixer.v_mix]
    for i, w in widths[1:]:
        if w != widths[0][1]:
            raise ConfigError(f"config.json: layers[{i}].mixer.v_mix: {w} value channels, layer {widths[0][0]} has {widths[0][1]}")


@dataclass(frozen=True)
class ZuvevikConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    streams: int
    logit_scale: float
    pairs: PairTableConfig
    layers: Tuple[ZuvevikLayerConfig, ...]
    max_position_embeddings: int = 1 << 20      # the design has no position limit of its own; engines clamp to their cache
    eos_token_ids: Tuple[int, ...] = ()
    raw: dict = field(default_factory=dict, compare=False, repr=False)

    ARCHITECTURES = ("Zuvevik",)

    @classmethod
    def from_dict(cls, d: dict) -> "ZuvevikConfig":
        arch = architecture_name(d)
        vocab = _positive("vocab", _get(d, "vocab", int))
        width = _positive("width", _get(d, "width", int))
        eps = _get(_get(d, "norm", dict), "eps", float)
        if not eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps}")
        bigram = _get(_get(d, "embedding", dict), "bigram", dict)
        pairs = PairTableConfig(_positive("embedding.bigram.buckets", _get(bigram, "buckets", int)), _get(bigram, "mul_prev", int),
                                _get(bigram, "mul_cur", int))
        entries = _get(d, "layers", list)
        if not entries:
            raise ConfigError("config.json: 'layers' lists no layer")
        layers = []
        for i, e in enumerate(entries):
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = _get(e, "type", str)
            layers.append(ZuvevikLayerConfig(kind, _mixer(kind, _get(e, "mixer", dict), f"layers[{i}].mixer"),
                                             _mlp(e.get("mlp"), f"layers[{i}].mlp")))
        _check_blends(layers)
        known = {"architecture", "architectures", "model_type", "vocab", "width", "norm", "streams", "logit_scale", "embedding", "layers",
                 "max_position_embeddings", "eos_token_id"}
        unknown = sorted(k for k in d if k not in known and not k.startswith("_"))
        if unknown:
            warnings.warn(f"config.json: keys not used by {arch}: {', '.join(unknown)}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(x) for x in eos))
        return cls(architecture=arch, vocab_size=vocab, width=width, norm_eps=float(eps),
                   streams=_positive("streams", _get(d, "streams", int)), logit_scale=float(_get(d, "logit_scale", float, 1.0)),
                   pairs=pairs, layers=tuple(layers),
                   max_position_embeddings=_positive("max_position_embeddings", _get(d, "max_position_embeddings", int, 1 << 20)),
                   eos_token_ids=eos_ids, raw=dict(d))

    def value_mix_roles(self) -> List[Optional[str]]:
        """Per layer: None (its values are its own), "first" (the others blend with its values) or "follow"."""
        roles, seen = [], False
        for layer in self.layers:
            roles.append(None if not layer.mixer.v_mix else ("follow" if seen else "first"))
            seen = seen or layer.mixer.v_mix
        return roles

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
             "streams": self.streams, "logit_scale": self.logit_scale, "embedding": self.pairs.to_dict(),
             "layers": [l.to_dict() for l in self.layers]}
        if self.max_position_embeddings != 1 << 20:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
