"""Typed configuration of the Gipinex decoder, read from its own config.json keys.

    {"architecture": "Gipinex", "vocab": V, "width": d, "norm": {"eps": e}, "residual_mult": a,
     "loop": {"start", "stop", "times"} (optional),
     "layers": [{"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {...} | null}, ...]}

    attention mixer:         {"heads", "kv_heads", "dim", "vdim", "scale"}                    (vdim = dim: the values are the keys)
    latent attention mixer:  {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}}
    mlp:                     {"kind": "dense", "ff", "limit"}
                             {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"}, "shared": {"ff", "limit"} (optional)}

Every size and every constant that can differ between models of the design is a field. `loop`: layers start .. stop-1 run
`times` times in a row with the same tensors, each pass with caches of its own.
"""
from __future__ import annotations

import warnings
from dataclasses import dataclass, field
from typing import List, Optional, Tuple, Union

from .model_config import ConfigError, _get, _positive, architecture_name


@dataclass(frozen=True)
class MixedAttentionConfig:
    """'attention': heads whose scores are mixed before the softmax; the values are the keys before their norm."""
    heads: int
    kv_heads: int
    dim: int
    scale: float

    def to_dict(self):
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim, "scale": self.scale}


@dataclass(frozen=True)
class LatentMixerConfig:
    """'latent_attention': a cached latent of `kv_rank` values and one rotated key part of `rot_dim` values per token, queries
    through a latent of `q_rank`; a head has `dim` unrotated and `rot_dim` rotated query/key values and `vdim` channels."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dims}}


@dataclass(frozen=True)
class DenseFFConfig:
    """down(clamped_glu(gate h, up h)) with hidden size `ff` and biases on all three products."""
    ff: int
    limit: float

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class ExpertsConfig:
    """`experts` clamped-GLU experts of hidden size `ff` behind a router with a bias, `top` a token, weighted by the softmax
    over the chosen logits; an optional expert of hidden size `shared_ff` that every token uses."""
    ff: int
    limit: float
    experts: int
    top: int
    shared_ff: int = 0
    shared_limit: float = 0.0

    def to_dict(self):
        d = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return d


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int

    def to_dict(self):
        return {"start": self.start, "stop": self.stop, "times": self.times}


@dataclass(frozen=True)
class GipinexLayerConfig:
    type: str
    mixer: Union[MixedAttentionConfig, LatentMixerConfig]
    mlp: Union[DenseFFConfig, ExpertsConfig, None] = None

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}


def _sizes(m: dict, where: str, keys) -> dict:
    return {k: _positive(f"{where}.{k}", _get(m, k, int)) for k in keys}


def _limit(m: dict, where: str) -> float:
    v = _get(m, "limit", float)
    if not v > 0:
        raise ConfigError(f"config.json: {where}.limit must be positive, got {v}")
    return float(v)


def _mixer(kind: str, m: dict, where: str):
    if kind == "attention":
        n = _sizes(m, where, ("heads", "kv_heads", "dim"))
        if n["heads"] % n["kv_heads"] != 0:
            raise ConfigError(f"config.json: {where}: {n['heads']} heads cannot share {n['kv_heads']} key/value heads")
        vdim = _positive(f"{where}.vdim", _get(m, "vdim", int, n["dim"]))
        if vdim != n["dim"]:
            raise ConfigError(f"config.json: {where}.vdim ({vdim}) must equal dim ({n['dim']}): the values are the keys")
        return MixedAttentionConfig(n["heads"], n["kv_heads"], n["dim"], float(_get(m, "scale", float)))
    if kind == "latent_attention":
        n = _sizes(m, where, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
        rot = _get(m, "rot", dict)
        base = float(_get(rot, "base", float))
        if not base > 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive, got {base}")
        dims = _get(rot, "dims", int, n["rot_dim"])
        if dims < 0 or dims % 2 != 0 or dims > n["rot_dim"]:
            raise ConfigError(f"config.json: {where}.rot.dims ({dims}) must be even and at most rot_dim ({n['rot_dim']})")
        return LatentMixerConfig(n["heads"], n["dim"], n["rot_dim"], n["vdim"], n["q_rank"], n["kv_rank"],
                                 float(_get(m, "scale", float)), base, dims)
    raise ConfigError(f"config.json: {where}: unknown layer type {kind!r} (attention, latent_attention)")


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where} must be an object or null")
    kind = _get(mlp, "kind", str)
    if kind == "dense":
        return DenseFFConfig(_positive(f"{where}.ff", _get(mlp, "ff", int)), _limit(mlp, where))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not supported (dense, moe)")
    expert, router = _get(mlp, "expert", dict), _get(mlp, "router", dict)
    experts = _positive(f"{where}.router.experts", _get(router, "experts", int))
    top = _positive(f"{where}.router.top", _get(router, "top", int))
    if top > experts:
        raise ConfigError(f"config.json: {where}.router: {top} experts a token out of {experts}")
    shared_ff, shared_limit = 0, 0.0
    if mlp.get("shared") is not None:
        sh = _get(mlp, "shared", dict)
        shared_ff, shared_limit = _positive(f"{where}.shared.ff", _get(sh, "ff", int)), _limit(sh, where + ".shared")
    return ExpertsConfig(_positive(f"{where}.expert.ff", _get(expert, "ff", int)), _limit(expert, where + ".expert"), experts, top,
                         shared_ff, shared_limit)


def _loop(d: dict, n_layers: int) -> Optional[LoopConfig]:
    if d.get("loop") is None:
        return None
    loop = _get(d, "loop", dict)
    start, stop, times = (_get(loop, k, int) for k in ("start", "stop", "times"))
    if not 0 <= start < stop <= n_layers:
        raise ConfigError(f"config.json: loop from layer {start} to {stop} does not lie inside {n_layers} layers")
    return LoopConfig(start, stop, _positive("loop.times", times))


@dataclass(frozen=True)
class GipinexConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[GipinexLayerConfig, ...]
    loop: Optional[LoopConfig] = None
    max_position_embeddings: int = 1 << 20      # the design has no position limit of its own; engines clamp to their cache
    eos_token_ids: Tuple[int, ...] = ()
    raw: dict = field(default_factory=dict, compare=False, repr=False)

    ARCHITECTURES = ("Gipinex",)

    @classmethod
    def from_dict(cls, d: dict) -> "GipinexConfig":
        arch = architecture_name(d)
        vocab = _positive("vocab", _get(d, "vocab", int))
        width = _positive("width", _get(d, "width", int))
        eps = _get(_get(d, "norm", dict), "eps", float)
        if not eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps}")
        mult = float(_get(d, "residual_mult", float, 1.0))
        if not mult > 0:
            raise ConfigError(f"config.json: residual_mult must be positive, got {mult}")
        entries = _get(d, "layers", list)
        if not entries:
            raise ConfigError("config.json: 'layers' lists no layer")
        layers = []
        for i, e in enumerate(entries):
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = _get(e, "type", str)
            layers.append(GipinexLayerConfig(kind, _mixer(kind, _get(e, "mixer", dict), f"layers[{i}].mixer"),
                                             _mlp(e.get("mlp"), f"layers[{i}].mlp")))
        known = {"architecture", "architectures", "model_type", "vocab", "width", "norm", "residual_mult", "loop", "layers",
                 "max_position_embeddings", "eos_token_id"}
        unknown = sorted(k for k in d if k not in known and not k.startswith("_"))
        if unknown:
            warnings.warn(f"config.json: keys not used by {arch}: {', '.join(unknown)}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(x) for x in eos))
        return cls(architecture=arch, vocab_size=vocab, width=width, norm_eps=float(eps), residual_mult=mult, layers=tuple(layers),
                   loop=_loop(d, len(layers)),
                   max_position_embeddings=_positive("max_position_embeddings", _get(d, "max_position_embeddings", int, 1 << 20)),
                   eos_token_ids=eos_ids, raw=dict(d))

    def run_order(self) -> List[Tuple[int, bool]]:
        """[(layer, begins a pass of the loop)] in the order in which the layers run."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [(i, False) for i in range(n)]
        body = [(i, i == loop.start) for i in range(loop.start, loop.stop)]
        return [(i, False) for i in range(loop.start)] + body * loop.times + [(i, False) for i in range(loop.stop, n)]

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "layers": [l.to_dict() for l in self.layers]}
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        if self.max_position_embeddings != 1 << 20:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
