"""The Zuvevik decoder as a list of parts, and its checkpoint tensor names.

A `PairEmbedding` fills a residual of `streams` streams. A layer is a `HyperBlock` (RMS norms, a `HyperConnection` around each
sublayer) of a `GatedSinkAttention` (window, norms over the whole projections, values blended with those of the first blending
layer, a gate per channel, heads padded to a size of the tensor-core kernels) and an optional feed-forward: `GluMLP` with SiLU, or
`RoutedExperts` with clamped activations whose weights multiply what the experts read. An RMS norm of the streams' sum, with
`logit_scale` in its weight, and an untied head end the model.

Layer i's tensors are `l<i>.*`: `norm1`, `norm2`, `hc1.{in, out, mix}`, `hc2.*`, `mix.{q, k, v, q.norm, k.norm, vmix, g, o}`,
`mlp.{gate, up, down}` or `mlp.{router, e<j>.gate / .up / .down}`.
"""
from __future__ import annotations

from ..config import register_architecture
from ..config.zuvevik_config import DenseFFConfig, ExpertsConfig, ZuvevikConfig
from ..parts import (DecoderModel, GatedSinkAttention, GluMLP, HyperBlock, HyperConnection, OutputHead, PairEmbedding, RMSNorm,
                     RotaryTable, RoutedExperts)


def _norm(cfg: ZuvevikConfig, name, gain: float = 1.0):
    return RMSNorm(cfg.width, cfg.norm_eps, {"weight": name}, gain=gain)


def _connection(cfg: ZuvevikConfig, p: str):
    return HyperConnection(cfg.streams, {"in": p + "in", "out": p + "out", "mix": p + "mix"})


def _mixer(cfg: ZuvevikConfig, m, p: str, role):
    names = {"wq": p + "q", "wk": p + "k", "wv": p + "v", "wo": p + "o", "q_norm": p + "q.norm", "k_norm": p + "k.norm",
             "wg": p + "g", "vmix": p + "vmix"}
    return GatedSinkAttention(cfg.width, m.heads, m.kv_heads, m.dim, m.vdim,
                              RotaryTable(m.dim, m.rot_base, n_rot=m.rot_dims, pairs="halves"), names, window=m.window,
                              scale=m.scale, qk_norm="whole", qk_norm_eps=cfg.norm_eps, out_gate="channel", value_mix=role,
                              pad_heads=True)


def _feed_forward(cfg: ZuvevikConfig, f, p: str):
    d = cfg.width
    if isinstance(f, DenseFFConfig):
        return GluMLP(d, f.ff, {"w_gate": p + "gate", "w_up": p + "up", "w_down": p + "down"}, activation="silu")
    if isinstance(f, ExpertsConfig):
        names = {"router": p + "router"}
        for j in range(f.experts):
            names.update({f"gate{j}": f"{p}e{j}.gate", f"up{j}": f"{p}e{j}.up", f"down{j}": f"{p}e{j}.down"})
        return RoutedExperts(d, f.ff, f.experts, f.top, names, correction=False, activation="clamped", limit=f.limit,
                             weight_on="input")
    raise TypeError(f"no feed-forward for {type(f).__name__}")


def build_zuvevik(cfg: ZuvevikConfig) -> DecoderModel:
    d = cfg.width
    blocks, spare = [], []
    for i, (layer, role) in enumerate(zip(cfg.layers, cfg.value_mix_roles())):
        p = f"l{i}."
        ff = {}
        if role != "follow":
            spare.append(p + "mix.vmix")      # the layer that the others blend with has the number too and does not use it
        if layer.mlp is None:                 # a file may keep the tensors around a feed-forward that the layer does not have
            spare += [p + "norm2"] + [p + "hc2." + n for n in ("in", "out", "mix")]
        else:
            ff = dict(ffn_norm=_norm(cfg, p + "norm2"), ffn=_feed_forward(cfg, layer.mlp, p + "mlp."),
                      ffn_connection=_connection(cfg, p + "hc2."))
        blocks.append(HyperBlock(_norm(cfg, p + "norm1"), _mixer(cfg, layer.mixer, p + "mix.", role), _connection(cfg, p + "hc1."), **ff))
    embedding = PairEmbedding(cfg.vocab_size, d, cfg.pairs.buckets, cfg.pairs.mul_prev, cfg.pairs.mul_cur,
                              {"table": "embed", "pairs": "bigram"})
    return DecoderModel(embedding, blocks, _norm(cfg, "final.norm", gain=cfg.logit_scale),
                        OutputHead(cfg.vocab_size, d, {"weight": "head"}), ignorable_tensors=spare, streams=cfg.streams)


register_architecture(ZuvevikConfig.ARCHITECTURES, ZuvevikConfig, build_zuvevik)
