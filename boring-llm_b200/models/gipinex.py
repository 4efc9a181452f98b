"""The Gipinex decoder as a list of parts, and its checkpoint tensor names.

A layer is a `PreNormBlock` (RMS norms whose weights are stored around zero) around a `MixedScoreAttention` ('attention') or a
`LatentAttention` with interleaved rotation and a gate per head ('latent_attention'), and an optional feed-forward: `GluMLP`
with the clamped activation and biases, or `RoutedExperts` with a router bias and weights from the chosen logits plus a
`GluMLP` that every token uses. With `loop` the run order names the blocks of layers start .. stop-1 `times` times, each entry
with a cache layer of its own, and a `StreamReentry` runs ahead of each pass. The output head is the embedding table.

`residual_mult` a (x <- x + a f(N(x))) costs nothing: the stream is kept divided by a. With y = x / a the layers are
y <- y + f(N(a y)), N(a y) is the same norm of y with eps / a^2, the reentry is linear, and the embedding rows are scaled by
1 / a as they are read.

Layer i's tensors are `l<i>.*`: `norm1`, `norm2`, `mix.{q, k, talk, g, o}` or `mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o}`,
`mlp.{gate, up, down}` (+ `.b`) or `mlp.{router, router.b, e<j>.gate / .up / .down, shared.gate / .up / .down}`; `loop.in`.
"""
from __future__ import annotations

from ..config import register_architecture
from ..config.gipinex_config import DenseFFConfig, ExpertsConfig, GipinexConfig, LatentMixerConfig, MixedAttentionConfig
from ..parts import (DecoderModel, Embedding, GluMLP, LatentAttention, LayerCall, MixedScoreAttention, OutputHead, PreNormBlock,
                     RMSNorm, RotaryTable, RoutedExperts, StreamReentry, SumFeedForward, distance_slopes)


def _norm(cfg: GipinexConfig, name):
    return RMSNorm(cfg.width, cfg.norm_eps / cfg.residual_mult ** 2, {"weight": name}, around_zero=True)


def _mixer(cfg: GipinexConfig, m, p: str):
    d, eps = cfg.width, cfg.norm_eps
    if isinstance(m, MixedAttentionConfig):
        return MixedScoreAttention(d, m.heads, m.kv_heads, m.dim,
                                   {"wq": p + "q", "wk": p + "k", "talk": p + "talk", "wg": p + "g", "wo": p + "o"},
                                   scale=m.scale, qk_norm_eps=eps, slopes=distance_slopes(m.heads), out_gate=True)
    if isinstance(m, LatentMixerConfig):
        names = {"wdq": p + "dq", "dq_norm": p + "dq.norm", "wuq": p + "uq", "wdkv": p + "dkv", "dkv_norm": p + "dkv.norm",
                 "wuk": p + "uk", "wuv": p + "uv", "wg": p + "g", "wo": p + "o"}
        rotary = RotaryTable(m.rot_dim, m.rot_base, n_rot=m.rot_dims, pairs="interleaved") if m.rot_dims else None
        return LatentAttention(d, m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, rotary, names, scale=m.scale,
                               norm_eps=eps, out_gate="head")
    raise TypeError(f"no mixer for {type(m).__name__}")


def _feed_forward(cfg: GipinexConfig, f, p: str):
    d = cfg.width
    if isinstance(f, DenseFFConfig):
        return GluMLP(d, f.ff, {"w_gate": p + "gate", "w_up": p + "up", "w_down": p + "down", "b_gate": p + "gate.b",
                                "b_up": p + "up.b", "b_down": p + "down.b"}, activation="clamped", limit=f.limit, bias=True)
    if isinstance(f, ExpertsConfig):
        names = {"router": p + "router", "router_bias": p + "router.b"}
        for j in range(f.experts):
            names.update({f"gate{j}": f"{p}e{j}.gate", f"up{j}": f"{p}e{j}.up", f"down{j}": f"{p}e{j}.down"})
        experts = RoutedExperts(d, f.ff, f.experts, f.top, names, correction=False, activation="clamped", limit=f.limit,
                                score="chosen", router_bias=True)
        if not f.shared_ff:
            return experts
        shared = GluMLP(d, f.shared_ff, {"w_gate": p + "shared.gate", "w_up": p + "shared.up", "w_down": p + "shared.down"},
                        activation="clamped", limit=f.shared_limit)
        return SumFeedForward([experts, shared])
    raise TypeError(f"no feed-forward for {type(f).__name__}")


def build_gipinex(cfg: GipinexConfig) -> DecoderModel:
    d = cfg.width
    blocks, spare = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ff = {}
        if layer.mlp is None:
            spare.append(p + "norm2")         # a file may keep the norm of a feed-forward that the layer does not have
        else:
            ff = dict(ffn_norm=_norm(cfg, p + "norm2"), ffn=_feed_forward(cfg, layer.mlp, p + "mlp."))
        blocks.append(PreNormBlock(_norm(cfg, p + "norm1"), _mixer(cfg, layer.mixer, p + "mix."), **ff))
    order = [LayerCall(i, n, enters=enters) for n, (i, enters) in enumerate(cfg.run_order())]
    embedding = Embedding(cfg.vocab_size, d, {"table": "embed"}, scale=1.0 / cfg.residual_mult)
    return DecoderModel(embedding, blocks, _norm(cfg, "final.norm"), OutputHead(cfg.vocab_size, d, {}, tied_to=embedding),
                        schedule=order, ignorable_tensors=spare,
                        reentry=StreamReentry(d, {"weight": "loop.in"}) if cfg.loop is not None else None)


register_architecture(GipinexConfig.ARCHITECTURES, GipinexConfig, build_gipinex)
