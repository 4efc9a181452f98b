"""Gipinex without a GPU: configuration keys and errors, declared tensors, the run order of looped layers and their caches, the
stream kept divided by the residual multiplier, interleaved pairs as reordered rows, and the plain implementation against
closed forms."""
import copy
import math

import pytest
import torch

import plain_gipinex as pg
from boring_llm_b200 import ConfigError, GipinexConfig
from boring_llm_b200.cache import CacheManager, PagedKVSpec
from boring_llm_b200.models import build_model
from boring_llm_b200.parts import (Embedding, LatentAttention, LayerCall, DecoderModel, OutputHead, RMSNorm, RotaryTable, distance_slopes)
from boring_llm_b200.weights.random_init import random_tensor

F64 = torch.float64

ATT = {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 10, "scale": 0.3}
LAT = {"heads": 5, "dim": 8, "rot_dim": 6, "vdim": 12, "q_rank": 14, "kv_rank": 18, "scale": 0.25, "rot": {"base": 700.0, "dims": 6}}
MOE = {"kind": "moe", "expert": {"ff": 12, "limit": 1.25}, "router": {"experts": 7, "top": 3}, "shared": {"ff": 20, "limit": 0.75}}
CFG = {"architecture": "Gipinex", "vocab": 77, "width": 36, "norm": {"eps": 2e-5}, "residual_mult": 0.8, "layers": [
    {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 28, "limit": 2.0}},
    {"type": "latent_attention", "mixer": LAT, "mlp": MOE},
    {"type": "attention", "mixer": dict(ATT, heads=2, kv_heads=2), "mlp": None},
    {"type": "latent_attention", "mixer": dict(LAT, heads=1), "mlp": {k: v for k, v in MOE.items() if k != "shared"}}],
    "loop": {"start": 1, "stop": 3, "times": 3}}


def test_config_round_trip_and_fields():
    cfg = GipinexConfig.from_dict(CFG)
    assert cfg.to_dict() == CFG
    assert (cfg.vocab_size, cfg.width, cfg.norm_eps, cfg.residual_mult) == (77, 36, 2e-5, 0.8)
    a, m, f = cfg.layers[0].mixer, cfg.layers[1].mixer, cfg.layers[1].mlp
    assert (a.heads, a.kv_heads, a.dim, a.scale) == (6, 3, 10, 0.3)
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot_base, m.rot_dims) == (5, 8, 6, 12, 14, 18, 0.25, 700.0, 6)
    assert (f.ff, f.limit, f.experts, f.top, f.shared_ff, f.shared_limit) == (12, 1.25, 7, 3, 20, 0.75)
    assert (cfg.layers[0].mlp.ff, cfg.layers[0].mlp.limit) == (28, 2.0)
    assert cfg.layers[2].mlp is None and cfg.layers[3].mlp.shared_ff == 0
    for loop in (None, "absent"):
        d = {k: v for k, v in CFG.items() if k != "loop"} if loop else dict(CFG, loop=None)
        assert GipinexConfig.from_dict(d).loop is None


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "gla", "unknown layer type"),
    (("layers", 0, "mixer", "kv_heads"), 4, "cannot share"),
    (("layers", 0, "mixer", "vdim"), 12, "the values are the keys"),
    (("layers", 1, "mixer", "rot", "dims"), 5, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 8, "rot.dims"),
    (("layers", 1, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 1, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 1, "mlp", "router", "top"), 8, "out of 7"),
    (("layers", 1, "mlp", "expert", "limit"), 0.0, "limit"),
    (("layers", 1, "mlp", "shared", "limit"), -1.0, "limit"),
    (("layers", 0, "mlp", "kind"), "swiglu", "not supported"),
    (("loop", "stop"), 5, "does not lie inside"),
    (("loop", "start"), 3, "does not lie inside"),
    (("loop", "times"), 0, "loop.times"),
    (("residual_mult",), 0.0, "residual_mult"),
    (("norm", "eps"), 0.0, "norm.eps"),
])
def test_config_errors_name_the_key(path, value, word):
    d = copy.deepcopy(CFG)
    at = d
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        GipinexConfig.from_dict(d)


def test_declared_tensors_run_order_and_caches():
    cfg = GipinexConfig.from_dict(CFG)
    model = build_model(cfg)
    specs = {k: tuple(v.shape) for k, v in model.tensor_specs().items()}
    assert specs["embed"] == (77, 36) and specs["loop.in"] == (36, 72) and specs["final.norm"] == (36,) and "head" not in specs
    assert specs["l0.mix.q"] == (60, 36) and specs["l0.mix.k"] == (30, 36) and specs["l0.mix.talk"] == (6, 6) and specs["l0.mix.g"] == (60, 36)
    assert "l0.mix.v" not in specs and specs["l0.mlp.gate.b"] == (28,) and specs["l0.mlp.down.b"] == (36,)
    assert specs["l1.mix.g"] == (5, 36) and specs["l1.mix.uq"] == (5 * 14, 14) and specs["l1.mix.dkv"] == (24, 36)
    assert specs["l1.mlp.router.b"] == (7,) and specs["l1.mlp.e6.down"] == (36, 12) and specs["l1.mlp.shared.up"] == (20, 36)
    assert "l2.norm2" not in specs and "l2.norm2" in model.ignorable_tensors and "l3.mlp.shared.up" not in specs
    assert [(c.block, c.cache, c.enters) for c in model.schedule] == [
        (0, 0, False), (1, 1, True), (2, 2, False), (1, 3, True), (2, 4, False), (1, 5, True), (2, 6, False), (3, 7, False)]
    assert [n for n, e in cfg.run_order()] == [i for i, _ in pg.run_order(CFG)]
    caches = model.cache_specs()
    assert caches[1] == caches[3] == PagedKVSpec(1, 24, 0, 18, values_in_keys=True)
    assert caches[0] == PagedKVSpec(3, 10, 0, 2) and caches[2] == caches[6] == PagedKVSpec(2, 10, 0, 2)
    groups = CacheManager(caches, 16, 128, 2).paged_groups          # one block table for all runs of a layer
    assert sorted(len(g.cache_layers) for g in groups) == [1, 3, 4]
    plain = build_model(GipinexConfig.from_dict(dict(CFG, loop=None)))
    assert "loop.in" not in plain.tensor_specs() and [c.block for c in plain.schedule] == [0, 1, 2, 3]
    assert not any(c.enters for c in plain.schedule)


def test_entries_that_begin_a_pass_need_a_reentry():
    e = Embedding(5, 4, {"table": "e"})
    block = build_model(GipinexConfig.from_dict(CFG)).blocks[0]
    with pytest.raises(ValueError, match="reentry"):
        DecoderModel(e, [block], RMSNorm(4, 1e-5, {"weight": "n"}), OutputHead(5, 4, {}, tied_to=e), schedule=[LayerCall(0, 0, enters=True)])


def test_norm_weights_around_zero():
    cfg = GipinexConfig.from_dict(CFG)
    spec = build_model(cfg).tensor_specs()["l0.norm1"]
    w = random_tensor("l0.norm1", spec, 3, torch.float32, std=0.02)
    assert abs(float(w.mean())) < 0.02                       # the random-weights mode draws them around zero, not one
    n = RMSNorm(3, 1e-5, {"weight": "w"}, around_zero=True)
    n.place({"weight": torch.tensor([0.25, -1.0, 2.0]).bfloat16()}, torch.bfloat16, "cpu")
    assert n.weight.dtype == torch.float32 and n.weight.tolist() == [1.25, 0.0, 3.0]


def test_the_stream_divided_by_the_residual_multiplier():
    """x <- x + a f(N_eps(x)) against y <- y + f(N_(eps / a^2)(y)) with y = x / a."""
    g = torch.Generator().manual_seed(1)
    x = torch.randn(4, 9, generator=g, dtype=F64)
    w, eps, a = torch.randn(9, generator=g, dtype=F64), 0.3, 0.37
    y = x / a
    for _ in range(3):
        x = x + a * torch.tanh(pg.offset_norm(x, w, eps))
        y = y + torch.tanh(pg.offset_norm(y, w, eps / a ** 2))
    assert (y * a - x).abs().max() < 1e-12
    model = build_model(GipinexConfig.from_dict(CFG))
    assert model.embedding.scale == 1.0 / 0.8 and model.final_norm.eps == 2e-5 / 0.8 ** 2
    assert model.blocks[0].mixer.qk_norm_eps == 2e-5 and model.blocks[1].mixer.eps == 2e-5       # the inner norms keep their eps


@pytest.mark.parametrize("dims", [6, 4, 2])
def test_interleaved_pairs_are_reordered_rows(dims):
    """Rows in the order that the mixer places them, rotated in halves, give the scores of the interleaved rotation."""
    n, lead = 6, 3
    part = LatentAttention(8, 2, lead, n, 4, 5, 7, RotaryTable(n, 50.0, n_rot=dims, pairs="interleaved"),
                           {k: k for k in ("wdq", "dq_norm", "wuq", "wdkv", "dkv_norm", "wuk", "wuv", "wo")})
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(5, lead + n, generator=g, dtype=F64), torch.randn(5, lead + n, generator=g, dtype=F64)
    pos = torch.tensor([0, 3, 11, 64, 200])
    want = pg.rotate_pairs(q[:, lead:], pos, dims, 50.0) @ pg.rotate_pairs(k[:, lead:], pos, dims, 50.0).T

    def halves(x):
        x = part._halves(x.T, lead).T[:, lead:]
        h = dims // 2
        a = pos.to(F64)[:, None] * torch.tensor([50.0 ** (-2.0 * i / dims) for i in range(h)], dtype=F64)
        u, v = x[:, :h], x[:, h:dims]
        return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), x[:, dims:]], dim=1)
    assert (halves(q) @ halves(k).T - want).abs().max() < 1e-12
    assert torch.equal(part._halves(q.T, lead).T[:, :lead], q[:, :lead])


def test_slopes():
    assert distance_slopes(4) == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    assert distance_slopes(1) == [2.0 ** -8]
    assert pg.distance_slopes(12).tolist() == pytest.approx(distance_slopes(12))


# ---- the plain implementation against closed forms -----------------------------------------------------------------------
def test_plain_mixing_moves_to_the_query_and_the_slope():
    """What the kernels rest on: mixed scores equal scores of mixed queries over all key heads with a mixed slope."""
    g = torch.Generator().manual_seed(3)
    T, H, G, d = 7, 6, 3, 4
    q, k = torch.randn(T, H, d, generator=g, dtype=F64), torch.randn(T, G, d, generator=g, dtype=F64)
    talk, scale, eps = torch.randn(H, H, generator=g, dtype=F64), 0.7, 1e-3
    qn, kn = pg.rms_unit(q, eps), pg.rms_unit(k, eps)
    s = pg.mix_heads(talk, pg.biased_scores(qn.permute(1, 0, 2), kn.repeat_interleave(2, dim=1).permute(1, 0, 2), scale))
    Q = torch.stack([torch.einsum("hg,tgd->thd", talk[:, 2 * c:2 * c + 2], qn[:, 2 * c:2 * c + 2]) for c in range(G)], dim=2)
    slope = talk @ pg.distance_slopes(H)
    i = torch.arange(T, dtype=F64)
    mine = torch.einsum("ihcd,jcd->hij", Q, kn) * scale - slope[:, None, None] * (i[:, None] - i[None, :])
    assert (mine - s).abs().max() < 1e-12


def test_plain_attention_closed_forms():
    g = torch.Generator().manual_seed(4)
    T, d = 6, 5
    k = torch.randn(T, 1, d, generator=g, dtype=F64)
    # one token sees itself: its value is its key as projected, whatever the scores are
    out = pg.mixed_score_attention(torch.randn(T, 2, d, generator=g, dtype=F64), k, 3.0, torch.randn(2, 2, generator=g, dtype=F64), 1e-5)
    assert (out[0, 0] - k[0, 0]).abs().max() < 1e-12 and (out[0, 1] - k[0, 0]).abs().max() < 1e-12
    # a mix of zeros: every visible key weighs the same
    out = pg.mixed_score_attention(torch.randn(T, 2, d, generator=g, dtype=F64), k, 3.0, torch.zeros(2, 2, dtype=F64), 1e-5)
    assert (out[-1, 0] - k[:, 0].mean(0)).abs().max() < 1e-12
    # no content (scale 0), the identity as the mix: weights fall off by e^-slope a position
    out = pg.mixed_score_attention(torch.randn(T, 1, d, generator=g, dtype=F64), k, 0.0, torch.ones(1, 1, dtype=F64), 1e-5)
    w = torch.exp(-(2.0 ** -8) * torch.arange(T - 1, -1, -1, dtype=F64))
    assert (out[-1, 0] - (w[:, None] * k[:, 0]).sum(0) / w.sum()).abs().max() < 1e-12
    # a large key keeps its direction in the score and its length in the value
    k2 = k.clone()
    k2[2] *= 1000.0
    s1 = pg.biased_scores(pg.rms_unit(k, 1e-9).permute(1, 0, 2), pg.rms_unit(k, 1e-9).permute(1, 0, 2), 1.0)
    s2 = pg.biased_scores(pg.rms_unit(k, 1e-9).permute(1, 0, 2), pg.rms_unit(k2, 1e-9).permute(1, 0, 2), 1.0)
    assert (s1 - s2).abs().max() < 1e-6


def test_plain_rotation_routing_and_activation():
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0, 5.0]], dtype=F64)
    y = pg.rotate_pairs(x, torch.tensor([3]), 4, 100.0)
    f1 = 100.0 ** -0.5
    assert y[0].tolist() == pytest.approx([math.cos(3), math.sin(3), -2 * math.sin(3 * f1), 2 * math.cos(3 * f1), 5.0])
    ids, w = pg.choose_experts(torch.tensor([[0.5, 2.0, 2.0, -1.0], [3.0, 0.0, 1.0, 1.0]], dtype=F64), 2)
    assert ids.tolist() == [[1, 2], [0, 2]] and w[0].tolist() == pytest.approx([0.5, 0.5])
    assert float(w[1, 0] / w[1, 1]) == pytest.approx(math.exp(2.0))
    g, u = torch.tensor([3.0, -2.0], dtype=F64), torch.tensor([-4.0, 0.25], dtype=F64)
    out = pg.clamped_glu(g, u, 1.5)
    assert out.tolist() == pytest.approx([1.5 / (1 + math.exp(-1.702 * 1.5)) * -0.5, -2.0 / (1 + math.exp(1.702 * 2.0)) * 1.25])


def test_plain_run_order():
    base = {"layers": [None] * 4}
    assert pg.run_order(base) == [(0, False), (1, False), (2, False), (3, False)]
    assert pg.run_order(dict(base, loop={"start": 0, "stop": 4, "times": 1})) == [(0, True), (1, False), (2, False), (3, False)]
    assert pg.run_order(dict(base, loop={"start": 2, "stop": 3, "times": 2})) == [(0, False), (1, False), (2, True), (2, True), (3, False)]


def _in_halves(real):
    def rotate(x, positions, dims, base):
        h = dims // 2
        inter = torch.stack([x[..., :h], x[..., h:dims]], dim=-1).flatten(-2)         # pairs (i, i + h) side by side
        y = real(inter, positions, dims, base)
        return torch.cat([y[..., 0::2], y[..., 1::2], x[..., dims:]], dim=-1)
    return rotate


def _bias_behind_the_mix(real):
    def mix(talk, s):
        i = torch.arange(s.shape[-1], dtype=F64)
        bias = pg.distance_slopes(s.shape[0])[:, None, None] * (i[:, None] - i[None, :])
        return real(talk, s + bias) - bias
    return mix


# name of the mechanism's function in the plain implementation -> a wrong one made from it
MISTAKES = {
    "no distance bias": ("distance_slopes", lambda real: lambda H: real(H) * 0.0),
    "bias behind the mix": ("mix_heads", _bias_behind_the_mix),
    "heads not mixed": ("mix_heads", lambda real: lambda talk, s: s),
    "rotation in halves": ("rotate_pairs", _in_halves),
    "no rotation": ("rotate_pairs", lambda real: lambda x, p, dims, base: x),
    "norm weights not around zero": ("offset_norm", lambda real: lambda x, w, eps: real(x, w - 1.0, eps)),
    "up branch without the one": ("clamped_glu", lambda real: lambda g, u, limit: real(g, u - 1.0, limit)),
    "no clamp": ("clamped_glu", lambda real: lambda g, u, limit: real(g, u, 1e9)),
    "weights over all logits": ("choose_experts", lambda real: lambda z, top: (real(z, top)[0], torch.gather(torch.softmax(z, -1), 1, real(z, top)[0]))),
    "one pass less": ("run_order", lambda real: lambda c: real(dict(c, loop=dict(c["loop"], times=c["loop"]["times"] - 1)))),
    "reentry once": ("run_order", lambda real: lambda c: [(i, e and n == c["loop"]["start"]) for n, (i, e) in enumerate(real(c))]),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_random_models_show_mistakes(mistake, monkeypatch):
    """A mistake in any mechanism moves the logits of a random test model far beyond the float32 tolerance of the GPU tests."""
    from boring_llm_b200.weights.random_init import RandomTensors
    W = RandomTensors(build_model(GipinexConfig.from_dict(CFG)).tensor_specs(), 5, torch.bfloat16, 0.25)
    W = {k: W[k] for k in W}
    toks = [3, 70, 12, 12, 45, 8, 61, 0, 33, 29, 5, 17] * 3
    right = pg.forward(CFG, W, toks)
    name, make = MISTAKES[mistake]
    monkeypatch.setattr(pg, name, make(getattr(pg, name)))
    wrong = pg.forward(CFG, W, toks)
    assert (wrong - right).abs().max() > 50 * 1e-4 * right.abs().max()
