"""Zuvevik without a GPU: configuration keys and errors, declared tensors and caches, padded heads, the plain implementation
against closed forms, and mistakes planted in it that a random test model must show."""
import copy
import math

import pytest
import torch

import plain_zuvevik as pz
from boring_llm_b200 import ConfigError, ZuvevikConfig
from boring_llm_b200.cache import CacheManager, PagedKVSpec, StateSpec
from boring_llm_b200.models import build_model
from boring_llm_b200.parts import DecoderModel, GatedSinkAttention, HyperConnection, RMSNorm, RoutedExperts, RotaryTable
from boring_llm_b200.parts.attention import padded_head
from boring_llm_b200.weights import MIXING
from boring_llm_b200.weights.random_init import RandomTensors, random_tensor

F64 = torch.float64

ATT = {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.4, "rot": {"base": 700.0, "dims": 6}, "mask": {"size": 9}, "v_mix": True}
MOE = {"kind": "moe", "expert": {"ff": 12, "limit": 1.25}, "router": {"experts": 7, "top": 3}}
CFG = {"architecture": "Zuvevik", "vocab": 77, "width": 36, "norm": {"eps": 2e-5}, "streams": 4, "logit_scale": 0.7,
       "embedding": {"bigram": {"buckets": 31, "mul_prev": 1000003, "mul_cur": 53}}, "layers": [
           {"type": "attention", "mixer": dict(ATT, v_mix=False, kv_heads=2, vdim=8), "mlp": {"kind": "dense", "ff": 28}},
           {"type": "attention", "mixer": ATT, "mlp": MOE},
           {"type": "attention", "mixer": dict(ATT, heads=4, kv_heads=2, dim=40, vdim=21, rot={"base": 90.0, "dims": 40}), "mlp": None},
           {"type": "attention", "mixer": dict(ATT, mask={"size": 4}), "mlp": dict(MOE, router={"experts": 2, "top": 1})}]}


def test_config_round_trip_and_fields():
    cfg = ZuvevikConfig.from_dict(CFG)
    assert cfg.to_dict() == CFG
    assert (cfg.vocab_size, cfg.width, cfg.norm_eps, cfg.streams, cfg.logit_scale) == (77, 36, 2e-5, 4, 0.7)
    assert (cfg.pairs.buckets, cfg.pairs.mul_prev, cfg.pairs.mul_cur) == (31, 1000003, 53)
    m, f = cfg.layers[1].mixer, cfg.layers[1].mlp
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.rot_base, m.rot_dims, m.window, m.v_mix) == (6, 3, 10, 14, 0.4, 700.0, 6, 9, True)
    assert (f.ff, f.limit, f.experts, f.top) == (12, 1.25, 7, 3)
    assert cfg.layers[0].mlp.ff == 28 and cfg.layers[2].mlp is None
    assert cfg.value_mix_roles() == [None, "first", "follow", "follow"]
    none = ZuvevikConfig.from_dict(dict(CFG, layers=[{"type": "attention", "mixer": {k: v for k, v in ATT.items() if k not in ("mask", "v_mix")}}]))
    assert none.layers[0].mixer.window == 0 and none.value_mix_roles() == [None] and none.layers[0].mlp is None


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "gla", "unknown layer type"),
    (("layers", 0, "mixer", "kv_heads"), 4, "cannot share"),
    (("layers", 1, "mixer", "rot", "dims"), 5, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 12, "rot.dims"),
    (("layers", 1, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 1, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 2, "mixer", "vdim"), 20, "layers.2..mixer.v_mix"),
    (("layers", 1, "mlp", "router", "top"), 8, "out of 7"),
    (("layers", 1, "mlp", "expert", "limit"), 0.0, "limit"),
    (("layers", 0, "mlp", "kind"), "swiglu", "not supported"),
    (("embedding", "bigram", "buckets"), 0, "buckets"),
    (("embedding", "bigram", "mul_prev"), None, "mul_prev"),
    (("streams",), 0, "streams"),
    (("norm", "eps"), 0.0, "norm.eps"),
])
def test_config_errors_name_the_key(path, value, word):
    d = copy.deepcopy(CFG)
    at = d
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        ZuvevikConfig.from_dict(d)


def test_declared_tensors_and_caches():
    model = build_model(ZuvevikConfig.from_dict(CFG))
    specs = {k: tuple(v.shape) for k, v in model.tensor_specs().items()}
    assert specs["embed"] == specs["head"] == (77, 36) and specs["bigram"] == (32, 36) and specs["final.norm"] == (36,)
    assert specs["l1.mix.q"] == (60, 36) and specs["l1.mix.k"] == (30, 36) and specs["l1.mix.v"] == (42, 36) and specs["l1.mix.g"] == (84, 36)
    assert specs["l1.mix.o"] == (36, 84) and specs["l1.mix.q.norm"] == (60,) and specs["l1.mix.k.norm"] == (30,)
    assert specs["l2.mix.vmix"] == specs["l3.mix.vmix"] == ()
    assert "l0.mix.vmix" not in specs and "l1.mix.vmix" not in specs and {"l0.mix.vmix", "l1.mix.vmix"} <= set(model.ignorable_tensors)
    assert specs["l0.hc1.in"] == specs["l0.hc2.out"] == (4,) and specs["l0.hc1.mix"] == (4, 4)
    assert "l2.norm2" not in specs and "l2.hc2.mix" not in specs and {"l2.norm2", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix"} <= set(model.ignorable_tensors)
    assert specs["l1.mlp.e6.down"] == (36, 12) and specs["l3.mlp.router"] == (2, 36) and specs["l0.mlp.up"] == (28, 36)
    caches = model.cache_specs()
    assert caches == [PagedKVSpec(2, 16, 9), PagedKVSpec(3, 16, 9), PagedKVSpec(2, 48, 9), PagedKVSpec(3, 16, 4), StateSpec((1,), "int32")]
    assert model.embedding_cache == 4
    mgr = CacheManager(caches, 16, 128, 2)
    assert len(mgr.paged_groups) == 4 and mgr.state_groups[0].cache_layers == [4]
    assert model.final_norm.gain == 0.7


def test_heads_padded_to_one_built_size():
    assert [padded_head(*n) for n in ((1, 1), (16, 16), (10, 14), (40, 21), (21, 50), (64, 65), (128, 3))] == [16, 16, 16, 48, 64, 96, 128]
    assert padded_head(129, 4) == padded_head(4, 200) == 0           # no build holds them: they stay as they are
    part = GatedSinkAttention(6, 4, 2, 5, 7, RotaryTable(5, 10.0, n_rot=4), {k: k for k in ("wq", "wk", "wv", "wo", "wg", "q_norm", "k_norm")},
                              qk_norm="whole", out_gate="channel", pad_heads=True)
    g = torch.Generator().manual_seed(1)
    w = {k: torch.randn(*s.shape, generator=g) for k, s in part.local_specs().items()}
    part.load(w, torch.float32, "cpu")
    assert part.w_in.shape == ((4 + 2 + 2 + 4) * 16, 6) and part.wo.shape == (6, 64) and part.q_norm.shape == (64,)
    heads = part.w_in.view(12, 16, 6)
    assert torch.equal(heads[1, :5], w["wq"][5:10]) and torch.equal(heads[5, :5], w["wk"][5:]) and torch.equal(heads[7, :7], w["wv"][7:])
    assert torch.equal(heads[11, :7], w["wg"][21:]) and torch.equal(part.wo.view(6, 4, 16)[:, 2, :7], w["wo"][:, 14:21])
    assert not heads[:6, 5:].any() and not heads[6:, 7:].any() and not part.wo.view(6, 4, 16)[:, :, 7:].any() and not part.k_norm.view(2, 16)[:, 5:].any()
    off = GatedSinkAttention(6, 4, 2, 5, 7, None, {}, out_gate="channel")
    assert (off.pk, off.pv, off.n_in) == (5, 7, 20 + 10 + 14 + 28)


def test_parts_refuse_what_they_cannot_do():
    with pytest.raises(ValueError, match="streams"):
        HyperConnection(17, {})
    with pytest.raises(ValueError, match="weight_on"):
        RoutedExperts(8, 8, 4, 1, {}, weight_on="input", n_identity=1)
    with pytest.raises(ValueError, match="value_mix"):
        GatedSinkAttention(8, 2, 1, 4, None, None, {}, value_mix="second")
    model = build_model(ZuvevikConfig.from_dict(CFG))
    with pytest.raises(ValueError, match="several streams"):
        DecoderModel(model.embedding, model.blocks, model.final_norm, model.head, depth_mix=[None] * 4, streams=2)
    n = RMSNorm(2, 1e-5, {"weight": "w"}, gain=0.3)
    n.place({"weight": torch.tensor([2.0, -1.0]).bfloat16()}, torch.bfloat16, "cpu")
    assert n.weight.dtype == torch.float32 and n.weight.tolist() == pytest.approx([0.6, -0.3])


def test_random_mixing_matrices_are_around_the_identity():
    spec = build_model(ZuvevikConfig.from_dict(CFG)).tensor_specs()["l0.hc1.mix"]
    assert spec.kind == MIXING
    w = random_tensor("l0.hc1.mix", spec, 3, torch.float32, std=0.02)
    assert (w - torch.eye(4)).abs().max() < 0.1 and (w - torch.eye(4)).abs().min() > 0


# ---- the plain implementation against closed forms -----------------------------------------------------------------------
def test_plain_pair_rows():
    assert pz.pair_rows([5], 7, 3, 11).tolist() == [11]                       # no previous token: the last row
    assert pz.pair_rows([5, 2, 2], 7, 3, 11).tolist() == [11, (35 + 6) % 11, (14 + 6) % 11]
    assert pz.pair_rows([40000, 39999], 10 ** 12 + 39, 10 ** 11 + 3, 65521).tolist() == [65521, (40000 * (10 ** 12 + 39) + 39999 * (10 ** 11 + 3)) % 65521]
    table, pairs = torch.arange(12, dtype=F64).view(6, 2), 100.0 * torch.arange(8, dtype=F64).view(4, 2)
    x = pz.embed(torch.tensor([3, 1]), table, pairs, {"mul_prev": 2, "mul_cur": 5, "buckets": 3})
    assert x.tolist() == [[6.0 + 600.0, 7.0 + 700.0], [2.0 + 400.0, 3.0 + 500.0]]           # (2 * 3 + 5) mod 3 = 2


def test_plain_streams():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=F64)
    assert pz.read_streams(X, torch.tensor([2.0, -1.0], dtype=F64)).tolist() == [[-8.0, -16.0]]
    M = torch.tensor([[1.0, 3.0], [0.0, 0.5]], dtype=F64)                    # [from, to]: stream 0 goes to 0 once and to 1 three times
    out = pz.write_streams(X, M, torch.tensor([1.0, -2.0], dtype=F64), torch.tensor([[100.0, 0.0]], dtype=F64))
    assert out[0].tolist() == [[101.0, 2.0]] and out[1].tolist() == [[3.0 + 5.0 - 200.0, 6.0 + 10.0]]
    # one stream, ones everywhere: a plain residual
    x, y = torch.randn(1, 3, 4, dtype=F64), torch.randn(3, 4, dtype=F64)
    one = torch.ones(1, dtype=F64)
    assert torch.equal(pz.write_streams(x, one.view(1, 1), one, y)[0], x[0] + y)


def test_plain_rotation_window_and_values():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]], dtype=F64)
    y = pz.rotate_halves(x, torch.tensor([3]), 4, 100.0)[0, 0]
    f1 = 100.0 ** -0.5
    assert y.tolist() == pytest.approx([math.cos(3), -2 * math.sin(3 * f1), math.sin(3), 2 * math.cos(3 * f1), 5.0])
    assert pz.visible(4, 2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False], [False, False, True, True]]
    assert pz.visible(3, 0).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    g = torch.Generator().manual_seed(4)
    v = torch.randn(6, 2, 3, generator=g, dtype=F64)
    out = pz.attend(torch.zeros(6, 4, 5, dtype=F64), torch.randn(6, 2, 5, generator=g, dtype=F64), v, 1.0, 3)
    assert (out[5, 1] - v[3:, 0].mean(0)).abs().max() < 1e-12 and (out[5, 2] - v[3:, 1].mean(0)).abs().max() < 1e-12
    assert torch.equal(pz.attend(torch.randn(6, 4, 5, dtype=F64), torch.randn(6, 2, 5, dtype=F64), v, 1.0, 1), v.repeat_interleave(2, dim=1))
    a, b = torch.tensor([4.0], dtype=F64), torch.tensor([8.0], dtype=F64)
    assert pz.blend_values(a, b, torch.tensor(0.25, dtype=F64)).tolist() == [5.0]
    assert pz.channel_gate(torch.ones(1, 2, dtype=F64), torch.tensor([[1.0]], dtype=F64), torch.tensor([[0.0], [50.0]], dtype=F64))[0].tolist() == pytest.approx([0.5, 1.0])


def test_plain_routing_and_activation():
    ids, w = pz.choose_experts(torch.tensor([[0.5, 2.0, 2.0, -1.0], [-3.0, -9.0, -1.0, -1.0]], dtype=F64), 2)
    sig = lambda z: 1.0 / (1.0 + math.exp(-z))
    assert ids.tolist() == [[1, 2], [2, 3]] and w.flatten().tolist() == pytest.approx([sig(2.0), sig(2.0), sig(-1.0), sig(-1.0)])
    g, u = torch.tensor([3.0, -2.0], dtype=F64), torch.tensor([-4.0, 0.25], dtype=F64)
    assert pz.clamped_glu(g, u, 1.5).tolist() == pytest.approx([1.5 * sig(1.702 * 1.5) * -0.5, -2.0 * sig(-1.702 * 2.0) * 1.25])
    one = torch.ones(1, 1, dtype=F64)
    W = {"router": 0.0 * one, "e0.gate": one, "e0.up": one, "e0.down": one}
    out = pz.routed_experts(4.0 * one, W, {"router": {"top": 1}, "expert": {"limit": 9.0}})         # score 1/2: the expert reads 2
    assert float(out) == pytest.approx(2.0 * sig(1.702 * 2.0) * 3.0)
    assert float(pz.dense_ff(2.0 * one, {"gate": one, "up": one, "down": one})) == pytest.approx(2.0 * sig(2.0) * 2.0)


def _weight_behind(real):
    def routed(h, w, c, forced=None, info=None):
        ids, wts = pz.choose_experts(h @ w["router"].T, c["router"]["top"])
        return torch.stack([sum(p * pz.expert(h[t:t + 1], w, f"e{e}", c["expert"]["limit"])[0] for e, p in zip(ids[t].tolist(), wts[t]))
                            for t in range(h.shape[0])])
    return routed


def _per_head_norm(real):
    def norm(x, w, eps):
        if w.shape[0] in (60, 30):                        # a projection's norm: over each head of 10 instead of the whole row
            return real(x.view(x.shape[0], -1, 10), torch.ones(1, dtype=F64), eps).reshape(x.shape) * w
        return real(x, w, eps)
    return norm


# name of the mechanism's function in the plain implementation -> a wrong one made from it
MISTAKES = {
    "pairs the other way round": ("pair_rows", lambda real: lambda t, a, b, n: real(t, b, a, n)),
    "first token paired with token 0": ("pair_rows", lambda real: lambda t, a, b, n: torch.cat([torch.tensor([int(t[0]) * b % n]), real(t, a, b, n)[1:]])),
    "mix indexed [to, from]": ("write_streams", lambda real: lambda X, M, b, y: real(X, M.T, b, y)),
    "streams updated one after another": ("write_streams", lambda real: lambda X, M, b, y: _in_turn(X, M, b, y)),
    "plain sum read": ("read_streams", lambda real: lambda X, a: real(X, torch.ones_like(a))),
    "window one longer": ("visible", lambda real: lambda T, w: real(T, w + 1)),
    "window one shorter": ("visible", lambda real: lambda T, w: real(T, w - 1)),
    "no window": ("visible", lambda real: lambda T, w: real(T, 0)),
    "no rotation": ("rotate_halves", lambda real: lambda x, p, dims, base: x),
    "norms over heads": ("rms_norm", _per_head_norm),
    "values not blended": ("blend_values", lambda real: lambda v, f, lam: v),
    "blended the other way round": ("blend_values", lambda real: lambda v, f, lam: real(f, v, lam)),
    "no gate": ("channel_gate", lambda real: lambda o, h, wg: o),
    "weight on the result": ("routed_experts", _weight_behind),
    "weights renormalised": ("choose_experts", lambda real: lambda z, top: (real(z, top)[0], real(z, top)[1] / real(z, top)[1].sum(-1, keepdim=True))),
    "up branch without the one": ("clamped_glu", lambda real: lambda g, u, limit: real(g, u - 1.0, limit)),
    "no clamp": ("clamped_glu", lambda real: lambda g, u, limit: real(g, u, 1e9)),
}


def _in_turn(X, M, b, y):
    X = X.clone()
    for t in range(X.shape[0]):
        X[t] = torch.einsum("s,snd->nd", M[:, t], X) + b[t] * y
    return X


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_random_models_show_mistakes(mistake, monkeypatch):
    """A mistake in any mechanism moves the logits of a random test model far beyond the float32 tolerance of the GPU tests."""
    W = RandomTensors(build_model(ZuvevikConfig.from_dict(CFG)).tensor_specs(), 5, torch.bfloat16, 0.25)
    W = {k: W[k] for k in W}
    W["l2.mix.vmix"], W["l3.mix.vmix"] = torch.tensor(0.3), torch.tensor(-0.4)
    toks = [3, 70, 12, 12, 45, 8, 61, 0, 33, 29, 5, 17] * 3
    right = pz.forward(CFG, W, toks)
    name, make = MISTAKES[mistake]
    monkeypatch.setattr(pz, name, make(getattr(pz, name)))
    wrong = pz.forward(CFG, W, toks)
    assert (wrong - right).abs().max() > 50 * 1e-4 * right.abs().max()
