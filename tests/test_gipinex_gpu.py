"""The Gipinex decoder on the GPU against the plain float64 implementation in `plain_gipinex`: each mechanism alone through its
kernels and parts, then whole models of several small shapes through the runner (prompts whole, tails token by token,
portions down to two tokens, mixed batches with pages used again, long decoding), and greedy generation through `Engine`. The
test models are random; where random weights would hide a fault the inputs are made so that it shows."""
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import helpers
import plain_gipinex as pg
import plain_model as plain
from part_harness import run_portions, runner_for

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64
BF16_TOL = 6e-2


# ---- small shapes -----------------------------------------------------------------------------------------------------
def att(heads, kv, dim, scale):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, limit, experts, top, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


def layer(mixer, mlp=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, mult, layers, loop=None):
    d = {"architecture": "Gipinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


SHAPES = {
    # sizes in multiples of 8 (tensor cores in bfloat16); a loop in the middle (a layer before it, two after it), run three
    # times; a layer without feed-forward inside the loop; groups of three and of one head; both kinds of feed-forward behind
    # both kinds of mixer
    "A": model(101, 64, 1e-5, 0.6, [
        layer(att(6, 2, 24, 0.9), moe(24, 1.25, 5, 2, (40, 0.8))),
        layer(lat(3, 16, 8, 24, 24, 32), dense(48, 0.7)),
        layer(att(4, 4, 16, 1.3)),
        layer(lat(5, 8, 16, 8, 16, 48, base=500.0), moe(16, 0.5, 3, 1)),
        layer(att(3, 1, 40, 0.7), dense(40, 2.0))], loop=(1, 3, 3)),
    # sizes that are 1 or equal, and no multiple of 8 anywhere (plain kernels in both dtypes): one head, one pass, a multiplier
    # of one, one expert, every expert taken
    "B": model(61, 36, 1e-6, 1.0, [
        layer(att(1, 1, 6, 1.0), moe(12, 1.5, 2, 2, (12, 1.5))),
        layer(lat(1, 6, 4, 6, 6, 12, base=100.0), moe(20, 3.0, 1, 1)),
        layer(att(3, 3, 7, 0.8), dense(30, 1.0))], loop=(0, 1, 1)),
    # more heads than a block has rows in a decode step, several key/value heads to a row tile, no loop, a multiplier above one
    "D": model(83, 96, 1e-5, 1.7, [
        layer(att(35, 7, 8, 1.1), dense(64, 1.0)),
        layer(att(20, 5, 16, 1.4), moe(32, 1.0, 4, 3)),
        layer(lat(18, 8, 8, 16, 40, 72), moe(24, 0.75, 6, 2, (48, 1.0)))]),
    # head size 64 and 160 latent values: prompts of a few hundred tokens send the joined products through the tcgen05 kernels;
    # the whole model is the loop
    "C": model(300, 128, 1e-6, 0.4, [
        layer(lat(6, 64, 32, 40, 48, 160, base=500000.0), dense(256, 3.0)),
        layer(att(6, 3, 64, 0.5), moe(64, 1.5, 8, 2, (96, 2.5)))], loop=(0, 2, 2)),
}
SEEDS = {"A": 51, "B": 52, "C": 53, "D": 54}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from boring_llm_b200 import GipinexConfig, write_random_model
    made = {}

    def get(name, std=0.25):
        key = (name, std)
        if key not in made:
            d = str(tmp_path_factory.mktemp(f"gip_{name}"))
            write_random_model(d, GipinexConfig.from_dict(SHAPES[name]), SEEDS[name], "bfloat16", std)
            made[key] = d
        return made[key]
    return get


def std_for(dtype):
    return 0.25 if dtype == "float32" else 0.1


def plain_logits(folder, tokens):
    cfg, W = plain.read_model_folder(folder)
    return pg.forward(cfg, W, tokens).numpy()


def experts_of(block):
    from boring_llm_b200.parts import RoutedExperts, SumFeedForward
    f = block.ffn
    if isinstance(f, SumFeedForward):
        f = f.parts[0]
    return f if isinstance(f, RoutedExperts) else None


def run_recording(folder, dtype, steps, max_tokens, debug_poison=False):
    """`helpers.run_inprocess` with kernels launched singly, which also returns the experts every routed run chose:
    {place in the run order: {(request, position): experts}}. A block that several entries name records once per entry."""
    from boring_llm_b200.config import EngineOptions
    from boring_llm_b200.engine.runner import ModelRunner, StepEntry
    from boring_llm_b200.models import load_model
    _, mdl = load_model(folder, dtype, DEV)
    cap = -(-max_tokens // 16) * 16
    runner = ModelRunner(mdl, EngineOptions(dtype=dtype, page_size=16, max_tokens=cap, ctx_size=cap, max_num_seqs=8,
                                            cuda_graphs=False, debug_poison=debug_poison))
    parts = [experts_of(b) for b in mdl.blocks]
    for p in parts:
        if p is not None:
            p.record = []
    routed = [i for i, call in enumerate(mdl.schedule) if parts[call.block] is not None]
    outputs, chosen, at = {}, {i: {} for i in routed}, {}
    for s in steps:
        logits = runner.step([StepEntry(e["id"], e["tokens"], e["want"]) for e in s["entries"]])
        if logits.shape[0]:
            outputs[s["step"]] = logits.float().cpu().numpy()
        for i in routed:                                 # the entries of the run order recorded in order
            ids = parts[mdl.schedule[i].block].record.pop(0).cpu()
            t = 0
            for e in s["entries"]:
                for j in range(len(e["tokens"])):
                    chosen[i][(e["id"], at.get(e["id"], 0) + j)] = ids[t]
                    t += 1
        assert all(p is None or not p.record for p in parts)
        for e in s["entries"]:
            at[e["id"]] = at.get(e["id"], 0) + len(e["tokens"])
        for rid in s["end"]:
            runner.free_request(rid)
            at.pop(rid, None)
    runner.cache.check()
    return outputs, runner, chosen


def check_trace(folder, dtype, reqs, steps, max_tokens, what, **kw):
    """float32: the engine against the plain implementation, experts and all. bfloat16: rounding may turn a close choice
    between two experts the other way, so the plain implementation is told which experts the engine took, and the engine's
    choice must be the plain one wherever that is not close."""
    if dtype == "float32":
        outputs, runner = helpers.run_inprocess(folder, dtype, steps, max_tokens, **kw)
        chosen = None
    else:
        outputs, runner, chosen = run_recording(folder, dtype, steps, max_tokens, **kw)
    rows = helpers.collect_rows(steps, outputs)
    cfg, W = plain.read_model_folder(folder)
    errors, scale = [], 1e-6
    for rid, toks in reqs.items():
        forced = None if chosen is None else {i: torch.stack([c[(rid, p)] for p in range(len(toks))]) for i, c in chosen.items()}
        info = {}
        want = pg.forward(cfg, W, toks, forced=forced, info=info).numpy()
        got = np.stack([rows[(rid, p)] for p in range(len(toks))])
        assert np.isfinite(got).all(), f"{what} {rid}: non-finite logits"
        if dtype == "float32":
            helpers.assert_close(got, want, dtype, f"{what} {rid}")
            continue
        errors.append(np.abs(got - want).max(-1))
        scale = max(scale, np.abs(want).max())
        for i, rec in info.items():
            z = rec["logits"]
            gap = (torch.sort(z, dim=-1).values.diff(dim=-1).min(-1).values if z.shape[1] > 1 else torch.ones(z.shape[0], dtype=F64))
            same = (rec["own"].sort(-1).values == forced[i].long().sort(-1).values).all(-1)
            assert bool((same | (gap < 0.05 * z.abs().max())).all()), f"{what} {rid}: run {i} chose other experts where the choice is clear"
    if errors:
        e = np.concatenate(errors) / scale
        over = int((e > BF16_TOL).sum())
        assert over <= max(1, int(0.04 * e.size)), f"{what}: {over} of {e.size} positions differ by more than {BF16_TOL} (worst {e.max():.3f})"
        assert np.median(e) <= BF16_TOL / 4, f"{what}: median difference {np.median(e):.4f}"
    return runner


def solo_steps(reqs, cut):
    steps, n0 = [], 0
    for i, (rid, toks) in enumerate(reqs.items()):
        s = helpers.solo_trace(rid, toks, cut(toks, i), n0)
        steps += s
        n0 += len(s)
    return steps


# ---- whole models ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_whole_tails_singly_and_portions(folders, name, dtype):
    folder = folders(name, std_for(dtype))
    vocab = SHAPES[name]["vocab"]
    reqs = {f"r{i}": helpers.random_tokens(vocab, n, 100 + i) for i, n in enumerate([1, 2, 19, 75, 130])}
    check_trace(folder, dtype, reqs, solo_steps(reqs, lambda t, i: helpers.cut_whole(t)), 256, f"{name} whole")
    check_trace(folder, dtype, reqs, solo_steps(reqs, lambda t, i: helpers.cut_tail_singly(t, 45)), 256, f"{name} tail")
    check_trace(folder, dtype, reqs, solo_steps(reqs, lambda t, i: helpers.cut_varying(t, i)), 256, f"{name} portions")
    check_trace(folder, dtype, reqs, solo_steps(reqs, lambda t, i: [2] * (len(t) // 2) + [1] * (len(t) % 2)), 256, f"{name} pairs")


@pytest.mark.parametrize("name", ["A", "B", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reuse_pages(folders, name, dtype):
    folder = folders(name, std_for(dtype))
    vocab = SHAPES[name]["vocab"]
    reqs = {f"m{i}": helpers.random_tokens(vocab, n, 200 + i) for i, n in enumerate([33, 7, 90, 41, 2, 64, 17, 58])}
    steps, peak = helpers.mixed_trace(reqs, seed=5, max_live=3)
    runner = check_trace(folder, dtype, reqs, steps, peak, f"{name} mixed", debug_poison=True)
    assert all(hw <= runner.cache.num_pages for hw in runner.cache.stats()["pages_high_water"])
    # every run of a layer has a cache layer of its own
    assert sum(len(g.cache_layers) for g in runner.cache.paged_groups) == len(pg.run_order(SHAPES[name]))


def test_float32_does_not_depend_on_the_cut_or_the_batch(folders):
    folder = folders("A")
    reqs = {f"c{i}": helpers.random_tokens(101, n, 300 + i) for i, n in enumerate([50, 21, 77])}
    a, _ = helpers.run_inprocess(folder, "float32", solo_steps(reqs, lambda t, i: helpers.cut_whole(t)), 256)
    whole = helpers.collect_rows(solo_steps(reqs, lambda t, i: helpers.cut_whole(t)), a)
    steps, peak = helpers.mixed_trace(reqs, seed=9, max_live=3)
    b, _ = helpers.run_inprocess(folder, "float32", steps, peak)
    mixed = helpers.collect_rows(steps, b)
    for key, row in whole.items():
        assert np.abs(row - mixed[key]).max() <= 2e-5 * max(1.0, np.abs(row).max()), key


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    """300 tokens decoded one by one behind a prompt of 30, over page and key-block edges."""
    folder = folders("A", std_for(dtype))
    toks = helpers.random_tokens(101, 330, 7)
    check_trace(folder, dtype, {"long": toks}, helpers.solo_trace("long", toks, [30] + [1] * 300), 384, "long decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_shape_on_the_tensor_core_kernels(folders, dtype):
    """Prompts of 300 and 90 tokens: in bfloat16 the products run on tcgen05 and decode steps replay captured graphs."""
    folder = folders("C", 0.25 if dtype == "float32" else 0.06)
    reqs = {"w0": helpers.random_tokens(300, 300, 1), "w1": helpers.random_tokens(300, 90, 2)}
    steps = solo_steps(reqs, lambda t, i: helpers.cut_tail_singly(t, 24))
    check_trace(folder, dtype, reqs, steps, 512, "wide tail").check_kernels()
    steps, peak = helpers.mixed_trace(reqs, seed=3, max_live=2)
    check_trace(folder, dtype, reqs, steps, peak, "wide mixed").check_kernels()


@pytest.mark.parametrize("name", ["A", "D"])
def test_captured_steps_replay_the_same_bits(folders, name):
    folder = folders(name, 0.1)
    reqs = {f"g{i}": helpers.random_tokens(SHAPES[name]["vocab"], n, 400 + i) for i, n in enumerate([40, 23, 31])}
    steps, peak = helpers.mixed_trace(reqs, seed=4, max_live=3)
    twice = steps + [dict(s, step=s["step"] + len(steps)) for s in steps]
    out, runner = helpers.run_inprocess(folder, "bfloat16", twice, peak, step_graph_after=1)
    assert runner.graph_steps > 0
    single, _ = helpers.run_inprocess(folder, "bfloat16", steps, peak, cuda_graphs=False)
    for s in steps:
        if s["step"] in out:
            np.testing.assert_array_equal(out[s["step"]], out[s["step"] + len(steps)])
            np.testing.assert_allclose(out[s["step"]], single[s["step"]], atol=0.05 * np.abs(single[s["step"]]).max())


def test_greedy_generation_through_the_engine(folders):
    import boring_llm_b200 as b
    for name, dtype, std in (("A", "float32", 0.25), ("B", "float32", 0.25), ("A", "bfloat16", 0.1)):
        folder = folders(name, std)
        vocab = SHAPES[name]["vocab"]
        prompts = [helpers.random_tokens(vocab, n, 500 + n) for n in (5, 26, 61)]
        eng = b.Engine(folder, dtype=dtype, ctx_size=128, max_num_seqs=2, max_tokens=192, prefill_chunk=16)
        outs = eng.generate(prompts, n_predict=12, ignore_eos=True)
        for p, o in zip(prompts, outs):
            assert len(o) == 12
            logits = plain_logits(folder, p + o)
            for i, tok in enumerate(o):
                row = logits[len(p) - 1 + i]
                gap = row.max() - row[tok]
                assert gap <= (1e-4 if dtype == "float32" else 0.05) * np.abs(logits).max(), (name, i, gap)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_layer_streams_one_by_one(folders, name):
    """float32: the residual stream behind every entry of the run order (kept divided by the residual multiplier) against
    the plain implementation's."""
    from boring_llm_b200.config import EngineOptions
    from boring_llm_b200.engine.runner import ModelRunner, StepEntry
    from boring_llm_b200.models import load_model
    folder = folders(name)
    toks = helpers.random_tokens(SHAPES[name]["vocab"], 70, 3)
    cfg, W = plain.read_model_folder(folder)
    _, want = pg.forward(cfg, W, toks, streams=True)
    _, mdl = load_model(folder, "float32", DEV)
    runner = ModelRunner(mdl, EngineOptions(dtype="float32", max_tokens=128, ctx_size=128, max_num_seqs=2, cuda_graphs=False))
    mdl.keep_streams = []
    runner.step([StepEntry("s", toks, [])])
    assert len(mdl.keep_streams) == len(pg.run_order(cfg)) == len(want)
    for i, got in enumerate(mdl.keep_streams):
        w = want[i].numpy()
        assert np.abs(got.cpu().numpy() * cfg["residual_mult"] - w).max() <= 1e-4 * np.abs(w).max(), i


def test_passes_of_a_loop_keep_apart(folders):
    """Each pass reads the keys that the same pass of earlier tokens wrote. Two requests that differ in their first token only,
    decoded token by token, must match the plain implementation, in which every pass has keys of its own; and the cache layers
    of a layer's passes must differ."""
    from boring_llm_b200.config import EngineOptions
    from boring_llm_b200.engine.runner import ModelRunner, StepEntry
    from boring_llm_b200.models import load_model
    folder = folders("C")
    toks = helpers.random_tokens(300, 20, 11)
    reqs = {"p": toks, "q": [(toks[0] + 1) % 300] + toks[1:]}
    check_trace(folder, "float32", reqs, solo_steps(reqs, lambda t, i: [1] * len(t)), 64, "passes")
    _, mdl = load_model(folder, "float32", DEV)
    runner = ModelRunner(mdl, EngineOptions(dtype="float32", max_tokens=64, ctx_size=64, max_num_seqs=2, cuda_graphs=False))
    runner.step([StepEntry("p", toks, [])])
    passes = [c.cache for c in mdl.schedule if c.block == 1]
    assert len(passes) == 2
    a, b = (runner.storage.keys(c) for c in passes)
    assert bool((a != 0).any()) and not torch.equal(a, b)


# ---- mechanisms alone --------------------------------------------------------------------------------------------------
def rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g, dtype=F64) * scale


def dev(t, dtype=torch.float32):
    return t.to(dtype).to(DEV).contiguous()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def scattered_tables(lengths, seed):
    """A block table over scattered pages for requests of these lengths; (table, number of pages)."""
    n_pages = sum(-(-n // 16) for n in lengths) + 3
    order = torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
    table = torch.full((len(lengths), max(-(-n // 16) for n in lengths)), -1, dtype=torch.int32)
    for r, n in enumerate(lengths):
        for p in range(-(-n // 16)):
            table[r, p] = order.pop()
    return table, n_pages


@pytest.mark.parametrize("H,KV,dh", [(6, 2, 24), (1, 1, 6), (7, 7, 5), (14, 2, 64), (9, 3, 128)])
def test_mixed_queries_keys_and_their_root_mean_squares(H, KV, dh):
    from boring_llm_b200.kernels import ops
    eps, positions, reqs = 0.05, [37, 5, 16, 0, 15], [0, 1, 2, 2, 2]
    T = len(positions)
    off_k = -(-H * dh // 8) * 8
    proj = rnd(T, off_k + KV * dh + 5, seed=1, scale=2.0)
    proj[2, :H * dh] = 0.0                                         # a query of zeros stays zero
    talk = rnd(H, H, seed=2)
    table = i32([[4, 7, 2], [6, 1, 0], [3, 5, 8]])
    proj32 = dev(proj)
    p64 = proj32.double().cpu()
    q = pg.rms_unit(p64[:, :H * dh].view(T, H, dh), eps)
    G = H // KV
    want_q = torch.stack([torch.einsum("hg,tgd->thd", talk.float().double()[:, c * G:(c + 1) * G], q[:, c * G:(c + 1) * G]) for c in range(KV)], dim=2)
    k = p64[:, off_k:off_k + KV * dh].view(T, KV, dh)
    rms = torch.sqrt((k * k).mean(-1) + eps)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 8e-3)):
        q_out = torch.full((T, H, KV, dh), float("nan"), dtype=dtype, device=DEV)
        kc = torch.full((9, KV, 16, dh), float("nan"), dtype=dtype, device=DEV)
        kr = torch.full((9, KV, 16, 2), float("nan"), dtype=dtype, device=DEV)
        ops.mixed_prep(proj32, off_k, dev(talk), eps, i32(positions), i32(reqs), table, q_out, kc, kr)
        assert (q_out.double().cpu() - want_q).abs().max() <= tol * want_q.abs().max()
        nums = kr.view(torch.float32)[..., 0] if dtype == torch.bfloat16 else kr[..., 0]       # one 32-bit number either way
        for t, (pos, r) in enumerate(zip(positions, reqs)):
            page = int(table[r, pos // 16])
            got_r = nums[page, :, pos % 16].double().cpu()
            assert (got_r - rms[t]).abs().max() <= 1e-6 * rms.max()
            got = kc[page, :, pos % 16].double().cpu()
            assert (got - k[t] / rms[t][:, None]).abs().max() <= tol * 3
            assert (got * got_r[:, None] - k[t]).abs().max() <= tol * k.abs().max()            # the value is the key as projected
        assert int(torch.isfinite(kc.float()).all(-1).sum()) == T * KV                         # no other row was touched


def attention_case(H, KV, dh, seed):
    """Three requests in one step: a portion of 70 tokens behind 130 cached ones, a single token at position 149, a prompt of
    5 tokens. Keys are planted along the queries: the very first key, keys at a page's and a key block's edge, the token
    itself, and, twice as strongly, the key just behind the query, which must not be seen."""
    ctx, q_lens = [200, 150, 5], [70, 1, 5]
    keys = [rnd(n, KV, dh, seed=seed + r, scale=0.4) for r, n in enumerate(ctx)]
    rms = [rnd(n, KV, seed=seed + 20 + r).abs() + 0.3 for r, n in enumerate(ctx)]
    qs = []
    for r, (n, ql) in enumerate(zip(ctx, q_lens)):
        q = rnd(ql, H, KV, dh, seed=seed + 10 + r, scale=0.4)
        for t in range(ql):
            pos = n - ql + t
            a = (t * 5 + r) % dh
            for edge in (0, (pos // 16) * 16, max(0, (pos // 16) * 16 - 1), (pos // 64) * 64, max(0, (pos // 64) * 64 - 1), pos)[t % 6:t % 6 + 1]:
                q[t, :, :, a] += 5.0
                keys[r][edge, :, a] += 5.0
            if pos + 1 < n:
                keys[r][pos + 1, :, a] += 10.0
        qs.append(q)
    return ctx, q_lens, keys, rms, torch.cat(qs)


def attention_oracle(ctx, q_lens, keys, rms, q, scale, slopes, gate):
    out, t0 = [], 0
    H, KV, dh = q.shape[1:]
    for r, (n, ql) in enumerate(zip(ctx, q_lens)):
        s = torch.einsum("ihcd,jcd->hij", q[t0:t0 + ql], keys[r]) * scale
        i = torch.arange(n - ql, n, dtype=F64)[:, None]
        j = torch.arange(n, dtype=F64)[None, :]
        s = s - slopes[:, None, None] * (i - j)
        p = torch.softmax(s.masked_fill((j > i)[None], float("-inf")), dim=-1)
        v = (keys[r] * rms[r][:, :, None]).repeat_interleave(H // KV, dim=1)
        o = torch.einsum("hij,jhd->ihd", p, v).reshape(ql, H * dh)
        out.append(o * torch.sigmoid(gate[t0:t0 + ql]) if gate is not None else o)
        t0 += ql
    return torch.cat(out)


@pytest.mark.parametrize("H,KV,dh", [(6, 2, 24), (4, 4, 16), (1, 1, 64), (14, 2, 64), (35, 7, 8), (12, 3, 128), (16, 8, 128), (5, 1, 88), (3, 3, 7)])
def test_attention_kernels(H, KV, dh):
    from boring_llm_b200.kernels import ops
    from boring_llm_b200.parts.attention import attention_plan
    scale = 0.5
    ctx, q_lens, keys, rms, q = attention_case(H, KV, dh, seed=H)
    slopes = rnd(H, seed=98, scale=0.05)                            # mixed slopes have either sign
    T = q.shape[0]
    gate = rnd(T, H * dh + 8, seed=97)
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    tok_req = i32([r for r, n in enumerate(q_lens) for _ in range(n)])
    table, n_pages = scattered_tables(ctx, 5)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        keys_d = [k.to(dtype).to(F64) for k in keys]                # the keys as the dtype stores them are the oracle's inputs as well
        rms_d = [x.float().double() for x in rms]
        q_d = q.to(dtype).to(F64)
        g32 = dev(gate)
        want = attention_oracle(ctx, q_lens, keys_d, rms_d, q_d, scale, slopes.float().double(), g32.double().cpu()[:, 8:])
        kc = torch.full((n_pages, KV, 16, dh), float("nan"), dtype=F64)
        kr = torch.full((n_pages, KV, 16), float("nan"), dtype=torch.float32)
        for r, n in enumerate(ctx):
            for j in range(n):
                kc[table[r, j // 16], :, j % 16] = keys_d[r][j]
                kr[table[r, j // 16], :, j % 16] = rms_d[r][j].float()
        kc = dev(kc, dtype)
        if dtype == torch.bfloat16:
            kr_pages = kr.to(DEV).view(torch.bfloat16).view(n_pages, KV, 16, 2)
        else:
            kr_pages = torch.stack([kr, torch.full_like(kr, float("nan"))], dim=-1).to(DEV).contiguous()
        out = torch.full((T, H * dh), float("nan"), dtype=dtype, device=DEV)
        sl, gt, tb = dev(slopes), g32[:, 8:], table.to(DEV)
        ops.attention_mixed_plain(dev(q_d, dtype), kc, kr_pages, tok_req, i32(cu), i32(ctx), tb, out, scale, sl, gt)
        err = (out.double().cpu() - want).abs().max().item()
        assert err <= tol * want.abs().max().item(), ("plain", dtype, err)
        if dtype != torch.bfloat16:
            continue
        supported = ops.attention_mixed_supported(dtype, KV, dh, 16)
        assert supported == (dh % 8 == 0)
        if not supported:
            continue
        plan = attention_plan(q_lens, ctx)
        tiles, singles = (torch.from_numpy(plan.arrays[k]).to(DEV) for k in ("tiles64", "singles"))
        for splits in (1, 2, 5, 16):                               # the single token's keys in one block, in slices, in more slices than key blocks
            out.fill_(float("nan"))
            ops.attention_mixed_prefill(dev(q_d, dtype), kc, kr_pages, i32(cu), i32(ctx), tb, tiles, out, scale, sl, gt)
            ops.attention_mixed_decode(dev(q_d, dtype), kc, kr_pages, i32(cu), i32(ctx), tb, singles, splits, out, scale, sl, gt)
            got = out.double().cpu()
            assert torch.isfinite(got).all()
            err = (got - want).abs().max().item()
            assert err <= tol * want.abs().max().item(), ("tensor cores", splits, err)
        # neither slopes nor a gate
        bare = attention_oracle(ctx, q_lens, keys_d, rms_d, q_d, scale, torch.zeros(H, dtype=F64), None)
        ops.attention_mixed_prefill(dev(q_d, dtype), kc, kr_pages, i32(cu), i32(ctx), tb, tiles, out, scale)
        ops.attention_mixed_decode(dev(q_d, dtype), kc, kr_pages, i32(cu), i32(ctx), tb, singles, 3, out, scale)
        assert (out.double().cpu() - bare).abs().max().item() <= tol * bare.abs().max().item()


CUTS = {"whole": [90], "single": [1] * 90, "portions": [2, 3, 17, 31, 2, 1, 1, 33], "page edges": [15, 1, 16, 1, 31, 1, 25]}


@pytest.mark.parametrize("cut", sorted(CUTS))
@pytest.mark.parametrize("H,KV,dh", [(6, 2, 24), (3, 3, 7)])
def test_mixed_score_attention_part(H, KV, dh, cut):
    """The part in the engine's step machinery, keys of very different lengths (a long key must weigh by its direction and
    count by its length), a distance bias, a far key that stands out for the last tokens; in float32, and in bfloat16."""
    from boring_llm_b200.parts import MixedScoreAttention, distance_slopes
    d, T, scale, eps = 40, 90, 2.5, 1e-3
    x = rnd(T, d, seed=1)
    x[1] *= 30.0
    x[T - 4:] = x[3] * 0.5 + x[T - 4:] * 0.05                      # the last tokens look for token 3
    w = {"wq": rnd(H * dh, d, seed=2, scale=0.3), "wk": rnd(KV * dh, d, seed=3, scale=0.3), "talk": rnd(H, H, seed=4, scale=0.7),
         "wg": rnd(H * dh, d, seed=5, scale=0.3), "wo": rnd(d, H * dh, seed=6, scale=0.3)}
    for g in range(H):                                             # queries that look along the keys
        w["wq"][g * dh:(g + 1) * dh] += w["wk"][(g // (H // KV)) * dh:(g // (H // KV) + 1) * dh]
    w = {k: v.bfloat16().double() for k, v in w.items()}
    xb = x.bfloat16().double()
    want = pg.attention_mixer(xb, {"q": w["wq"], "k": w["wk"], "talk": w["talk"], "g": w["wg"], "o": w["wo"]},
                              {"heads": H, "kv_heads": KV, "dim": dh, "scale": scale}, eps)
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 4e-2)):
        part = MixedScoreAttention(d, H, KV, dh, {k: k for k in w}, scale=scale, qk_norm_eps=eps, slopes=distance_slopes(H), out_gate=True)
        tdt = getattr(torch, dtype)
        part.load({k: v.bfloat16() for k, v in w.items()}, tdt, DEV)

        def body(ctx, h):
            out = torch.zeros((h.shape[0], d), dtype=torch.float32, device=DEV)
            part.forward(ctx, h, out, 0)
            return out
        runner = runner_for(dev(xb, tdt), body, [part.cache_spec()], dtype=dtype)
        got = run_portions(runner, "r", T, CUTS[cut]).double().cpu()
        assert (got - want).abs().max() <= tol * want.abs().max(), (dtype, (got - want).abs().max())


@pytest.mark.parametrize("cut", ["whole", "single", "portions"])
@pytest.mark.parametrize("H,dn,dr,dv,qr,kr", [(3, 16, 8, 24, 24, 32), (2, 5, 6, 7, 9, 11)])
def test_latent_attention_part_with_interleaved_rotation_and_head_gates(H, dn, dr, dv, qr, kr, cut):
    from boring_llm_b200.parts import LatentAttention, RotaryTable
    d, T, scale, eps, base = 40, 90, 0.6, 1e-3, 300.0
    x = rnd(T, d, seed=1).bfloat16().double()
    w = {"wdq": rnd(qr, d, seed=2, scale=0.3), "wuq": rnd(H * (dn + dr), qr, seed=3, scale=0.6), "wdkv": rnd(kr + dr, d, seed=4, scale=0.4),
         "wuk": rnd(H * dn, kr, seed=5, scale=0.5), "wuv": rnd(H * dv, kr, seed=6, scale=0.4), "wg": rnd(H, d, seed=7, scale=0.4),
         "wo": rnd(d, H * dv, seed=8, scale=0.3), "dq_norm": rnd(qr, seed=9) * 0.1 + 1.0, "dkv_norm": rnd(kr, seed=10) * 0.1 + 1.0}
    w = {k: v.bfloat16().double() for k, v in w.items()}
    names = {"wdq": "dq", "wuq": "uq", "wdkv": "dkv", "wuk": "uk", "wuv": "uv", "wg": "g", "wo": "o", "dq_norm": "dq.norm", "dkv_norm": "dkv.norm"}
    want = pg.latent_attention_mixer(x, {names[k]: v for k, v in w.items()},
                                     {"heads": H, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": kr, "scale": scale,
                                      "rot": {"base": base, "dims": dr}}, eps, torch.arange(T))
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 4e-2)):
        part = LatentAttention(d, H, dn, dr, dv, qr, kr, RotaryTable(dr, base, pairs="interleaved"), {k: k for k in w}, scale=scale,
                               norm_eps=eps, out_gate="head")
        tdt = getattr(torch, dtype)
        part.load({k: v.bfloat16() for k, v in w.items()}, tdt, DEV)

        def body(ctx, h):
            out = torch.zeros((h.shape[0], d), dtype=torch.float32, device=DEV)
            part.forward(ctx, h, out, 0)
            return out
        runner = runner_for(dev(x, tdt), body, [part.cache_spec()], dtype=dtype)
        got = run_portions(runner, "r", T, CUTS[cut]).double().cpu()
        assert (got - want).abs().max() <= tol * want.abs().max(), (dtype, (got - want).abs().max())


def test_biases_in_the_gated_and_the_residual_epilogue_of_every_product():
    """Every kernel the row count can send a product to, with and without vectorised stores, and the products that begin the
    next norm while they add."""
    from boring_llm_b200.kernels import ops
    K, limit, seen = 256, 0.7, set()
    for N in (192, 198):
        for M in (3, 16, 40, 130, 600):
            x = rnd(M, K, seed=M, scale=0.5).bfloat16().double()
            w = rnd(2 * N, K, seed=M + 1, scale=0.2).bfloat16().double()
            b = rnd(2 * N, seed=M + 2).bfloat16().double()
            sums = x @ w.T + b
            g, u = sums[:, :N], sums[:, N:]
            res = rnd(M, N, seed=M + 3).float().double()
            for dtype, tol in ((torch.bfloat16, 2e-2), (torch.float32, 1e-5)):
                for kind, want in ((ops.GLU_CLAMPED, pg.clamped_glu(g, u, limit)), (ops.GLU_SILU, g * torch.sigmoid(g) * u)):
                    args = ops.glu_args(kind, limit, DEV, dev(b[:N], torch.bfloat16), dev(b[N:], torch.bfloat16))
                    out = torch.full((M, N), float("nan"), dtype=dtype, device=DEV)
                    seen.add(ops.gemm_kernel(dev(x, dtype), dev(w, dtype), N, args, ops.EPI_SWIGLU))
                    ops.gemm(dev(x, dtype), dev(w, dtype), out, args, ops.EPI_SWIGLU)
                    assert (out.double().cpu() - want).abs().max() <= tol * max(1.0, want.abs().max().item()), (kind, M, N, dtype)
                stream = dev(res)
                bias = dev(b[:N], torch.bfloat16)
                seen.add(ops.gemm_kernel(dev(x, dtype), dev(w[:N], dtype), N, bias, ops.EPI_RESIDUAL))
                ops.gemm(dev(x, dtype), dev(w[:N], dtype), stream, bias, ops.EPI_RESIDUAL)
                want = res + sums[:, :N]
                assert (stream.double().cpu() - want).abs().max() <= 1e-4 * want.abs().max(), (M, N, dtype)
            if N % 8 == 0 and M in (3, 600):
                fn = ops.gemm_skinny_residual_norm if M == 3 else ops.gemm_residual_norm
                stream, nw = dev(res), dev(rnd(N, seed=5) + 1.0)
                hw, ss = fn(dev(x, torch.bfloat16), dev(w[:N], torch.bfloat16), stream, nw, dev(b[:N], torch.bfloat16))
                assert (stream.double().cpu() - want).abs().max() <= 1e-4 * want.abs().max()
                assert (ss.double().cpu().sum(1) - (want * want).sum(1)).abs().max() <= 1e-3 * (want * want).sum(1).max()
                assert (hw.double().cpu() - want * nw.double().cpu()).abs().max() <= 1e-2 * want.abs().max()
    K = 4096                                                       # a long K: the kernel that cuts it among a cluster's blocks
    x, w = rnd(100, K, seed=1, scale=0.3).bfloat16().double(), rnd(192, K, seed=2, scale=0.1).bfloat16().double()
    b, res = rnd(192, seed=3).bfloat16().double(), rnd(100, 192, seed=4).float().double()
    stream = dev(res)
    seen.add(ops.gemm_kernel(dev(x, torch.bfloat16), dev(w, torch.bfloat16), 192, dev(b), ops.EPI_RESIDUAL))
    ops.gemm(dev(x, torch.bfloat16), dev(w, torch.bfloat16), stream, dev(b), ops.EPI_RESIDUAL)
    want = res + x @ w.T + b
    assert (stream.double().cpu() - want).abs().max() <= 1e-4 * want.abs().max()
    assert {"plain", "skinny", "tc", "pair", "splitk"} <= seen, seen


def test_dense_layer_with_biases():
    from boring_llm_b200.parts import GluMLP
    d, F, limit = 48, 56, 0.8
    x = rnd(20, d, seed=1).bfloat16().double()
    names = {"w_gate": "gate", "w_up": "up", "w_down": "down", "b_gate": "gate.b", "b_up": "up.b", "b_down": "down.b"}
    w = {"gate": rnd(F, d, seed=2, scale=0.3), "up": rnd(F, d, seed=3, scale=0.3), "down": rnd(d, F, seed=4, scale=0.3),
         "gate.b": rnd(F, seed=5), "up.b": rnd(F, seed=6), "down.b": rnd(d, seed=7)}
    w = {k: v.bfloat16().double() for k, v in w.items()}
    want = pg.dense_ff(x, w, limit)
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 2e-2)):
        tdt = getattr(torch, dtype)
        part = GluMLP(d, F, names, activation="clamped", limit=limit, bias=True)
        part.load({k: v.bfloat16() for k, v in w.items()}, tdt, DEV)
        for how in ("add", "write"):
            def body(ctx, h):
                out = torch.ones((h.shape[0], d), dtype=torch.float32, device=DEV)
                (part.forward if how == "add" else part.apply)(ctx, h, out)
                return out
            got = run_portions(runner_for(dev(x, tdt), body, [], dtype=dtype), "r", 20, [20]).double().cpu()
            assert (got - want - (1.0 if how == "add" else 0.0)).abs().max() <= tol * want.abs().max(), (dtype, how)


def test_routing_by_the_chosen_logits():
    from boring_llm_b200.kernels import ops
    for E, top in ((16, 4), (5, 1), (3, 3), (40, 7)):
        z = rnd(30, E, seed=E, scale=3.0)
        z[0] += 500.0                                              # weights only depend on differences
        z[1, :] = 0.0                                              # ties: the lower indices
        z32 = dev(z)
        ids = torch.empty((30, top), dtype=torch.int32, device=DEV)
        wts = torch.empty((30, top), dtype=torch.float32, device=DEV)
        ops.moe_route(z32, None, top, 1, 1, ids, wts, ops.SCORE_CHOSEN, 2)
        want_ids, want_w = pg.choose_experts(z32.double().cpu(), top)
        assert torch.equal(ids.cpu().long(), want_ids)
        assert (wts.double().cpu() - want_w).abs().max() <= 1e-6


def test_routed_experts_with_a_router_bias_and_a_shared_expert():
    from boring_llm_b200.parts import GluMLP, RoutedExperts, SumFeedForward
    d, F, E, top = 40, 24, 6, 2
    c = {"expert": {"limit": 0.6}, "router": {"experts": E, "top": top}, "shared": {"limit": 1.1}}
    w = {"router": rnd(E, d, seed=1), "router.b": rnd(E, seed=2, scale=6.0)}                      # the bias decides most choices
    for e in range(E):
        w.update({f"e{e}.gate": rnd(F, d, seed=10 + e, scale=0.3), f"e{e}.up": rnd(F, d, seed=30 + e, scale=0.3),
                  f"e{e}.down": rnd(d, F, seed=50 + e, scale=0.3)})
    w.update({"shared.gate": rnd(32, d, seed=70, scale=0.3), "shared.up": rnd(32, d, seed=71, scale=0.3), "shared.down": rnd(d, 32, seed=72, scale=0.3)})
    w = {k: v.bfloat16().double() for k, v in w.items()}
    x = rnd(30, d, seed=3).bfloat16().double()
    want = pg.routed_experts(x, w, c)
    names = {"router": "router", "router_bias": "router.b"}
    for e in range(E):
        names.update({f"gate{e}": f"e{e}.gate", f"up{e}": f"e{e}.up", f"down{e}": f"e{e}.down"})
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 2e-2)):
        tdt = getattr(torch, dtype)
        part = SumFeedForward([RoutedExperts(d, F, E, top, names, correction=False, activation="clamped", limit=0.6, score="chosen", router_bias=True),
                               GluMLP(d, 32, {"w_gate": "shared.gate", "w_up": "shared.up", "w_down": "shared.down"}, activation="clamped", limit=1.1)])
        part.load({k: v.bfloat16() for k, v in w.items()}, tdt, DEV)

        def body(ctx, h):
            out = torch.zeros((h.shape[0], d), dtype=torch.float32, device=DEV)
            part.forward(ctx, h, out)
            return out
        got = run_portions(runner_for(dev(x, tdt), body, [], dtype=dtype), "r", 30, [13, 1, 16]).double().cpu()
        assert (got - want).abs().max() <= tol * want.abs().max(), dtype


def test_norm_around_zero_and_the_reentry():
    from boring_llm_b200.kernels import ops
    from boring_llm_b200.parts import RMSNorm, StreamReentry
    for d in (36, 40):
        x, x0 = rnd(9, d, seed=1, scale=3.0).float().double(), rnd(9, d, seed=2).float().double()
        nw, w = rnd(d, seed=3, scale=0.2).bfloat16().double(), rnd(d, 2 * d, seed=4, scale=0.2).bfloat16().double()
        for dtype, tol in (("float32", 1e-5), ("bfloat16", 1e-2)):
            tdt = getattr(torch, dtype)
            both = torch.empty((9, 2 * d), dtype=tdt, device=DEV)
            ops.concat_rows(dev(x), dev(x0), both)
            assert torch.equal(both.cpu(), torch.cat([x, x0], dim=1).to(tdt))
            n = RMSNorm(d, 0.01, {"weight": "n"}, around_zero=True)
            n.load({"n": nw.bfloat16()}, tdt, DEV)
            r = StreamReentry(d, {"weight": "w"})
            r.load({"w": w.bfloat16()}, tdt, DEV)
            x0_dev = dev(x0)

            def body(ctx, h):
                y = r.forward(ctx, dev(x), x0_dev)
                return torch.cat([y, n.forward(ctx, y).float()], dim=1)
            got = run_portions(runner_for(dev(x, tdt), body, [], dtype=dtype), "r", 9, [9]).double().cpu()
            want = torch.cat([x, x0], dim=1) @ w.T
            assert (got[:, :d] - want).abs().max() <= tol * want.abs().max()
            assert (got[:, d:] - pg.offset_norm(got[:, :d], nw, 0.01)).abs().max() <= tol * 4
            assert torch.equal(x0_dev.cpu().double(), x0)


def test_the_command_line_and_the_trace_program_on_a_model_folder(folders, tmp_path):
    """`bin/boring-llm` generates what the plain implementation's arg-max gives, and `bin/trace_run`, started as a user
    would start it, writes the logits of a mixed trace (float32, and bfloat16 on poisoned pools)."""
    folder = folders("A")
    exe = [sys.executable, os.path.join(helpers.ROOT, "bin", "boring-llm")]
    prompt = helpers.random_tokens(101, 9, 3)
    p = subprocess.run(exe + ["--model", folder, "--prompt-tokens", ",".join(map(str, prompt)), "--n-predict", "6", "--dtype", "f32",
                              "--ctx-size", "64", "--ignore-eos"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    toks = list(prompt)
    for _ in range(6):
        toks.append(int(plain_logits(folder, toks)[-1].argmax()))
    assert p.stdout.strip().splitlines()[-1] == "generated: " + ",".join(map(str, toks[9:]))
    reqs = {f"t{i}": helpers.random_tokens(101, n, 600 + i) for i, n in enumerate([30, 12, 45])}
    steps, peak = helpers.mixed_trace(reqs, seed=2, max_live=2)
    outputs = helpers.run_trace_program(folder, "float32", steps, peak, str(tmp_path / "out"), 101)
    rows = helpers.collect_rows(steps, outputs)
    for rid, t in reqs.items():
        helpers.assert_close(np.stack([rows[(rid, i)] for i in range(len(t))]), plain_logits(folder, t), "float32", rid)
    outputs = helpers.run_trace_program(folders("A", 0.1), "bfloat16", steps, peak, str(tmp_path / "out16"), 101, extra=["--poison"])
    rows = helpers.collect_rows(steps, outputs)
    for rid, t in reqs.items():
        got = np.stack([rows[(rid, i)] for i in range(len(t))])
        want = plain_logits(folders("A", 0.1), t)
        assert np.isfinite(got).all() and np.median(np.abs(got - want).max(-1)) <= BF16_TOL / 2 * np.abs(want).max(), rid
