"""The Zuvevik decoder on the GPU against the plain float64 implementation in `plain_zuvevik`: each mechanism alone through its
kernels and parts, then whole models of several small shapes through the runner (prompts whole, tails token by token,
portions down to two tokens, mixed batches with pages and slots used again, long decoding), and greedy generation through
`Engine`. The test models are random; where random weights would hide a fault the inputs are made so that it shows."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import helpers
import plain_model as plain
import plain_zuvevik as pz
from part_harness import run_portions, runner_for

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64
BF16_TOL = 6e-2


# ---- small shapes -----------------------------------------------------------------------------------------------------
def att(heads, kv, dim, vdim, window, scale, dims=None, base=10000.0, v_mix=True):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dim if dims is None else dims},
         "v_mix": v_mix}
    if window:
        d["mask"] = {"size": window}
    return d


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, limit, experts, top):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, streams, logit_scale, pairs, layers):
    return {"architecture": "Zuvevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "logit_scale": logit_scale,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))}, "layers": layers}


SHAPES = {
    # sizes in multiples of 8 (tensor cores in bfloat16), heads that are padded; a first layer that does not blend, values that
    # blend across different numbers of heads, a layer without feed-forward, windows of one page, less than one, several
    "A": model(101, 64, 1e-5, 4, 0.6, (97, 31, 7), [
        layer(att(6, 2, 24, 16, 16, 0.35, dims=16, v_mix=False), moe(24, 1.25, 5, 2)),
        layer(att(4, 2, 24, 40, 21, 0.3), dense(48)),
        layer(att(4, 4, 16, 20, 50, 0.4, dims=8, base=300.0)),
        layer(att(5, 1, 40, 80, 7, 0.2), moe(16, 0.5, 3, 1))]),
    # sizes that are 1 or equal, and no multiple of 4 anywhere: one stream, one head, one bucket, a window of the token alone, one
    # expert, every expert taken, a factor of one on the logits, a layer without a window
    "B": model(61, 38, 1e-6, 1, 1.0, (1, 5, 3), [
        layer(att(1, 1, 6, 6, 1, 1.0), moe(10, 1.5, 2, 2)),
        layer(att(3, 3, 7, 2, 0, 0.8, dims=6, base=100.0), moe(18, 3.0, 1, 1)),
        layer(att(2, 1, 10, 6, 5, 0.5, dims=0), dense(30))]),
    # five streams (more than the built kernels' four), more heads to a key/value head than a decode block has rows, heads too
    # wide to be padded, multipliers beyond 32 bits
    "D": model(83, 96, 1e-5, 5, 1.7, (1009, 10 ** 12 + 39, 10 ** 11 + 3), [
        layer(att(35, 1, 8, 8, 33, 1.1), dense(64)),
        layer(att(2, 1, 136, 8, 30, 0.3, dims=64), moe(32, 1.0, 4, 3)),
        layer(att(6, 3, 96, 48, 64, 0.2, v_mix=False), moe(24, 0.75, 6, 2))]),
    # head size 64 and 128 in the cache: prompts of a few hundred tokens run on the tcgen05 kernels, single tokens on the TMA-fed one
    "C": model(300, 128, 1e-6, 3, 0.25, (499, 1237, 611), [
        layer(att(6, 2, 64, 64, 150, 0.125), dense(256)),
        layer(att(4, 2, 80, 64, 129, 0.11, dims=32), moe(64, 1.5, 8, 2)),
        layer(att(6, 2, 50, 64, 20, 0.14), moe(64, 2.5, 4, 4))]),
}
SEEDS = {"A": 61, "B": 62, "C": 63, "D": 64}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """Random model folders; the learned numbers between the layers' values are set to ones that tell the layers apart."""
    from boring_llm_b200 import ZuvevikConfig
    from boring_llm_b200.models import build_model
    from boring_llm_b200.weights import write_model_folder
    from boring_llm_b200.weights.random_init import RandomTensors
    made = {}

    def get(name, std=0.25):
        key = (name, std)
        if key not in made:
            d = str(tmp_path_factory.mktemp(f"zuv_{name}"))
            cfg = ZuvevikConfig.from_dict(SHAPES[name])
            W = RandomTensors(build_model(cfg).tensor_specs(), SEEDS[name], torch.bfloat16, std)
            W = {k: W[k] for k in W}
            for i, k in enumerate(sorted(k for k in W if k.endswith("vmix"))):
                W[k] = torch.tensor([0.4, -0.3, 0.7][i % 3]).to(W[k].dtype)
            write_model_folder(d, cfg.to_dict(), W)
            made[key] = d
        return made[key]
    return get


def std_for(dtype):
    return 0.25 if dtype == "float32" else 0.1


def plain_logits(folder, tokens):
    cfg, W = plain.read_model_folder(folder)
    return pz.forward(cfg, W, tokens).numpy()


def experts_of(block):
    from boring_llm_b200.parts import RoutedExperts
    return block.ffn if isinstance(block.ffn, RoutedExperts) else None


def run_recording(folder, dtype, steps, max_tokens, debug_poison=False):
    """`helpers.run_inprocess` with kernels launched singly, which also returns the experts every routed run chose:
    {layer: {(request, position): experts}}."""
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
        want = pz.forward(cfg, W, toks, forced=forced, info=info).numpy()
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
def test_mixed_batches_reuse_pages_and_slots(folders, name, dtype):
    folder = folders(name, std_for(dtype))
    vocab = SHAPES[name]["vocab"]
    reqs = {f"m{i}": helpers.random_tokens(vocab, n, 200 + i) for i, n in enumerate([33, 7, 90, 41, 2, 64, 17, 58])}
    steps, peak = helpers.mixed_trace(reqs, seed=5, max_live=3)
    runner = check_trace(folder, dtype, reqs, steps, peak, f"{name} mixed", debug_poison=True)
    assert all(hw <= runner.cache.num_pages for hw in runner.cache.stats()["pages_high_water"])


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
    """300 tokens decoded one by one behind a prompt of 30, over page and window edges, pages given back on the way."""
    folder = folders("A", std_for(dtype))
    toks = helpers.random_tokens(101, 330, 7)
    check_trace(folder, dtype, {"long": toks}, helpers.solo_trace("long", toks, [30] + [1] * 300), 384, "long decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_shape_on_the_tensor_core_kernels(folders, dtype):
    """Prompts of 300 and 90 tokens: in bfloat16 products and attention run on tcgen05."""
    folder = folders("C", 0.25 if dtype == "float32" else 0.06)
    reqs = {"w0": helpers.random_tokens(300, 300, 1), "w1": helpers.random_tokens(300, 90, 2)}
    steps = solo_steps(reqs, lambda t, i: helpers.cut_tail_singly(t, 24))
    check_trace(folder, dtype, reqs, steps, 512, "wide tail").check_kernels()
    steps, peak = helpers.mixed_trace(reqs, seed=3, max_live=2)
    check_trace(folder, dtype, reqs, steps, peak, "wide mixed").check_kernels()


@pytest.mark.parametrize("name", ["A", "C"])
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


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_stream_sums_layer_by_layer(folders, name):
    """float32: the sum of the streams behind every layer against the plain implementation's."""
    from boring_llm_b200.config import EngineOptions
    from boring_llm_b200.engine.runner import ModelRunner, StepEntry
    from boring_llm_b200.models import load_model
    folder = folders(name)
    toks = helpers.random_tokens(SHAPES[name]["vocab"], 70, 3)
    cfg, W = plain.read_model_folder(folder)
    _, want = pz.forward(cfg, W, toks, streams=True)
    _, mdl = load_model(folder, "float32", DEV)
    runner = ModelRunner(mdl, EngineOptions(dtype="float32", max_tokens=128, ctx_size=128, max_num_seqs=2, cuda_graphs=False))
    mdl.keep_streams = []
    runner.step([StepEntry("s", toks, [])])
    assert len(mdl.keep_streams) == len(want)
    for i, got in enumerate(mdl.keep_streams):
        w = want[i].numpy()
        assert np.abs(got.cpu().numpy() - w).max() <= 1e-4 * np.abs(w).max(), i


def test_a_slot_used_again_starts_without_a_previous_token(folders):
    """Requests one after another in the same slot: the first token of each takes the row for sequences' beginnings."""
    folder = folders("A")
    reqs = {f"s{i}": helpers.random_tokens(101, n, 700 + i) for i, n in enumerate([9, 1, 5, 1, 12])}
    check_trace(folder, "float32", reqs, solo_steps(reqs, lambda t, i: [1] * len(t)), 64, "one slot")
    from boring_llm_b200.engine.runner import StepError
    from boring_llm_b200.config import EngineOptions
    from boring_llm_b200.engine.runner import ModelRunner, StepEntry
    from boring_llm_b200.models import load_model
    _, mdl = load_model(folder, "float32", DEV)
    runner = ModelRunner(mdl, EngineOptions(dtype="float32", max_tokens=64, ctx_size=64, max_num_seqs=1, cuda_graphs=False))
    runner.step([StepEntry("x", [5, 6, 7], [])])
    with pytest.raises(StepError):                               # the previous token is state: a cut-back request is computed again
        runner.truncate("x", 2)


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


@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("d", [40, 1300, 37])
def test_stream_pass(S, d):
    """`hyper_step` in every form: streams that are still equal, written beside themselves and in place, read with and without
    a norm, chosen rows, and a sublayer's result that lies in the rows of routed pairs."""
    from boring_llm_b200.kernels import ops
    T, eps = 7, 0.01
    X = rnd(S, T, d, seed=1).float().double()
    M, b, a = rnd(S, S, seed=2).float().double(), rnd(S, seed=3).float().double(), rnd(S, seed=4).float().double()
    y, w = rnd(T, d, seed=5).float().double(), rnd(d, seed=6).bfloat16().double()
    write, read = dev(torch.cat([b, M.reshape(-1)])), dev(a)
    new = pz.write_streams(X, M, b, y)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 8e-3)):
        h = torch.full((T, d), float("nan"), dtype=dtype, device=DEV)
        out = torch.full((S, T, d), float("nan"), device=DEV)
        want = pz.rms_norm(pz.read_streams(new, a), w, eps)
        ops.hyper_step(dev(X), S, x_out=out, write=write, y=dev(y), read=read, norm_w=dev(w, torch.bfloat16), eps=eps, h=h)
        assert (out.double().cpu() - new).abs().max() <= 1e-5 * new.abs().max()
        assert (h.double().cpu() - want).abs().max() <= tol * want.abs().max()
        x = dev(X)                                                 # in place
        ops.hyper_step(x, S, x_out=x, write=write, y=dev(y), read=read, norm_w=dev(w), eps=eps, h=h)
        assert torch.equal(x, out) and (h.double().cpu() - want).abs().max() <= tol * want.abs().max()
        ops.hyper_step(dev(X), S, read=read, norm_w=dev(w), eps=eps, h=h)                         # nothing to write back
        want = pz.rms_norm(pz.read_streams(X, a), w, eps)
        assert (h.double().cpu() - want).abs().max() <= tol * want.abs().max()
        equal = X[:1].repeat(S, 1, 1)                              # all streams equal, kept once
        ops.hyper_step(dev(X[0]), S, x_out=out, write=write, y=dev(y), read=read, norm_w=dev(w), eps=eps, h=h)
        new_e = pz.write_streams(equal, M, b, y)
        want = pz.rms_norm(pz.read_streams(new_e, a), w, eps)
        assert (out.double().cpu() - new_e).abs().max() <= 1e-5 * new_e.abs().max()
        assert (h.double().cpu() - want).abs().max() <= tol * want.abs().max()
        rows = [5, 0, 5]                                           # the end of a model: the sum, normed, of some rows; nothing stored
        few = torch.full((3, d), float("nan"), dtype=dtype, device=DEV)
        ops.hyper_step(dev(X), S, write=write, y=dev(y), norm_w=dev(w), eps=eps, h=few, row_idx=i32(rows))
        want = pz.rms_norm(new.sum(0), w, eps)[rows]
        assert (few.double().cpu() - want).abs().max() <= tol * want.abs().max()
        ops.hyper_step(dev(X), S, h=h)                             # the plain sum
        assert (h.double().cpu() - X.sum(0)).abs().max() <= tol * X.sum(0).abs().max()
    top = 3
    rows = rnd(T * top + 40, d, seed=7).float().double()
    pos = torch.randperm(T * top + 40, generator=torch.Generator().manual_seed(8))[:T * top].view(T, top)
    wts = rnd(T, top, seed=9).float().double()
    for y_pos, y_wts in ((pos, None), (pos, wts), (None, None), (None, wts)):
        src = rows[y_pos] if y_pos is not None else rows[:T * top].view(T, top, d)
        res = (src * (y_wts[:, :, None] if y_wts is not None else 1.0)).sum(1)
        out = torch.empty((S, T, d), device=DEV)
        ops.hyper_step(dev(X), S, x_out=out, write=write, y=dev(rows if y_pos is not None else rows[:T * top]),
                       y_pos=i32(y_pos.reshape(-1).tolist()) if y_pos is not None else None,
                       y_wts=dev(y_wts) if y_wts is not None else None, top=top)
        new = pz.write_streams(X, M, b, res)
        assert (out.double().cpu() - new).abs().max() <= 1e-5 * new.abs().max()


@pytest.mark.parametrize("cut", [[40], [1] * 40, [2, 3, 17, 1, 1, 16]])
def test_pair_embedding(cut):
    """Portions of every kind: a portion's first token is paired with the last of the portion before. Two requests share the
    batch, and the second one's slot is one that another request has left."""
    from boring_llm_b200.config import EngineOptions
    from boring_llm_b200.engine.runner import ModelRunner, StepEntry
    from boring_llm_b200.parts import PairEmbedding
    vocab, d, buckets, a, b = 50, 24, 13, 10 ** 12 + 39, 77
    table, pairs = rnd(vocab, d, seed=1).bfloat16(), rnd(buckets + 1, d, seed=2).bfloat16()
    for dtype in ("float32", "bfloat16"):
        part = PairEmbedding(vocab, d, buckets, a, b, {"table": "t", "pairs": "p"})
        part.load({"t": table, "p": pairs}, getattr(torch, dtype), DEV)

        class Probe:
            vocab_size = vocab

            def cache_specs(self):
                return [part.cache_spec()]

            def forward(self, ctx):
                return part.forward(ctx, None, 0)
        r = ModelRunner(Probe(), EngineOptions(dtype=dtype, max_tokens=256, ctx_size=64, max_num_seqs=2, cuda_graphs=False))
        r.step([StepEntry("gone", [7, 8, 9], [])])
        r.free_request("gone")
        toks = {"x": helpers.random_tokens(vocab, 40, 3), "y": helpers.random_tokens(vocab, 40, 4)}
        got = {k: [] for k in toks}
        at = 0
        for i, n in enumerate(cut):
            order = ["x", "y"] if i % 2 else ["y", "x"]
            out = r.step([StepEntry(k, toks[k][at:at + n], []) for k in order]).double().cpu()
            for j, k in enumerate(order):
                got[k].append(out[j * n:(j + 1) * n])
            at += n
        for k in toks:
            want = pz.embed(torch.tensor(toks[k]), table.double(), pairs.double(), {"mul_prev": a, "mul_cur": b, "buckets": buckets})
            assert (torch.cat(got[k]) - want).abs().max() <= 1e-6 * want.abs().max()


def attention_case(H, KV, dh, window, seed):
    """Four requests in one step: a portion of 70 tokens behind 180 cached ones, a single token at position 199, a prompt of 5
    tokens, a single token at position 300. Along each query one key is planted at the window's inner edge, the key just
    outside the window gets twice that, and so does the key just behind the query; neither may be seen."""
    ctx, q_lens = [250, 200, 5, 301], [70, 1, 5, 1]
    keys = [rnd(n, KV, dh, seed=seed + r, scale=0.3) for r, n in enumerate(ctx)]
    vals = [rnd(n, KV, dh, seed=seed + 30 + r) for r, n in enumerate(ctx)]
    qs = []
    for r, (n, ql) in enumerate(zip(ctx, q_lens)):
        q = rnd(ql, H, dh, seed=seed + 10 + r, scale=0.3)
        for t in range(ql):
            pos, a = n - ql + t, (t * 5 + r) % dh
            q[t, :, a] += 5.0
            inner = max(0, pos - window + 1) if window else 0
            keys[r][inner if t % 3 else pos, :, a] += 4.0
            if inner > 0:
                keys[r][inner - 1, :, a] += 8.0
            if pos + 1 < n:
                keys[r][pos + 1, :, a] += 8.0
        qs.append(q)
    return ctx, q_lens, keys, vals, torch.cat(qs)


def attention_oracle(ctx, q_lens, keys, vals, q, scale, window, gate):
    out, t0 = [], 0
    for r, (n, ql) in enumerate(zip(ctx, q_lens)):
        full = torch.cat([torch.zeros(n - ql, *q.shape[1:], dtype=F64), q[t0:t0 + ql]])
        o = pz.attend(full, keys[r], vals[r], scale, window)[n - ql:].reshape(ql, -1)
        out.append(o * torch.sigmoid(gate[t0:t0 + ql]))
        t0 += ql
    return torch.cat(out)


@pytest.mark.parametrize("window", [0, 1, 15, 16, 17, 63, 64, 65, 130])
@pytest.mark.parametrize("H,KV,dh", [(6, 2, 64), (4, 4, 128), (35, 1, 16), (12, 3, 48), (3, 1, 96), (14, 2, 32), (5, 5, 7)])
def test_a_gate_per_channel_in_every_attention_kernel(H, KV, dh, window):
    from boring_llm_b200.kernels import ops
    from boring_llm_b200.parts.attention import attention_plan
    scale = 0.4
    ctx, q_lens, keys, vals, q = attention_case(H, KV, dh, window, seed=H)
    T = q.shape[0]
    gate = dev(rnd(T, H * dh + 8, seed=97, scale=2.0))
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    tok_req = i32([r for r, n in enumerate(q_lens) for _ in range(n)])
    table, n_pages = scattered_tables(ctx, 5)
    tb = table.to(DEV)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        store = lambda x: [k.to(dtype).to(F64) for k in x]          # what the dtype stores is the oracle's input as well
        keys_d, vals_d, q_d = store(keys), store(vals), q.to(dtype).to(F64)
        want = attention_oracle(ctx, q_lens, keys_d, vals_d, q_d, scale, window, gate.double().cpu()[:, 8:])
        kc = torch.full((n_pages, KV, 16, dh), float("nan"), dtype=F64)
        vc = kc.clone()
        for r, n in enumerate(ctx):
            for j in range(n):
                kc[table[r, j // 16], :, j % 16] = keys_d[r][j]
                vc[table[r, j // 16], :, j % 16] = vals_d[r][j]
        kc, vc, qd, g = dev(kc, dtype), dev(vc, dtype), dev(q_d.reshape(T, -1), dtype), gate[:, 8:]
        out = torch.full((T, H * dh), float("nan"), dtype=dtype, device=DEV)

        def check(what):
            got = out.double().cpu()
            assert torch.isfinite(got).all(), what
            err = (got - want).abs().max().item()
            assert err <= tol * want.abs().max().item(), (what, dtype, err)
            out.fill_(float("nan"))
        ops.attention_plain(qd, kc, vc, tok_req, i32(cu), i32(ctx), tb, out, H, window, scale, None, g, gate_dim=dh)
        check("plain")
        if dtype != torch.bfloat16 or not ops.attention_mma_supported(dtype, dh, 16):
            continue
        plan = attention_plan(q_lens, ctx)
        tiles, singles = (torch.from_numpy(plan.arrays[k]).to(DEV) for k in ("tiles64", "singles"))
        tiles128 = i32([[0, 0], [2, 0]])
        args = (qd, kc, vc, i32(cu), i32(ctx), tb)
        for splits in (1, 3, 16):
            ops.attention_prefill(*args, tiles, out, H, window, scale, None, g, gate_dim=dh)
            ops.attention_decode(*args, singles, splits, out, H, window, scale, None, None, g, gate_dim=dh)
            check(f"mma, {splits} slices")
        scratch = torch.empty(ops.attention_decode_scratch(2, H, dh, 5), dtype=torch.float32, device=DEV)
        ops.attention_prefill(*args, tiles, out, H, window, scale, None, g, gate_dim=dh)
        ops.attention_decode(*args, singles, 5, out, H, window, scale, scratch, None, g, gate_dim=dh)
        check("mma, slices through memory")
        if ops.attention_prefill_tc_supported(dtype, dh, 16):
            for splits in (1, 2, 5):
                ops.attention_prefill_tc(*args, tiles128, out, H, window, scale, None, g, gate_dim=dh)
                ops.attention_decode_tma(*args, singles, splits, out, H, window, scale, None, g, gate_dim=dh)
                check(f"tcgen05 and TMA, {splits} slices")
            ops.check_status()


def test_a_channel_gate_that_does_not_fit_is_refused():
    from boring_llm_b200.kernels import ops
    kc = torch.zeros((2, 1, 16, 64), dtype=torch.bfloat16, device=DEV)
    q = torch.zeros((2, 64), dtype=torch.bfloat16, device=DEV)
    tiles = i32([[0, 0]])
    gate = torch.zeros((2, 66), device=DEV)
    for g, dim in ((gate[:, 1:65], 64), (gate[:, :64], 64), (gate[:, :64], 32)):       # off a 16-byte boundary, rows that are, another head size
        with pytest.raises(ops.KernelError):
            ops.attention_prefill(q, kc, kc, i32([0, 2]), i32([2]), i32([[0]]), tiles, q.clone(), 1, 0, 1.0, None, g, gate_dim=dim)


@pytest.mark.parametrize("pairs", ["halves", "interleaved"])
@pytest.mark.parametrize("H,KV,dk,dv,pk,pv,n_rot,first", [
    (6, 2, 24, 20, 32, 32, 16, (2, 20, 32)),       # padded heads, values of the same layout
    (4, 4, 16, 10, 16, 16, 16, (2, 20, 32)),       # ... of two heads of 20, 32 places apart
    (3, 3, 7, 5, 7, 5, 6, (5, 3, 4)),              # nothing is a multiple of four
    (5, 1, 8, 12, 8, 12, 4, None),
    (16, 2, 64, 64, 64, 64, 64, (2, 64, 64)),
    (16, 2, 128, 128, 128, 128, 0, (4, 64, 64)),
])
def test_norm_rotation_and_blended_values_into_the_pages(H, KV, dk, dv, pk, pv, n_rot, first, pairs):
    from boring_llm_b200.kernels import ops
    from boring_llm_b200.parts import RotaryTable
    from plain_gipinex import rotate_pairs
    eps, base, lam = 0.05, 500.0, 0.375
    positions, reqs = [37, 5, 16, 0, 15], [0, 1, 2, 2, 2]
    T = len(positions)
    table = i32([[4, 7, 2], [6, 1, 0], [3, 5, 8]])

    def padded(x, places):                                          # [T, heads, n] -> [T, heads * places]
        return torch.cat([x, torch.zeros(T, x.shape[1], places - x.shape[2], dtype=F64)], dim=2).reshape(T, -1)
    q, k, v = (rnd(T, h, n, seed=s).float().double() for h, n, s in ((H, dk, 1), (KV, dk, 2), (KV, dv, 3)))
    proj = dev(torch.cat([padded(q, pk), padded(k, pk), padded(v, pv), rnd(T, 8, seed=4)], dim=1))
    qw, kw = rnd(H * dk, seed=5).bfloat16().double(), rnd(KV * dk, seed=6).bfloat16().double()
    place_w = lambda w, heads: torch.cat([w.view(heads, dk), torch.zeros(heads, pk - dk, dtype=F64)], dim=1).reshape(-1)
    rot = RotaryTable(pk, base, n_rot=n_rot, pairs=pairs).to(DEV)

    def turned(x, w, heads):
        y = pz.rms_norm(x.reshape(T, -1), w, eps).view(T, heads, dk)
        if n_rot == 0:
            return y
        if pairs == "halves":
            return pz.rotate_halves(y, torch.tensor(positions), n_rot, base)
        return rotate_pairs(y.permute(1, 0, 2), torch.tensor(positions), n_rot, base).permute(1, 0, 2)
    want_q, want_k, want_v, blend = turned(q, qw, H), turned(k, kw, KV), v, None
    if first is not None:
        heads1, dv1, places1 = first
        v1 = rnd(T, heads1, dv1, seed=7).float().double()
        rows = dev(torch.cat([rnd(T, 8, seed=8), padded(v1, places1), rnd(T, 4, seed=9)], dim=1))[:, 8:]
        blend = (rows, dv1, places1, dv, dev(torch.tensor([lam])))
        want_v = pz.blend_values(v.reshape(T, -1), v1.reshape(T, -1), lam).view(T, KV, dv)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 8e-3)):
        qo = torch.full((T, H * pk), float("nan"), dtype=dtype, device=DEV)
        kc = torch.full((9, KV, 16, pk), float("nan"), dtype=dtype, device=DEV)
        vc = torch.full((9, KV, 16, pv), float("nan"), dtype=dtype, device=DEV)
        ops.qk_norm_rope_write(proj, H * pk, (H + KV) * pk, dev(place_w(qw, H), torch.bfloat16), dev(place_w(kw, KV), torch.bfloat16), eps,
                               i32(positions), i32(reqs), table, rot.inv_freq, n_rot // 2, rot.pair_layout, qo, kc, vc, H, KV, pk, pv,
                               norm_q=H * dk if pk != dk else 0, norm_k=KV * dk if pk != dk else 0, blend=blend)
        got = qo.double().cpu().view(T, H, pk)
        assert (got[:, :, :dk] - want_q).abs().max() <= tol * want_q.abs().max() and not got[:, :, dk:].any()
        for t, (pos, r) in enumerate(zip(positions, reqs)):
            page = int(table[r, pos // 16])
            gk, gv = kc[page, :, pos % 16].double().cpu(), vc[page, :, pos % 16].double().cpu()
            assert (gk[:, :dk] - want_k[t]).abs().max() <= tol * want_k.abs().max() and not gk[:, dk:].any()
            assert (gv[:, :dv] - want_v[t]).abs().max() <= tol * want_v.abs().max() and not gv[:, dv:].any()
        assert int(torch.isfinite(kc.float()).all(-1).sum()) == T * KV == int(torch.isfinite(vc.float()).all(-1).sum())


CUTS = {"whole": [90], "single": [1] * 90, "portions": [2, 3, 17, 31, 2, 1, 1, 33], "page edges": [15, 1, 16, 1, 31, 1, 25]}


@pytest.mark.parametrize("cut", sorted(CUTS))
@pytest.mark.parametrize("H,KV,dk,dv,window", [(6, 2, 24, 16, 16), (3, 3, 7, 5, 21), (2, 1, 136, 9, 40)])
def test_two_attention_layers_that_blend_their_values(H, KV, dk, dv, window, cut):
    """The first blending layer and one that follows it, in the engine's step machinery: the first one's values of the same
    tokens, in whatever step they come. The last tokens look for a token at the window's inner edge and for one just outside."""
    from boring_llm_b200.parts import GatedSinkAttention, RotaryTable
    d, T, scale, eps, base = 40, 90, 0.8, 1e-3, 5000.0
    x = rnd(T, d, seed=1)
    for t in range(T - 6, T):
        x[t - window + 1] = x[t] * 0.9 + x[t - window + 1] * 0.1       # seen
        x[t - window] = x[t] * 0.9 + x[t - window] * 0.1               # not seen by t (but by t - 1)
    xb = x.bfloat16().double()
    layers, want = [], []
    first = None
    for i, role in enumerate(("first", "follow")):
        w = {"wq": rnd(H * dk, d, seed=10 * i + 2, scale=0.3), "wk": rnd(KV * dk, d, seed=10 * i + 3, scale=0.3),
             "wv": rnd(KV * dv, d, seed=10 * i + 4, scale=0.3), "wg": rnd(H * dv, d, seed=10 * i + 5, scale=0.3),
             "wo": rnd(d, H * dv, seed=10 * i + 6, scale=0.3), "q_norm": rnd(H * dk, seed=10 * i + 7, scale=0.1) + 1.0,
             "k_norm": rnd(KV * dk, seed=10 * i + 8, scale=0.1) + 1.0, "vmix": torch.tensor(0.625, dtype=F64)}
        for g in range(H):                                             # queries that look along the keys
            w["wq"][g * dk:(g + 1) * dk] += w["wk"][(g // (H // KV)) * dk:(g // (H // KV) + 1) * dk]
        w = {k: v.bfloat16().double() for k, v in w.items()}
        names = {"wq": "q", "wk": "k", "wv": "v", "wg": "g", "wo": "o", "q_norm": "q.norm", "k_norm": "k.norm", "vmix": "vmix"}
        c = {"heads": H, "kv_heads": KV, "dim": dk, "vdim": dv, "scale": scale, "rot": {"base": base, "dims": dk // 2 * 2}, "mask": {"size": window}}
        y, own = pz.attention_mixer(xb, {names[k]: v for k, v in w.items()}, c, eps, torch.arange(T), first)
        first = own if first is None else first
        layers.append((role, w))
        want.append(y)
    want = torch.cat(want, dim=1)
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 4e-2)):
        tdt = getattr(torch, dtype)
        parts = []
        for role, w in layers:
            p = GatedSinkAttention(d, H, KV, dk, dv, RotaryTable(dk, base, n_rot=dk // 2 * 2), {k: k for k in w}, window=window, scale=scale,
                                   qk_norm="whole", qk_norm_eps=eps, out_gate="channel", value_mix=role, pad_heads=True)
            p.load({k: v.bfloat16() for k, v in w.items()}, tdt, DEV)
            parts.append(p)

        def body(ctx, h):
            ctx.memo.clear()
            outs = []
            for i, p in enumerate(parts):
                o = torch.full((h.shape[0], d), float("nan"), dtype=torch.float32, device=DEV)
                p.mix(ctx, h, o, i)
                outs.append(o)
            return torch.cat(outs, dim=1)
        runner = runner_for(dev(xb, tdt), body, [p.cache_spec() for p in parts], dtype=dtype)
        got = run_portions(runner, "r", T, CUTS[cut]).double().cpu()
        assert (got - want).abs().max() <= tol * want.abs().max(), (dtype, (got - want).abs().max())


@pytest.mark.parametrize("d,F,E,top", [(40, 24, 6, 2), (48, 16, 3, 3), (30, 10, 4, 1)])
def test_experts_with_the_weight_on_their_input(d, F, E, top):
    """The three ways a feed-forward hands its result on, on the grouped tensor-core product and on the plain one; router logits
    on both sides of zero, so that the scores differ much and a weight in the wrong place shows in the clamped activation."""
    from boring_llm_b200.parts import RoutedExperts
    limit, T = 0.6, 150
    c = {"expert": {"limit": limit}, "router": {"top": top}}
    w = {"router": rnd(E, d, seed=1, scale=0.4)}
    for e in range(E):
        w.update({f"e{e}.gate": rnd(F, d, seed=10 + e, scale=0.3), f"e{e}.up": rnd(F, d, seed=30 + e, scale=0.3),
                  f"e{e}.down": rnd(d, F, seed=50 + e, scale=0.3)})
    w = {k: v.bfloat16().double() for k, v in w.items()}
    x = rnd(T, d, seed=3).bfloat16().double()
    want = pz.routed_experts(x, w, c)
    names = {"router": "router"}
    for e in range(E):
        names.update({f"gate{e}": f"e{e}.gate", f"up{e}": f"e{e}.up", f"down{e}": f"e{e}.down"})
    for dtype, tol, fast in (("float32", 1e-5, True), ("bfloat16", 2e-2, True), ("bfloat16", 2e-2, False)):
        tdt = getattr(torch, dtype)
        part = RoutedExperts(d, F, E, top, names, correction=False, activation="clamped", limit=limit, weight_on="input")
        part.load({k: v.bfloat16() for k, v in w.items()}, tdt, DEV)
        for how in ("forward", "apply", "apply_pairs"):
            def body(ctx, h):
                out = torch.full((h.shape[0], d), 1.0 if how == "forward" else float("nan"), dtype=torch.float32, device=DEV)
                if how != "apply_pairs":
                    getattr(part, how)(ctx, h, out)
                    return out - 1.0 if how == "forward" else out
                y, pos, wts = part.apply_pairs(ctx, h)
                assert wts is None
                return y[pos.long() if pos is not None else slice(None)].view(h.shape[0], top, d).sum(1)
            runner = runner_for(dev(x, tdt), body, [], dtype=dtype, fast=fast)
            got = run_portions(runner, "r", T, [130, 1, 2, 17]).double().cpu()
            assert (got - want).abs().max() <= tol * want.abs().max(), (dtype, how)


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
