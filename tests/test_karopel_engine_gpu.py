"""Whole Karopel models against the plain implementation (``plain_karopel``): small configurations made here, with random
weights from the package's random-weights mode, run through the model runner (the step function, cache manager and kernels
of generation) whole, with the last tokens one by one, in portions down to two tokens, and as mixed batches with so few
pages that they are used again; then through ``bin/trace_run`` and through the engine's own entry point with its scheduler."""
import json
import os
import random

import numpy as np
import pytest
import torch

import plain_karopel as pk
from conftest import plain_weights
from replay_driver import Replay
from test_getizen_engine_gpu import run_schedule
from test_karopel_config import attention, parallel, with_mlp

pytestmark = pytest.mark.gpu
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# relative error of a row of logits (root mean square of the difference over that of the row).  float32: the order of sums.  bfloat16: activations are
# rounded between kernels, and every norm behind a sublayer scales a small output up together with its rounding error.  So a row may
# differ by this much or by three times what rounding moves it by in the plain implementation; one row in fifty may go up to twice that.
TOL = {"float32": 3e-4, "bfloat16": 0.06}


CONFIGS = {
    # the repeated stretch lies in the middle (layers 1 and 2, twice); windows and a number of kept tokens that are no multiples of
    # a page; a layer without a feed-forward; three query heads a key head; key and value sizes differ wherever they can
    "k_a": dict(architecture="Karopel", vocab=150, width=48, norm=dict(eps=1e-5), residual_mult=0.6, logit_scale=0.3, loop=dict(start=1, stop=3, times=2), layers=[
        with_mlp(parallel(3, 1, 24, 21, 0.25, 0.8, 1.3, 4, 2, 12, 20, 3), 64),
        with_mlp(attention(6, 2, 16, 32, dict(size=24, keep_first=19), 8, 100.0, dict(factor=4.0, low=1.0, high=4.0, original=50), 0.7), None),
        with_mlp(parallel(2, 2, 16, 40, 0.4, 1.5, 0.7, 3, 3, 32, 8, 5), 40),
        with_mlp(attention(3, 3, 32, 16, dict(size=40, keep_first=3), 32, 5e3, dict(factor=2.0, low=1.0, high=2.0, original=300), 0.4), 96)]),
    # nothing is repeated; heads of 64 and 128 (in bfloat16 the tcgen05 kernel, page copies by TMA in decoding); a window of exactly a
    # page that keeps exactly a page; a window that keeps nothing; one head; no rescaling; scales and constants of 1
    "k_b": dict(architecture="Karopel", vocab=97, width=64, norm=dict(eps=1e-4), residual_mult=1.0, logit_scale=1.0, layers=[
        with_mlp(attention(4, 1, 64, 64, dict(size=16, keep_first=16), 64, 500.0, None, 0.2), 128),
        with_mlp(parallel(4, 2, 64, 33, 0.15, 1.0, 1.0, 2, 1, 64, 128, 4), 72),
        with_mlp(attention(1, 1, 128, 96, dict(size=33), 0, 1e4, None, 0.15), 8),
        with_mlp(parallel(2, 1, 128, 16, 0.1, 0.3, 2.0, 1, 1, 128, 64, 1), None)]),
    # the whole model three times; heads that are multiples of nothing; a window of one that keeps one; attention over everything;
    # heads beyond 128 (in bfloat16 the CUDA-core attention kernel)
    "k_c": dict(architecture="Karopel", vocab=211, width=52, norm=dict(eps=1e-6), residual_mult=0.25, logit_scale=2.5, loop=dict(start=0, stop=3, times=3), layers=[
        with_mlp(attention(5, 1, 20, 12, dict(size=1, keep_first=1), 6, 40.0, dict(factor=8.0, low=0.5, high=3.0, original=40), 0.9), 36),
        with_mlp(parallel(2, 1, 144, 60, 0.09, 0.9, -0.8, 6, 3, 20, 36, 2), 60),
        with_mlp(attention(2, 1, 36, 40, None, 12, 1e3, dict(factor=2.0, low=1.0, high=4.0, original=64), 0.5), 20)]),
}
LENGTHS = {"k_a": [5, 77, 130, 2, 49, 24, 25], "k_b": [1, 70, 33, 129, 16, 17, 64], "k_c": [3, 100, 47, 150, 48, 49, 9]}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from mini_inference_engine_b200.config import load_config
    from mini_inference_engine_b200.weights import write_model_folder
    out = {}
    for i, (name, c) in enumerate(CONFIGS.items()):
        d = str(tmp_path_factory.mktemp(name))
        write_model_folder(d, load_config(json.loads(json.dumps(c))), seed=90 + i)
        with open(os.path.join(d, "config.json")) as f:
            assert json.load(f) == json.loads(json.dumps(c)), "the configuration must survive writing and reading"
        out[name] = d
    return out


def requests_for(name, seed=0):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(CONFIGS[name]["vocab"]) for _ in range(n)] for i, n in enumerate(LENGTHS[name])}


_plain: dict = {}


def plain_logits(name, folder, tokens, rnd=pk.exact):
    key = (name, tuple(tokens), rnd is pk.exact)
    if key not in _plain:
        _plain[key] = pk.forward(CONFIGS[name], plain_weights(folder), tokens, rnd=rnd)
    return _plain[key]


_models: dict = {}


def model_for(name, folder, dtype_name):
    from mini_inference_engine_b200.models import load_model
    key = (name, dtype_name)
    if key not in _models:
        _models[key] = load_model(folder, DTYPES[dtype_name], "cuda:0")[1]
    return _models[key]


def runner_for(name, folder, dtype_name, max_tokens, slots):
    from mini_inference_engine_b200.engine.runner import ModelRunner
    return ModelRunner(model_for(name, folder, dtype_name), -(-max_tokens // 16) + 1, 16, slots)


def check(name, folder, dtype_name, got, reqs):
    """got[id][position] = logits row; every position of every request must be there and close to the plain row."""
    errs = []
    for rid, toks in reqs.items():
        assert sorted(got[rid]) == list(range(len(toks))), f"{rid}: positions missing"
        want = plain_logits(name, folder, toks)
        size = want.pow(2).mean(-1).sqrt()
        limit = torch.full((len(toks),), TOL[dtype_name])
        if dtype_name == "bfloat16":
            limit = torch.maximum(limit, 3.0 * (plain_logits(name, folder, toks, pk.to_bf16) - want).pow(2).mean(-1).sqrt() / size)
        for p in range(len(toks)):
            d = torch.from_numpy(got[rid][p]) - want[p]
            assert torch.isfinite(d).all(), f"{name} {dtype_name} {rid}: position {p} is not finite"
            errs.append((float(d.pow(2).mean().sqrt() / size[p] / limit[p]), rid, len(toks), p, p % 16))
    bad = sorted((e for e in errs if e[0] > 1.0), reverse=True)
    allowed = len(errs) // 50 if dtype_name == "bfloat16" else 0
    assert len(bad) <= allowed and (not bad or bad[0][0] <= 2.0), (
        f"{name} {dtype_name}: {len(bad)} of {len(errs)} positions differ; worst (error over limit, request, length, position, page offset): {bad[:6]}")


CASES = [(n, d) for n in CONFIGS for d in DTYPES]


@pytest.mark.parametrize("name,dtype_name", CASES)
def test_whole_then_token_by_token_then_portions(name, dtype_name, folders):
    reqs = requests_for(name)
    runner = runner_for(name, folders[name], dtype_name, 192, 2)
    whole = [[(rid, len(t))] for rid, t in reqs.items()]
    check(name, folders[name], dtype_name, run_schedule(runner, reqs, whole), reqs)
    # most of a request in one step, its last tokens (up to 40: past the edges of every window) one by one
    decode = []
    for rid, t in reqs.items():
        tail = min(40, len(t) - 1)
        decode += ([[(rid, len(t) - tail)]] if len(t) > tail else []) + [[(rid, 1)]] * tail
    check(name, folders[name], dtype_name, run_schedule(runner, reqs, decode), reqs)
    rng = random.Random(1)
    portions = []
    for rid, t in reqs.items():
        left = len(t)
        while left:
            n = min(left, rng.choice([2, 2, 3, 5, 15, 16, 17, 31, 40, 1]))
            portions.append([(rid, n)])
            left -= n
    check(name, folders[name], dtype_name, run_schedule(runner, reqs, portions), reqs)


@pytest.mark.parametrize("name,dtype_name", CASES)
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype_name, folders):
    """Up to three live requests: portions of some beside single tokens of others; the pool holds 208 positions and
    three state slots for seven requests, so both are used again, by requests of other lengths."""
    reqs = requests_for(name, seed=2)
    rng = random.Random(3)
    waiting, live, left, schedule = list(reqs), [], {r: len(t) for r, t in reqs.items()}, []
    held = lambda: sum(-(-(len(reqs[r]) - left[r]) // 16) * 16 for r in live)
    while waiting or live:
        while waiting and len(live) < 3 and held() + -(-len(reqs[waiting[0]]) // 16) * 16 + 16 * len(live) <= 208 - 16 * 3:
            live.append(waiting.pop(0))
        step = []
        for r in list(live):
            if rng.random() < 0.2 and len(live) > 1 and step:
                continue                                   # left out of this step, goes on later
            n = min(left[r], rng.choice([1, 1, 2, 7, 16, 33]))
            step.append((r, n))
            left[r] -= n
            if left[r] == 0:
                live.remove(r)
        schedule.append(step)
    assert any(len(s) == 3 for s in schedule) and any(len({n for _, n in s}) > 1 for s in schedule)
    runner = runner_for(name, folders[name], dtype_name, 416, 3)
    check(name, folders[name], dtype_name, run_schedule(runner, reqs, schedule), reqs)


@pytest.mark.parametrize("dtype_name", list(DTYPES))
def test_long_decoding_far_beyond_every_window_and_page(dtype_name, folders):
    name = "k_a"
    rng = random.Random(4)
    reqs = {"long": [rng.randrange(150) for _ in range(330)]}
    runner = runner_for(name, folders[name], dtype_name, 336, 1)
    check(name, folders[name], dtype_name, run_schedule(runner, reqs, [[("long", 3)]] + [[("long", 1)]] * 327), reqs)


@pytest.mark.parametrize("dtype_name", list(DTYPES))
def test_trace_replay_program(dtype_name, folders, tmp_path):
    name = "k_b"
    reqs = requests_for(name, seed=5)
    got = {}
    with Replay(folders[name], dtype_name, tmp_path / "out", max_tokens=448, vocab=CONFIGS[name]["vocab"]) as rp:
        ids = list(reqs)
        for a, b in zip(ids[0::2], ids[1::2] + [None]):
            ta, tb = reqs[a], reqs[b] if b else []
            ca = max(1, len(ta) // 2)
            first = [(a, ta[:ca], list(range(ca)))] + ([(b, tb, list(range(len(tb))))] if b else [])
            for (rid, toks, want), rows in zip(first, np.split(rp.step(first, end=[b] if b else []), [ca])):
                got.setdefault(rid, {}).update({p: rows[p] for p in want})
            if len(ta) > ca:
                rows = rp.step([(a, ta[ca:], list(range(len(ta) - ca)))], end=[a])
                got[a].update({ca + p: rows[p] for p in range(len(ta) - ca)})
    check(name, folders[name], dtype_name, got, reqs)


def plain_greedy(name, folder, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(plain_logits(name, folder, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_through_the_engine(name, folders):
    """The engine's own entry point and scheduler, four ways: default (captured decode graphs), a token budget of 16
    (prompts go in portions beside decoding requests), no graphs, and a pool so small that requests are pushed out
    and recomputed (their pages and slots are used again).  float32: the plain implementation's tokens."""
    from mini_inference_engine_b200 import EngineConfig, LLMEngine, SamplingParams
    rng = random.Random(6)
    vocab = CONFIGS[name]["vocab"]
    prompts = [[rng.randrange(vocab) for _ in range(n)] for n in (5, 37, 20, 66, 2)]
    crowded = [[rng.randrange(vocab) for _ in range(n)] for n in (30, 29, 31, 5)]      # three of them outgrow seven pages together
    for overrides in (dict(), dict(max_num_batched_tokens=16), dict(use_cuda_graphs=False),
                      dict(num_blocks=8, max_num_seqs=3, max_num_batched_tokens=48)):
        ps = crowded if "num_blocks" in overrides else prompts
        want = [plain_greedy(name, folders[name], p, 12) for p in ps]
        eng = LLMEngine(folders[name], EngineConfig(max_model_len=128, **overrides), dtype=torch.float32, load_tokenizer=False,
                        verbose=False)
        outs = eng.generate(ps, SamplingParams(max_tokens=12, ignore_eos=True))
        assert [o.output_ids for o in outs] == want, f"{name} with {overrides}"
        if "num_blocks" in overrides:
            assert eng.scheduler.num_preemptions > 0
        eng.cache.check()


def test_greedy_generation_in_bfloat16_follows_the_plain_scores(folders):
    from mini_inference_engine_b200 import EngineConfig, LLMEngine, SamplingParams
    name = "k_b"
    rng = random.Random(7)
    prompts = [[rng.randrange(CONFIGS[name]["vocab"]) for _ in range(n)] for n in (9, 40)]
    eng = LLMEngine(folders[name], EngineConfig(max_model_len=128), dtype=torch.bfloat16, load_tokenizer=False, verbose=False)
    outs = eng.generate(prompts, SamplingParams(max_tokens=10, ignore_eos=True))
    for p, o in zip(prompts, outs):
        ids = list(p)
        for n, tok in enumerate(o.output_ids):
            row = plain_logits(name, folders[name], ids)[-1]
            assert row[tok] >= row.max() - 4 * TOL["bfloat16"] * row.pow(2).mean().sqrt(), f"output {n}: token {tok} is far from the plain top"
            ids.append(tok)


def test_command_line_generates_with_a_karopel_folder(folders, capsys):
    from mini_inference_engine_b200.__main__ import main
    main(["generate", "--model", folders["k_a"], "--dtype", "float32", "--prompt-ids", "5,6,7", "--max-tokens", "4", "--ignore-eos",
          "--overrides", '{"num_blocks": 64, "max_model_len": 128}'])
    lines = [json.loads(l) for l in capsys.readouterr().out.splitlines() if l.startswith("{")]
    assert lines[0]["output_ids"] == plain_greedy("k_a", folders["k_a"], [5, 6, 7], 4)
