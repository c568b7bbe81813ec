"""What of the Radenex design runs without a GPU: reading and writing its config.json, the model's description as data (tensor
names, the run order of a repeated stretch with a cache per run, the groups of a window that keeps the first tokens),
refusals, the cache manager's rule for kept pages, rotary frequencies, and the plain implementation on a model from the
random-weights mode."""
import copy
import json
import math
import os

import pytest
import torch

import plain_radenex as pr


def latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=20, scaling=dict(factor=3.0, original=64, fast=16.0, slow=1.0), base=900.0, scale=0.21):
    rot = dict(base=base, dims=rot_dim)
    if scaling:
        rot["scaling"] = scaling
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=rot))


def attention(heads=4, kv_heads=2, dim=16, vdim=10, mask=dict(size=20, keep_first=5), dims=6, base=70.0, factor=1.5, scale=0.4):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=dims))
    if factor:
        m["rot"]["scaling"] = dict(factor=factor)
    if mask:
        m["mask"] = mask
    return dict(type="attention", mixer=m)


CFG = dict(architecture="Radenex", vocab=90, width=24, norm=dict(eps=1e-5), loop=dict(start=1, stop=3, times=3), layers=[
    dict(latent(), mlp=dict(kind="dense", ff=40)), dict(attention(), mlp=None),
    dict(latent(heads=3, scaling=None, vdim=8), mlp=dict(kind="dense", ff=16)), dict(attention(mask=None, factor=None), mlp=dict(kind="dense", ff=8))])


def test_config_round_trip_and_tensor_names(tmp_path):
    from mini_inference_engine_b200.config import load_config
    from mini_inference_engine_b200.models import expected_tensors
    from mini_inference_engine_b200.weights import write_model_folder
    cfg = load_config(json.loads(json.dumps(CFG)))
    assert type(cfg).__name__ == "RadenexConfig" and cfg.to_dict() == json.loads(json.dumps(CFG))
    spec = cfg.model_spec()
    names = {spec.aliases.get(n, n): tuple(t.shape) for n, t in expected_tensors(spec).items()}
    assert names["embed"] == names["head"] == (90, 24) and names["final.norm"] == (24,)
    assert names["l0.norm1"] == (24,) and names["l0.mix.q"] == (2 * 24, 24) and names["l0.mix.dkv"] == (28, 24) and names["l0.mix.dkv.norm"] == (20,)
    assert names["l0.mix.uk"] == (32, 20) and names["l0.mix.uv"] == (48, 20) and names["l0.mix.sink"] == (2,) and names["l0.mix.g"] == (2, 24)
    assert names["l0.mix.o"] == (24, 48) and names["l0.mlp.up"] == (40, 24) and names["l0.mlp.down"] == (24, 40)
    assert names["l1.mix.q"] == (64, 24) and names["l1.mix.k"] == (32, 24) and names["l1.mix.v"] == (20, 24) and names["l1.mix.o"] == (24, 40)
    assert {n for n in names if n.startswith("l1.")} == {"l1.norm1", "l1.mix.q", "l1.mix.k", "l1.mix.v", "l1.mix.o"}     # no feed-forward, nothing learned beside
    assert not any("norm2" in n or ".act" in n for n in names)
    # the random-weights mode writes the checkpoint's own names, and the plain implementation runs on them
    folder = write_model_folder(str(tmp_path / "m"), cfg, seed=1)
    from safetensors.torch import load_file
    W = load_file(os.path.join(folder, "model.safetensors"))
    assert set(W) == set(names)
    trace = []
    logits = pr.forward(CFG, {k: v.float() for k, v in W.items()}, [3, 1, 4, 1, 5, 9, 2, 6], trace)
    assert logits.shape == (8, 90) and torch.isfinite(logits).all() and len(trace) == 8


def test_run_order_and_cache_groups():
    from mini_inference_engine_b200.config import load_config
    from mini_inference_engine_b200.models import DecoderModel, expected_tensors
    from mini_inference_engine_b200.parts import Runtime
    from mini_inference_engine_b200.weights.random_init import random_state
    cfg = load_config(json.loads(json.dumps(CFG)))
    assert cfg.run_plan() == pr.run_order(CFG) == [0, 1, 2, 1, 2, 1, 2, 3]
    spec = cfg.model_spec()
    assert [e.layer for e in spec.run_order] == cfg.run_plan() and len({e.cache for e in spec.run_order}) == 8
    state = {spec.aliases.get(n, n): t for n, t in random_state(expected_tensors(spec), 3).items()}
    model = DecoderModel(spec, state, Runtime("cpu", torch.float32))
    lay = model.cache_layout
    assert [(g.name, g.window, g.keep) for g in lay.groups] == [("full", None, 0), ("window20+first5", 20, 5)] and not lay.state
    group_of = {c: g for c, (g, _) in lay.kv.items()}
    assert [group_of[i] for i in range(8)] == [0, 1, 0, 1, 0, 1, 0, 0]
    assert (lay.kv[0][1].num_kv_heads, lay.kv[0][1].head_dim) == (2, 32) and (lay.kv[1][1].num_kv_heads, lay.kv[1][1].head_dim) == (2, 16)
    # the same window with and without kept tokens, or with other ones, are groups of their own
    from mini_inference_engine_b200.cache.storage import CacheLayout
    from mini_inference_engine_b200.parts import KVNeed
    lay = CacheLayout.from_needs({0: KVNeed(1, 16, 20, None, 5), 1: KVNeed(1, 16, 20), 2: KVNeed(1, 16, 20, None, 7), 3: KVNeed(2, 16, 20, None, 5),
                                  4: KVNeed(1, 16), 5: KVNeed(1, 16, None, None, 9)})
    assert [(g.window, g.keep) for g in lay.groups] == [(None, 0), (20, 0), (20, 5), (20, 7)]
    assert lay.kv[0][0] == lay.kv[3][0] and lay.kv[4][0] == lay.kv[5][0] == 0
    plain = copy.deepcopy(CFG)
    del plain["loop"]
    assert [e.layer for e in load_config(plain).model_spec().run_order] == [0, 1, 2, 3]


@pytest.mark.parametrize("window,keep,page", [(20, 5, 16), (20, 16, 16), (20, 17, 16), (1, 1, 16), (8, 0, 16), (40, 100, 16), (7, 33, 8)])
def test_pages_of_the_first_tokens_stay_while_the_window_moves_on(window, keep, page):
    from mini_inference_engine_b200.cache import RELEASED, CacheManager, GroupSpec, RequestCache
    m = CacheManager([GroupSpec("full"), GroupSpec("w", window, None, keep)], [40, 40], page)
    rc, total = RequestCache(), 0
    for n in (3, 50, 1, 1, 30, 1, 64, 1, 1, 20):
        assert m.reserve(rc, n)
        m.advance(rc, n)
        total += n
        for j in range(total):                     # the next query is at position ``total``
            needed = j < keep or total - j < window
            if needed:
                assert rc.tables[1][j // page] != RELEASED, (total, j)
        held = sum(p != RELEASED for p in rc.tables[1])
        assert held <= -(-keep // page) + -(-window // page) + 1
        assert all(p != RELEASED for p in rc.tables[0])
        m.check()
    m.free(rc)
    assert m.num_free(0) == m.num_free(1) == 39


@pytest.mark.parametrize("edit,word", [
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["layers"][0].update(type="lightning"), "lightning"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rot_dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=9), "vdim"),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
])
def test_configurations_that_are_refused(edit, word):
    from mini_inference_engine_b200.config import ConfigError, load_config
    c = json.loads(json.dumps(CFG))
    edit(c)
    with pytest.raises(ConfigError, match=word):
        load_config(c)


def test_rotary_frequencies_linear_and_yarn():
    from mini_inference_engine_b200.parts.rope import rotary_frequencies, rotary_gain
    cases = [(24, 1.5e5, dict(factor=4.0, original=700, fast=24.0, slow=1.0)), (64, 1e4, dict(factor=40.0, original=4096, fast=32.0, slow=1.0)),
             (8, 50.0, dict(factor=1.0, original=64, fast=4.0, slow=2.0)),
             (32, 1e6, dict(factor=8.0, original=100000, fast=500.0, slow=0.01)),       # the ramp's ends lie beyond both ends of the pairs
             (12, 1e3, dict(factor=2.0, original=30, fast=1.5, slow=1.5))]             # both ends on one pair
    for dims, base, s in cases:
        speeds, gain = pr.yarn_speeds(dims, base, s)
        got = rotary_frequencies(dims, base, dict(s, kind="yarn"))
        assert got.dtype == torch.float32 and torch.equal(got, torch.tensor(speeds, dtype=torch.float32))
        assert rotary_gain(dict(s, kind="yarn")) == pytest.approx(gain) and gain == pytest.approx(0.1 * math.log(s["factor"]) + 1.0)
    assert torch.equal(rotary_frequencies(10, 300.0, dict(kind="linear", factor=2.5)), torch.tensor(pr.linear_speeds(10, 300.0, 2.5), dtype=torch.float32))
    assert rotary_gain(dict(kind="linear", factor=2.5)) == rotary_gain(None) == 1.0
    # a mixture: some pairs keep their frequency, some get f / factor, some lie between
    f, s = rotary_frequencies(24, 1.5e5), rotary_frequencies(24, 1.5e5, dict(cases[0][2], kind="yarn"))
    ratio = (s / f).tolist()
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(0.25) and any(0.26 < r < 0.99 for r in ratio)
    with pytest.raises(ValueError):
        rotary_frequencies(8, 10.0, dict(kind="ntk", factor=2.0))


def test_norm_before_the_rotation_is_norm_after_it():
    """The kernels take a head's statistic before turning it; the design norms the turned head."""
    v = torch.randn(9, 3, 24, dtype=torch.float64)
    pos = torch.arange(9) * 7
    speeds = pr.linear_speeds(16, 40.0, 3.0)
    assert torch.allclose(pr.rms(pr.turn(v, pos, speeds), 1e-3), pr.turn(pr.rms(v, 1e-3), pos, speeds), atol=1e-12)


def test_preset_and_the_benchmark_pair_of_equal_size():
    """The shipped tiny preset reads back, and bench.py's --design option builds a Radenex and a Llama configuration of the
    same width, heads and number of layer runs, the feed-forward's two matrices as large as Llama's three."""
    import importlib.util

    from mini_inference_engine_b200.config import load_preset, preset_names
    assert "tiny-radenex" in preset_names()
    cfg = load_preset("tiny-radenex")
    assert type(cfg).__name__ == "RadenexConfig" and cfg.loop is not None
    assert {l["type"] for l in cfg.layers} == {"latent_attention", "attention"}
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    spec = importlib.util.spec_from_file_location("bench_for_test", os.path.join(root, "bench.py"))
    bench = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(bench)
    for size in bench.DESIGN_SIZES.values():
        r, l = bench.radenex_configs(size)
        assert r.width == l.hidden_size == size["width"] and len(r.run_plan()) == l.num_hidden_layers == size["layers"]
        assert {x["type"] for x in r.layers} == {"latent_attention", "attention"}
        assert abs(2 * r.layers[0]["mlp"]["ff"] - 3 * l.intermediate_size) <= 0.05 * 3 * l.intermediate_size
        m = next(x["mixer"] for x in r.layers if x["type"] == "attention")
        assert m["heads"] == l.num_attention_heads and m["kv_heads"] == l.num_key_value_heads and m["dim"] == l.head_dim
