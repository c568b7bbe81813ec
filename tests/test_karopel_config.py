"""What of the Karopel design runs without a GPU: reading and writing its config.json, the model's description as data (tensor
names, the run order of a repeated stretch with its shifts and a cache per run, pages that hold keys only), refusals, and the plain
implementation on a model from the random-weights mode."""
import copy
import json
import os

import pytest
import torch

import plain_karopel as pk


def attention(heads=4, kv_heads=2, dim=16, vdim=10, mask=dict(size=20, keep_first=5), dims=6, base=70.0,
              scaling=dict(factor=3.0, low=1.0, high=4.0, original=64), scale=0.4):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=dims))
    if scaling:
        m["rot"]["scaling"] = scaling
    if mask:
        m["mask"] = mask
    return dict(type="attention", mixer=m)


def parallel(heads=4, kv_heads=2, dim=16, size=24, scale=0.3, left_scale=0.8, right_scale=1.3, d_heads=4, d_kv=2, d_dim=12, d_vdim=20, conv=3):
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask=dict(size=size))
    right = dict(heads=d_heads, kv_heads=d_kv, dim=d_dim, vdim=d_vdim, conv=conv)
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale))


def with_mlp(layer, ff):
    return dict(layer, mlp=dict(kind="dense", ff=ff) if ff else None)


CFG = dict(architecture="Karopel", vocab=90, width=24, norm=dict(eps=1e-5), residual_mult=0.6, logit_scale=0.3, loop=dict(start=1, stop=3, times=3),
           layers=[with_mlp(parallel(), 40), with_mlp(attention(), None), with_mlp(parallel(heads=3, kv_heads=1, d_heads=1, d_kv=1, conv=1), 16),
                   with_mlp(attention(mask=None, scaling=None), 8)])


def test_config_round_trip_and_tensor_names(tmp_path):
    from mini_inference_engine_b200.config import load_config
    from mini_inference_engine_b200.models import expected_tensors
    from mini_inference_engine_b200.weights import write_model_folder
    cfg = load_config(json.loads(json.dumps(CFG)))
    assert type(cfg).__name__ == "KaropelConfig" and cfg.to_dict() == json.loads(json.dumps(CFG))
    spec = cfg.model_spec()
    names = {spec.aliases.get(n, n): tuple(t.shape) for n, t in expected_tensors(spec).items()}
    assert names["embed"] == names["head"] == (90, 24) and names["final.norm"] == (24,) and names["loop.step"] == (3, 24)
    assert {n for n in names if n.startswith("l0.") and ".mix." not in n} == {"l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down"}
    assert {n[len("l0.mix."):]: s for n, s in names.items() if n.startswith("l0.mix.")} == {
        "left.q": (64, 24), "left.k": (32, 24), "left.o": (24, 64), "right.q": (24, 24), "right.k": (24, 24), "right.v": (80, 24), "right.q.conv": (24, 3),
        "right.k.conv": (24, 3), "right.v.conv": (80, 3), "right.b": (4, 24), "right.a": (4, 24), "right.A_log": (4,), "right.dt_bias": (4,),
        "right.norm": (20,), "right.g": (80, 24), "right.o": (24, 80)}
    assert {n: s for n, s in names.items() if n.startswith("l1.")} == {
        "l1.norm1": (24,), "l1.norm1b": (24,), "l1.mix.q": (64, 24), "l1.mix.k": (32, 24), "l1.mix.v": (20, 24), "l1.mix.q.norm": (16,), "l1.mix.k.norm": (16,),
        "l1.mix.sink": (4,), "l1.mix.o": (24, 40)}
    # the random-weights mode writes the checkpoint's own names, and the plain implementation runs on them
    folder = write_model_folder(str(tmp_path / "m"), cfg, seed=1)
    from safetensors.torch import load_file
    W = load_file(os.path.join(folder, "model.safetensors"))
    assert set(W) == set(names)
    trace = []
    logits = pk.forward(CFG, {k: v.float() for k, v in W.items()}, [3, 1, 4, 1, 5, 9, 2, 6], trace)
    assert logits.shape == (8, 90) and torch.isfinite(logits).all() and len(trace) == 8


def test_run_order_caches_and_what_they_hold():
    from mini_inference_engine_b200.config import load_config
    from mini_inference_engine_b200.models import DecoderModel, expected_tensors
    from mini_inference_engine_b200.parts import Runtime
    from mini_inference_engine_b200.weights.random_init import random_state
    cfg = load_config(json.loads(json.dumps(CFG)))
    assert cfg.run_plan() == pk.run_order(CFG) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    spec = cfg.model_spec()
    # entries 4, 5 and 6 of the layer list are the shifts in front of the passes
    assert [e.layer for e in spec.run_order] == [0, 4, 1, 2, 5, 1, 2, 6, 1, 2, 3] and len({e.cache for e in spec.run_order}) == 11
    assert [spec.layers[i].shift.params["with_embedding"] for i in (4, 5, 6)] == [False, True, True]
    assert [spec.layers[i].shift.params["index"] for i in (4, 5, 6)] == [0, 1, 2]
    assert spec.embedding.params["keep_output"] and spec.final_norm.params["gain"] == 0.3 and spec.layers[0].mixer_out_norm.params["gain"] == 0.6
    state = {spec.aliases.get(n, n): t for n, t in random_state(expected_tensors(spec), 3).items()}
    model = DecoderModel(spec, state, Runtime("cpu", torch.float32))
    lay = model.cache_layout
    assert [(g.window, g.keep) for g in lay.groups] == [(None, 0), (20, 5), (24, 0)]
    assert len(lay.kv) == 8 and len(lay.state) == 2 * 4                  # a parallel layer keeps pages, the delta rule's state and the convolution's inputs
    shared = {k for k, (_, n) in lay.kv.items() if n.shared}
    assert shared == {(0, 0), (2, 0), (4, 0), (6, 0)}
    # keys that serve as values are stored once: half the bytes, and the two views are one tensor
    model.allocate_cache(5, 16, 2)
    lc = model.storage.layer_cache(0).parts[0]
    assert lc.k.data_ptr() == lc.v.data_ptr() and tuple(lc.k.shape) == (5, 2, 16, 16)
    other = model.storage.layer_cache(1)
    assert other.k.data_ptr() != other.v.data_ptr()
    group = lay.kv[(0, 0)][0]
    assert lay.bytes_per_page(group, 16, torch.float32) == 16 * 16 * 4 * (2 + 1 + 1 + 1)
    plain = copy.deepcopy(CFG)
    del plain["loop"]
    spec = load_config(plain).model_spec()
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 3] and not spec.embedding.params["keep_output"] and len(spec.layers) == 4
    once = copy.deepcopy(CFG)
    once["loop"]["times"] = 1                                            # one pass: its vector is added, the embedding's output is not
    spec = load_config(once).model_spec()
    assert [e.layer for e in spec.run_order] == [0, 4, 1, 2, 3] and not spec.embedding.params["keep_output"]


def test_constants_that_may_be_absent():
    from mini_inference_engine_b200.config import load_config
    c = copy.deepcopy(CFG)
    for k in ("residual_mult", "logit_scale"):
        del c[k]
    cfg = load_config(c)
    assert cfg.residual_mult == cfg.logit_scale == 1.0
    assert cfg.model_spec().layers[0].parts["feed_forward_out_norm"].params["gain"] == 1.0


@pytest.mark.parametrize("edit,word", [
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["layers"][0].update(type="lightning"), "lightning"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=3), "keeps no first"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("original"), "original"),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
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


def test_parts_refuse_what_they_cannot_compute():
    from mini_inference_engine_b200.config.model_config import PartSpec
    from mini_inference_engine_b200.parts import NormedDelta
    from mini_inference_engine_b200.parts.base import build_part
    base = dict(hidden_size=32, num_heads=4, num_kv_heads=2, dim=16, vdim=16, scale=1.0, rot_dims=0, rot_base=1.0, eps=1e-5, qk_norm=False, head_temp=False, gate=False)
    for bad in (dict(rot_dims=4), dict(qk_norm="head"), dict(bias=True), dict(vdim=8), dict(rotate_values=True)):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("gated_attention", {**base, "keys_as_values": True, **bad}))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("gated_attention", dict(base, slopes=(1.0, 2.0))))
    shift = build_part("connection", PartSpec("stream_shift", dict(hidden_size=8, rows=2, index=0, with_embedding=False)))
    shift.shift = torch.zeros(8)
    first = shift.pending(None, None)
    assert isinstance(first, NormedDelta) and first.y is None and first.shift is shift.shift
    with pytest.raises(ValueError):
        shift.pending(first, None)                                       # one shift at a time
    with pytest.raises(ValueError):
        build_part("connection", PartSpec("stream_shift", dict(hidden_size=8, rows=2, index=2, with_embedding=False)))


def test_frequencies_rescaled_by_wavelength():
    from mini_inference_engine_b200.parts.rope import rotary_frequencies
    for dims, base, s in [(24, 1.5e5, dict(factor=4.0, low=1.0, high=4.0, original=700)), (64, 1e4, dict(factor=32.0, low=1.0, high=8.0, original=256)),
                          (6, 70.0, dict(factor=3.0, low=1.0, high=4.0, original=64)), (128, 5e5, dict(factor=8.0, low=1.0, high=4.0, original=8192))]:
        got = rotary_frequencies(dims, base, dict(s, kind="wavelength"))
        want = pk.speeds(dict(dims=dims, base=base, scaling=s))
        assert torch.equal(got, torch.tensor(want, dtype=torch.float32))
        share = [w / f for w, f in zip(want, pk.speeds(dict(dims=dims, base=base)))]
        assert share[0] == 1.0 and min(share) < 1.0


def test_the_plain_delta_rule_in_closed_form():
    """Two steps by hand: S_1 = b_1 k_1 v_1^T, o_2 = (g_2 S_1)^T q_2 + (k_2 . q_2) u_2 with u_2 = b_2 (v_2 - g_2 S_1^T k_2)."""
    q, k, v = torch.randn(2, 1, 5, dtype=torch.float64), torch.randn(2, 1, 5, dtype=torch.float64), torch.randn(2, 1, 3, dtype=torch.float64)
    b, g = torch.rand(2, 1, dtype=torch.float64), torch.rand(2, 1, dtype=torch.float64)
    o = pk.delta_steps(q, k, v, b, g)
    S1 = b[0, 0] * torch.outer(k[0, 0], v[0, 0])
    assert torch.allclose(o[0, 0], S1.T @ q[0, 0])
    u2 = b[1, 0] * (v[1, 0] - g[1, 0] * (S1.T @ k[1, 0]))
    assert torch.allclose(o[1, 0], g[1, 0] * (S1.T @ q[1, 0]) + (k[1, 0] @ q[1, 0]) * u2)


def test_preset_and_the_benchmark_pair_of_equal_size():
    """The shipped tiny preset reads back, and bench.py's --design option builds a Karopel and a Llama configuration of the
    same width, feed-forward, heads and number of layer runs."""
    import importlib.util

    from mini_inference_engine_b200.config import load_preset, preset_names
    assert "tiny-karopel" in preset_names()
    cfg = load_preset("tiny-karopel")
    assert type(cfg).__name__ == "KaropelConfig" and cfg.loop is not None and {l["type"] for l in cfg.layers} == {"parallel", "attention"}
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    spec = importlib.util.spec_from_file_location("bench_for_test", os.path.join(root, "bench.py"))
    bench = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(bench)
    for size in bench.DESIGN_SIZES.values():
        r, l = bench.karopel_configs(size)
        assert r.width == l.hidden_size == size["width"] and len(r.run_plan()) == l.num_hidden_layers == size["layers"]
        assert {x["type"] for x in r.layers} == {"parallel", "attention"} and all(x["mlp"]["ff"] == l.intermediate_size for x in r.layers)
        m = next(x["mixer"] for x in r.layers if x["type"] == "attention")
        assert m["heads"] == l.num_attention_heads and m["kv_heads"] == l.num_key_value_heads and m["dim"] == l.head_dim
