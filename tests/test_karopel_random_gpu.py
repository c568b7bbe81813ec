"""Randomly drawn Karopel configurations -- width, layer order, the repeated stretch, head counts and groupings, key and value
sizes, windows and kept tokens, rotated dimensions and their rescaling, taps of the convolution, scales and constants, layers
without a feed-forward -- each with random weights, run through the model runner whole and in portions beside single tokens,
against the plain implementation."""
import json
import random

import pytest

import test_karopel_engine_gpu as eng

pytestmark = pytest.mark.gpu


def draw(seed: int) -> dict:
    rng = random.Random(seed)
    width = rng.choice([32, 40, 52, 64, 72, 96, 128])
    layers = []
    for _ in range(rng.randint(2, 5)):
        if rng.random() < 0.55:
            kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 16, 20, 32, 64, 96, 128])
            left = dict(heads=kv * rng.choice([1, 2, 4]), kv_heads=kv, dim=dim, vdim=dim, scale=round(rng.uniform(0.7, 1.8) * dim ** -0.5, 5),
                        mask=dict(size=rng.choice([1, 7, 16, 24, 33, 64, 96])))
            kv = rng.choice([1, 2, 3])
            right = dict(heads=kv * rng.choice([1, 2, 3]), kv_heads=kv, dim=rng.choice([8, 16, 20, 32, 64, 128]), vdim=rng.choice([6, 16, 32, 48, 64, 128]),
                         conv=rng.randint(1, 6))
            m, kind = dict(left=left, right=right, left_scale=round(rng.uniform(0.3, 1.5), 3), right_scale=round(rng.uniform(0.3, 1.5), 3)), "parallel"
        else:
            kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 16, 20, 32, 64, 96, 128])
            rot = dict(base=rng.choice([30.0, 1e3, 1e4, 2.5e5, 3e6]), dims=rng.choice([d for d in (0, 2, 8, 12, 16, 32, 64, 128) if d <= dim]))
            if rng.random() < 0.8:
                rot["scaling"] = dict(factor=rng.choice([1.0, 2.0, 8.0]), low=rng.choice([0.5, 1.0]), high=rng.choice([2.0, 4.0]), original=rng.choice([32, 200, 2048]))
            m = dict(heads=kv * rng.choice([1, 2, 4]), kv_heads=kv, dim=dim, vdim=rng.choice([6, 16, 32, 48, 64, 128]),
                     scale=round(rng.uniform(0.7, 1.8) * dim ** -0.5, 5), rot=rot)
            if rng.random() < 0.85:
                m["mask"] = dict(size=rng.choice([1, 7, 16, 24, 33, 64, 96]), keep_first=rng.choice([0, 1, 4, 16, 21, 40]))
            kind = "attention"
        mlp = dict(kind="dense", ff=rng.choice([24, 40, 64, 100, 160])) if rng.random() > 0.2 else None
        layers.append(dict(type=kind, mixer=m, mlp=mlp))
    cfg = dict(architecture="Karopel", vocab=rng.randint(50, 300), width=width, norm=dict(eps=rng.choice([1e-6, 1e-5, 1e-3])),
               residual_mult=round(rng.uniform(0.2, 1.2), 3), logit_scale=round(rng.uniform(0.1, 3.0), 3), layers=layers)
    if rng.random() < 0.75:
        lo = rng.randrange(len(layers))
        cfg["loop"] = dict(start=lo, stop=rng.randint(lo + 1, len(layers)), times=rng.randint(1, 3))
    return cfg


@pytest.mark.parametrize("seed,dtype_name", [(s, d) for s in range(14) for d in ("float32", "bfloat16")])
def test_a_drawn_configuration_whole_and_in_portions(seed, dtype_name, tmp_path):
    from mini_inference_engine_b200.config import load_config
    from mini_inference_engine_b200.weights import write_model_folder
    cfg = draw(seed)
    name = f"draw{seed}"
    eng.CONFIGS[name] = cfg
    try:
        folder = write_model_folder(str(tmp_path / name), load_config(json.loads(json.dumps(cfg))), seed=300 + seed)
        rng = random.Random(2000 + seed)
        reqs = {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(n)] for i, n in enumerate((rng.randint(1, 140), rng.randint(17, 200), 33))}
        runner = eng.runner_for(name, folder, dtype_name, 416, 3)
        eng.check(name, folder, dtype_name, eng.run_schedule(runner, reqs, [[(rid, len(t))] for rid, t in reqs.items()]), reqs)
        # all three at once: a portion of each, then single tokens of one beside portions of the others, on reused pages
        left, schedule = {r: len(t) for r, t in reqs.items()}, []
        while any(left.values()):
            step = []
            for r in reqs:
                if left[r]:
                    n = min(left[r], rng.choice([1, 1, 2, 9, 16, 31]))
                    step.append((r, n))
                    left[r] -= n
            schedule.append(step)
        eng.check(name, folder, dtype_name, eng.run_schedule(runner, reqs, schedule), reqs)
    finally:
        eng.CONFIGS.pop(name, None)
        eng._models.pop((name, dtype_name), None)
        for k in [k for k in eng._plain if k[0] == name]:
            eng._plain.pop(k)
