"""The mechanisms of the Radenex design one by one, built through the part registry with sizes of their own, against the plain
functions of ``plain_radenex``: the RMS norm over a sum of two outputs, the squared-relu feed-forward, heads of unit root mean
square and rotated values, the attention kernels' window with kept first keys, windowed attention, latent attention with a
rescaled rotation, a sink and a gate per head.  Mixers run a sequence whole, in portions down to one token, and several
requests in one batch, from pages that other requests used before."""
import random

import pytest
import torch

import plain_radenex as pr
from helpers import close as close_at, scattered_tables
from test_getizen_parts_gpu import DEV, DTYPES, PAGE, Harness, bind_random, build, inputs, rt_for, run_in_portions

pytestmark = pytest.mark.gpu
BF16 = torch.bfloat16


def close(got, want, dtype, what="", bf16=4e-2):
    """bfloat16 mixers round their projections, keys, values and heads in turn: twice the bound of a single kernel."""
    if dtype == torch.float32:
        return close_at(got, want, dtype, what)
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    err, scale = (got - want).abs().max().item(), max(want.abs().max().item(), 1e-6)
    assert err <= bf16 * scale, f"{what}: max abs error {err:.3e} > {bf16} x {scale:.3e}"


# ----------------------------------------------------------------------------------------------- norm, feed-forward, layer

@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n", [40, 42, 1024])
def test_rms_norm_over_the_sum_of_both_sublayers(dt, n):
    from mini_inference_engine_b200.parts import Branches
    rt = rt_for(dt)
    norm = build("norm", "layernorm", size=n, eps=2e-3, center=False)
    W = bind_random(norm, rt, 3, {"weight": torch.randn(n)})
    res, a, b = torch.randn(6, n) * 0.1 + 0.2, torch.randn(6, n), torch.randn(6, n) * 0.3
    r = res.clone().to(DEV)
    out = norm(Branches((a.to(DEV), b.to(DEV))), r)
    close_at(r, res + a + b, torch.float32, "stream")
    close_at(out, pr.rms(res + a + b, 2e-3) * W["p.weight"], dt, "normed")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T", [1, 9, 40, 200])
@pytest.mark.parametrize("hidden,ff", [(64, 144), (50, 36)])
def test_squared_relu_feed_forward(dt, T, hidden, ff):
    rt = rt_for(dt)
    part = build("feed_forward", "activated_mlp", hidden_size=hidden, intermediate_size=ff, activation="relu2")
    assert set(part.tensor_specs()) == {"up", "down"}
    W = bind_random(part, rt, 4)
    x = inputs(T, hidden, 1, dt) * 2
    close(part.forward(x.to(dt).to(DEV), None), pr.feed_forward(x, W, "p."), dt, f"{T} tokens", bf16=2e-2)


@pytest.mark.parametrize("M,N,K,force", [(1, 264, 320, {}), (8, 2048, 1024, {}), (24, 520, 96, {}), (40, 256, 512, {}), (8, 384, 512, dict(splits=1)),
                                         (300, 384, 96, {}), (300, 264, 72, dict(splits=2)), (2048, 2560, 256, {}), (64, 640, 1024, dict(bn=64, splits=8))])
def test_squared_relu_in_the_epilogue_of_the_tcgen05_products(M, N, K, force):
    from mini_inference_engine_b200.kernels import gemm_tc
    g = torch.Generator().manual_seed(M + N)
    x, w = torch.randn(M, K, generator=g).to(BF16), (torch.randn(N, K, generator=g) * K ** -0.5).to(BF16)
    want = torch.relu(x.float() @ w.float().T).square()
    for out_dt in (BF16, torch.float32):
        out = torch.empty(M, N, dtype=out_dt, device=DEV)
        gemm_tc.gemm(x.to(DEV), w.to(DEV), out, relu2=True, **force)
        close_at(out, want, out_dt if out_dt == BF16 else torch.float32, f"gemm {force}")
        if M >= 128:
            out.fill_(7.0)
            gemm_tc.gemm_pair(x.to(DEV), w.to(DEV), out, relu2=True)
            close_at(out, want, out_dt if out_dt == BF16 else torch.float32, "pair")
    torch.cuda.synchronize()
    gemm_tc.check_error()


# ----------------------------------------------------------------------------------------------- projections -> heads

SHAPES = [dict(H=4, G=2, D=32, Dv=32, rot=16), dict(H=3, G=1, D=16, Dv=48, rot=16), dict(H=5, G=5, D=128, Dv=96, rot=32), dict(H=1, G=1, D=64, Dv=64, rot=0),
          dict(H=6, G=2, D=10, Dv=6, rot=4), dict(H=2, G=1, D=144, Dv=192, rot=144), dict(H=20, G=4, D=128, Dv=128, rot=128)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("s", SHAPES)
@pytest.mark.parametrize("interleaved", [False, True])
def test_unit_heads_rotated_values_and_the_turn_back(dt, s, interleaved):
    """The kernel between the projection and attention, and the one behind attention, alone; bfloat16 takes the kernels of whole
    16-byte pieces where the sizes allow.  Positions are far apart and out of order."""
    from mini_inference_engine_b200.kernels import ops
    H, G, D, Dv, rot = s["H"], s["G"], s["D"], s["Dv"], s["rot"]
    DP, T, eps, pages = -(-max(D, Dv) // 16) * 16, 7, 1e-3, 5
    g = torch.Generator().manual_seed(D + Dv)
    width = H * D + G * (D + Dv) + (-(H * D + G * (D + Dv))) % 8
    rows = torch.randn(T, width, generator=g).to(dt)
    pos = torch.tensor([0, 1, 2, 77, 1030, 5, 40000], dtype=torch.int32)
    slots = torch.tensor([16, 33, 17, 70, 64, 18, 79], dtype=torch.int32)
    speeds, v_speeds = pr.plain_speeds(rot, 300.0), pr.plain_speeds(Dv, 1000.0)
    freq, v_freq = torch.tensor(speeds, dtype=torch.float32), torch.tensor(v_speeds, dtype=torch.float32)
    k_cache = torch.full((pages, G, PAGE, DP), 3.0, dtype=dt, device=DEV)
    v_cache, q_out = k_cache.clone(), torch.empty(T, H, DP, dtype=dt, device=DEV)
    ops.qk_norm_rope(rows.to(DEV), pos.to(DEV), slots.to(DEV), freq.to(DEV), q_out, k_cache, v_cache, num_heads=H, num_kv_heads=G, dim=D,
                     vdim=Dv, rot=rot, page_size=PAGE, eps=eps, head_norm=True, interleaved=interleaved, v_freq=v_freq.to(DEV))

    def turn(x, sp, sign=1):
        if not interleaved:
            return pr.turn(x, sign * pos, sp)
        n = 2 * len(sp)                            # neighbours as pairs: the same rotation with the entries laid out otherwise
        y = torch.cat([x[..., 0:n:2], x[..., 1:n:2], x[..., n:]], -1)
        y = pr.turn(y, sign * pos, sp)
        out = y.clone()
        out[..., 0:n:2], out[..., 1:n:2] = y[..., :n // 2], y[..., n // 2:n]
        return out

    x = rows.double()
    q, k, v = x[:, :H * D].reshape(T, H, D), x[:, H * D:(H + G) * D].reshape(T, G, D), x[:, (H + G) * D:(H + G) * D + G * Dv].reshape(T, G, Dv)
    pad = lambda t: torch.nn.functional.pad(t, (0, DP - t.shape[-1]))
    # float32 angles: a position of 40,000 turns the fastest pair by an angle that float32 holds to 2e-3

    def chk(got, want, what):
        close(got[:6], want[:6], dt, what, bf16=2e-2)
        close(got[6:], want[6:], BF16, what + " (far position)", bf16=2e-2)

    chk(q_out, pad(pr.rms(turn(q, speeds), eps)), "queries")
    page, off = slots // PAGE, slots % PAGE
    stored = lambda c: c.cpu()[page.long(), :, off.long()]
    chk(stored(k_cache), pad(pr.rms(turn(k, speeds), eps)), "keys")
    chk(stored(v_cache), pad(turn(v, v_speeds)), "values")
    assert (k_cache.cpu()[0] == 3.0).all() and int((k_cache.cpu() != 3.0).any(-1).sum()) == T * G, "only the tokens' own slots are written"
    attn = torch.randn(T, H, DP, generator=g).to(dt)
    out = torch.empty(T, H * Dv, dtype=dt, device=DEV)
    ops.turn_heads(attn.to(DEV), pos.to(DEV), v_freq.to(DEV), out, H, Dv, interleaved=interleaved)
    chk(out, turn(attn[..., :Dv].double(), v_speeds, -1).reshape(T, H * Dv), "turned back")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,Dv,DP", [(3, 16, 16), (5, 24, 32), (2, 10, 16), (8, 128, 128)])
def test_gate_per_head(dt, H, Dv, DP):
    from mini_inference_engine_b200.kernels import ops
    T = 9
    attn, wide = torch.randn(T, H, DP).to(dt), torch.randn(T, 3 + H + 2).to(dt)
    out = torch.empty(T, H * Dv, dtype=dt, device=DEV)
    ops.sigmoid_gate(attn.to(DEV), wide.to(DEV)[:, 3:3 + H], out, H, Dv)
    close_at(out, (attn[..., :Dv].float() * torch.sigmoid(wide[:, 3:3 + H].float())[..., None]).reshape(T, H * Dv), dt, "gate per head")


# ----------------------------------------------------------------------------------------------- kept keys, kernel by kernel

def kept_case(ops, kernel, dt, H, G, D, page, rows, window, keep, seed=0, sink=True, loud=(), **more):
    """Rows of (new tokens, context) through one attention kernel.  Pages that lie wholly between the kept keys and the window of
    the row's first new token have been given back: their table entries name page 0, which holds large numbers.  ``loud``:
    key positions scaled so that their scores stand out."""
    g = torch.Generator().manual_seed(seed)
    T, n_pages = sum(a for a, _ in rows), sum(-(-c // page) for _, c in rows) + 3
    tables = scattered_tables([c for _, c in rows], page, n_pages, seed)
    kc = (50.0 * torch.randn(n_pages, G, page, D, generator=g)).to(dt)
    vc = (50.0 * torch.randn(n_pages, G, page, D, generator=g)).to(dt)
    q_all = torch.randn(T, H, D, generator=g).to(dt)
    sinks = torch.randn(H, generator=g) if sink else torch.zeros(H)
    scale, want, at = 1.3 * D ** -0.5, [], 0
    width = max(len(t) for t in tables)
    block = torch.zeros(len(rows), width, dtype=torch.int32)
    for r, (n, ctx) in enumerate(rows):
        k, v = torch.randn(ctx, G, D, generator=g).to(dt), torch.randn(ctx, G, D, generator=g).to(dt)
        for j in loud:
            if j < ctx:
                k[j] = (q_all[at + n - 1].view(G, H // G, D).mean(1) * 3.0).to(dt)
        for j in range(ctx):
            p = tables[r][j // page]
            kc[p, :, j % page], vc[p, :, j % page] = k[j], v[j]
        first = max(0, ctx - n - window + 1)
        for i, p in enumerate(tables[r]):
            gone = i >= -(-keep // page) and (i + 1) * page <= first
            block[r, i] = 0 if gone else p
        q = torch.zeros(ctx, H, D)
        q[ctx - n:] = q_all[at:at + n].float()
        o = pr.softmax_attention(q, k.float(), v.float(), scale, dict(size=window, keep_first=keep), sinks)
        want.append(o[ctx - n:])
        at += n
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    starts = [sum(a for a, _ in rows[:i]) for i in range(len(rows))]
    out = torch.full((T, H, D), 9.0, dtype=dt, device=DEV)
    args = (q_all.to(DEV), H * D, kc.to(DEV), vc.to(DEV), block.to(DEV), i32(starts), i32([a for a, _ in rows]), i32([c for _, c in rows]))
    mods = ops.ScoreMods(sink=sinks.to(DEV))
    if kernel == "decode":
        ops.decode_attention(*args, out, H, G, D, page, scale, window, keep=keep, mods=mods, max_ctx=max(c for _, c in rows), **more)
    elif kernel == "simt":
        ops.paged_attention(*args, T, out, H, G, D, page, scale, window, keep=keep, mods=mods)
    else:
        fn = ops.prefill_attention_tc if kernel == "prefill_tc" else ops.prefill_attention
        fn(*args, T, out, H, G, D, page, scale, window, keep=keep, mods=mods, min_q_len=1)
    torch.cuda.synchronize()
    ops.check_range_errors()
    ops.check_tc_errors()
    return out, torch.cat(want, 0)


PORTIONS = [(1, 1), (2, 30), (5, 5), (130, 130), (40, 300), (200, 700), (3, 515), (129, 385)]
KEPT = [(20, 5), (20, 16), (1, 1), (64, 64), (65, 63), (100, 129), (33, 200), (128, 17), (300, 65), (16, 0)]


@pytest.mark.parametrize("window,keep", KEPT)
@pytest.mark.parametrize("kernel,dt,D,page", [("simt", torch.float32, 48, 16), ("simt", BF16, 32, 64), ("prefill", BF16, 48, 16), ("prefill", BF16, 80, 128),
                                              ("prefill_tc", BF16, 64, 16), ("prefill_tc", BF16, 128, 32), ("prefill_tc", BF16, 64, 256)])
def test_kept_keys_in_portions(kernel, dt, D, page, window, keep):
    from mini_inference_engine_b200.kernels import ops
    out, want = kept_case(ops, kernel, dt, 4, 2, D, page, PORTIONS, window, keep, seed=window + keep, loud=(0, keep - 1, keep, 250))
    close_at(out, want, dt, f"{kernel} window {window} keep {keep}")


@pytest.mark.parametrize("window,keep", KEPT)
@pytest.mark.parametrize("how", [dict(), dict(splits=1), dict(splits=2, merge="cluster"), dict(splits=8, merge="cluster", tma=True),
                                 dict(splits=5, merge="scratch", min_part_tiles=1), dict(splits=3, merge="scratch", tma=True, stages=2)])
@pytest.mark.parametrize("H,G,D,page", [(6, 2, 64, 16), (4, 4, 48, 32), (20, 1, 128, 16)])
def test_kept_keys_in_decoding(H, G, D, page, how, window, keep):
    from mini_inference_engine_b200.kernels import ops
    rows = [(1, c) for c in (1, 2, 17, 64, 65, 130, 257, 300, 705)]
    out, want = kept_case(ops, "decode", BF16, H, G, D, page, rows, window, keep, seed=window + keep, loud=(0, keep - 1, keep, 250), **how)
    close_at(out, want, BF16, f"decode window {window} keep {keep} {how}")


def test_kept_keys_where_a_block_takes_two_query_tiles():
    from mini_inference_engine_b200.kernels import ops
    for D in (64, 128):
        out, want = kept_case(ops, "prefill_tc", BF16, 32, 4, D, 16, [(900, 900), (400, 1000), (7, 300)], 150, 140, seed=D)
        close_at(out, want, BF16, f"pairs of query tiles, heads of {D}")


# ----------------------------------------------------------------------------------------------- windowed attention

def windowed(heads, kv_heads, dim, vdim, scale, rot_dims, base, factor, window, keep):
    part = dict(num_heads=heads, num_kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot_dims=rot_dims, rot_base=base, window=window, keep_first=keep,
                rot_scaling=dict(kind="linear", factor=factor) if factor else None)
    cfg = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=rot_dims))
    if factor:
        cfg["rot"]["scaling"] = dict(factor=factor)
    if window:
        cfg["mask"] = dict(size=window, keep_first=keep)
    return part, cfg


WINDOWED = [windowed(4, 2, 32, 32, 0.3, 16, 50.0, 2.0, 24, 5), windowed(3, 3, 16, 48, 0.5, 16, 1e4, None, 16, 20), windowed(6, 1, 64, 32, 0.15, 0, 1e6, 3.0, None, 0),
            windowed(2, 1, 128, 96, 0.09, 64, 1e3, 1.0, 1, 1), windowed(5, 1, 48, 64, 0.2, 2, 200.0, 0.5, 40, 0), windowed(1, 1, 144, 160, 0.1, 32, 9e3, 7.0, 33, 70)]


def windowed_part(hidden, part):
    return build("mixer", "gated_attention", hidden_size=hidden, eps=1e-3, qk_norm="unit", head_temp=False, gate=False, rotate_values=True, sink="one", **part)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", WINDOWED)
def test_windowed_attention_whole_in_portions_token_by_token_and_in_batches(dt, case):
    rt = rt_for(dt)
    hidden, T, (params, cfg) = 40, 150, case
    mixer = windowed_part(hidden, params)
    assert set(mixer.tensor_specs()) == {"q", "k", "v", "o"}
    W = bind_random(mixer, rt, 14)
    x = inputs(T, hidden, 5, dt)
    want = pr.windowed_attention(x, W, "p.", cfg, 1e-3)
    h = Harness(mixer, rt, pages=40)
    close(run_in_portions(h, x, [T]), want, dt, "whole")
    close(run_in_portions(h, x, [23, 2, 30, 1, 1, 20, 2, 21, 50]), want, dt, "portions")
    close(run_in_portions(h, x, [1] * T), want, dt, "token by token")
    close(run_in_portions(h, x, [2] * (T // 2)), want, dt, "two by two")
    xs = [inputs(n, hidden, 40 + n, dt) for n in (90, 3, 131)]
    rcs, cuts = [h.new() for _ in xs], [(60, 30), (2, 1), (130, 1)]
    first = h.step([(rc, xi[:a]) for rc, xi, (a, _) in zip(rcs, xs, cuts)])
    second = h.step([(rc, xi[a:]) for rc, xi, (a, _) in zip(rcs, xs, cuts)])
    for i, (f, s) in enumerate(zip(first, second)):
        close(torch.cat([f, s], 0), pr.windowed_attention(xs[i], W, "p.", cfg, 1e-3), dt, f"request {i} of a batch")
        h.free(rcs[i])
    h.manager.check()


STANDOUT = windowed(2, 2, 16, 16, 0.8, 0, 1e4, None, 24, 5)
PAIRS = [(70, 47), (70, 46), (70, 4), (70, 5), (70, 0), (95, 72), (95, 71), (23, 0), (24, 0), (28, 4), (28, 5), (29, 5), (29, 4), (200, 177), (200, 176),
         (200, 4), (200, 5), (200, 15), (200, 16), (40, 39), (300, 0), (300, 4), (300, 5), (300, 130)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
def test_a_key_that_stands_out_at_the_edges_of_the_window_and_of_the_kept_tokens(dt, decode):
    """W_k = -W_q and the planted input is minus the query's: its key equals the query (whose own key is its opposite), so it takes
    nearly the whole softmax wherever it can be seen."""
    rt = rt_for(dt)
    params, cfg = STANDOUT
    mixer = windowed_part(32, params)
    wq = torch.randn(32, 32, generator=torch.Generator().manual_seed(1)) * 32 ** -0.5
    W = bind_random(mixer, rt, 15, {"q": wq, "k": -wq})
    for query, planted in PAIRS:
        x = inputs(query + 1, 32, 100 + query, dt)
        x[planted] = -x[query]
        want = pr.windowed_attention(x, W, "p.", cfg, 1e-3)
        moved = x.clone()
        moved[planted] = inputs(1, 32, 999, dt)[0]
        seen = bool((want[query] - pr.windowed_attention(moved, W, "p.", cfg, 1e-3)[query]).abs().max() > 0.2 * want[query].abs().max())
        assert seen == (query - planted < 24 or planted < 5), "the plain implementation disagrees with the rule"
        h = Harness(mixer, rt, pages=24)
        got = run_in_portions(h, x, [query, 1] if decode else ([5, query - 4] if query > 5 else [query + 1]))
        close(got[query], want[query], dt, f"query {query}, planted key {planted}")


@pytest.mark.parametrize("dt", DTYPES)
def test_values_mix_by_relative_position_and_the_sink_takes_its_share(dt):
    """With equal keys and inputs everywhere, values turned by their positions and turned back differ from plain values by a phase per
    distance; and the softmax over n equal scores s gives each key e^s / (1 + n e^s): both show at the first tokens."""
    rt = rt_for(dt)
    params, cfg = windowed(1, 1, 16, 16, 1e-4, 0, 3.0, None, 12, 2)
    mixer = windowed_part(16, params)
    W = bind_random(mixer, rt, 16)
    x = inputs(1, 16, 3, dt).expand(30, 16).contiguous()
    want = pr.windowed_attention(x, W, "p.", cfg, 1e-3)
    v = x[:1] @ W["p.v"].T
    assert torch.allclose(want[0], 0.5 * v[0] @ W["p.o"].T, atol=1e-3 * v.abs().max().item())       # one key beside the constant
    unturned = pr.softmax_attention(torch.zeros(30, 1, 16), torch.zeros(30, 1, 16), v.expand(30, 16)[:, None], 1.0, cfg["mask"], torch.zeros(1))
    assert (unturned.reshape(30, 16) @ W["p.o"].T - want)[20:].abs().max() > 0.1 * want.abs().max(), "the rotation of the values must matter"
    h = Harness(mixer, rt)
    close(run_in_portions(h, x, [30]), want, dt, "whole", bf16=2e-2)
    close(run_in_portions(h, x, [1] * 30), want, dt, "token by token", bf16=2e-2)


# ----------------------------------------------------------------------------------------------- latent attention

def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, scaling, hidden=40):
    part = dict(hidden_size=hidden, num_heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=None, kv_rank=kv_rank, scale=scale, rot_dims=rot_dim,
                rot_base=base, eps=1e-3, gate="head", sink=True, rot_pairing="half", rot_scaling=dict(scaling, kind="yarn") if scaling else None)
    cfg = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    if scaling:
        cfg["rot"]["scaling"] = scaling
    return part, cfg


YARN = dict(factor=6.0, original=40, fast=8.0, slow=1.0)
LATENT = [latent(3, 16, 8, 32, 24, 0.3, 500.0, YARN), latent(1, 48, 16, 64, 16, 0.15, 1e4, dict(factor=1.0, original=300, fast=20.0, slow=1.0)),
          latent(2, 96, 32, 128, 40, 0.1, 3e4, dict(factor=32.0, original=30, fast=2.0, slow=0.5)), latent(5, 10, 6, 20, 9, 0.4, 100.0, YARN),
          latent(2, 120, 24, 40, 32, 0.1, 1e4, YARN), latent(4, 16, 48, 16, 48, 0.2, 1e3, None), latent(7, 56, 56, 40, 112, 0.1, 2e5, YARN, hidden=72)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", LATENT)
def test_latent_attention_whole_in_portions_token_by_token_and_in_batches(dt, case):
    rt = rt_for(dt)
    params, cfg = case
    mixer = build("mixer", "latent_attention", **params)
    assert set(mixer.tensor_specs()) == {"q", "dkv", "dkv.norm", "uk", "uv", "o", "g", "sink"} and mixer.tensor_specs()["g"].shape == (params["num_heads"], params["hidden_size"])
    sinks = torch.tensor([1.0, -0.5, 3.0, 0.0, 2.0, -4.0, 0.5, 1.5][:params["num_heads"]])
    W = bind_random(mixer, rt, 27, {"sink": sinks})
    hid = params["hidden_size"]
    x = inputs(120, hid, 1, dt)
    want = pr.latent_attention(x, W, "p.", cfg, 1e-3)
    far_sink = dict(W, **{"p.sink": torch.full_like(sinks, -30.0)})
    assert (pr.latent_attention(x, far_sink, "p.", cfg, 1e-3) - want).abs().max() > 0.05 * want.abs().max(), "the sink must matter"
    h = Harness(mixer, rt, pages=32, slots=3)
    close(run_in_portions(h, x, [120]), want, dt, "whole")
    close(run_in_portions(h, x, [33, 1, 1, 14, 2, 17, 2, 50]), want, dt, "portions")
    close(run_in_portions(h, x, [1] * 120), want, dt, "token by token")
    xs = [inputs(n, hid, 20 + i, dt) for i, n in enumerate((40, 9, 131))]
    rcs, cuts = [h.new() for _ in xs], [(17, 23), (8, 1), (130, 1)]
    first = h.step([(rc, xi[:a]) for rc, xi, (a, _) in zip(rcs, xs, cuts)])
    second = h.step([(rc, xi[a:]) for rc, xi, (a, _) in zip(rcs, xs, cuts)])
    for i, (f, s) in enumerate(zip(first, second)):
        close(torch.cat([f, s], 0), pr.latent_attention(xs[i], W, "p.", cfg, 1e-3), dt, f"request {i} of a batch")
        h.free(rcs[i])
    h.manager.check()


@pytest.mark.parametrize("dt", DTYPES)
def test_rescaled_rotation_shows_in_the_scores(dt):
    """Queries and keys that live in the rotated part alone: angles (frequencies) and lengths (the gain) both decide the output."""
    rt = rt_for(dt)
    params, cfg = latent(2, 8, 16, 16, 16, 0.5, 30.0, dict(factor=5.0, original=48, fast=6.0, slow=1.0))
    mixer = build("mixer", "latent_attention", **params)
    q = torch.randn(2, 24, 40, generator=torch.Generator().manual_seed(2)) * 0.3
    q[:, :8] = 0.0
    W = bind_random(mixer, rt, 31, {"q": q.reshape(48, 40), "sink": torch.zeros(2)})
    x = inputs(100, 40, 4, dt)
    want = pr.latent_attention(x, W, "p.", cfg, 1e-3)
    plain = {**cfg, "rot": dict(base=30.0, dims=16)}
    assert (pr.latent_attention(x, W, "p.", plain, 1e-3) - want).abs().max() > 0.05 * want.abs().max(), "the rescaling must matter"
    h = Harness(mixer, rt)
    close(run_in_portions(h, x, [100]), want, dt, "whole")
    close(run_in_portions(h, x, [60, 2] + [1] * 38), want, dt, "decoded")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("far", [0, 15, 16, 31, 32, 63, 64, 127, 128, 250, 296])
def test_a_key_far_back_that_stands_out(dt, far):
    """W_q = -W_uk W_dkv, so that a key made from minus the query's input scores |q|^2 against a softmax of hundreds, while the
    query's own key scores the opposite."""
    rt = rt_for(dt)
    params, cfg = latent(2, 32, 8, 48, 24, 1.0, 100.0, YARN)
    mixer = build("mixer", "latent_attention", **params)
    g = torch.Generator().manual_seed(5)
    dkv, uk = torch.randn(32, 40, generator=g) * 40 ** -0.5, torch.randn(64, 24, generator=g) * 24 ** -0.5
    q = torch.zeros(2, 40, 40)
    q[:, :32] = -(uk @ dkv[:24]).reshape(2, 32, 40)
    W = bind_random(mixer, rt, 28, {"dkv": dkv, "uk": uk, "q": q.reshape(80, 40), "dkv.norm": torch.ones(24), "sink": torch.zeros(2)})
    T = 300
    x = inputs(T, 40, 2, dt)
    without = x.clone()
    x[T - 3:] = x[T - 1] + 0.05 * inputs(3, 40, 77, dt)
    x[T - 3:] = x[T - 3:].to(dt).float()
    without[T - 3:] = x[T - 3:]
    x[far] = -x[T - 1]
    want, lost = pr.latent_attention(x, W, "p.", cfg, 1e-3), pr.latent_attention(without, W, "p.", cfg, 1e-3)
    assert (want[-3:] - lost[-3:]).abs().max() > 0.2 * want[-3:].abs().max(), "the planted key must matter"
    h = Harness(mixer, rt, pages=24, slots=1)
    close(run_in_portions(h, x, [T]), want, dt, "whole")
    close(run_in_portions(h, x, [T - 5, 2, 1, 1, 1]), want, dt, "the last queries decoded alone")
    close(run_in_portions(h, x, [7, 9, 1, 15, 2, 200, 61, 3, 2]), want, dt, "portions cut inside pages")
