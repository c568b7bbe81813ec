"""The mechanisms of the Karopel design one by one, built through the part registry with sizes of their own, against the plain
functions of ``plain_karopel``: the norms on both sides of a sublayer with what comes between layers, the silu-gated feed-forward,
the slope by distance in every attention kernel, attention that keeps the first tokens, attention whose keys serve as values, the
gated delta rule with one decay per head, and the two side by side.  Mixers run a sequence whole, in portions down to one token,
and several requests in one batch, from pages and slots that other requests used before."""
from types import SimpleNamespace

import pytest
import torch

import plain_karopel as pk
from helpers import close as close_at, scattered_tables
from test_getizen_parts_gpu import DEV, DTYPES, Harness, bind_random, build, inputs, rt_for, run_in_portions

pytestmark = pytest.mark.gpu
BF16 = torch.bfloat16


def close(got, want, dtype, what="", bf16=4e-2, rounded=None):
    """bfloat16 mixers round their projections, keys, values and heads in turn: twice the bound of a single kernel, or three times what
    rounding alone does to the plain implementation (``rounded``: its result with rounding) where that is more -- a head whose
    read-out is small before its norm, or a key of one entry, magnifies it."""
    if dtype == torch.float32:
        return close_at(got, want, dtype, what)
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    err, scale = (got - want).abs().max().item(), max(want.abs().max().item(), 1e-6)
    bound = max(bf16 * scale, 3.0 * (rounded - want).abs().max().item() if rounded is not None else 0.0)
    assert err <= bound, f"{what}: max abs error {err:.3e} > {bound:.3e}, scale {scale:.3e}"


# ----------------------------------------------------------------------------------------------- norms, shifts, feed-forward

@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n", [40, 42, 52, 260, 1024, 4096, 8192])
@pytest.mark.parametrize("T", [6, 200])
def test_norms_on_both_sides_of_a_sublayer_and_what_comes_between_layers(dt, n, T):
    from mini_inference_engine_b200.parts import Branches, NormedDelta
    from mini_inference_engine_b200.parts.norm import apply_pending
    rt = rt_for(dt)
    eps, mult = 3e-3, 0.7
    norm, after = build("norm", "zero_centered_rmsnorm", size=n, eps=eps, gain=1.0), build("norm", "zero_centered_rmsnorm", size=n, eps=eps, gain=mult)
    g = torch.Generator().manual_seed(n)
    rnd = lambda *s: torch.randn(*s, generator=g)
    w, wb = (bind_random(p, rt, s, {"weight": 0.3 * rnd(n)})["p.weight"] for p, s in ((norm, 1), (after, 2)))
    res, a, b, e, step = rnd(T, n) * 0.2 + 0.1, rnd(T, n) * 0.05, rnd(T, n) * 0.1, rnd(T, n), rnd(n)
    added = lambda y: mult * pk.norm_about_one(y, wb, eps)
    d = lambda t: t.to(DEV)
    cases = {
        "nothing pending": (None, res),
        "one output": (NormedDelta(d(a), after), res + added(a)),
        "two outputs with coefficients": (NormedDelta(Branches((d(a), d(b)), coefs=(1.5, -0.4)), after), res + added(1.5 * a - 0.4 * b)),
        "a bfloat16 output": (NormedDelta(d(a.to(BF16)), after), res + added(a.to(BF16).float())),
        "a shift": (NormedDelta(shift=d(step)), res + step),
        "an output, the embedding and a shift": (NormedDelta(d(b), after, d(e), d(step)), res + added(b) + e + step),
    }
    for what, (pending, x) in cases.items():
        r = d(res.clone())
        out = norm(pending, r)
        close_at(r, x, torch.float32, what + ": stream")
        close_at(out, pk.norm_about_one(x, w, eps), dt, what + ": normed")
        rows = torch.tensor([5, 0, 5, 3], dtype=torch.int32, device=DEV)
        r = d(res.clone())
        close_at(norm(pending, r, rows), pk.norm_about_one(x, w, eps)[[5, 0, 5, 3]], dt, what + ": gathered")
        assert torch.equal(r.cpu(), res), "gathering leaves the stream as it is"
        if pending is not None:
            r = d(res.clone())
            assert apply_pending(pending, r, eps) is None
            close_at(r, x, torch.float32, what + ": without a reader")
    with pytest.raises(ValueError):
        norm(d(a), d(res))                                                # an output without its norm
    # a norm's gain in front of the head is a factor on the logits
    scaled = build("norm", "zero_centered_rmsnorm", size=n, eps=eps, gain=0.37)
    bind_random(scaled, rt, 1, {"weight": w})
    close_at(scaled(None, d(res.clone())), 0.37 * pk.norm_about_one(res, w, eps), dt, "gain")


def test_a_row_that_does_not_exist_is_reported_and_not_read():
    from mini_inference_engine_b200.kernels import ops
    norm = build("norm", "zero_centered_rmsnorm", size=64, eps=1e-5)
    bind_random(norm, rt_for(torch.float32), 1)
    norm(None, torch.randn(4, 64, device=DEV), torch.tensor([1, 4], dtype=torch.int32, device=DEV))
    torch.cuda.synchronize()
    with pytest.raises(ops.KernelError, match="sandwich_norm"):
        ops.check_range_errors()


@pytest.mark.parametrize("with_embedding", [False, True])
def test_shift_in_front_of_a_pass(with_embedding):
    from mini_inference_engine_b200.parts import NormedDelta
    rt = rt_for(torch.float32)
    part = build("connection", "stream_shift", hidden_size=24, rows=3, index=1, with_embedding=with_embedding)
    W = bind_random(part, rt, 7)
    e = torch.randn(5, 24, device=DEV)
    pending = part.pending(NormedDelta(e, None), SimpleNamespace(extras={"embedding_output": e}))
    assert torch.equal(pending.shift.cpu(), W["p.step"][1]) and (pending.extra is e) == with_embedding and pending.y is e
    if with_embedding:
        with pytest.raises(ValueError):
            part.pending(None, SimpleNamespace(extras={}))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T", [1, 9, 40, 200])
@pytest.mark.parametrize("hidden,ff", [(64, 144), (50, 36)])
def test_silu_gated_feed_forward(dt, T, hidden, ff):
    rt = rt_for(dt)
    part = build("feed_forward", "clamped_glu", hidden_size=hidden, intermediate_size=ff, limit=0.0, slope=1.0, shift=0.0)
    W = bind_random(part, rt, 4)
    x = inputs(T, hidden, 1, dt) * 4                                       # large enough for a clamp to bite
    close(part.forward(x.to(dt).to(DEV), None), pk.feed_forward(x, W, "p."), dt, f"{T} tokens", bf16=2e-2)


# ----------------------------------------------------------------------------------------------- the slope, kernel by kernel

def sloped_case(ops, kernel, dt, H, G, D, page, rows, window, slope, seed=0, sinks=None, shared=False, keep=0, loud=(), **more):
    """Rows of (new tokens, context) through one attention kernel, scores minus slope times distance.  ``shared``: one tensor is
    given as keys and values.  ``loud``: key positions whose scores stand out by what the slope takes off at that distance."""
    g = torch.Generator().manual_seed(seed)
    T, n_pages = sum(a for a, _ in rows), sum(-(-c // page) for _, c in rows) + 3
    tables = scattered_tables([c for _, c in rows], page, n_pages, seed)
    kc, vc = torch.zeros(n_pages, G, page, D).to(dt), torch.zeros(n_pages, G, page, D).to(dt)
    q_all = torch.randn(T, H, D, generator=g).to(dt)
    scale, want, at = D ** -0.5, [], 0
    block = torch.zeros(len(rows), max(len(t) for t in tables), dtype=torch.int32)
    for r, (n, ctx) in enumerate(rows):
        k = torch.randn(ctx, G, D, generator=g)
        for j in loud:
            if j < ctx:
                q = q_all[at + n - 1].float().view(G, H // G, D)[:, 0]
                k[j] = q * ((slope[0] * (ctx - 1 - j) + 4.0) / scale / (q * q).sum(-1, keepdim=True))
        k = k.to(dt)
        v = k if shared else torch.randn(ctx, G, D, generator=g).to(dt)
        for j in range(ctx):
            kc[tables[r][j // page], :, j % page], vc[tables[r][j // page], :, j % page] = k[j], v[j]
        block[r, :len(tables[r])] = torch.tensor(tables[r], dtype=torch.int32)
        q = torch.zeros(ctx, H, D)
        q[ctx - n:] = q_all[at:at + n].float()
        mask = dict(size=window, keep_first=keep) if window else None
        o = pk.softmax_heads(q, k.float(), v.float(), scale, pk.visible(ctx, mask), sink=sinks, slope=slope)
        want.append(o[ctx - n:])
        at += n
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    starts = [sum(a for a, _ in rows[:i]) for i in range(len(rows))]
    out = torch.full((T, H, D), 9.0, dtype=dt, device=DEV)
    kd = kc.to(DEV)
    args = (q_all.to(DEV), H * D, kd, kd if shared else vc.to(DEV), block.to(DEV), i32(starts), i32([a for a, _ in rows]), i32([c for _, c in rows]))
    mods = ops.ScoreMods(sink=None if sinks is None else sinks.to(DEV), slope=torch.tensor(slope, dtype=torch.float32, device=DEV))
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
SLOPES = [(0.5, 0.01, 0.0, 2.0), (0.0625, 0.25, 1e-3, 0.7)]


@pytest.mark.parametrize("slope", SLOPES)
@pytest.mark.parametrize("window,with_sink,shared", [(None, False, False), (72, False, True), (130, True, False), (None, True, True), (1, False, True)])
@pytest.mark.parametrize("kernel,dt,D,page", [("simt", torch.float32, 48, 16), ("simt", BF16, 32, 64), ("prefill", BF16, 48, 16), ("prefill", BF16, 80, 128),
                                              ("prefill_tc", BF16, 64, 16), ("prefill_tc", BF16, 128, 32), ("prefill_tc", BF16, 64, 256)])
def test_slope_in_portions(kernel, dt, D, page, window, with_sink, shared, slope):
    from mini_inference_engine_b200.kernels import ops
    sinks = torch.tensor([1.0, -0.5, 2.0, 0.0]) if with_sink else None
    out, want = sloped_case(ops, kernel, dt, 4, 2, D, page, PORTIONS, window, slope, seed=D, sinks=sinks, shared=shared, loud=(0, 17, 250))
    close_at(out, want, dt, f"{kernel} window {window} sink {with_sink}")


@pytest.mark.parametrize("how", [dict(), dict(splits=1), dict(splits=2, merge="cluster"), dict(splits=8, merge="cluster", tma=True),
                                 dict(splits=5, merge="scratch", min_part_tiles=1), dict(splits=3, merge="scratch", tma=True, stages=2)])
@pytest.mark.parametrize("window,with_sink,shared", [(None, False, False), (72, False, True), (200, True, True)])
@pytest.mark.parametrize("H,G,D,page", [(6, 2, 64, 16), (4, 4, 48, 32), (20, 1, 128, 16)])
def test_slope_in_decoding(H, G, D, page, window, with_sink, shared, how):
    from mini_inference_engine_b200.kernels import ops
    rows = [(1, c) for c in (1, 2, 17, 64, 65, 130, 257, 300, 705)]
    slope = [0.4 / (1 + h) for h in range(H)]
    sinks = torch.linspace(-1.0, 2.0, H) if with_sink else None
    out, want = sloped_case(ops, "decode", BF16, H, G, D, page, rows, window, slope, seed=H, sinks=sinks, shared=shared, loud=(0, 17, 250), **how)
    close_at(out, want, BF16, f"decode window {window} {how}")


def test_slope_beside_kept_keys_takes_the_kernels_that_have_both():
    from mini_inference_engine_b200.kernels import ops
    mods = ops.ScoreMods(slope=torch.zeros(1))
    assert mods.tcgen05_takes(0) and not mods.tcgen05_takes(3)
    assert not ops.ScoreMods(softcap=2.0, slope=torch.zeros(1)).tcgen05_takes(0) and ops.ScoreMods(softcap=2.0).tcgen05_takes(0)
    for kernel, dt in (("simt", torch.float32), ("prefill", BF16)):
        out, want = sloped_case(ops, kernel, dt, 4, 2, 64, 16, PORTIONS, 40, (0.03, 0.01, 0.2, 0.0), keep=7, loud=(0, 6, 7))
        close_at(out, want, dt, kernel)
    out, want = sloped_case(ops, "decode", BF16, 4, 2, 64, 16, [(1, c) for c in (3, 50, 300)], 40, (0.03, 0.01, 0.2, 0.0), keep=7, loud=(0, 6, 7))
    close_at(out, want, BF16, "decode")


def test_slope_where_a_block_takes_two_query_tiles():
    from mini_inference_engine_b200.kernels import ops
    for D in (64, 128):
        slope = [2.0 ** (-8.0 * (h + 1) / 32) for h in range(32)]
        out, want = sloped_case(ops, "prefill_tc", BF16, 32, 4, D, 16, [(900, 900), (400, 1000), (7, 300)], 150, slope, seed=D, shared=True)
        close_at(out, want, BF16, f"pairs of query tiles, heads of {D}")


# ----------------------------------------------------------------------------------------------- mixers: shared checks

def check_mixer(mixer, rt, dt, plain, hidden, T=150, pages=40, slots=4, tail_lengths=(90, 3, 131), batch_cuts=((60, 30), (2, 1), (130, 1))):
    x = inputs(T, hidden, 5, dt)
    want, rounded = plain(x), plain(x, pk.to_bf16)
    h = Harness(mixer, rt, pages=pages, slots=slots)
    close(run_in_portions(h, x, [T]), want, dt, rounded=rounded, what="whole")
    close(run_in_portions(h, x, [T - 127, 2, 30, 1, 1, 20, 2, 21, 50]), want, dt, rounded=rounded, what="portions")
    close(run_in_portions(h, x, [1] * T), want, dt, rounded=rounded, what="token by token")
    close(run_in_portions(h, x, [2] * (T // 2)), want, dt, rounded=rounded, what="two by two")
    xs = [inputs(n, hidden, 40 + n, dt) for n in tail_lengths]
    rcs = [h.new() for _ in xs]                                            # pages and slots that the runs above used and gave back
    first = h.step([(rc, xi[:a]) for rc, xi, (a, _) in zip(rcs, xs, batch_cuts)])
    second = h.step(list(reversed([(rc, xi[a:]) for rc, xi, (a, _) in zip(rcs, xs, batch_cuts)])))
    for i, (f, s) in enumerate(zip(first, reversed(second))):
        close(torch.cat([f, s], 0), plain(xs[i]), dt, rounded=plain(xs[i], pk.to_bf16), what=f"request {i} of a batch")
        h.free(rcs[i])
    h.manager.check()


# ----------------------------------------------------------------------------------------------- attention that keeps the first tokens

def windowed(heads, kv_heads, dim, vdim, scale, dims, base, scaling, window, keep):
    part = dict(num_heads=heads, num_kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot_dims=dims, rot_base=base, window=window, keep_first=keep,
                rot_scaling=dict(scaling, kind="wavelength") if scaling else None)
    cfg = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=dims))
    if scaling:
        cfg["rot"]["scaling"] = scaling
    if window:
        cfg["mask"] = dict(size=window, keep_first=keep)
    return part, cfg


def windowed_part(hidden, part):
    return build("mixer", "gated_attention", hidden_size=hidden, eps=1e-3, qk_norm="head", head_temp=False, gate=False, sink=True, rot_pairing="interleaved", **part)


LLAMA3 = dict(factor=4.0, low=1.0, high=4.0, original=60)
WINDOWED = [windowed(4, 2, 32, 32, 0.3, 16, 50.0, LLAMA3, 24, 5), windowed(3, 3, 16, 48, 0.5, 16, 1e4, dict(factor=8.0, low=0.5, high=2.0, original=300), 16, 20),
            windowed(6, 1, 64, 32, 0.15, 0, 1e6, None, None, 0), windowed(2, 1, 128, 96, 0.09, 64, 1e3, LLAMA3, 1, 1),
            windowed(5, 1, 48, 64, 0.2, 2, 200.0, None, 40, 0), windowed(1, 1, 144, 160, 0.1, 32, 9e3, LLAMA3, 33, 70), windowed(6, 2, 10, 6, 0.6, 4, 30.0, LLAMA3, 17, 3)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", WINDOWED)
def test_windowed_attention(dt, case):
    rt = rt_for(dt)
    params, cfg = case
    mixer = windowed_part(40, params)
    assert set(mixer.tensor_specs()) == {"q", "k", "v", "o", "q.norm", "k.norm", "sink"}
    sinks = torch.tensor([1.0, -0.5, 3.0, 0.0, 2.0, -4.0][:params["num_heads"]])
    W = bind_random(mixer, rt, 14, {"sink": sinks})
    x = inputs(150, 40, 5, dt)
    no_sink = dict(W, **{"p.sink": torch.full_like(sinks, -30.0)})
    want = pk.attention(x, W, "p.", cfg, 1e-3)
    assert (pk.attention(x, no_sink, "p.", cfg, 1e-3) - want).abs().max() > 0.05 * want.abs().max(), "the sink must matter"
    check_mixer(mixer, rt, dt, lambda z, *r: pk.attention(z, W, "p.", cfg, 1e-3, *r), 40)


EDGE_PAIRS = [(70, 47), (70, 46), (70, 4), (70, 5), (70, 0), (95, 72), (95, 71), (23, 0), (24, 0), (28, 4), (28, 5), (29, 5), (29, 4), (200, 177), (200, 176),
              (200, 4), (200, 5), (200, 15), (200, 16), (40, 39), (300, 0), (300, 4), (300, 5), (300, 130)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
def test_a_key_that_stands_out_at_the_edges_of_the_window_and_of_the_kept_tokens(dt, decode):
    """W_k = -W_q and the planted input is minus the query's: its key equals the query (whose own key is its opposite), so it takes
    nearly the whole softmax wherever it can be seen."""
    rt = rt_for(dt)
    params, cfg = windowed(2, 2, 16, 16, 0.8, 0, 1e4, None, 24, 5)
    mixer = windowed_part(32, params)
    wq = torch.randn(32, 32, generator=torch.Generator().manual_seed(1)) * 32 ** -0.5
    W = bind_random(mixer, rt, 15, {"q": wq, "k": -wq, "q.norm": torch.ones(16), "k.norm": torch.ones(16), "sink": torch.zeros(2)})
    plain = lambda z: pk.attention(z, W, "p.", cfg, 1e-3)
    for query, planted in EDGE_PAIRS:
        x = inputs(query + 1, 32, 100 + query, dt)
        x[planted] = -x[query]
        want = plain(x)
        moved = x.clone()
        moved[planted] = inputs(1, 32, 999, dt)[0]
        seen = bool((want[query] - plain(moved)[query]).abs().max() > 0.2 * want[query].abs().max())
        assert seen == (query - planted < 24 or planted < 5), "the plain implementation disagrees with the rule"
        h = Harness(mixer, rt, pages=24)
        got = run_in_portions(h, x, [query, 1] if decode else ([5, query - 4] if query > 5 else [query + 1]))
        close(got[query], want[query], dt, f"query {query}, planted key {planted}")


@pytest.mark.parametrize("dt", DTYPES)
def test_kept_first_tokens_turn_by_their_true_positions(dt):
    """Queries and keys that live in one fast pair: a kept key whose position were counted from the window's start would score
    otherwise."""
    rt = rt_for(dt)
    params, cfg = windowed(1, 1, 16, 16, 2.0, 2, 1e4, dict(factor=2.0, low=1.0, high=4.0, original=4096), 10, 6)
    mixer = windowed_part(16, params)
    only = torch.zeros(16, 16)
    only[:2] = torch.randn(2, 16, generator=torch.Generator().manual_seed(3)) * 0.5
    W = bind_random(mixer, rt, 16, {"q": only, "k": only, "q.norm": torch.ones(16), "k.norm": torch.ones(16), "sink": torch.full((1,), -2.0)})
    x = inputs(220, 16, 9, dt)
    want = pk.attention(x, W, "p.", cfg, 1e-3)
    h = Harness(mixer, rt)
    close(run_in_portions(h, x, [220]), want, dt, "whole")
    close(run_in_portions(h, x, [100] + [1] * 120), want, dt, "decoded")


# ----------------------------------------------------------------------------------------------- keys that serve as values

def keyed(heads, kv_heads, dim, scale, window):
    part = dict(num_heads=heads, num_kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, window=window, slopes=tuple(pk.slopes(heads)))
    cfg = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask=dict(size=window) if window else None)
    return part, cfg


def keyed_part(hidden, part):
    return build("mixer", "gated_attention", hidden_size=hidden, eps=1e-3, rot_dims=0, rot_base=1.0, qk_norm=False, head_temp=False, gate=False,
                 keys_as_values=True, **part)


KEYED = [keyed(4, 2, 32, 0.3, 24), keyed(3, 3, 16, 0.5, 16), keyed(6, 1, 64, 0.15, 50), keyed(2, 1, 128, 0.09, 1), keyed(5, 1, 48, 0.2, 40), keyed(1, 1, 160, 0.1, 33),
         keyed(12, 4, 10, 0.4, 130), keyed(7, 7, 64, 0.2, None)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", KEYED)
def test_keys_as_values_with_a_slope(dt, case):
    rt = rt_for(dt)
    params, cfg = case
    mixer = keyed_part(40, params)
    assert set(mixer.tensor_specs()) == {"q", "k", "o"} and mixer.cache_need().shared
    W = bind_random(mixer, rt, 18)
    check_mixer(mixer, rt, dt, lambda z, *r: pk.keys_as_values(z, W, "p.", cfg, 1e-3, *r), 40)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
def test_a_key_that_stands_out_at_the_edge_of_a_sloped_window(dt, decode):
    """W_k = -W_q and the planted input is -1.5 times the query's: its score beats what the slope takes off at that distance, so it takes the
    softmax just inside the window and is not there just outside."""
    rt = rt_for(dt)
    params, cfg = keyed(2, 2, 16, 1.0, 24)
    mixer = keyed_part(32, params)
    wq = torch.randn(32, 32, generator=torch.Generator().manual_seed(1)) * 32 ** -0.5
    W = bind_random(mixer, rt, 19, {"q": wq, "k": -wq})
    plain = lambda z: pk.keys_as_values(z, W, "p.", cfg, 1e-3)
    for query, planted in [(70, 47), (70, 46), (70, 48), (95, 72), (95, 71), (23, 0), (24, 0), (25, 1), (31, 8), (32, 8), (40, 17), (40, 16), (200, 177), (200, 176), (48, 47)]:
        x = inputs(query + 1, 32, 100 + query, dt)
        x[planted] = -x[query] * 1.5
        want = plain(x)
        moved = x.clone()
        moved[planted] = inputs(1, 32, 999, dt)[0]
        seen = bool((want[query] - plain(moved)[query]).abs().max() > 0.2 * want[query].abs().max())
        assert seen == (query - planted < 24), "the plain implementation disagrees with the rule"
        h = Harness(mixer, rt, pages=24)
        got = run_in_portions(h, x, [query, 1] if decode else ([3, query - 2] if query > 3 else [query + 1]))
        close(got[query], want[query], dt, f"query {query}, planted key {planted}")


@pytest.mark.parametrize("dt", DTYPES)
def test_slope_alone_decides_between_equal_scores(dt):
    """Queries are zero: the weights are exp(-slope x distance) over the window, and nothing else."""
    rt = rt_for(dt)
    params, cfg = keyed(4, 1, 16, 1.0, 30)
    mixer = keyed_part(24, params)
    W = bind_random(mixer, rt, 20, {"q": torch.zeros(64, 24)})
    x = inputs(100, 24, 3, dt)
    k = (x @ W["p.k"].T)
    want = []
    for i in range(100):
        j = torch.arange(max(0, i - 29), i + 1)
        heads = [torch.softmax(-s * (i - j).float(), 0) @ k[j] for s in pk.slopes(4)]
        want.append(torch.cat(heads) @ W["p.o"].T)
    want = torch.stack(want)
    close_at(pk.keys_as_values(x, W, "p.", cfg, 1e-3), want, torch.float32, "the plain implementation")
    h = Harness(mixer, rt)
    close(run_in_portions(h, x, [100]), want, dt, "whole", bf16=2e-2)
    close(run_in_portions(h, x, [40] + [1] * 60), want, dt, "decoded", bf16=2e-2)


# ----------------------------------------------------------------------------------------------- gated delta rule, one decay per head

def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, hidden=40, eps=1e-5):
    return (dict(hidden_size=hidden, num_heads=heads, num_kv_heads=kv_heads, dim=dim, vdim=vdim, taps=conv, eps=eps),
            dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv))


DELTA = [delta(), delta(1, 1, 48, 8, 1), delta(2, 2, 128, 40, 2), delta(3, 1, 200, 16, 6), delta(2, 1, 8, 130, 3), delta(4, 4, 64, 64, 4), delta(6, 2, 128, 128, 4, hidden=72),
         delta(1, 1, 1, 3, 5), delta(2, 1, 100, 33, 4), delta(5, 5, 36, 256, 2)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("chunked_from", [2, 112])
@pytest.mark.parametrize("case", DELTA)
def test_delta_rule(dt, case, chunked_from, monkeypatch):
    from mini_inference_engine_b200.parts import delta as delta_parts
    monkeypatch.setattr(delta_parts, "CHUNKED_FROM", chunked_from)
    rt = rt_for(dt)
    params, cfg = case
    mixer = build("mixer", "head_delta", **params)
    assert mixer.tensor_specs()["a"].shape == (params["num_heads"], params["hidden_size"]) and mixer.tensor_specs()["dt_bias"].shape == (params["num_heads"],)
    W = bind_random(mixer, rt, 13)
    check_mixer(mixer, rt, dt, lambda z, *r: pk.gated_delta(z, W, "p.", cfg, params["eps"], *r), params["hidden_size"], pages=40, slots=3)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("rate", [-9.0, -2.0, 0.5, 4.0])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 64, 32), (2, 128, 128), (1, 40, 24)])
@pytest.mark.parametrize("chunked_from", [1, 40, 112])
def test_delta_rule_over_long_portions_at_every_rate_of_decay(dt, rate, heads, dim, vdim, chunked_from, monkeypatch):
    """Portions of several hundred tokens, of lengths around the multiples of 16, 32 and 64, from decays of almost 1 to states that
    vanish within a token; keys that repeat, so that the corrections of a token by the ones before it are large.  Which portions go
    in chunks and which token by token makes no difference."""
    from mini_inference_engine_b200.parts import delta as delta_parts
    monkeypatch.setattr(delta_parts, "CHUNKED_FROM", chunked_from)
    rt = rt_for(dt)
    params, cfg = delta(heads, 1, dim, vdim, 4)
    mixer = build("mixer", "head_delta", **params)
    W = bind_random(mixer, rt, 17, {"A_log": torch.full((heads,), rate), "dt_bias": torch.linspace(-1.0, 1.0, heads)})
    x = inputs(400, 40, 6, dt)
    x[100:300] = x[100:104].repeat(50, 1)
    want = pk.gated_delta(x.double(), {k: v.double() for k, v in W.items()}, "p.", cfg, params["eps"]).float()
    h = Harness(mixer, rt, pages=30, slots=1)
    for portions in ([400], [63, 64, 65, 127, 81], [15, 17, 31, 33, 96, 1, 128, 79], [1, 255, 144]):
        close(run_in_portions(h, x, portions), want, dt, f"portions {portions}")


@pytest.mark.parametrize("dt", DTYPES)
def test_delta_rule_state_holds_a_far_token_and_long_decoding(dt):
    """Decays of almost 1 (A_log far below zero): what the first token wrote is still read 260 tokens later, most of
    them decoded one by one.  A state that is lost, or cleared between steps, shows at once."""
    rt = rt_for(dt)
    params, cfg = delta(2, 2, 64, 16)
    mixer = build("mixer", "head_delta", **params)
    W = bind_random(mixer, rt, 14, {"A_log": torch.full((2,), -9.0)})
    x = inputs(260, 40, 4, dt)
    x[0] *= 4.0
    want, gone = pk.gated_delta(x, W, "p.", cfg, 1e-5), pk.gated_delta(x[1:], W, "p.", cfg, 1e-5)
    assert (want[-1] - gone[-1]).abs().max() > 0.02 * want[-1].abs().max(), "the first token must still matter at the end"
    h = Harness(mixer, rt, pages=24, slots=1)
    close(run_in_portions(h, x, [10] + [1] * 250), want, dt, "long decoding")
    close(run_in_portions(h, x, [130, 2, 1, 1, 126]), want, dt, "portions")


@pytest.mark.parametrize("dt", DTYPES)
def test_a_slot_that_is_used_again_starts_from_zero_and_rows_do_not_mix(dt):
    rt = rt_for(dt)
    params, cfg = delta(2, 1, 32, 32, 4)
    mixer = build("mixer", "head_delta", **params)
    W = bind_random(mixer, rt, 15, {"A_log": torch.full((2,), -9.0)})
    h = Harness(mixer, rt, pages=24, slots=2)
    plain = lambda z, *r: pk.gated_delta(z, W, "p.", cfg, 1e-5, *r)
    big = inputs(70, 40, 1, dt) * 8
    close(run_in_portions(h, big, [70]), plain(big), dt, "first user")
    for n in (1, 2, 3, 90):
        x = inputs(n, 40, 50 + n, dt)
        close(run_in_portions(h, x, [n]), plain(x), dt, f"{n} tokens on a used slot", rounded=plain(x, pk.to_bf16))
    # one row decodes while another takes long portions, in either order
    a, b = inputs(40, 40, 2, dt), inputs(200, 40, 3, dt)
    ra, rb, ga, gb = h.new(), h.new(), [], []
    ga += h.step([(ra, a[:20])])
    at = 0
    for i, n in enumerate((1, 130, 2, 1, 66)):
        entries = [(ra, a[20 + i:21 + i]), (rb, b[at:at + n])]
        outs = h.step(entries if i % 2 else entries[::-1])
        ga.append(outs[0 if i % 2 else 1])
        gb.append(outs[1 if i % 2 else 0])
        at += n
    close(torch.cat(ga, 0), plain(a[:25]), dt, "the row that decodes")
    close(torch.cat(gb, 0), plain(b), dt, "the row that takes portions")


@pytest.mark.parametrize("groups,dim,vdim,least", [(1, 128, 48, 1), (2, 64, 16, 30), (3, 36, 100, 64)])
def test_chunks_and_single_steps_of_several_rows_in_one_launch(groups, dim, vdim, least):
    """The chunked kernel and the token-by-token one share a batch: rows of ``least`` tokens or more and the others, each from a state of its own
    that is not zero, in slots out of order; both against the plain recurrence, outputs and states."""
    from mini_inference_engine_b200.kernels import ops
    H, G, lens, slots = 2 * groups, groups, (70, 1, 128, 29, 30, 64, 200, 3), (5, 2, 8, 1, 7, 3, 4, 6)
    T = sum(lens)
    g = torch.Generator().manual_seed(dim)
    unit = lambda z: z / z.norm(dim=-1, keepdim=True)
    q, k = unit(torch.randn(T, G, dim, generator=g)) * dim ** -0.5, unit(torch.randn(T, G, dim, generator=g) + 0.7)
    v, beta = torch.randn(T, H, vdim, generator=g), torch.rand(T, H, generator=g)
    log_decay = -torch.rand(T, H, generator=g) ** 4
    state = torch.randn(9, H, vdim, dim, generator=g)
    want, after, at = torch.zeros(T, H, vdim), state.clone(), 0
    for n, slot in zip(lens, slots):
        S = state[slot].double().transpose(1, 2)                       # [H, dim, vdim]
        for t in range(at, at + n):
            kk, qq = (z[t].double().repeat_interleave(H // G, 0) for z in (k, q))
            S = log_decay[t].double().exp()[:, None, None] * S
            u = beta[t].double()[:, None] * (v[t].double() - torch.einsum("hdv,hd->hv", S, kk))
            S = S + kk[:, :, None] * u[:, None, :]
            want[t] = torch.einsum("hdv,hd->hv", S, qq).float()
        after[slot] = S.transpose(1, 2).float()
        at += n
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    d = lambda t: t.reshape(t.shape[0], -1).contiguous().to(DEV)
    st, out = state.to(DEV), torch.full((T, H * vdim), 7.0, device=DEV)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    args = (i32(starts), i32(lens), i32(slots), st, out)
    sizes = dict(num_heads=H, num_kv_heads=G, dim=dim, vdim=vdim)
    long = [n for n in lens if n >= least]
    ops.delta_chunks(d(q), d(k), d(v), d(beta), d(log_decay), *args, min_len=least, work=(len(long), sum(long)) if groups != 2 else None, **sizes)
    torch.cuda.synchronize()
    for n, s0, slot in zip(lens, starts, slots):
        if n < least:
            assert (out[s0:s0 + n] == 7.0).all() and torch.equal(st[slot].cpu(), state[slot]), "a row below the bound is left alone"
    kq = (k * q).sum(-1)
    ops.delta_scan(d(q), d(k), d(v), d(beta), d(log_decay.exp()), d(kq), *args, below=least, **sizes)
    close_at(out.reshape(T, H, vdim), want, torch.float32, "outputs")
    close_at(st, after, torch.float32, "states")


# ----------------------------------------------------------------------------------------------- side by side

@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("left,right,scales", [(keyed(4, 2, 32, 0.3, 24), delta(4, 2, 16, 24), (1.4, 0.6)), (keyed(2, 1, 128, 0.1, 40), delta(1, 1, 64, 64, 2), (-0.5, 2.0))])
def test_both_side_by_side_under_the_norms_around_them(dt, left, right, scales):
    from mini_inference_engine_b200.config.model_config import PartSpec
    from mini_inference_engine_b200.parts import NormedDelta
    rt = rt_for(dt)
    (lp, lc), (rp, rc) = left, right
    lp = dict(lp, hidden_size=40, eps=1e-3, rot_dims=0, rot_base=1.0, qk_norm=False, head_temp=False, gate=False, keys_as_values=True)
    mixer = build("mixer", "parallel", hidden_size=40, branches={"left": PartSpec("gated_attention", lp), "right": PartSpec("head_delta", dict(rp, eps=1e-3))}, scales=scales)
    W = bind_random(mixer, rt, 21)
    m = dict(left=lc, right=rc, left_scale=scales[0], right_scale=scales[1])
    after = build("norm", "zero_centered_rmsnorm", size=40, eps=1e-3, gain=0.5)
    reader = build("norm", "zero_centered_rmsnorm", size=40, eps=1e-3)
    wb, w = bind_random(after, rt, 22)["p.weight"], bind_random(reader, rt, 23)["p.weight"]
    T = 120
    x, res = inputs(T, 40, 8, dt), inputs(T, 40, 9, torch.float32)
    stream = res + 0.5 * pk.norm_about_one(pk.parallel(x, W, "p.", m, 1e-3), wb, 1e-3)

    class Normed:                                                          # the harness runs a mixer: this one applies the norms behind it
        def __init__(self):
            self.at = 0

        def cache_need(self):
            return mixer.cache_need()

        def forward(self, rows, ctx, cache):
            r = res[self.at:self.at + rows.shape[0]].clone().to(DEV)
            self.at += rows.shape[0]
            out = reader(NormedDelta(mixer.forward(rows, ctx, cache), after), r)
            self.streams.append(r.cpu())
            return out

    for portions in ([T], [50, 2, 1, 1, 66]):
        runner = Normed()
        runner.streams = []
        got = run_in_portions(Harness(runner, rt, pages=20), x, portions)
        close(torch.cat(runner.streams, 0), stream, dt, f"stream {portions}", bf16=2e-2)
        close(got, pk.norm_about_one(stream, w, 1e-3), dt, f"normed {portions}")
