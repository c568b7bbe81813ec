"""Plain, slow Karopel: the oracle that the tests of this design compare with.

Whole sequences, no cache, no batching, on the CPU, one function per mechanism, written from the design's
equations and sharing no code with the package.  ``cfg`` is the parsed config.json, ``W`` a
``{tensor name: tensor}`` dict in the precision to compute in (float32 or float64).

The design in this file's notation (t: token index = position, x_t: residual stream):

  norm               n(v; w) = v / sqrt(mean v^2 + eps) * (1 + w)
  embedding          e_t = E[token_t], x_t = e_t
  order of layers    layers lo .. hi-1 run ``times`` times in a row with the same weights, the others once, in their place; right
                     before pass t of the stretch, x <- x + step[t], and before every pass but the first also x <- x + e
  layer              x <- x + m n(mixer(n(x; w1)); w1b), then x <- x + m n(ff(n(x; w2)); w2b); the second half may be absent
  attention          grouped query heads; q and k divided by their root mean square per head times a weight shared by the heads, then
                     their first dims turned (pairs of neighbours, frequencies rescaled by wavelength); score = q . k * scale;
                     keys j in (i - size, i] and the first ``keep`` of the sequence; exp(sink_head) in the denominator; Wo
  parallel           a * left(h) + b * right(h):
    left             grouped query heads, the value is the key; nothing turns; score = q . k * scale - slope_h (i - j) with
                     slope_h = 2^(-8 (h + 1) / heads); keys j in (i - size, i]; plain softmax; Wo
    right            q, k, v: causal convolution over time per channel, then silu; q, k to unit length per head, q / sqrt(dim);
                     S <- g S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q   with b = sigmoid(Wb h) and
                     g = exp(-exp(A_log) softplus(Wa h + dt_bias)) per head; o / rms(o) * w * silu(Wg h); Wo
  feed-forward       Wd (silu(Wgate h) * (Wup h))
  head               logits = W_head n(x; w_final) * logit_scale

``rnd`` (default: nothing) is applied where an implementation in 16 bits rounds -- operands and results of matrix products, heads before
and after attention -- so that a run with it shows how much rounding alone moves each row of logits.
"""
from __future__ import annotations

import math

import torch


def exact(z: torch.Tensor) -> torch.Tensor:
    return z


def to_bf16(z: torch.Tensor) -> torch.Tensor:
    return z.to(torch.bfloat16).to(z.dtype)


def over_rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def norm_about_one(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return over_rms(v, eps) * (1 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0)


# --------------------------------------------------------------------------- rotation

def speeds(rot: dict) -> list:
    """Radians a position for every pair, rescaled by wavelength when ``scaling`` says so."""
    out = []
    for i in range(int(rot["dims"]) // 2):
        f = float(rot["base"]) ** (-2.0 * i / int(rot["dims"]))
        s = rot.get("scaling")
        if s:
            wave, orig = 2.0 * math.pi / f, float(s["original"])
            if wave > orig / s["low"]:
                f = f / s["factor"]
            elif wave >= orig / s["high"]:
                share = (orig / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return out


def turn_neighbours(v: torch.Tensor, pos: torch.Tensor, per_pair: list) -> torch.Tensor:
    """v [T, heads, D]: entries 2i and 2i + 1 are a pair, turned by pos * per_pair[i]; what has no speed passes unchanged."""
    out = v.clone()
    for i, f in enumerate(per_pair):
        a = pos.to(torch.float64) * f
        c, s = torch.cos(a).to(v.dtype)[:, None], torch.sin(a).to(v.dtype)[:, None]
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


# --------------------------------------------------------------------------- softmax attention

def visible(T: int, mask: dict | None) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask:
        seen = seen & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))
    return seen


def slopes(heads: int) -> list:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def softmax_heads(q, k, v, scale: float, seen, sink=None, slope=None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    away = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if slope is not None:
            s = s - slope[h] * away
        s = s.masked_fill(~seen, float("-inf"))
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h].to(s.dtype).reshape(1, 1))
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(sink[h].to(s.dtype) - top)
        out[:, h] = (e / total) @ v[:, g]
    return out


def attention(h, W, p, m, eps, rnd=exact):
    T, H, G, D, Dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = over_rms(rnd(h @ W[p + "q"].T).reshape(T, H, D), eps) * W[p + "q.norm"]
    k = over_rms(rnd(h @ W[p + "k"].T).reshape(T, G, D), eps) * W[p + "k.norm"]
    v = rnd(h @ W[p + "v"].T).reshape(T, G, Dv)
    f = speeds(m["rot"])
    o = softmax_heads(rnd(turn_neighbours(q, pos, f)), rnd(turn_neighbours(k, pos, f)), v, float(m["scale"]), visible(T, m.get("mask")), sink=W[p + "sink"])
    return rnd(o.reshape(T, H * Dv)) @ W[p + "o"].T


def keys_as_values(h, W, p, m, eps, rnd=exact):
    T, H, G, D = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = rnd(h @ W[p + "q"].T).reshape(T, H, D)
    k = rnd(h @ W[p + "k"].T).reshape(T, G, D)
    o = softmax_heads(q, k, k, float(m["scale"]), visible(T, m.get("mask")), slope=slopes(H))
    return rnd(o.reshape(T, H * D)) @ W[p + "o"].T


# --------------------------------------------------------------------------- gated delta rule

def short_convolution(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, K], the last column for the token itself."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u], 0)
    return silu(sum(padded[j:j + T] * taps[:, j] for j in range(K)))


def delta_steps(q, k, v, beta, g):
    """q, k [T, H, D], v [T, H, Dv], beta, g [T, H] -> [T, H, Dv]; the state starts at zero."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def gated_delta(h, W, p, m, eps, rnd=exact):
    T, H, G, D, Dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (short_convolution(rnd(h @ W[p + n].T), W[p + n + ".conv"]) for n in "qkv")
    unit = lambda z: z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q.reshape(T, G, D)) * D ** -0.5, unit(k.reshape(T, G, D))
    q, k = (z.repeat_interleave(H // G, 1) for z in (q, k))
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = over_rms(delta_steps(q, k, v.reshape(T, H, Dv), beta, g), eps) * W[p + "norm"]
    return rnd(o.reshape(T, H * Dv) * silu(rnd(h @ W[p + "g"].T))) @ W[p + "o"].T


def parallel(h, W, p, m, eps, rnd=exact):
    return (float(m["left_scale"]) * keys_as_values(h, W, p + "left.", m["left"], eps, rnd)
            + float(m["right_scale"]) * gated_delta(h, W, p + "right.", m["right"], eps, rnd))


MIXERS = {"attention": attention, "parallel": parallel}


def feed_forward(h, W, p, rnd=exact):
    return rnd(silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# --------------------------------------------------------------------------- the model

def run_order(cfg: dict) -> list:
    """[(layer, pass number with the first layer of a pass, else None)]"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    lo, hi = int(loop["start"]), int(loop["stop"])
    order = [(i, None) for i in range(lo)]
    for t in range(int(loop["times"])):
        order += [(i, t if i == lo else None) for i in range(lo, hi)]
    return order + [(i, None) for i in range(hi, n)]


def before_pass(x, e, W, t: int):
    if t > 0:
        x = x + e
    return x + W["loop.step"][t]


def layer(x, W, p, spec, eps, m, rnd=exact):
    y = MIXERS[spec["type"]](rnd(norm_about_one(x, W[p + "norm1"], eps)), W, p + "mix.", spec["mixer"], eps, rnd)
    x = x + m * norm_about_one(y, W[p + "norm1b"], eps)
    if spec.get("mlp") is not None:
        y = feed_forward(rnd(norm_about_one(x, W[p + "norm2"], eps)), W, p + "mlp.", rnd)
        x = x + m * norm_about_one(y, W[p + "norm2b"], eps)
    return x


def forward(cfg: dict, W: dict, tokens, trace: list | None = None, rnd=exact) -> torch.Tensor:
    """Logits [T, vocab]; ``trace`` collects the stream after every layer run."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = e = W["embed"][torch.as_tensor(list(tokens))]
    for i, t in run_order(cfg):
        if t is not None:
            x = before_pass(x, e, W, t)
        x = layer(x, W, f"l{i}.", cfg["layers"][i], eps, m, rnd)
        if trace is not None:
            trace.append(x)
    return (rnd(norm_about_one(x, W["final.norm"], eps)) @ W["head"].T) * float(cfg.get("logit_scale", 1.0))
