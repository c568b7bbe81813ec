"""Plain, slow Radenex: the oracle that the tests of this design compare with.

Whole sequences, no cache, no batching, on the CPU, one function per mechanism, written from the design's
equations and sharing no code with the package.  ``cfg`` is the parsed config.json, ``W`` a
``{tensor name: tensor}`` dict in the precision to compute in (float32 or float64).

The design in this file's notation (t: token index = position, x_t: residual stream):

  embedding          x_t = E[token_t]
  order of layers    layers lo .. hi-1 run ``times`` times in a row with the same weights; the others run once, in their place
  layer              h = rms(x) w;  x <- x + (mixer(h) + ff(h)), rms(v) = v / sqrt(mean v^2 + eps); ff may be absent
  latent attention   q = Wq h, per head [plain | turned]; W_dkv h = [c | r]: c <- rms(c) w is a latent from which every head's
                     plain key (W_uk c) and value (W_uv c) come, r one turned key part for all heads; score =
                     (q_plain . k_plain + q_turned . r) scale; causal; exp(sink_head) in the softmax's denominator; the head's
                     output times sigmoid(Wg h)[head]; then Wo
  windowed attention q, k turned over a head's first dims, then divided by their root mean square over the head; the value at j
                     turned by j over all its dims, the output at i turned back by i; keys j in (i - w, i] and the first n keys;
                     1 more in the softmax's denominator; then Wo
  feed-forward       Wd relu(Wu h)^2
  head               logits = W_head (rms(x) w_final)

Turning by an angle a: the pair (u_i, u_{i + n/2}) becomes (u_i cos a - u_{i+n/2} sin a, u_{i+n/2} cos a + u_i sin a).
"""
from __future__ import annotations

import math

import torch


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


# --------------------------------------------------------------------------- rotation

def plain_speeds(dims: int, base: float) -> list:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def linear_speeds(dims: int, base: float, factor: float) -> list:
    return [f / factor for f in plain_speeds(dims, base)]


def yarn_speeds(dims: int, base: float, s: dict) -> tuple:
    """(speeds, factor on cos and sin)."""
    at = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_speeds(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def turn(v: torch.Tensor, pos: torch.Tensor, speeds: list, gain: float = 1.0) -> torch.Tensor:
    """v [T, heads, D]: the first 2 * len(speeds) entries of every head are turned by pos * speed, the rest passes unchanged."""
    n = len(speeds)
    a = pos.to(torch.float64)[:, None, None] * torch.tensor(speeds, dtype=torch.float64)
    c, s = (gain * torch.cos(a)).to(v.dtype), (gain * torch.sin(a)).to(v.dtype)
    u, w, rest = v[..., :n], v[..., n:2 * n], v[..., 2 * n:]
    return torch.cat([u * c - w * s, w * c + u * s, rest], -1)


# --------------------------------------------------------------------------- softmax attention

def visible(T: int, mask: dict | None) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask:
        seen = seen & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return seen


def softmax_attention(q, k, v, scale: float, mask: dict | None, sink: torch.Tensor) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv], sink [H]: exp(sink) is one more term of the denominator.  Returns [T, H, Dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(T, mask)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, float("-inf"))
        top = torch.maximum(s.max(-1, keepdim=True).values, sink[h].to(s.dtype).reshape(1, 1))
        e = torch.exp(s - top)
        out[:, h] = (e / (e.sum(-1, keepdim=True) + torch.exp(sink[h].to(s.dtype) - top))) @ v[:, g]
    return out


# --------------------------------------------------------------------------- mixers

def windowed_attention(h, W, p, m, eps):
    T, H, G, D, Dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    rot = m.get("rot")
    q = (h @ W[p + "q"].T).reshape(T, H, D)
    k = (h @ W[p + "k"].T).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, Dv)
    scaling = rot.get("scaling")
    speeds = linear_speeds(int(rot["dims"]), float(rot["base"]), float(scaling["factor"]) if scaling else 1.0)
    q, k = rms(turn(q, pos, speeds), eps), rms(turn(k, pos, speeds), eps)
    v_speeds = plain_speeds(Dv, float(rot["base"]))
    o = softmax_attention(q, k, turn(v, pos, v_speeds), float(m["scale"]), m.get("mask"), torch.zeros(H, dtype=h.dtype))
    return turn(o, -pos, v_speeds).reshape(T, H * Dv) @ W[p + "o"].T


def latent_attention(h, W, p, m, eps):
    T, H, D, R, Dv, C = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = torch.arange(T)
    rot = m["rot"]
    scaling = rot.get("scaling")
    speeds, gain = yarn_speeds(R, float(rot["base"]), scaling) if scaling else (plain_speeds(R, float(rot["base"])), 1.0)
    q = (h @ W[p + "q"].T).reshape(T, H, D + R)
    q = torch.cat([q[..., :D], turn(q[..., D:], pos, speeds, gain)], -1)
    down = h @ W[p + "dkv"].T
    c = rms(down[:, :C], eps) * W[p + "dkv.norm"]
    r = turn(down[:, None, C:], pos, speeds, gain)
    k = torch.cat([(c @ W[p + "uk"].T).reshape(T, H, D), r.expand(T, H, R)], -1)
    v = (c @ W[p + "uv"].T).reshape(T, H, Dv)
    o = softmax_attention(q, k, v, float(m["scale"]), None, W[p + "sink"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * Dv) @ W[p + "o"].T


MIXERS = {"attention": windowed_attention, "latent_attention": latent_attention}


def feed_forward(h, W, p):
    return torch.relu(h @ W[p + "up"].T).square() @ W[p + "down"].T


# --------------------------------------------------------------------------- the model

def run_order(cfg: dict) -> list:
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    lo, hi, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return list(range(lo)) + list(range(lo, hi)) * times + list(range(hi, n))


def layer(x, W, p, spec, eps):
    h = rms(x, eps) * W[p + "norm1"]
    y = MIXERS[spec["type"]](h, W, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        y = y + feed_forward(h, W, p + "mlp.")
    return x + y


def forward(cfg: dict, W: dict, tokens, trace: list | None = None) -> torch.Tensor:
    """Logits [T, vocab]; ``trace`` collects the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(list(tokens))]
    for i in run_order(cfg):
        x = layer(x, W, f"l{i}.", cfg["layers"][i], eps)
        if trace is not None:
            trace.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T
