"""Karopel: a decoder whose layers norm each sublayer's input and its output (weights stored around zero), listed one by one in
config.json, each with a mixer of its own kind and sizes, and of which a stretch may run several times in a row with the same
weights.

config.json: ``architecture`` "Karopel", ``vocab``, ``width``, ``norm`` {eps}, ``residual_mult`` (the constant on every branch, 1 if
absent), ``logit_scale`` (1 if absent), ``loop`` {start, stop, times} (optional) and ``layers``, a list of {type, mixer, mlp}:

* type "attention": mixer {heads, kv_heads, dim, vdim, scale, mask {size, keep_first} (optional), rot {base, dims, scaling {factor, low,
  high, original} (optional)}} -- parts.attention.GatedAttention with weighted per-head norms of q and k, a rotation of neighbouring
  pairs with frequencies rescaled by wavelength, a sliding window that keeps the first tokens, and a sink;
* type "parallel": mixer {left_scale, right_scale, left {heads, kv_heads, dim, vdim, scale, mask {size}}, right {heads, kv_heads, dim, vdim,
  conv}} -- parts.parallel.ParallelMixers of windowed attention whose keys serve as values, with a slope by distance
  (GatedAttention), and a gated delta rule with one decay per head (parts.delta.HeadDelta);
* mlp {kind "dense", ff} -- a silu-gated feed-forward (parts.feedforward.ClampedGLU without clamps) -- or null.

The layers ``loop.start`` .. ``loop.stop`` - 1 run ``loop.times`` times in a row, every pass on caches and states of its own; in front
of every pass the row of 'loop.step' that belongs to it is added to the stream, and in front of every pass but the first the
embedding's output too (parts.block.StreamShift).

Tensors: 'embed', 'head', 'final.norm', 'loop.step', and per layer i 'l<i>.norm1', 'l<i>.norm1b', 'l<i>.norm2', 'l<i>.norm2b', 'l<i>.mix.*',
'l<i>.mlp.*'.  This class is the only place that knows these names; everything else works from the ``ModelSpec`` it returns."""
from __future__ import annotations

import copy
from dataclasses import dataclass

from .model_config import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

MAX_POSITION = 1 << 20       # the design has no position limit (angles come from the position itself); the engine wants a bound
SLOPE_SPAN = 8.0             # head h of H takes 2^(-SLOPE_SPAN (h + 1) / H) off a score for every position between query and key
UNIT_EPS = 1e-6              # under the root of the delta rule's unit vectors

_SIZES = {"attention": ("heads", "kv_heads", "dim", "vdim"), "left": ("heads", "kv_heads", "dim", "vdim"),
          "right": ("heads", "kv_heads", "dim", "vdim", "conv")}


def _need(d, keys, where: str):
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    missing = [k for k in keys if k not in d]
    if missing:
        raise ConfigError(f"config.json: {where} lacks key(s): {', '.join(missing)}")


def _check_sizes(m, kind: str, where: str):
    _need(m, _SIZES[kind] + (() if kind == "right" else ("scale",)), where)
    if any(int(m[k]) < 1 for k in _SIZES[kind]):
        raise ConfigError(f"config.json: {where}: sizes must be positive")
    if int(m["heads"]) % int(m["kv_heads"]):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    mask = m.get("mask")
    if mask is not None:
        _need(mask, ("size",), where + ".mask")
        if int(mask["size"]) < 1 or int(mask.get("keep_first") or 0) < 0:
            raise ConfigError(f"config.json: {where}.mask: size must be positive and keep_first not negative")


def _check_mixer(kind, m, where: str):
    if kind == "attention":
        _check_sizes(m, "attention", where)
        rot = m.get("rot")
        if rot is not None:
            _need(rot, ("base", "dims"), where + ".rot")
            if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= int(m["dim"]):
                raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
            if rot.get("scaling") is not None:
                _need(rot["scaling"], ("factor", "low", "high", "original"), where + ".rot.scaling")
    elif kind == "parallel":
        _need(m, ("left", "right", "left_scale", "right_scale"), where)
        _check_sizes(m["left"], "left", where + ".left")
        _check_sizes(m["right"], "right", where + ".right")
        if int(m["left"]["vdim"]) != int(m["left"]["dim"]):
            raise ConfigError(f"config.json: {where}.left.vdim must be its dim: the keys serve as values")
        if (m["left"].get("mask") or {}).get("keep_first"):
            raise ConfigError(f"config.json: {where}.left.mask keeps no first tokens in this design")
    else:
        raise ConfigError(f"config.json: {where}: type {kind!r} is not a mixer of this design (attention, parallel)")


@dataclass(frozen=True)
class KaropelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple            # the config's own dicts, checked
    loop: tuple | None       # (start, stop, times)
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    architecture: str = "Karopel"

    @classmethod
    def from_dict(cls, c: dict) -> "KaropelConfig":
        _need(c, ("vocab", "width", "norm", "layers"), "the model")
        _need(c["norm"], ("eps",), "norm")
        if not isinstance(c["layers"], list) or not c["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, layer in enumerate(c["layers"]):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            _check_mixer(layer["type"], layer["mixer"], where + ".mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                _need(mlp, ("kind",), where + ".mlp")
                if mlp["kind"] != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp['kind']!r} is not a feed-forward of this design (dense)")
                _need(mlp, ("ff",), where + ".mlp")
            layers.append(copy.deepcopy(layer))
        loop = None
        if c.get("loop") is not None:
            _need(c["loop"], ("start", "stop", "times"), "loop")
            loop = (int(c["loop"]["start"]), int(c["loop"]["stop"]), int(c["loop"]["times"]))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"config.json: loop {c['loop']} does not name a stretch of the {len(layers)} layers run at least once")
        number = lambda key: float(c[key]) if c.get(key) is not None else 1.0
        cfg = cls(vocab=int(c["vocab"]), width=int(c["width"]), norm_eps=float(c["norm"]["eps"]), layers=tuple(layers), loop=loop,
                  residual_mult=number("residual_mult"), logit_scale=number("logit_scale"), architecture=str(c.get("architecture", "Karopel")))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    # ------------------------------------------------------------------ description as data
    def _norm(self, prefix: str, gain: float = 1.0) -> PartSpec:
        return PartSpec("zero_centered_rmsnorm", dict(size=self.width, eps=self.norm_eps, gain=gain), prefix)

    def _attention(self, m: dict, **more) -> dict:
        mask = m.get("mask")
        return dict(hidden_size=self.width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                    scale=float(m["scale"]), eps=self.norm_eps, head_temp=False, gate=False, window=int(mask["size"]) if mask else None,
                    keep_first=int(mask.get("keep_first") or 0) if mask else 0, **more)

    def _mixer(self, layer: dict, prefix: str) -> PartSpec:
        m = layer["mixer"]
        if layer["type"] == "attention":
            rot = m.get("rot") or dict(base=1.0, dims=0)
            scaling = rot.get("scaling")
            return PartSpec("gated_attention", self._attention(
                m, rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_pairing="interleaved", qk_norm="head", sink=True,
                rot_scaling=dict(kind="wavelength", **{k: float(scaling[k]) for k in ("factor", "low", "high", "original")}) if scaling else None), prefix)
        left, right = m["left"], m["right"]
        heads = int(left["heads"])
        keys = PartSpec("gated_attention", self._attention(
            left, rot_dims=0, rot_base=1.0, qk_norm=False, keys_as_values=True,
            slopes=tuple(2.0 ** (-SLOPE_SPAN * (h + 1) / heads) for h in range(heads))))
        delta = PartSpec("head_delta", dict(hidden_size=self.width, num_heads=int(right["heads"]), num_kv_heads=int(right["kv_heads"]),
                                            dim=int(right["dim"]), vdim=int(right["vdim"]), taps=int(right["conv"]), eps=self.norm_eps, unit_eps=UNIT_EPS))
        return PartSpec("parallel", dict(hidden_size=self.width, branches={"left": keys, "right": delta},
                                         scales=(float(m["left_scale"]), float(m["right_scale"]))), prefix)

    def run_plan(self) -> list:
        """[(layer, pass or None)] in running order: a pass number stands with the first layer of a pass of the repeated stretch."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        lo, hi, times = self.loop
        plan = [(i, None) for i in range(lo)]
        for t in range(times):
            plan += [(i, t if i == lo else None) for i in range(lo, hi)]
        return plan + [(i, None) for i in range(hi, n)]

    def model_spec(self) -> ModelSpec:
        layers, aliases = [], {"embed.weight": "embed", "head.weight": "head", "final.norm.weight": "final.norm"}
        for i, layer in enumerate(self.layers):
            p, parts = f"l{i}.", {}

            def norms(role, name):
                parts[role + "_norm"], parts[role + "_out_norm"] = self._norm(p + name + "."), self._norm(p + name + "b.", self.residual_mult)
                for n in (name, name + "b"):
                    aliases[p + n + ".weight"] = p + n

            parts["mixer"] = self._mixer(layer, p + "mix.")
            norms("mixer", "norm1")
            if layer.get("mlp") is not None:
                # silu is the gated feed-forward's sigmoid with slope 1; nothing is clamped and nothing shifts the second factor
                parts["feed_forward"] = PartSpec("clamped_glu", dict(hidden_size=self.width, intermediate_size=int(layer["mlp"]["ff"]), limit=0.0,
                                                                     slope=1.0, shift=0.0), p + "mlp.")
                norms("feed_forward", "norm2")
            layers.append(LayerSpec("sandwich_residual", parts))
        # the steps in front of the passes are entries of the layer list too (they share 'loop.step'); every run of a layer has a
        # cache id of its own, so every pass keeps its own keys, values and states
        run, shifts = [], {}
        for cache_id, (i, t) in enumerate(self.run_plan()):          # (such a step keeps nothing: its cache id is a negative number)
            if t is not None:
                if t not in shifts:
                    shifts[t] = len(layers)
                    layers.append(LayerSpec("stream_shift_step", dict(shift=PartSpec("stream_shift", dict(
                        hidden_size=self.width, rows=self.loop[2], index=t, with_embedding=t > 0), "loop."))))
                run.append(RunEntry(shifts[t], -1 - t))
            run.append(RunEntry(i, cache_id))
        return ModelSpec(
            vocab_size=self.vocab, hidden_size=self.width,
            embedding=PartSpec("embedding", dict(vocab_size=self.vocab, hidden_size=self.width,
                                                 keep_output=self.loop is not None and self.loop[2] > 1), "embed."),
            layers=tuple(layers), run_order=tuple(run), final_norm=self._norm("final.norm.", self.logit_scale),
            head=PartSpec("linear_head", dict(vocab_size=self.vocab, hidden_size=self.width), "head."),
            max_position=MAX_POSITION, eos_token_id=-1, aliases=aliases)
