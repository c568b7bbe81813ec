"""Radenex: a decoder of parallel layers (one RMS norm, mixer and feed-forward side by side on its output, one sum) that are
listed one by one in config.json, each with a mixer of its own kind and sizes, and of which a stretch may run several times
in a row with the same weights.

config.json: ``architecture`` "Radenex", ``vocab``, ``width``, ``norm`` {eps}, ``loop`` {start, stop, times} (optional) and
``layers``, a list of {type, mixer, mlp}:

* type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims, scaling {factor, original, fast, slow}
  (optional)}} -- parts.attention.LatentAttention without a query latent, rotate-half pairs, "yarn" frequencies, a sink and a
  gate per head;
* type "attention": mixer {heads, kv_heads, dim, vdim, scale, mask {size, keep_first} (optional), rot {base, dims, scaling {factor}
  (optional)}} -- parts.attention.GatedAttention with heads of unit root mean square, rotated values, a sliding window that keeps
  the first tokens, and a constant 1 in the softmax's denominator;
* mlp {kind "dense", ff} -- parts.feedforward.ActivatedMLP with the square of relu -- or null.

The layers ``loop.start`` .. ``loop.stop`` - 1 run ``loop.times`` times in a row, every pass on caches of its own.

Tensors: 'embed', 'head', 'final.norm', and per layer i 'l<i>.norm1', 'l<i>.mix.*', 'l<i>.mlp.*'.  This class is the only place
that knows these names; everything else works from the ``ModelSpec`` it returns."""
from __future__ import annotations

import copy
from dataclasses import dataclass

from .model_config import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

MAX_POSITION = 1 << 20       # the design has no position limit (angles come from the position itself); the engine wants a bound

_MIXER_KEYS = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"),
               "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "rot")}
_SCALING_KEYS = {"latent_attention": ("factor", "original", "fast", "slow"), "attention": ("factor",)}


def _need(d, keys, where: str):
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    missing = [k for k in keys if k not in d]
    if missing:
        raise ConfigError(f"config.json: {where} lacks key(s): {', '.join(missing)}")


def _check_mixer(kind, m, where: str):
    if kind not in _MIXER_KEYS:
        raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design ({', '.join(_MIXER_KEYS)})")
    where += ".mixer"
    _need(m, _MIXER_KEYS[kind], where)
    if any(int(m[k]) < 1 for k in _MIXER_KEYS[kind] if k not in ("scale", "rot", "rot_dim")):
        raise ConfigError(f"config.json: {where}: sizes must be positive")
    rot = m["rot"]
    _need(rot, ("base", "dims"), where + ".rot")
    if rot.get("scaling") is not None:
        _need(rot["scaling"], _SCALING_KEYS[kind], where + ".rot.scaling")
    if kind == "latent_attention":
        if int(rot["dims"]) != int(m["rot_dim"]) or int(m["rot_dim"]) < 0 or int(m["rot_dim"]) % 2:
            raise ConfigError(f"config.json: {where}.rot.dims must be the (even) rot_dim: the rotated part turns as a whole")
        return
    if int(m["heads"]) % int(m["kv_heads"]):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= int(m["dim"]) or int(m["vdim"]) % 2:
        raise ConfigError(f"config.json: {where}: rot.dims must be even and at most dim, and vdim even (values rotate in pairs)")
    if m.get("mask") is not None:
        _need(m["mask"], ("size",), where + ".mask")
        if int(m["mask"]["size"]) < 1 or int(m["mask"].get("keep_first") or 0) < 0:
            raise ConfigError(f"config.json: {where}.mask: size must be positive and keep_first not negative")


@dataclass(frozen=True)
class RadenexConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple            # the config's own dicts, checked
    loop: tuple | None       # (start, stop, times)
    architecture: str = "Radenex"

    @classmethod
    def from_dict(cls, c: dict) -> "RadenexConfig":
        _need(c, ("vocab", "width", "norm", "layers"), "the model")
        _need(c["norm"], ("eps",), "norm")
        if not isinstance(c["layers"], list) or not c["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, layer in enumerate(c["layers"]):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            _check_mixer(layer["type"], layer["mixer"], where)
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
        cfg = cls(vocab=int(c["vocab"]), width=int(c["width"]), norm_eps=float(c["norm"]["eps"]), layers=tuple(layers), loop=loop,
                  architecture=str(c.get("architecture", "Radenex")))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    # ------------------------------------------------------------------ description as data
    def _norm(self, prefix: str) -> PartSpec:
        # an RMS norm that adds both sublayers' outputs of the layer before to the stream first
        return PartSpec("layernorm", dict(size=self.width, eps=self.norm_eps, center=False), prefix)

    def _mixer(self, layer: dict, prefix: str) -> PartSpec:
        m, rot = layer["mixer"], layer["mixer"]["rot"]
        scaling = rot.get("scaling")
        common = dict(hidden_size=self.width, num_heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                      rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_pairing="half", eps=self.norm_eps)
        if layer["type"] == "latent_attention":
            return PartSpec("latent_attention", dict(
                common, rot_dim=int(m["rot_dim"]), q_rank=None, kv_rank=int(m["kv_rank"]), gate="head", sink=True,
                rot_scaling=dict(kind="yarn", **{k: float(scaling[k]) for k in _SCALING_KEYS["latent_attention"]}) if scaling else None), prefix)
        mask = m.get("mask")
        return PartSpec("gated_attention", dict(
            common, num_kv_heads=int(m["kv_heads"]), qk_norm="unit", head_temp=False, gate=False, rotate_values=True, sink="one",
            rot_scaling=dict(kind="linear", factor=float(scaling["factor"])) if scaling else None,
            window=int(mask["size"]) if mask else None, keep_first=int(mask.get("keep_first") or 0) if mask else 0), prefix)

    def run_plan(self) -> list:
        """The layers in running order."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        lo, hi, times = self.loop
        return list(range(lo)) + list(range(lo, hi)) * times + list(range(hi, n))

    def model_spec(self) -> ModelSpec:
        layers, aliases = [], {"embed.weight": "embed", "head.weight": "head", "final.norm.weight": "final.norm"}
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            parts = dict(mixer=self._mixer(layer, p + "mix."), norm=self._norm(p + "norm1."))
            aliases[p + "norm1.weight"] = p + "norm1"
            if layer.get("mlp") is not None:
                parts["feed_forward"] = PartSpec("activated_mlp", dict(hidden_size=self.width, intermediate_size=int(layer["mlp"]["ff"]),
                                                                       activation="relu2"), p + "mlp.")
            layers.append(LayerSpec("parallel_residual", parts))
        # every run of a layer has a cache id of its own, so every pass keeps its own keys and values
        run = tuple(RunEntry(i, n) for n, i in enumerate(self.run_plan()))
        return ModelSpec(
            vocab_size=self.vocab, hidden_size=self.width,
            embedding=PartSpec("embedding", dict(vocab_size=self.vocab, hidden_size=self.width), "embed."),
            layers=tuple(layers), run_order=run, final_norm=self._norm("final.norm."),
            head=PartSpec("linear_head", dict(vocab_size=self.vocab, hidden_size=self.width), "head."),
            max_position=MAX_POSITION, eos_token_id=-1, aliases=aliases)
