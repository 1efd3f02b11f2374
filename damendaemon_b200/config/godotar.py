"""Typed Godotar configuration, parsed from the architecture's own config.json keys.

    architecture   "Godotar"
    vocab, width   sizes of the token table and the residual stream
    norm           {eps}: of every norm
    logit_scale    multiplies the logits
    loop           {start, stop, times} (optional): layers start .. stop - 1 run `times` times in a row
    layers         a list; each entry {type, mixer: {...}, mlp: {...} | null}
      wkv               {heads, dim}: time mixing with a matrix state per head; the rank of its decay's low-rank projection is
                        not in config.json: the tensors' shapes give it (``with_tensor_shapes``); a configuration that is to
                        be filled with random weights may name it (decay_rank)
      latent_attention  {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot: {dims, base}, mask: {size} (optional)}
      mlp               {kind: "dense", ff} | {kind: "moe", router: {experts, top, identity (optional)}, expert: {ff, limit}}

The configuration names no context length: the engine's cache sets it.
"""
from __future__ import annotations

import dataclasses
import math
from dataclasses import dataclass
from typing import Optional, Tuple

from .reader import ConfigError

ARCHITECTURE = "Godotar"


def _get(config, name, where):
    if not isinstance(config, dict) or name not in config:
        raise ConfigError(f"{where}: '{name}' is missing")
    return config[name]


def _int(config, name, where, least=1):
    value = _get(config, name, where)
    if type(value) is not int or value < least:
        raise ConfigError(f"{where}.{name} must be an integer of at least {least}, got {value!r}")
    return value


def _number(config, name, where, positive=True):
    value = _get(config, name, where)
    if type(value) not in (int, float) or not math.isfinite(value) or (positive and value <= 0):
        raise ConfigError(f"{where}.{name} must be a finite{' positive' if positive else ''} number, got {value!r}")
    return float(value)


@dataclass(frozen=True)
class TimeMixer:
    heads: int
    dim: int
    decay_rank: Optional[int] = None


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_dims: int
    rot_base: float
    mask_size: Optional[int] = None


@dataclass(frozen=True)
class Mlp:
    kind: str            # 'dense' | 'moe'
    ff: int
    experts: int = 0
    top: int = 0
    identity: int = 0
    limit: float = 0.0


@dataclass(frozen=True)
class Layer:
    type: str            # 'wkv' | 'latent_attention'
    mixer: object
    mlp: Optional[Mlp]


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


def _time_mixer(raw, where):
    return TimeMixer(_int(raw, "heads", where), _int(raw, "dim", where),
                     None if raw.get("decay_rank") is None else _int(raw, "decay_rank", where))


def _latent(raw, where):
    sizes = {n: _int(raw, n, where) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")}
    rot = _get(raw, "rot", where)
    dims, base = _int(rot, "dims", where + ".rot"), _number(rot, "base", where + ".rot")
    if dims % 2 or dims > sizes["rot_dim"]:
        raise ConfigError(f"{where}.rot.dims must be even and at most the rotated part's size {sizes['rot_dim']}, got {dims}")
    mask = raw.get("mask")
    return LatentMixer(scale=_number(raw, "scale", where, positive=False), rot_dims=dims, rot_base=base,
                       mask_size=None if mask is None else _int(mask, "size", where + ".mask"), **sizes)


def _mlp(raw, where):
    if raw is None:
        return None
    kind = _get(raw, "kind", where)
    if kind == "dense":
        return Mlp("dense", ff=_int(raw, "ff", where))
    if kind == "moe":
        router, expert = _get(raw, "router", where), _get(raw, "expert", where)
        experts, top = _int(router, "experts", where + ".router"), _int(router, "top", where + ".router")
        identity = 0 if router.get("identity") is None else _int(router, "identity", where + ".router", 0)
        if top > experts + identity:
            raise ConfigError(f"{where}.router: {top} experts per token of {experts} + {identity}")
        return Mlp("moe", ff=_int(expert, "ff", where + ".expert"), experts=experts, top=top, identity=identity,
                   limit=_number(expert, "limit", where + ".expert"))
    raise ConfigError(f"{where}.kind must be 'dense' or 'moe', got {kind!r}")


_MIXERS = {"wkv": _time_mixer, "latent_attention": _latent}


@dataclass(frozen=True)
class GodotarConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[Layer, ...]
    loop: Optional[Loop] = None
    eos_token_ids: tuple = ()

    architecture = ARCHITECTURE

    @property
    def vocab_size(self):
        return self.vocab

    @classmethod
    def from_dict(cls, config: dict) -> "GodotarConfig":
        if config.get("architecture") != ARCHITECTURE:
            raise ConfigError(f"architecture must be {ARCHITECTURE!r}, got {config.get('architecture')!r}")
        raw_layers = _get(config, "layers", "config")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, raw in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = _get(raw, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}.type must be one of {sorted(_MIXERS)}, got {kind!r}")
            layers.append(Layer(kind, _MIXERS[kind](_get(raw, "mixer", where), where + ".mixer"), _mlp(raw.get("mlp"), where + ".mlp")))
        loop = config.get("loop")
        if loop is not None:
            loop = Loop(_int(loop, "start", "loop", 0), _int(loop, "stop", "loop", 0), _int(loop, "times", "loop"))
            if not loop.start <= loop.stop <= len(layers):
                raise ConfigError(f"loop: layers {loop.start} to {loop.stop} are not a run of the model's {len(layers)} layers")
        return cls(vocab=_int(config, "vocab", "config"), width=_int(config, "width", "config"),
                   norm_eps=_number(_get(config, "norm", "config"), "eps", "norm"),
                   logit_scale=_number(config, "logit_scale", "config", positive=False), layers=tuple(layers), loop=loop)

    def with_tensor_shapes(self, shapes: dict) -> "GodotarConfig":
        """The sizes that config.json does not name, from the checkpoint's tensor shapes ({name: shape}): the rank of a time
        mixer's decay projection, the rows of 'l<i>.mix.w1'."""
        layers = []
        for i, layer in enumerate(self.layers):
            if layer.type == "wkv":
                name, named = f"l{i}.mix.w1", layer.mixer.decay_rank
                shape = shapes.get(name)
                if shape is not None and len(shape) == 2:
                    if named is not None and named != shape[0]:
                        raise ConfigError(f"layers[{i}].mixer.decay_rank is {named}, but {name} has {shape[0]} rows")
                    layer = dataclasses.replace(layer, mixer=dataclasses.replace(layer.mixer, decay_rank=int(shape[0])))
                elif named is None:
                    raise ConfigError(f"layers[{i}]: neither config.json nor a tensor {name} gives the mixer's decay_rank")
            layers.append(layer)
        return dataclasses.replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        """The config.json this configuration round-trips through."""
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            if layer.type == "wkv":
                mixer = {"heads": m.heads, "dim": m.dim}
                if m.decay_rank is not None:
                    mixer["decay_rank"] = m.decay_rank
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank,
                         "scale": m.scale, "rot": {"dims": m.rot_dims, "base": m.rot_base}}
                if m.mask_size is not None:
                    mixer["mask"] = {"size": m.mask_size}
            if f is None:
                mlp = None
            elif f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            else:
                mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top, "identity": f.identity},
                       "expert": {"ff": f.ff, "limit": f.limit}}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "logit_scale": self.logit_scale, "layers": layers}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out
