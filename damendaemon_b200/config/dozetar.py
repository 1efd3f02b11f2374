"""Typed Dozetar configuration, parsed from the architecture's own config.json keys.

    architecture   "Dozetar"
    vocab, width   sizes of the token table and the residual stream
    norm           {eps}: of every norm
    residual_mult  c: every sublayer's normed result is added c times
    logit_softcap  s (optional): logits become s * tanh(logits / s)
    layers         a list; each entry {type, mixer: {...}, mlp: {kind: "moe", router: {experts, top}, expert: {ff}} | null}
      mlstm        {heads, dim, vdim, gate_cap}: a matrix memory with exponential gates
      parallel     {left: {heads, kv_heads, dim, vdim, scale, rot: {dims, base}, mask (optional): {size, keep_first (optional)}},
                    right: {heads, dim, vdim, decay: one per head}, left_scale, right_scale}: softmax attention beside linear
                   attention with fixed decays

The configuration names no context length: the engine's cache sets it.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple

from .reader import ConfigError

ARCHITECTURE = "Dozetar"


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
class Rotation:
    dims: int
    base: float


@dataclass(frozen=True)
class Mask:
    size: int
    keep_first: int = 0


@dataclass(frozen=True)
class SoftmaxMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation
    mask: Optional[Mask] = None


@dataclass(frozen=True)
class DecayMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class ParallelMixer:
    left: SoftmaxMixer
    right: DecayMixer
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class MemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class Experts:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class Layer:
    type: str            # 'mlstm' | 'parallel'
    mixer: object
    mlp: Optional[Experts]


def _softmax(raw, where):
    sizes = {n: _int(raw, n, where) for n in ("heads", "kv_heads", "dim", "vdim")}
    if sizes["heads"] % sizes["kv_heads"]:
        raise ConfigError(f"{where}: {sizes['heads']} heads cannot share {sizes['kv_heads']} key heads")
    rot = _get(raw, "rot", where)
    rot = Rotation(_int(rot, "dims", where + ".rot"), _number(rot, "base", where + ".rot"))
    if rot.dims % 2 or rot.dims > sizes["dim"]:
        raise ConfigError(f"{where}.rot.dims must be even and at most the head size {sizes['dim']}, got {rot.dims}")
    mask = raw.get("mask")
    if mask is not None:
        mask = Mask(_int(mask, "size", where + ".mask"), _int(mask, "keep_first", where + ".mask", 0) if "keep_first" in mask else 0)
    return SoftmaxMixer(scale=_number(raw, "scale", where), rot=rot, mask=mask, **sizes)


def _decayed(raw, where):
    sizes = {n: _int(raw, n, where) for n in ("heads", "dim", "vdim")}
    decay = _get(raw, "decay", where)
    if not isinstance(decay, list) or len(decay) != sizes["heads"] or \
            any(type(d) not in (int, float) or not 0.0 <= d <= 1.0 for d in decay):
        raise ConfigError(f"{where}.decay must list a number from 0 to 1 for each of the {sizes['heads']} heads, got {decay!r}")
    return DecayMixer(decay=tuple(float(d) for d in decay), **sizes)


def _parallel(raw, where):
    return ParallelMixer(_softmax(_get(raw, "left", where), where + ".left"), _decayed(_get(raw, "right", where), where + ".right"),
                         _number(raw, "left_scale", where, positive=False), _number(raw, "right_scale", where, positive=False))


def _memory(raw, where):
    return MemoryMixer(gate_cap=_number(raw, "gate_cap", where), **{n: _int(raw, n, where) for n in ("heads", "dim", "vdim")})


def _mlp(raw, where):
    if raw is None:
        return None
    kind = _get(raw, "kind", where)
    if kind != "moe":
        raise ConfigError(f"{where}.kind must be 'moe', got {kind!r}")
    router = _get(raw, "router", where)
    m = Experts(_int(router, "experts", where + ".router"), _int(router, "top", where + ".router"),
                _int(_get(raw, "expert", where), "ff", where + ".expert"))
    if m.top > m.experts:
        raise ConfigError(f"{where}.router: {m.top} experts a token of {m.experts}")
    return m


_MIXERS = {"mlstm": _memory, "parallel": _parallel}


@dataclass(frozen=True)
class DozetarConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[Layer, ...]
    logit_softcap: Optional[float] = None
    eos_token_ids: tuple = ()

    architecture = ARCHITECTURE

    @property
    def vocab_size(self):
        return self.vocab

    @classmethod
    def from_dict(cls, config: dict) -> "DozetarConfig":
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
        cap = config.get("logit_softcap")
        if cap is not None:
            cap = _number(config, "logit_softcap", "config")
        return cls(vocab=_int(config, "vocab", "config"), width=_int(config, "width", "config"),
                   norm_eps=_number(_get(config, "norm", "config"), "eps", "norm"),
                   residual_mult=_number(config, "residual_mult", "config", positive=False), layers=tuple(layers), logit_softcap=cap)

    def to_dict(self) -> dict:
        """The config.json this configuration round-trips through."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if layer.type == "mlstm":
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
            else:
                l, r = m.left, m.right
                left = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale,
                        "rot": {"dims": l.rot.dims, "base": l.rot.base}}
                if l.mask is not None:
                    left["mask"] = {"size": l.mask.size, "keep_first": l.mask.keep_first}
                mixer = {"left": left, "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)},
                         "left_scale": m.left_scale, "right_scale": m.right_scale}
            f = layer.mlp
            mlp = None if f is None else {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "residual_mult": self.residual_mult, "layers": layers}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out
