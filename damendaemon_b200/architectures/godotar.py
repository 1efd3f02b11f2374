"""Godotar described with the framework's parts.

A decoder over a float32 stream that starts as the token's normed row. A run of layers may be repeated: every pass has caches
and states of its own (a stop of the run order each) and starts by adding its row of a table of vectors to the stream. A layer
is x <- x + mixer(norm1(x)) + ff(norm2(x)), both of the same x, with RMS norms whose weights are stored around zero. A mixer
is one of
  wkv               time mixing: a matrix state per head with a decay per key channel that depends on the token, a bonus for
                    the current token, every branch fed by its own blend with the token before;
  latent_attention  attention whose keys and values are projections of one cached latent row per token, with a rotated key
                    part that all heads share, queries through a latent of their own, a sliding window and a gate per head.
The feed-forward is a silu gated unit, or experts chosen by the softmax of a router (a correction per output moves the choice
only, the weights are renormalised, the last outputs are the input itself), or absent. The final norm, the token table as the
head and a factor give the logits.

Tensor names: embed, embed.norm, loop.step, l<i>.{norm1, norm2}, l<i>.mix.* (wkv: mu.{r, k, v, g, w}, r, k, v, g, w1, w2, w0,
u, norm, o; latent_attention: dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o), l<i>.mlp.{gate, up, down} or
l<i>.mlp.{router, correction, e<j>.{gate, up, down}}, final.norm; matrices [out, in].
"""
from __future__ import annotations

import math

import torch

from ..config.godotar import ARCHITECTURE, GodotarConfig
from ..parts.spec import (EmbeddingSpec, GatedFeedForwardSpec, GatedUnitSpec, HeadSpec, LatentAttentionSpec, LayerSpec, ModelSpec,
                          NoFeedForwardSpec, NormSpec, PositionSpec, RotarySpec, RunEntry, ScoreRoutedExpertsSpec, TimeMixSpec)
from ..registry import Architecture, register_architecture

SWISH_ALPHA = 1.702       # the design fixes the sigmoid's slope in an expert's unit


def _norm(c, name):
    return NormSpec("rmsnorm", c.width, c.norm_eps, name, weight_offset=1.0)


def _mixer_spec(c: GodotarConfig, i: int):
    layer, p = c.layers[i], f"l{i}.mix."
    m = layer.mixer
    if layer.type == "wkv":
        if m.decay_rank is None:
            raise ValueError(f"layer {i}: the rank of the time mixer's decay projection is not known; read it from the tensors' "
                             "shapes (GodotarConfig.with_tensor_shapes) or name it")
        return TimeMixSpec("time_mix", width=c.width, n_heads=m.heads, head_dim=m.dim, decay_rank=m.decay_rank, norm_eps=c.norm_eps,
                           mix_weights=tuple(p + "mu." + s for s in "rkvgw"), receptance_weight=p + "r", key_weight=p + "k",
                           value_weight=p + "v", gate_weight=p + "g", decay_down=p + "w1", decay_up=p + "w2", decay_bias=p + "w0",
                           bonus=p + "u", out_norm=p + "norm", out_weight=p + "o")
    return LatentAttentionSpec("latent_attention", width=c.width, n_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim,
                               value_dim=m.vdim, rank=m.kv_rank, scale=m.scale, norm_eps=c.norm_eps,
                               rotary=RotarySpec("rotary", head_dim=m.rot_dim, dims=m.rot_dims, base=m.rot_base, interleaved=False),
                               query_weight=p + "uq", down_weight=p + "dkv", latent_norm=p + "dkv.norm", up_key_weight=p + "uk",
                               up_value_weight=p + "uv", out_weight=p + "o", window=m.mask_size, gate_weight=p + "g",
                               query_down=p + "dq", query_norm=p + "dq.norm", query_rank=m.q_rank)


def _layer_spec(c: GodotarConfig, i: int):
    f, p = c.layers[i].mlp, f"l{i}."
    norms = (_norm(c, p + "norm1"), _norm(c, p + "norm2"))
    if f is None:
        return LayerSpec("pre_norm_mixer", _mixer_spec(c, i), NoFeedForwardSpec(), norms[:1])
    if f.kind == "dense":
        unit = GatedUnitSpec(f.ff, 0.0, p + "mlp.gate", p + "mlp.up", p + "mlp.down", activation="silu")
        return LayerSpec("parallel", _mixer_spec(c, i), GatedFeedForwardSpec("gated", c.width, unit), norms)
    experts = tuple(GatedUnitSpec(f.ff, f.limit, f"{p}mlp.e{j}.gate", f"{p}mlp.e{j}.up", f"{p}mlp.e{j}.down", alpha=SWISH_ALPHA,
                                  activation="clamped_swish") for j in range(f.experts))
    return LayerSpec("parallel", _mixer_spec(c, i),
                     ScoreRoutedExpertsSpec("experts_by_score", c.width, f.top, p + "mlp.router", experts, score="softmax",
                                            correction=p + "mlp.correction", renormalize=True, identity=f.identity), norms)


def run_order(c: GodotarConfig):
    """The stops: layers before the loop once, the loop's layers ``times`` times (a pass's first stop adds its row of the
    pass vectors), then the rest."""
    n = len(c.layers)
    if c.loop is None:
        return tuple(RunEntry(i) for i in range(n))
    a, b = c.loop.start, c.loop.stop
    stops = [RunEntry(i) for i in range(a)]
    for t in range(c.loop.times):
        stops += [RunEntry(i, add_vector=t if i == a else None) for i in range(a, b)]
    return tuple(stops + [RunEntry(i) for i in range(b, n)])


def build_spec(c: GodotarConfig) -> ModelSpec:
    looped = c.loop is not None and c.loop.stop > c.loop.start
    # a layer without a feed-forward has no use for its second norm, should the checkpoint hold one
    ignored = tuple(rf"l{i}\.norm2" for i, l in enumerate(c.layers) if l.mlp is None)
    return ModelSpec(
        architecture=ARCHITECTURE, vocab_size=c.vocab, width=c.width, max_positions=None,
        embedding=EmbeddingSpec("tokens", c.vocab, c.width, table="embed", norm=_norm(c, "embed.norm")),
        position=PositionSpec("none", 0, c.width), layers=tuple(_layer_spec(c, i) for i in range(len(c.layers))),
        run_order=run_order(c),
        head=HeadSpec("linear", c.vocab, c.width, norm=_norm(c, "final.norm"), weight="embed", tied=True, scale=c.logit_scale),
        pass_vectors=("loop.step", c.loop.times) if looped else None,
        ignored_tensors=ignored + (() if looped or c.loop is None else (r"loop\.step",)), eos_token_ids=tuple(c.eos_token_ids))


def with_tensor_shapes(c: GodotarConfig, shapes: dict) -> GodotarConfig:
    return c.with_tensor_shapes(shapes)


def random_tensors(c: GodotarConfig, seed: int, matrix_dtype=torch.float32, device="cpu") -> dict:
    """Seeded random weights under their checkpoint names, in a fixed draw order: the token table ~N(0, 1), matrices
    ~N(0, 1/in), norm weights ~N(0, 0.1) around zero or one as they are stored, blend weights uniform in [0, 1], decay biases
    spread so that fast and slow channels both occur, corrections ~N(0, 0.02). A time mixer whose decay rank the configuration
    does not name gets half its key size (at least 8)."""
    g = torch.Generator(device=device)
    g.manual_seed(int(seed))
    out = {}
    normal = lambda *shape: torch.randn(shape, generator=g, dtype=torch.float32, device=device)

    def matrix(name, rows, cols, gain=1.0):
        out[name] = (normal(rows, cols) * gain / math.sqrt(cols)).to(matrix_dtype)

    def around(name, n, centre=1.0, spread=0.1):
        out[name] = centre + normal(n) * spread

    out["embed"] = normal(c.vocab, c.width).to(matrix_dtype)
    around("embed.norm", c.width, centre=0.0)
    if c.loop is not None:
        out["loop.step"] = normal(c.loop.times, c.width) * 0.3
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        around(p + "norm1", c.width, centre=0.0)
        if layer.type == "wkv":
            inner, rank = m.heads * m.dim, m.decay_rank or max(8, m.dim // 2)
            for s in "rkvgw":
                out[p + "mix.mu." + s] = torch.rand((c.width,), generator=g, dtype=torch.float32, device=device)
            for s in "rkvg":
                matrix(p + "mix." + s, inner, c.width)
            matrix(p + "mix.w1", rank, c.width)
            matrix(p + "mix.w2", inner, rank)
            around(p + "mix.w0", inner, centre=-2.0, spread=1.5)
            out[p + "mix.u"] = normal(m.heads, m.dim) * 0.5
            around(p + "mix.norm", inner)
            matrix(p + "mix.o", c.width, inner)
        else:
            matrix(p + "mix.dq", m.q_rank, c.width)
            around(p + "mix.dq.norm", m.q_rank)
            matrix(p + "mix.uq", m.heads * (m.dim + m.rot_dim), m.q_rank)
            matrix(p + "mix.dkv", m.kv_rank + m.rot_dim, c.width)
            around(p + "mix.dkv.norm", m.kv_rank)
            matrix(p + "mix.uk", m.heads * m.dim, m.kv_rank)
            matrix(p + "mix.uv", m.heads * m.vdim, m.kv_rank)
            matrix(p + "mix.g", m.heads, c.width)
            matrix(p + "mix.o", c.width, m.heads * m.vdim)
        if f is None:
            continue
        around(p + "norm2", c.width, centre=0.0)
        units = [""] if f.kind == "dense" else [f"e{j}." for j in range(f.experts)]
        for u in units:
            matrix(p + "mlp." + u + "gate", f.ff, c.width)
            matrix(p + "mlp." + u + "up", f.ff, c.width)
            matrix(p + "mlp." + u + "down", c.width, f.ff)
        if f.kind == "moe":
            matrix(p + "mlp.router", f.experts + f.identity, c.width)
            around(p + "mlp.correction", f.experts + f.identity, centre=0.0, spread=0.02)
    around("final.norm", c.width, centre=0.0)
    return out


register_architecture(Architecture(ARCHITECTURE, GodotarConfig.from_dict, build_spec, random_tensors,
                                   sizes_from_shapes=with_tensor_shapes), replace=True)
