"""Dozetar described with the framework's parts.

A decoder over a float32 stream that starts as the token's row. A layer is post-norm: a sublayer reads the stream itself, its
result is divided by its root mean square, weighted and added with a fixed factor. A mixer is one of
  mlstm       a matrix memory per head with exponential gates (a running maximum keeps them in range), its read-out over a
              normalizer, normed per head, weighted and gated;
  parallel    two mixers of the same input, added with a fixed factor each: grouped softmax attention (biases, queries and
              keys normed over the whole projection, part of a head rotated with neighbours paired, a window behind which
              the first keys stay visible, a learned sink) and linear attention with a fixed decay per head whose queries,
              keys and values pass silu, normed over all heads together, weighted and gated.
The feed-forward is a choice of squared-relu experts by sigmoid scores, which multiply the experts' inputs, or absent. The
final norm, a head matrix of its own and a tanh cap give the logits.

Tensor names: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.* (mlstm: q, k, v, g, o, norm, i, i.b, f, f.b; parallel: left.{q, k, v}
each with .b, left.{q.norm, k.norm, sink, o, o.b}, right.{q, k, v, g, o, norm}), l<i>.mlp.{router, e<j>.up, e<j>.down},
final.norm, head; matrices [out, in].
"""
from __future__ import annotations

import math

import torch

from ..config.dozetar import ARCHITECTURE, DozetarConfig
from ..parts.spec import (AttentionSpec, EmbeddingSpec, HeadSpec, LayerSpec, MatrixMemorySpec, ModelSpec, NoFeedForwardSpec, NormSpec,
                          PlainUnitSpec, PositionSpec, RotarySpec, RunEntry, ScoreRoutedExpertsSpec, SideBySideSpec)
from ..registry import Architecture, register_architecture

DENOMINATOR_EPS = 1e-6      # the design fixes what is added to the memory's denominator


def _norm(c, name):
    return NormSpec("rmsnorm", c.width, c.norm_eps, name)


def _memory(c, m, p, **more):
    return MatrixMemorySpec("matrix_memory", width=c.width, n_heads=m.heads, head_dim=m.dim, value_dim=m.vdim, norm_eps=c.norm_eps,
                            query_weight=p + "q", key_weight=p + "k", value_weight=p + "v", gate_weight=p + "g", out_norm=p + "norm",
                            out_weight=p + "o", **more)


def _mixer_spec(c: DozetarConfig, i: int):
    layer, p = c.layers[i], f"l{i}.mix."
    m = layer.mixer
    if layer.type == "mlstm":
        return _memory(c, m, p, query_scale=m.dim ** -0.5, input_gate=p + "i", input_gate_bias=p + "i.b", forget_gate=p + "f",
                       forget_gate_bias=p + "f.b", gate_cap=m.gate_cap, denominator_eps=DENOMINATOR_EPS)
    l = m.left
    left = AttentionSpec("attention", width=c.width, n_heads=l.heads, n_kv_heads=l.kv_heads, head_dim=l.dim, scale=l.scale,
                         window=None if l.mask is None else l.mask.size, keep_first=0 if l.mask is None else l.mask.keep_first,
                         qkv_weight=tuple(p + "left." + n for n in "qkv"), qkv_bias=tuple(p + f"left.{n}.b" for n in "qkv"),
                         out_weight=p + "left.o", out_bias=p + "left.o.b", value_dim=l.vdim,
                         rotary=RotarySpec("rotary", head_dim=l.dim, dims=l.rot.dims, base=l.rot.base, interleaved=True),
                         query_norm=p + "left.q.norm", key_norm=p + "left.k.norm", head_norm_eps=c.norm_eps,
                         norm_whole_projection=True, sink=p + "left.sink", exact_weights=True)
    right = _memory(c, m.right, p + "right.", activation="silu", norm_together=True, decay=m.right.decay)
    return SideBySideSpec("side_by_side", width=c.width, left=left, right=right, left_scale=m.left_scale, right_scale=m.right_scale)


def _layer_spec(c: DozetarConfig, i: int):
    f, p = c.layers[i].mlp, f"l{i}."
    if f is None:
        return LayerSpec("post_norm", _mixer_spec(c, i), NoFeedForwardSpec(), (_norm(c, p + "norm1"),), residual_factor=c.residual_mult)
    units = tuple(PlainUnitSpec(f.ff, p + f"mlp.e{j}.up", p + f"mlp.e{j}.down", "relu2") for j in range(f.experts))
    feed = ScoreRoutedExpertsSpec("experts_by_score", width=c.width, top=f.top, router=p + "mlp.router", experts=units, weight_input=True)
    return LayerSpec("post_norm", _mixer_spec(c, i), feed, (_norm(c, p + "norm1"), _norm(c, p + "norm2")), residual_factor=c.residual_mult)


def build_spec(c: DozetarConfig) -> ModelSpec:
    n = len(c.layers)
    return ModelSpec(
        architecture=ARCHITECTURE, vocab_size=c.vocab, width=c.width, max_positions=None,
        embedding=EmbeddingSpec("tokens", c.vocab, c.width, table="embed"), position=PositionSpec("none", 0, c.width),
        layers=tuple(_layer_spec(c, i) for i in range(n)), run_order=tuple(RunEntry(i) for i in range(n)),
        head=HeadSpec("linear", c.vocab, c.width, norm=_norm(c, "final.norm"), weight="head", softcap=c.logit_softcap),
        eos_token_ids=tuple(c.eos_token_ids))


def random_tensors(c: DozetarConfig, seed: int, matrix_dtype=torch.float32, device="cpu") -> dict:
    """Seeded random weights under their checkpoint names, in a fixed draw order: tables ~N(0, 1), matrices ~N(0, 1/in), norm
    weights ~N(1, 0.1), biases ~N(0, 0.1), the gates' biases such that memories last for some tens of tokens, sinks ~N(0, 1)."""
    g = torch.Generator(device=device)
    g.manual_seed(int(seed))
    out = {}
    normal = lambda *shape: torch.randn(shape, generator=g, dtype=torch.float32, device=device)

    def matrix(name, rows, cols, gain=1.0):
        out[name] = (normal(rows, cols) * gain / math.sqrt(cols)).to(matrix_dtype)

    def around(name, n, centre=1.0, spread=0.1):
        out[name] = centre + normal(n) * spread

    def memory(p, m):
        for name, n in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
            matrix(p + name, n, c.width)
        matrix(p + "o", c.width, m.heads * m.vdim)
        around(p + "norm", m.heads * m.vdim)

    out["embed"] = normal(c.vocab, c.width).to(matrix_dtype)
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        around(p + "norm1", c.width)
        if layer.type == "mlstm":
            memory(p + "mix.", m)
            matrix(p + "mix.i", m.heads, c.width)
            around(p + "mix.i.b", m.heads, centre=-1.0, spread=1.0)
            matrix(p + "mix.f", m.heads, c.width)
            around(p + "mix.f.b", m.heads, centre=3.0, spread=1.0)
        else:
            l, q = m.left, p + "mix.left."
            for name, n in (("q", l.heads * l.dim), ("k", l.kv_heads * l.dim), ("v", l.kv_heads * l.vdim)):
                matrix(q + name, n, c.width)
                around(q + name + ".b", n, centre=0.0)
            around(q + "q.norm", l.heads * l.dim)
            around(q + "k.norm", l.kv_heads * l.dim)
            out[q + "sink"] = normal(l.heads)
            matrix(q + "o", c.width, l.heads * l.vdim)
            around(q + "o.b", c.width, centre=0.0)
            memory(p + "mix.right.", m.right)
        if layer.mlp is not None:
            f = layer.mlp
            around(p + "norm2", c.width)
            matrix(p + "mlp.router", f.experts, c.width)
            for j in range(f.experts):
                matrix(p + f"mlp.e{j}.up", f.ff, c.width)
                matrix(p + f"mlp.e{j}.down", c.width, f.ff)
    around("final.norm", c.width)
    matrix("head", c.vocab, c.width)
    return out


register_architecture(Architecture(ARCHITECTURE, DozetarConfig.from_dict, build_spec, random_tensors), replace=True)
