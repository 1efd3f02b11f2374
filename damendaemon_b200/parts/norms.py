"""Norms. LayerNorm with weight and optional bias (damendaemon/starcoder.py:53-55); RMS norm,
x / sqrt(mean(x^2) + eps) * (offset + weight), with the offset a parameter of the spec, and optionally in groups:
the row in equal consecutive stretches, each divided by its own root mean square; a norm without statistics,
tanh(alpha x) * weight + bias with one learned number alpha."""
from __future__ import annotations

from .. import kernels
from .interfaces import Norm
from .registry import register_norm
from .spec import TensorDecl


@register_norm("layernorm")
class LayerNorm(Norm):
    def __init__(self, spec, weights, runtime):
        self.spec, self.runtime = spec, runtime
        self.gamma = weights[spec.weight]
        self.beta = weights[spec.bias] if spec.bias else None

    @staticmethod
    def tensor_decls(spec):
        decls = [TensorDecl(spec.weight, (spec.width,), "vector")]
        if spec.bias:
            decls.append(TensorDecl(spec.bias, (spec.width,), "vector"))
        return decls

    def forward(self, x, row_index=None, out_dtype=None):
        return kernels.layernorm(x, self.gamma, self.beta, self.spec.eps, out_dtype or self.runtime.dtype, row_index)

    def scale_output(self, factor):
        self.gamma = self.gamma * factor
        self.beta = None if self.beta is None else self.beta * factor


@register_norm("rmsnorm")
class RmsNorm(Norm):
    def __init__(self, spec, weights, runtime):
        if spec.bias:
            raise ValueError("an RMS norm has no bias")
        if spec.groups < 1 or spec.width % spec.groups:
            raise ValueError(f"a row of {spec.width} does not fall into {spec.groups} equal stretches")
        self.spec, self.runtime = spec, runtime
        self.weight, self.offset = weights[spec.weight], spec.weight_offset

    @staticmethod
    def tensor_decls(spec):
        return [TensorDecl(spec.weight, (spec.width,), "vector")]

    def forward(self, x, row_index=None, out_dtype=None):
        return kernels.rmsnorm(x, self.weight, self.spec.eps, out_dtype or self.runtime.dtype, row_index,
                               offset=self.offset, groups=self.spec.groups)

    def scale_output(self, factor):
        """Multiply everything the norm returns (folded into the weight, which then is the factor itself)."""
        self.weight, self.offset = (self.offset + self.weight) * factor, 0.0

    def add_normed(self, x, terms, factor=1.0, rounded=True):
        """x += factor * norm(y) in place, y given as a sublayer's ``forward_terms``; returns x in the engine dtype (x itself
        in a float32 engine), or None where that is not asked for. One pass over the stream."""
        if self.spec.groups != 1:
            raise ValueError("a result that is normed and added is normed whole, not in groups")
        if self.offset:
            self.weight, self.offset = self.offset + self.weight, 0.0
        low = rounded and self.runtime.dtype != x.dtype
        out = kernels.post_norm(x, weight=self.weight, eps=self.spec.eps, factor=factor,
                                rounded_dtype=self.runtime.dtype if low else None, **terms)
        return out if low or not rounded else x

    def forward_pair(self, other, x):
        """This norm's and another RMS norm's rows of the same x, in one pass over it."""
        y, z, _ = kernels.token_mix(x, self.weight, self.spec.eps, self.runtime.dtype, offset=self.offset, weight2=other.weight)
        return y, z

    def forward_mixes(self, x, mu, state, ctx, other=None, rows_per_mix=None):
        """Blends of every normed row with the normed row before it (kernels.token_mix), and, of the same x, the rows of
        ``other`` (an RMS norm with the same eps and offset, or None), in one pass: (mixes, the other norm's rows)."""
        if self.spec.groups != 1:
            raise ValueError("blends with the row before are made of rows normed whole, not in groups")
        _, z, mixes = kernels.token_mix(x, self.weight, self.spec.eps, self.runtime.dtype, offset=self.offset, keep=False,
                                        weight2=None if other is None else other.weight, mu=mu, state=state,
                                        token_entry=ctx.token_entry, entry_start=ctx.entry_start, entry_slot=ctx.entry_slot,
                                        rows_per_mix=rows_per_mix)
        return mixes, z

    def pairs_with(self, other):
        """Whether one pass can compute both norms of the same row: RMS norms of one width, eps and offset, in one group."""
        return isinstance(other, RmsNorm) and self.spec.groups == other.spec.groups == 1 and self.spec.width == other.spec.width and \
            self.spec.eps == other.spec.eps and self.offset == other.offset

    def forward_shifted(self, x, shift, state, ctx):
        """The norm of every row blended with the norm of the token before it (kernels.rmsnorm_shift), one kernel."""
        return kernels.rmsnorm_shift(x, self.weight, self.spec.eps, self.runtime.dtype, shift, state, ctx.token_entry,
                                     ctx.entry_start, ctx.entry_slot, offset=self.offset, groups=self.spec.groups)


@register_norm("tanh")
class TanhNorm(Norm):
    """tanh(alpha * x) * weight + bias: no mean, no variance, so a row needs no reduction."""

    def __init__(self, spec, weights, runtime):
        if not spec.bias or not spec.alpha:
            raise ValueError("a tanh norm has a weight, a bias and the number alpha")
        self.spec, self.runtime = spec, runtime
        self.weight, self.bias = weights[spec.weight], weights[spec.bias]
        self.alpha = weights[spec.alpha].reshape(1)

    @staticmethod
    def tensor_decls(spec):
        return [TensorDecl(spec.weight, (spec.width,), "vector"), TensorDecl(spec.bias, (spec.width,), "vector"),
                TensorDecl(spec.alpha, (), "vector")]

    def forward(self, x, row_index=None, out_dtype=None):
        return kernels.tanh_norm(x, self.alpha, self.weight, self.bias, out_dtype or self.runtime.dtype, row_index)

    def scale_output(self, factor):
        self.weight, self.bias = self.weight * factor, self.bias * factor
