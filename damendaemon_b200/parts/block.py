"""Block arrangements: how a layer's norms, mixer and feed-forward are wired.

'pre_norm': x = x + mixer(norm[0](x)); x = x + feed_forward(norm[1](x))  (damendaemon/gpt2.py:47-64).
'pre_norm_mixer': x = x + mixer(norm[0](x)), a layer without a feed-forward.
'parallel': y = norm[0](x); x = x + mixer(y) + feed_forward(y): one norm, both read its output, both results are added
to the float32 stream (by the epilogues of their last products, one after the other). With two norms the mixer reads
norm[0](x) and the feed-forward norm[1](x), both of the same x and, where the norms allow it, from one pass over it; a mixer
that reads blends of its input with the token before gets them from that pass as well.
'pre_norm_shift': 'pre_norm' (or, with one norm, 'pre_norm_mixer') whose mixer reads s[t] = n[t] + (n[t-1] - n[t]) * mu
with n = norm[0](x) and mu one number per channel; n[t-1] of a sequence's first token is zero, and across steps it is kept
per request (a state named 'shift' at the layer's cache site).
'post_norm': x = x + c norm[0](mixer(x)); x = x + c norm[1](feed_forward(x)) (with one norm there is no feed-forward): a
sublayer reads the stream itself, in the engine dtype. Norm, add and the rounding that the next sublayer reads are one pass.
"""
from __future__ import annotations

from .. import kernels
from ..cache.manager import RequestState
from .registry import register_arrangement
from .spec import TensorDecl


def normed_mixer(norm, mixer, x, ctx, cache, position):
    """x + mixer(norm(x)). A mixer that reads blends of its input with the token before gets them from the norm's own pass."""
    if hasattr(mixer, "forward_mixes"):
        mixes, _ = norm.forward_mixes(x, mixer.mix_weights, cache.named["shift"], ctx, rows_per_mix=mixer.mix_rows(ctx.n_tokens))
        return mixer.forward_mixes(mixes, x, ctx, cache, position)
    return mixer.forward(norm.forward(x), x, ctx, cache, position)


def check_mixes(norm, mixer):
    if hasattr(mixer, "forward_mixes") and not hasattr(norm, "forward_mixes"):
        raise ValueError("the norm before a mixer that reads blends with the token before must offer forward_mixes (the RMS norm does)")


@register_arrangement("pre_norm")
class PreNormBlock:
    def __init__(self, spec, norms, mixer, feed_forward):
        if len(norms) != 2:
            raise ValueError(f"a pre-norm block takes two norms (before the mixer, before the feed-forward), got {len(norms)}")
        check_mixes(norms[0], mixer)
        self.spec, self.norms, self.mixer, self.feed_forward = spec, list(norms), mixer, feed_forward

    def forward(self, x, ctx, cache, position):
        x = normed_mixer(self.norms[0], self.mixer, x, ctx, cache, position)
        return self.feed_forward.forward(self.norms[1].forward(x), x, ctx)


@register_arrangement("pre_norm_mixer")
class PreNormMixerOnly:
    def __init__(self, spec, norms, mixer, feed_forward):
        if len(norms) != 1:
            raise ValueError(f"a mixer-only block takes one norm, got {len(norms)}")
        check_mixes(norms[0], mixer)
        self.spec, self.norms, self.mixer, self.feed_forward = spec, list(norms), mixer, feed_forward

    def forward(self, x, ctx, cache, position):
        return normed_mixer(self.norms[0], self.mixer, x, ctx, cache, position)


@register_arrangement("parallel")
class ParallelBlock:
    def __init__(self, spec, norms, mixer, feed_forward):
        if len(norms) not in (1, 2):
            raise ValueError(f"a parallel block takes one norm or two, got {len(norms)}")
        self.spec, self.norms, self.mixer, self.feed_forward = spec, list(norms), mixer, feed_forward
        self.together = len(norms) == 2 and getattr(norms[0], "pairs_with", lambda _: False)(norms[1])
        check_mixes(norms[0], mixer)
        self.mixes = hasattr(mixer, "forward_mixes")

    def forward(self, x, ctx, cache, position):
        # both norms read the stream before either branch adds to it
        if self.mixes:
            mixes, z = self.norms[0].forward_mixes(x, self.mixer.mix_weights, cache.named["shift"], ctx,
                                                   other=self.norms[1] if self.together else None,
                                                   rows_per_mix=self.mixer.mix_rows(ctx.n_tokens))
            if not self.together:
                z = self.norms[-1].forward(x)
            x = self.mixer.forward_mixes(mixes, x, ctx, cache, position)
            return self.feed_forward.forward(z, x, ctx)
        if self.together:
            y, z = self.norms[0].forward_pair(self.norms[1], x)
        else:
            y = self.norms[0].forward(x)
            z = self.norms[1].forward(x) if len(self.norms) == 2 else y
        x = self.mixer.forward(y, x, ctx, cache, position)
        return self.feed_forward.forward(z, x, ctx)


@register_arrangement("pre_norm_shift")
class ShiftedPreNormBlock:
    def __init__(self, spec, norms, mixer, feed_forward):
        if len(norms) not in (1, 2):
            raise ValueError(f"a shifted pre-norm block takes one norm (no feed-forward) or two, got {len(norms)}")
        if not spec.shift_weight:
            raise ValueError("a shifted pre-norm block needs the name of its shift weights")
        if not hasattr(norms[0], "forward_shifted"):
            raise ValueError("the norm before a shifted mixer must offer forward_shifted (the RMS norm does)")
        self.spec, self.norms, self.mixer, self.feed_forward = spec, list(norms), mixer, feed_forward
        self.shift = None

    def bind(self, weights):
        self.shift = weights[self.spec.shift_weight]

    @staticmethod
    def tensor_decls(spec):
        return [TensorDecl(spec.shift_weight, (spec.norms[0].width,), "vector")]

    @staticmethod
    def cache_needs(spec):
        return [RequestState((spec.norms[0].width,), "float32", name="shift")]

    def forward(self, x, ctx, cache, position):
        y = self.norms[0].forward_shifted(x, self.shift, cache.named["shift"], ctx)
        x = self.mixer.forward(y, x, ctx, cache, position)
        if len(self.norms) == 1:
            return x
        return self.feed_forward.forward(self.norms[1].forward(x), x, ctx)


ROUNDED = "rounded stream"       # StepContext.shared: (the stream's tensor, its values in the engine dtype)


@register_arrangement("post_norm")
class PostNormBlock:
    leaves_rounded = True        # forward() leaves ctx.shared[ROUNDED] in step with the stream it returns

    def __init__(self, spec, norms, mixer, feed_forward):
        if len(norms) not in (1, 2):
            raise ValueError(f"a post-norm block takes one norm (no feed-forward) or two, got {len(norms)}")
        if any(not hasattr(n, "add_normed") for n in norms):
            raise ValueError("the norms of a post-norm block must offer add_normed (the RMS norm does)")
        if hasattr(mixer, "forward_mixes"):
            raise ValueError("a mixer that reads blends with the token before needs a norm in front of it that makes them")
        self.spec, self.norms, self.mixer, self.feed_forward = spec, list(norms), mixer, feed_forward

    def forward(self, x, ctx, cache, position):
        known, y = ctx.shared.get(ROUNDED, (None, None))
        if known is not x:
            y = kernels.round_rows(x, self.norms[0].runtime.dtype)
        factor = self.spec.residual_factor
        y = self.norms[0].add_normed(x, self.mixer.forward_terms(y, ctx, cache, position), factor)
        if len(self.norms) == 2:
            y = self.norms[1].add_normed(x, self.feed_forward.forward_terms(y, ctx), factor)
        ctx.shared[ROUNDED] = (x, y)
        return x
