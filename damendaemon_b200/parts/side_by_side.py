"""Two mixers side by side: both read the same input; each output is divided by its root mean square over the model width
and multiplied by a weight, and ``factor`` times their sum is added to the stream; or, without norms, the two are added with
a factor each.

The two are mixers of any registered kind, built from their own specs; they share the stop's cache site, so their cache
needs must not collide (at most one paged need, one state without a name, and names that differ). Each runs as it would
alone, without a residual: its last product leaves the bare result in float32.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.manager import PagedNeed, RequestState
from .interfaces import Mixer
from .registry import MIXERS, lookup, register_mixer
from .spec import TensorDecl


def _both(spec):
    return ((spec.left, lookup(MIXERS, spec.left, "mixer")), (spec.right, lookup(MIXERS, spec.right, "mixer")))


@register_mixer("side_by_side")
class SideBySide(Mixer):
    def __init__(self, spec, weights, runtime):
        self.spec, self.runtime = spec, runtime
        self.left, self.right = (cls(sub, weights, runtime) for sub, cls in _both(spec))
        if (spec.left_norm is None) != (spec.right_norm is None):
            raise ValueError("two mixers side by side are both normed or neither is")
        self.normed = spec.left_norm is not None
        if self.normed:
            self.left_norm, self.right_norm = weights[spec.left_norm], weights[spec.right_norm]
        self.graph_safe = bool(getattr(self.left, "graph_safe", False) and getattr(self.right, "graph_safe", False))
        self.portion_multiple = max(int(getattr(self.left, "portion_multiple", 1)), int(getattr(self.right, "portion_multiple", 1)))

    @staticmethod
    def tensor_decls(spec):
        decls = [d for sub, cls in _both(spec) for d in cls.tensor_decls(sub)]
        if spec.left_norm is None:
            return decls
        return decls + [TensorDecl(spec.left_norm, (spec.width,), "vector"), TensorDecl(spec.right_norm, (spec.width,), "vector")]

    @staticmethod
    def cache_needs(spec):
        needs = [n for sub, cls in _both(spec) for n in cls.cache_needs(sub)]
        paged = [n for n in needs if isinstance(n, PagedNeed)]
        names = [n.name for n in needs if isinstance(n, RequestState)]
        if len(paged) > 1 or len(set(names)) != len(names):
            raise ValueError("two mixers side by side share one cache site: at most one of them may keep pages, and their states "
                             f"must differ in name (pages: {len(paged)}, states: {names})")
        return needs

    def forward(self, y, residual, ctx, cache, position):
        if residual is None:
            residual = torch.zeros((y.shape[0], self.spec.width), dtype=torch.float32, device=y.device)
        if not self.normed:
            kernels.post_norm(residual, **self.forward_terms(y, ctx, cache, position))
            return residual
        left, right = (m.forward(y, None, ctx, cache, position) for m in (self.left, self.right))
        return kernels.norm_pair_add(residual, left, right, self.left_norm, self.right_norm, self.spec.norm_eps, self.spec.factor)

    def forward_terms(self, y, ctx, cache, position):
        if self.normed:
            return super().forward_terms(y, ctx, cache, position)
        left, right = (m.forward(y, None, ctx, cache, position) for m in (self.left, self.right))
        return {"a": left, "scale": self.spec.left_scale, "other": right, "other_scale": self.spec.right_scale}
