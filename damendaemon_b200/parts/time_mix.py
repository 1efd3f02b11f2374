"""The time mixer: a matrix state per head whose rows decay per key channel by a factor that depends on the token.

Each of the five branches (receptance, key, value, gate, decay) reads its own blend of the mixer's input with that of the token
before. The block arrangement has its norm make the blends in the pass that norms the rows (``forward_mixes``). The four
square products of a step of few tokens are one grouped launch over the blends laid out plane by plane; the decay goes
through two small products with tanh in the first one's epilogue. A step of single tokens then takes one kernel (``kernels.time_step``: decay, recurrence over the request's float32 state, norm,
weight and gate of the read-out); a step with portions takes ``kernels.time_prepare``, ``kernels.time_scan`` and
``kernels.retention_finish``. The output projection adds into the stream in its epilogue. The state S (without a name) and the
last token's normed row ('shift') are per request, so a portion of a prompt continues exactly where the portion before stopped.
Everything between the projections' outputs and the operand of the output projection is float32.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.manager import RequestState
from .interfaces import Mixer
from .linear import linear
from .registry import register_mixer
from .spec import TensorDecl


def _square_names(spec):
    return (spec.receptance_weight, spec.key_weight, spec.value_weight, spec.gate_weight)


@register_mixer("time_mix")
class TimeMix(Mixer):
    graph_safe = True
    GROUPED_TOKENS = 128       # up to this many tokens the four products of a step are one grouped launch

    def __init__(self, spec, weights, runtime):
        self.spec, self.runtime = spec, runtime
        s = spec
        kernels.delta_state_shape(s.n_heads, s.head_dim, s.head_dim)            # raises for sizes the kernels do not take
        self.inner = s.n_heads * s.head_dim
        self.mix_weights = weights["+".join(s.mix_weights)].view(5, s.width)
        self.square_w = weights["+".join(_square_names(s))].view(4, self.inner, s.width)
        self.decay_down, self.decay_up = weights[s.decay_down], weights[s.decay_up]
        self.decay_bias, self.bonus = weights[s.decay_bias], weights[s.bonus].view(-1)
        self.out_norm, self.out_w = weights[s.out_norm], weights[s.out_weight]
        self.grouped = runtime.dtype == torch.bfloat16 and runtime.gemm != "simt" and s.width % 8 == 0
        self.groups = torch.arange(4, dtype=torch.int32, device=runtime.device)

    @staticmethod
    def tensor_decls(spec):
        s = spec
        inner = s.n_heads * s.head_dim
        return [TensorDecl("+".join(s.mix_weights), (5 * s.width,), "vector", False, tuple((n, (s.width,)) for n in s.mix_weights)),
                TensorDecl("+".join(_square_names(s)), (4 * inner, s.width), "matrix", False,
                           tuple((n, (inner, s.width)) for n in _square_names(s))),
                TensorDecl(s.decay_down, (s.decay_rank, s.width), "matrix"),
                TensorDecl(s.decay_up, (inner, s.decay_rank), "matrix"),
                TensorDecl(s.decay_bias, (inner,), "vector"),
                TensorDecl(s.bonus, (s.n_heads, s.head_dim), "vector"),
                TensorDecl(s.out_norm, (inner,), "vector"),
                TensorDecl(s.out_weight, (s.width, inner), "matrix")]

    @staticmethod
    def cache_needs(spec):
        s = spec
        return [RequestState(kernels.delta_state_shape(s.n_heads, s.head_dim, s.head_dim), "float32"),
                RequestState((s.width,), "float32", name="shift")]

    def mix_rows(self, n_tokens):
        """Rows a blend takes in ``forward_mixes``'s operand: a row tile of the grouped product where that runs."""
        if self.grouped and n_tokens <= self.GROUPED_TOKENS:
            return next(t for t in kernels.GROUPED_TCGEN05_TILES if t >= n_tokens)
        return n_tokens

    def _products(self, mixes, n):
        """r, k, v and the gate's input, row views [n, inner] of one buffer."""
        rows = mixes.shape[1]
        if self.grouped and n <= self.GROUPED_TOKENS and rows in kernels.GROUPED_TCGEN05_TILES:
            out = kernels.gemm_grouped_tcgen05(mixes[:4].view(4 * rows, -1), self.square_w, self.groups, rows).view(4, rows, self.inner)
        else:
            out = torch.empty((4, rows, self.inner), dtype=mixes.dtype, device=mixes.device)
            for i in range(4):
                linear(self.runtime, mixes[i, :n], self.square_w[i], out=out[i, :n])
        return tuple(out[i, :n] for i in range(4))

    def forward(self, y, residual, ctx, cache, position):
        raise ValueError("the time mixer reads blends of its input with the token before: it needs an arrangement whose norm makes "
                         "them (forward_mixes)")

    def forward_mixes(self, mixes, residual, ctx, cache, position):
        """mixes: [5, rows, width], rows at least the step's tokens (see mix_rows)."""
        s, rt, n = self.spec, self.runtime, residual.shape[0]
        if cache.state is None:
            raise ValueError("the time mixer needs its per-request state (a stop of the run order with a cache of its own)")
        r, k, v, gate = self._products(mixes, n)
        low = linear(rt, mixes[4, :n], self.decay_down, activation="tanh")
        decay_in = linear(rt, low, self.decay_up, out_dtype=torch.float32)
        if ctx.decode_only:
            mixed = kernels.time_step(r, k, v, gate, decay_in, self.decay_bias, self.bonus, self.out_norm, s.norm_eps, ctx.entry_slot,
                                      cache.state, s.n_heads, s.head_dim, s.head_dim)
        else:
            operands = kernels.time_prepare(r, k, v, decay_in, self.decay_bias, self.bonus, s.n_heads, s.head_dim, s.head_dim)
            read = kernels.time_scan(*operands, ctx.entry_start, ctx.entry_slot, cache.state, s.n_heads, s.head_dim, s.head_dim)
            mixed = kernels.retention_finish(read, gate, s.n_heads, s.norm_eps, r.dtype, weight=self.out_norm)
        return linear(rt, mixed, self.out_w, residual=residual, out_dtype=torch.float32, out=residual)
