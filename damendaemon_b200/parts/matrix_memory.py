"""The matrix memory mixer: linear attention whose state per head fades by one number per head and token.

One fused projection gives queries, keys, values and the output gate; with exponential gates a second, small one gives their
logarithms' inputs in float32. A step with portions runs ``kernels.memory_gates`` (where there are gates),
``memory_prepare``, ``memory_scan`` and ``memory_finish``; a step of single tokens runs ``memory_step`` alone where the read-out
is normed per head, and ``memory_finish`` behind it where all heads are normed together. The state is float32 and lives in the
request's slot (a ``RequestState`` need; with gates also the running maximum, a state named 'peak'), so a portion of a prompt
continues exactly where the portion before stopped. Everything between the projections' outputs and the operand of the output
projection is float32; the residual add is the last product's epilogue.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.manager import RequestState
from .interfaces import Mixer
from .linear import linear
from .registry import register_mixer
from .spec import TensorDecl


def _names(spec):
    return (spec.query_weight, spec.key_weight, spec.value_weight, spec.gate_weight)


@register_mixer("matrix_memory")
class MatrixMemory(Mixer):
    graph_safe = True

    def __init__(self, spec, weights, runtime):
        self.spec, self.runtime = spec, runtime
        s = spec
        gates = (s.input_gate, s.input_gate_bias, s.forget_gate, s.forget_gate_bias)
        self.gated = s.decay is None
        if any(g is None for g in gates) if self.gated else any(g is not None for g in gates):
            raise ValueError("a matrix memory fades by fixed decays or by its gates (input and forget, each with a bias)")
        if not self.gated and len(s.decay) != s.n_heads:
            raise ValueError(f"{len(s.decay)} decays for {s.n_heads} heads")
        if self.gated and s.gate_cap <= 0:
            raise ValueError("the cap of a matrix memory's gates must be positive")
        if s.activation not in (None, "silu"):
            raise ValueError(f"activation {s.activation!r} is not supported; known: [None, 'silu']")
        kernels.memory_state_shape(s.n_heads, s.head_dim, s.value_dim, self.gated)       # raises for sizes the kernels do not take
        key = "+".join(_names(s))
        self.proj_w = weights[key]
        if self.proj_w.shape[0] % 8:
            # rows of zeros make the projection's row stride a multiple of eight elements (their outputs are never read)
            pad = torch.zeros((-self.proj_w.shape[0] % 8, self.proj_w.shape[1]), dtype=self.proj_w.dtype, device=self.proj_w.device)
            self.proj_w = weights[key] = torch.cat([self.proj_w, pad], dim=0)
        self.qk_width, self.v_width = s.n_heads * s.head_dim, s.n_heads * s.value_dim
        self.out_norm, self.out_w = weights[s.out_norm], weights[s.out_weight]
        if self.gated:
            self.gates_w, self.gates_b = weights[s.input_gate + "+" + s.forget_gate], weights[s.input_gate_bias + "+" + s.forget_gate_bias]
        else:
            # the distance from one is formed in double precision: a decay near one has few float32 digits of it
            self.fade = torch.tensor([1.0 - d for d in s.decay], dtype=torch.float64).to(torch.float32).to(runtime.device)

    @staticmethod
    def tensor_decls(spec):
        s = spec
        qk, v = s.n_heads * s.head_dim, s.n_heads * s.value_dim
        shapes = ((qk, s.width), (qk, s.width), (v, s.width), (v, s.width))
        decls = [TensorDecl("+".join(_names(s)), (2 * qk + 2 * v, s.width), "matrix", False, tuple(zip(_names(s), shapes))),
                 TensorDecl(s.out_norm, (v,), "vector"),
                 TensorDecl(s.out_weight, (s.width, v), "matrix")]
        if s.decay is None:
            names = (s.input_gate, s.forget_gate)
            decls.append(TensorDecl("+".join(names), (2 * s.n_heads, s.width), "matrix", False, tuple((n, (s.n_heads, s.width)) for n in names)))
            names = (s.input_gate_bias, s.forget_gate_bias)
            decls.append(TensorDecl("+".join(names), (2 * s.n_heads,), "vector", False, tuple((n, (s.n_heads,)) for n in names)))
        return decls

    @staticmethod
    def cache_needs(spec):
        s = spec
        gated = s.decay is None
        needs = [RequestState(kernels.memory_state_shape(s.n_heads, s.head_dim, s.value_dim, gated), "float32")]
        return needs + ([RequestState((s.n_heads,), "float32", name="peak")] if gated else [])

    def forward(self, y, residual, ctx, cache, position):
        s, a, b = self.spec, self.qk_width, self.v_width
        if cache.state is None:
            raise ValueError("the matrix memory needs its per-request state (a stop of the run order with a cache of its own)")
        proj = linear(self.runtime, y, self.proj_w)
        q, k, v, gate = proj[:, :a], proj[:, a:2 * a], proj[:, 2 * a:2 * a + b], proj[:, 2 * a + b:2 * a + 2 * b]
        sizes = (s.n_heads, s.head_dim, s.value_dim)
        silu = s.activation == "silu"
        z = linear(self.runtime, y, self.gates_w, self.gates_b, out_dtype=torch.float32) if self.gated else None
        if ctx.decode_only:
            source = {"gates": (z, s.gate_cap, cache.named["peak"])} if self.gated else {"fade": self.fade}
            mixed = kernels.memory_step(q, k, v, gate, ctx.entry_slot, cache.state, *sizes, weight=None if s.norm_together else self.out_norm,
                                        eps=s.norm_eps, den_eps=s.denominator_eps, scale=s.query_scale, silu=silu, **source)
            if s.norm_together:
                read, floor = mixed
        else:
            fade, take, floor = self.fade if not self.gated else None, None, None
            if self.gated:
                fade, take, floor = kernels.memory_gates(z, s.gate_cap, ctx.entry_start, ctx.entry_slot, cache.named["peak"])
            operands = kernels.memory_prepare(q, k, v, *sizes, scale=s.query_scale, silu=silu, take=take)
            read = kernels.memory_scan(*operands, fade, ctx.entry_start, ctx.entry_slot, cache.state, s.head_dim, s.value_dim)
        if s.norm_together or not ctx.decode_only:
            mixed = kernels.memory_finish(read, gate, self.out_norm, s.n_heads, s.value_dim, s.norm_eps, s.denominator_eps, floor=floor,
                                          together=s.norm_together)
        return linear(self.runtime, mixed, self.out_w, residual=residual, out_dtype=torch.float32, out=residual)
