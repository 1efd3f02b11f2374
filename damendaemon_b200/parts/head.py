"""Heads: from the residual stream to float32 logits at the wanted rows.

'linear': the final norm on the wanted rows only, then logits = y . W^T (+ bias); W may be the embedding's
table (damendaemon/gpt2.py:18,65-66: ``head is embed``, the norm after the last prompt row was picked); with ``softcap`` c
the logits become c * tanh(logits / c). A scale of the logits is folded into the
weights of the head's own norm (and into the bias), so it costs no pass over the logits.
"""
from __future__ import annotations

import torch

from .. import kernels
from .interfaces import Head
from .linear import linear
from .registry import NORMS, lookup, register_head
from .spec import TensorDecl


@register_head("linear")
class LinearHead(Head):
    def __init__(self, spec, weights, runtime):
        self.spec, self.runtime = spec, runtime
        self.norm = lookup(NORMS, spec.norm, "norm")(spec.norm, weights, runtime)
        self.weight = weights[spec.weight]
        self.bias = weights[spec.bias] if spec.bias else None
        if spec.scale != 1.0:
            self.norm.scale_output(spec.scale)
            self.bias = None if self.bias is None else self.bias * spec.scale

    @staticmethod
    def tensor_decls(spec):
        decls = list(lookup(NORMS, spec.norm, "norm").tensor_decls(spec.norm))
        if not spec.tied:
            decls.append(TensorDecl(spec.weight, (spec.vocab_size, spec.width), "matrix"))
        if spec.bias:
            decls.append(TensorDecl(spec.bias, (spec.vocab_size,), "vector"))
        return decls

    def forward(self, x, ctx):
        y = self.norm.forward(x, row_index=ctx.want_rows)
        logits = linear(self.runtime, y, self.weight, self.bias, out_dtype=torch.float32)
        if self.spec.softcap:
            kernels.tanh_cap(logits, self.spec.softcap)
        return logits
