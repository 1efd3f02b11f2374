"""What a part must look like. Parts are chosen by the spec's ``kind`` and built as
``cls(spec, weights, runtime)``; none of them knows which model it is in.

``weights``  {checkpoint name: device tensor}, already checked and placed.
``runtime``  a ``Runtime`` (below): engine dtype, device and kernel choices.
``ctx``      the step's ``StepContext`` (engine/context.py): flattened token metadata
             on the device, block tables per cache group, and ``ctx.attend(q, k, v, cache,
             heads, scale, window)``: cache write plus paged causal attention with the best
             kernel for the step.
``cache``    a ``LayerCache`` (cache/manager.py): ``kv`` pages of this layer
             [pages, 2, kv_heads, page_size, head_dim], ``group`` (its block table is
             ``ctx.block_table(cache.group)``), ``state`` rows [max_requests, ...],
             ``writable`` (False when the stop reads another stop's cache).

Embedding         tensor_decls(spec); forward(ctx, position) -> float32 residual stream [N,width]
Head              tensor_decls(spec); forward(x, ctx) -> float32 logits [ctx.n_wanted, vocab] at rows ctx.want_rows
Norm              tensor_decls(spec); forward(x_f32 [N,width], row_index=None) -> [N,width] engine dtype;
                  scale_output(factor): everything it returns is multiplied by factor from then on;
                  optionally add_normed(x, terms, factor, rounded): x += factor * norm(the terms), in place, and x
                  rounded to the engine dtype if asked
PositionEncoding  tensor_decls(spec); embedding_table() -> table or None (added to the token
                  embedding by the fused embedding kernel); on_embedding(x, ctx) -> x for
                  encodings that act there without a table; on_query_key(q, k, ctx) -> (q, k)
                  for encodings that rotate or bias inside the mixer
Mixer             tensor_decls(spec); cache_needs(spec) -> [a paged need (cache/manager.py: PagedKeyValues, or any
                  PagedNeed of the mixer's own) | RequestState]; forward(y, residual, ctx, cache, position) ->
                  residual + mix(y)   (float32 [N,width]); optionally portion_multiple: where the mixer likes a
                  prompt to be cut (the engine passes the largest one on to the scheduler). A mixer that reads
                  blends of its input with the token before (mix_weights [S, width], a state named 'shift') may
                  offer forward_mixes(mixes [S, >= N, width], residual, ctx, cache, position) and
                  mix_rows(n_tokens) (rows it wants a blend padded to): the arrangement then has the norm make them
FeedForward       tensor_decls(spec); forward(y, residual, ctx) -> residual + ff(y)
Arrangement       cls(layer_spec, norms, mixer, feed_forward), norms being the built norms of layer_spec.norms in
                  order; forward(x, ctx, cache, position) -> x

``residual`` is the float32 residual stream; a part returns the updated stream and may
write it in place (the GEMM epilogues add into it). ``residual`` None: the part returns its bare
result, float32. ``forward_terms(y, ctx[, cache, position])`` of a mixer or feed-forward is its bare
result as operands of ``kernels.post_norm`` (a tensor; or two with factors; or rows and which of them a
token adds up), so that whatever norms and adds the result does not need it made first.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from .paged_attention import AttentionTuning


@dataclass
class Runtime:
    dtype: torch.dtype            # engine dtype: torch.bfloat16 or torch.float32
    device: torch.device
    gemm: str = "auto"            # 'auto' | 'simt' | 'tcgen05'
    attention: str = "auto"       # 'auto' | 'mma' (no tcgen05 prompt kernel) | 'rows' (the general kernel only)
    attention_tuning: AttentionTuning = field(default_factory=AttentionTuning)   # measured thresholds of the kernel choice
    page_size: int = 16           # tokens per cache page (mixers ask their kernels what they support at this size)


class Part:
    @staticmethod
    def tensor_decls(spec):
        return []


class Mixer(Part):
    # True if forward() launches the same kernels with the same arguments whenever the step's
    # counts are the same (everything that varies is read from device memory), so that a
    # decode step may be replayed from a CUDA graph. Parts that plan on the host say False.
    graph_safe = False

    @staticmethod
    def cache_needs(spec):
        return []

    def forward(self, y, residual, ctx, cache, position):
        raise NotImplementedError

    def forward_terms(self, y, ctx, cache, position):
        return {"a": self.forward(y, None, ctx, cache, position)}


class FeedForward(Part):
    graph_safe = False

    def forward(self, y, residual, ctx):
        raise NotImplementedError

    def forward_terms(self, y, ctx):
        return {"a": self.forward(y, None, ctx)}


class Norm(Part):
    def forward(self, x, row_index=None):
        raise NotImplementedError


class Embedding(Part):
    def forward(self, ctx, position):
        raise NotImplementedError


class Head(Part):
    def forward(self, x, ctx):
        raise NotImplementedError


class PositionEncoding(Part):
    def embedding_table(self):
        return None

    def on_embedding(self, x, ctx):
        return x

    def on_query_key(self, q, k, ctx):
        return q, k
