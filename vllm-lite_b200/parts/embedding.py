"""Token embedding: x[t] = table[id[t]] * scale, a row gather into the float32 residual stream; the reference has no scaling
(crates/model/src/causal_lm/mod.rs:28-46 of the reference).

An embedding part offers
    declare(spec) -> {relative tensor name: TensorDecl}            static
    __init__(spec, weights, ctx)
    __call__(step, x)        fills x float32 [T, hidden] from step.tokens (and step.positions if it likes)
    (with `keeps_state` True also cache_need(spec), static, and __call__(step, x, cache): something of the request is kept
    from step to step)
    tied_weight()            the [vocab, hidden] matrix an output head may share, or None
and may say `graph_safe = True` (parts/base.py)."""
from __future__ import annotations

from ..cache.spec import FixedState
from .registry import EMBEDDINGS
from .spec import EmbeddingSpec, PairEmbeddingSpec, TensorDecl


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding:
    graph_safe = True

    @staticmethod
    def declare(spec: EmbeddingSpec) -> dict:
        return {spec.tensor: TensorDecl((spec.vocab_size, spec.hidden_size))}

    def __init__(self, spec: EmbeddingSpec, weights: dict, ctx):
        self.spec = spec
        self.table = weights[spec.tensor]

    def tied_weight(self):
        return self.table

    def __call__(self, step, x):
        from ..csrc import ops
        return ops.embed(step.tokens, self.table, x, step.err, self.spec.scale)     # an id outside the table is flagged, not read


@EMBEDDINGS.register("pair_embedding")
class PairEmbedding:
    """x[t] = table[id_t] * scale + pairs[row(id_(t-1), id_t)]: a row of a second table chosen by the token before and this
    one (`PairEmbeddingSpec`).  The token before a portion is part of the request's state, on the device like the tokens
    themselves, so a decode step launched before the host knows its token works as any other."""
    graph_safe = True
    keeps_state = True

    @staticmethod
    def declare(spec: PairEmbeddingSpec) -> dict:
        return {spec.tensor: TensorDecl((spec.vocab_size, spec.hidden_size)),
                spec.pair_tensor: TensorDecl((spec.buckets + 1, spec.hidden_size))}

    @staticmethod
    def cache_need(spec: PairEmbeddingSpec):
        return FixedState((1,), "int32")

    def __init__(self, spec: PairEmbeddingSpec, weights: dict, ctx):
        self.spec = spec
        self.table, self.pairs = weights[spec.tensor], weights[spec.pair_tensor]

    def tied_weight(self):
        return self.table

    def __call__(self, step, x, cache):
        from ..csrc import ops
        s = self.spec
        return ops.embed_pair(step.tokens, self.table, self.pairs, x, s.scale, s.buckets, s.mul_prev, s.mul_cur, cache.state,
                              step.cu_seqlens, step.state_slots, step.req_index, step.positions, step.err)
