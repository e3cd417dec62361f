"""A causal language model assembled from a `ModelPlan`:
embedding -> the calls of the running order -> final norm -> output head
(crates/model/src/causal_lm/mod.rs:180-221 of the reference).  Only the rows
whose logits are wanted go through the final norm and the head."""
from __future__ import annotations

import torch

from ..cache.spec import widened
from .base import BuildContext, Residual, StreamSum, prefixed, sub_weights
from .registry import BLOCKS, EMBEDDINGS, HEADS, NORMS
from .spec import ModelPlan, TensorDecl


def declare_model(plan: ModelPlan) -> dict:
    """Every tensor the model binds: {checkpoint name: TensorDecl}."""
    emb, head = plan.embedding_spec, plan.head_spec
    d = prefixed(EMBEDDINGS.get(emb.kind).declare(emb), plan.embed_prefix)
    for i, block in enumerate(plan.layers):
        d.update(prefixed(BLOCKS.get(block.kind).declare(block), plan.layer_prefix.format(i)))
    d.update(prefixed(NORMS.get(plan.final_norm.kind).declare(plan.final_norm), plan.final_norm_prefix))
    d.update(prefixed(HEADS.get(head.kind).declare(head), plan.head_prefix))
    d.update({name: TensorDecl((rows, plan.hidden_size)) for name, rows in plan.stream_tables})
    return d


def cache_needs(plan: ModelPlan) -> list:
    """The need of every entry of the running order (None for an entry that
    keeps nothing or that reads another entry's cache; what such a reader can reach is
    kept by the owner), then the embedding's, if it keeps something (`cache_sources` beside it)."""
    needs = []
    for call in plan.order:
        block = plan.layers[call.layer]
        need = BLOCKS.get(block.kind).cache_need(block)
        if call.cache_of is not None:
            needs[call.cache_of] = widened(needs[call.cache_of], need)
            need = None
        needs.append(need)
    emb = plan.embedding_spec
    own = getattr(EMBEDDINGS.get(emb.kind), "cache_need", None)
    if own is not None:
        needs.append(own(emb))
    return needs


def cache_sources(plan: ModelPlan) -> list:
    """For every entry of `cache_needs`: the earlier entry whose cache it reads, or None."""
    sources = [c.cache_of for c in plan.order]
    return sources + [None] * (len(cache_needs(plan)) - len(sources))


class CausalLM:
    def __init__(self, plan: ModelPlan, weights: dict, ctx: BuildContext):
        plan.validate()
        self.plan = plan
        self.ctx = ctx
        emb, head = plan.embedding_spec, plan.head_spec
        self.embedding = EMBEDDINGS.get(emb.kind)(emb, sub_weights(weights, plan.embed_prefix), ctx)
        self.layers = [BLOCKS.get(b.kind)(b, sub_weights(weights, plan.layer_prefix.format(i)), ctx)
                       for i, b in enumerate(plan.layers)]
        self.final_norm = NORMS.get(plan.final_norm.kind)(plan.final_norm,
                                                          sub_weights(weights, plan.final_norm_prefix), ctx)
        self.head = HEADS.get(head.kind)(head, sub_weights(weights, plan.head_prefix), ctx, embedding=self.embedding)
        # rows that are added to the stream between two calls, in float32 like the stream
        self.stream_tables = {name: weights[name].to(device=ctx.device, dtype=torch.float32).contiguous()
                              for name, _ in plan.stream_tables}
        self.keeps_embedding = any(call.add_embedding for call in plan.order)
        self.graph_safe = all(getattr(part, "graph_safe", False) for part in [self.embedding, self.head] + self.layers)

    def forward(self, step, caches, watch=None) -> torch.Tensor:
        """Logits float32 [len(step.logit_rows), vocab].  `watch(i, x)`, when given, is called after every entry of
        the running order with the stream brought up to date (a reader for tests and comparisons)."""
        ws = step.workspace
        x = ws.get(step.tag + "residual", (step.num_tokens, self.plan.hidden_size), torch.float32)
        # the embedding's output is kept apart when a later call adds it again: the stream then starts as a sum with that base
        first = ws.get(step.tag + "embedded", tuple(x.shape), torch.float32) if self.keeps_embedding else x
        if getattr(self.embedding, "keeps_state", False):
            self.embedding(step, first, caches[len(self.plan.order)])
        else:
            self.embedding(step, first)
        residual = Residual(x)
        if self.keeps_embedding:
            residual.pending = StreamSum(base=first)
        order = self.plan.order
        for i, (call, cache) in enumerate(zip(order, caches)):
            layer = self.layers[call.layer]
            residual.add_before_next(first if call.add_embedding else None,
                                     self.stream_tables[call.add_row[0]][call.add_row[1]] if call.add_row is not None else None)
            if (residual.deferred is not None and not getattr(layer, "takes_deferred", False)) or \
                    (isinstance(residual.pending, StreamSum) and not getattr(layer, "takes_sum", False)):
                residual.settle()
            if getattr(layer, "chains_norms", False):
                # a block may leave the next block's first norm in factored form (parts/base.py, ScaledRows)
                nxt = self.layers[order[i + 1].layer] if i + 1 < len(order) else None
                if nxt is not None and (order[i + 1].add_embedding or order[i + 1].add_row is not None):
                    nxt = None
                ask = getattr(nxt, "input_norm_for_fusion", None)
                layer(residual, step, cache, next_norm=ask(step.num_tokens) if ask else None)
            else:
                layer(residual, step, cache)
            if watch is not None:
                residual.settle()
                if residual.pending is not None or residual.normed is not None:
                    raise NotImplementedError("watching a model whose blocks leave their results pending")
                watch(i, residual.x)
        if residual.deferred is not None or not getattr(self.final_norm, "takes_sum", False):
            residual.settle()
        R = step.logit_rows.shape[0]
        if R == 0:
            return ws.get(step.tag + "logits", (0, self.plan.vocab_size), torch.float32)
        h = self.final_norm(residual.x, residual.pending, step, rows=step.logit_rows, tag="final_norm")   # pending: the last block has no next norm
        return self.head(h, step)
