"""Two mixers side by side on the same input: out = left_scale * left(h) + right_scale * right(h).

Each side is a mixer of any registered kind with its own tensors (under `prefixes`) and its own cache or state: the
part asks for `Several` needs and hands each side its own `CallCache`.  A caller whose next step reads the sum anyway (a norm
on the mixer's output) may ask for the two results as they are (`as_pair`) and form the sum itself.  With `out_norms` each
side's result passes an RMS norm of its own first; these norms, too, are left to the caller that takes the pair."""
from __future__ import annotations

import torch

from ..cache.spec import Several
from .base import prefixed, sub_weights
from .registry import MIXERS, NORMS
from .spec import ParallelMixerSpec


@MIXERS.register("parallel_mixer")
class ParallelMixer:
    @staticmethod
    def declare(s: ParallelMixerSpec) -> dict:
        d = {}
        for side, prefix in zip((s.left, s.right), s.prefixes):
            d.update(prefixed(MIXERS.get(side.kind).declare(side), prefix))
        for norm, prefix in zip(s.out_norms or (), s.out_norm_prefixes):
            d.update(prefixed(NORMS.get(norm.kind).declare(norm), prefix))
        return d

    @staticmethod
    def cache_need(s: ParallelMixerSpec):
        needs = [MIXERS.get(side.kind).cache_need(side) for side in (s.left, s.right)]
        return Several(tuple(needs))

    def __init__(self, s: ParallelMixerSpec, weights: dict, ctx):
        self.spec, self.dtype = s, ctx.dtype
        self.left = MIXERS.get(s.left.kind)(s.left, sub_weights(weights, s.prefixes[0]), ctx)
        self.right = MIXERS.get(s.right.kind)(s.right, sub_weights(weights, s.prefixes[1]), ctx)
        self.norms = None
        if s.out_norms is not None:
            if any(n.kind != "rms_norm" for n in s.out_norms) or s.out_norms[0].eps != s.out_norms[1].eps:
                raise ValueError("the norms of two mixers side by side are RMS norms with one eps")
            self.norms = [NORMS.get(n.kind)(n, sub_weights(weights, p), ctx) for n, p in zip(s.out_norms, s.out_norm_prefixes)]
        self.graph_safe = bool(getattr(self.left, "graph_safe", False) and getattr(self.right, "graph_safe", False))

    returns_pair = True        # __call__(as_pair=True) leaves the sum to the caller (`ScaledPair`)

    def take_out_bias(self):
        """The bias of the sum, if the sides' last products have one and nothing stands between them and the sum; the sides
        then leave it out."""
        if self.norms is not None:
            return None
        total = None
        for side, scale in ((self.left, self.spec.left_scale), (self.right, self.spec.right_scale)):
            bias = side.take_out_bias() if hasattr(side, "take_out_bias") else None
            if bias is not None:
                total = scale * bias if total is None else total + scale * bias
        return total

    def __call__(self, h, step, cache, as_pair=False):
        from ..csrc import ops
        a = self.left(h, step, cache.parts[0])
        b = self.right(h, step, cache.parts[1])
        if as_pair:
            from .base import ScaledPair
            if self.norms is not None:
                return ScaledPair(a, self.spec.left_scale, b, self.spec.right_scale, self.norms[0].weight, self.norms[1].weight,
                                  self.norms[0].spec.eps)
            return ScaledPair(a, self.spec.left_scale, b, self.spec.right_scale)
        out = step.workspace.get(step.tag + "par.out", tuple(a.shape), self.dtype)
        if self.norms is not None:
            total = step.workspace.get(step.tag + "par.sum", tuple(a.shape), torch.float32).zero_()
            for y, norm, scale in ((a, self.norms[0], self.spec.left_scale), (b, self.norms[1], self.spec.right_scale)):
                ops.rmsnorm_add(y, norm.weight, norm.spec.eps, scale, total)
            return total if self.dtype == torch.float32 else ops.cast(total, out)
        return ops.scaled_sum(a, self.spec.left_scale, b, self.spec.right_scale, out)
