"""Attention whose heads are the difference of two softmax maps over the same values (`DifferentialAttentionSpec`).

    [q | k | v] = W h (+ b)   one stacked product; a norm and a rotation on every map of every head (`ops.head_work`)
    a_1, a_2 = the maps' attentions;  o = a_1 - lambda a_2, normed per head, times a factor (`ops.combine_maps`);  W_o o

On the attention kernels both maps of all query heads of a key head are ONE group: a cached key row is [k_1 | k_2 | 0], the
query row of map m holds q_m in the features of k_m and zeros in the others' (their products add exact zeros), and the value
row serves both maps.  So a request's keys and values are cached and read once, whatever the number of maps, and where
2 dim = vdim (the usual choice) nothing is padded.

A call without keys and values of its own (`own_kv` False) reads the pages an earlier call of the same heads wrote.
"""
from __future__ import annotations

import dataclasses
import math

import torch

from ..cache.spec import PagedKV
from .attention import MAX_HEAD_DIM, _pad_heads, neighbour_order, round_up
from .linear import Linear
from .registry import MIXERS, POSITIONS
from .spec import DifferentialAttentionSpec, TensorDecl

MAPS = 2


@dataclasses.dataclass(frozen=True)
class _KernelHeads:
    """What the attention kernels are told: every map a query head of the padded row's size."""
    num_heads: int
    num_kv_heads: int
    head_dim: int
    window: object


@MIXERS.register("differential_attention")
class DifferentialAttention:
    graph_safe = True

    @staticmethod
    def row_width(s: DifferentialAttentionSpec) -> int:
        """Features of a cached row: the maps' keys side by side, or a value head where that is wider."""
        return round_up(max(MAPS * round_up(s.dim, 8), round_up(s.vdim, 8)), 16)

    @staticmethod
    def declare(s: DifferentialAttentionSpec) -> dict:
        q, k, v, o = s.names
        rows = {q: s.num_heads * MAPS * s.dim}
        if s.own_kv:
            rows.update({k: s.num_kv_heads * MAPS * s.dim, v: s.num_kv_heads * s.vdim})
        d = {n: TensorDecl((r, s.hidden_size)) for n, r in rows.items()}
        if s.bias:
            d.update({n + s.bias_suffix: TensorDecl((r,)) for n, r in rows.items()})
        if s.qk_norm is not None:
            d.update({n + s.norm_suffix: TensorDecl((s.dim,), init="norm") for n in ((q, k) if s.own_kv else (q,))})
        d.update({n: TensorDecl((s.dim,), init="linear") for n in s.lambda_names})
        d[o] = TensorDecl((s.hidden_size, s.num_heads * s.vdim))
        return d

    @staticmethod
    def cache_need(s: DifferentialAttentionSpec):
        return PagedKV(s.num_kv_heads, DifferentialAttention.row_width(s), s.window,
                       keep=s.keep_first if s.window is not None else None)

    def __init__(self, s: DifferentialAttentionSpec, weights: dict, ctx):
        nq, nkv = s.num_heads, s.num_kv_heads
        if nq <= 0 or nkv <= 0 or nq % nkv:
            raise ValueError(f"{nkv} kv heads do not divide {nq} query heads")
        if s.window is not None and s.window <= 0:
            raise ValueError(f"window {s.window} must be positive (None reads every earlier key)")
        self.P = self.row_width(s)
        if self.P > MAX_HEAD_DIM:
            raise ValueError(f"differential attention: two maps of {s.dim} features and values of {s.vdim} need rows of {self.P}; "
                             f"the attention kernels take up to {MAX_HEAD_DIM}")
        if s.qk_norm is not None and (s.qk_norm.kind != "rms_norm" or s.qk_norm.size != s.dim):
            raise ValueError("differential attention: the norm of a map is an RMS norm over its features")
        self.spec, self.dtype = s, ctx.dtype
        self.D, self.V = round_up(s.dim, 8), round_up(s.vdim, 8)
        f32 = lambda t: t.to(device=ctx.device, dtype=torch.float32).contiguous()
        q, k, v, o = s.names
        rot = s.position
        order = neighbour_order(s.dim, rot.dim if rot is not None else 0, rot is None or rot.interleaved, weights[q].device)
        units = lambda t, n: _pad_heads(t.reshape((n, s.dim) + tuple(t.shape[1:]))[:, order].reshape(t.shape), n, s.dim, self.D)
        rows = lambda suffix, cast: ([units(cast(weights[q + suffix]), nq * MAPS)] +
                                     ([units(cast(weights[k + suffix]), nkv * MAPS), _pad_heads(cast(weights[v + suffix]), nkv, s.vdim, self.V)]
                                      if s.own_kv else []))
        self.in_proj = Linear(torch.cat(rows("", lambda t: t), dim=0).contiguous())
        self.bias = f32(torch.cat(rows(s.bias_suffix, lambda t: t.float()))) if s.bias else None
        self.norms = (None, None)
        if s.qk_norm is not None:
            qw = units(f32(weights[q + s.norm_suffix]), 1).contiguous()
            # (a call that reads another's keys norms no key: the kernel is given the query's weight for both)
            self.norms = (qw, units(f32(weights[k + s.norm_suffix]), 1).contiguous() if s.own_kv else qw)
        lq1, lk1, lq2, lk2 = (weights[n].detach().to("cpu", torch.float64) for n in s.lambda_names)
        self.lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + s.diff
        self.o_proj = Linear(_pad_heads(weights[o].t().contiguous(), nq, s.vdim, self.V).t().contiguous())
        self.rotary = None
        if rot is not None:
            self.rotary = POSITIONS.get(rot.kind)(rot, {}, ctx).fused_rotary()
            if self.rotary is None:
                raise TypeError(f"position kind {rot.kind!r} offers no table of frequencies to the head-work kernel")
        self.scale = s.scale if s.scale is not None else s.dim ** -0.5
        self.kernel_heads = _KernelHeads(nq * MAPS, nkv, self.P, s.window)

    def __call__(self, h, step, cache):
        from ..csrc import ops
        from . import attention_dispatch
        s, ws, tag = self.spec, step.workspace, step.tag
        group = step.groups[cache.group]
        T = h.shape[0]
        if s.own_kv != cache.writes:
            raise ValueError("differential attention: a call has key and value tensors if and only if it owns its cache")
        rows = self.in_proj(h, step, "diff.in")
        q = ws.get(tag + "diff.q", (T, s.num_heads * MAPS, self.P), self.dtype)
        ops.head_work(rows, self.bias, step.positions, group.slots if s.own_kv else None, self.norms[0], self.norms[1],
                      s.qk_norm.eps if s.qk_norm is not None else 0.0, self.rotary, None, q, cache.k if s.own_kv else None,
                      cache.v if s.own_kv else None, s.num_heads, s.num_kv_heads, MAPS, self.D, self.V, step.err, true_dim=s.dim)
        width = s.num_heads * MAPS * self.P
        maps = ws.get(tag + "diff.maps", (T, width), self.dtype)
        attention_dispatch.run(q.view(T, width), maps, cache, group, step, self.kernel_heads, self.scale, keep=s.keep_first)
        out = ws.get(tag + "diff.out", (T, s.num_heads * self.V), self.dtype)
        ops.combine_maps(maps.view(T, s.num_heads * MAPS, self.P), self.lam, 1.0 - s.diff, s.eps, s.vdim, out)
        return self.o_proj(out, step, "diff.o")
