"""Mixers whose recurrence runs element by element, S_t = a_t S_(t-1) + b_t: a minimal gated recurrence (its gates depend on the
token at hand, not on the state) and a real-gated linear recurrent unit behind a short convolution.

Each is: one stacked projection of the input -> (a short causal convolution, a product per block of channels for the gates)
-> one kernel that makes a, b and the output's gate, walks the step's tokens from the state in the request's slot and
multiplies by the gate (csrc/linear_scan.cu) -> the output projection.  The state of a request is one row of float32 numbers
(`FixedState`), zero when the slot is handed out: the convolution's last inputs first, then S.  Gates, decays with their
logarithms, the recurrence and its state are float32 whatever the model's dtype; the gates' products leave float32 sums.
"""
from __future__ import annotations

import torch

from ..cache.spec import FixedState
from .linear import Linear
from .registry import MIXERS
from .spec import GatedLruSpec, MinGruSpec, TensorDecl


def _f32(t, ctx):
    return t.to(device=ctx.device, dtype=torch.float32).contiguous()


@MIXERS.register("min_gru")
class MinGru:
    graph_safe = True

    @staticmethod
    def declare(s: MinGruSpec) -> dict:
        z, x, g, o = s.names
        d = {n: TensorDecl((s.width, s.hidden_size)) for n in (z, x, g)}
        d.update({n + s.bias_suffix: TensorDecl((s.width,), init="unit") for n in (z, x)})
        d[o] = TensorDecl((s.hidden_size, s.width))
        return d

    @staticmethod
    def cache_need(s: MinGruSpec):
        return FixedState((s.width,))

    def __init__(self, s: MinGruSpec, weights: dict, ctx):
        if s.width <= 0:
            raise ValueError(f"gated recurrence: {s.width} channels")
        self.spec, self.dtype = s, ctx.dtype
        z, x, g, o = s.names
        self.in_proj = Linear(torch.cat([weights[n] for n in (z, x, g)], dim=0).contiguous())
        self.o_proj = Linear(weights[o])
        self.biases = tuple(_f32(weights[n + s.bias_suffix], ctx) for n in (z, x))

    def __call__(self, h, step, cache):
        from ..csrc import ops
        proj = self.in_proj(h, step, "mg.in")
        out = step.workspace.get(step.tag + "mg.out", (h.shape[0], self.spec.width), self.dtype)
        ops.linear_scan("min_gru", proj, self.biases, cache.state, 0, step.cu_seqlens, step.state_slots, out,
                        longest=step.max_query_len)
        return self.o_proj(out, step, "mg.o")


@MIXERS.register("gated_lru")
class GatedLru:
    graph_safe = True

    @staticmethod
    def declare(s: GatedLruSpec) -> dict:
        y, x, conv, r, i, lam, o = s.names
        C, K, b = s.width, s.width // max(s.blocks, 1), s.bias_suffix
        return {y: TensorDecl((C, s.hidden_size)), y + b: TensorDecl((C,)), x: TensorDecl((C, s.hidden_size)), x + b: TensorDecl((C,)),
                conv: TensorDecl((C, s.conv), init="conv"), conv + b: TensorDecl((C,)), r: TensorDecl((s.blocks, K, K)),
                r + b: TensorDecl((s.blocks, K), init="unit"), i: TensorDecl((s.blocks, K, K)), i + b: TensorDecl((s.blocks, K), init="unit"),
                lam: TensorDecl((C,), init="unit"), o: TensorDecl((s.hidden_size, C))}

    @staticmethod
    def cache_need(s: GatedLruSpec):
        return FixedState((s.conv * s.width,))             # conv - 1 rows of inputs, then S

    def __init__(self, s: GatedLruSpec, weights: dict, ctx):
        if s.width <= 0 or s.blocks <= 0 or s.width % s.blocks or s.conv < 1:
            raise ValueError(f"linear recurrent unit: {s.width} channels in {s.blocks} blocks, {s.conv} taps")
        self.spec, self.dtype = s, ctx.dtype
        y, x, conv, r, i, lam, o = s.names
        b = s.bias_suffix
        self.in_proj = Linear(torch.cat([weights[y], weights[x]], dim=0).contiguous())
        self.o_proj = Linear(weights[o])
        self.taps, self.conv_bias, self.x_bias = _f32(weights[conv], ctx), _f32(weights[conv + b], ctx), _f32(weights[x + b], ctx)
        self.gates = torch.cat([weights[r], weights[i]], dim=1).contiguous()                 # [blocks, r rows then i rows, K]
        self.biases = (_f32(weights[r + b].reshape(-1), ctx), _f32(weights[i + b].reshape(-1), ctx), _f32(weights[y + b], ctx))
        # log a = decay * r
        self.decay = _f32(-float(s.rate) * torch.nn.functional.softplus(weights[lam].double()), ctx)

    def __call__(self, h, step, cache):
        from ..csrc import ops
        s, ws, tag = self.spec, step.workspace, step.tag
        T, C = h.shape[0], s.width
        proj = self.in_proj(h, step, "lru.in")                                               # [y | x]
        u = ws.get(tag + "lru.u", (T, C), self.dtype)
        ops.short_conv(proj, C, C, self.taps, self.conv_bias, cache.state, 0, step.cu_seqlens, step.state_slots, u, act=False,
                       longest=step.max_query_len, in_bias=self.x_bias)
        gates = ops.gemm_heads(u, self.gates, ws.get(tag + "lru.gates", (T, 2 * C), torch.float32))
        out = ws.get(tag + "lru.out", (T, C), self.dtype)
        ops.linear_scan("gated_lru", proj, self.biases, cache.state, (s.conv - 1) * C, step.cu_seqlens, step.state_slots, out,
                        conv=u, gates=gates, block=C // s.blocks, decay=self.decay, longest=step.max_query_len)
        return self.o_proj(out, step, "lru.o")
