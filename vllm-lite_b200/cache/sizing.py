"""How many pages the cache gets when nobody says: what is left of the GPU after the weights.

The reference takes `--kv-blocks` with a default of 1,024 (crates/server/src/cli/args.rs:161-162); on
a GPU with 180 GB that is 16,384 tokens of cache beside a hundred and more GB unused.  Here an explicit
count still wins; without one the pools are sized from the free device memory: a fraction of what is
free once the weights are resident, less a reserve for the step's activations, shared out among the
paged groups by the bytes a page of each costs.  Plain arithmetic on numbers: nothing here touches
a device, the caller brings the free bytes.
"""
from __future__ import annotations

from typing import List, Optional

from .manager import CacheLayout

MIN_RESERVE = 512 << 20


def page_bytes(layout: CacheLayout, page_size: int, itemsize: int) -> List[int]:
    """Bytes of one page in every paged group: keys and values of every call of the group."""
    return [len(members) * page_size * need.bytes_per_token(itemsize)
            for need, members in zip(layout.paged_groups, layout.paged_members)]


def state_bytes(layout: CacheLayout, max_requests: int) -> int:
    sizes = {"float32": 4, "bfloat16": 2, "int32": 4}
    total = 0
    for need, members in zip(layout.state_groups, layout.state_members):
        n = sizes[need.dtype]
        for s in need.shape:
            n *= int(s)
        total += n * len(members) * max_requests
    return total


def _mixer_width(mixer) -> int:
    """Elements per token of a mixer's intermediates (float32 buffers count twice), a bound for the reserve."""
    if mixer is None:
        return 0
    if hasattr(mixer, "inner"):                                         # a mixer behind a token shift: the mixed rows
        return _mixer_width(mixer.inner) + getattr(mixer, "hidden_size", 0)
    if hasattr(mixer, "conv") and hasattr(mixer, "num_kv_heads") and hasattr(mixer, "head_dim"):
        # attention behind convolutions: the stacked projection, its convolved float32 copy, queries and context
        hd = -(-mixer.head_dim // 16) * 16
        return (mixer.num_heads + mixer.num_kv_heads) * mixer.head_dim * 3 + mixer.num_heads * (2 * hd + 1)
    if hasattr(mixer, "left") and hasattr(mixer, "right"):              # two mixers side by side, plus their sum
        return _mixer_width(mixer.left) + _mixer_width(mixer.right) + 2 * getattr(mixer.left, "hidden_size", 0)
    if hasattr(mixer, "num_kv_heads") and hasattr(mixer, "head_dim"):
        hd = max(mixer.head_dim, getattr(mixer, "v_head_dim", None) or 0)
        gate = mixer.num_heads if getattr(mixer, "gate", None) else 0  # an output gate as wide as the heads
        if getattr(mixer, "whole_norm", False) or getattr(mixer, "head_temp", None):
            gate += mixer.num_heads                                    # the head work writes its queries to rows of their own
        return (2 * mixer.num_heads + 2 * mixer.num_kv_heads + gate) * (-(-hd // 16) * 16)
    if hasattr(mixer, "diff"):
        # differential attention: the stacked product, padded query rows and outputs of both maps, the combined heads
        row = -(-max(2 * mixer.dim, mixer.vdim) // 16) * 16 + 16
        return 6 * mixer.num_heads * row + 2 * mixer.num_kv_heads * row + mixer.num_heads * mixer.vdim
    if hasattr(mixer, "width") and hasattr(mixer, "blocks"):           # linear recurrent unit: y, x, conv, float32 gates, gated
        return (2 + 1 + 4 + 1) * mixer.width
    if hasattr(mixer, "width") and not hasattr(mixer, "kv_rank"):      # minimal gated recurrence: z, x, gate, gated
        return 4 * mixer.width
    if hasattr(mixer, "kv_rank"):
        # latent attention: both latents (and the rotated key part), the queries, their absorbed form and the context
        # (heads x cached row, the row rounded up to 16), the expanded values, the output gate
        rot = getattr(mixer, "rot_dim", 0)
        step = 16 if mixer.kv_rank + rot <= 256 else 64
        row = -(-(mixer.kv_rank + rot) // step) * step
        gate = mixer.num_heads * mixer.vdim if getattr(mixer, "gate", None) else 0
        gate += mixer.num_heads if getattr(mixer, "head_gate", None) else 0
        return mixer.q_rank + mixer.kv_rank + rot + gate + 7 + mixer.num_heads * (mixer.dim + rot + 2 * row + mixer.vdim)
    if hasattr(mixer, "state") and hasattr(mixer, "norm_groups"):       # state space: projection, convolved copy, scan, gated
        inner = mixer.num_heads * mixer.vdim
        conv = inner + 2 * mixer.groups * mixer.state
        return (inner + conv + mixer.num_heads) + 2 * conv + 2 * inner + inner
    if hasattr(mixer, "gate_cap"):                                      # matrix memory
        hp, hd = mixer.num_heads * mixer.vdim, mixer.num_heads * mixer.dim
        return (2 * hd + 2 * hp + 2 * mixer.num_heads) + 2 * hp + hp
    if hasattr(mixer, "decay_rank") and not hasattr(mixer, "gate_rank"):
        # time mixing: five mixes of the input, r, k, v and the raw decay in float32, the gate, the scan's result, the gated rows
        hd = mixer.num_heads * mixer.dim
        return 5 * mixer.hidden_size + 8 * hd + hd + 2 * mixer.decay_rank + 2 * hd + hd
    if hasattr(mixer, "unit_eps") and not hasattr(mixer, "decay_rank"):
        # delta rule with one decay per head: one product (with the gate, two numbers a head and up to 7 rows of padding), its
        # convolved float32 copy, the scan's float32 result, the gated rows
        hp = mixer.num_heads * mixer.vdim
        conv = 2 * mixer.num_kv_heads * mixer.dim + hp
        # ... and, in chunks of 64 tokens, per head two matrices of 64 numbers a row of the state, one of 64 x 64, the chunk's state
        chunks = 2 * mixer.num_heads * (mixer.dim + mixer.vdim + 64 + 3 + mixer.dim * mixer.vdim // 64)
        return (conv + hp + 2 * mixer.num_heads + 7) + 2 * conv + 2 * hp + hp + chunks
    if hasattr(mixer, "decay_rank"):                                    # delta rule
        hp, hd = mixer.num_heads * mixer.vdim, mixer.num_heads * mixer.dim
        conv = 2 * mixer.num_kv_heads * mixer.dim + hp
        return (conv + mixer.num_heads) + (mixer.decay_rank + mixer.gate_rank) + (hd + hp) + 2 * conv + 2 * hp + hp
    return 0


def activation_reserve(plan, max_step_tokens: int, max_requests: int, max_context: int, itemsize: int) -> int:
    """A bound on what steps allocate beside weights and cache: the buffers of the longest step (the
    float32 stream, a layer's widest intermediates) and, for every decode graph that may be recorded
    (batch buckets up to max_requests, context bounds from 1,024 up), its own logits."""
    H, V = plan.hidden_size, plan.vocab_size
    widest, streams = 0, 1
    for block in plan.layers:
        mixer, ffn = getattr(block, "mixer", None), getattr(block, "ffn", None)
        streams = max(streams, int(getattr(block, "streams", 1) or 1))
        w = _mixer_width(mixer)
        if hasattr(ffn, "top"):
            # routed experts: every token's row `top` times (sorted copy, gate and up, activation, result), tiles padded
            w += 2 * ffn.top * (3 * ffn.intermediate_size + 2 * H)
        elif hasattr(ffn, "intermediate_size"):
            w += 3 * ffn.intermediate_size
        widest = max(widest, w)
    if any(getattr(call, "add_embedding", False) for call in getattr(plan, "order", ())):
        streams += 1                                          # the embedding's output is kept for the whole step
    per_token = 4 * H * (1 + (streams if streams > 1 else 0)) + itemsize * (widest + 4 * H)
    bounds, b = 1, 1024
    while b < max_context:
        b, bounds = b * 2, bounds + 1
    graph_logits = 2 * max_requests * V * 4 * bounds          # buckets 1, 2, 4, ... sum to under twice the largest
    return int(1.25 * per_token * max_step_tokens) + graph_logits + MIN_RESERVE


def pages_from_memory(layout: CacheLayout, page_size: int, itemsize: int, free_bytes: int, fraction: float,
                      reserve_bytes: int, max_requests: int, max_context: int,
                      max_step_tokens: Optional[int] = None) -> List[int]:
    """Pages for every paged group.  budget = free_bytes * fraction - reserve_bytes - state slots; every
    group gets the same count, except that no group gets more pages than its requests could ever hold
    at once (max_requests at max_context; a windowed group: the window plus the longest step), and
    what such a group leaves goes to the others.  Raises ValueError when not even one request of
    max_context fits."""
    if not 0.0 < fraction <= 1.0:
        raise ValueError(f"the memory fraction must lie in (0, 1], got {fraction}")
    costs = page_bytes(layout, page_size, itemsize)
    if not costs:
        return []
    budget = int(free_bytes * fraction) - int(reserve_bytes) - state_bytes(layout, max_requests)
    per_request = -(-max_context // page_size)
    caps, least = [], []
    for need in layout.paged_groups:
        most = per_request
        if need.window is not None:
            most = min(most, -(-(need.window + (max_step_tokens or max_context)) // page_size) + 1
                       + -(-(getattr(need, "keep", None) or 0) // page_size))
        if getattr(need, "chunk", None):
            most = min(most, -(-(need.chunk + (max_step_tokens or max_context)) // page_size) + 1)
        least.append(most)                                    # what one request alone may come to hold
        caps.append(max_requests * most + 1)
    counts: List[Optional[int]] = [None] * len(costs)
    while True:
        open_groups = [g for g, c in enumerate(counts) if c is None]
        if not open_groups:
            break
        left = budget - sum(costs[g] * c for g, c in enumerate(counts) if c is not None)
        share = left // sum(costs[g] for g in open_groups)
        capped = [g for g in open_groups if caps[g] <= share]
        if not capped:
            for g in open_groups:
                counts[g] = int(share)
            break
        for g in capped:
            counts[g] = caps[g]
    if any(c < l for c, l in zip(counts, least)):
        raise ValueError(f"{free_bytes / 2**30:.1f} GiB free x {fraction} less {reserve_bytes / 2**30:.1f} GiB of reserve "
                         f"holds {counts} pages; one request of {max_context} tokens needs {least}")
    return counts
