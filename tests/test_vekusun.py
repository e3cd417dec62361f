"""The Vekusun decoder in the engine against the plain implementation (tests/plain_vekusun.py).

Small configurations of their own that differ in every size, per layer too (head sizes that are no multiple of 4, value heads
wider and narrower than key heads, latent rows of 13 to 320 numbers, layers in other orders, loops over the first, the middle, the
last and all layers, one without a loop) and in every constant, also values that are equal or 1 (one head, one expert, one tap,
one pass, factors of 1).  Seeded random weights with edits where random numbers would hide a fault: routers with wide gaps, sharp
scores so that one far key stands out among hundreds, decays near 1 so that a state that is lost shows.
Each mechanism alone against one function of the plain implementation, with state carried across steps and slots; then
whole prompts, the stream after every layer run, decoding token by token, portions down to two tokens, mixed batches with
pages and slots used again, long prompts and decoding, and greedy generation through the engine's entry point, the command
line and the replay program.
"""
import copy
import functools
import json
import math

import numpy as np
import pytest
import torch

import helpers as H
import plain_vekusun as P

DEV = "cuda:0"


def delta(heads, kv, dim, vdim, conv):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv))


def one(heads, dim, vdim, q_rank, kv_rank, scale):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale))


def rot(dims, base, yarn=None):
    r = dict(dims=dims, base=base)
    if yarn is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return r


def two(heads, dim, vdim, kv_rank, scale, r):
    return dict(type="latent_attention_2", mixer=dict(heads=heads, dim=dim, rot_dim=r["dims"], vdim=vdim, kv_rank=kv_rank, scale=scale, rot=r))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def model(vocab, width, eps, mult, cap, loop, layers):
    c = dict(architecture="Vekusun", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult,
             layers=[dict(mix, mlp=mlp) for mix, mlp in layers])
    if cap is not None:
        c["logit_softcap"] = cap
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# A: every layer its own sizes, a loop over the middle, all three stretches of the frequency ramp, a layer without a feed-forward.
# B: the values that are equal or 1: one head, one pass over ALL layers, one expert, every expert chosen, one tap, factors of 1.
# C: pages of 64 positions and the sizes of the tensor-core kernels (latent rows of 128, heads of 64 and 128), a loop over the last
#    layers, no scaling of the frequencies.
# D: sizes that are multiples of two at best (the delta rule's general scan), a loop over the first layers, no cap on the logits.
# E: latent rows of 192, 256 and 320 numbers, no loop.
CONFIGS = {
    "A": model(150, 64, 1e-5, 0.4, 20.0, (1, 3, 3),
               [(delta(4, 2, 12, 20, 3), moe(40, 5, 2)), (one(3, 10, 14, 24, 18, 0.4), dense(96)),
                (two(4, 12, 6, 22, 0.3, rot(8, 100.0, (3.0, 64, 8.0, 1.0))), None), (delta(6, 6, 8, 4, 1), dense(40))]),
    "B": model(211, 96, 3e-6, 1.0, 5.0, (0, 3, 1),
               [(two(1, 16, 16, 16, 1.0, rot(16, 50.0, (1.0, 16, 2.0, 1.0))), moe(16, 1, 1)), (delta(1, 1, 16, 16, 1), moe(32, 4, 4)),
                (one(1, 16, 16, 16, 16, 1.0), dense(16))]),
    "C": model(301, 128, 1e-6, 0.7, 12.0, (2, 4, 2),
               [(delta(4, 2, 64, 64, 4), moe(64, 6, 2)), (one(8, 32, 48, 96, 128, 0.2), dense(160)),
                (two(4, 48, 32, 64, 0.12, rot(64, 9000.0)), moe(48, 3, 1)), (delta(2, 1, 128, 128, 2), None)]),
    "D": model(97, 72, 2e-5, 0.55, None, (0, 2, 4),
               [(two(3, 10, 14, 7, 0.5, rot(6, 7.0, (2.5, 10, 3.0, 0.5))), moe(20, 3, 2)), (delta(6, 3, 10, 6, 5), dense(18)),
                (one(2, 6, 10, 5, 9, 0.9), moe(6, 7, 3))]),
    "E": model(133, 80, 1e-5, 0.9, 30.0, None,
               [(one(5, 24, 8, 40, 192, 0.3), dense(24)), (two(3, 20, 12, 300, 0.25, rot(20, 500.0, (4.0, 300, 16.0, 2.0))), moe(24, 4, 2)),
                (two(6, 12, 20, 224, 0.2, rot(32, 2000.0, (8.0, 40, 4.0, 1.0))), dense(48)), (delta(2, 2, 36, 100, 3), dense(32))]),
}
PAGE = {"A": 8, "B": 16, "C": 64, "D": 4, "E": 16}
SEED = {"A": 81, "B": 82, "C": 83, "D": 84, "E": 85}
# max |engine - plain| / max |plain| over a row of logits
TOL = {"float32": 5e-5, "bfloat16": 5e-2}
NAMES = ["A", "B", "C", "D", "E"]
CASES = [(w, d) for w in NAMES for d in ("float32", "bfloat16")]


def edited(cfg, sharp=1.0):
    """The same model with every attention's scale multiplied."""
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        if "scale" in l["mixer"]:
            l["mixer"]["scale"] *= sharp
    return cfg


def store_of(dtype):
    return "float32" if dtype == "float32" else "bfloat16"


@functools.lru_cache(maxsize=None)
def model_dir(which, store="bfloat16", sharp=1.0):
    """A folder with the configuration and seeded weights.  The float32 folders get routers with wide logits, so that the
    choice of experts changes from token to token; the bfloat16 folders corrections that lie far apart in a shuffled order: a
    choice there hardly ever rests on a close call, which a rounding could turn.  The rates of the decays are moved down so that
    the states forget slowly; the sinks are as large as scores."""
    from vllm_lite_b200.weights import write_model_dir
    from vllm_lite_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    d = H.tmp_root() / f"vekusun_{which}_{store}_{sharp}"
    write_model_dir(d, edited(CONFIGS[which], sharp), SEED[which], std=0.12, dtype=torch.float32 if store == "float32" else torch.bfloat16)
    f = SafetensorsFile(d / "model.safetensors")
    tensors = {n: f.read(n).clone() for n in f.names()}
    f.close()
    for name, t in tensors.items():
        if name.endswith(".mlp.router") and store == "float32":
            tensors[name] = (t.float() * 4.0).to(t.dtype)
        if name.endswith(".mlp.correction"):
            tensors[name] = (t.float() * 0.3).to(t.dtype)
            if store != "float32":
                order = np.random.default_rng(t.numel() + len(name)).permutation(t.numel())
                tensors[name] = torch.tensor(1.5 * order, dtype=torch.float32).to(t.dtype)
        if name.endswith(".A_log"):
            tensors[name] = (t.float() - 2.5).to(t.dtype)
        if name.endswith(".sink"):
            tensors[name] = (t.float() * 10.0 + 1.0).to(t.dtype)
        if name == "loop.step":
            tensors[name] = (t.float() * 5.0).to(t.dtype)
    write_safetensors(d / "model.safetensors", tensors, metadata={"format": "pt"})
    return d


@functools.lru_cache(maxsize=None)
def plain_model(which, store, sharp=1.0):
    return P.read_model_dir(model_dir(which, store, sharp))


_plain = {}


def plain_run(which, tokens, dtype, sharp=1.0):
    key = (which, store_of(dtype), sharp, tuple(tokens))
    if key not in _plain:
        cfg, w = plain_model(which, store_of(dtype), sharp)
        logits, after = P.forward(cfg, w, list(tokens))
        _plain[key] = (logits.float(), [a.float() for a in after])
    return _plain[key]


def tokens_for(which, length, seed):
    rng = np.random.default_rng(13000 + seed)
    return [int(t) for t in rng.integers(0, CONFIGS[which]["vocab"], size=length)]


def make_runner(which, dtype, num_pages, sharp=1.0, page_size=None, max_requests=4, max_context=1024, **kw):
    from vllm_lite_b200.engine import ModelRunner, load_model_dir
    _, plan, weights = load_model_dir(model_dir(which, store_of(dtype), sharp), dtype, DEV)
    return ModelRunner(plan, weights, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32, device=DEV,
                       page_size=page_size or PAGE[which], num_pages=num_pages, max_requests=max_requests,
                       max_context=max_context, **kw)


def assert_rows(rows, which, requests, dtype, what, sharp=1.0, loosen=1.0):
    """float32: every row within the tolerance.  bfloat16: a row's rounding can change which expert a router takes where
    two choice scores lie close; up to a twentieth of the rows (or one row) may, the mechanisms' own tests hold every row."""
    assert rows, "nothing was compared"
    errs = []
    for (rid, pos), row in rows.items():
        ref = plain_run(which, requests[rid], dtype, sharp)[0][pos]
        err = float((row - ref).abs().max()) / max(float(ref.abs().max()), 1e-12)
        if dtype == "float32":
            assert err <= loosen * TOL[dtype], f"{what} {which}/{dtype}: request {rid} position {pos}: {err:.3e}"
        errs.append(err)
    over = [e for e in errs if not e <= loosen * TOL[dtype]]
    assert len(over) <= max(1, len(errs) // 20), f"{what} {which}/{dtype}: {len(over)} of {len(errs)} rows, worst {max(errs):.3e}"
    errs.sort()
    key = ("vekusun " + what, which, dtype)
    H.WORST[key] = max(H.WORST.get(key, 0.0), errs[len(errs) - 1 - len(errs) // 20])


def pages_for(which, tokens):
    return -(-tokens // PAGE[which])


# ----------------------------------------------------------------------------------------------
# without a GPU: configuration, plan, running order, cache layout, frequencies, the plain implementation's own behaviour
# ----------------------------------------------------------------------------------------------

def test_config_reads_every_size_and_constant():
    from vllm_lite_b200.config import plan_from_config_json
    from vllm_lite_b200.parts.model import declare_model
    cfg, plan = plan_from_config_json(CONFIGS["A"])
    assert (cfg.vocab_size, cfg.hidden_size, cfg.eps, cfg.residual_mult, cfg.logit_softcap, cfg.loop) == (150, 64, 1e-5, 0.4, 20.0, (1, 3, 3))
    assert (plan.head.kind, plan.head.softcap, plan.head.scale) == ("capped_head", 20.0, 1.0) and not plan.tie_word_embeddings
    assert plan.embedding.scale == 1.0
    assert all(b.kind == "shared_norm" and b.residual_mult == 0.4 and b.norm1.eps == 1e-5 and b.scales == ("ls1", "ls2") for b in plan.layers)
    b0, b1, b2, b3 = plan.layers
    m = b0.mixer
    assert (m.kind, m.num_heads, m.num_kv_heads, m.dim, m.vdim, m.conv, m.eps, m.unit_eps) == ("head_delta", 4, 2, 12, 20, 3, 1e-5, 1e-6)
    m = b1.mixer
    assert (m.kind, m.num_heads, m.dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.sink, m.rot_dim, m.position, m.window) == \
        ("latent_attention", 3, 10, 14, 24, 18, 0.4, True, 0, None, None)
    m = b2.mixer
    assert (m.kind, m.num_heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.sink, m.head_gate, m.gate) == \
        ("latent_attention", 4, 12, 8, 6, 0, 22, 0.3, False, "g", None)
    s = m.position.scaling
    assert (m.position.dim, m.position.theta, m.position.interleaved, s.factor, s.original, s.fast, s.slow) == (8, 100.0, True, 3.0, 64.0, 8.0, 1.0)
    f = b0.ffn
    assert (f.num_experts, f.top, f.intermediate_size, f.activation, f.score, f.renormalize, f.scale_input, f.choice_bias, f.groups, f.shared) == \
        (5, 2, 40, "silu", "softmax", False, False, "correction", 1, None)
    assert (b1.ffn.activation, b1.ffn.gated, b1.ffn.intermediate_size) == ("gelu", False, 96) and b2.ffn is None
    names = declare_model(plan)
    shape = lambda n: names[n].shape
    assert shape("embed") == (150, 64) and shape("head") == (150, 64) and shape("final.norm") == (64,) and shape("loop.step") == (3, 64)
    assert shape("l0.mix.q") == (24, 64) and shape("l0.mix.v") == (80, 64) and shape("l0.mix.v.conv") == (80, 3) and shape("l0.mix.g") == (80, 64)
    assert shape("l0.mix.a") == (4, 64) and shape("l0.mix.dt_bias") == (4,) and shape("l0.mix.norm") == (20,) and shape("l0.mix.o") == (64, 80)
    assert shape("l0.mlp.router") == (5, 64) and shape("l0.mlp.correction") == (5,) and shape("l0.mlp.e4.gate") == (40, 64)
    assert shape("l1.mix.dq") == (24, 64) and shape("l1.mix.uq") == (30, 24) and shape("l1.mix.dkv") == (18, 64) and shape("l1.mix.sink") == (3,)
    assert shape("l1.mlp.up") == (96, 64) and "l1.mlp.gate" not in names and shape("l1.ls1") == (64,) and shape("l1.ls2") == (64,)
    assert shape("l2.mix.q") == (80, 64) and shape("l2.mix.dkv") == (30, 64) and shape("l2.mix.dkv.norm") == (22,) and shape("l2.mix.g") == (4, 64)
    assert "l2.mix.dq" not in names and "l2.mix.dq.norm" not in names and "l2.mix.sink" not in names
    assert "l2.ls2" not in names and "l2.ls2" in plan.unused_tensors and not any(n.endswith("norm2") for n in names)
    _, bare = plan_from_config_json(CONFIGS["E"])
    assert "loop.step" not in declare_model(bare) and bare.stream_tables == ()
    assert plan_from_config_json(CONFIGS["D"])[1].head.softcap is None


def test_running_order_of_the_loop():
    from vllm_lite_b200.config import plan_from_config_json
    for which in NAMES:
        _, plan = plan_from_config_json(CONFIGS[which])
        want = P.run_order(CONFIGS[which])
        assert [c.layer for c in plan.order] == [i for i, _ in want] and all(c.cache_of is None for c in plan.order)
        for c, (_, t) in zip(plan.order, want):
            assert c.add_row == (None if t is None else ("loop.step", t)) and c.add_embedding == bool(t)
    order = plan_from_config_json(CONFIGS["A"])[1].order
    assert [c.layer for c in order] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [c.add_embedding for c in order] == [False, False, False, True, False, True, False, False]
    from vllm_lite_b200.parts.spec import LayerCall
    from dataclasses import replace
    plan = plan_from_config_json(CONFIGS["A"])[1]
    with pytest.raises(ValueError, match="stream tables"):
        replace(plan, order=(LayerCall(0, add_row=("loop.step", 3)),)).validate()


def test_config_errors_name_the_field():
    from vllm_lite_b200.config import InvalidField, MissingField, plan_from_config_json
    def bad(edit):
        c = copy.deepcopy(CONFIGS["A"])
        edit(c)
        return c
    L = lambda c, i: c["layers"][i]["mixer"]
    with pytest.raises(MissingField, match=r"layers\[0\]\.mixer\.conv"):
        plan_from_config_json(bad(lambda c: L(c, 0).pop("conv")))
    with pytest.raises(MissingField, match=r"layers\[1\]\.mixer\.q_rank"):
        plan_from_config_json(bad(lambda c: L(c, 1).pop("q_rank")))
    with pytest.raises(MissingField, match=r"layers\[2\]\.mixer\.rot"):
        plan_from_config_json(bad(lambda c: L(c, 2).pop("rot")))
    with pytest.raises(MissingField, match=r"rot\.scaling\.fast"):
        plan_from_config_json(bad(lambda c: L(c, 2)["rot"]["scaling"].pop("fast")))
    with pytest.raises(InvalidField, match=r"rot\.dims"):
        plan_from_config_json(bad(lambda c: L(c, 2)["rot"].update(dims=10)))
    with pytest.raises(InvalidField, match="kv_heads"):
        plan_from_config_json(bad(lambda c: L(c, 0).update(kv_heads=3)))
    with pytest.raises(InvalidField, match=r"layers\[2\]\.type"):
        plan_from_config_json(bad(lambda c: c["layers"][2].update(type="something_else")))
    with pytest.raises(InvalidField, match="router"):
        plan_from_config_json(bad(lambda c: c["layers"][0]["mlp"]["router"].update(top=6)))
    with pytest.raises(InvalidField, match=r"mlp\.kind"):
        plan_from_config_json(bad(lambda c: c["layers"][0]["mlp"].update(kind="other")))
    with pytest.raises(InvalidField, match="loop"):
        plan_from_config_json(bad(lambda c: c["loop"].update(stop=5)))
    with pytest.raises(InvalidField, match="loop"):
        plan_from_config_json(bad(lambda c: c["loop"].update(start=3)))
    with pytest.raises(MissingField, match=r"loop\.times"):
        plan_from_config_json(bad(lambda c: c["loop"].pop("times")))
    for key in ("residual_mult", "norm", "vocab", "width"):
        with pytest.raises(MissingField, match=key):
            plan_from_config_json(bad(lambda c: c.pop(key)))


def test_every_pass_keeps_its_own():
    """A layer inside the loop has pages or a state per pass; latent rows are stored once."""
    from vllm_lite_b200.cache import CacheLayout, FixedState
    from vllm_lite_b200.cache.spec import PagedLatent
    from vllm_lite_b200.config import plan_from_config_json
    from vllm_lite_b200.parts.model import cache_needs, cache_sources
    _, plan = plan_from_config_json(CONFIGS["A"])
    needs = cache_needs(plan)
    assert needs[0] == FixedState((2 * (48 + 80) + 4 * 12 * 20,)) and needs[7] == FixedState((0 + 6 * 8 * 4,))
    assert needs[1] == needs[3] == needs[5] == PagedLatent(32) and needs[2] == needs[4] == PagedLatent(32)
    lay = CacheLayout.from_needs(needs, cache_sources(plan))
    assert len({lay.call_place[i][:3] for i in range(1, 7)}) == 6
    assert cache_needs(plan_from_config_json(CONFIGS["E"])[1])[1] == PagedLatent(320)          # wide rows: a multiple of 64
    from vllm_lite_b200.csrc import ops
    scan = cache_needs(plan_from_config_json(CONFIGS["D"])[1])[1]
    assert scan == FixedState((4 * (60 + 36) + ops.scan_state_floats(6, 10, 6),))


@pytest.mark.parametrize("r", [rot(8, 100.0), rot(32, 9000.0, (2.5, 512, 16.0, 1.0)), rot(24, 3000.0, (6.0, 64, 4.0, 1.0)), rot(64, 50.0, (1.0, 16, 2.0, 1.0)),
                               rot(2, 5.0, (8.0, 8192, 32.0, 1.0)), rot(16, 500000.0, (32.0, 100, 1.0, 1.0)), rot(12, 7.0, (3.0, 5, 64.0, 0.25))])
def test_yarn_frequencies_and_amplitude(r):
    from vllm_lite_b200.parts.rope import RotaryTable, amplitude, inverse_frequencies, scaled_frequencies
    from vllm_lite_b200.parts.base import BuildContext
    from vllm_lite_b200.parts.spec import RotarySpec, YarnScaling
    sc = r.get("scaling")
    want = np.array(P.frequencies(r))
    got = inverse_frequencies(r["dims"], r["base"]) if sc is None else scaled_frequencies(r["dims"], r["base"], YarnScaling(**sc))
    assert got.dtype == np.float32 and np.allclose(got, want, rtol=1e-6, atol=0)
    assert math.isclose(amplitude(None if sc is None else YarnScaling(**sc)), P.magnitude(r))
    table = RotaryTable(RotarySpec(r["dims"], r["base"], scaling=None if sc is None else YarnScaling(**sc)), {}, BuildContext(torch.device("cpu"), torch.float32))
    assert table.scaled_rotary()[1:] == (r["dims"], P.magnitude(r))
    if P.magnitude(r) != 1.0:                    # a mixer that knows no amplitude must not take it silently
        with pytest.raises(NotImplementedError):
            table.fused_rotary()


def test_interleaved_pairs_reordered():
    from vllm_lite_b200.parts.latent_attention import half_order
    assert half_order(6, 8) == [0, 2, 4, 1, 3, 5, 6, 7]
    x, y = torch.randn(5, 3, 8, dtype=torch.float64), torch.randn(5, 3, 8, dtype=torch.float64)
    r = rot(6, 30.0, (2.0, 20, 4.0, 1.0))
    half = lambda v: torch.cat([v[..., :3] * c - v[..., 3:6] * s, v[..., 3:6] * c + v[..., :3] * s, v[..., 6:]], -1)
    a = torch.arange(5, dtype=torch.float64)[:, None] * torch.tensor(P.frequencies(r))
    c, s = P.magnitude(r) * torch.cos(a)[:, None], P.magnitude(r) * torch.sin(a)[:, None]
    o = half_order(6, 8)
    want = (P.rotate(x, r) * P.rotate(y, r)).sum(-1)
    assert torch.allclose((half(x[..., o]) * half(y[..., o])).sum(-1), want)


@pytest.mark.parametrize("which", NAMES)
def test_cache_sizing_counts_the_buffers_of_every_mixer(which):
    from vllm_lite_b200.cache.sizing import _mixer_width, activation_reserve
    from vllm_lite_b200.config import plan_from_config_json
    from dataclasses import replace
    _, plan = plan_from_config_json(CONFIGS[which])
    for b in plan.layers:
        m = b.mixer
        if m.kind == "head_delta":
            conv = 2 * m.num_kv_heads * m.dim + m.num_heads * m.vdim
            assert _mixer_width(m) >= 3 * conv + 4 * m.num_heads * m.vdim + 2 * m.num_heads * (m.dim + m.vdim + 64)
        else:
            row = -(-(m.kv_rank + m.rot_dim) // 16) * 16
            assert _mixer_width(m) >= m.kv_rank + m.rot_dim + m.num_heads * (m.dim + m.rot_dim + 2 * row + m.vdim) + (m.num_heads if m.head_gate else 0)
    if any(c.add_embedding for c in plan.order):
        without = replace(plan, order=tuple(replace(c, add_embedding=False) for c in plan.order))
        assert activation_reserve(plan, 512, 4, 1024, 2) > activation_reserve(without, 512, 4, 1024, 2)


def test_plain_pieces_behave():
    d = lambda v: torch.tensor(v, dtype=torch.float64)
    assert P.run_order(dict(layers=[0] * 4, loop=dict(start=1, stop=3, times=2))) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    w = P.causal_weights(d([[0.0, 9.0], [0.0, 0.0]]), d(0.0))
    assert torch.allclose(w, d([[0.5, 0.0], [1 / 3, 1 / 3]]))                            # the sink takes its part, the future is masked
    x = torch.randn(5, 2, 8, dtype=torch.float64)
    y = P.rotate(x, rot(4, 100.0, (4.0, 64, 8.0, 1.0)))
    amp = 0.1 * math.log(4.0) + 1.0
    assert torch.allclose(y[0, :, :4], amp * x[0, :, :4]) and torch.equal(y[..., 4:], x[..., 4:])
    assert torch.allclose(y[..., 2] ** 2 + y[..., 3] ** 2, amp ** 2 * (x[..., 2] ** 2 + x[..., 3] ** 2))
    assert torch.allclose(P.gelu(d([0.0, 1.0, -30.0])), d([0.0, 0.8413447460685429, 0.0]))
    assert torch.allclose(P.softplus(d([0.0, 800.0, -800.0])), d([math.log(2.0), 800.0, 0.0]))
    c = P.causal_conv(d([[1.0], [2.0], [3.0]]), torch.tensor([[10.0, 1.0]]))
    assert torch.allclose(c, d([[1.0], [12.0], [23.0]]))                                 # the last tap is the current token's
    q = k = d([[[1.0, 0.0]], [[1.0, 0.0]]])
    o = P.delta_steps(q, k, d([[[4.0]], [[6.0]]]), d([[1.0], [0.5]]), d([[0.9], [0.5]]))
    assert torch.allclose(o, d([[[4.0]], [[2.0 + 0.5 * (6.0 - 2.0)]]]))                  # decayed, corrected, read after the write
    ids, wt = P.route(torch.eye(4, dtype=torch.float64)[:1], torch.tensor([[0.0, 0, 0, 0], [2.0, 0, 0, 0], [1.0, 0, 0, 0]]),
                      torch.tensor([5.0, 0.0, 0.5]), 2)
    sc = torch.softmax(d([0.0, 2.0, 1.0]), 0)
    assert ids[0] == [0, 2] and torch.allclose(wt[0], sc[[0, 2]])                        # the correction chooses, nothing is renormalised


# ----------------------------------------------------------------------------------------------
# each mechanism alone, against one function of the plain implementation
# ----------------------------------------------------------------------------------------------

def ops():
    from vllm_lite_b200.csrc import ops as o
    return o


def rand(shape, seed, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * scale).to(dtype).to(DEV)


def close(got, want, dtype, what, tol=None):
    tol = tol or (2e-5 if dtype in (torch.float32, "float32") else 2.5e-2)
    err = float((got.double().cpu() - want.double().cpu()).abs().max()) / max(float(want.abs().max()), 1e-12)
    assert err <= tol, f"{what} ({dtype}): {err:.3e}"


def ints(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def build_part(spec, dtype, seed, family="MIXERS", edit=None):
    """(the part with seeded weights, those weights on the CPU)."""
    from vllm_lite_b200.parts import registry
    from vllm_lite_b200.parts.base import BuildContext
    from vllm_lite_b200.weights.random_init import random_tensors
    cls = getattr(registry, family).get(spec.kind)
    tensors = random_tensors(cls.declare(spec), seed, std=0.2, dtype=dtype)
    if edit is not None:
        edit(tensors)
    return cls(spec, {k: v.to(DEV) for k, v in tensors.items()}, BuildContext(torch.device(DEV), dtype)), tensors


class Pages:
    """A paged latent cache for parts under test: pages handed out in a shuffled order, NaN in every slot not yet written."""

    def __init__(self, width, page, requests, longest, dtype, seed=3):
        self.page, self.blocks = page, -(-longest // page)
        n = requests * self.blocks + 2
        self.cache = torch.full((n, 1, page, width), float("nan"), dtype=dtype, device=DEV)
        self.table = torch.tensor(np.random.default_rng(seed).permutation(n)[:requests * self.blocks].reshape(requests, self.blocks), dtype=torch.int32)

    def call(self):
        from vllm_lite_b200.parts.base import CallCache
        return CallCache(group=0, k=self.cache, v=self.cache)


def step_of(live, lengths, starts, slots=None, pages=None):
    """A step's description: request live[i] brings lengths[i] tokens from position starts[i] on, owns state row slots[live[i]] and
    row live[i] of the pages' table."""
    from vllm_lite_b200.parts.base import QUERY_TILE, GroupView, StepBatch, Workspace
    T = int(sum(lengths))
    req = [i for i, n in enumerate(lengths) for _ in range(n)]
    pos = [s + i for s, n in zip(starts, lengths) for i in range(n)]
    groups, tiles, single, t0 = [], [], [], 0
    if pages is not None:
        table = pages.table[live]
        at = [int(table[r, p // pages.page]) * pages.page + p % pages.page for r, p in zip(req, pos)]
        groups = [GroupView(page_size=pages.page, block_table=table.to(DEV).contiguous(), slots=ints(at), max_context=max(pos) + 1)]
    for i, (n, s) in enumerate(zip(lengths, starts)):
        if n == 1:
            single.append(t0)
        for lo in range(0, n if n > 1 else 0, QUERY_TILE):
            tiles.append([i, t0 + lo, min(QUERY_TILE, n - lo), s + lo])
        t0 += n
    return StepBatch(tokens=ints([0] * T), positions=ints(pos), req_index=ints(req),
                     cu_seqlens=ints(np.concatenate([[0], np.cumsum(lengths)])), state_slots=ints([slots[b] for b in live] if slots else live),
                     logit_rows=ints([]), groups=groups, entries=[], err=torch.zeros(1, dtype=torch.int32, device=DEV),
                     workspace=Workspace(torch.device(DEV)), num_tokens=T, num_entries=len(lengths), max_query_len=max(lengths),
                     query_tiles=ints(np.array(tiles).reshape(-1)).view(-1, 4) if tiles else None,
                     single_tokens=ints(single) if single and tiles else None,
                     single_context=max([s + 1 for s, n in zip(starts, lengths) if n == 1], default=0))


def in_portions(part, h, cuts, dtype, slots=None, pages=None, state=None):
    """The rows of every request (h: one tensor a request), fed through the part in the steps of `cuts` (tokens a request, 0: it
    pauses)."""
    from vllm_lite_b200.parts.base import CallCache
    got, at = [[] for _ in h], [0] * len(h)
    for lens in cuts:
        live = [b for b in range(len(h)) if lens[b]]
        step = step_of(live, [lens[b] for b in live], [at[b] for b in live], slots, pages)
        rows = torch.cat([h[b][at[b]:at[b] + lens[b]] for b in live]).contiguous()
        out = part(rows, step, pages.call() if pages is not None else CallCache(state=state)).clone()
        assert int(step.err.item()) == 0
        o = 0
        for b in live:
            got[b].append(out[o:o + lens[b]])
            o += lens[b]
            at[b] += lens[b]
    assert at == [x.shape[0] for x in h]
    return [torch.cat(g) for g in got]


CUTS = ([1, 2], [1, 0], [2, 1], [14, 3], [15, 0], [16, 64], [64, 1], [65, 63], [1, 130], [130, 0], [1, 1])
TOTAL = [sum(c[b] for c in CUTS) for b in (0, 1)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,dim,vdim,conv,W", [(4, 2, 12, 20, 3, 64), (1, 1, 16, 16, 1, 32), (6, 3, 64, 64, 4, 128), (3, 3, 128, 128, 2, 96), (2, 1, 36, 100, 3, 80),
                                                      (4, 1, 128, 64, 4, 64), (2, 2, 4, 128, 5, 48), (6, 3, 10, 6, 5, 72), (2, 1, 160, 40, 3, 64), (3, 1, 20, 7, 2, 40)])
def test_delta_rule_in_portions_and_slots(dtype, heads, kv, dim, vdim, conv, W):
    """The whole mixer (one product, convolution, unit vectors, decay, recurrence, gated norm, output) for two requests in
    portions on both sides of every border (chunks of 64, portions of 16), single tokens between; then one slot freed, zeroed and used
    by a third request.  Slow decays: a state that is lost or written twice shows for the rest of the sequence."""
    from vllm_lite_b200.parts import spec as S
    spec = S.HeadDeltaSpec(W, heads, kv, dim, vdim, conv, 1e-5)

    def slow(t):
        t["A_log"] = (t["A_log"].float() - 3.0).to(dtype)

    part, tensors = build_part(spec, dtype, 61, edit=slow)
    need = type(part).cache_need(spec)
    state = torch.zeros((3,) + need.shape, dtype=torch.float32, device=DEV)
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim)
    h = [rand((TOTAL[b], W), 62 + b, dtype) for b in (0, 1)]
    got = in_portions(part, h, CUTS, dtype, slots=[2, 0], state=state)
    tol = 3e-5 if dtype == torch.float32 else 2.5e-2
    for b in (0, 1):
        close(got[b], P.delta(h[b].double().cpu(), tensors, m, 1e-5), dtype, f"delta rule of request {b}", tol=tol)
    assert float(state[1].abs().max()) == 0.0
    state[0].zero_()                                                  # what the cache does when it hands a slot out
    h2 = [rand((150, W), 70, dtype)]
    got = in_portions(part, h2, ([3], [146], [1]), dtype, slots=[0], state=state)
    close(got[0], P.delta(h2[0].double().cpu(), tensors, m, 1e-5), dtype, "a slot used again", tol=tol)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_rule_with_strong_and_uneven_decays(dtype):
    """Decays from nearly 1 to e^-50 a token, within one chunk: running sums of their logarithms reach hundreds while single
    differences stay small."""
    from vllm_lite_b200.parts import spec as S
    spec = S.HeadDeltaSpec(64, 4, 2, 32, 32, 2, 1e-5)

    def uneven(t):
        t["A_log"] = torch.tensor([2.5, 1.0, -1.0, -4.0]).to(dtype)
        t["a"] = (t["a"].float() * 4).to(dtype)

    part, tensors = build_part(spec, dtype, 71, edit=uneven)
    state = torch.zeros((1,) + type(part).cache_need(spec).shape, dtype=torch.float32, device=DEV)
    h = [rand((300, 64), 72, dtype)]
    m = dict(heads=4, kv_heads=2, dim=32, vdim=32)
    g = P.head_decay(P.lin(tensors["a"], h[0].double().cpu()), tensors["A_log"], tensors["dt_bias"])
    assert float(g.min()) < 1e-15 and float(g.max()) > 0.99
    got = in_portions(part, h, ([200], [1], [99]), dtype, slots=[0], state=state)
    close(got[0], P.delta(h[0].double().cpu(), tensors, m, 1e-5), dtype, "uneven decays", tol=3e-5 if dtype == torch.float32 else 2.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_rule_of_many_unequal_requests(dtype):
    """Forty requests of 1 to 200 tokens in one step: every chunk finds its request and its state."""
    from vllm_lite_b200.parts import spec as S
    spec = S.HeadDeltaSpec(48, 2, 1, 24, 40, 3, 1e-5)
    part, tensors = build_part(spec, dtype, 73)
    lens = [1, 15, 16, 17, 63, 64, 65, 200] * 5
    state = torch.zeros((41,) + type(part).cache_need(spec).shape, dtype=torch.float32, device=DEV)
    slots = [int(s) for s in np.random.default_rng(5).permutation(41)[:40]]
    h = [rand((n, 48), 100 + i, dtype) for i, n in enumerate(lens)]
    got = in_portions(part, h, (lens,), dtype, slots=slots, state=state)
    m = dict(heads=2, kv_heads=1, dim=24, vdim=40)
    for b in range(40):
        close(got[b], P.delta(h[b].double().cpu(), tensors, m, 1e-5), dtype, f"request {b} of {lens[b]}", tol=3e-5 if dtype == torch.float32 else 2.5e-2)


LATENT = [("one", 3, 10, 14, 24, 18, None, 8), ("one", 8, 32, 48, 96, 128, None, 64), ("one", 1, 16, 16, 16, 16, None, 16), ("one", 5, 24, 8, 40, 192, None, 16),
          ("one", 16, 20, 12, 33, 250, None, 64),
          ("two", 4, 12, 6, 0, 22, rot(8, 100.0, (3.0, 64, 8.0, 1.0)), 8), ("two", 4, 48, 32, 0, 64, rot(64, 9000.0), 64),
          ("two", 3, 10, 14, 0, 7, rot(6, 7.0, (2.5, 10, 3.0, 0.5)), 4), ("two", 1, 16, 16, 0, 16, rot(16, 50.0, (1.0, 16, 2.0, 1.0)), 16),
          ("two", 6, 12, 20, 0, 224, rot(32, 2000.0, (8.0, 40, 4.0, 1.0)), 64), ("two", 3, 20, 12, 0, 300, rot(20, 500.0, (4.0, 300, 16.0, 2.0)), 16)]


def score_scale(spread, dim, q_rank, kv_rank, r, W):
    """The scale that gives scores of about this standard deviation, for inputs of variance 1 and weights of 0.2."""
    var = dim * 0.2 ** 4 * (q_rank or W) * kv_rank
    if r is not None:
        var += r["dims"] * (0.2 ** 2 * W * P.magnitude(r) ** 2) ** 2
    return spread / math.sqrt(var)


def latent_part(kind, heads, dim, vdim, q_rank, kv_rank, r, W, dtype, scale, seed, edit=None):
    from vllm_lite_b200.config.vekusun import VekusunLayer, _mixer, _rotation
    m = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, scale=scale)
    if kind == "one":
        m["q_rank"] = q_rank
        spec = _mixer(VekusunLayer("latent_attention", m, None), W, 1e-5)
    else:
        spec = _mixer(VekusunLayer("latent_attention_2", dict(m, rot_dim=r["dims"], rot=_rotation(r, r["dims"], "rot")), None), W, 1e-5)
        m.update(rot_dim=r["dims"], rot=r)
    part, tensors = build_part(spec, dtype, seed, edit=edit)
    plain = {"one": P.sink_attention, "two": P.rotated_attention}[kind]
    return part, tensors, lambda h: plain(h.double().cpu(), tensors, m, 1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,heads,dim,vdim,q_rank,kv_rank,r,page", LATENT)
def test_latent_attention_in_portions(dtype, kind, heads, dim, vdim, q_rank, kv_rank, r, page):
    """Whole mixers over shuffled pages, portions and single tokens mixed; scores sharp enough that for most queries one key, as
    often as not hundreds of positions back, takes most of the weight; sinks from nothing to most of the denominator."""
    W = 64
    spread = 6.0 if dtype == torch.float32 else 3.0            # bfloat16 rounds scores in proportion to their size

    def sinks(t):
        if "sink" in t:
            t["sink"] = torch.linspace(-2.0, 6.0, heads).to(dtype)

    part, tensors, plain = latent_part(kind, heads, dim, vdim, q_rank, kv_rank, r, W, dtype,
                                       score_scale(spread, dim, q_rank, kv_rank, r, W), 81, sinks)
    pages = Pages(part.rank, page, 2, max(TOTAL), dtype)
    h = [rand((TOTAL[b], W), 82 + b, dtype) for b in (0, 1)]
    got = in_portions(part, h, CUTS, dtype, pages=pages)
    for b in (0, 1):
        close(got[b], plain(h[b]), dtype, f"{kind} of request {b}", tol=4e-5 if dtype == torch.float32 else 6e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("q_rank,kv_rank,rot_dim,dims,heads,dim", [(2048, 64, 0, 0, 0, 0), (1024, 512, 64, 64, 0, 0), (72, 40, 24, 16, 0, 0), (0, 96, 32, 32, 5, 24),
                                                                   (0, 200, 16, 16, 3, 8), (0, 24, 40, 16, 2, 16), (0, 18, 6, 4, 3, 10)])
def test_norm_rotation_and_cache_row_of_a_token(dtype, q_rank, kv_rank, rot_dim, dims, heads, dim):
    """Both forms of the kernel (eight numbers a thread, one): the query latent or the finished query heads before the key and value
    latent, the rotated key part behind it (only its first features turned), sine and cosine with a factor, zeros behind."""
    pos, page, amp = [0, 1, 7, 130, 1000], 4, 1.25
    T, kv_col = len(pos), q_rank or heads * (dim + rot_dim)
    width = -(-(kv_rank + rot_dim) // 16) * 16 + 16
    ld = -(-(kv_col + kv_rank + rot_dim + 3) // 8) * 8
    proj = rand((T, ld), 100, dtype, 1.5)
    wq, wkv = rand((max(q_rank, 1),), 101) + 1, rand((kv_rank,), 102) + 1
    r = rot(dims, 300.0) if dims else None
    inv = torch.tensor(P.frequencies(r), dtype=torch.float32, device=DEV) if dims else None
    cache = torch.full((2, 1, page, width), 9.0, dtype=dtype, device=DEV)
    slots = [6, 1, 4, -1, 7]
    cq = torch.empty((T, q_rank), dtype=dtype, device=DEV) if q_rank else None
    e = torch.zeros(1, dtype=torch.int32, device=DEV)
    p64 = proj.double().cpu()
    ops().latent_norm_write(proj, q_rank, kv_rank, wq if q_rank else None, wkv, 1e-5, cq, ints(slots), cache, e, rot_dim=rot_dim,
                            rotary=(inv, dims, amp) if dims else None, positions=ints(pos), kv_col=kv_col,
                            q_heads=(dim, dim + rot_dim, heads) if heads else None)
    assert int(e.item()) == 0

    def turned(x):                                  # pairs i, i + dims / 2
        a = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor(P.frequencies(r))
        c, s, h = (amp * torch.cos(a)).view(T, *[1] * (x.dim() - 2), -1), (amp * torch.sin(a)).view(T, *[1] * (x.dim() - 2), -1), dims // 2
        return torch.cat([x[..., :h] * c - x[..., h:dims] * s, x[..., h:dims] * c + x[..., :h] * s, x[..., dims:]], -1)

    tol = 2e-5 if dtype == torch.float32 else 1e-2
    if q_rank:
        close(cq, P.rms_norm(p64[:, :q_rank], wq.cpu(), 1e-5), dtype, "query latent", tol=tol)
    if heads:
        q = p64[:, :kv_col].reshape(T, heads, dim + rot_dim)
        want = torch.cat([q[..., :dim], turned(q[..., dim:])], -1).reshape(T, kv_col)
        close(proj[:, :kv_col], want, dtype, "query heads", tol=10 * tol)
    want = P.rms_norm(p64[:, kv_col:kv_col + kv_rank], wkv.cpu(), 1e-5)
    key = p64[:, kv_col + kv_rank:kv_col + kv_rank + rot_dim]
    for t, s in enumerate(slots):
        if s < 0:
            continue
        row = cache[s // page, 0, s % page]
        close(row[:kv_rank], want[t], dtype, "cached latent", tol=tol)
        if rot_dim:
            close(row[kv_rank:kv_rank + rot_dim], turned(key)[t], dtype, "cached key part", tol=10 * tol)
        assert float(row[kv_rank + rot_dim:].abs().max()) == 0.0
    assert float(cache[0, 0, 3, 0]) == 9.0                           # slot 3 belongs to nobody


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [0, 1, 3, 5, 6, 9, 10])
def test_one_far_key_among_hundreds(dtype, case):
    """Every key but one the same: with another token in that one place the outputs of queries hundreds of positions on are
    others, and the engine's are the right ones, in a long portion and in single tokens, at the first position and at pages' borders."""
    kind, heads, dim, vdim, q_rank, kv_rank, r, page = LATENT[case]
    W, n = 64, 340
    part, tensors, plain = latent_part(kind, heads, dim, vdim, q_rank, kv_rank, r, W, dtype,
                                       score_scale(4.0 if dtype == torch.float32 else 2.5, dim, q_rank, kv_rank, r, W), 91)
    base = rand((n, W), 92, torch.float32)
    for far in (0, page - 1, page, 64, 129):
        h = base.clone()
        h[far] = 3.0 * rand((W,), 93)
        h = h.to(dtype)
        without = h.clone()
        without[far] = base[(far + 7) % n].to(dtype)
        want, other = plain(h), plain(without)
        moved = (want - other).abs().amax(-1)[200:]
        assert float(moved.max()) > 0.01 * float(want.abs().max())
        pages = Pages(part.rank, page, 1, n, dtype, seed=far)
        got = in_portions(part, [h], ([200], [100], [1], [39]), dtype, pages=pages)
        close(got[0], want, dtype, f"far key {far}", tol=4e-5 if dtype == torch.float32 else 6e-2)
        if dtype == torch.float32:
            assert float((got[0].double().cpu() - other).abs().max()) > 100 * float((got[0].double().cpu() - want).abs().max())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hd", [128, 192, 256, 320, 576])
@pytest.mark.parametrize("sink", [False, True])
def test_attention_kernels_on_wide_shared_rows(dtype, hd, sink):
    """Keys and values as one plane of pages, every kernel that takes the width: a prompt's portion of several tiles and single
    tokens, one key far back made to take nearly all of the weight; NaN behind the last key."""
    o, heads, page, n, new = ops(), 5, 64, 460, 200
    if dtype == torch.bfloat16 and hd > 256:
        pytest.skip("the tensor-core kernels end at 256")
    c = rand((n, hd), 7, dtype, 0.5)
    q = rand((new, heads * hd), 8, dtype, 0.3)
    far = 70
    q.view(new, heads, hd)[:, 2] = (c[far].float() * 2.0).to(dtype)
    scale = 2.0 / math.sqrt(hd)
    sinks = torch.linspace(-1.0, 3.0, heads, device=DEV) if sink else None
    pages = Pages(hd, page, 1, n, dtype)
    for i in range(n):
        pages.cache[int(pages.table[0, i // page]), 0, i % page] = c[i]
    s = torch.einsum("thd,jd->thj", q.double().cpu().view(new, heads, hd), c.double().cpu()) * scale
    i, j = torch.arange(n - new, n)[:, None], torch.arange(n)[None]
    s = s.masked_fill((j > i)[:, None], -math.inf)
    z = torch.exp(s - 50.0)
    den = z.sum(-1, keepdim=True) + (torch.exp(sinks.double().cpu() - 50.0)[None, :, None] if sink else 0.0)
    want = torch.einsum("thj,jd->thd", z / den, c.double().cpu()).reshape(new, heads * hd)
    assert float((z / den)[:, 2, far].min()) > 0.5
    table, err = pages.table.to(DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    pos, req = ints(range(n - new, n)), ints([0] * new)
    tiles = ints([0, 0, 128, n - new, 0, 128, new - 128, n - new + 128]).view(2, 4)
    args = (heads, 1, hd, scale, None)
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    out = torch.full((new, heads * hd), float("nan"), dtype=dtype, device=DEV)
    o.paged_attention(q, out, pages.cache, pages.cache, table, req, pos, *args, err, sinks=sinks)
    close(out, want, dtype, "a token and head a block", tol)
    if dtype == torch.bfloat16:
        for fn in (lambda out: o.flash_prefill_tc5(q, out, pages.cache, pages.cache, table, tiles, *args, err, sinks=sinks),
                   lambda out: o.flash_prefill(q, out, pages.cache, pages.cache, table, tiles, *args, err, tile_rows=128, sinks=sinks)):
            out = torch.full((new, heads * hd), float("nan"), dtype=dtype, device=DEV)
            fn(out)
            close(out, want, dtype, "prompt tiles", tol)
        S, na, nm = o.decode_attention_scratch(new, heads, hd, n, 256)
        out = torch.full((new, heads * hd), float("nan"), dtype=dtype, device=DEV)
        o.flash_decode(q, out, pages.cache, pages.cache, table, req, pos, *args, n, torch.empty(na, device=DEV), torch.empty(nm, device=DEV), err,
                       chunk=256, sinks=sinks)
        close(out, want, dtype, "single tokens", tol)
    assert int(err.item()) == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [6, 72, 300, 2048, 5000, 9000])
@pytest.mark.parametrize("parts", ["a", "b", "ab", "none"])
@pytest.mark.parametrize("around", [True, False])
def test_stream_sum_and_norm(dtype, W, parts, around):
    """x <- (base) + m (s1 a + s2 b) + rows + vector and its norm in one pass, for every row and for picked rows (x then stays)."""
    from vllm_lite_b200.parts.base import StreamSum
    a, b = rand((7, W), 34, dtype, 2.0), rand((7, W), 35, dtype, 0.5)
    s1, s2, w, vec = (rand((W,), 30 + i) * 0.3 + 1.0 for i in range(4))
    base, rows = rand((7, W), 40, torch.float32, 3.0), rand((7, W), 41)
    total = StreamSum(a=a if "a" in parts else None, a_scale=s1, b=b if "b" in parts else None, b_scale=s2 if around else None, mult=0.37,
                      base=base if around else None, rows=rows if around else None, vector=vec if around else None)
    x = rand((7, W), 36, torch.float32, 3.0)
    d = lambda t: t.double().cpu()
    want = d(base) if around else d(x)
    if "a" in parts:
        want = want + 0.37 * d(a) * d(s1)
    if "b" in parts:
        want = want + 0.37 * d(b) * (d(s2) if around else 1.0)
    if around:
        want = want + d(rows) + d(vec)
    normed = P.rms_norm(want, w.cpu(), 1e-5)
    pick = ints([5, 0, 5])
    before = x.clone()
    out = torch.empty((3, W), dtype=dtype, device=DEV)
    ops().stream_norm(x, total, w, 1e-5, out, rows=pick)
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    close(out, normed[[5, 0, 5]], dtype, "norm of picked rows", tol)
    assert torch.equal(x, before)
    y, out = x.clone(), torch.empty((7, W), dtype=dtype, device=DEV)
    ops().stream_norm(y, total, w, 1e-5, out)
    close(y, want, torch.float32, "the stream", 2e-6)
    close(out, normed, dtype, "its norm", tol)
    ops().stream_norm(x, total)
    assert torch.equal(x, y)                                          # without a norm: the same stream


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sums_that_wait_for_the_next_norm(dtype):
    """A model of blocks of several kinds: what a shared-norm block leaves, and what is added between calls, reaches blocks
    that take it and blocks that do not (post-norm), and the last norm."""
    from vllm_lite_b200.parts import spec as S
    from vllm_lite_b200.parts.model import CausalLM, declare_model
    from vllm_lite_b200.parts.base import BuildContext
    from vllm_lite_b200.weights.random_init import random_tensors
    W, V = 48, 50
    norm = S.NormSpec(W, 1e-5, tensor="")
    mix = lambda: S.HeadDeltaSpec(W, 2, 1, 8, 8, 2, 1e-5)
    ff = S.GatedMlpSpec(W, 32, activation="gelu", gated=False, names=("gate", "up", "down"))
    names = ("norm1", "mix.", "norm2", "mlp.")
    shared = S.BlockSpec(mix(), ff, norm, norm, kind="shared_norm", residual_mult=0.6, names=names, scales=("ls1", "ls2"))
    bare = S.BlockSpec(mix(), ff, norm, norm, kind="shared_norm", names=names)
    post = S.BlockSpec(mix(), ff, norm, norm, kind="post_norm", residual_mult=0.5, names=names)
    order = (S.LayerCall(0), S.LayerCall(1, add_embedding=True), S.LayerCall(2, add_row=("steps", 1)), S.LayerCall(1, add_row=("steps", 0)),
             S.LayerCall(0, add_embedding=True, add_row=("steps", 2)))
    plan = S.ModelPlan("x", V, W, (shared, post, bare), order, norm, False, 64, layer_prefix="l{}.", embed_prefix="", final_norm_prefix="final",
                       head_prefix="", embedding=S.EmbeddingSpec(V, W, tensor="embed"), head=S.HeadSpec(V, W, tensor="head"),
                       stream_tables=(("steps", 3),)).validate()
    t = random_tensors(declare_model(plan), 3, std=0.3, dtype=dtype)
    model = CausalLM(plan, {k: v.to(DEV) for k, v in t.items()}, BuildContext(torch.device(DEV), dtype))
    from vllm_lite_b200.parts.base import CallCache
    from vllm_lite_b200.parts.model import cache_needs
    T = 9
    step = step_of([0], [T], [0])
    toks = [3, 1, 4, 1, 5, 9, 2, 6, 5]
    step.tokens, step.logit_rows = ints(toks), ints([8, 0, 4])
    new = lambda: [CallCache(state=torch.zeros((1,) + n.shape, device=DEV)) for n in cache_needs(plan)]
    seen = []
    watched = model.forward(step, new(), watch=lambda i, x: seen.append(x.double().cpu().clone())).clone()
    logits = model.forward(step, new()).clone()
    w = {k: v.double() for k, v in t.items()}
    first = w["embed"][toks]
    m = dict(heads=2, kv_heads=1, dim=8, vdim=8)

    def block(x, i):
        lw = P.sub(w, f"l{i}.")
        run = lambda h: (P.delta(h, P.sub(lw, "mix."), m, 1e-5), P.dense_ff(h, P.sub(lw, "mlp.")))
        if i == 1:
            x = x + 0.5 * P.rms_norm(run(x)[0], lw["norm1"], 1e-5)
            return x + 0.5 * P.rms_norm(run(x)[1], lw["norm2"], 1e-5)
        y, z = run(P.rms_norm(x, lw["norm1"], 1e-5))
        return x + 0.6 * (y * lw["ls1"] + z * lw["ls2"]) if i == 0 else x + y + z

    x = first
    for n, call in enumerate(order):
        if call.add_embedding:
            x = x + first
        if call.add_row is not None:
            x = x + w["steps"][call.add_row[1]]
        x = block(x, call.layer)
        close(seen[n], x, dtype, f"stream after call {n}", tol=2e-5 if dtype == torch.float32 else 3e-2)
    want = P.lin(w["head"], P.rms_norm(x, w["final"], 1e-5))[[8, 0, 4]]
    close(logits, want, dtype, "logits", tol=2e-5 if dtype == torch.float32 else 3e-2)
    close(watched, logits, dtype, "watched", tol=1e-6 if dtype == torch.float32 else 1e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H_,K,N,extra", [(5, 3, 24, 20, 8), (16, 6, 128, 80, 0), (100, 4, 64, 128, 24), (700, 2, 136, 272, 16), (530, 5, 256, 128, 0), (33, 3, 10, 7, 5)])
def test_product_per_head_with_a_gate_per_head(dtype, T, H_, K, N, extra):
    """Rows wider than the heads (the columns behind them are not read), a sigmoid per head and row on the sums."""
    a, w = rand((T, H_ * K + extra), 140, dtype), rand((H_, N, K), 141, dtype, 0.2)
    gate = rand((T, H_ + 13), 142, dtype, 2.0)
    if extra:
        a[:, H_ * K:] = float("nan")
    d = lambda t: t.double().cpu()
    sums = torch.einsum("thk,hnk->thn", d(a)[:, :H_ * K].reshape(T, H_, K), d(w))
    for g, want in ((None, sums), (gate, sums * torch.sigmoid(d(gate)[:, 4:4 + H_])[..., None])):
        out = torch.full((T, H_ * N), float("nan"), dtype=dtype, device=DEV)
        ops().gemm_heads(a, w, out, **({} if g is None else dict(gate=g, gate_col=4)))
        close(out, want.reshape(T, H_ * N), dtype, "per-head product", tol=3e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,W,T", [(96, 64, 37), (18, 72, 5), (160, 128, 300), (7, 40, 3)])
def test_dense_feed_forward_with_the_erf_gelu(dtype, ff, W, T):
    from vllm_lite_b200.parts import spec as S
    spec = S.GatedMlpSpec(W, ff, activation="gelu", gated=False, names=("gate", "up", "down"))
    part, tensors = build_part(spec, dtype, 18, "FEED_FORWARDS")
    assert sorted(tensors) == ["down", "up"]
    h = rand((T, W), 19, dtype)
    close(part(h, step_of([0], [T], [0])), P.dense_ff(h.double().cpu(), tensors), dtype, "dense feed-forward")
    z = torch.linspace(-9.0, 9.0, 4001, device=DEV).to(dtype)
    out = ops().unary_act(z, torch.empty_like(z), "gelu")
    want = P.gelu(z.double().cpu())
    assert torch.allclose(out.double().cpu(), want, rtol=3e-5 if dtype == torch.float32 else 5e-3, atol=3e-7)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,ff,W,T", [(8, 2, 40, 64, 37), (5, 5, 24, 64, 5), (1, 1, 17, 72, 37), (16, 4, 64, 128, 700), (7, 3, 6, 72, 20), (4, 1, 9, 72, 1)])
def test_experts_by_score_plus_correction_weighted_by_the_score(dtype, E, top, ff, W, T):
    from vllm_lite_b200.parts import spec as S
    spec = S.RoutedExpertsSpec(W, ff, E, top, activation="silu", score="softmax", renormalize=False, scale_input=False, choice_bias="correction")

    def edit(t):
        t["router"] = (t["router"].float() * 6).to(dtype)                   # wide gaps between the scores
        t["correction"] = (t["correction"].float() * 0.5).to(dtype)

    part, tensors = build_part(spec, dtype, 8, "FEED_FORWARDS", edit)
    h = rand((T, W), 9, dtype)
    want = P.expert_mixture(h.double().cpu(), tensors, dict(router=dict(experts=E, top=top)))
    close(part(h, step_of([0], [T], [0])), want, dtype, "experts", tol=2e-5 if dtype == torch.float32 else 2.5e-2)
    ids, wt = P.route(h.double().cpu(), tensors["router"], tensors["correction"], top)
    if 1 < top < E:
        plain_ids, _ = P.route(h.double().cpu(), tensors["router"], 0 * tensors["correction"].float(), top)
        assert any(sorted(a) != sorted(b) for a, b in zip(plain_ids, ids))              # the correction is not idle
        assert min(float(w.sum()) for w in wt) < 0.9                                    # renormalising would show


# ----------------------------------------------------------------------------------------------
# the model in the engine
# ----------------------------------------------------------------------------------------------

@pytest.mark.gpu
@pytest.mark.parametrize("which,dtype", CASES)
def test_whole_prompts(which, dtype):
    reqs = {f"r{i}": tokens_for(which, n, i) for i, n in enumerate([1, 2, 37, 230])}
    runner = make_runner(which, dtype, num_pages=pages_for(which, 230) + 1)
    rows = {}
    for rid, toks in reqs.items():
        rows.update(H.run_schedule(runner, [([(rid, toks, list(range(len(toks))))], [rid])]))
    assert_rows(rows, which, reqs, dtype, "whole")


@pytest.mark.gpu
@pytest.mark.parametrize("which", NAMES)
def test_stream_after_every_layer_run(which):
    from vllm_lite_b200.engine import StepEntry
    toks = tokens_for(which, 100, 5)
    runner = make_runner(which, "float32", num_pages=pages_for(which, 128))
    seen = []
    batch = runner.prepare([StepEntry("a", toks, [])])
    runner.model.forward(batch, runner.storage.call_caches, watch=lambda i, x: seen.append(x.clone().cpu()))
    runner.finish(batch)
    runner.check_device_errors()
    want = plain_run(which, toks, "float32")[1]
    assert len(seen) == len(want)
    for i, (a, b) in enumerate(zip(seen, want)):
        close(a, b, "float32", f"stream after run {i}", tol=2e-5)


def without_sinks(P_, cfg, w):
    return cfg, {k: (torch.full_like(t, -1e4) if k.endswith(".sink") else t) for k, t in w.items()}


def one_row_for_all_passes(P_, cfg, w):
    return cfg, dict(w, **{"loop.step": w["loop.step"][:1].expand_as(w["loop.step"])})


def no_feed_forward_factor(P_, cfg, w):
    return cfg, {k: (torch.ones_like(t) if k.endswith(".ls2") else t) for k, t in w.items()}


def plain_frequencies(P_, cfg, w):
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        l["mixer"].get("rot", {}).pop("scaling", None)
    return cfg, w


def one_pass_less(P_, cfg, w):
    cfg = copy.deepcopy(cfg)
    cfg["loop"]["times"] -= 1
    return cfg, w


@pytest.mark.parametrize("which,wrong", [("A", without_sinks), ("C", without_sinks), ("E", without_sinks), ("A", one_row_for_all_passes), ("C", one_row_for_all_passes),
                                         ("D", one_row_for_all_passes), ("A", no_feed_forward_factor), ("A", plain_frequencies), ("D", plain_frequencies),
                                         ("E", plain_frequencies), ("A", one_pass_less), ("D", one_pass_less)])
def test_a_left_out_mechanism_shows_in_the_logits(which, wrong):
    """In the plain implementation, on the CPU: what the engine's tests compare against moves by far more than their tolerance
    when a mechanism is left out."""
    cfg, w = plain_model(which, "float32")
    toks = tokens_for(which, 60, 33)
    right = P.forward(cfg, w, toks)[0]
    other = P.forward(*wrong(P, cfg, w), toks)[0]
    gap = float((other - right).abs().max()) / float(right.abs().max())
    assert gap > 20 * TOL["float32"], f"{wrong.__name__} would not show ({gap:.2e})"


@pytest.mark.gpu
@pytest.mark.parametrize("which,dtype", CASES)
def test_prompt_then_token_by_token(which, dtype):
    """Most of a prompt in one step, then single tokens (replayed from a graph) across page borders; and a request fed one token
    at a time from its first (states start from zeros)."""
    n, cut = 180, 60
    toks, first = tokens_for(which, n, 11), tokens_for(which, 12, 12)
    runner = make_runner(which, dtype, num_pages=pages_for(which, n) + pages_for(which, 12) + 1)
    schedule = [([("r", toks[:cut], [0, cut - 1])], [])] + [([("r", [toks[p]], [0])], []) for p in range(cut, n)]
    schedule += [([("s", [first[p]], [0])], []) for p in range(12)]
    rows = H.run_schedule(runner, schedule)
    assert_rows(rows, which, {"r": toks, "s": first}, dtype, "decode")


@pytest.mark.gpu
@pytest.mark.parametrize("which,dtype", CASES)
def test_portions_of_changing_size(which, dtype):
    toks = tokens_for(which, 235, 21)
    runner = make_runner(which, dtype, num_pages=pages_for(which, 235) + 1)
    sizes, schedule, at = [2, 37, 3, 2, 64, 1, 5, 33, 2, 22, 62, 2], [], 0
    for n in sizes:
        schedule.append(([("r", toks[at:at + n], list(range(n)))], []))
        at += n
    assert at == 235
    rows = H.run_schedule(runner, schedule)
    assert_rows(rows, which, {"r": toks}, dtype, "portions")


def mixed_schedule(which):
    """Up to three live requests in three state slots: portions beside single tokens, requests that pause, end and are
    replaced, so that pages and slots change hands."""
    reqs = {k: tokens_for(which, n, 260 + i) for i, (k, n) in enumerate([("a", 90), ("b", 41), ("c", 7), ("d", 66), ("e", 30)])}
    fed = {k: 0 for k in reqs}
    plan = [[("a", 30), ("b", 2)], [("a", 1), ("b", 17), ("c", 3)], [("a", 29), ("c", 1)], [("b", 1), ("c", 3)],
            [("a", 2), ("b", 21), ("d", 40)], [("a", 28), ("d", 1)], [("d", 2), ("e", 9)], [("d", 23), ("e", 1)], [("e", 20)]]
    schedule = []
    for step in plan:
        entries, end = [], []
        for k, n in step:
            lo = fed[k]
            entries.append((k, reqs[k][lo:lo + n], sorted({0, n - 1})))
            fed[k] += n
            if fed[k] == len(reqs[k]):
                end.append(k)
        schedule.append((entries, end))
    assert all(fed[k] == len(v) for k, v in reqs.items())
    return reqs, schedule


@pytest.mark.gpu
@pytest.mark.parametrize("which,dtype", CASES)
@pytest.mark.parametrize("native", [True, False])
def test_mixed_batches_with_pages_and_slots_used_again(which, dtype, native):
    reqs, schedule = mixed_schedule(which)
    runner = make_runner(which, dtype, num_pages=pages_for(which, 90) + pages_for(which, 66) + pages_for(which, 41) + 1, max_requests=3,
                         native_host=native)
    rows = H.run_schedule(runner, schedule)
    assert_rows(rows, which, reqs, dtype, "mixed")
    assert runner.cache.slots.free_count == 3 and all(p.held_count == 0 for p in runner.cache.pools)


@pytest.mark.gpu
@pytest.mark.parametrize("which", NAMES)
def test_cuts_and_batches_agree_in_float32(which):
    """Beyond the rounding of the delta rule's chunks nothing depends on how a prompt was cut or on what else ran."""
    reqs, schedule = mixed_schedule(which)
    runner = make_runner(which, "float32", num_pages=4 * pages_for(which, 90), max_requests=3)
    mixed = H.run_schedule(runner, schedule)
    for rid, toks in reqs.items():
        alone = H.run_schedule(runner, [([(rid, toks, list(range(len(toks))))], [rid])])
        for (r, pos), row in mixed.items():
            if r == rid:
                close(row, alone[(r, pos)], "float32", f"{rid} position {pos}", tol=2e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "C", "E"])
def test_sharp_scores_in_prompts_and_decoding(which):
    """Scores several times as sharp: most weight on single keys, far ones among them, in a prompt and in decoding."""
    n, sharp = 200, 6.0
    toks = tokens_for(which, n, 34)
    runner = make_runner(which, "float32", num_pages=pages_for(which, n) + 1, sharp=sharp)
    schedule = [([("r", toks[:100], list(range(100)))], [])] + [([("r", [toks[p]], [0])], []) for p in range(100, n)]
    assert_rows(H.run_schedule(runner, schedule), which, {"r": toks}, "float32", "sharp", sharp, loosen=2.0)


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["B", "C", "E"])
def test_long_prompt_whole_against_portions(which):
    """A prompt of 2,300 tokens in one step (products, experts and attention of many rows run on their kernels for long
    steps) against the same prompt in portions of a few hundred tokens and of two: they agree to rounding."""
    from vllm_lite_b200.engine import ModelRunner, load_model_dir
    n = 2300
    toks = tokens_for(which, n, 71)
    want = sorted(set(range(0, n, 97)) | set(range(n - 8, n)))
    for dtype in ("bfloat16", "float32"):
        _, plan, weights = load_model_dir(model_dir(which, store_of(dtype)), dtype, DEV)
        runner = ModelRunner(plan, weights, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32, device=DEV,
                             page_size=PAGE[which], num_pages=pages_for(which, n) + 2, max_requests=2, max_context=4096)
        whole = H.run_schedule(runner, [([("w", toks, want)], ["w"])])
        cuts, schedule, at = [300, 411, 2, 600, 87, 900], [], 0
        for c in cuts:
            schedule.append(([("p", toks[at:at + c], [p - at for p in want if at <= p < at + c])], []))
            at += c
        assert at == n
        parts = H.run_schedule(runner, schedule)
        errs = sorted(float((whole[("w", p)] - parts[("p", p)]).abs().max()) / max(float(parts[("p", p)].abs().max()), 1e-12) for p in want)
        if dtype == "float32":
            assert errs[-1] <= 2e-5, errs[-3:]
        else:
            assert errs[len(errs) // 2] <= TOL[dtype] and errs[int(0.8 * len(errs))] <= 2 * TOL[dtype], errs[-5:]
        del runner


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "D"])
def test_long_decoding(dtype, which):
    """300 tokens one by one after a prompt of four: states, convolutions and caches of every pass carry on."""
    length = 300
    toks = tokens_for(which, length, 31)
    runner = make_runner(which, dtype, num_pages=pages_for(which, length) + 1)
    schedule = [([("r", toks[:4], [3])], [])] + [([("r", [toks[p]], [0])], []) for p in range(4, length)]
    rows = H.run_schedule(runner, schedule)
    assert_rows(rows, which, {"r": toks}, dtype, "long decode")


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "C", "D", "E"])
def test_greedy_generation_through_the_engine(which):
    """More prompts than the batch holds, portions of prompts beside decoding, decode steps launched ahead of the host."""
    from vllm_lite_b200 import LLMEngine
    prompts = [tokens_for(which, n, 50 + i) for i, n in enumerate([5, 17, 33, 64])]
    eng = LLMEngine(str(model_dir(which, "float32")), dtype="float32", kv_blocks=64, block_size=PAGE[which],
                    max_batch_size=3, max_num_batched_tokens=48, prefill_chunk_size=13, max_model_len=256)
    outs = eng.generate(prompts, max_tokens=16)
    for p, o in zip(prompts, outs):
        toks = list(p)
        assert len(o) == 16
        for t in o:
            row = plain_run(which, toks, "float32")[0][-1]
            assert int(row.argmax()) == t or float(row.max() - row[t]) < 1e-4 * float(row.abs().max())
            toks.append(t)
    assert eng.stats()["finished"] == len(prompts)


@pytest.mark.gpu
def test_greedy_generation_bfloat16_with_the_cache_sized_from_memory():
    from vllm_lite_b200 import LLMEngine
    which = "C"
    prompts = [tokens_for(which, n, 80 + i) for i, n in enumerate([9, 70])]
    eng = LLMEngine(str(model_dir(which, "bfloat16")), dtype="bfloat16", kv_blocks=None, block_size=PAGE[which], max_batch_size=4,
                    max_model_len=256)
    outs = eng.generate(prompts, max_tokens=10)
    far = 0
    for p, o in zip(prompts, outs):
        toks = list(p)
        assert len(o) == 10
        for t in o:
            row = plain_run(which, toks, "bfloat16")[0][-1]
            far += float(row.max() - row[t]) > 2 * TOL["bfloat16"] * float(row.abs().max())
            toks.append(t)
    assert far <= 2


@pytest.mark.gpu
def test_command_line_and_replay_program(tmp_path):
    """The command line writes a folder from config.json and generates from it (greedy, float32: the plain implementation's
    tokens); bin/trace_run replays steps on the folder: a portion, then a portion beside another request's, then one token."""
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(CONFIGS["D"]))
    folder = tmp_path / "model"
    run = lambda *a, **k: subprocess.run([sys.executable, *a], capture_output=True, text=True, cwd=root, timeout=900, **k)
    made = run("-m", "vllm_lite_b200", "init", "--config", str(cfg), "--out", str(folder), "--seed", "5", "--std", "0.08")
    assert made.returncode == 0, made.stderr[-2000:]
    prompt = tokens_for("D", 14, 77)
    out = run("-m", "vllm_lite_b200", "--model", str(folder), "--dtype", "float32", "--kv-blocks", "32", "--max-tokens", "6",
              "--prompt-ids", ",".join(map(str, prompt)), "--log-level", "warn")
    assert out.returncode == 0, out.stderr[-2000:]
    got = [int(t) for t in out.stdout.strip().split(",")]
    pc, pw = P.read_model_dir(folder)
    toks = list(prompt)
    for t in got:
        row = P.forward(pc, pw, toks)[0][-1]
        assert int(row.argmax()) == t or float(row.max() - row[t]) < 1e-4 * float(row.abs().max())
        toks.append(t)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompt[:9], "want": [8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": prompt[9:], "want": [0, 4]}, {"id": "b", "tokens": [3, 1], "want": []}],
              "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [4], "want": [0]}], "end": ["b"]}]
    outdir = tmp_path / "logits"
    rep = run(str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(outdir),
              "--max-tokens", "64", "--page-size", "8", input="".join(json.dumps(x) + "\n" for x in steps))
    assert rep.returncode == 0, rep.stderr[-2000:]
    assert [l for l in rep.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = P.forward(pc, pw, prompt)[0].float()
    rows = np.fromfile(outdir / "1.f32", dtype="<f4").reshape(2, CONFIGS["D"]["vocab"])
    for row, pos in zip(rows, (9, 13)):
        assert float(np.abs(row - ref[pos].numpy()).max()) <= TOL["float32"] * float(ref[pos].abs().max())
    last = np.fromfile(outdir / "2.f32", dtype="<f4")
    refb = P.forward(pc, pw, [3, 1, 4])[0].float()[2].numpy()
    assert float(np.abs(last - refb).max()) <= TOL["float32"] * float(np.abs(refb).max())
