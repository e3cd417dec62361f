"""The Pafelorn decoder in the engine against the plain implementation (tests/plain_pafelorn.py).

Small configurations of their own that differ in every size, per layer too (head sizes that are no multiple of 8, value
heads wider and narrower than key heads, a layer that reads an earlier layer's keys through a wider and through a narrower
window, a layer without a feed-forward, layers in other orders) and in every constant, also values that are equal or 1 (one
head, a window of one key, one tap, one block, one bucket, no identity expert, every expert chosen and one, scales of 1).
Seeded random weights with edits where random numbers would hide a fault: routers with wide gaps, one far key made to stand
out among hundreds, sharp scores so that a window or a kept token that is one off moves the logits.
Each mechanism alone against one function of the plain implementation, with state carried across steps and slots; then
whole prompts, the stream after every layer, decoding token by token, portions down to two tokens, mixed batches with
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
import plain_pafelorn as P

DEV = "cuda:0"


def rot(dims, base, factor=None, llama=None):
    r = dict(dims=dims, base=base)
    if llama is not None:
        r["scaling"] = dict(factor=factor, low=llama[0], high=llama[1], original=llama[2])
    elif factor is not None:
        r["scaling"] = dict(factor=factor)
    return r


def diff(heads, kv, dim, vdim, scale, d, window, r, kv_from=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, diff=d, mask=dict(size=window), rot=r)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m)


def par(heads, kv, dim, vdim, scale, window, r, width, ls, rs):
    return dict(type="parallel", mixer=dict(left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window), rot=r),
                                            right=dict(width=width), left_scale=ls, right_scale=rs))


def par2(heads, kv, dim, vdim, scale, cap, window, keep, r, width, blocks, conv):
    return dict(type="parallel_2", mixer=dict(left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, softcap=cap,
                                                        mask=dict(size=window, keep_first=keep), rot=r),
                                              right=dict(width=width, blocks=blocks, conv=conv)))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, limit, experts, top, identity, sff=None, slimit=None):
    m = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top, identity=identity))
    if sff is not None:
        m["shared"] = dict(ff=sff, limit=slimit)
    return m


def model(vocab, width, eps, emb, bigram, cap, layers):
    return dict(architecture="Pafelorn", vocab=vocab, width=width, norm=dict(eps=eps), logit_softcap=cap,
                embedding=dict(scale=emb, bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2])),
                layers=[dict(mix, mlp=mlp) for mix, mlp in layers])


# A: every layer its own sizes; a reader of layer 0's keys through a WIDER window (its owner's pages must stay); all three
#    stretches of the frequency ramp occur; a layer without a feed-forward.
# B: the values that are equal or 1: one head, windows of one key and beyond the context, ONE bucket, one tap, one block,
#    no identity expert and every expert chosen, no kept token, factors and scales of 1.
# C: pages of 64 positions, rows of 64 and 128 numbers (the sizes of the tensor-core attention kernels), kept tokens beyond
#    a page's border, a reader through a narrower window, only identity experts beside one.
# D: sizes that are multiples of two at best: heads of 6 and 10, blocks of 6 channels, a width of 72, pages of 4.
CONFIGS = {
    "A": model(150, 64, 1e-5, 3.0, (37, 5, 11), 20.0,
               [(diff(4, 2, 12, 20, 0.5, 0.2, 11, rot(8, 10000.0, 3.0)), dense(96)),
                (par2(6, 3, 16, 24, 0.9, 5.0, 9, 3, rot(16, 500.0, 2.0), 36, 3, 3), moe(40, 0.6, 5, 2, 3, 24, 0.4)),
                (diff(4, 2, 12, 20, 0.8, 0.6, 30, rot(8, 10000.0, 3.0), kv_from=0), moe(24, 1.1, 6, 3, 2, 8, 0.8)),
                (par(3, 1, 24, 16, 0.7, 13, rot(24, 3000.0, 6.0, (1.0, 4.0, 64)), 40, 1.3, 0.6), None)]),
    "B": model(211, 96, 3e-6, 1.0, (1, 1, 1), 1.0,
               [(par2(1, 1, 48, 48, 1.0, 1.0, 500, 0, rot(48, 100.0, 1.0), 96, 1, 1), moe(48, 1.0, 5, 5, 0, 16, 1.0)),
                (diff(1, 1, 16, 32, 1.0, 0.5, 1, rot(16, 1234.0, 1.0)), moe(32, 0.5, 4, 1, 4)),
                (par(6, 6, 16, 16, 1.0, 1, rot(2, 50.0, 1.0, (1.0, 2.0, 16)), 16, 1.0, 1.0), dense(32))]),
    "C": model(301, 128, 1e-6, 0.7, (503, 17, 3), 12.0,
               [(par(8, 2, 64, 64, 0.2, 90, rot(32, 20000.0, 4.0, (1.0, 4.0, 512)), 160, 0.7, 1.1), moe(64, 0.9, 1, 2, 5, 96, 1.2)),
                (diff(4, 2, 64, 128, 0.15, 0.35, 150, rot(64, 9000.0, 2.0)), dense(160)),
                (par2(4, 2, 128, 96, 0.1, 30.0, 70, 66, rot(64, 800.0, 5.0), 128, 8, 4), moe(48, 0.7, 6, 2, 2, 64, 0.5)),
                (diff(4, 2, 64, 128, 0.25, 0.1, 65, rot(64, 9000.0, 2.0), kv_from=1), None)]),
    "D": model(97, 72, 2e-5, 0.5, (13, 2, 0), 7.0,
               [(par2(3, 3, 10, 6, 0.6, 3.0, 7, 5, rot(6, 30.0, 1.5), 30, 5, 5), moe(20, 0.3, 3, 2, 1, 10, 0.9)),
                (diff(6, 3, 6, 10, 1.1, 0.7, 6, rot(4, 3.0, 2.5)), dense(18)),
                (par(2, 2, 10, 14, 0.4, 5, rot(10, 77.0, 2.0, (0.5, 1.5, 12)), 18, 0.2, 2.0), moe(6, 2.0, 4, 4, 1))]),
}
PAGE = {"A": 8, "B": 16, "C": 64, "D": 4}
SEED = {"A": 61, "B": 62, "C": 63, "D": 64}
# max |engine - plain| / max |plain| over a row of logits
TOL = {"float32": 8e-5, "bfloat16": 5e-2}
CASES = [(w, d) for w in ("A", "B", "C", "D") for d in ("float32", "bfloat16")]


def attentions(cfg):
    return [l["mixer"] if l["type"] == "attention" else l["mixer"]["left"] for l in cfg["layers"]]


def edited(cfg, sharp=1.0, window=0, keep=0):
    """The same model with every attention's scale multiplied and every window and number of kept tokens moved."""
    cfg = copy.deepcopy(cfg)
    for a in attentions(cfg):
        a["scale"] *= sharp
        a["mask"]["size"] = max(1, a["mask"]["size"] + window)
        if a["mask"].get("keep_first"):
            a["mask"]["keep_first"] = max(0, a["mask"]["keep_first"] + keep)
    return cfg


def store_of(dtype):
    return "float32" if dtype == "float32" else "bfloat16"


@functools.lru_cache(maxsize=None)
def model_dir(which, store="bfloat16", sharp=1.0):
    """A folder with the configuration and seeded weights.  The float32 folders get routers with wide logits, so that the
    choice of experts changes from token to token; the bfloat16 folders corrections that lie far apart in a shuffled order: a
    choice there hardly ever rests on a close call, which a rounding could turn (the float32 tests, and the router's own
    test, hold the choice token by token).  The decays' `lam` are moved below zero so that the recurrences forget slowly."""
    from vllm_lite_b200.weights import write_model_dir
    from vllm_lite_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    cfg = edited(CONFIGS[which], sharp)
    d = H.tmp_root() / f"pafelorn_{which}_{store}_{sharp}"
    write_model_dir(d, cfg, SEED[which], std=0.12, dtype=torch.float32 if store == "float32" else torch.bfloat16)
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
        if name.endswith(".right.lam"):
            tensors[name] = (t.float() * 2.0 - 2.0).to(t.dtype)
        if name.split(".")[-1] in ("lq1", "lk1", "lq2", "lk2"):
            tensors[name] = (t.float() * 3.0).to(t.dtype)
    write_safetensors(d / "model.safetensors", tensors, metadata={"format": "pt"})
    return d


@functools.lru_cache(maxsize=None)
def plain_model(which, store, sharp=1.0):
    return P.read_model_dir(model_dir(which, store, sharp))


_plain = {}


def plain_run(which, tokens, dtype, sharp=1.0, **off):
    key = (which, store_of(dtype), sharp, tuple(sorted(off.items())), tuple(tokens))
    if key not in _plain:
        cfg, w = plain_model(which, store_of(dtype), sharp)
        logits, after = P.forward(edited(cfg, 1.0, **off), w, list(tokens))
        _plain[key] = (logits.float(), [a.float() for a in after])
    return _plain[key]


def tokens_for(which, length, seed):
    rng = np.random.default_rng(11000 + seed)
    return [int(t) for t in rng.integers(0, CONFIGS[which]["vocab"], size=length)]


def make_runner(which, dtype, num_pages, sharp=1.0, page_size=None, max_requests=4, max_context=1024, **kw):
    from vllm_lite_b200.engine import ModelRunner, load_model_dir
    _, plan, weights = load_model_dir(model_dir(which, store_of(dtype), sharp), dtype, DEV)
    return ModelRunner(plan, weights, dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32, device=DEV,
                       page_size=page_size or PAGE[which], num_pages=num_pages, max_requests=max_requests,
                       max_context=max_context, **kw)


def assert_rows(rows, which, requests, dtype, what, sharp=1.0, loosen=1.0):
    """float32: every row within the tolerance.  bfloat16: a row's rounding can change which expert a router takes where
    two choice scores lie close, and then that row and those that read it differ by far more than rounding; up to a
    twentieth of the rows (or one row) may, the mechanisms' own tests hold every row."""
    assert rows, "nothing was compared"
    errs = []
    for (rid, pos), row in rows.items():
        ref = plain_run(which, requests[rid], dtype, sharp)[0][pos]
        err = float((row - ref).abs().max()) / max(float(ref.abs().max()), 1e-12)
        if dtype == "float32":
            assert err <= loosen * TOL[dtype], f"{what} {which}/{dtype}: request {rid} position {pos}: {err:.3e}"
        errs.append(err)
    over = [e for e in errs if e > loosen * TOL[dtype]]
    assert len(over) <= max(1, len(errs) // 20), f"{what} {which}/{dtype}: {len(over)} of {len(errs)} rows, worst {max(errs):.3e}"
    errs.sort()
    worst = errs[len(errs) - 1 - len(errs) // 20]
    key = ("pafelorn " + what, which, dtype)
    H.WORST[key] = max(H.WORST.get(key, 0.0), worst)


def pages_for(which, tokens):
    return -(-tokens // PAGE[which])


# ----------------------------------------------------------------------------------------------
# without a GPU: configuration, plan, cache layout, frequencies, the plain implementation's own behaviour
# ----------------------------------------------------------------------------------------------

def test_config_reads_every_size_and_constant():
    from vllm_lite_b200.config import plan_from_config_json
    from vllm_lite_b200.parts.model import declare_model
    cfg, plan = plan_from_config_json(CONFIGS["A"])
    assert (cfg.vocab_size, cfg.hidden_size, cfg.eps, cfg.embedding_scale, cfg.bigram, cfg.logit_softcap) == (150, 64, 1e-5, 3.0, (37, 5, 11), 20.0)
    e = plan.embedding
    assert (e.kind, e.scale, e.buckets, e.mul_prev, e.mul_cur) == ("pair_embedding", 3.0, 37, 5, 11)
    assert (plan.head.kind, plan.head.softcap, plan.head.scale) == ("capped_head", 20.0, 1.0) and not plan.tie_word_embeddings
    assert all(b.kind == "post_norm" and b.residual_mult == 1.0 and b.norm1.eps == 1e-5 and not b.norm1.offset for b in plan.layers)
    b0, b1, b2, b3 = plan.layers
    m = b0.mixer
    assert (m.kind, m.num_heads, m.num_kv_heads, m.dim, m.vdim, m.scale, m.diff, m.window, m.own_kv, m.bias) == \
        ("differential_attention", 4, 2, 12, 20, 0.5, 0.2, 11, True, True)
    assert (m.position.dim, m.position.theta, m.position.interleaved, m.position.scaling.factor, m.position.scaling.original) == (8, 10000.0, False, 3.0, None)
    assert (b2.mixer.own_kv, b2.mixer.window, b2.mixer.diff) == (False, 30, 0.6) and plan.order[2].cache_of == 0 and plan.order[1].cache_of is None
    p2 = b1.mixer
    assert (p2.left_scale, p2.right_scale, len(p2.out_norms), p2.out_norm_prefixes) == (0.5, 0.5, 2, ("left.out", "right.out"))
    a = p2.left
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.v_head_dim, a.scale, a.softcap, a.window, a.keep_first, a.gate, a.bias) == \
        (6, 3, 16, 24, 0.9, 5.0, 9, 3, "g", False)
    assert a.whole_norm and a.position.interleaved and a.sink is None and a.head_temp is None
    assert (p2.right.kind, p2.right.width, p2.right.blocks, p2.right.conv, p2.right.rate) == ("gated_lru", 36, 3, 3, 8.0)
    p1 = b3.mixer
    assert (p1.left_scale, p1.right_scale, p1.out_norms, p1.right.kind, p1.right.width) == (1.3, 0.6, None, "min_gru", 40)
    s = p1.left.position.scaling
    assert (s.factor, s.low, s.high, s.original) == (6.0, 1.0, 4.0, 64.0) and p1.left.position.dim == 24
    assert (p1.left.head_temp, p1.left.sink, p1.left.bias, p1.left.out_bias, p1.left.whole_norm) == ("temp", "sink", True, True, False) and b3.ffn is None
    assert (b0.ffn.activation, b0.ffn.gated, b0.ffn.intermediate_size, b0.ffn.eps) == ("poly_norm", False, 96, 1e-5)
    f = b1.ffn
    assert (f.num_experts, f.top, f.identity, f.limit, f.alpha, f.up_shift, f.score, f.renormalize, f.scale_input) == (5, 2, 3, 0.6, 1.702, 1.0, "softmax", True, False)
    assert (f.shared.intermediate_size, f.shared.limit, f.shared_gate, f.choice_bias, f.renorm_eps) == (24, 0.4, "shared.sg", "correction", 1e-20)
    names = declare_model(plan)
    shape = lambda n: names[n].shape
    assert shape("embed") == (150, 64) and shape("bigram") == (38, 64) and shape("head") == (150, 64) and shape("final.norm") == (64,)
    assert shape("l0.mix.q") == (96, 64) and shape("l0.mix.k") == (48, 64) and shape("l0.mix.v.b") == (40,) and shape("l0.mix.o") == (64, 80)
    assert shape("l0.mix.q.norm") == (12,) and shape("l0.mix.lq2") == (12,) and shape("l0.mlp.act") == (4,) and "l0.mlp.gate" not in names
    assert shape("l1.mix.left.q.norm") == (96,) and shape("l1.mix.left.k.norm") == (48,) and shape("l1.mix.left.g") == (144, 64)
    assert shape("l1.mix.right.ra") == (3, 12, 12) and shape("l1.mix.right.ri.b") == (3, 12) and shape("l1.mix.right.conv") == (36, 3)
    assert shape("l1.mix.left.out") == (64,) and shape("l1.mlp.router") == (8, 64) and shape("l1.mlp.correction") == (8,)
    assert shape("l1.mlp.shared.sg") == (1, 64) and shape("l1.mlp.e4.gate") == (40, 64) and "l1.mlp.e5.gate" not in names
    assert shape("l2.mix.q.b") == (96,) and not any(n.startswith(("l2.mix.k", "l2.mix.v")) for n in names)
    assert shape("l3.mix.left.temp") == (3,) and shape("l3.mix.left.sink") == (3,) and shape("l3.mix.left.o.b") == (64,)
    assert shape("l3.mix.right.z") == (40, 64) and shape("l3.mix.right.x.b") == (40,) and "l3.norm2" not in names and "l3.norm2" in plan.unused_tensors


def test_config_errors_name_the_field():
    from vllm_lite_b200.config import InvalidField, MissingField, plan_from_config_json
    def bad(edit):
        c = copy.deepcopy(CONFIGS["A"])
        edit(c)
        return c
    L = lambda c, i: c["layers"][i]["mixer"]
    with pytest.raises(MissingField, match=r"layers\[0\]\.mixer\.diff"):
        plan_from_config_json(bad(lambda c: L(c, 0).pop("diff")))
    with pytest.raises(InvalidField, match=r"layers\[2\]\.type"):
        plan_from_config_json(bad(lambda c: c["layers"][2].update(type="something_else")))
    with pytest.raises(InvalidField, match=r"layers\[2\]\.mixer\.kv_from"):
        plan_from_config_json(bad(lambda c: L(c, 2).update(kv_from=1)))              # no differential attention
    with pytest.raises(InvalidField, match=r"layers\[2\]\.mixer\.kv_from"):
        plan_from_config_json(bad(lambda c: L(c, 2).update(kv_heads=4)))             # other heads than layer 0
    with pytest.raises(InvalidField, match=r"layers\[0\]\.mixer\.kv_from"):
        plan_from_config_json(bad(lambda c: L(c, 0).update(kv_from=2)))              # not an earlier layer
    with pytest.raises(InvalidField, match="router"):
        plan_from_config_json(bad(lambda c: c["layers"][1]["mlp"]["router"].update(top=9)))
    with pytest.raises(InvalidField, match="kv_heads"):
        plan_from_config_json(bad(lambda c: L(c, 1)["left"].update(kv_heads=4)))
    with pytest.raises(InvalidField, match=r"rot\.dims"):
        plan_from_config_json(bad(lambda c: L(c, 3)["left"]["rot"].update(dims=7)))
    with pytest.raises(InvalidField, match=r"rot\.scaling"):
        plan_from_config_json(bad(lambda c: L(c, 3)["left"]["rot"]["scaling"].update(high=1.0)))
    with pytest.raises(InvalidField, match="blocks"):
        plan_from_config_json(bad(lambda c: L(c, 1)["right"].update(blocks=5)))
    with pytest.raises(MissingField, match=r"layers\[1\]\.mixer\.right"):
        plan_from_config_json(bad(lambda c: L(c, 1).pop("right")))
    with pytest.raises(InvalidField, match=r"mlp\.kind"):
        plan_from_config_json(bad(lambda c: c["layers"][0]["mlp"].update(kind="other")))
    with pytest.raises(MissingField, match=r"embedding\.bigram"):
        plan_from_config_json(bad(lambda c: c["embedding"].pop("bigram")))
    for key in ("embedding", "norm", "vocab", "width"):
        with pytest.raises(MissingField, match=key):
            plan_from_config_json(bad(lambda c: c.pop(key)))


def test_what_layers_and_the_embedding_keep():
    """Pages with windows and kept tokens, states beside them, the token before; an owner keeps what its reader reaches."""
    from vllm_lite_b200.cache import CacheLayout, FixedState, PagedKV, Several
    from vllm_lite_b200.config import plan_from_config_json
    from vllm_lite_b200.parts.model import cache_needs, cache_sources
    _, plan = plan_from_config_json(CONFIGS["A"])
    needs, src = cache_needs(plan), cache_sources(plan)
    assert needs[0] == PagedKV(2, 32, window=30) and needs[2] is None and src == [None, None, 0, None, None]      # the reader's window is wider
    assert needs[1] == Several((PagedKV(3, 32, window=9, keep=3), FixedState((3 * 36,))))
    assert needs[3] == Several((PagedKV(1, 32, window=13), FixedState((40,)))) and needs[4] == FixedState((1,), "int32")
    lay = CacheLayout.from_needs(needs, src)
    assert lay.call_place[2][:3] == lay.call_place[0][:3] and not lay.call_place[2][3] and lay.call_place[4][0] == "state"
    _, plan = plan_from_config_json(CONFIGS["C"])
    assert cache_needs(plan)[1] == PagedKV(2, 128, window=150)                          # the reader's window is narrower


@pytest.mark.parametrize("r", [rot(8, 100.0), rot(32, 9000.0, 2.5), rot(24, 3000.0, 6.0, (1.0, 4.0, 64)), rot(64, 50.0, 1.0, (1.0, 2.0, 16)),
                               rot(2, 5.0, 8.0, (1.0, 4.0, 8192)), rot(16, 500000.0, 32.0, (1.0, 4.0, 8192))])
def test_frequencies_slowed_down(r):
    from vllm_lite_b200.parts.rope import inverse_frequencies, scaled_frequencies
    from vllm_lite_b200.parts.spec import RotaryScaling
    sc = r.get("scaling")
    want = np.array(P.frequencies(r))
    got = inverse_frequencies(r["dims"], r["base"]) if sc is None else scaled_frequencies(r["dims"], r["base"], RotaryScaling(**sc))
    assert got.dtype == np.float32 and np.allclose(got, want, rtol=1e-6, atol=0)


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_cache_sizing_counts_the_buffers_of_every_mixer(which):
    from vllm_lite_b200.cache.sizing import _mixer_width
    from vllm_lite_b200.config import plan_from_config_json
    for b in plan_from_config_json(CONFIGS[which])[1].layers:
        m = b.mixer
        if m.kind == "differential_attention":
            P_ = -(-max(2 * m.dim, m.vdim) // 16) * 16
            assert _mixer_width(m) >= m.num_heads * (2 * m.dim + 4 * P_ + m.vdim) + m.num_kv_heads * (2 * m.dim + m.vdim)
        else:
            a = m.left
            P_ = -(-max(a.head_dim, a.v_head_dim) // 16) * 16
            attention = (a.num_heads + a.num_kv_heads) * a.head_dim + a.num_kv_heads * a.v_head_dim + (2 + (a.gate is not None)) * a.num_heads * P_
            assert _mixer_width(a) >= attention
            assert _mixer_width(m.right) == (8 if m.right.kind == "gated_lru" else 4) * m.right.width
            assert _mixer_width(m) >= _mixer_width(a) + _mixer_width(m.right)


def test_plain_pieces_behave():
    d = lambda v: torch.tensor(v, dtype=torch.float64)
    assert P.bigram_rows([4, 2, 7], dict(buckets=10, mul_prev=3, mul_cur=5)) == [10, (12 + 10) % 10, (6 + 35) % 10]
    seen = P.visible(6, dict(size=2, keep_first=1))
    assert seen[5].tolist() == [True, False, False, False, True, True] and seen[0].tolist() == [True] + [False] * 5
    x = torch.randn(5, 2, 8, dtype=torch.float64)
    for inter in (True, False):
        y = P.rotate(x, rot(4, 100.0), inter)
        assert torch.allclose(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
        a, b = (0, 1) if inter else (0, 2)
        assert torch.allclose(y[..., a] ** 2 + y[..., b] ** 2, x[..., a] ** 2 + x[..., b] ** 2)
    w = P.softmax_rows(d([[0.0, 0.0]]), torch.tensor([[True, True]]), 0.0)
    assert torch.allclose(w, d([[1 / 3, 1 / 3]]))                                       # the sink takes a third
    assert torch.allclose(P.candidate(d([0.0, 2.0, -1.0])), d([0.5, 2.5, 1 / (1 + math.e)]))
    S = P.linear_recurrence(d([[0.5], [0.5]]), d([[1.0], [1.0]]))
    assert torch.allclose(S, d([[1.0], [1.5]]))
    c = P.causal_conv(d([[1.0], [2.0], [3.0]]), torch.tensor([[10.0, 1.0]]), torch.tensor([0.5]))
    assert torch.allclose(c, d([[1.5], [12.5], [23.5]]))                                # the last tap is the current token's
    z = d([[1.0, -2.0]])
    p = P.poly_norm(z, torch.tensor([1.0, 2.0, 3.0, 4.0]), 0.0)
    assert torch.allclose(p, z / d(2.5).sqrt() + 2 * z ** 2 / d(8.5).sqrt() + 3 * z ** 3 / d(32.5).sqrt() + 4)
    o = P.combine_maps(d([[3.0, 4.0]]), d([[1.0, 0.0]]), 0.5, 0.2, 0.0)
    assert torch.allclose(o, 0.8 * d([[2.5, 4.0]]) / d((2.5 ** 2 + 16) / 2).sqrt())
    ids, wt = P.route(torch.eye(4, dtype=torch.float64)[:1], torch.tensor([[0.0, 0, 0, 0], [2.0, 0, 0, 0], [1.0, 0, 0, 0]]),
                      torch.tensor([5.0, 0.0, 0.5]), 2)
    sc = torch.softmax(d([0.0, 2.0, 1.0]), 0)
    assert ids[0] == [0, 2] and torch.allclose(wt[0], sc[[0, 2]] / sc[[0, 2]].sum())    # the correction chooses, it does not weigh


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


def mini_step(lengths, slots, starts=None, tokens=None):
    """A step's description for parts that keep a state: request b brings lengths[b] tokens from position starts[b] on and
    owns state row slots[b]."""
    from vllm_lite_b200.parts.base import StepBatch, Workspace
    starts = starts or [0] * len(lengths)
    T = int(sum(lengths))
    req = [b for b, n in enumerate(lengths) for _ in range(n)]
    pos = [starts[b] + i for b, n in enumerate(lengths) for i in range(n)]
    return StepBatch(tokens=ints(tokens if tokens is not None else [0] * T), positions=ints(pos), req_index=ints(req),
                     cu_seqlens=ints(np.concatenate([[0], np.cumsum(lengths)])), state_slots=ints(slots), logit_rows=ints([]),
                     groups=[], entries=[], err=torch.zeros(1, dtype=torch.int32, device=DEV), workspace=Workspace(torch.device(DEV)),
                     num_tokens=T, num_entries=len(lengths), max_query_len=max(lengths))


# portions of two requests of 13 and 6 tokens: single tokens, portions of two, one request pausing
CUTS = ([1, 2], [1, 0], [2, 1], [1, 3], [8, 0])


def in_portions(n, fn, cuts=CUTS):
    """fn(live, lengths, starts) -> rows of the step, for every step of the cuts; returns every request's rows in order."""
    got, at = [[], []], [0, 0]
    for lens in cuts:
        live = [b for b in (0, 1) if lens[b]]
        out = fn(live, [lens[b] for b in live], [at[b] for b in live])
        o = 0
        for b in live:
            got[b].append(out[o:o + lens[b]].clone())
            o += lens[b]
            at[b] += lens[b]
    assert at == n
    return [torch.cat(g) for g in got]


def build_part(spec, dtype, seed, registry="MIXERS", edit=None, std=0.15):
    """(part, its tensors as the plain implementation reads them) with seeded random weights."""
    from vllm_lite_b200.parts import registry as R
    from vllm_lite_b200.parts.base import BuildContext
    from vllm_lite_b200.weights import random_tensors
    cls = getattr(R, registry).get(spec.kind)
    tensors = random_tensors(cls.declare(spec), seed, std, 0.1, dtype=dtype)
    if edit:
        edit(tensors)
    part = cls(spec, {k: v.to(DEV) for k, v in tensors.items()}, BuildContext(torch.device(DEV), dtype))
    return part, tensors


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,V,bigram,scale", [(64, 50, (37, 5, 11), 3.0), (6, 9, (1, 1, 1), 1.0), (300, 70, (13, 2, 0), 0.5),
                                              (66, 40, (1009, 2147483647, 2147483629), 0.25)])
def test_embedding_reads_the_token_before_across_portions(dtype, W, V, bigram, scale):
    """Token ids in portions and single tokens in slots that are not the requests' numbers; the table's last row for a first
    token; multipliers whose products leave 32 bits; then a slot freed, zeroed and used again."""
    from vllm_lite_b200.parts import spec as S
    from vllm_lite_b200.parts.base import CallCache
    spec = S.PairEmbeddingSpec(V, W, *bigram, scale=scale)
    part, w = build_part(spec, dtype, 7, "EMBEDDINGS", std=1.0)
    cfg = dict(embedding=dict(scale=scale, bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))))
    state = torch.zeros((4, 1), dtype=torch.int32, device=DEV)
    n, slots = [13, 6], [3, 1]
    toks = [[int(t) for t in np.random.default_rng(5 + b).integers(0, V, size=n[b])] for b in (0, 1)]

    def fn(live, lens, starts):
        ids = [t for b, s, c in zip(live, starts, lens) for t in toks[b][s:s + c]]
        step = mini_step(lens, [slots[b] for b in live], starts, ids)
        x = torch.full((len(ids), W), float("nan"), device=DEV)
        part(step, x, CallCache(state=state))
        assert int(step.err.item()) == 0
        return x

    got = in_portions(n, fn)
    for b in (0, 1):
        close(got[b], P.embedding(toks[b], w, cfg), torch.float32, f"embedding of request {b}", tol=1e-6)
        assert int(state[slots[b], 0]) == toks[b][-1]
    assert int(state[0, 0]) == 0 and int(state[2, 0]) == 0
    state[slots[0]].zero_()
    x = torch.empty((2, W), device=DEV)
    step = mini_step([2], [slots[0]], None, [1, 3])
    part(step, x, CallCache(state=state))
    close(x, P.embedding([1, 3], w, cfg), torch.float32, "a slot used again", tol=1e-6)
    step = mini_step([2], [slots[0]], [2], [V, 1])                     # an id outside the table: flagged, not read
    part(step, x, CallCache(state=state))
    assert int(step.err.item()) != 0 and float(x[0].abs().max()) == 0.0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H_,G_,M,D_,V_,rd,whole,many", [(4, 2, 2, 16, 24, 8, False, False), (3, 1, 1, 24, 16, 24, False, False), (6, 3, 1, 16, 24, 16, True, False),
                                                         (8, 2, 1, 128, 128, 64, False, True), (4, 2, 2, 64, 128, 64, False, True), (1, 1, 2, 8, 8, 2, False, False),
                                                         (40, 8, 1, 128, 96, 32, True, False), (12, 4, 1, 64, 64, 64, True, True), (2, 1, 3, 40, 64, 40, False, False)])
def test_head_work(dtype, H_, G_, M, D_, V_, rd, whole, many):
    """Biases, a norm per map of a head or over the whole projection, rotation of neighbours far out, a factor per head, and
    the padded rows of queries, keys and values; what pads them is zero, slots of nobody are left alone."""
    o, eps = ops(), 1e-5
    pos = [0, 1, 5, 63, 64, 1000, 4097] + (list(range(300)) if many else [])
    T, page = len(pos), 4
    PD = -(-max(M * D_, V_) // 16) * 16 + (16 if D_ == 24 else 0)
    Cq, Ck, Cv = H_ * M * D_, G_ * M * D_, G_ * V_
    rows = rand((T, Cq + Ck + Cv + 8), 100, dtype, 1.5)
    bias = rand((Cq + Ck + Cv,), 101, scale=0.5)
    qw, kw = (rand((n,), 102 + i) * 0.3 + 1 for i, n in enumerate((Cq, Ck) if whole else (D_, D_)))
    factor = rand((H_,), 104) + 0.2
    r = rot(rd, 777.0, 1.5)
    inv = torch.tensor(P.frequencies(r), dtype=torch.float32, device=DEV)
    pages = -(-T // page) + 2
    slots = np.random.default_rng(3).permutation(pages * page)[:T].tolist()
    kc = torch.full((pages, G_, page, PD), 9.0, dtype=dtype, device=DEV)
    vc = torch.full((pages, G_, page, PD), 9.0, dtype=dtype, device=DEV)
    q = torch.full((T, H_ * M, PD), float("nan"), dtype=dtype, device=DEV)
    e = torch.zeros(1, dtype=torch.int32, device=DEV)
    o.head_work(rows, bias, ints(pos), ints(slots), qw, kw, eps, (inv, rd), factor, q, kc, vc, H_, G_, M, D_, V_, e, whole=whole)
    assert int(e.item()) == 0
    x = rows.double().cpu()[:, :Cq + Ck + Cv] + bias.double().cpu()

    def turned(u):                                                    # u [T, n, D]: at the tokens' own positions
        out = u.clone()
        for i, f in enumerate(P.frequencies(r)):
            # the angle as the design computes it, one 32-bit product (far out a rounding of it is a visible turn)
            a = torch.tensor((np.array(pos, dtype=np.float32) * np.float32(f)).astype(np.float64))[:, None]
            c, s = torch.cos(a), torch.sin(a)
            out[..., 2 * i], out[..., 2 * i + 1] = u[..., 2 * i] * c - u[..., 2 * i + 1] * s, u[..., 2 * i + 1] * c + u[..., 2 * i] * s
        return out

    def normed(u, w, n):
        return P.rms_norm(u, w.cpu(), eps).reshape(T, n, D_) if whole else P.rms_norm(u.reshape(T, n, D_), w.cpu(), eps)

    wq = turned(normed(x[:, :Cq], qw, H_ * M)) * factor.double().cpu().repeat_interleave(M)[:, None]
    wk = turned(normed(x[:, Cq:Cq + Ck], kw, G_ * M)).reshape(T, G_, M * D_)
    wv = x[:, Cq + Ck:].reshape(T, G_, V_)
    tol = 5e-6 if dtype == torch.float32 else 1e-2
    for m in range(M):
        got = q[:, m::M]
        close(got[..., m * D_:(m + 1) * D_], wq[:, m::M], dtype, f"queries of map {m}", tol=tol)
        rest = got.clone()
        rest[..., m * D_:(m + 1) * D_] = 0
        assert float(rest.abs().max()) == 0.0
    at = torch.tensor(slots)
    kk, vv = kc[at // page, :, at % page], vc[at // page, :, at % page]
    close(kk[..., :M * D_], wk, dtype, "cached keys", tol=tol)
    close(vv[..., :V_], wv, dtype, "cached values", tol=tol)
    assert M * D_ == PD or float(kk[..., M * D_:].abs().max()) == 0.0
    assert V_ == PD or float(vv[..., V_:].abs().max()) == 0.0
    free = sorted(set(range(pages * page)) - set(slots))
    assert all(float(kc[s // page, 0, s % page, 0]) == 9.0 for s in free)
    # a token without a slot writes nothing; rows of queries alone serve a call that reads another's cache
    kc.fill_(5.0)
    o.head_work(rows, bias, ints(pos), ints([-1] * T), qw, kw, eps, (inv, rd), factor, q, kc, vc, H_, G_, M, D_, V_, e, whole=whole)
    assert bool((kc == 5.0).all())
    if not whole:
        q2 = torch.empty_like(q)
        o.head_work(rows[:, :-(-Cq // 8) * 8].contiguous(), bias, ints(pos), None, qw, kw, eps, (inv, rd), factor, q2, None, None, H_, G_, M, D_, V_, e)
        assert torch.equal(q2, q)
    o.head_work(rows, bias, ints(pos), ints([pages * page] + slots[1:]), qw, kw, eps, (inv, rd), factor, q, kc, vc, H_, G_, M, D_, V_, e, whole=whole)
    assert int(e.item()) != 0                                         # a slot beyond the pool: flagged, not written


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H_,V_,n,PD", [(4, 24, 20, 32), (1, 8, 6, 16), (6, 64, 64, 64), (5, 128, 128, 128), (3, 256, 250, 256)])
def test_difference_of_two_maps(dtype, H_, V_, n, PD):
    a = rand((7, 2 * H_, PD), 110, dtype)
    a[..., n:] = 0
    out = torch.empty((7, H_ * V_), dtype=dtype, device=DEV)
    ops().combine_maps(a, 0.83, 0.7, 1e-5, n, out)
    x = a.double().cpu()[..., :n]
    want = P.unit_rms(x[:, 0::2] - float(np.float32(0.83)) * x[:, 1::2], 1e-5) * 0.7
    got = out.view(7, H_, V_)
    close(got[..., :n], want, dtype, "combined maps", tol=3e-6 if dtype == torch.float32 else 8e-3)
    assert n == V_ or float(got[..., n:].abs().max()) == 0.0


def paged(seqs, page, G_, Dp, dtype, seed):
    """Scatter every sequence's rows [n, G, Dp] (keys, values) into shuffled pages: (k cache, v cache, block table)."""
    total = sum(-(-k.shape[0] // page) for k, _ in seqs) + 3
    perm = np.random.default_rng(seed).permutation(total).tolist()
    kc = torch.full((total, G_, page, Dp), float("nan"), dtype=dtype)
    vc = torch.full((total, G_, page, Dp), float("nan"), dtype=dtype)
    table = torch.full((len(seqs), max(-(-k.shape[0] // page) for k, _ in seqs)), -1, dtype=torch.int32)
    for b, (k, v) in enumerate(seqs):
        for blk in range(-(-k.shape[0] // page)):
            pg = perm.pop()
            table[b, blk] = pg
            n = min(page, k.shape[0] - blk * page)
            kc[pg, :, :n] = k[blk * page:blk * page + n].transpose(0, 1).to(dtype)
            vc[pg, :, :n] = v[blk * page:blk * page + n].transpose(0, 1).to(dtype)
    return kc.to(DEV), vc.to(DEV), table.to(DEV)


def give_back(table, page, lens, new, window, keep):
    """Takes the pages out of the tables that no query of the step can read, as the cache does."""
    for b, (n, c) in enumerate(zip(lens, new)):
        first = n - c - window + 1
        for blk in range(-(-keep // page), max(0, first) // page):
            table[b, blk] = -1


def plain_masked(q, k, v, scale, cap, window, keep, sink, first):
    """Rows `first` .. of a sequence: q [n, H, D], k, v [n, G, D]."""
    n, H_, _ = q.shape
    G_ = k.shape[1]
    seen = P.visible(n, dict(size=window, keep_first=keep))[first:]
    out = torch.zeros(n - first, H_, v.shape[2], dtype=torch.float64)
    for a in range(H_):
        s = q[first:, a] @ k[:, a // (H_ // G_)].t() * scale
        s = P.capped(s, cap) if cap else s
        out[:, a] = P.softmax_rows(s, seen, None if sink is None else float(sink[a])) @ v[:, a // (H_ // G_)]
    return out


def want_masked(seqs, lens, new, req, q, H_, D_, scale, cap, window, keep, sink):
    """Per request: its tokens of the step and the plain rows."""
    wants = []
    for b, (n, c) in enumerate(zip(lens, new)):
        k, v = (t.double() for t in seqs[b])
        mine = [t for t in range(len(req)) if req[t] == b]
        full = torch.zeros(n, H_, D_, dtype=torch.float64)
        full[n - c:] = q[mine].double().cpu().view(c, H_, D_)
        wants.append((mine, plain_masked(full, k, v, scale, cap, window, keep, sink, n - c)))
    return wants


def check_masked(out, wants, dtype, what, tol):
    for b, (mine, want) in enumerate(wants):
        close(out[mine].view(want.shape), want, dtype, f"{what}, request {b}", tol=tol)


def masked_case(dtype, H_, G_, D_, page, lens, new, window, keep, seed):
    seqs = [(rand((n, G_, D_), 70 + b + seed, dtype).cpu(), rand((n, G_, D_), 72 + b + seed, dtype).cpu()) for b, n in enumerate(lens)]
    kc, vc, table = paged(seqs, page, G_, D_, dtype, 5 + seed)
    give_back(table, page, lens, new, window, keep)
    req = [b for b, c in enumerate(new) for _ in range(c)]
    pos = [p for n, c in zip(lens, new) for p in range(n - c, n)]
    return seqs, kc, vc, table, req, pos, rand((len(req), H_ * D_), 74 + seed, dtype)


MASKS = [(40, 6), (17, 0), (64, 64), (1, 1), (33, 70), (200, 130), (500, 9), (64, 1)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("H_,G_,D_,page", [(4, 2, 16, 8), (6, 6, 32, 16), (8, 2, 64, 64), (3, 1, 48, 4)])
def test_window_beside_kept_tokens(dtype, window, keep, H_, G_, D_, page):
    """Portions and a single token over shuffled pages of which the unreadable ones are given back, in the kernel whose
    sums depend on positions alone; a cap and a learned sink ride along."""
    lens, new = [150, 83, 300], [61, 1, 2]
    scale = 2.0 * D_ ** -0.5
    seqs, kc, vc, table, req, pos, q = masked_case(dtype, H_, G_, D_, page, lens, new, window, keep, 0)
    out = torch.empty((len(req), H_ * D_), dtype=dtype, device=DEV)
    e = torch.zeros(1, dtype=torch.int32, device=DEV)
    sink = rand((H_,), 77)
    ops().paged_attention(q, out, kc, vc, table, ints(req), ints(pos), H_, G_, D_, scale, window, e, sinks=sink, softcap=4.0, keep=keep)
    assert int(e.item()) == 0
    wants = want_masked(seqs, lens, new, req, q, H_, D_, scale, 4.0, window, keep, sink.cpu())
    check_masked(out, wants, dtype, "kept tokens", 2e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("H_,G_,D_,page,cap", [(4, 2, 16, 8, 3.0), (8, 2, 64, 64, None), (40, 2, 32, 16, 5.0), (2, 1, 128, 16, 2.0), (9, 1, 80, 32, None)])
def test_tensor_core_kernels_keep_the_first_tokens(window, keep, H_, G_, D_, page, cap):
    """The bfloat16 kernels of a mixed step: tiles of a prompt's portion, and single tokens whose readable keys are cut into
    chunks that merge as a cluster, through scratch, or not at all."""
    dtype = torch.bfloat16
    lens, new = [300, 83, 1200, 5], [170, 1, 1, 1]
    scale = 2.0 * D_ ** -0.5
    seqs, kc, vc, table, req, pos, q = masked_case(dtype, H_, G_, D_, page, lens, new, window, keep, 3)
    T = len(req)
    e = torch.zeros(1, dtype=torch.int32, device=DEV)
    sink = rand((H_,), 78)
    opt = dict(softcap=cap, keep=keep, sinks=sink)
    tiles = torch.tensor([[0, 0, 128, 130], [0, 128, 42, 258]], dtype=torch.int32, device=DEV)
    singles = ints([170, 171, 172])
    wants = want_masked(seqs, lens, new, req, q, H_, D_, scale, cap, window, keep, sink.cpu())
    for chunk in (64, 256, 1024):
        reach = min(1200, window + keep) if keep else 1200         # kept keys: the launch counts readable keys, not positions
        out = torch.full((T, H_ * D_), float("nan"), dtype=dtype, device=DEV)
        ops().flash_prefill(q, out, kc, vc, table, tiles, H_, G_, D_, scale, window, e, tile_rows=128, **opt)
        S, na, nm = ops().decode_attention_scratch(3, H_, D_, reach, chunk)
        arrivals = torch.zeros(ops().flash_decode_arrivals(3, H_, G_), dtype=torch.int32, device=DEV)
        ops().flash_decode(q, out, kc, vc, table, ints(req), ints(pos), H_, G_, D_, scale, window, reach, torch.empty(na, device=DEV),
                           torch.empty(nm, device=DEV), e, chunk=chunk, token_index=singles, arrivals=arrivals, **opt)
        assert int(e.item()) == 0 and int(arrivals.abs().max()) == 0
        check_masked(out, wants, dtype, f"chunks of {chunk}", 1.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("H_,G_,D_,page,cap", [(4, 2, 64, 16, None), (2, 1, 128, 64, 3.0), (2, 2, 128, 16, None), (8, 2, 64, 32, 4.0)])
def test_tcgen05_prompt_kernel_keeps_the_first_tokens(window, keep, H_, G_, D_, page, cap):
    dtype = torch.bfloat16
    lens, new = [700, 300], [300, 129]
    scale = 2.0 * D_ ** -0.5
    seqs, kc, vc, table, req, pos, q = masked_case(dtype, H_, G_, D_, page, lens, new, window, keep, 9)
    e = torch.zeros(1, dtype=torch.int32, device=DEV)
    sink = rand((H_,), 79)
    tiles = torch.tensor([[0, 0, 128, 400], [0, 128, 128, 528], [0, 256, 44, 656], [1, 300, 128, 171], [1, 428, 1, 299]],
                         dtype=torch.int32, device=DEV)
    out = torch.full((len(req), H_ * D_), float("nan"), dtype=dtype, device=DEV)
    ops().flash_prefill_tc5(q, out, kc, vc, table, tiles, H_, G_, D_, scale, window, e, softcap=cap, keep=keep, sinks=sink)
    assert int(e.item()) == 0
    check_masked(out, want_masked(seqs, lens, new, req, q, H_, D_, scale, cap, window, keep, sink.cpu()), dtype, "tcgen05", 1.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H_,G_,D_,page", [(8, 2, 64, 64), (4, 4, 32, 16), (2, 1, 128, 8)])
@pytest.mark.parametrize("n,window,keep", [(700, 65, 4), (700, 64, 64), (513, 128, 1), (1300, 300, 200), (130, 40, 90)])
def test_one_key_that_stands_out_at_every_edge(dtype, H_, G_, D_, page, n, window, keep):
    """One key whose score stands out among hundreds, placed at the last kept token, the one behind it, the last key outside
    the window, the first inside, a page's border: its marker shows in the last query's output if and only if it is readable
    (as the last row of a portion and as a single token)."""
    lo = n - window
    places = {0, keep - 1, keep, lo - 1, lo, lo + 1, n - 1, min(max(page - 1, 0), n - 1), min(page, n - 1), (n // 2) // page * page}
    for far in sorted(p for p in places if 0 <= p < n):
        k, v = rand((n, G_, D_), 120, dtype, 0.05).cpu(), rand((n, G_, D_), 121, dtype, 0.05).cpu()
        k[far], v[far] = 0, 0
        k[far, :, 0], v[far, :, 1] = 6.0, 40.0
        kc, vc, table = paged([(k, v)], page, G_, D_, dtype, 7)
        e = torch.zeros(1, dtype=torch.int32, device=DEV)
        seen = far >= lo or far < keep
        for new in (1, 37, 90):
            mine = table.clone()
            give_back(mine, page, [n], [new], window, keep)
            q = rand((new, H_ * D_), 123, dtype, 0.05)
            q.view(new, H_, D_)[-1, :, 0] = 5.0
            args = (H_, G_, D_, 1.0, window, e)
            outs = [torch.full((new, H_ * D_), float("nan"), dtype=dtype, device=DEV) for _ in range(3)]
            pos = ints(range(n - new, n))
            ops().paged_attention(q, outs[0], kc, vc, mine, ints([0] * new), pos, *args, softcap=25.0, keep=keep)
            ran = [outs[0]]
            if dtype == torch.bfloat16 and new > 1:
                tiles = torch.tensor([[0, 0, new, n - new]], dtype=torch.int32, device=DEV)
                ops().flash_prefill(q, outs[1], kc, vc, mine, tiles, *args, tile_rows=128, softcap=25.0, keep=keep)
                ran.append(outs[1])
                if ops().flash_tc5_supported(dtype, D_, page):
                    ops().flash_prefill_tc5(q, outs[2], kc, vc, mine, tiles, *args, softcap=25.0, keep=keep)
                    ran.append(outs[2])
            elif dtype == torch.bfloat16:
                reach = window + keep
                S, na, nm = ops().decode_attention_scratch(1, H_, D_, reach, 128)
                arrivals = torch.zeros(ops().flash_decode_arrivals(1, H_, G_), dtype=torch.int32, device=DEV)
                ops().flash_decode(q, outs[1], kc, vc, mine, ints([0]), pos, H_, G_, D_, 1.0, window, reach, torch.empty(na, device=DEV),
                                   torch.empty(nm, device=DEV), e, chunk=128, arrivals=arrivals, softcap=25.0, keep=keep)
                ran.append(outs[1])
            assert int(e.item()) == 0
            for i, out in enumerate(ran):
                marker = out[-1].view(H_, D_)[:, 1].float()
                assert bool((marker > 30.0).all()) if seen else bool((marker.abs() < 1.0).all()), (far, new, i, seen, marker.tolist())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["min_gru", "gated_lru"])
@pytest.mark.parametrize("C,blocks", [(18, 3), (64, 1), (160, 5), (300, 2), (35, 5), (1, 1)])
def test_element_wise_recurrences(dtype, kind, C, blocks):
    """The scan alone: states carried over single tokens, short portions and portions of several stretches, in slots used in
    another order; the neighbours of its state columns are left alone."""
    o, K = ops(), C // blocks
    cuts = ([1, 2], [1, 0], [300, 1], [2, 257], [9, 0])
    n = [313, 260]
    ld = 3 * C if kind == "min_gru" else C + 5
    proj = [rand((n[b], ld), 20 + b, dtype, 1.5) for b in (0, 1)]
    u = [rand((n[b], C), 22 + b, dtype) for b in (0, 1)]
    gates = [rand((n[b], 2 * C), 24 + b) for b in (0, 1)]
    b0, b1, b2 = (rand((C,), 26 + i, scale=0.5) for i in range(3))
    decay = -8.0 * torch.nn.functional.softplus(rand((C,), 29) * 2 - 3)
    state = torch.zeros((3, 5 + C + 2), dtype=torch.float32, device=DEV)
    slots = [1, 2]

    def fn(live, lens, starts):
        step = mini_step(lens, [slots[b] for b in live], starts)
        cat = lambda xs: torch.cat([xs[b][s:s + c] for b, s, c in zip(live, starts, lens)]).contiguous()
        out = torch.full((sum(lens), C), float("nan"), dtype=dtype, device=DEV)
        kw = {} if kind == "min_gru" else dict(conv=cat(u), gates=cat(gates), block=K, decay=decay)
        o.linear_scan(kind, cat(proj), (b0, b1) if kind == "min_gru" else (b0, b1, b2), state, 5, step.cu_seqlens, step.state_slots, out,
                      longest=max(lens), **kw)
        return out

    got = in_portions(n, fn, cuts)
    d = lambda t: t.double().cpu()
    for b in (0, 1):
        x = d(proj[b])
        if kind == "min_gru":
            z = torch.sigmoid(x[:, :C] + d(b0))
            S = P.linear_recurrence(1 - z, z * P.candidate(x[:, C:2 * C] + d(b1)))
            want = S * torch.nn.functional.silu(x[:, 2 * C:])
        else:
            g = d(gates[b]).view(n[b], blocks, 2, K)
            r, i = torch.sigmoid(g[:, :, 0].reshape(n[b], C) + d(b0)), torch.sigmoid(g[:, :, 1].reshape(n[b], C) + d(b1))
            la = d(decay) * r
            S = P.linear_recurrence(torch.exp(la), torch.sqrt(-torch.expm1(2 * la)) * i * d(u[b]))
            want = S * P.gelu_tanh(x[:, :C] + d(b2))
        close(got[b], want, dtype, f"{kind} of request {b}", tol=1e-5 if dtype == torch.float32 else 8e-3)
        close(state[slots[b], 5:5 + C], S[-1], torch.float32, "state", tol=1e-5)
    assert float(state[0].abs().max()) == 0.0 and float(state[:, :5].abs().max()) == 0.0 and float(state[:, 5 + C:].abs().max()) == 0.0


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["min_gru", "gated_lru"])
@pytest.mark.parametrize("n", [64, 65, 512, 513, 1024, 2500])
def test_long_stretches_do_not_depend_on_the_number_of_blocks(kind, n):
    """A long portion alone (one cluster walks it), as a portion of a launch whose longest request is longer, and in two portions
    cut at a stretch's border: the same bits; and the plain recurrence."""
    o, C, dtype = ops(), 70, torch.bfloat16
    ld = 3 * C if kind == "min_gru" else C
    proj, u, gates = rand((n, ld), 20, dtype, 1.5), rand((n, C), 22, dtype), rand((n, 2 * C), 24)
    b0, b1, b2 = (rand((C,), 26 + i, scale=0.5) for i in range(3))
    decay = -8.0 * torch.nn.functional.softplus(rand((C,), 29) * 2 - 5)

    def run(lo, hi, state, longest):
        step = mini_step([hi - lo], [0], [lo])
        out = torch.full((hi - lo, C), float("nan"), dtype=dtype, device=DEV)
        kw = {} if kind == "min_gru" else dict(conv=u[lo:hi].contiguous(), gates=gates[lo:hi].contiguous(), block=C // 2, decay=decay)
        o.linear_scan(kind, proj[lo:hi].contiguous(), (b0, b1) if kind == "min_gru" else (b0, b1, b2), state, 0, step.cu_seqlens,
                      step.state_slots, out, longest=longest, **kw)
        return out

    fresh = lambda: torch.zeros((1, C), dtype=torch.float32, device=DEV)
    sa, sb, sc = fresh(), fresh(), fresh()
    whole = run(0, n, sa, n)
    assert torch.equal(whole, run(0, n, sb, n + 3000)) and torch.equal(sa, sb)
    cut = n // 2 // 64 * 64
    if cut:
        assert torch.equal(whole, torch.cat([run(0, cut, sc, cut), run(cut, n, sc, n - cut)])) and torch.equal(sa, sc)
    d = lambda t: t.double().cpu()
    x = d(proj)
    if kind == "min_gru":
        z = torch.sigmoid(x[:, :C] + d(b0))
        S = P.linear_recurrence(1 - z, z * P.candidate(x[:, C:2 * C] + d(b1)))
    else:
        g = d(gates).view(n, 2, 2, C // 2)
        r, i = torch.sigmoid(g[:, :, 0].reshape(n, C) + d(b0)), torch.sigmoid(g[:, :, 1].reshape(n, C) + d(b1))
        S = P.linear_recurrence(torch.exp(d(decay) * r), torch.sqrt(-torch.expm1(2 * d(decay) * r)) * i * d(u))
    close(sa[0], S[-1], torch.float32, "state", tol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,out_dtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
@pytest.mark.parametrize("C,col0", [(64, 8), (40, 0), (36, 4), (1100, 16), (7, 3)])
def test_convolution_in_portions(dtype, out_dtype, taps, C, col0):
    """Both kernels of the short convolution (16-byte accesses, and any size): biases on its rows and on its sums, an
    activation, requests in portions, single tokens and portions of several runs."""
    n, cuts = [83, 42], ([1, 2], [1, 0], [2, 1], [1, 39], [78, 0])
    ld = col0 + C + (5 if C == 7 else 8)
    x = [rand((n[b], ld), 130 + b, dtype) for b in (0, 1)]
    w, bias, ib = rand((C, taps), 132), rand((C,), 133), rand((C,), 134)
    state = torch.zeros((3, 4 + max(taps - 1, 1) * C + (-(taps - 1) * C) % 4), dtype=torch.float32, device=DEV)
    slots = [2, 0]
    for act in (False, True):
        state.zero_()

        def fn(live, lens, starts):
            step = mini_step(lens, [slots[b] for b in live], starts)
            rows = torch.cat([x[b][s:s + c] for b, s, c in zip(live, starts, lens)]).contiguous()
            out = torch.full((rows.shape[0], C), float("nan"), dtype=out_dtype, device=DEV)
            ops().short_conv(rows, col0, C, w, bias, state, 4, step.cu_seqlens, step.state_slots, out, act=act, longest=max(lens), in_bias=ib)
            return out

        got = in_portions(n, fn, cuts)
        for b in (0, 1):
            src = x[b].double().cpu()[:, col0:col0 + C] + ib.double().cpu()
            want = P.causal_conv(src, w.cpu(), bias.cpu())
            want = torch.nn.functional.silu(want) if act else want
            close(got[b], want, dtype, f"convolution of request {b}", tol=3e-6 if out_dtype == torch.float32 else 8e-3)
            if taps > 1:
                kept = state[slots[b], 4:4 + (taps - 1) * C].view(taps - 1, C)
                close(kept, src[-(taps - 1):], torch.float32, "kept inputs", tol=1e-6)
        assert float(state[1].abs().max()) == 0.0 and float(state[:, :4].abs().max()) == 0.0


@pytest.mark.gpu
@pytest.mark.parametrize("T,H_,K,N", [(512, 3, 64, 128), (700, 2, 136, 272), (1030, 5, 40, 100), (600, 1, 256, 512), (16, 4, 64, 128), (100, 4, 24, 48)])
def test_product_per_block_with_float32_sums(T, H_, K, N):
    """The gates' product: bfloat16 operands, the float32 sums as they are, few rows and many."""
    a, w = rand((T, H_ * K), 140, torch.bfloat16), rand((H_, N, K), 141, torch.bfloat16, 0.2)
    out = torch.full((T, H_ * N), float("nan"), device=DEV)
    ops().gemm_heads(a, w, out)
    want = torch.einsum("thk,hnk->thn", a.double().cpu().view(T, H_, K), w.double().cpu()).reshape(T, H_ * N)
    close(out, want, torch.float32, "product", tol=2e-6)


@pytest.mark.gpu
@pytest.mark.parametrize("window", [1, 17, 64, 200])
@pytest.mark.parametrize("H_,G_,D_,page", [(4, 2, 16, 8), (8, 2, 64, 64), (40, 2, 32, 16)])
def test_single_tokens_count_the_keys_of_a_window(window, H_, G_, D_, page):
    """The decode kernel with chunks over the readable keys instead of positions, on pages of which those behind the window are
    given back."""
    dtype, lens, new = torch.bfloat16, [300, 83, 1200, 5, 64], [1, 1, 1, 1, 1]
    scale = 2.0 * D_ ** -0.5
    seqs, kc, vc, table, req, pos, q = masked_case(dtype, H_, G_, D_, page, lens, new, window, 0, 4)
    sink = rand((H_,), 81)
    wants = want_masked(seqs, lens, new, req, q, H_, D_, scale, None, window, 0, sink.cpu())
    e = torch.zeros(1, dtype=torch.int32, device=DEV)
    for chunk in (64, 256):
        out = torch.full((5, H_ * D_), float("nan"), dtype=dtype, device=DEV)
        S, na, nm = ops().decode_attention_scratch(5, H_, D_, window, chunk)
        arrivals = torch.zeros(ops().flash_decode_arrivals(5, H_, G_), dtype=torch.int32, device=DEV)
        ops().flash_decode(q, out, kc, vc, table, ints(req), ints(pos), H_, G_, D_, scale, window, window, torch.empty(na, device=DEV),
                           torch.empty(nm, device=DEV), e, chunk=chunk, arrivals=arrivals, sinks=sink, numbered=True)
        assert int(e.item()) == 0 and int(arrivals.abs().max()) == 0
        check_masked(out, wants, dtype, f"chunks of {chunk}", 1.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,C,blocks,conv,W", [("min_gru", 40, 1, 1, 64), ("min_gru", 18, 1, 1, 72), ("min_gru", 320, 1, 1, 128), ("gated_lru", 36, 3, 3, 64),
                                                  ("gated_lru", 30, 5, 5, 72), ("gated_lru", 96, 1, 1, 96), ("gated_lru", 256, 4, 4, 128), ("gated_lru", 64, 8, 2, 64)])
def test_recurrent_mixers_in_portions_and_slots(dtype, kind, C, blocks, conv, W):
    """The whole right-hand mixers: projections with biases, (the convolution with its own state, the gates' product per
    block), the recurrence, the gate, the output; two requests in portions, then one slot freed, zeroed and used by a third."""
    from vllm_lite_b200.parts import spec as S
    from vllm_lite_b200.parts.base import CallCache
    spec = S.MinGruSpec(W, C) if kind == "min_gru" else S.GatedLruSpec(W, C, blocks, conv)
    part, tensors = build_part(spec, dtype, 61)
    need = type(part).cache_need(spec)
    state = torch.zeros((3,) + need.shape, dtype=torch.float32, device=DEV)
    n, slots = [13, 6], [2, 0]
    h = [rand((n[b], W), 62 + b, dtype) for b in (0, 1)]

    def fn(live, lens, starts):
        step = mini_step(lens, [slots[b] for b in live], starts)
        rows = torch.cat([h[b][s:s + c] for b, s, c in zip(live, starts, lens)]).contiguous()
        return part(rows, step, CallCache(state=state)).clone()

    got = in_portions(n, fn)
    plain = {"min_gru": P.min_gru, "gated_lru": P.gated_lru}[kind]
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    for b in (0, 1):
        close(got[b], plain(h[b].double().cpu(), tensors, None, None), dtype, f"{kind} of request {b}", tol=tol)
    state[slots[1]].zero_()                                           # what the cache does when it hands a slot out
    h2 = rand((150, W), 70, dtype)
    out = torch.cat([part(h2[:4].contiguous(), mini_step([4], [slots[1]]), CallCache(state=state)).clone(),
                     part(h2[4:].contiguous(), mini_step([146], [slots[1]], [4]), CallCache(state=state)).clone()])
    close(out, plain(h2.double().cpu(), tensors, None, None), dtype, "a slot used again", tol=tol)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [6, 72, 300, 2048, 5000, 9000])
@pytest.mark.parametrize("normed", [True, False])
def test_norm_after_two_mixers_that_are_normed_themselves(dtype, W, normed):
    """x += n(s1 n(a) w1 + s2 n(b) w2) w in float32 in one pass, also with a bias on the sum; without the inner norms the
    plain scaled sum."""
    w, w1, w2, bias = (rand((W,), 30 + i) * 0.3 + 1.0 for i in range(4))
    a, b = rand((7, W), 34, dtype, 2.0), rand((7, W), 35, dtype, 0.05)
    d = lambda t: t.double().cpu()
    for extra in (None, bias):
        x = rand((7, W), 36, torch.float32, 3.0)
        x0 = d(x)
        y = (0.5 * P.rms_norm(d(a), w1.cpu(), 1e-5) + 0.7 * P.rms_norm(d(b), w2.cpu(), 1e-5)) if normed else 0.5 * d(a) + 0.7 * d(b)
        y = y if extra is None else y + d(extra)
        cast = torch.empty((7, W), dtype=dtype, device=DEV)
        ops().rmsnorm_add(a, w, 1e-5, 1.0, x, cast, bias=extra, pair=(b, 0.5, 0.7, w1, w2) if normed else (b, 0.5, 0.7))
        want = x0 + P.rms_norm(y, w.cpu(), 1e-5)
        close(x, want, torch.float32, "norm of a pair", tol=3e-6)
        close(cast, want, dtype, "its rounding", tol=3e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [2, 18, 160, 1024, 3001, 5000, 12288, 20000])
def test_polynomial_of_normed_powers(dtype, n):
    """Every row length the kernel holds in registers and those it reads twice; one value that stands out, whose cube leads
    the third mean; the four numbers far apart."""
    z = rand((5, n), 40, dtype, 1.3)
    z[2, n // 2] = 30.0
    z[3] *= 1e-3
    coef = torch.tensor([0.7, -1.3, 0.9, 0.25], device=DEV)
    out = torch.empty_like(z)
    ops().poly_norm(z, coef, 1e-5, out)
    want = P.poly_norm(z.double().cpu(), coef.cpu(), 1e-5)
    for r in range(5):
        close(out[r], want[r], dtype, f"row {r}", tol=5e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,W,T", [(96, 64, 37), (18, 72, 5), (160, 128, 300)])
def test_dense_feed_forward(dtype, ff, W, T):
    from vllm_lite_b200.parts import spec as S
    spec = S.GatedMlpSpec(W, ff, activation="poly_norm", gated=False, names=("gate", "up", "down"), eps=1e-5)
    part, tensors = build_part(spec, dtype, 18, "FEED_FORWARDS")
    assert sorted(tensors) == ["act", "down", "up"]
    h = rand((T, W), 19, dtype)
    close(part(h, mini_step([T], [0])), P.dense_ff(h.double().cpu(), tensors, 1e-5), dtype, "dense feed-forward")


@pytest.mark.gpu
@pytest.mark.parametrize("E,top,identity", [(8, 2, 4), (5, 5, 0), (1, 2, 5), (6, 1, 2), (3, 4, 1), (64, 6, 16)])
def test_choice_by_softmax_score_plus_correction(E, top, identity):
    """Corrections as large as the scores, so that choice and weight fall apart; identity experts chosen like the others; the
    shared feed-forward's gate is one more row of the router."""
    o, T, K = ops(), 64, 32
    h = rand((T, K), 90)
    router = rand((E + identity + 1, K), 91, scale=0.5)
    corr = rand((E + identity,), 92, scale=0.3)
    ids = torch.empty((T, top), dtype=torch.int32, device=DEV)
    w = torch.empty((T, top), dtype=torch.float32, device=DEV)
    share = torch.empty((T,), dtype=torch.float32, device=DEV)
    logits = torch.empty((o.router_slices(K), T, E + identity + 1), dtype=torch.float32, device=DEV)
    o.moe_route(h, router, top, ids, w, logits, "softmax", True, choice_bias=corr, renorm_eps=1e-20, extra_out=share)
    want_ids, want_w = P.route(h.double().cpu(), router[:-1].cpu(), corr.cpu(), top)
    for t in range(T):
        assert ids[t].tolist() == want_ids[t], f"token {t}: {ids[t].tolist()} against {want_ids[t]}"
        close(w[t], want_w[t], torch.float32, "expert weights", tol=1e-5)
    close(share, torch.sigmoid(P.lin(router[-1:].cpu(), h.double().cpu()))[:, 0], torch.float32, "shared gate", tol=1e-6)
    if 1 < top < E + identity:
        plain_ids, _ = P.route(h.double().cpu(), router[:-1].cpu(), 0 * corr.cpu(), top)
        assert any(sorted(a) != sorted(b) for a, b in zip(plain_ids, want_ids))       # the correction is not idle


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,identity,ff,sff,W,T", [(8, 2, 4, 40, 24, 64, 37), (5, 5, 0, 24, 8, 64, 5), (1, 2, 5, 17, 30, 72, 37), (16, 4, 4, 64, 96, 128, 700),
                                                       (4, 2, 2, 9, None, 72, 1), (3, 4, 1, 6, None, 72, 20)])
def test_experts_identity_experts_and_gated_shared_expert(dtype, E, top, identity, ff, sff, W, T):
    from vllm_lite_b200.parts import spec as S
    act = dict(activation="capped_swish", alpha=1.702, up_shift=1.0, names=("gate", "up", "down"))
    shared = S.GatedMlpSpec(W, sff, limit=0.4, **act) if sff else None
    spec = S.RoutedExpertsSpec(W, ff, E, top, limit=0.7, score="softmax", renormalize=True, scale_input=False, choice_bias="correction",
                               renorm_eps=1e-20, identity=identity, shared=shared, shared_gate="shared.sg" if sff else None, **act)

    def edit(t):
        t["router"] = (t["router"].float() * 6).to(dtype)                   # wide gaps between the scores
        t["correction"] = (t["correction"].float() * 0.5).to(dtype)

    part, tensors = build_part(spec, dtype, 8, "FEED_FORWARDS", edit)
    h = rand((T, W), 9, dtype)
    got = part(h, mini_step([T], [0]))
    mlp = dict(router=dict(experts=E, top=top, identity=identity), expert=dict(limit=0.7))
    if sff:
        mlp["shared"] = dict(limit=0.4)
    h64 = h.double().cpu()
    want = P.expert_mixture(h64, tensors, mlp)
    close(got, want, dtype, "experts", tol=2e-5 if dtype == torch.float32 else 2.5e-2)
    ids, _ = P.route(h64, tensors["router"], tensors["correction"], top)
    if identity and T > 4:
        assert any(e >= E for row in ids for e in row) and any(e < E for row in ids for e in row)
    pre = P.lin(tensors["e0.gate"], h64)
    assert float(pre.max()) > 0.7 and float(pre.min()) < -0.7                         # the limits bite


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
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_stream_after_every_layer(which):
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
        close(a, b, "float32", f"stream after layer {i}", tol=2e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("which,dtype", CASES)
def test_prompt_then_token_by_token(which, dtype):
    """Most of a prompt in one step, then single tokens (replayed from a graph) across page borders and every window's and
    the kept tokens' edges; and a request fed one token at a time from its first (states start from zeros)."""
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
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_cuts_and_batches_agree_in_float32(which):
    """Beyond the rounding of the recurrences' stretches nothing depends on how a prompt was cut or on what else ran."""
    reqs, schedule = mixed_schedule(which)
    runner = make_runner(which, "float32", num_pages=4 * pages_for(which, 90), max_requests=3)
    mixed = H.run_schedule(runner, schedule)
    for rid, toks in reqs.items():
        alone = H.run_schedule(runner, [([(rid, toks, list(range(len(toks))))], [rid])])
        for (r, pos), row in mixed.items():
            if r == rid:
                close(row, alone[(r, pos)], "float32", f"{rid} position {pos}", tol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("which,off", [("A", dict(window=1)), ("A", dict(window=-1)), ("A", dict(keep=1)), ("A", dict(keep=-1)), ("C", dict(window=1)),
                                       ("C", dict(window=-1)), ("C", dict(keep=1)), ("C", dict(keep=-1)), ("D", dict(window=-1)), ("D", dict(keep=1)), ("B", dict(window=1))])
def test_edges_of_windows_and_kept_tokens_show_in_the_logits(which, off):
    """Sharp scores: windows or kept tokens one off move the logits by far more than the tolerance in the plain
    implementation, and the engine agrees with the right ones, in prompts and in decoding."""
    sharp, n = 4.0, 200
    toks = tokens_for(which, n, 33)
    right = plain_run(which, toks, "float32", sharp)[0]
    wrong = plain_run(which, toks, "float32", sharp, **off)[0]
    gap = float((wrong - right).abs().max()) / float(right.abs().max())
    assert gap > 30 * TOL["float32"], f"{off} would not show ({gap:.2e})"
    runner = make_runner(which, "float32", num_pages=pages_for(which, n) + 1, sharp=sharp)
    schedule = [([("r", toks[:100], list(range(100)))], [])] + [([("r", [toks[p]], [0])], []) for p in range(100, n)]
    assert_rows(H.run_schedule(runner, schedule), which, {"r": toks}, "float32", "edges", sharp, loosen=2.0)


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "C"])
def test_the_cache_gives_back_what_no_layer_reads(which):
    """A pool too small for the whole request serves it in portions and single tokens: pages behind every window are given
    back and used again, the kept tokens' pages and those that a reader with a wider window needs stay."""
    n = {"A": 420, "C": 620}[which]
    toks = tokens_for(which, n, 91)
    longest = max(a["mask"]["size"] for a in attentions(CONFIGS[which])) + max(a["mask"].get("keep_first", 0) for a in attentions(CONFIGS[which]))
    runner = make_runner(which, "float32", num_pages=pages_for(which, longest + 40) + 3)
    assert (pages_for(which, longest + 40) + 3) * PAGE[which] < n
    schedule, at = [], 0
    while at < n:
        c = min(1 if at > 300 and at % 3 else 30, n - at)
        schedule.append(([("r", toks[at:at + c], [0, c - 1] if c > 1 else [0])], []))
        at += c
    assert_rows(H.run_schedule(runner, schedule), which, {"r": toks}, "float32", "small pool")


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["B", "C"])
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
            assert errs[-1] <= 1e-5, errs[-3:]
        else:
            assert errs[len(errs) // 2] <= TOL[dtype] and errs[int(0.8 * len(errs))] <= 2 * TOL[dtype], errs[-5:]
        del runner


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    """300 tokens one by one after a prompt of four: recurrences, convolution, the token before and the caches carry on."""
    which, length = "D", 300
    toks = tokens_for(which, length, 31)
    runner = make_runner(which, dtype, num_pages=pages_for(which, length) + 1)
    schedule = [([("r", toks[:4], [3])], [])] + [([("r", [toks[p]], [0])], []) for p in range(4, length)]
    rows = H.run_schedule(runner, schedule)
    assert_rows(rows, which, {"r": toks}, dtype, "long decode")


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "C", "D"])
def test_greedy_generation_through_the_engine(which):
    """More prompts than the batch holds, portions of prompts beside decoding, decode steps launched ahead of the host: the
    token before must be the device's own."""
    from vllm_lite_b200 import LLMEngine
    prompts = [tokens_for(which, n, 50 + i) for i, n in enumerate([5, 17, 33, 64])]
    eng = LLMEngine(str(model_dir(which, "float32")), dtype="float32", kv_blocks=64, block_size=PAGE[which],
                    max_batch_size=3, max_num_batched_tokens=48, prefill_chunk_size=13, max_model_len=256)
    outs = eng.generate(prompts, max_tokens=20)
    for p, o in zip(prompts, outs):
        toks = list(p)
        assert len(o) == 20
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
