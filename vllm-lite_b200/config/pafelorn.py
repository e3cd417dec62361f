"""Configuration of the Pafelorn decoder and its plan of parts.

config.json: `architecture` (a string), `vocab`, `width`, `embedding` {"scale", "bigram": {"buckets", "mul_prev", "mul_cur"}},
`norm.eps`, `logit_softcap` and `layers`, one object per layer:

    {"type": "attention",
     "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "mask", "rot", "kv_from"?}, "mlp": ...}
    {"type": "parallel",
     "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"}, "right": {"width"},
               "left_scale", "right_scale"}, "mlp": ...}
    {"type": "parallel_2",
     "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask", "rot"},
               "right": {"width", "blocks", "conv"}}, "mlp": ...}
    "mask": {"size", "keep_first"?}
    "rot": {"dims", "base", "scaling"?: {"factor"} | {"factor", "low", "high", "original"}}
    "mlp": null | {"kind": "dense", "ff"}
               | {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top", "identity"?},
                  "shared"?: {"ff", "limit"}}

Every size and every constant the file gives is read from it.  What the design fixes stands in `pafelorn_plan` as arguments
of the parts: a second embedding hashed from the token before and this one; blocks that norm their sub-layers' outputs (plain
RMS norms); differential attention (biases on q, k and v, a norm per map, rotate-half, `kv_from`: the keys and values of an
earlier layer); beside each other an attention with biases, head norms, an interleaved rotation, a factor per head and a
learned sink and a minimal gated recurrence; or an attention with a norm over the whole projection,
capped scores, kept first tokens and an output gate and a gated linear recurrent unit behind a convolution, each normed
before half their sum; a dense feed-forward with a polynomial of normed powers, or experts with a capped swish chosen by
softmax score plus a correction, identity experts among them, weights renormalised, and a gated shared expert.  Tensor names
are flat: `embed`, `bigram`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.<t>`, `l<i>.mlp.<t>`, `final.norm`, `head`.
`max_position_embeddings` is optional (an engine bound on a request's length, not part of the design).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..parts.spec import (AttentionSpec, BlockSpec, CappedHeadSpec, DifferentialAttentionSpec, GatedLruSpec, GatedMlpSpec,
                          LayerCall, MinGruSpec, ModelPlan, NormSpec, PairEmbeddingSpec, ParallelMixerSpec, RotaryScaling,
                          RotarySpec, RoutedExpertsSpec)
from .errors import ConfigError, InvalidField, MissingField
from .kikepel import _field, _pos_int
from .registry import register_architecture

ARCHITECTURE = "Pafelorn"
MIXER_TYPES = ("attention", "parallel", "parallel_2")
DEFAULT_MAX_POSITIONS = 32768

# what the design fixes
EXPERT_ACTIVATION, EXPERT_ALPHA, EXPERT_UP_SHIFT = "capped_swish", 1.702, 1.0
RENORM_EPS = 1e-20
LRU_RATE = 8.0
NORMED_PAIR_SCALE = 0.5            # two mixers that are normed one by one count half each


def _number(d, key, where):
    return float(_field(d, key, where))


def _positive(d, key, where):
    v = _number(d, key, where)
    if not v > 0:
        raise InvalidField(f"{where}.{key}" if where else key, f"must be positive, got {v}")
    return v


def _count(d, key, where, default=None):
    """A non-negative integer; absent (or null): `default`, when one is given."""
    if d.get(key) is None and default is not None:
        return default
    v = _field(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise InvalidField(f"{where}.{key}", f"expected a non-negative integer, got {v!r}")
    return v


def _attention(m, where):
    """What every attention of the design has: heads, sizes, scale, mask, rotation."""
    a = {k: _pos_int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    if a["heads"] % a["kv_heads"]:
        raise InvalidField(f"{where}.kv_heads", "must divide heads")
    a["scale"] = _number(m, "scale", where)
    a["window"], a["keep_first"] = None, 0
    if m.get("mask") is not None:
        mask = _field(m, "mask", where, dict)
        a["window"] = _pos_int(mask, "size", f"{where}.mask")
        a["keep_first"] = _count(mask, "keep_first", f"{where}.mask", 0)
    a["rot"] = None
    if m.get("rot") is not None:
        rw, rot = f"{where}.rot", _field(m, "rot", where, dict)
        dims = _pos_int(rot, "dims", rw)
        if dims % 2 or dims > a["dim"]:
            raise InvalidField(f"{rw}.dims", "must be even and at most dim")
        scaling = None
        if rot.get("scaling") is not None:
            sw, sc = f"{rw}.scaling", _field(rot, "scaling", rw, dict)
            scaling = RotaryScaling(_positive(sc, "factor", sw))
            if "original" in sc:
                scaling = RotaryScaling(_positive(sc, "factor", sw), _positive(sc, "low", sw), _positive(sc, "high", sw),
                                        _positive(sc, "original", sw))
                if not scaling.high > scaling.low:
                    raise InvalidField(sw, "high must lie above low")
        a["rot"] = (dims, _positive(rot, "base", rw), scaling)
    return a


@dataclass(frozen=True)
class PafelornLayer:
    type: str
    mixer: dict
    mlp: Optional[dict]


@dataclass(frozen=True)
class PafelornConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    embedding_scale: float
    bigram: Tuple[int, int, int]               # buckets, mul_prev, mul_cur
    logit_softcap: Optional[float]
    layers: Tuple[PafelornLayer, ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, d: dict) -> "PafelornConfig":
        if not isinstance(d, dict):
            raise ConfigError("config.json must hold a JSON object")
        layers_json = d.get("layers")
        if not isinstance(layers_json, list) or not layers_json:
            raise MissingField("layers")
        layers = []
        for i, lj in enumerate(layers_json):
            where = f"layers[{i}]"
            if not isinstance(lj, dict):
                raise InvalidField(where, "expected an object")
            typ = lj.get("type")
            if typ not in MIXER_TYPES:
                raise InvalidField(f"{where}.type", f"{typ!r}; known: {', '.join(MIXER_TYPES)}")
            m, mw = lj.get("mixer"), f"{where}.mixer"
            if not isinstance(m, dict):
                raise MissingField(mw)
            if typ == "attention":
                mixer = _attention(m, mw)
                mixer["diff"] = _number(m, "diff", mw)
                mixer["kv_from"] = None
                if m.get("kv_from") is not None:
                    j = mixer["kv_from"] = _count(m, "kv_from", mw)
                    if j >= i or layers[j].type != "attention" or layers[j].mixer["kv_from"] is not None:
                        raise InvalidField(f"{mw}.kv_from", f"{j} is no earlier attention layer with keys and values of its own")
                    if any(layers[j].mixer[k] != mixer[k] for k in ("heads", "kv_heads", "dim", "vdim", "rot")):
                        raise InvalidField(f"{mw}.kv_from", f"layer {j} has other heads or another rotation")
            else:
                left, right = _field(m, "left", mw, dict), _field(m, "right", mw, dict)
                lm, rm = _attention(left, f"{mw}.left"), {"width": _pos_int(right, "width", f"{mw}.right")}
                mixer = {"left": lm, "right": rm}
                if typ == "parallel":
                    mixer.update(left_scale=_number(m, "left_scale", mw), right_scale=_number(m, "right_scale", mw))
                else:
                    lm["softcap"] = _positive(left, "softcap", f"{mw}.left") if left.get("softcap") is not None else None
                    rm.update(blocks=_pos_int(right, "blocks", f"{mw}.right"), conv=_pos_int(right, "conv", f"{mw}.right"))
                    if rm["width"] % rm["blocks"]:
                        raise InvalidField(f"{mw}.right.blocks", "must divide width")
            mj, mlp = lj.get("mlp"), None
            if mj is not None:
                fw = f"{where}.mlp"
                kind = mj.get("kind") if isinstance(mj, dict) else None
                if kind == "dense":
                    mlp = {"kind": "dense", "ff": _pos_int(mj, "ff", fw)}
                elif kind == "moe":
                    ex, ro = _field(mj, "expert", fw, dict), _field(mj, "router", fw, dict)
                    mlp = {"kind": "moe", "ff": _pos_int(ex, "ff", f"{fw}.expert"), "limit": _positive(ex, "limit", f"{fw}.expert"),
                           "experts": _pos_int(ro, "experts", f"{fw}.router"), "top": _pos_int(ro, "top", f"{fw}.router"),
                           "identity": _count(ro, "identity", f"{fw}.router", 0), "shared": None}
                    if mlp["top"] > mlp["experts"] + mlp["identity"]:
                        raise InvalidField(f"{fw}.router.top", f"{mlp['experts']} + {mlp['identity']} experts cannot offer {mlp['top']} choices")
                    if mj.get("shared") is not None:
                        sh = _field(mj, "shared", fw, dict)
                        mlp["shared"] = (_pos_int(sh, "ff", f"{fw}.shared"), _positive(sh, "limit", f"{fw}.shared"))
                else:
                    raise InvalidField(f"{fw}.kind", f"{kind!r}; known: dense, moe")
            layers.append(PafelornLayer(typ, mixer, mlp))
        emb = _field(d, "embedding", "", dict)
        bg = _field(emb, "bigram", "embedding", dict)
        maxpos = d.get("max_position_embeddings", DEFAULT_MAX_POSITIONS)
        if isinstance(maxpos, bool) or not isinstance(maxpos, int) or maxpos <= 0:
            raise InvalidField("max_position_embeddings", f"expected a positive integer, got {maxpos!r}")
        return cls(vocab_size=_pos_int(d, "vocab"), hidden_size=_pos_int(d, "width"),
                   eps=_positive(_field(d, "norm", "", dict), "eps", "norm"), embedding_scale=_number(emb, "scale", "embedding"),
                   bigram=(_pos_int(bg, "buckets", "embedding.bigram"), _count(bg, "mul_prev", "embedding.bigram"),
                           _count(bg, "mul_cur", "embedding.bigram")),
                   logit_softcap=_positive(d, "logit_softcap", "") if d.get("logit_softcap") is not None else None,
                   layers=tuple(layers), max_position_embeddings=maxpos)


def _rotary(a, interleaved):
    if a["rot"] is None:
        return None
    dims, base, scaling = a["rot"]
    return RotarySpec(a["dim"], base, rotary_dim=dims, interleaved=interleaved, scaling=scaling)


def _grouped(a, W, eps, **kw):
    return AttentionSpec(hidden_size=W, num_heads=a["heads"], num_kv_heads=a["kv_heads"], head_dim=a["dim"], v_head_dim=a["vdim"],
                         qk_norm=NormSpec(a["dim"], eps, tensor=""), position=_rotary(a, True), window=a["window"],
                         keep_first=a["keep_first"] or None, scale=a["scale"], names=("q", "k", "v", "o"),
                         bias_names=("q.b", "k.b", "v.b", "o.b"), norm_prefixes=("q.norm", "k.norm"), **kw)


def _mixer(layer: PafelornLayer, W: int, eps: float):
    m = layer.mixer
    if layer.type == "attention":
        return DifferentialAttentionSpec(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                         eps=eps, diff=m["diff"], scale=m["scale"], qk_norm=NormSpec(m["dim"], eps, tensor=""),
                                         position=_rotary(m, False), window=m["window"], keep_first=m["keep_first"] or None,
                                         own_kv=m["kv_from"] is None)
    lm, rm = m["left"], m["right"]
    if layer.type == "parallel":
        left = _grouped(lm, W, eps, bias=True, out_bias=True, head_temp="temp", sink="sink")
        return ParallelMixerSpec(left, MinGruSpec(W, rm["width"]), m["left_scale"], m["right_scale"])
    left = _grouped(lm, W, eps, whole_norm=True, softcap=lm["softcap"], gate="g")
    norm = NormSpec(W, eps, tensor="")
    return ParallelMixerSpec(left, GatedLruSpec(W, rm["width"], rm["blocks"], rm["conv"], rate=LRU_RATE), NORMED_PAIR_SCALE,
                             NORMED_PAIR_SCALE, out_norms=(norm, norm))


def pafelorn_plan(cfg: PafelornConfig) -> ModelPlan:
    W, eps = cfg.hidden_size, cfg.eps
    norm = NormSpec(W, eps, tensor="")
    blocks, order, unused = [], [], []
    for i, layer in enumerate(cfg.layers):
        ffn, p = None, layer.mlp
        if p is None:
            unused.append(f"l{i}.norm2")               # a layer without a feed-forward may still store its norm
        elif p["kind"] == "dense":
            ffn = GatedMlpSpec(W, p["ff"], activation="poly_norm", gated=False, names=("gate", "up", "down"), coef="act", eps=eps)
        else:
            act = dict(activation=EXPERT_ACTIVATION, alpha=EXPERT_ALPHA, up_shift=EXPERT_UP_SHIFT, names=("gate", "up", "down"))
            shared = GatedMlpSpec(W, p["shared"][0], limit=p["shared"][1], **act) if p["shared"] is not None else None
            ffn = RoutedExpertsSpec(W, p["ff"], p["experts"], p["top"], limit=p["limit"], score="softmax", renormalize=True,
                                    scale_input=False, choice_bias="correction", renorm_eps=RENORM_EPS, identity=p["identity"],
                                    shared=shared, shared_gate="shared.sg" if shared is not None else None, **act)
        blocks.append(BlockSpec(mixer=_mixer(layer, W, eps), ffn=ffn, norm1=norm, norm2=norm, kind="post_norm",
                                names=("norm1", "mix.", "norm2", "mlp.")))
        order.append(LayerCall(i, layer.mixer["kv_from"] if layer.type == "attention" else None))
    buckets, mul_prev, mul_cur = cfg.bigram
    return ModelPlan(architecture=ARCHITECTURE, vocab_size=cfg.vocab_size, hidden_size=W, layers=tuple(blocks), order=tuple(order),
                     final_norm=norm, tie_word_embeddings=False, max_position_embeddings=cfg.max_position_embeddings,
                     layer_prefix="l{}.", embed_prefix="", final_norm_prefix="final.norm", head_prefix="",
                     embedding=PairEmbeddingSpec(cfg.vocab_size, W, buckets, mul_prev, mul_cur, scale=cfg.embedding_scale),
                     head=CappedHeadSpec(cfg.vocab_size, W, softcap=cfg.logit_softcap, tensor="head"), unused_tensors=tuple(unused))


register_architecture(ARCHITECTURE, PafelornConfig, pafelorn_plan, model_types=("pafelorn",), replace=True)
