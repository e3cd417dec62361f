"""Configuration of the Vekusun decoder and its plan of parts.

config.json: `architecture` (a string), `vocab`, `width`, `norm.eps`, `residual_mult`, `logit_softcap`, `loop`
{"start", "stop", "times"} and `layers`, one object per layer:

    {"type": "delta", "mixer": {"heads", "kv_heads", "dim", "vdim", "conv"}, "mlp": ...}
    {"type": "latent_attention", "mixer": {"heads", "dim", "vdim", "q_rank", "kv_rank", "scale"}, "mlp": ...}
    {"type": "latent_attention_2",
     "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale",
               "rot": {"dims", "base", "scaling"?: {"factor", "original", "fast", "slow"}}}, "mlp": ...}
    "mlp": null | {"kind": "dense", "ff"} | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}

Every size and every constant the file gives is read from it.  What the design fixes stands in `vekusun_plan` as arguments of
the parts: blocks whose mixer and feed-forward read ONE norm's output and are added with a factor per channel each and one for
both; a stretch of layers that runs several times with the same weights, each time from caches and states of its own, the
embedding added again before every pass but the first and a vector per pass before each; latent attention without positions, with
a query latent and a sink, or with an interleaved rotation whose frequencies and amplitude follow YaRN, queries straight from the
input and a gate per head; a delta rule with one decay per head behind short convolutions, with a silu gate; a dense
feed-forward with the erf gelu, or silu experts chosen by softmax score plus a correction and weighted by the score as it
is.  Tensor names are flat: `embed`, `loop.step`, `l<i>.norm1`, `l<i>.ls1`, `l<i>.ls2`, `l<i>.mix.<t>`, `l<i>.mlp.<t>`, `final.norm`,
`head`.  `loop`, `rot.scaling` and `logit_softcap` may be absent (the option is then off).  `max_position_embeddings` is optional (an
engine bound on a request's length, not part of the design).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..parts.spec import (BlockSpec, CappedHeadSpec, EmbeddingSpec, GatedMlpSpec, HeadDeltaSpec, LatentAttentionSpec, LayerCall,
                          ModelPlan, NormSpec, RotarySpec, RoutedExpertsSpec, YarnScaling)
from .errors import ConfigError, InvalidField, MissingField
from .kikepel import _field, _pos_int
from .pafelorn import _count, _number, _positive
from .registry import register_architecture

ARCHITECTURE = "Vekusun"
MIXER_SIZES = {"delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
               "latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank"),
               "latent_attention_2": ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
DEFAULT_MAX_POSITIONS = 32768

# what the design fixes
DENSE_ACTIVATION = "gelu"
EXPERT_ACTIVATION = "silu"
UNIT_EPS = 1e-6                    # under the root of the delta rule's unit vectors


def _rotation(rot, rot_dim, where):
    dims, base = _pos_int(rot, "dims", where), _positive(rot, "base", where)
    if dims % 2 or dims > rot_dim:
        raise InvalidField(f"{where}.dims", "must be even and at most rot_dim")
    scaling = None
    if rot.get("scaling") is not None:
        sw, sc = f"{where}.scaling", _field(rot, "scaling", where, dict)
        scaling = YarnScaling(*(_positive(sc, k, sw) for k in ("factor", "original", "fast", "slow")))
        if base == 1.0:
            raise InvalidField(f"{where}.base", "frequencies that are all equal cannot be told apart by a scaling")
    return dims, base, scaling


@dataclass(frozen=True)
class VekusunLayer:
    type: str
    mixer: dict
    mlp: Optional[dict]


@dataclass(frozen=True)
class VekusunConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    residual_mult: float
    logit_softcap: Optional[float]
    loop: Optional[Tuple[int, int, int]]       # start, stop, times
    layers: Tuple[VekusunLayer, ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, d: dict) -> "VekusunConfig":
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
            if typ not in MIXER_SIZES:
                raise InvalidField(f"{where}.type", f"{typ!r}; known: {', '.join(MIXER_SIZES)}")
            m, mw = lj.get("mixer"), f"{where}.mixer"
            if not isinstance(m, dict):
                raise MissingField(mw)
            mixer = {k: _pos_int(m, k, mw) for k in MIXER_SIZES[typ]}
            if typ == "delta":
                if mixer["heads"] % mixer["kv_heads"]:
                    raise InvalidField(f"{mw}.kv_heads", "must divide heads")
            else:
                mixer["scale"] = _number(m, "scale", mw)
                if typ == "latent_attention_2":
                    mixer["rot"] = _rotation(_field(m, "rot", mw, dict), mixer["rot_dim"], f"{mw}.rot")
            mj, mlp = lj.get("mlp"), None
            if mj is not None:
                fw = f"{where}.mlp"
                kind = mj.get("kind") if isinstance(mj, dict) else None
                if kind == "dense":
                    mlp = {"kind": "dense", "ff": _pos_int(mj, "ff", fw)}
                elif kind == "moe":
                    ex, ro = _field(mj, "expert", fw, dict), _field(mj, "router", fw, dict)
                    mlp = {"kind": "moe", "ff": _pos_int(ex, "ff", f"{fw}.expert"), "experts": _pos_int(ro, "experts", f"{fw}.router"),
                           "top": _pos_int(ro, "top", f"{fw}.router")}
                    if mlp["top"] > mlp["experts"]:
                        raise InvalidField(f"{fw}.router.top", f"{mlp['experts']} experts cannot offer {mlp['top']} choices")
                else:
                    raise InvalidField(f"{fw}.kind", f"{kind!r}; known: dense, moe")
            layers.append(VekusunLayer(typ, mixer, mlp))
        loop = None
        if d.get("loop") is not None:
            lo = _field(d, "loop", "", dict)
            loop = (_count(lo, "start", "loop"), _pos_int(lo, "stop", "loop"), _pos_int(lo, "times", "loop"))
            if not loop[0] < loop[1] <= len(layers):
                raise InvalidField("loop", f"layers {loop[0]} .. {loop[1] - 1} of {len(layers)}")
        maxpos = d.get("max_position_embeddings", DEFAULT_MAX_POSITIONS)
        if isinstance(maxpos, bool) or not isinstance(maxpos, int) or maxpos <= 0:
            raise InvalidField("max_position_embeddings", f"expected a positive integer, got {maxpos!r}")
        return cls(vocab_size=_pos_int(d, "vocab"), hidden_size=_pos_int(d, "width"),
                   eps=_positive(_field(d, "norm", "", dict), "eps", "norm"), residual_mult=_number(d, "residual_mult", ""),
                   logit_softcap=_positive(d, "logit_softcap", "") if d.get("logit_softcap") is not None else None,
                   loop=loop, layers=tuple(layers), max_position_embeddings=maxpos)


def _mixer(layer: VekusunLayer, W: int, eps: float):
    m = layer.mixer
    if layer.type == "delta":
        return HeadDeltaSpec(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                             conv=m["conv"], eps=eps, unit_eps=UNIT_EPS)
    sizes = dict(hidden_size=W, num_heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], eps=eps, scale=m["scale"])
    if layer.type == "latent_attention":
        return LatentAttentionSpec(q_rank=m["q_rank"], sink=True, **sizes)
    dims, base, scaling = m["rot"]
    return LatentAttentionSpec(q_rank=0, names=("dq", "dq.norm", "q", "dkv", "dkv.norm", "uk", "uv", "o", "sink"), rot_dim=m["rot_dim"],
                               position=RotarySpec(m["rot_dim"], base, rotary_dim=dims, interleaved=True, scaling=scaling),
                               head_gate="g", **sizes)


def _order(cfg: VekusunConfig):
    """The running order: the layers before the loop, its passes, the layers behind it."""
    n = len(cfg.layers)
    if cfg.loop is None:
        return tuple(LayerCall(i) for i in range(n))
    start, stop, times = cfg.loop
    calls = [LayerCall(i) for i in range(start)]
    for t in range(times):
        calls.append(LayerCall(start, add_embedding=t > 0, add_row=("loop.step", t)))
        calls += [LayerCall(i) for i in range(start + 1, stop)]
    return tuple(calls + [LayerCall(i) for i in range(stop, n)])


def vekusun_plan(cfg: VekusunConfig) -> ModelPlan:
    W, eps = cfg.hidden_size, cfg.eps
    norm = NormSpec(W, eps, tensor="")
    blocks, unused = [], []
    for i, layer in enumerate(cfg.layers):
        ffn, p = None, layer.mlp
        if p is None:
            unused.append(f"l{i}.ls2")                 # a layer without a feed-forward may still store its factors
        elif p["kind"] == "dense":
            ffn = GatedMlpSpec(W, p["ff"], activation=DENSE_ACTIVATION, gated=False, names=("gate", "up", "down"))
        else:
            ffn = RoutedExpertsSpec(W, p["ff"], p["experts"], p["top"], activation=EXPERT_ACTIVATION, score="softmax",
                                    renormalize=False, scale_input=False, choice_bias="correction")
        blocks.append(BlockSpec(mixer=_mixer(layer, W, eps), ffn=ffn, norm1=norm, norm2=norm, kind="shared_norm",
                                residual_mult=cfg.residual_mult, names=("norm1", "mix.", "norm2", "mlp."), scales=("ls1", "ls2")))
    return ModelPlan(architecture=ARCHITECTURE, vocab_size=cfg.vocab_size, hidden_size=W, layers=tuple(blocks), order=_order(cfg),
                     final_norm=norm, tie_word_embeddings=False, max_position_embeddings=cfg.max_position_embeddings,
                     layer_prefix="l{}.", embed_prefix="", final_norm_prefix="final.norm", head_prefix="",
                     embedding=EmbeddingSpec(cfg.vocab_size, W, tensor="embed"),
                     head=CappedHeadSpec(cfg.vocab_size, W, softcap=cfg.logit_softcap, tensor="head"), unused_tensors=tuple(unused),
                     stream_tables=(("loop.step", cfg.loop[2]),) if cfg.loop is not None else ())


register_architecture(ARCHITECTURE, VekusunConfig, vekusun_plan, model_types=("vekusun",), replace=True)
