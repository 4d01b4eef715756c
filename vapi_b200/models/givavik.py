"""Givavik (``"architecture": "Givavik"``) as a plan of parts.

A decoder-only model.  The embedding's rows are multiplied by ``embedding.scale``, and a row of a second table, picked by
a hash of the token and the one before it, is added (``embedding.bigram``; the previous token is part of a request's
state).  Every layer is parallel: one RMS norm whose weight is stored around zero, and the mixer and the feed-forward
both read its output, the mixer through a token shift (a request's last normed row is part of its state, in every
layer); each result is multiplied column by column by a stored vector (layer scale) before both are added to the
stream.  A layer's mixer is one of

* ``latent_attention``: queries straight from the input, keys and values expanded from a normed latent that is all the
  cache keeps, beside one rotated key part that the heads share (interleaved pairs over the whole part), with a learned
  sink per head in the softmax's denominator; with ``kv_from`` the layer has no latent of its own and reads the cache of
  an earlier layer;
* ``parallel``: ``left_scale * left + right_scale * right`` on the same input, with ``left`` grouped-query attention
  (biases on all four projections, interleaved rotary pairs over ``rot.dims`` elements, RMS norms of q and k per head
  without a weight, capped scores, weights that are sigmoids of score + a stored number per head, not normalised over
  the keys) and ``right`` Mamba-2.

Its feed-forward is one hidden layer with the xIELU activation, or absent.  The model ends on such an RMS norm and a head
of its own.  Everything here is data handed to parameterised parts.

config.json keys: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``embedding.bigram{buckets mul_prev mul_cur}``
and ``layers[i] = {type, mixer, mlp}`` with ``mixer`` = ``{heads dim rot_dim vdim kv_rank scale rot{base dims} kv_from?}`` |
``{left{heads kv_heads dim vdim scale softcap rot{base dims}} left_scale right{heads vdim state groups conv norm_groups}
right_scale}`` and ``mlp`` = null | ``{kind: dense, ff}``.
Tensors: ``embed``, ``bigram``, ``l<i>.norm1 ls1 ls2 shift``, ``l<i>.mix.{q, dkv, dkv.norm, uk, uv, sink, o}`` |
``l<i>.mix.left.{q,k,v,o}(.b) pb``, ``l<i>.mix.right.{in, conv, conv.b, dt_bias, A_log, D, norm, o}``,
``l<i>.mlp.{up, down, act}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from ..config.model import Architecture, ConfigError, register_architecture, require_int
from ..parts import (GQAttention, LatentAttention, Mamba2Mixer, OutputHead, ParallelBlock, ParallelMixer, RMSNorm,
                     ScaledRotaryEncoding, TokenEmbedding, XIELU)
from .plan import LayerCall, ModelPlan

#: positions are counted in float32, which holds integers exactly up to here
MAX_POSITIONS = 1 << 24
#: norm weights are stored as what is added to one
NORM_OFFSET = 1.0

MIXER_TYPES = ("latent_attention", "parallel")


def _num(v: Any, key: str, where: str) -> float:
    x = v.get(key) if isinstance(v, dict) else None
    if isinstance(x, bool) or not isinstance(x, (int, float)):
        raise ConfigError(f"config.json: {where} needs the number `{key}`")
    return float(x)


def _opt_num(v: Any, key: str, where: str, default: Optional[float]) -> Optional[float]:
    return default if not isinstance(v, dict) or v.get(key) is None else _num(v, key, where)


def _int(v: Any, key: str, where: str, least: int = 1) -> int:
    x = v.get(key) if isinstance(v, dict) else None
    if isinstance(x, bool) or not isinstance(x, int) or x < least:
        raise ConfigError(f"config.json: {where} needs the integer `{key}` >= {least}")
    return int(x)


def _rotation(v: Any, most: int, where: str) -> Optional[Tuple[int, float]]:
    """(rotated elements, base) of a mixer's ``rot``; None: no rotation."""
    rot = v.get("rot")
    if rot is None:
        return None
    dims, base = _int(rot, "dims", where + " rot"), _num(rot, "base", where + " rot")
    if dims % 2 or dims > most or base <= 0:
        raise ConfigError(f"config.json: {where}: {dims} rotated elements of {most}, base {base}")
    return dims, base


@dataclass(frozen=True)
class GivavikLayer:
    kind: str                                    # latent_attention | parallel
    mixer: Tuple[Tuple[str, Any], ...]           # the mixer's sizes and constants, as sorted items
    ff: Optional[int]                            # None: no feed-forward


@dataclass(frozen=True)
class GivavikConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: Optional[Tuple[int, int, int]]       # (buckets, mul_prev, mul_cur)
    layers: Tuple[GivavikLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_json(cls, v: Dict[str, Any]) -> "GivavikConfig":
        norm = v.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json: missing `norm`")
        raw = v.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: `layers` must be a non-empty list")
        layers = []
        for i, e in enumerate(raw):
            where = f"layer {i}"
            if not isinstance(e, dict) or e.get("type") not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}: type must be one of {', '.join(MIXER_TYPES)}")
            kind, mx = e["type"], e.get("mixer")
            if not isinstance(mx, dict):
                raise ConfigError(f"config.json: {where} needs `mixer`")
            m = cls._latent(mx, where) if kind == "latent_attention" else cls._parallel(mx, where)
            source = m.get("kv_from")
            if source is not None:
                if not 0 <= source < i or layers[source].kind != "latent_attention":
                    raise ConfigError(f"config.json: {where}: kv_from {source} must name an earlier latent attention layer")
                theirs = dict(layers[source].mixer)
                if theirs["kv_from"] is not None or any(theirs[k] != m[k] for k in ("kv_rank", "rot_dim", "rot")):
                    raise ConfigError(f"config.json: {where}: layer {source} must have a latent of its own, of the same size and rotation")
            mlp = e.get("mlp")
            ff = None
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}: the feed-forward kind must be `dense`")
                ff = _int(mlp, "ff", where + " mlp")
            layers.append(GivavikLayer(kind, tuple(sorted(m.items())), ff))
        emb = v.get("embedding")
        scale = _opt_num(emb, "scale", "embedding", 1.0)
        bigram = None
        bg = emb.get("bigram") if isinstance(emb, dict) else None
        if bg is not None:
            bigram = (_int(bg, "buckets", "embedding.bigram"), _int(bg, "mul_prev", "embedding.bigram", 0),
                      _int(bg, "mul_cur", "embedding.bigram", 0))
        eos = v.get("eos_token_id")
        eos_ids = (int(eos),) if isinstance(eos, int) and not isinstance(eos, bool) else \
            tuple(int(x) for x in eos if isinstance(x, int)) if isinstance(eos, list) else ()
        return cls(vocab=require_int(v, "vocab"), width=require_int(v, "width"), norm_eps=_num(norm, "eps", "norm"),
                   embedding_scale=scale, bigram=bigram, layers=tuple(layers), eos_token_ids=tuple(sorted(set(eos_ids))))

    @staticmethod
    def _latent(mx: Dict[str, Any], where: str) -> Dict[str, Any]:
        m: Dict[str, Any] = {k: _int(mx, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
        m["scale"] = _num(mx, "scale", where)
        m["rot"] = _rotation(mx, m["rot_dim"], where)
        m["kv_from"] = _int(mx, "kv_from", where, 0) if mx.get("kv_from") is not None else None
        return m

    @staticmethod
    def _parallel(mx: Dict[str, Any], where: str) -> Dict[str, Any]:
        le, ri = mx.get("left"), mx.get("right")
        if not isinstance(le, dict) or not isinstance(ri, dict):
            raise ConfigError(f"config.json: {where} needs `mixer.left` and `mixer.right`")
        left: Dict[str, Any] = {k: _int(le, k, where + " left") for k in ("heads", "kv_heads", "dim", "vdim")}
        if left["heads"] % left["kv_heads"]:
            raise ConfigError(f"config.json: {where}: {left['heads']} heads over {left['kv_heads']} kv heads")
        left["scale"] = _num(le, "scale", where + " left")
        left["softcap"] = _opt_num(le, "softcap", where + " left", None)
        if left["softcap"] is not None and left["softcap"] <= 0:
            raise ConfigError(f"config.json: {where}: softcap {left['softcap']}")
        left["rot"] = _rotation(le, left["dim"], where + " left")
        right = {k: _int(ri, k, where + " right") for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}
        if right["heads"] % right["groups"] or (right["heads"] * right["vdim"]) % right["norm_groups"]:
            raise ConfigError(f"config.json: {where}: {right['heads']} heads of {right['vdim']} in {right['groups']} groups and "
                              f"{right['norm_groups']} norm groups")
        return {"left": tuple(sorted(left.items())), "right": tuple(sorted(right.items())),
                "left_scale": _num(mx, "left_scale", where), "right_scale": _num(mx, "right_scale", where)}


def givavik_plan(cfg: GivavikConfig) -> ModelPlan:
    W, eps = cfg.width, cfg.norm_eps
    emb = TokenEmbedding(cfg.vocab, W, "embed", scale=cfg.embedding_scale,
                         bigram=("bigram",) + cfg.bigram if cfg.bigram is not None else None)
    ropes: Dict[Any, ScaledRotaryEncoding] = {}

    def rope(rot: Optional[Tuple[int, float]]) -> Optional[str]:
        if rot is None:
            return None
        if rot not in ropes:              # layers that agree share one pair of tables
            ropes[rot] = ScaledRotaryEncoding(rot[0], rot[1], None, name=f"rope{len(ropes)}")
        return ropes[rot].name

    layers, prefixes, order = [], [], []
    for i, layer in enumerate(cfg.layers):
        m = dict(layer.mixer)
        source = m.get("kv_from")
        if layer.kind == "latent_attention":
            mixer = LatentAttention(W, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], None, scale=m["scale"],
                                    norm_eps=eps, pos=rope(m["rot"]), rot=m["rot"][0] if m["rot"] else 0, weight_suffix="",
                                    rope_layout="interleaved", sink=True, own_latent=source is None,
                                    names={"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o",
                                           "sink": "sink"})
        else:
            le, ri = dict(m["left"]), dict(m["right"])
            left = GQAttention(W, le["heads"], le["kv_heads"], le["dim"], qk_norm_eps=eps, qk_norm_weight=False,
                               pos=rope(le["rot"]), rot_dim=le["rot"][0] if le["rot"] else None, rope_layout="interleaved",
                               bias=True, scale=le["scale"], v_head_dim=le["vdim"], softcap=le["softcap"], weights="sigmoid",
                               score_bias=True, weight_suffix="", bias_suffix=".b",
                               names={"q": "q", "k": "k", "v": "v", "o": "o", "score_bias": "pb"})
            right = Mamba2Mixer(W, ri["heads"], ri["vdim"], ri["state"], ri["groups"], ri["conv"], ri["norm_groups"], eps,
                                weight_suffix="", names={"in": "in", "conv": "conv", "conv_bias": "conv.b", "norm": "norm",
                                                         "o": "o"})
            mixer = ParallelMixer(W, [("left.", left), ("right.", right)], factors=(m["left_scale"], m["right_scale"]))
        ffn = XIELU(W, layer.ff, {"up": "up", "down": "down", "act": "act"}, weight_suffix="") if layer.ff is not None else None
        layers.append(ParallelBlock(RMSNorm(W, eps, "norm1", offset=NORM_OFFSET), mixer, ffn, {"mixer": "mix.", "ffn": "mlp."},
                                    scales=("ls1", "ls2"), hidden=W, shift="shift"))
        prefixes.append(f"l{i}.")
        order.append(LayerCall(i, cache_of=source))
    return ModelPlan(
        architecture="Givavik", vocab_size=cfg.vocab, hidden_size=W, max_positions=MAX_POSITIONS, embedding=emb,
        layers=layers, layer_prefixes=prefixes, order=order, final_norm=RMSNorm(W, eps, "norm", offset=NORM_OFFSET),
        final_norm_prefix="final.", head=OutputHead(cfg.vocab, W, False, emb, "head"),
        position_encodings=list(ropes.values()), eos_token_ids=cfg.eos_token_ids, config=cfg)


register_architecture(Architecture(name="Givavik", model_types=("givavik",), parse=GivavikConfig.from_json, plan=givavik_plan))
