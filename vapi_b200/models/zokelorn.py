"""Zokelorn (``"architecture": "Zokelorn"``) as a plan of parts.

A decoder-only model.  Every layer is parallel: one RMS norm, and the mixer and the feed-forward both read its output;
both results are added to the stream.  A layer's mixer is one of

* ``attention``: grouped-query attention within chunks of ``mask.size`` positions counted from position 0, interleaved
  rotary pairs over ``rot.dims`` elements of a head with the frequency rule of Llama 3.1 (``rot.scaling``), a free
  ``scale`` and a sigmoid gate per head;
* ``lightning``: linear attention with a fixed decay per head, SiLU on q, k and v, one RMS norm with a weight over all
  heads together and a sigmoid gate as wide;
* ``retention``: the same recurrence on plain q, k and v (times ``dim^-1/2``), a weightless RMS norm per head and a SiLU
  gate.

Its feed-forward is a dense one gated by the tanh form of GELU, a mixture of SiLU-gated experts (scores are sigmoids of the
router's logits, grouped choice by the sum of a group's two largest, weights normalised over the chosen) with a shared
expert behind a sigmoid gate per token, or absent.  ``loop`` = {start, stop, times} runs layers start .. stop-1 that many
times in a row with the same weights, every pass with caches and states of its own.  The model ends on an RMS norm and a
head of its own.  Everything here is data handed to parameterised parts.

config.json keys: ``vocab``, ``width``, ``norm.eps``, ``loop{start stop times}`` and ``layers[i] = {type, mixer, mlp}`` with
``mixer`` = ``{heads kv_heads dim vdim scale mask{size} rot{base dims scaling{factor low high original}}}`` |
``{heads dim vdim decay[heads]}`` and ``mlp`` = null | ``{kind: dense, ff}`` | ``{kind: moe, expert{ff}, router{experts top
groups{count keep}}, shared{ff}}``.
Tensors: ``embed``, ``l<i>.norm1``, ``l<i>.mix.{q,k,v,g,o}``, ``l<i>.mix.norm`` (lightning), ``l<i>.mlp.{gate,up,down}`` or
``l<i>.mlp.{e<j>.gate, e<j>.up, e<j>.down, router, shared.gate, shared.up, shared.down, shared.sg}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from ..config.model import Architecture, ConfigError, register_architecture, require_int
from ..parts import (FixedDecayMixer, GQAttention, OutputHead, ParallelBlock, RMSNorm, ScaledRotaryEncoding, SparseMoE, SwiGLU,
                     TokenEmbedding)
from .plan import ModelPlan, looped_order

#: positions are counted in float32, which holds integers exactly up to here
MAX_POSITIONS = 1 << 24
#: how many of a group's largest scores make the group's own
GROUP_TOP = 2

MIXER_TYPES = ("attention", "lightning", "retention")


def _num(v: Any, key: str, where: str) -> float:
    x = v.get(key) if isinstance(v, dict) else None
    if isinstance(x, bool) or not isinstance(x, (int, float)):
        raise ConfigError(f"config.json: {where} needs the number `{key}`")
    return float(x)


def _int(v: Any, key: str, where: str, least: int = 1) -> int:
    x = v.get(key) if isinstance(v, dict) else None
    if isinstance(x, bool) or not isinstance(x, int) or x < least:
        raise ConfigError(f"config.json: {where} needs the integer `{key}` >= {least}")
    return int(x)


Items = Tuple[Tuple[str, Any], ...]


@dataclass(frozen=True)
class ZokelornLayer:
    kind: str                                    # attention | lightning | retention
    mixer: Items                                 # the mixer's sizes and constants, as sorted items
    mlp: Optional[Items]                         # None: no feed-forward


@dataclass(frozen=True)
class ZokelornConfig:
    vocab: int
    width: int
    norm_eps: float
    loop: Optional[Tuple[int, int, int]]         # (start, stop, times); None: every layer runs once
    layers: Tuple[ZokelornLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_json(cls, v: Dict[str, Any]) -> "ZokelornConfig":
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
            mx = e.get("mixer")
            if not isinstance(mx, dict):
                raise ConfigError(f"config.json: {where} needs `mixer`")
            m = cls._attention(mx, where) if e["type"] == "attention" else cls._decayed(mx, where)
            f = cls._mlp(e["mlp"], where) if e.get("mlp") is not None else None
            layers.append(ZokelornLayer(e["type"], tuple(sorted(m.items())), tuple(sorted(f.items())) if f is not None else None))
        loop = None
        lp = v.get("loop")
        if lp is not None:
            a, b, t = _int(lp, "start", "loop", 0), _int(lp, "stop", "loop"), _int(lp, "times", "loop")
            if not a < b <= len(layers):
                raise ConfigError(f"config.json: loop from {a} to {b} over {len(layers)} layers")
            loop = (a, b, t)
        eos = v.get("eos_token_id")
        eos_ids = (int(eos),) if isinstance(eos, int) and not isinstance(eos, bool) else \
            tuple(int(x) for x in eos if isinstance(x, int)) if isinstance(eos, list) else ()
        return cls(vocab=require_int(v, "vocab"), width=require_int(v, "width"), norm_eps=_num(norm, "eps", "norm"), loop=loop,
                   layers=tuple(layers), eos_token_ids=tuple(sorted(set(eos_ids))))

    @staticmethod
    def _attention(mx: Dict[str, Any], where: str) -> Dict[str, Any]:
        m: Dict[str, Any] = {k: _int(mx, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"config.json: {where}: {m['heads']} heads over {m['kv_heads']} kv heads")
        m["scale"] = _num(mx, "scale", where)
        m["chunk"] = _int(mx["mask"], "size", where + " mask") if mx.get("mask") is not None else 0
        m["rot"] = None
        rot = mx.get("rot")
        if rot is not None:
            dims, base = _int(rot, "dims", where + " rot"), _num(rot, "base", where + " rot")
            if dims % 2 or dims > m["dim"] or base <= 0:
                raise ConfigError(f"config.json: {where}: {dims} rotated elements of {m['dim']}, base {base}")
            scaling = None
            if rot.get("scaling") is not None:
                sc = {k: _num(rot["scaling"], k, where + " rot.scaling") for k in ("factor", "low", "high", "original")}
                if sc["factor"] <= 0 or sc["low"] <= 0 or sc["high"] < sc["low"] or sc["original"] <= 0:
                    raise ConfigError(f"config.json: {where}: rot.scaling {sc}")
                scaling = tuple(sorted(sc.items()))
            m["rot"] = (dims, base, scaling)
        return m

    @staticmethod
    def _decayed(mx: Dict[str, Any], where: str) -> Dict[str, Any]:
        m: Dict[str, Any] = {k: _int(mx, k, where) for k in ("heads", "dim", "vdim")}
        decay = mx.get("decay")
        if not isinstance(decay, list) or len(decay) != m["heads"] or \
                any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
            raise ConfigError(f"config.json: {where}: `decay` must list one number per head ({m['heads']})")
        m["decay"] = tuple(float(d) for d in decay)
        return m

    @staticmethod
    def _mlp(mlp: Any, where: str) -> Dict[str, Any]:
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"config.json: {where}: the feed-forward kind must be `dense` or `moe`")
        if mlp["kind"] == "dense":
            return {"kind": "dense", "ff": _int(mlp, "ff", where + " mlp")}
        r = mlp.get("router")
        f: Dict[str, Any] = {"kind": "moe", "ff": _int(mlp.get("expert"), "ff", where + " mlp.expert"),
                             "experts": _int(r, "experts", where + " mlp.router"), "top": _int(r, "top", where + " mlp.router")}
        g = r.get("groups")
        f["groups"] = _int(g, "count", where + " mlp.router.groups") if g is not None else 1
        f["keep"] = _int(g, "keep", where + " mlp.router.groups") if g is not None else 1
        if f["experts"] % f["groups"] or f["keep"] > f["groups"] or (f["experts"] // f["groups"]) * f["keep"] < f["top"]:
            raise ConfigError(f"config.json: {where}: {f['experts']} experts in {f['groups']} groups, {f['keep']} kept, top {f['top']}")
        sh = mlp.get("shared")
        f["shared_ff"] = _int(sh, "ff", where + " mlp.shared") if sh is not None else None
        return f


def zokelorn_plan(cfg: ZokelornConfig) -> ModelPlan:
    W, eps = cfg.width, cfg.norm_eps
    emb = TokenEmbedding(cfg.vocab, W, "embed")
    ropes: Dict[Any, ScaledRotaryEncoding] = {}
    layers, prefixes = [], []
    for i, layer in enumerate(cfg.layers):
        m = dict(layer.mixer)
        if layer.kind == "attention":
            rot = m["rot"]
            if rot is not None and rot not in ropes:          # layers that agree share one pair of tables
                ropes[rot] = ScaledRotaryEncoding(rot[0], rot[1], dict(rot[2]) if rot[2] else None, name=f"rope{len(ropes)}")
            mixer = GQAttention(W, m["heads"], m["kv_heads"], m["dim"], qk_norm_eps=None, scale=m["scale"], v_head_dim=m["vdim"],
                                pos=ropes[rot].name if rot is not None else None, rot_dim=rot[0] if rot is not None else None,
                                rope_layout="interleaved", chunk=m["chunk"], head_gate=True, weight_suffix="",
                                names={"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g"})
        else:
            lightning = layer.kind == "lightning"
            mixer = FixedDecayMixer(W, m["heads"], m["dim"], m["vdim"], m["decay"], eps, act="silu" if lightning else None,
                                    norm="all" if lightning else "head", gate="sigmoid" if lightning else "silu",
                                    qk_scale=1.0 if lightning else m["dim"] ** -0.5, weight_suffix="",
                                    names={"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm"})
        ffn = None
        if layer.mlp is not None:
            f = dict(layer.mlp)
            if f["kind"] == "dense":
                ffn = SwiGLU(W, f["ff"], {"gate": "gate", "up": "up", "down": "down"}, weight_suffix="", act="gelu_tanh")
            else:
                ffn = SparseMoE(W, f["ff"], f["experts"], f["top"], groups=f["groups"], keep=f["keep"], shared_ff=f["shared_ff"],
                                gated=True, score="sigmoid", correction=False, group_top=GROUP_TOP,
                                shared_gate=f["shared_ff"] is not None, weight_suffix="",
                                names={"expert": "e{}.", "gate": "gate", "up": "up", "down": "down", "router": "router",
                                       "shared": "shared.", "shared_gate": "sg"})
        layers.append(ParallelBlock(RMSNorm(W, eps, "norm1"), mixer, ffn, {"mixer": "mix.", "ffn": "mlp."}, hidden=W))
        prefixes.append(f"l{i}.")
    return ModelPlan(
        architecture="Zokelorn", vocab_size=cfg.vocab, hidden_size=W, max_positions=MAX_POSITIONS, embedding=emb,
        layers=layers, layer_prefixes=prefixes, order=looped_order(len(layers), cfg.loop), final_norm=RMSNorm(W, eps, "norm"),
        final_norm_prefix="final.", head=OutputHead(cfg.vocab, W, False, emb, "head"),
        position_encodings=list(ropes.values()), eos_token_ids=cfg.eos_token_ids, config=cfg)


register_architecture(Architecture(name="Zokelorn", model_types=("zokelorn",), parse=ZokelornConfig.from_json, plan=zokelorn_plan))
