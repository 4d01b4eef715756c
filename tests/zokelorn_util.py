"""Small Zokelorn configurations and model folders whose small parameters make faults show."""
from __future__ import annotations

import zlib
from typing import Optional, Sequence

import torch

import givavik_util
import plain_zokelorn as plain


def attention(heads=4, kv_heads=2, dim=20, vdim=12, scale=0.3, size: Optional[int] = 24, dims=12, base=30.0,
              scaling: Optional[Sequence[float]] = (3.0, 1.0, 5.0, 40.0)) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if size is not None:
        m["mask"] = {"size": size}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def memory(kind: str, heads=3, dim=12, vdim=20, decay: Optional[Sequence[float]] = None) -> dict:
    decay = list(decay) if decay is not None else [1.0 - 0.4 * 0.3 ** i for i in range(heads)]
    return {"type": kind, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def dense(ff=72) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(ff=20, experts=12, top=3, groups=(3, 2), shared: Optional[int] = 28) -> dict:
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer: dict, mlp: Optional[dict] = None) -> dict:
    return {**mixer, "mlp": mlp}


def config(layers: Sequence[dict], width=64, vocab=200, loop=None, eps=1e-5) -> dict:
    c = {"architecture": "Zokelorn", "layers": list(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


#: sizes that all differ from one another: every mixer with every kind of feed-forward, two chunk sizes (neither a page's),
#: unlike key and value widths, a loop that neither starts nor stops at the ends
MIXED = config([layer(memory("retention"), dense()),
                layer(attention(), moe()),
                layer(memory("lightning", heads=5, dim=8, vdim=28), moe(ff=12, experts=8, top=2, groups=(4, 3), shared=None)),
                layer(memory("retention", heads=2, dim=40, vdim=16, decay=[0.5, 0.995]), None),
                layer(attention(heads=3, kv_heads=1, dim=16, vdim=36, scale=0.2, size=37, dims=16, base=500.0, scaling=None), dense(40)),
                layer(memory("lightning", heads=1, dim=28, vdim=44, decay=[0.97]), moe(groups=None, top=5))], loop=(1, 4, 3))
#: tiny, for runs where plain Python stands in for the kernels
TINY = config([layer(memory("lightning", heads=2, dim=4, vdim=8), dense(24)),
               layer(attention(heads=2, kv_heads=1, dim=8, vdim=12, size=7, dims=4), moe(ff=8, experts=4, top=2, groups=(2, 1), shared=12)),
               layer(memory("retention", heads=2, dim=8, vdim=4), None)], width=32, vocab=61, loop=(0, 2, 2))
#: values that a model may happen to make equal or one: one head, one expert, one group, a factor of one, decays of one and of
#: nearly nothing, a chunk of one token, no loop; a width and a vocabulary that fit no vector access
PLAIN = config([layer(memory("lightning", heads=1, dim=16, vdim=16, decay=[1.0]), dense(50)),
                layer(attention(heads=1, kv_heads=1, dim=16, vdim=16, scale=1.0, size=1, dims=16, scaling=(1.0, 1.0, 1.0, 16.0)),
                      moe(ff=18, experts=1, top=1, groups=(1, 1), shared=18)),
                layer(memory("retention", heads=1, dim=1, vdim=3, decay=[1e-3]), moe(ff=10, experts=4, top=4, groups=(4, 4), shared=6)),
                layer(attention(heads=2, kv_heads=2, dim=8, vdim=8, size=None, dims=2, base=1.5, scaling=(2.0, 0.5, 0.5, 9.0)), None),
                layer(memory("retention", heads=3, dim=7, vdim=5, decay=[1.0, 0.0, 0.9]), dense(33))], width=66, vocab=91)
#: the same for bfloat16: a head of one key element that forgets at once reads nothing but the sign of q times k, which is no
#: matter of rounding
PLAIN_16 = config(PLAIN["layers"][:2] + [layer(memory("retention", heads=1, dim=9, vdim=3, decay=[0.95]), PLAIN["layers"][2]["mlp"])] + PLAIN["layers"][3:4],
                  width=66, vocab=91)
#: sizes of the serving kernels (the tensor cores for bfloat16: head sizes of 64 and 128 in the attention, states that the
#: chunked form takes, also with padding on both sides)
SERVING_HEADS = config([layer(attention(heads=6, kv_heads=2, dim=64, vdim=64, scale=0.12, size=90, dims=48, base=1e4, scaling=(4.0, 1.0, 4.0, 64.0)), dense(160)),
                        layer(memory("lightning", heads=3, dim=64, vdim=128), moe(ff=64, experts=16, top=4, groups=(4, 2), shared=96)),
                        layer(memory("retention", heads=2, dim=128, vdim=72, decay=[0.8, 0.996]), dense(96)),
                        layer(attention(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.08, size=64, dims=128, base=1e4), None),
                        layer(memory("lightning", heads=4, dim=24, vdim=40), moe(ff=40, experts=6, top=2, groups=(2, 1), shared=32)),
                        layer(memory("retention", heads=2, dim=200, vdim=64), dense(64))], width=128, vocab=300, loop=(1, 3, 2))
#: one kind of mixer, and one kind of feed-forward, alone
ONE = {"attention": config([layer(attention())] * 2), "lightning": config([layer(memory("lightning"))] * 2),
       "retention": config([layer(memory("retention"))] * 2),
       "experts": config([layer(memory("retention", heads=1, dim=4, vdim=4), moe())] * 2, loop=(1, 2, 2))}


def write_model(folder: str, cfg: dict, seed: int = 0, dtype=torch.float32, std: float = 0.12, planted_routes: bool = False) -> str:
    """A model folder whose small parameters are far from their neutral values: norm weights that differ, gates that open and
    shut, routers that spread their scores.

    With ``planted_routes`` no router's choice is a close call, so that a model in reduced precision chooses as the plain one
    does: the last channels of the width carry a code of the token that no sublayer writes to (their rows of the
    out-projections are zero), and each expert's router row reads one of these channels."""
    from vapi_b200.config.model import resolve_architecture
    from vapi_b200.weights import write_random_model
    arch = resolve_architecture(cfg)
    W, V = cfg["width"], cfg["vocab"]
    most = max([e["mlp"]["router"]["experts"] for e in cfg["layers"] if e["mlp"] and e["mlp"]["kind"] == "moe"] or [0])
    code = slice(W - most, W) if planted_routes and most > 0 else slice(0, 0)
    over = {}
    for s in arch.plan(arch.parse(cfg)).tensor_specs():
        g = torch.Generator().manual_seed(seed * 7919 + zlib.crc32(s.name.encode()) % 100003)
        tail = ".".join(s.name.split(".")[1:])
        if tail in ("norm1", "norm", "mix.norm"):
            t = 1.0 + 0.3 * torch.randn(s.shape, generator=g)
            if tail != "mix.norm":
                t[code] = 1.0
        elif tail in ("mlp.router", "mlp.shared.sg"):
            t = (0.004 if planted_routes and tail == "mlp.router" else 0.3) * torch.randn(s.shape, generator=g)
            if planted_routes and tail == "mlp.router":
                for e in range(s.shape[0]):
                    t[e, W - most + e] = 2.0
        elif s.name == "embed":
            t = 0.5 * torch.randn(s.shape, generator=g)
            if code.stop > 0:             # channel j of token t holds ((t + j) mod most) in steps of a quarter, around zero
                step = (torch.arange(V)[:, None] + torch.arange(most)[None, :]) % most
                t[:, code] = (step.float() - (most - 1) / 2) * 0.25
        elif s.name.endswith((".o", ".down")):
            t = std * torch.randn(s.shape, generator=g)
            t[code] = 0.0
        else:
            continue
        over[s.name] = t
    return write_random_model(folder, cfg, seed, std=std, norm_init="perturbed", dtype=dtype, overrides=over)


prompt = givavik_util.prompt
batch = givavik_util.batch
step_index = givavik_util.step_index
within = givavik_util.within


class Oracle(givavik_util.Oracle):
    """The plain model on a folder, float64 (the error measures are those of the other models)."""
    model = plain
