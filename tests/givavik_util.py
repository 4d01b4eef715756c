"""Small Givavik configurations and model folders whose small parameters make faults show."""
from __future__ import annotations

import zlib
from typing import Dict, Optional, Sequence

import numpy as np
import torch

import plain_givavik as plain


def latent(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=24, scale=0.25, base=100.0, kv_from: Optional[int] = None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def left(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, softcap: Optional[float] = 1.5, dims=12, base=50.0) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if softcap is not None:
        m["softcap"] = softcap
    return m


def right(heads=6, vdim=10, state=20, groups=3, conv=3, norm_groups=2) -> dict:
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(le: Optional[dict] = None, ri: Optional[dict] = None, left_scale=0.7, right_scale=1.4) -> dict:
    return {"type": "parallel", "mixer": {"left": le or left(), "right": ri or right(), "left_scale": left_scale,
                                          "right_scale": right_scale}}


def layer(mixer: dict, ff: Optional[int] = 72) -> dict:
    return {**mixer, "mlp": {"kind": "dense", "ff": ff} if ff is not None else None}


def config(layers: Sequence[dict], width=64, vocab=200, scale=1.7, bigram=(37, 91, 13), eps=1e-5) -> dict:
    e: Dict[str, object] = {"scale": scale}
    if bigram is not None:
        e["bigram"] = {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    return {"architecture": "Givavik", "embedding": e, "layers": list(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width}


#: sizes that all differ from one another: two layers share the first one's latents (with heads of other counts and
#: sizes), a layer without a feed-forward, a cap that bites, unlike key and value widths, three state groups
MIXED = config([layer(parallel()),
                layer(latent(), ff=40),
                layer(latent(heads=2, dim=20, vdim=16, scale=0.3, kv_from=1), ff=None),
                layer(parallel(left(heads=3, kv_heads=3, dim=24, vdim=16, scale=0.2, softcap=0.9, dims=24, base=7.0),
                               right(heads=2, vdim=40, state=12, groups=1, conv=5, norm_groups=4), 1.3, 0.6), ff=136),
                layer(latent(heads=5, dim=8, rot_dim=12, vdim=12, kv_rank=40, base=7.0)),
                layer(latent(heads=4, dim=16, vdim=8, scale=0.2, kv_from=1), ff=24)])
#: tiny, for runs where plain Python stands in for the kernels
TINY = config([layer(latent(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=12), ff=16),
               layer(parallel(left(heads=2, kv_heads=1, dim=8, vdim=12, dims=4), right(heads=2, vdim=8, state=8, groups=1, conv=3, norm_groups=1)), ff=None),
               layer(latent(heads=3, dim=12, rot_dim=4, vdim=4, kv_rank=12, kv_from=0), ff=24)], width=32, vocab=61, bigram=(17, 5, 3))
#: values that a model may happen to make equal or one: one head, one group, one tap, factors and scale of one, no cap,
#: no second table; a width and a vocabulary that fit no vector access
PLAIN = config([layer(parallel(left(heads=1, kv_heads=1, dim=16, vdim=16, scale=1.0, softcap=None, dims=16),
                               right(heads=1, vdim=16, state=16, groups=1, conv=1, norm_groups=1), 1.0, 1.0), ff=64),
                layer(latent(heads=1, dim=16, rot_dim=16, vdim=16, kv_rank=16), ff=50)], width=66, vocab=91, scale=1.0, bigram=None)
#: the head sizes of the serving kernels (keys and values of 64 and of 128, latent rows of 80 and 160: tensor cores for
#: bfloat16); no two sizes alike where the kernels allow it
SERVING_HEADS = config([layer(parallel(left(heads=6, kv_heads=2, dim=64, vdim=64, scale=0.12, softcap=30.0, dims=48, base=1e4),
                                       right(heads=4, vdim=64, state=64, groups=2, conv=4, norm_groups=2)), ff=160),
                        layer(latent(heads=4, dim=32, rot_dim=16, vdim=48, kv_rank=64, scale=0.14), ff=96),
                        layer(parallel(left(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.08, softcap=2.0, dims=128, base=1e4),
                                       right(heads=2, vdim=32, state=32, groups=1, conv=2, norm_groups=1), 1.5, 0.5), ff=None),
                        layer(latent(heads=3, dim=48, rot_dim=16, vdim=32, kv_rank=64, scale=0.1, kv_from=1), ff=64),
                        layer(latent(heads=2, dim=64, rot_dim=32, vdim=64, kv_rank=128, scale=0.1), ff=64)], width=128, vocab=300)
#: one kind of mixer alone
ONE = {"latent": config([layer(latent())] * 2), "parallel": config([layer(parallel())] * 2),
       "shared": config([layer(latent()), layer(latent(heads=2, dim=16, vdim=16, kv_from=0))], bigram=(11, 1, 0))}


def write_model(folder: str, cfg: dict, seed: int = 0, dtype=torch.float32, std: float = 0.12) -> str:
    """A model folder whose small parameters are far from their neutral values: norm weights and layer scales that
    differ, shifts between nothing and all of the token before, sinks and score biases that matter, decays from fast to
    slow, convolutions with a bias, a second embedding table as strong as the first."""
    from vapi_b200.config.model import resolve_architecture
    from vapi_b200.weights import write_random_model
    arch = resolve_architecture(cfg)
    over = {}
    for s in arch.plan(arch.parse(cfg)).tensor_specs():
        g = torch.Generator().manual_seed(seed * 7919 + zlib.crc32(s.name.encode()) % 100003)
        tail = ".".join(s.name.split(".")[1:])
        if tail in ("ls1", "ls2"):
            over[s.name] = 0.7 + 0.5 * torch.rand(s.shape, generator=g)
        elif tail == "shift":
            over[s.name] = torch.rand(s.shape, generator=g)
        elif tail in ("norm1", "norm") and s.name != "norm":
            over[s.name] = 0.2 * torch.randn(s.shape, generator=g)
        elif tail in ("mix.sink", "mix.left.pb", "mlp.act"):
            over[s.name] = torch.randn(s.shape, generator=g)
        elif tail == "mix.right.A_log":
            over[s.name] = torch.rand(s.shape, generator=g) * 2.5 - 1.0
        elif tail == "mix.right.dt_bias":
            over[s.name] = torch.randn(s.shape, generator=g)
        elif tail == "mix.right.D":
            over[s.name] = 1.0 + 0.5 * torch.randn(s.shape, generator=g)
        elif tail == "mix.right.conv":
            over[s.name] = 0.5 * torch.randn(s.shape, generator=g)
        elif tail.endswith(".b"):
            over[s.name] = 0.3 * torch.randn(s.shape, generator=g)
        elif s.name in ("embed", "bigram"):
            over[s.name] = 0.5 * torch.randn(s.shape, generator=g)
    return write_random_model(folder, cfg, seed, std=std, norm_init="perturbed", dtype=dtype, overrides=over)


def prompt(cfg: dict, n: int, seed: int):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


class Oracle:
    """The plain model on a folder, float64."""
    model = plain

    def __init__(self, folder: str):
        self.cfg = self.model.read_config(folder)
        self.w = self.model.read_weights(folder, torch.float64)
        self._memo: Dict[tuple, object] = {}

    def logits(self, tokens: Sequence[int]) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._memo:
            self._memo[key] = self.model.forward(self.cfg, self.w, tokens)
        return self._memo[key]

    def rounding(self, tokens: Sequence[int], dtype: str = "float32") -> np.ndarray:
        """What reduced precision alone does to each position's logits, as a part of the logits' range.  float32: the
        plain model in float32 against itself in float64, the larger of two draws (the weights as they are, and once
        with every element moved by up to 2^-23 of itself).  bfloat16: the plain model with every matrix moved by up to
        2^-8 of each element against itself."""
        key = (dtype,) + tuple(tokens)
        if key not in self._memo:
            want = self.logits(tokens)
            g = torch.Generator().manual_seed(99)

            def moved(by, to):
                return {k: (v * (1.0 + by * (2.0 * torch.rand(v.shape, generator=g, dtype=v.dtype) - 1.0))).to(to)
                        if v.dim() >= 2 or to == torch.float32 else v for k, v in self.w.items()}
            if dtype == "float32":
                draws = [self.model.forward(self.cfg, moved(by, torch.float32), tokens).double() for by in (0.0, 2.0 ** -23)]
            else:
                draws = [self.model.forward(self.cfg, moved(2.0 ** -8, torch.float64), tokens)]
            err = torch.stack([(got - want).abs().amax(-1) for got in draws]).amax(0)
            self._memo[key] = (err / float(want.max() - want.min())).numpy()
        return self._memo[key]

    def greedy(self, tokens: Sequence[int], n: int):
        toks, out = list(tokens), []
        for _ in range(n):
            t = int(torch.argmax(self.logits(toks)[-1]))
            out.append(t)
            toks.append(t)
        return out


def batch(lens: Sequence[int], klens: Sequence[int], page: int, row: int, seed: int, dtype=torch.float32, spread: float = 0.5):
    """A paged cache of random rows (``row`` elements a token) for sequences with ``lens`` new tokens over ``klens`` keys,
    its pages taken in a scrambled order: (cache, block table, cu_q, seqlens_k)."""
    g = torch.Generator().manual_seed(seed)
    pages = sum(-(-k // page) for k in klens)
    cache = (torch.randn((pages + 2, page * row), generator=g) * spread).to(dtype)
    order = torch.randperm(pages + 2, generator=g).to(torch.int32)
    table = torch.zeros((len(klens), max(-(-k // page) for k in klens)), dtype=torch.int32)
    at = 0
    for s, k in enumerate(klens):
        m = -(-k // page)
        table[s, :m] = order[at:at + m]
        at += m
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    return cache, table, cu, torch.tensor(klens, dtype=torch.int32)


def step_index(lens: Sequence[int], starts: Sequence[int], slots: Sequence[int]):
    """What a step knows of its tokens: (cu_q, tok_seq, positions, state_slots) for sequences that bring ``lens`` tokens
    from positions ``starts``."""
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    seq = torch.tensor([s for s, n in enumerate(lens) for _ in range(n)], dtype=torch.int32)
    pos = torch.tensor([p + i for n, p in zip(lens, starts) for i in range(n)], dtype=torch.int32)
    return cu, seq, pos, torch.tensor(slots, dtype=torch.int32)


def within(e, slack, dtype: str, what: str, limit: float) -> None:
    """``e``: errors as parts of the logit range; ``slack``: what reduced precision alone does to the plain model at the
    same positions.  An error counts as far as it exceeds three times that."""
    e, slack = np.asarray(e, dtype=np.float64), np.asarray(slack, dtype=np.float64)
    assert np.isfinite(e).all(), what
    if dtype == "bfloat16":
        ex = np.maximum(0.0, e - 3.0 * slack)
        assert ex.mean() <= 0.01 and ex.max() <= limit, f"{what}: mean {ex.mean():.3e}, worst {ex.max():.3e} at {int(ex.argmax())}"
    else:
        over = e - np.maximum(limit, 3.0 * slack)
        pos = int(over.argmax())
        assert over[pos] <= 0, f"{what}: {e[pos]:.3e} of the logit range at {pos} of {len(e)}"
