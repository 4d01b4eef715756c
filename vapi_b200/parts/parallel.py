"""Several mixers side by side on one input."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Sequence, Tuple

import torch

from .. import ops
from .base import CacheView, Mixer, TensorSpec, register_mixer


@dataclass
class DeferredBranches:
    """The branches' outputs before their norms and their mean: ``scale * sum_b rmsnorm(outs[b]) * weights[b]``.
    A block whose next kernel reads every row anyway (:class:`~vapi_b200.parts.hyper.HyperBlock`) takes the
    norms and the mean on there; :meth:`tensor` computes them with a kernel of their own."""

    outs: List[torch.Tensor]
    weights: List[torch.Tensor]
    eps: float
    scale: float

    def tensor(self) -> torch.Tensor:
        return ops.branch_rmsnorm_mean(self.outs, self.weights, self.eps, self.scale)


class ParallelMixer(Mixer):
    """``mean_b rmsnorm(branch_b(a)) * w_b``: every branch reads the same normed input; each output is
    RMS-normed over the model width with a plain weight of its own (``<sub_b><norm_name>``) and the results
    are averaged.  ``branches`` is a sequence of ``(sub-prefix, mixer)``.  Each branch keeps the cache it
    asks for: the mixer's ``cache_spec`` is the tuple of the branches' specs, and it is handed a ``multi``
    view with one part per branch.  With ``deferred`` (and at most two branches) ``forward`` returns a
    :class:`DeferredBranches` instead of a tensor, for a block that folds the norms and the mean into its next read.

    ``factors`` (one number per branch) stand in the norms' and the mean's place: ``sum_b factor_b * branch_b(a)``, and
    there are no norm tensors.  The branches must offer themselves in pieces (:meth:`Mixer.pieces`) and share two
    products: one in-projection with all branches' rows, and one out-projection over their inner results side by side,
    each already multiplied by its factor (in float32, before its one rounding).
    """

    def __init__(self, hidden: int, branches: Sequence[Tuple[str, Mixer]], eps: float = 0.0, norm_name: str = "out",
                 deferred: bool = False, factors: Optional[Sequence[float]] = None):
        if not 1 <= len(branches) <= 4:
            raise ValueError("one to four branches")
        self.hidden, self.eps, self.norm_name = int(hidden), float(eps), norm_name
        self.factors = [float(f) for f in factors] if factors is not None else None
        if self.factors is not None and (len(self.factors) != len(branches) or deferred):
            raise ValueError("one factor per branch, and no norms to defer")
        self.deferred = bool(deferred) and len(branches) <= 2
        self._joined = False
        self.w_in = self.b_in = self.w_out = self.b_out = None
        self.subs = [s for s, _ in branches]
        self.branches: List[Mixer] = [m for _, m in branches]
        self.weights: List[torch.Tensor] = []

    def members(self):
        return tuple(self.branches)

    def cache_spec(self):
        return tuple(m.cache_spec() for m in self.branches)

    def tensor_specs(self, prefix: str) -> List[TensorSpec]:
        out: List[TensorSpec] = []
        for sub, m in zip(self.subs, self.branches):
            out += m.tensor_specs(prefix + sub)
            if self.factors is not None:
                continue
            out.append(TensorSpec(f"{prefix}{sub}{self.norm_name}", (self.hidden,), role="vector", init="ones"))
        return out

    def bind(self, tensors, prefix, dtype):
        self.weights = []
        for sub, m in zip(self.subs, self.branches):
            m.bind(tensors, prefix + sub, dtype)
            if self.factors is not None:
                continue
            self.weights.append(tensors[f"{prefix}{sub}{self.norm_name}"].contiguous())

        if self.factors is not None:
            self._join()

    def _join(self) -> None:
        """The branches' projections as one in-product and one out-product."""
        pieces = [m.pieces() for m in self.branches]
        if any(p is None for p in pieces) or any(p.first for p in pieces[1:]):
            raise ValueError("factors need branches that offer their projections, at most one of which wants to lead the "
                             "product's rows, and that one first")

        def joined(ts, dim):
            wd = ts[0].dtype if all(t.dtype == ts[0].dtype for t in ts) else torch.float32
            return torch.cat([t.to(wd) for t in ts], dim)

        dev = pieces[0].w_in.device
        self._at, ins, at = [], [], 0
        for p in pieces:                                     # every branch's rows start at a multiple of eight
            rows = p.w_in.shape[0]
            self._at.append(at)
            ins.append(p.w_in if rows % 8 == 0 else
                       torch.cat([p.w_in, p.w_in.new_zeros((8 - rows % 8, self.hidden))], 0))
            at += ins[-1].shape[0]
        self.w_in = joined(ins, 0).contiguous()
        self.b_in = self.b_out = None
        if any(p.b_in is not None for p in pieces):
            self.b_in = torch.zeros(at, dtype=torch.float32, device=dev)
            for p, a in zip(pieces, self._at):
                if p.b_in is not None:
                    self.b_in[a:a + p.b_in.numel()] = p.b_in
        # the out-product's inner size is padded to a multiple of 32, which is what the decode products want
        widths = [p.w_out.shape[1] for p in pieces]
        pad = -sum(widths) % 32
        outs = [p.w_out for p in pieces] + ([pieces[0].w_out.new_zeros((self.hidden, pad))] if pad else [])
        self.w_out = joined(outs, 1).contiguous()
        self._pad, self._cols, c = pad, [], 0
        for w in widths:
            self._cols.append((c, c + w))
            c += w
        if any(p.b_out is not None for p in pieces):
            self.b_out = torch.zeros(self.hidden, dtype=torch.float32, device=dev)
            for p, f in zip(pieces, self.factors):
                if p.b_out is not None:
                    self.b_out += f * p.b_out
        self._joined = True
        for m in self.branches:
            m.give_up_projections()

    def _forward_joined(self, a: torch.Tensor, ctx: Any, views) -> torch.Tensor:
        h = ops.linear(a, self.w_in, self.b_in)
        y = torch.empty((a.shape[0], self.w_out.shape[1]), dtype=a.dtype, device=a.device)
        if self._pad:
            y[:, -self._pad:].zero_()                        # nothing but zeros may meet the padding's zeros
        for m, at, (c0, c1), f, v in zip(self.branches, self._at, self._cols, self.factors, views):
            m.inner(h, at, ctx, v, y[:, c0:c1], f)
        return ops.linear(y, self.w_out, self.b_out)

    def decode_splits(self, batch, max_context, page_size, dtype):
        return max(m.decode_splits(batch, max_context, page_size, dtype) for m in self.branches)

    def forward(self, a: torch.Tensor, ctx: Any, cache: CacheView) -> torch.Tensor:
        views = cache.parts if cache.kind == "multi" else [cache] * len(self.branches)
        if self._joined:
            return self._forward_joined(a, ctx, views)
        outs = [m.forward(a, ctx, v) for m, v in zip(self.branches, views)]
        if self.deferred:
            return DeferredBranches(outs, self.weights, self.eps, 1.0 / len(outs))
        return ops.branch_rmsnorm_mean(outs, self.weights, self.eps, 1.0 / len(outs))


register_mixer("parallel", ParallelMixer)
