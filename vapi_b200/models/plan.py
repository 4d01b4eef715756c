"""A model as data: parts, their tensor names, and the order in which layers run."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..parts.base import Norm, Part, PositionEncoding, TensorSpec
from ..parts.embedding import OutputHead, TokenEmbedding


@dataclass(frozen=True)
class LayerCall:
    """One entry of the run order.

    ``layer`` indexes ``ModelPlan.layers`` (a layer may be named more than once: its weights
    are shared, each call site has a cache of its own).  ``cache_of`` = k makes this call
    site read the cache that call site k owns instead of having one (k < this index, and
    that site's mixer must want the same kind of cache).  ``before`` names an entry of ``ModelPlan.stream_parts``
    that acts on the residual stream right before this call (a looped stack's input product).
    """

    layer: int
    cache_of: Optional[int] = None
    before: Optional[str] = None


def looped_order(n_layers: int, loop: Optional[Tuple[int, int, int]], before: Optional[str] = None) -> List[LayerCall]:
    """Every layer once, but those of ``loop`` = (start, stop, times) that many times in a row (each pass with caches of its
    own), each pass led by the stream part ``before`` names."""
    if loop is None:
        return [LayerCall(i) for i in range(n_layers)]
    a, b, times = loop
    order = [LayerCall(i) for i in range(a)]
    for _ in range(times):
        order += [LayerCall(i, before=before if i == a else None) for i in range(a, b)]
    return order + [LayerCall(i) for i in range(b, n_layers)]


@dataclass
class ModelPlan:
    architecture: str
    vocab_size: int
    hidden_size: int
    max_positions: int
    embedding: TokenEmbedding
    layers: List[Part]                 # blocks
    layer_prefixes: List[str]          # checkpoint prefix of each block, e.g. "model.layers.3."
    order: List[LayerCall]
    final_norm: Norm
    final_norm_prefix: str
    head: OutputHead
    position_encodings: List[PositionEncoding] = field(default_factory=list)
    eos_token_ids: Tuple[int, ...] = ()
    config: Any = None
    #: parts that act on the whole stream between layers (``part.forward(x, pending, ctx) -> (x, pending)``), by the
    #: key that ``LayerCall.before`` names; their tensors carry no layer prefix
    stream_parts: Dict[str, Part] = field(default_factory=dict)

    def __post_init__(self) -> None:
        if len(self.layers) != len(self.layer_prefixes):
            raise ValueError("one checkpoint prefix per layer is needed")
        for i, c in enumerate(self.order):
            if not 0 <= c.layer < len(self.layers):
                raise ValueError(f"run order entry {i} names layer {c.layer} of {len(self.layers)}")
            if c.before is not None and c.before not in self.stream_parts:
                raise ValueError(f"run order entry {i} names the stream part `{c.before}`, which the plan does not have")
            if c.cache_of is not None:
                if not 0 <= c.cache_of < i or self.order[c.cache_of].cache_of is not None:
                    raise ValueError(f"run order entry {i}: cache_of must name an earlier entry that owns its cache")
                a = self.layers[c.layer].mixer.cache_spec()
                b = self.layers[self.order[c.cache_of].layer].mixer.cache_spec()
                if a != b:
                    raise ValueError(f"run order entry {i} cannot read the cache of entry {c.cache_of}: {a} != {b}")

    # ---- tensors -------------------------------------------------------------------
    def tensor_specs(self) -> List[TensorSpec]:
        specs: List[TensorSpec] = list(self.embedding.tensor_specs(""))
        for blk, pre in zip(self.layers, self.layer_prefixes):
            specs += blk.tensor_specs(pre)
        specs += self.final_norm.tensor_specs(self.final_norm_prefix)
        specs += self.head.tensor_specs("")
        for pe in self.position_encodings:
            specs += pe.tensor_specs("")
        for part in self.stream_parts.values():
            specs += part.tensor_specs("")
        seen: Dict[str, TensorSpec] = {}
        for s in specs:
            if s.name in seen and seen[s.name].shape != s.shape:
                raise ValueError(f"tensor `{s.name}` is wanted with two shapes")
            seen[s.name] = s
        return list(seen.values())

    def bind(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype) -> None:
        self.embedding.bind(tensors, "", dtype)
        for blk, pre in zip(self.layers, self.layer_prefixes):
            blk.bind(tensors, pre, dtype)
        self.final_norm.bind(tensors, self.final_norm_prefix, dtype)
        self.head.bind(tensors, "", dtype)
        for pe in self.position_encodings:
            pe.bind(tensors, "", dtype)
        for part in self.stream_parts.values():
            part.bind(tensors, "", dtype)

    # ---- caches --------------------------------------------------------------------
    def cache_sites(self) -> List[Tuple[object, object]]:
        """(site, spec) of every cache that a call site owns.  A site is the call site's index in the run
        order, or ``(index, member)`` for each member of a mixer that is several mixers side by side (its
        ``cache_spec`` is a tuple); what a block keeps for itself is ``("block", index)``, whoever owns its mixer's
        cache, and what the embedding keeps ``"embedding"``."""
        out = []
        spec = self.embedding.block_cache_spec()
        if spec is not None:
            out.append(("embedding", spec))
        for i, c in enumerate(self.order):
            spec = self.layers[c.layer].block_cache_spec()
            if spec is not None:
                out.append((("block", i), spec))
            if c.cache_of is None:
                spec = self.layers[c.layer].mixer.cache_spec()
                if isinstance(spec, tuple):
                    out += [((i, j), sp) for j, sp in enumerate(spec) if sp is not None]
                elif spec is not None:
                    out.append((i, spec))
        return out
