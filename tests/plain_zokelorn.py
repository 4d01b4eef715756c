"""Zokelorn, plainly: one function per mechanism, loops over tokens, float64 by default.

Nothing here is shared with the package: the folder is read with a few lines of its own, the model is
a function of (configuration, weights, tokens) without cache or state, and every mechanism is
written from its equations.

The model.  ``x = embed[token]``.  A layer is parallel: ``h = norm(x)``; ``x <- x + mixer(h) + ff(h)``.  The mixer is
grouped-query attention within chunks of positions (interleaved rotary pairs whose slow frequencies are stretched, a
sigmoid gate per head), lightning attention or retention (both a decayed sum of outer products per head, with a fixed
decay).  The feed-forward is a gated one with the tanh form of GELU, a mixture of SiLU-gated experts behind a sigmoid
router with grouped choice and a gated shared expert, or absent.  A run of layers may be passed several times.  The model
ends on a norm and a matrix of its own.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Any, Dict, List, Optional, Sequence, Tuple

import torch

_DT = {"F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16, "F64": torch.float64, "I32": torch.int32,
       "I64": torch.int64}


def read_config(folder: str) -> Dict[str, Any]:
    with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as f:
        return json.load(f)


def read_weights(folder: str, dtype=torch.float64) -> Dict[str, torch.Tensor]:
    """Eight bytes of length, that much json (name -> dtype, shape, data_offsets), then the data."""
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        lo, hi = e["data_offsets"]
        t = torch.frombuffer(bytearray(data[lo:hi]), dtype=_DT[e["dtype"]]).reshape(e["shape"])
        out[name] = t.to(dtype) if t.dtype.is_floating_point else t
    return out


# ---- small functions ----------------------------------------------------------------------------------

def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


# ---- rotation -------------------------------------------------------------------------------------------

def frequencies(rot: Dict[str, Any]) -> List[float]:
    """One per pair: short wavelengths stay, long ones are stretched by ``factor``, those between are a blend."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wavelength = 2.0 * math.pi / f
            if wavelength < sc["original"] / sc["high"]:
                pass
            elif wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(x: torch.Tensor, p: int, freqs: Sequence[float]) -> torch.Tensor:
    """x [..., n]: element 2i turns with element 2i + 1 by p * freqs[i]; what lies behind the pairs stays."""
    out = x.clone()
    for i, f in enumerate(freqs):
        c, s = math.cos(p * f), math.sin(p * f)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---- attention ------------------------------------------------------------------------------------------

def visible(i: int, chunk: Optional[int]) -> Tuple[int, int]:
    """Position i sees the positions from the first of these to the second, both included."""
    return (0 if not chunk else (i // chunk) * chunk), i


def attention(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).reshape(T, H, d)
    k = (h @ w[pre + "k"].T).reshape(T, G, d)
    v = (h @ w[pre + "v"].T).reshape(T, G, dv)
    gate = sigmoid(h @ w[pre + "g"].T)
    if m.get("rot"):
        fs = frequencies(m["rot"])
        q = torch.stack([rotate_pairs(q[t], t, fs) for t in range(T)])
        k = torch.stack([rotate_pairs(k[t], t, fs) for t in range(T)])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        a, b = visible(t, (m.get("mask") or {}).get("size"))
        for n in range(H):
            g = n // (H // G)
            s = (k[a:b + 1, g] @ q[t, n]) * float(m["scale"])
            e = torch.exp(s - s.max())
            out[t, n] = ((e / e.sum()) @ v[a:b + 1, g]) * gate[t, n]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


# ---- a decayed sum of outer products ------------------------------------------------------------------------

def decayed_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: Sequence[float]) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv]: S_t = decay_h S_{t-1} + k_t v_t^T from zero; returns S_t^T q_t [T, H, dv]."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for n in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=q.dtype)
        for t in range(T):
            S = float(decay[n]) * S + torch.outer(k[t, n], v[t, n])
            out[t, n] = S.T @ q[t, n]
    return out


def lightning(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ w[pre + "q"].T).reshape(T, H, d), silu(h @ w[pre + "k"].T).reshape(T, H, d)
    v = silu(h @ w[pre + "v"].T).reshape(T, H, dv)
    o = decayed_memory(q, k, v, m["decay"]).reshape(T, H * dv)
    return (norm(o, w[pre + "norm"], eps) * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def retention(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (h @ w[pre + "q"].T).reshape(T, H, d), (h @ w[pre + "k"].T).reshape(T, H, d) * d ** -0.5
    v = (h @ w[pre + "v"].T).reshape(T, H, dv)
    o = unit_rms(decayed_memory(q, k, v, m["decay"]), eps).reshape(T, H * dv)
    return (o * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- feed-forwards ------------------------------------------------------------------------------------------

def dense(w: Dict[str, torch.Tensor], pre: str, h: torch.Tensor) -> torch.Tensor:
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def expert(w: Dict[str, torch.Tensor], pre: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def choose(z: torch.Tensor, r: Dict[str, Any]) -> Tuple[List[int], torch.Tensor]:
    """z [experts]: one token's router logits.  The chosen experts, best first, and their weights."""
    s = sigmoid(z)
    E = s.numel()
    groups = r.get("groups") or {"count": 1, "keep": 1}
    C = int(groups["count"])
    per = E // C
    value = [float(torch.sort(s[c * per:(c + 1) * per], descending=True).values[:2].sum()) for c in range(C)]
    best = sorted(range(C), key=lambda c: (-value[c], c))[:int(groups["keep"])]
    open_to = [e for e in range(E) if e // per in best]
    chosen = sorted(open_to, key=lambda e: (-float(s[e]), e))[:int(r["top"])]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def mixture(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor) -> torch.Tensor:
    out = torch.zeros_like(h)
    z = h @ w[pre + "router"].T
    for t in range(h.shape[0]):
        for e, p in zip(*choose(z[t], m["router"])):
            out[t] += p * expert(w, f"{pre}e{e}.", h[t])
    if m.get("shared"):
        out = out + expert(w, pre + "shared.", h) * sigmoid(h @ w[pre + "shared.sg"].T)
    return out


# ---- the model ------------------------------------------------------------------------------------------------

def run_order(cfg: Dict[str, Any]) -> List[int]:
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def layer(cfg, w, i: int, x: torch.Tensor) -> torch.Tensor:
    e, eps, pre = cfg["layers"][i], float(cfg["norm"]["eps"]), f"l{i}."
    h = norm(x, w[pre + "norm1"], eps)
    m = e["mixer"]
    if e["type"] == "attention":
        mix = attention(w, pre + "mix.", m, h)
    elif e["type"] == "lightning":
        mix = lightning(w, pre + "mix.", m, h, eps)
    elif e["type"] == "retention":
        mix = retention(w, pre + "mix.", m, h, eps)
    else:
        raise ValueError(e["type"])
    f = e.get("mlp")
    if f is None:
        return x + mix
    return x + (mix + (dense(w, pre + "mlp.", h) if f["kind"] == "dense" else mixture(w, pre + "mlp.", f, h)))


def forward(cfg: Dict[str, Any], w: Dict[str, torch.Tensor], tokens: Sequence[int], keep_layers: bool = False):
    """Logits [T, vocab] of one sequence from position 0; with ``keep_layers`` also the stream after every layer run."""
    x = w["embed"][list(tokens)]
    kept = []
    for i in run_order(cfg):
        x = layer(cfg, w, i, x)
        kept.append(x)
    logits = norm(x, w["final.norm"], float(cfg["norm"]["eps"])) @ w["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits
