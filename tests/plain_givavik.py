"""Givavik, plainly: one function per mechanism, loops over tokens, float64 by default.

Nothing here is shared with the package: the folder is read with a few lines of its own, the model is
a function of (configuration, weights, tokens) without cache or state, and every mechanism is
written from its equations.

The model.  ``x = embed[token] * embedding.scale``, plus a row of a second table picked by a hash of the token and
the one before it.  A layer is parallel: ``h = norm(x)``; ``x <- x + ls1 * mixer(s) + ls2 * ff(h)`` where s_t mixes
h_t with h_{t-1} element by element (token shift).  The mixer is latent attention with a sink (a layer may read an
earlier layer's latents) or two mixers side by side whose results are added with fixed factors: grouped-query
attention whose weights are sigmoids of capped scores, not normalised over the keys, and Mamba-2.  The feed-forward
is one hidden layer with the xIELU activation, or absent.  Norm weights are stored around zero.  The model ends on
such a norm and a matrix of its own.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Any, Dict, Sequence

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


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * (1.0 + w)


def rotate_pairs(x: torch.Tensor, p: int, dims: int, base: float) -> torch.Tensor:
    """x [..., n]: its first ``dims`` elements turn, element 2i with element 2i + 1, by p * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---- the embedding --------------------------------------------------------------------------------------

def bigram_row(prev: int, cur: int, b: Dict[str, Any]) -> int:
    """Which row of the second table joins the token ``cur`` that follows ``prev``."""
    return (prev * int(b["mul_prev"]) + cur * int(b["mul_cur"])) % int(b["buckets"])


def embedding(cfg: Dict[str, Any], w: Dict[str, torch.Tensor], tokens: Sequence[int]) -> torch.Tensor:
    e = cfg["embedding"]
    rows = []
    for t, tok in enumerate(tokens):
        r = w["embed"][tok] * float(e["scale"])
        b = e.get("bigram")
        if b:
            r = r + w["bigram"][int(b["buckets"]) if t == 0 else bigram_row(tokens[t - 1], tok, b)]
        rows.append(r)
    return torch.stack(rows)


# ---- token shift ----------------------------------------------------------------------------------------

def token_shift(h: torch.Tensor, amount: torch.Tensor) -> torch.Tensor:
    """h [T, width] from position 0: every token's h moves towards the one before it (zeros before the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    return h + (before - h) * amount


# ---- latent attention -------------------------------------------------------------------------------------

def latent_rows(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], s: torch.Tensor, eps: float):
    """What a layer's cache holds: the normed latents [T, kv_rank] and the rotated key parts [T, rot_dim]."""
    R, T = int(m["kv_rank"]), s.shape[0]
    kv = s @ w[pre + "dkv"].T
    c = unit_rms(kv[:, :R], eps) * w[pre + "dkv.norm"]
    kr = torch.stack([rotate_pairs(kv[t, R:], t, int(m["rot"]["dims"]), float(m["rot"]["base"])) for t in range(T)])
    return c, kr


def latent_attention(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], s: torch.Tensor, c: torch.Tensor,
                     kr: torch.Tensor) -> torch.Tensor:
    """s [T, width] is the mixer's input; c and kr may come from an earlier layer."""
    T, H, d, r, dv = s.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (s @ w[pre + "q"].T).reshape(T, H, d + r)
    kn = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=s.dtype)
    for t in range(T):
        qr = rotate_pairs(q[t, :, d:], t, int(m["rot"]["dims"]), float(m["rot"]["base"]))
        for a in range(H):
            sc = (kn[: t + 1, a] @ q[t, a, :d] + kr[: t + 1] @ qr[a]) * float(m["scale"])
            sink = w[pre + "sink"][a]
            top = torch.maximum(sc.max(), sink)
            e = torch.exp(sc - top)
            out[t, a] = (e / (e.sum() + torch.exp(sink - top))) @ v[: t + 1, a]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


# ---- attention with sigmoid weights -------------------------------------------------------------------------

def sigmoid_attention(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], s: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, d, dv = s.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (s @ w[pre + "q"].T + w[pre + "q.b"]).reshape(T, H, d)
    k = (s @ w[pre + "k"].T + w[pre + "k.b"]).reshape(T, G, d)
    v = (s @ w[pre + "v"].T + w[pre + "v.b"]).reshape(T, G, dv)
    rot = m.get("rot")
    if rot:
        q = torch.stack([rotate_pairs(q[t], t, int(rot["dims"]), float(rot["base"])) for t in range(T)])
        k = torch.stack([rotate_pairs(k[t], t, int(rot["dims"]), float(rot["base"])) for t in range(T)])
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    cap = m.get("softcap")
    out = torch.zeros(T, H, dv, dtype=s.dtype)
    for t in range(T):
        for a in range(H):
            g = a // (H // G)
            sc = (k[: t + 1, g] @ q[t, a]) * float(m["scale"])
            if cap:
                sc = float(cap) * torch.tanh(sc / float(cap))
            out[t, a] = sigmoid(sc + w[pre + "pb"][a]) @ v[: t + 1, g]
    return out.reshape(T, H * dv) @ w[pre + "o"].T + w[pre + "o.b"]


# ---- Mamba-2 ------------------------------------------------------------------------------------------------

def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, L]: the last column is the current token's; zeros before the start."""
    T = x.shape[0]
    L = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = bias.clone()
        for j in range(L):
            u = t - (L - 1) + j
            if u >= 0:
                acc = acc + taps[:, j] * x[u]
        out[t] = acc
    return out


def mamba2(w: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], s: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, P, N, G, K = s.shape[0], m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"]
    inner = H * P
    p = s @ w[pre + "in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    step = softplus(dt + w[pre + "dt_bias"])                       # [T, H]
    y = torch.zeros(T, H, P, dtype=s.dtype)
    S = torch.zeros(H, N, P, dtype=s.dtype)
    for t in range(T):
        for a in range(H):
            g = a // (H // G)
            S[a] = torch.exp(-torch.exp(w[pre + "A_log"][a]) * step[t, a]) * S[a] + step[t, a] * torch.outer(B[t, g], x[t, a])
            y[t, a] = C[t, g] @ S[a] + w[pre + "D"][a] * x[t, a]
    u = (y.reshape(T, inner) * silu(z)).reshape(T, K, inner // K)
    return (unit_rms(u, eps).reshape(T, inner) * w[pre + "norm"]) @ w[pre + "o"].T


# ---- the feed-forward ---------------------------------------------------------------------------------------

def xielu(z: torch.Tensor, act: torch.Tensor) -> torch.Tensor:
    up, down = softplus(act[0]), 0.5 + softplus(act[1])
    low = torch.clamp(z, max=0.0)
    return torch.where(z > 0, up * z * z + 0.5 * z, down * (torch.expm1(low) - low) + 0.5 * z)


def feed_forward(w: Dict[str, torch.Tensor], pre: str, h: torch.Tensor) -> torch.Tensor:
    return xielu(h @ w[pre + "up"].T, w[pre + "act"]) @ w[pre + "down"].T


# ---- the model ------------------------------------------------------------------------------------------------

def layer(cfg, w, i: int, x: torch.Tensor, latents: Dict[int, tuple]) -> torch.Tensor:
    """One layer; ``latents`` collects what each latent layer's cache holds, for layers that read another's."""
    e, eps, pre = cfg["layers"][i], float(cfg["norm"]["eps"]), f"l{i}."
    m = e["mixer"]
    h = zero_centred_norm(x, w[pre + "norm1"], eps)
    s = token_shift(h, w[pre + "shift"])
    if e["type"] == "latent_attention":
        source = m.get("kv_from")
        if source is None:
            latents[i] = latent_rows(w, pre + "mix.", m, s, eps)
            source = i
        mix = latent_attention(w, pre + "mix.", m, s, *latents[source])
    elif e["type"] == "parallel":
        mix = (float(m["left_scale"]) * sigmoid_attention(w, pre + "mix.left.", m["left"], s, eps)
               + float(m["right_scale"]) * mamba2(w, pre + "mix.right.", m["right"], s, eps))
    else:
        raise ValueError(e["type"])
    x = x + mix * w[pre + "ls1"]
    if e.get("mlp") is not None:
        x = x + feed_forward(w, pre + "mlp.", h) * w[pre + "ls2"]
    return x


def forward(cfg: Dict[str, Any], w: Dict[str, torch.Tensor], tokens: Sequence[int], keep_layers: bool = False):
    """Logits [T, vocab] of one sequence from position 0; with ``keep_layers`` also the stream after every layer."""
    x = embedding(cfg, w, tokens)
    kept, latents = [], {}
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x, latents)
        kept.append(x)
    logits = zero_centred_norm(x, w["final.norm"], float(cfg["norm"]["eps"])) @ w["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits
