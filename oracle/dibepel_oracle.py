"""Plain, slow CPU implementation of the Dibepel decoder, one function per mechanism, in the dtype of the
weights it is given (float32 or float64). Whole sequences only: no cache, no state, no batching. It is written
from the equations and shares no code with ``flashrec_b200``.

Notation: ``x [T, width]`` residual stream, ``h = norm1(x)``, positions ``i`` (query) and ``j`` (key) count from 0."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1 + w)


def short_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Depthwise causal convolution: y[t] = sum_j w[:, j] * u[t - taps + 1 + j], zeros before the start."""
    t, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for i in range(t):
        for j in range(taps):
            s = i - taps + 1 + j
            if s >= 0:
                y[i] += w[:, j] * u[s]
    return y


def window_mask(t: int, size: int, keep_first: int) -> torch.Tensor:
    """visible[i, j]: j <= i and (i - j < size or j < keep_first)."""
    i = torch.arange(t)[:, None]
    j = torch.arange(t)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def chunk_mask(t: int, size: int) -> torch.Tensor:
    """visible[i, j]: j <= i and both in the same chunk of ``size`` positions."""
    i = torch.arange(t)[:, None]
    j = torch.arange(t)[None, :]
    return (j <= i) & (i // size == j // size)


def distance_slope(h: int, heads: int) -> float:
    return 2.0 ** (-8.0 * (h + 1) / heads)


def softmax_weights(q: torch.Tensor, k: torch.Tensor, visible: torch.Tensor, scale: float, slope: float = 0.0):
    """One head's attention weights [T, T]: softmax over the visible keys of (q . k) * scale - slope * (i - j)."""
    t = q.shape[0]
    s = (q @ k.T) * scale
    if slope:
        dist = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).to(s.dtype)
        s = s - slope * dist
    s = s.masked_fill(~visible, float("-inf"))
    return torch.softmax(s, dim=-1)


def differential_lambda(lq1, lk1, lq2, lk2, diff: float) -> float:
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def differential_attention(q, k, v, mixer: dict, lam: float, eps: float) -> torch.Tensor:
    """q [T, H, 2, dim], k [T, G, 2, dim], v [T, G, vdim] -> [T, H * vdim]."""
    t, heads = q.shape[0], q.shape[1]
    rep = heads // k.shape[1]
    vis = window_mask(t, mixer["mask"]["size"], mixer["mask"]["keep_first"])
    out = []
    for h in range(heads):
        g = h // rep
        a1 = softmax_weights(q[:, h, 0], k[:, g, 0], vis, mixer["scale"]) @ v[:, g]
        a2 = softmax_weights(q[:, h, 1], k[:, g, 1], vis, mixer["scale"]) @ v[:, g]
        out.append(rms(a1 - lam * a2, eps) * (1 - mixer["diff"]))
    return torch.cat(out, dim=-1)


def talking_attention(q, k, v, mixer: dict, talk: torch.Tensor) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H * vdim]; the heads' weights are mixed by ``talk``."""
    t, heads = q.shape[0], q.shape[1]
    rep = heads // k.shape[1]
    vis = chunk_mask(t, mixer["mask"]["size"])
    w = torch.stack([softmax_weights(q[:, h], k[:, h // rep], vis, mixer["scale"], distance_slope(h, heads))
                     for h in range(heads)])
    out = []
    for h in range(heads):
        mixed = sum(talk[h, g] * w[g] for g in range(heads))
        out.append(mixed @ v[:, h // rep])
    return torch.cat(out, dim=-1)


def swiglu(h, gate, up, down):
    z = h @ gate.T
    return ((z / (1 + torch.exp(-z))) * (h @ up.T)) @ down.T


def sublayer_gate(h, w, b):
    return 1 / (1 + torch.exp(-(h @ w.T + b)))


def mixer_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, entry: dict, eps: float) -> torch.Tensor:
    m = entry["mixer"]
    t, hq, g, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = h @ w[p + "mix.q"].T, h @ w[p + "mix.k"].T, h @ w[p + "mix.v"].T
    if entry["type"] == "attention":
        lam = differential_lambda(w[p + "mix.lq1"], w[p + "mix.lk1"], w[p + "mix.lq2"], w[p + "mix.lk2"], m["diff"])
        o = differential_attention(q.view(t, hq, 2, d), k.view(t, g, 2, d), v.view(t, g, vd), m, lam, eps)
    else:
        q, k, v = (short_conv(u, w[p + f"mix.{n}.conv"]) for u, n in ((q, "q"), (k, "k"), (v, "v")))
        o = talking_attention(q.view(t, hq, d), k.view(t, g, d), v.view(t, g, vd), m, w[p + "mix.talk"])
    return o @ w[p + "mix.o"].T


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float32,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, entry in enumerate(cfg["layers"]):
        p = f"l{entry.get('weights_of', i)}."
        h = zero_centred_norm(x, w[p + "norm1"], eps)
        y = sublayer_gate(h, w[p + "rg1"], w[p + "rg1.b"]) * mixer_forward(h, w, p, entry, eps)
        if entry.get("mlp") is not None:
            y = y + sublayer_gate(h, w[p + "rg2"], w[p + "rg2.b"]) * swiglu(h, w[p + "mlp.gate"], w[p + "mlp.up"],
                                                                           w[p + "mlp.down"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T
