"""Plain, slow CPU implementation of the Kotipel decoder, one function per mechanism, in the dtype of the weights it
is given (float32 or float64). Whole sequences only: no cache, no portions, no batching; recurrences run token by
token. It is written from the equations and shares no code with ``flashrec_b200``.

Notation: ``x [T, width]`` residual stream, ``h`` its normalised form, positions count from 0."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1 / (1 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- rotary attention ------------------------------------------------------------------------------------
def rotary_frequencies(rot: dict) -> List[float]:
    """Angle per position of every pair; long wavelengths are slowed down by ``factor``, medium ones in between."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            length = 2 * math.pi / f
            if length > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif length >= sc["original"] / sc["high"]:
                s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(v: torch.Tensor, pos: int, freqs: List[float]) -> torch.Tensor:
    """``v [heads, dim]``: dimension i turns with dimension i + len(freqs); the rest stays."""
    n = len(freqs)
    out = v.clone()
    for i, f in enumerate(freqs):
        c, s = math.cos(pos * f), math.sin(pos * f)
        out[:, i] = v[:, i] * c - v[:, i + n] * s
        out[:, i + n] = v[:, i + n] * c + v[:, i] * s
    return out


def causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]."""
    t, heads = q.shape[:2]
    rep = heads // k.shape[1]
    hidden = torch.ones(t, t, dtype=torch.bool).triu(1)
    out = []
    for h in range(heads):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        out.append(torch.softmax(s.masked_fill(hidden, float("-inf")), dim=-1) @ v[:, h // rep])
    return torch.stack(out, dim=1)


def rotary_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Norm over all heads at once, rotation, causal attention, one gate per head, output projection."""
    t = h.shape[0]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(t, m["heads"], m["dim"])
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(t, m["kv_heads"], m["dim"])
    v = (h @ w[p + "v"].T).view(t, m["kv_heads"], m["vdim"])
    freqs = rotary_frequencies(m["rot"])
    q = torch.stack([rotate(q[i], i, freqs) for i in range(t)])
    k = torch.stack([rotate(k[i], i, freqs) for i in range(t)])
    o = causal_attention(q, k, v, m["scale"]) * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(t, -1) @ w[p + "o"].T


# ---- recurrences -----------------------------------------------------------------------------------------
def recurrence(q, k, v, decay) -> torch.Tensor:
    """One head: S <- decay_t (per row of S, or one number) * S + k_t v_t^T, o_t = S^T q_t. q, k [T, N], v [T, V]."""
    s = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = []
    for t in range(q.shape[0]):
        s = decay[t].reshape(-1, 1) * s + torch.outer(k[t], v[t])
        out.append(s.T @ q[t])
    return torch.stack(out)


def gated_linear_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    t, n, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(t, n, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(t, n, d)
    v = (h @ w[p + "v"].T).view(t, n, vd)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    decay = torch.exp(-softplus(-z) / m["tau"]).view(t, n, d)  # sigmoid(z) ** (1 / tau)
    o = torch.stack([recurrence(q[:, i], k[:, i], v[:, i], decay[:, i]) for i in range(n)], dim=1)
    o = (rms(o, eps) * w[p + "norm"]).reshape(t, -1) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def short_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """silu of the depthwise causal convolution, whose last tap is the current token's; zeros before the start."""
    t, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for i in range(t):
        y[i] = b
        for j in range(taps):
            s = i - taps + 1 + j
            if s >= 0:
                y[i] += w[:, j] * u[s]
    return silu(y)


def state_space(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    t, n, vd, st, g = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = n * vd
    z, u, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * g * st, n], dim=1)
    x, b, c = torch.split(short_conv(u, w[p + "conv"], w[p + "conv.b"]), [inner, g * st, g * st], dim=1)
    x, b, c = x.reshape(t, n, vd), b.reshape(t, g, st), c.reshape(t, g, st)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    y = []
    for i in range(n):
        j = i // (n // g)
        o = recurrence(c[:, j], b[:, j], x[:, i] * dt[:, i:i + 1], decay[:, i])
        y.append(o + w[p + "D"][i] * x[:, i])
    y = torch.cat(y, dim=1) * silu(z)
    y = rms(y.view(t, m["norm_groups"], -1), eps).reshape(t, -1) * w[p + "norm"]
    return y @ w[p + "o"].T


# ---- the layer -------------------------------------------------------------------------------------------
def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    left = rotary_attention(h, w, p + "left.", m["left"], eps)
    right = gated_linear_attention(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


def clamped_glu(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def token_input(x: torch.Tensor, e: torch.Tensor, gate: torch.Tensor, proj: torch.Tensor, norm: torch.Tensor, eps: float):
    return rms((gelu_tanh(x @ gate.T) * e) @ proj.T, eps) * norm


def run_order(cfg: dict) -> List[tuple]:
    """(layer, pass or None for the first layer of a pass / no pass) of every layer run in order."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float32,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.tensor(tokens)
    x = w["embed"][ids]
    for i, step in run_order(cfg):
        entry, p = cfg["layers"][i], f"l{i}."
        if step is not None:
            x = x + w["loop.step"][step]
        h = rms(x, eps) * w[p + "norm1"]
        mixer = parallel_mixer if entry["type"] == "parallel" else state_space
        x = x + mixer(h, w, p + "mix.", entry["mixer"], eps)
        mlp = entry.get("mlp")
        if mlp is not None:
            h = rms(x, eps) * w[p + "norm2"]
            x = x + clamped_glu(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"], mlp["limit"])
        if cfg.get("token_side"):
            d = cfg["token_side"]["dim"]
            e = w["side.embed"][ids][:, i * d:(i + 1) * d]
            x = x + token_input(x, e, w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T
