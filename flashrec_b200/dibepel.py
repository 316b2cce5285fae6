"""Dibepel: a decoder whose layers add a mixer and a feed-forward of the same normalised input to the fp32
residual stream, each scaled element by element by a sigmoid of that input:

    h = norm(x);   x <- x + sigmoid(W1 h + b1) * mixer(h) + sigmoid(W2 h + b2) * ff(h)

Mixers: differential attention in a sliding window that keeps the first tokens, and chunked attention with short
convolutions on q, k and v, a linear distance bias and talking heads. ``config.json`` gives the order of the layers
and every size; layers may borrow another layer's weights.

Every projection of h (q, k, v, gate, up and both sigmoid gates) is one product with the merged weight, the output
projections of mixer and feed-forward are one gated two-part update of x: a layer is five kernels (norm, projections,
[convolution,] attention, update)."""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Sequence, Tuple

import torch

from flashrec_b200.core import ForwardBatch
from flashrec_b200.kvcache import CacheSpec, LayerCaches
from flashrec_b200.lm_layers import (MergedProjection, MixAttention, Partials, alibi_slopes, ceil_to, embed, gated_add,
                                     interleave_rows, pad_cols, pad_heads, rms_norm, short_conv)

DIFFERENTIAL, TALKING = "attention", "attention_2"


@dataclass(frozen=True)
class MixerConfig:
    kind: str  # DIFFERENTIAL or TALKING
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    mask_size: int
    keep_first: int = 0
    diff: float = 0.0
    conv: int = 1

    @staticmethod
    def from_json(kind: str, m: dict) -> "MixerConfig":
        if kind not in (DIFFERENTIAL, TALKING):
            raise ValueError(f"unknown mixer type {kind!r}")
        base = dict(kind=kind, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                    scale=float(m["scale"]), mask_size=int(m["mask"]["size"]))
        if kind == DIFFERENTIAL:
            return MixerConfig(**base, keep_first=int(m["mask"].get("keep_first", 0)), diff=float(m["diff"]))
        return MixerConfig(**base, conv=int(m["conv"]))

    @property
    def maps(self) -> int:
        return 2 if self.kind == DIFFERENTIAL else 1

    def cache_spec(self) -> CacheSpec:
        d, v = ceil_to(self.dim, 16), ceil_to(self.vdim, 16)
        k_cols, v_cols = self.kv_heads * self.maps * d, self.kv_heads * v
        if self.kind == DIFFERENTIAL:
            return CacheSpec(k_cols, v_cols, mask="window", size=self.mask_size, keep_first=self.keep_first)
        return CacheSpec(k_cols, v_cols, conv_channels=self.heads * d + k_cols + v_cols, conv_taps=self.conv,
                         mask="chunk", size=self.mask_size)


@dataclass(frozen=True)
class LayerConfig:
    mixer: MixerConfig
    ff: Optional[int]  # width of the dense SwiGLU feed-forward, or None
    weights_of: Optional[int] = None


@dataclass(frozen=True)
class DibepelConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: Tuple[LayerConfig, ...]

    @staticmethod
    def from_json(cfg: dict) -> "DibepelConfig":
        layers = []
        for e in cfg["layers"]:
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            wo = e.get("weights_of")
            layers.append(LayerConfig(MixerConfig.from_json(e["type"], e["mixer"]), None if mlp is None else int(mlp["ff"]),
                                      None if wo is None else int(wo)))
        return DibepelConfig(int(cfg["vocab"]), int(cfg["width"]), float(cfg["norm"]["eps"]),
                             float(cfg["embedding"]["scale"]), tuple(layers))

    def owner(self, i: int) -> int:
        """The layer whose weights layer ``i`` runs with."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError("layers borrow each other's weights in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def cache_specs(self) -> List[CacheSpec]:
        return [l.mixer.cache_spec() for l in self.layers]

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name and shape of every checkpoint tensor."""
        w = self.width
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, w), "final.norm": (w,), "head": (self.vocab, w)}
        for i, l in enumerate(self.layers):
            if l.weights_of is not None:
                continue
            m, p = l.mixer, f"l{i}."
            q, k, v = m.heads * m.maps * m.dim, m.kv_heads * m.maps * m.dim, m.kv_heads * m.vdim
            out.update({p + "norm1": (w,), p + "mix.q": (q, w), p + "mix.k": (k, w), p + "mix.v": (v, w),
                        p + "mix.o": (w, m.heads * m.vdim), p + "rg1": (w, w), p + "rg1.b": (w,)})
            if m.kind == DIFFERENTIAL:
                out.update({p + f"mix.{n}": (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
            else:
                out.update({p + f"mix.{n}.conv": (c, m.conv) for n, c in (("q", q), ("k", k), ("v", v))})
                out[p + "mix.talk"] = (m.heads, m.heads)
            if l.ff is not None:
                out.update({p + "mlp.gate": (l.ff, w), p + "mlp.up": (l.ff, w), p + "mlp.down": (w, l.ff),
                            p + "rg2": (w, w), p + "rg2.b": (w,)})
        return out


class DibepelLayer:
    """One layer's weights, laid out for the kernels; ``forward`` runs it on the caches of one layer run."""

    def __init__(self, cfg: DibepelConfig, layer: LayerConfig, tensors: Callable[[str], torch.Tensor], dtype, device):
        self.cfg, self.layer, self.dtype, self.device = cfg, layer, dtype, torch.device(device)
        m = layer.mixer
        dp, vp = ceil_to(m.dim, 16), ceil_to(m.vdim, 16)
        self.norm_w = tensors("norm1").to(device=device, dtype=torch.float32).contiguous()
        self.spec = m.cache_spec()
        q = pad_heads(tensors("mix.q"), m.dim, dp)
        k = pad_heads(tensors("mix.k"), m.dim, dp)
        v = pad_heads(tensors("mix.v"), m.vdim, vp)
        proj = MergedProjection(cfg.width)
        self.conv_w: Optional[torch.Tensor] = None
        if m.kind == DIFFERENTIAL:
            self.qkv = [proj.add("store", q), proj.add("store", k), proj.add("store", v)]
            lq1, lk1, lq2, lk2 = (tensors(f"mix.{n}").double() for n in ("lq1", "lk1", "lq2", "lk2"))
            lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + m.diff
            self.attn = MixAttention("diff", m.heads, m.kv_heads, m.dim, m.vdim, m.scale, self.spec, eps=cfg.eps, lam=lam,
                                     out_scale=1.0 - m.diff)
        else:
            self.qkv = [proj.add("store", torch.cat([q, k, v], dim=0))]
            self.conv_w = torch.cat([pad_heads(tensors("mix.q.conv"), m.dim, dp), pad_heads(tensors("mix.k.conv"), m.dim, dp),
                                     pad_heads(tensors("mix.v.conv"), m.vdim, vp)], dim=0)
            self.conv_w = self.conv_w.to(device=device, dtype=torch.float32).contiguous()
            if int(self.conv_w.shape[1]) != m.conv:
                raise ValueError("convolution taps differ between config and checkpoint")
            self.attn = MixAttention("talk", m.heads, m.kv_heads, m.dim, m.vdim, m.scale, self.spec,
                                     coef=tensors("mix.talk").float(), slopes=torch.tensor(alibi_slopes(m.heads)))
        self.ff_cols = 0
        if layer.ff is not None:
            gu = interleave_rows(tensors("mlp.gate"), tensors("mlp.up"))
            self.ff_cols = int(gu.shape[0]) // 2
            self.seg_ff = proj.add("swiglu", gu)
            self.down_w = pad_cols(tensors("mlp.down"), 32).to(device=device, dtype=dtype).contiguous()
        self.seg_g1 = proj.add("sigmoid", tensors("rg1"), bias=tensors("rg1.b"))
        if layer.ff is not None:
            self.seg_g2 = proj.add("sigmoid", tensors("rg2"), bias=tensors("rg2.b"))
        proj.finish(dtype, device)
        self.proj = proj
        self.o_w = pad_heads(tensors("mix.o").t(), m.vdim, vp).t().to(device=device, dtype=dtype).contiguous()
        self.attn.bind(device)

    def forward(self, x: torch.Tensor, batch: ForwardBatch, caches: LayerCaches, run: int, req_to_token: torch.Tensor,
                counters: torch.Tensor, partials: Optional[Partials], max_keys: Optional[int]) -> Optional[Partials]:
        cfg, t = self.cfg, int(x.shape[0])
        new = lambda cols: torch.empty((t, ceil_to(cols, 8)), dtype=self.dtype, device=self.device)
        h = rms_norm(x, self.norm_w, 1.0, cfg.eps, new(cfg.width), partials)
        kc, vc, loc = caches.k[run], caches.v[run], batch.out_cache_loc
        outs: List[Optional[torch.Tensor]] = [None] * len(self.proj.ranges)
        maps: List[Optional[torch.Tensor]] = [None] * len(self.proj.ranges)
        if self.conv_w is None:
            q = new(self.attn.q_cols)
            for seg, o, rm in zip(self.qkv, (q, kc, vc), (None, loc, loc)):
                outs[seg], maps[seg] = o, rm
        else:
            u = new(int(self.conv_w.shape[0]))
            outs[self.qkv[0]] = u
        g1 = outs[self.seg_g1] = new(cfg.width)
        if self.layer.ff is not None:
            act = outs[self.seg_ff] = new(self.ff_cols)
            g2 = outs[self.seg_g2] = new(cfg.width)
        self.proj(h, outs, maps)
        if self.conv_w is not None:
            q = new(self.attn.q_cols)
            nq, nk = self.attn.q_cols, self.spec.k_cols
            short_conv(u, self.conv_w, [(q, None, 0, nq), (kc, loc, nq, nk), (vc, loc, nq + nk, self.spec.v_cols)],
                       caches.conv[run], batch)
        o = self.attn.forward(q, kc, vc, req_to_token, batch, counters, max_keys)
        parts = [(o, self.o_w, g1)]
        if self.layer.ff is not None:
            parts.append((act, self.down_w, g2))
        return gated_add(x, parts)


class DibepelForCausalLM:
    """Embedding -> layer runs -> final norm -> logits. ``forward`` returns the residual stream (and the last
    layer's pending partials); ``logits`` turns chosen rows of it into fp32 logits."""

    SOURCES = ("capi", "dense_proj", "lm_rows", "attn_mix", "attn_talk")  # what a build of this family alone compiles

    def __init__(self, cfg: DibepelConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype, device):
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        for name, shape in cfg.tensor_shapes().items():
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            if tuple(tensors[name].shape) != shape:
                raise ValueError(f"{name}: shape {tuple(tensors[name].shape)}, expected {shape}")
        self.embed_table = tensors["embed"].to(device=device, dtype=dtype).contiguous()
        own: Dict[int, DibepelLayer] = {}
        self.layers: List[DibepelLayer] = []
        for i in range(len(cfg.layers)):
            j = cfg.owner(i)
            if j not in own:
                own[j] = DibepelLayer(cfg, cfg.layers[j], lambda n, j=j: tensors[f"l{j}.{n}"], dtype, device)
            self.layers.append(own[j])
        self.final_norm = tensors["final.norm"].to(device=device, dtype=torch.float32).contiguous()
        self.head = MergedProjection(cfg.width)
        self.head.add("store_f32", tensors["head"])
        self.head.finish(dtype, device)
        self.cache_specs = cfg.cache_specs()
        self.vocab = cfg.vocab

    def new_caches(self, n_pages: int, n_rows: int) -> LayerCaches:
        return LayerCaches(self.cache_specs, n_pages, n_rows, self.dtype, self.device)

    def forward(self, batch: ForwardBatch, caches: LayerCaches, req_to_token: torch.Tensor, counters: torch.Tensor,
                static_max_pos: Optional[int] = None, on_layer: Optional[Callable[[int, torch.Tensor], None]] = None):
        """``static_max_pos``: bound of the positions a captured step will ever see. ``on_layer(i, x)`` is called
        with the finished residual stream after every layer run (updates are then never left as partials)."""
        x = embed(self.embed_table, self.cfg.width, batch, self.cfg.embed_scale, req_to_token)
        partials: Optional[Partials] = None
        for i, layer in enumerate(self.layers):
            keys = layer.spec.max_keys(static_max_pos) if static_max_pos is not None else None
            partials = layer.forward(x, batch, caches, i, req_to_token, counters, partials, keys)
            if on_layer is not None:
                if partials is not None:
                    x += partials.buf.sum(dim=0)
                    partials = None
                on_layer(i, x)
        return x, partials

    def logits(self, x: torch.Tensor, partials: Optional[Partials], rows: torch.Tensor) -> torch.Tensor:
        """fp32 logits [n, vocab] of the rows ``rows`` (int64) of the residual stream."""
        n = int(rows.numel())
        h = torch.empty((n, ceil_to(self.cfg.width, 8)), dtype=self.dtype, device=self.device)
        rms_norm(x, self.final_norm, 1.0, self.cfg.eps, h, partials, rows)
        out = torch.empty((n, self.cfg.vocab), dtype=torch.float32, device=self.device)
        self.head(h, [out])
        return out


def random_tensors(cfg: DibepelConfig, seed: int = 0, std: Optional[float] = None, device="cpu",
                   dtype: torch.dtype = torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights of the checkpoint's names and shapes (benchmarks and tests). Matrices default to 1 / sqrt(fan in)."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        t = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
        if name.endswith(("norm1", "final.norm", ".b")):
            t *= 0.1
        elif name.endswith(("lq1", "lk1", "lq2", "lk2")):
            t *= 0.1
        elif name.endswith(".conv"):
            t *= 0.5
        elif name == "embed":
            t *= 1.0 / max(cfg.embed_scale, 1e-6)
        else:
            t *= std if std is not None else shape[-1] ** -0.5
        out[name] = t.to(dtype)
    return out
