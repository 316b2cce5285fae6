"""Kotipel: a pre-norm decoder whose mixers are recurrent, or attention and a recurrence side by side, and whose layers
take a per-layer embedding of the token as a third input:

    x <- x + mixer(norm1 x);   x <- x + ff(norm2 x);   x <- x + norm(P (gelu(G x) * e_layer[token]))

Mixer "parallel": causal rotary attention with a gate per head, and gated linear attention with a decay per key channel,
each divided by its root mean square before they are averaged. Mixer "mamba2": a state-space recurrence with a decay per
head behind a short convolution. A range of layers may run several times with the same weights, each pass with its own
cache and state. ``config.json`` gives the order of the layers and every size.

Everything that is added to the fp32 stream is added by the kernel that computes the next norm of it (or the copy that
the token input's gate reads): what a layer leaves behind travels as :class:`flashrec_b200.lm_layers.Pending`."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Tuple, Union

import torch

from flashrec_b200.core import ForwardBatch
from flashrec_b200.kvcache import CacheSpec, LayerCaches
from flashrec_b200.lm_layers import (LinearScan, MergedProjection, MixAttention, Pending, ceil_to, embed, gated_add, group_norm,
                                     interleave_rows, pad_cols, pad_heads, pad_rows, qk_norm_rope, rotary_frequencies,
                                     rotary_table, short_conv, split_product, update_norm)

PARALLEL, MAMBA2 = "parallel", "mamba2"
GLU_ALPHA, GLU_UP_BIAS = 1.702, 1.0  # fixed by the design
_FULL = 1 << 30  # every earlier key stays visible


@dataclass(frozen=True)
class RotaryAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    rot_scaling: Optional[Tuple[Tuple[str, float], ...]] = None


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class ParallelConfig:
    left: RotaryAttentionConfig
    right: GatedLinearConfig

    @staticmethod
    def from_json(m: dict) -> "ParallelConfig":
        a, g = m["left"], m["right"]
        sc = a["rot"].get("scaling")
        left = RotaryAttentionConfig(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                                     int(a["rot"]["dims"]), float(a["rot"]["base"]),
                                     tuple((k, float(sc[k])) for k in ("factor", "low", "high", "original")) if sc else None)
        return ParallelConfig(left, GatedLinearConfig(int(g["heads"]), int(g["dim"]), int(g["vdim"]), float(g["tau"])))

    def cache_spec(self) -> CacheSpec:
        a, g = self.left, self.right
        return CacheSpec(a.kv_heads * ceil_to(a.dim, 16), a.kv_heads * ceil_to(a.vdim, 16), size=_FULL, state_heads=g.heads,
                         state_dim=g.dim, state_vdim=g.vdim)

    def tensor_shapes(self, w: int) -> Dict[str, tuple]:
        a, g = self.left, self.right
        q, k, n, v = a.heads * a.dim, a.kv_heads * a.dim, g.heads * g.dim, g.heads * g.vdim
        return {"left.q": (q, w), "left.k": (k, w), "left.v": (a.kv_heads * a.vdim, w), "left.q.norm": (q,), "left.k.norm": (k,),
                "left.g": (a.heads, w), "left.o": (w, a.heads * a.vdim), "right.q": (n, w), "right.k": (n, w), "right.v": (v, w),
                "right.g": (v, w), "right.o": (w, v), "right.norm": (g.vdim,), "right.a1": (None, w), "right.a2": (n, None),
                "right.a2.b": (n,), "left.out": (w,), "right.out": (w,)}


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @staticmethod
    def from_json(m: dict) -> "Mamba2Config":
        return Mamba2Config(*(int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Of the convolution: x, B and C."""
        return self.inner + 2 * self.groups * self.state

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(0, 0, conv_channels=self.channels, conv_taps=self.conv, mask="none", state_heads=self.heads,
                         state_dim=self.state, state_vdim=self.vdim)

    def tensor_shapes(self, w: int) -> Dict[str, tuple]:
        h = (self.heads,)
        return {"in": (self.inner + self.channels + self.heads, w), "conv": (self.channels, self.conv), "conv.b": (self.channels,),
                "dt_bias": h, "A_log": h, "D": h, "norm": (self.inner,), "o": (w, self.inner)}


_MIXERS = {PARALLEL: ParallelConfig, MAMBA2: Mamba2Config}


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[ParallelConfig, Mamba2Config]
    ff: Optional[int]  # width of the feed-forward, or None
    limit: float = 0.0


@dataclass(frozen=True)
class LayerRun:
    """One pass over a layer: ``step`` is the number of the loop's pass that begins with it, if one does."""

    layer: int
    step: Optional[int] = None


@dataclass(frozen=True)
class KotipelConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerConfig, ...]
    loop: Optional[Tuple[int, int, int]] = None  # start, stop, times
    side_dim: int = 0  # 0: no per-layer token input

    @staticmethod
    def from_json(cfg: dict) -> "KotipelConfig":
        layers = []
        for e in cfg["layers"]:
            if e["type"] not in _MIXERS:
                raise ValueError(f"unknown mixer type {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            mixer = _MIXERS[e["type"]].from_json(e["mixer"])
            layers.append(LayerConfig(mixer, None, 0.0) if mlp is None else LayerConfig(mixer, int(mlp["ff"]), float(mlp["limit"])))
        lp = cfg.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        side = cfg.get("token_side")
        return KotipelConfig(int(cfg["vocab"]), int(cfg["width"]), float(cfg["norm"]["eps"]), tuple(layers), loop,
                             int(side["dim"]) if side else 0)

    def runs(self) -> List[LayerRun]:
        """The layer runs in order; every one has its own cache and state."""
        n = len(self.layers)
        start, stop, times = self.loop or (0, 0, 0)
        out = [LayerRun(i) for i in range(start)]
        for t in range(times):
            out += [LayerRun(i, t if i == start else None) for i in range(start, stop)]
        return out + [LayerRun(i) for i in range(stop, n)]

    def cache_specs(self) -> List[CacheSpec]:
        return [self.layers[r.layer].mixer.cache_spec() for r in self.runs()]

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name and shape of every checkpoint tensor; None is a size that only the checkpoint knows."""
        w, d = self.width, self.side_dim
        out: Dict[str, tuple] = {"embed": (self.vocab, w), "final.norm": (w,)}
        if self.loop:
            out["loop.step"] = (self.loop[2], w)
        if d:
            out["side.embed"] = (self.vocab, len(self.layers) * d)
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            out[p + "norm1"] = (w,)
            out.update({p + "mix." + n: s for n, s in l.mixer.tensor_shapes(w).items()})
            if l.ff is not None:
                out.update({p + "norm2": (w,), p + "mlp.gate": (l.ff, w), p + "mlp.up": (l.ff, w), p + "mlp.down": (w, l.ff)})
            if d:
                out.update({p + "side.gate": (d, w), p + "side.proj": (w, d), p + "side.norm": (w,)})
        return out


class _Context:
    """What a layer run works with besides its weights."""

    def __init__(self, batch: ForwardBatch, caches: LayerCaches, run: int, req_to_token, counters, max_keys, tables):
        self.batch, self.caches, self.run = batch, caches, run
        self.req_to_token, self.counters, self.max_keys = req_to_token, counters, max_keys
        self.tables = tables  # angles of the batch's positions by rotary configuration, shared by the layers


class _Mixer:
    def __init__(self, cfg: KotipelConfig, dtype, device):
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)

    def f32(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=torch.float32).contiguous()

    def weight(self, t: torch.Tensor) -> torch.Tensor:
        return pad_cols(t, 8).to(device=self.device, dtype=self.dtype).contiguous()

    def new(self, t: int, cols: int, dtype=None) -> torch.Tensor:
        return torch.empty((t, ceil_to(cols, 8)), dtype=dtype or self.dtype, device=self.device)

    def dense(self, weight: torch.Tensor) -> MergedProjection:
        p = MergedProjection(int(weight.shape[1]))
        p.add("store", weight)
        p.finish(self.dtype, self.device)
        return p

    def product(self, a: torch.Tensor, p: MergedProjection):
        """``a`` times the one matrix of ``p``, over the model width: whole or as K shares."""
        w = self.cfg.width
        y = split_product(a, p.weight[:w])
        if y is None:
            y = self.new(int(a.shape[0]), w)
            p(a, [y])
        return y


class ParallelMixer(_Mixer):
    """Rotary attention and gated linear attention of the same input, one product for all their projections."""

    def __init__(self, cfg: KotipelConfig, m: ParallelConfig, tensors: Callable[[str], torch.Tensor], dtype, device):
        super().__init__(cfg, dtype, device)
        a, g = m.left, m.right
        self.m, self.spec = m, m.cache_spec()
        dp, vp = ceil_to(a.dim, 16), ceil_to(a.vdim, 16)
        rank = int(tensors("right.a1").shape[0])
        if int(tensors("right.a2").shape[1]) != rank:
            raise ValueError("the two factors of the decay projection have different ranks")
        proj = MergedProjection(cfg.width)
        proj.add("store", pad_heads(tensors("left.q"), a.dim, dp))
        proj.add("store", pad_heads(tensors("left.k"), a.dim, dp))
        proj.add("store", pad_heads(tensors("left.v"), a.vdim, vp))
        for n in ("right.q", "right.k", "right.v", "right.g"):
            proj.add("store", tensors(n))
        proj.add("store_f32", tensors("left.g"))
        proj.add("store_f32", tensors("right.a1"))
        proj.finish(dtype, device)
        self.proj, self.rank = proj, rank
        self.q_norm = self.f32(pad_heads(tensors("left.q.norm"), a.dim, dp))
        self.k_norm = self.f32(pad_heads(tensors("left.k.norm"), a.dim, dp))
        self.rotary = (a.rot_dims, a.rot_base, a.rot_scaling)
        self.inv_freq = rotary_frequencies(a.rot_dims, a.rot_base, dict(a.rot_scaling) if a.rot_scaling else None).to(self.device)
        self.attn = MixAttention("plain", a.heads, a.kv_heads, a.dim, a.vdim, a.scale, self.spec)
        self.attn.bind(device)
        self.scan = LinearScan("channel", g.heads, g.heads, g.dim, g.vdim, tensors("right.a2.b"), scale=g.dim ** -0.5, tau=g.tau,
                               up=tensors("right.a2"), device=self.device)
        self.head_norm = self.f32(tensors("right.norm"))
        self.left_o = self.dense(pad_heads(tensors("left.o").t(), a.vdim, vp).t())
        self.right_o = self.dense(tensors("right.o"))
        self.left_out, self.right_out = self.f32(tensors("left.out")), self.f32(tensors("right.out"))

    def forward(self, x: torch.Tensor, h: torch.Tensor, c: _Context) -> Pending:
        a, g, t, b = self.m.left, self.m.right, int(x.shape[0]), c.batch
        f32 = torch.float32
        kc, vc = c.caches.k[c.run], c.caches.v[c.run]
        q, k = self.new(t, self.attn.q_cols), self.new(t, self.spec.k_cols)
        rq, rk = self.new(t, g.heads * g.dim), self.new(t, g.heads * g.dim)
        rv, rg = self.new(t, g.heads * g.vdim), self.new(t, g.heads * g.vdim)
        gate, low = self.new(t, a.heads, f32), self.new(t, self.rank, f32)
        self.proj(h, [q, k, vc, rq, rk, rv, rg, gate, low], [None, None, b.out_cache_loc] + [None] * 6)
        if self.rotary not in c.tables:
            c.tables[self.rotary] = rotary_table(self.inv_freq, b.positions)
        qk_norm_rope(q, k, a.heads, a.kv_heads, a.dim, self.q_norm, self.k_norm, self.cfg.eps, c.tables[self.rotary], b, kc)
        o = self.attn.forward(q, kc, vc, c.req_to_token, b, c.counters, c.max_keys, gate)
        left = self.product(o, self.left_o)
        y = self.scan.forward(rq, rk, rv, low, c.caches.state[c.run], b, self.new(t, g.heads * g.vdim))
        group_norm(y, g.heads, g.vdim, self.head_norm, self.cfg.eps, rv, rg)
        right = self.product(rv, self.right_o)
        return Pending(parts=[(left, self.left_out, 0.5), (right, self.right_out, 0.5)])


class Mamba2Mixer(_Mixer):
    def __init__(self, cfg: KotipelConfig, m: Mamba2Config, tensors: Callable[[str], torch.Tensor], dtype, device):
        super().__init__(cfg, dtype, device)
        self.m, self.spec = m, m.cache_spec()
        z, u, dt = torch.split(tensors("in"), [m.inner, m.channels, m.heads], dim=0)
        proj = MergedProjection(cfg.width)
        proj.add("store", z)
        proj.add("store", u)
        proj.add("store_f32", dt)
        proj.finish(dtype, device)
        self.proj = proj
        self.conv_w, self.conv_b = self.f32(tensors("conv")), self.f32(tensors("conv.b"))
        self.scan = LinearScan("head", m.heads, m.groups, m.state, m.vdim, tensors("dt_bias"),
                               rate=torch.exp(tensors("A_log").float()), skip=tensors("D"), device=self.device)
        self.norm = self.f32(tensors("norm"))
        self.o_w = self.weight(tensors("o"))

    def forward(self, x: torch.Tensor, h: torch.Tensor, c: _Context) -> Pending:
        m, t = self.m, int(x.shape[0])
        z, u, dt = self.new(t, m.inner), self.new(t, m.channels), self.new(t, m.heads, torch.float32)
        self.proj(h, [z, u, dt])
        xbc = self.new(t, m.channels)
        short_conv(u, self.conv_w, [(xbc, None, 0, m.channels)], c.caches.conv[c.run], c.batch, self.conv_b, silu=True)
        keys = m.groups * m.state
        b, cc = xbc[:, m.inner:m.inner + keys], xbc[:, m.inner + keys:m.inner + 2 * keys]
        y = self.scan.forward(cc, b, xbc[:, :m.inner], dt, c.caches.state[c.run], c.batch, self.new(t, m.inner))
        o = group_norm(y, m.norm_groups, m.inner // m.norm_groups, self.norm, self.cfg.eps, self.new(t, m.inner), z, gate_first=True)
        return Pending(gated_add(x, [(o, self.o_w, None)]))


class KotipelLayer(_Mixer):
    """One layer's weights, laid out for the kernels; ``forward`` runs it on the caches of one layer run."""

    def __init__(self, cfg: KotipelConfig, layer: LayerConfig, tensors: Callable[[str], torch.Tensor],
                 side_embed: Optional[torch.Tensor], dtype, device):
        super().__init__(cfg, dtype, device)
        self.layer = layer
        self.norm1 = self.f32(tensors("norm1"))
        mixer = ParallelMixer if isinstance(layer.mixer, ParallelConfig) else Mamba2Mixer
        self.mixer = mixer(cfg, layer.mixer, lambda n: tensors("mix." + n), dtype, device)
        self.spec = self.mixer.spec
        if layer.ff is not None:
            self.norm2 = self.f32(tensors("norm2"))
            gu = interleave_rows(tensors("mlp.gate"), tensors("mlp.up"))
            self.ff_cols = int(gu.shape[0]) // 2
            self.gate_up = MergedProjection(cfg.width)
            self.gate_up.add("glu_clamp", gu, limit=layer.limit, alpha=GLU_ALPHA, up_bias=GLU_UP_BIAS)
            self.gate_up.finish(dtype, device)
            self.down_w = pad_cols(tensors("mlp.down"), 32).to(device=device, dtype=dtype).contiguous()
        self.side_embed = side_embed  # [vocab, side_dim padded to 8]
        if side_embed is not None:
            self.side_gate = MergedProjection(cfg.width)
            self.side_gate.add("gelu_mul", pad_rows(tensors("side.gate"), 8))
            self.side_gate.finish(dtype, device)
            self.side_proj = self.dense(tensors("side.proj"))
            self.side_norm = self.f32(tensors("side.norm"))

    def forward(self, x: torch.Tensor, c: _Context, pending: Pending, add: Optional[torch.Tensor]) -> Pending:
        cfg, t, eps = self.cfg, int(x.shape[0]), self.cfg.eps
        h = update_norm(x, eps, self.new(t, cfg.width), self.norm1, pending=pending, add=add)
        pending = self.mixer.forward(x, h, c)
        if self.layer.ff is not None:
            h = update_norm(x, eps, self.new(t, cfg.width), self.norm2, pending=pending)
            act = self.new(t, self.ff_cols)
            self.gate_up(h, [act])
            copy = self.new(t, cfg.width) if self.side_embed is not None else None
            pending = Pending(gated_add(x, [(act, self.down_w, None)], copy=copy))
        if self.side_embed is not None:
            if self.layer.ff is None or not pending.empty:
                copy = update_norm(x, eps, self.new(t, cfg.width), pending=pending)
            g = self.new(t, int(self.side_embed.shape[1]))
            self.side_gate(copy, [g], mul=(self.side_embed, c.batch.input_ids))
            pending = Pending(parts=[(self.product(g, self.side_proj), self.side_norm, 1.0)])
        return pending


class KotipelForCausalLM:
    """Embedding -> layer runs -> final norm -> logits with the embedding table. ``forward`` returns the residual stream
    and what is still to be added to it; ``logits`` turns chosen rows of both into fp32 logits."""

    def __init__(self, cfg: KotipelConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype, device):
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        for name, shape in cfg.tensor_shapes().items():
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            have = tuple(tensors[name].shape)
            if len(have) != len(shape) or any(s is not None and s != n for s, n in zip(shape, have)):
                raise ValueError(f"{name}: shape {have}, expected {shape}")
        self.head = MergedProjection(cfg.width)
        self.head.add("store_f32", tensors["embed"])
        self.head.finish(dtype, device)
        self.embed_table = self.head.weight[:cfg.vocab]
        n = len(cfg.layers)
        side: Optional[torch.Tensor] = None
        if cfg.side_dim:  # one block of columns per layer, padded
            side = tensors["side.embed"].to(device=device, dtype=dtype).view(cfg.vocab, n, cfg.side_dim)
            side = torch.nn.functional.pad(side, (0, ceil_to(cfg.side_dim, 8) - cfg.side_dim)).contiguous()
        self.layers = [KotipelLayer(cfg, l, lambda name, i=i: tensors[f"l{i}.{name}"], None if side is None else side[:, i], dtype,
                                    device) for i, l in enumerate(cfg.layers)]
        self.runs = cfg.runs()
        self.loop_step = tensors["loop.step"].to(device=device, dtype=torch.float32).contiguous() if cfg.loop else None
        self.final_norm = tensors["final.norm"].to(device=device, dtype=torch.float32).contiguous()
        self.cache_specs = cfg.cache_specs()
        self.vocab = cfg.vocab

    def new_caches(self, n_pages: int, n_rows: int) -> LayerCaches:
        return LayerCaches(self.cache_specs, n_pages, n_rows, self.dtype, self.device)

    def forward(self, batch: ForwardBatch, caches: LayerCaches, req_to_token: torch.Tensor, counters: torch.Tensor,
                static_max_pos: Optional[int] = None, on_layer: Optional[Callable[[int, torch.Tensor], None]] = None):
        """``static_max_pos``: bound of the positions a captured step will ever see. ``on_layer(i, x)`` is called with the
        finished residual stream after every layer run (updates are then never left pending)."""
        x = embed(self.embed_table, self.cfg.width, batch, 1.0, req_to_token)
        pending, tables = Pending(), {}
        for i, run in enumerate(self.runs):
            layer = self.layers[run.layer]
            keys = layer.spec.max_keys(static_max_pos) if static_max_pos is not None else None
            add = self.loop_step[run.step] if run.step is not None else None
            pending = layer.forward(x, _Context(batch, caches, i, req_to_token, counters, keys, tables), pending, add)
            if on_layer is not None:
                if not pending.empty:
                    update_norm(x, self.cfg.eps, None, pending=pending)
                    pending = Pending()
                on_layer(i, x)
        return x, pending

    def logits(self, x: torch.Tensor, pending: Pending, rows: torch.Tensor) -> torch.Tensor:
        """fp32 logits [n, vocab] of the rows ``rows`` (int64) of the residual stream."""
        n = int(rows.numel())
        h = torch.empty((n, ceil_to(self.cfg.width, 8)), dtype=self.dtype, device=self.device)
        update_norm(x, self.cfg.eps, h, self.final_norm, pending=pending, row_idx=rows)
        out = torch.empty((n, self.cfg.vocab), dtype=torch.float32, device=self.device)
        self.head(h, [out])
        return out


def random_tensors(cfg: KotipelConfig, seed: int = 0, rank: int = 16, device="cpu",
                   dtype: torch.dtype = torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights of the checkpoint's names and shapes (benchmarks and tests); ``rank`` of the decay projections."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        shape = tuple(rank if s is None else s for s in shape)
        t = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
        if name.endswith(("norm", "norm1", "norm2", "left.out", "right.out")):
            t = 1 + 0.2 * t
        elif name.endswith((".b", "D")):
            t = 0.5 * t
        elif name.endswith("dt_bias"):
            t = t - 2
        elif name.endswith("A_log"):
            t = 0.7 * t
        elif name.endswith(".conv"):
            t *= 0.5
        elif name not in ("embed", "side.embed"):
            t *= shape[-1] ** -0.5
        out[name] = t.to(dtype)
    return out
