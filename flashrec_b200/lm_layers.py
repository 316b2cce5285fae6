"""Building blocks of the 16/32-bit decoder models, each a thin wrapper around one C-ABI entry point with its
constants as parameters: merged projections with per-range epilogues, the gated two-part residual update, RMS norm
of the fp32 residual stream (also fused with an update of the stream by normalised vectors), gated norms over groups,
norm and rotation of queries and keys, the short causal convolution, attention that mixes several softmax maps, and
recurrences with a matrix state per head.

``dtype`` (bfloat16 or float32) is the type of weights, activations and caches; the residual stream is fp32 in
both. bfloat16 runs on the tensor cores, float32 is true 32-bit arithmetic throughout."""

from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass, field
from typing import List, Optional, Sequence, Tuple, Union

import torch

from flashrec_b200 import _lib
from flashrec_b200._lib import (FrConvOut, FrGatedPart, FrGroupNorm, FrLinearScan, FrMixAttn, FrNormPart, FrNormUpdate,
                                FrOutSegment, FrQkRope, call, ptr, require_cuda, stream_ptr)
from flashrec_b200.core import ForwardBatch
from flashrec_b200.kvcache import CacheSpec

SEG = {"store": _lib.FR_SEG_STORE, "swiglu": _lib.FR_SEG_SWIGLU, "sigmoid": _lib.FR_SEG_SIGMOID,
       "store_f32": _lib.FR_SEG_STORE_F32, "glu_clamp": _lib.FR_SEG_GLU_CLAMP, "gelu_mul": _lib.FR_SEG_GELU_MUL}
_PAIRED = ("swiglu", "glu_clamp")  # weight rows in [32 gate | 32 up] blocks
MIX = {"diff": _lib.FR_MIX_DIFF, "talk": _lib.FR_MIX_TALK, "plain": _lib.FR_MIX_PLAIN}
ROW_PORTION = 8  # shorter portions run their attention and recurrences row by row
_SCORE_SCRATCH_BYTES = 256 << 20
_MAP_SCRATCH_BYTES = 1 << 30  # maps of talking heads between their kernels: every token tile of a large step at once


def ceil_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def dtype_code(dtype: torch.dtype) -> int:
    if dtype == torch.bfloat16:
        return 0
    if dtype == torch.float32:
        return 1
    raise NotImplementedError(f"{dtype}: these layers run in bfloat16 or float32")


def pad_heads(w: torch.Tensor, dim: int, padded: int) -> torch.Tensor:
    """Rows ``[heads * dim, ...]`` with every head's rows zero-padded to ``padded``."""
    w = w.reshape(-1, dim, *w.shape[1:])
    if padded != dim:
        w = torch.cat([w, w.new_zeros((w.shape[0], padded - dim, *w.shape[2:]))], dim=1)
    return w.reshape(-1, *w.shape[2:])


def pad_rows(w: torch.Tensor, multiple: int) -> torch.Tensor:
    extra = ceil_to(w.shape[0], multiple) - w.shape[0]
    return w if extra == 0 else torch.cat([w, w.new_zeros((extra, *w.shape[1:]))], dim=0)


def pad_cols(w: torch.Tensor, multiple: int) -> torch.Tensor:
    extra = ceil_to(w.shape[1], multiple) - w.shape[1]
    return w if extra == 0 else torch.cat([w, w.new_zeros((w.shape[0], extra))], dim=1)


def interleave_rows(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[32 gate | 32 up] blocks, both zero-padded to whole blocks (the SwiGLU epilogue's weight layout)."""
    g, u = pad_rows(gate, 32), pad_rows(up, 32)
    return torch.stack([g.reshape(-1, 32, g.shape[1]), u.reshape(-1, 32, u.shape[1])], dim=1).reshape(-1, g.shape[1])


@dataclass
class ColumnRange:
    """One output of a merged projection: ``rows`` weight rows (padded) of which ``n`` columns leave."""

    kind: str
    rows: int
    n: int
    bias: Optional[torch.Tensor] = None
    limit: float = 0.0
    alpha: float = 0.0
    up_bias: float = 0.0


class MergedProjection:
    """All projections of one input as a single product: one weight ``[N, K]``, column ranges with their own
    epilogues (``fr_dense_proj``)."""

    def __init__(self, k: int):
        self.k = int(k)
        self._parts: List[torch.Tensor] = []
        self.ranges: List[ColumnRange] = []
        self.weight: Optional[torch.Tensor] = None

    def add(self, kind: str, weight: torch.Tensor, n: Optional[int] = None, bias: Optional[torch.Tensor] = None,
            align: int = 32, limit: float = 0.0, alpha: float = 0.0, up_bias: float = 0.0) -> int:
        """Append a range; returns its index. ``swiglu`` and ``glu_clamp`` (with ``limit``, ``alpha``, ``up_bias``) take
        an interleaved weight and must stay 64-aligned."""
        if kind in _PAIRED:
            start = sum(r.rows for r in self.ranges)
            if start % 64:  # start the interleaved blocks on a 64-row boundary: widen the range before
                self._parts[-1] = pad_rows(self._parts[-1], 32)
                self._parts[-1] = torch.cat([self._parts[-1], self._parts[-1].new_zeros((32, self._parts[-1].shape[1]))])
                self.ranges[-1].rows += 32
            rows = weight.shape[0]
            n = rows // 2 if n is None else n
        else:
            n = weight.shape[0] if n is None else n
            weight = pad_rows(weight, align)
            rows = weight.shape[0]
        self._parts.append(weight)
        self.ranges.append(ColumnRange(kind, rows, int(n), bias, float(limit), float(alpha), float(up_bias)))
        return len(self.ranges) - 1

    def finish(self, dtype: torch.dtype, device) -> None:
        w = torch.cat(self._parts, dim=0)
        self.weight = pad_cols(w, 8).to(device=device, dtype=dtype).contiguous()
        for r in self.ranges:
            if r.bias is not None:
                r.bias = r.bias.to(device=device, dtype=torch.float32).contiguous()
        self._parts = []

    def __call__(self, a: torch.Tensor, outs: Sequence[torch.Tensor],
                 row_maps: Optional[Sequence[Optional[torch.Tensor]]] = None, algo: int = 0,
                 mul: Optional[Tuple[torch.Tensor, torch.Tensor]] = None) -> None:
        """``a`` [M, lda >= K padded]; ``outs`` one 2-D tensor per range (rows are ``row_maps[i][m]`` if given);
        ``mul`` = (table [rows, n], row of each m) of the ``gelu_mul`` ranges."""
        require_cuda(a)
        segs = (FrOutSegment * len(self.ranges))()
        n0 = 0
        for i, r in enumerate(self.ranges):
            o = outs[i]
            rm = row_maps[i] if row_maps is not None else None
            segs[i] = FrOutSegment(SEG[r.kind], n0, r.n, 0, ptr(o), o.stride(0), ptr(rm), ptr(r.bias), r.limit, r.alpha, r.up_bias)
            if r.kind == "gelu_mul":
                segs[i].mul, segs[i].ld_mul, segs[i].mul_map = ptr(mul[0]), mul[0].stride(0), ptr(mul[1])
            n0 += r.rows
        w, m, k = self.weight, int(a.shape[0]), int(self.weight.shape[1])
        code, s = dtype_code(w.dtype), stream_ptr(a.device)
        # a handful of tiles: their K extent is split over the SMs
        n_splits = _lib.load().fr_dense_gated_add_splits(code, m, n0, k, 0) if algo == 0 and n0 <= 1024 else 0
        if n_splits >= 4:
            buf = torch.empty((n_splits, m, n0), dtype=torch.float32, device=a.device)
            call("fr_dense_proj_split", code, ptr(a), a.stride(0), ptr(w), w.stride(0), m, n0, k, segs, len(segs), ptr(buf), n_splits, s)
        else:
            call("fr_dense_proj", code, ptr(a), a.stride(0), ptr(w), w.stride(0), m, n0, k, segs, len(segs), algo, s)


@dataclass
class Partials:
    """K shares of a residual update that the next norm adds (``fr_dense_gated_add`` with split K)."""

    buf: torch.Tensor
    n: int


def gated_add(x: torch.Tensor, parts: Sequence[Tuple[torch.Tensor, torch.Tensor, Optional[torch.Tensor]]],
              algo: int = 0, split: bool = True, copy: Optional[torch.Tensor] = None) -> Optional[Partials]:
    """``x += sum gate * (a @ w.T)`` over one or two ``(a, w, gate)`` parts; few-row products may come back as
    partials for the following ``rms_norm`` instead. ``copy`` gets the new x in its own type (not with partials)."""
    require_cuda(x)
    m, n = int(x.shape[0]), int(x.shape[1])
    arr = (FrGatedPart * len(parts))()
    for i, (a, w, g) in enumerate(parts):
        arr[i] = FrGatedPart(ptr(a), ptr(w), ptr(g), a.stride(0), w.stride(0), 0 if g is None else g.stride(0),
                             int(w.shape[1]), 0)
    code = dtype_code(parts[0][1].dtype)
    k = [int(p[1].shape[1]) for p in parts] + [0]
    n_splits = _lib.load().fr_dense_gated_add_splits(code, m, n, k[0], k[1]) if split and algo == 0 else 0
    buf = torch.empty((n_splits, m, n), dtype=torch.float32, device=x.device) if n_splits > 0 else None
    if n_splits > 0:
        copy = None
    call("fr_dense_gated_add", code, arr, len(parts), ptr(x), x.stride(0), m, n, ptr(buf), n_splits, ptr(copy),
         copy.stride(0) if copy is not None else 0, algo, stream_ptr(x.device))
    return Partials(buf, n_splits) if n_splits > 0 else None


def rms_norm(x: torch.Tensor, weight: torch.Tensor, offset: float, eps: float, out: torch.Tensor,
             partials: Optional[Partials] = None, row_idx: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out = x / sqrt(mean(x^2) + eps) * (offset + weight)`` of the fp32 stream; ``partials`` are added to ``x``
    first. ``offset`` 1 for weights stored around zero, 0 for plain ones."""
    require_cuda(x)
    m = int(out.shape[0])
    buf = partials.buf if partials is not None else None
    call("fr_lm_norm", dtype_code(out.dtype), ptr(x), x.stride(0), ptr(weight), float(offset), float(eps), ptr(buf),
         partials.n if partials is not None else 0, buf.stride(0) if buf is not None else 0, ptr(row_idx), ptr(out),
         out.stride(0), m, int(x.shape[1]), stream_ptr(x.device))
    return out


def split_product(a: torch.Tensor, w: torch.Tensor) -> Optional[Partials]:
    """``a @ w.T`` as K shares when it has so few tiles that they would leave SMs idle, else None."""
    require_cuda(a)
    m, n, code = int(a.shape[0]), int(w.shape[0]), dtype_code(w.dtype)
    n_splits = _lib.load().fr_dense_gated_add_splits(code, m, n, int(w.shape[1]), 0)
    if n_splits < 2:
        return None
    buf = torch.empty((n_splits, m, n), dtype=torch.float32, device=a.device)
    arr = (FrGatedPart * 1)(FrGatedPart(ptr(a), ptr(w), None, a.stride(0), w.stride(0), 0, int(w.shape[1]), 0))
    call("fr_dense_gated_add", code, arr, 1, ptr(buf), n, m, n, ptr(buf), n_splits, None, 0, 0, stream_ptr(a.device))
    return Partials(buf, n_splits)


@dataclass
class Pending:
    """What still has to be added to the residual stream: K shares of a product, and vectors (also as K shares) that are
    divided by their root mean square, weighted and scaled, ``(y [M, W], weight [W], coefficient)``."""

    partials: Optional[Partials] = None
    parts: List[Tuple[Union[torch.Tensor, Partials], torch.Tensor, float]] = field(default_factory=list)

    @property
    def empty(self) -> bool:
        return self.partials is None and not self.parts


def update_norm(x: torch.Tensor, eps: float, out: Optional[torch.Tensor], weight: Optional[torch.Tensor] = None,
                offset: float = 0.0, pending: Optional[Pending] = None, add: Optional[torch.Tensor] = None,
                row_idx: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """Adds ``pending`` and the vector ``add`` to the stream, then ``out`` = its norm (its rounded copy without a
    weight). With ``row_idx`` only those rows are read and the stream itself stays."""
    require_cuda(x)
    pending = pending or Pending()
    whole = [y for y, _, _ in pending.parts if isinstance(y, torch.Tensor)]
    dtype = out.dtype if out is not None else (whole[0].dtype if whole else torch.float32)
    u = FrNormUpdate(dtype=dtype_code(dtype), n_parts=len(pending.parts), eps=eps, offset=offset, x=ptr(x), ldx=x.stride(0),
                     add=ptr(add), row_idx=ptr(row_idx), weight=ptr(weight), out=ptr(out),
                     ldo=out.stride(0) if out is not None else 0)
    if pending.partials is not None:
        u.n_partials, u.partials = pending.partials.n, ptr(pending.partials.buf)
        u.partial_stride = pending.partials.buf.stride(0)
    for i, (y, w, coef) in enumerate(pending.parts):
        if isinstance(y, Partials):
            u.parts[i] = FrNormPart(ptr(y.buf), y.buf.stride(0), ptr(w), coef, y.n)
        else:
            u.parts[i] = FrNormPart(ptr(y), y.stride(0), ptr(w), coef, 0)
    m = int(x.shape[0]) if row_idx is None else int(row_idx.numel())
    call("fr_lm_update_norm", ctypes.byref(u), m, int(x.shape[1]), stream_ptr(x.device))
    return out


def group_norm(y: torch.Tensor, groups: int, size: int, weight: torch.Tensor, eps: float, out: torch.Tensor,
               gate: Optional[torch.Tensor] = None, gate_first: bool = False) -> torch.Tensor:
    """RMS norm over each of ``groups`` runs of ``size`` columns; ``gate``: times its silu, before or after. ``weight``
    has ``size`` values (every group the same) or one per column."""
    require_cuda(y)
    mode = _lib.FR_GATE_NONE if gate is None else (_lib.FR_GATE_BEFORE if gate_first else _lib.FR_GATE_AFTER)
    a = FrGroupNorm(dtype=dtype_code(y.dtype), gate_mode=mode, groups=groups, size=size,
                    weight_per_group=0 if weight.numel() == size else 1, eps=eps, y=ptr(y), ldy=y.stride(0), gate=ptr(gate),
                    ldg=gate.stride(0) if gate is not None else 0, weight=ptr(weight), out=ptr(out), ldo=out.stride(0))
    call("fr_lm_group_norm", ctypes.byref(a), int(y.shape[0]), stream_ptr(y.device))
    return out


def rotary_frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """Angle per position of each rotated pair, as a sum of two floats (fp32 [dims / 2, 2]). ``scaling`` (factor, low, high, original): pairs whose
    wavelength exceeds original / low turn ``factor`` times slower, those below original / high as they are, and a
    linear blend in original / wavelength between."""
    f = float(base) ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
    if scaling is not None:
        turns = float(scaling["original"]) * f / (2 * math.pi)  # within the original length
        low, high = float(scaling["low"]), float(scaling["high"])
        slow = f / float(scaling["factor"])
        s = (turns - low) / (high - low) if high != low else torch.zeros_like(f)
        f = torch.where(turns > high, f, torch.where(turns < low, slow, (1 - s) * slow + s * f))
    hi = f.float()
    return torch.stack([hi, (f - hi.double()).float()], dim=1).contiguous()


def rotary_table(inv_freq: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """Cosines, then sines of ``positions * inv_freq`` per token: [T, 2 * pairs] for :func:`qk_norm_rope`."""
    require_cuda(positions)
    pairs, t = int(inv_freq.shape[0]), int(positions.numel())
    table = torch.empty((t, 2 * pairs), dtype=torch.float32, device=positions.device)
    call("fr_lm_rotary_table", ptr(inv_freq), pairs, ptr(positions), ptr(table), t, stream_ptr(positions.device))
    return table


def qk_norm_rope(q: torch.Tensor, k: torch.Tensor, heads: int, kv_heads: int, dim: int, q_weight: torch.Tensor,
                 k_weight: torch.Tensor, eps: float, table: torch.Tensor, batch: ForwardBatch, k_cache: torch.Tensor) -> None:
    """Norms over all heads at once and rotation by the angles of ``table``; ``q`` in place, ``k`` into its cache slots.
    Heads are padded as the weights are."""
    require_cuda(q, k, k_cache)
    a = FrQkRope(dtype=dtype_code(q.dtype), heads=heads, kv_heads=kv_heads, dim=int(q_weight.numel()) // heads, dim_true=dim,
                 rot_dims=int(table.shape[1]), eps=eps, q=ptr(q), ldq=q.stride(0), k=ptr(k), ldk=k.stride(0),
                 q_weight=ptr(q_weight), k_weight=ptr(k_weight), table=ptr(table),
                 loc=ptr(batch.out_cache_loc), k_cache=ptr(k_cache), ldkc=k_cache.stride(0))
    call("fr_lm_qk_norm_rope", ctypes.byref(a), int(q.shape[0]), stream_ptr(q.device))


def embed(table: torch.Tensor, width: int, batch: ForwardBatch, scale: float, req_to_token: Optional[torch.Tensor],
          ) -> torch.Tensor:
    """fp32 residual stream ``table[id] * scale``; also enters the batch's new slots into the slot table."""
    ids = batch.input_ids
    x = torch.empty((ids.numel(), width), dtype=torch.float32, device=ids.device)
    call("fr_lm_embed", dtype_code(table.dtype), ptr(table), table.stride(0), ptr(ids), ptr(x), x.stride(0), ids.numel(),
         width, int(table.shape[0]), float(scale), ptr(req_to_token),
         req_to_token.stride(0) if req_to_token is not None else 0, ptr(batch.tok_rows), ptr(batch.positions),
         ptr(batch.out_cache_loc), stream_ptr(ids.device))
    return x


def short_conv(u: torch.Tensor, weight: torch.Tensor, outs, state: torch.Tensor, batch: ForwardBatch,
               bias: Optional[torch.Tensor] = None, silu: bool = False) -> None:
    """Causal depthwise convolution of ``u`` [T, C] with ``weight`` [C, taps] fp32, plus ``bias``, through a silu;
    ``outs`` = list of ``(tensor, row_map or None, first channel, channels)``; ``state`` [rows, taps - 1, C] is read and
    advanced."""
    require_cuda(u)
    arr = (FrConvOut * len(outs))()
    for i, (o, rm, c0, c) in enumerate(outs):
        arr[i] = FrConvOut(ptr(o), o.stride(0), ptr(rm), c0, c)
    call("fr_short_conv", dtype_code(u.dtype), ptr(u), u.stride(0), ptr(weight), ptr(bias),
         _lib.FR_CONV_SILU if silu else _lib.FR_CONV_LINEAR, int(weight.shape[1]),
         int(weight.shape[0]), arr, len(outs), ptr(state), ptr(batch.req_pool_indices), ptr(batch.tok_req),
         ptr(batch.qo_indptr), ptr(batch.positions), int(u.shape[0]), int(batch.req_pool_indices.numel()),
         1 if batch.one_token else 0, stream_ptr(u.device))


def alibi_slopes(heads: int) -> List[float]:
    """Distance-bias slopes 2^(-8 (h + 1) / heads)."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


class MixAttention:
    """Attention whose outputs are linear combinations of several softmax maps over the same values
    (``fr_mix_attn`` in the header). ``mix``: "diff" (two maps per head, second one subtracted ``lam`` times, output
    divided by its root mean square, times ``out_scale``), "talk" (all heads' maps through the matrix ``coef``) or "plain"
    (ordinary attention; ``forward`` may get a gate per head).
    ``dim`` / ``vdim`` are the model's sizes; caches and buffers use ``dim_p`` / ``vdim_p`` (multiples of 16)."""

    def __init__(self, mix: str, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, cache: CacheSpec, *,
                 eps: float = 0.0, lam: float = 0.0, out_scale: float = 1.0, coef: Optional[torch.Tensor] = None,
                 slopes: Optional[torch.Tensor] = None):
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        self.mix, self.heads, self.kv_heads = mix, int(heads), int(kv_heads)
        self.dim_p, self.vdim_p = ceil_to(dim, 16), ceil_to(vdim, 16)
        self.maps = 2 if mix == "diff" else 1
        self.cache = cache
        self.coef, self.slopes = coef, slopes
        big = (1 << 31) - 1
        self._args = FrMixAttn(mix=MIX[mix],
                               mask=_lib.FR_MASK_CHUNK if cache.mask == "chunk" else _lib.FR_MASK_WINDOW,
                               mask_size=min(cache.size, big), keep_first=min(cache.keep_first, big), heads=self.heads,
                               kv_heads=self.kv_heads, dim=self.dim_p, vdim=self.vdim_p, vdim_true=int(vdim),
                               scale=scale, lambda_=lam, eps=eps, out_scale=out_scale)
        self.tensor_cores = False

    @property
    def q_cols(self) -> int:
        return self.heads * self.maps * self.dim_p

    def bind(self, device) -> None:
        """Move the constants to ``device`` and ask the library whether the tensor-core kernel takes these sizes."""
        for name in ("coef", "slopes"):
            t = getattr(self, name)
            if t is not None:
                setattr(self, name, t.to(device=device, dtype=torch.float32).contiguous())
        self._args.coef, self._args.slopes = ptr(self.coef), ptr(self.slopes)
        self.tensor_cores = bool(_lib.load().fr_mix_attn_tc_fits(self._args.mix, self.heads, self.kv_heads, self.dim_p,
                                                                self.vdim_p))

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, req_to_token: torch.Tensor,
                batch: ForwardBatch, counters: torch.Tensor, max_keys: Optional[int] = None,
                head_gate: Optional[torch.Tensor] = None) -> torch.Tensor:
        """q [T, q_cols]; ``head_gate`` fp32 [T, heads], whose sigmoid multiplies the heads ("plain"); ``k`` / ``v`` the layer's caches (the batch's own keys are in already). bf16 prompts take
        the tensor-core kernel, short portions, decode steps and fp32 the row kernels."""
        require_cuda(q, k, v)
        t = int(q.shape[0])
        out = torch.empty((t, self.heads * self.vdim_p), dtype=q.dtype, device=q.device)
        a = FrMixAttn.from_buffer_copy(self._args)
        a.dtype = dtype_code(q.dtype)
        a.q, a.ldq, a.k, a.ldk, a.v, a.ldv = ptr(q), q.stride(0), ptr(k), k.stride(0), ptr(v), v.stride(0)
        a.out, a.ldo = ptr(out), out.stride(0)
        a.req_to_token, a.table_stride = ptr(req_to_token), req_to_token.stride(0)
        a.req_rows, a.tok_req, a.pos = ptr(batch.req_pool_indices), ptr(batch.tok_req), ptr(batch.positions)
        a.num_slots = int(k.shape[0])
        if head_gate is not None:
            a.head_gate, a.ld_gate = ptr(head_gate), head_gate.stride(0)
        s = stream_ptr(q.device)
        tc = self.tensor_cores and a.dtype == 0
        n_row = batch.n_row_tokens if tc else t
        if n_row > 0:
            keys = self.cache.max_keys(batch.max_pos) if max_keys is None else max_keys
            self._rows(a, n_row, keys, counters, s, q.device)
        if n_row < t:
            n_tiles = int(batch.tiles.shape[0])
            size = _lib.load().fr_mix_attn_tc_scratch(ctypes.byref(a), n_tiles, batch.max_pos, _MAP_SCRATCH_BYTES)
            scratch = torch.empty(size, dtype=torch.uint8, device=q.device) if size > 0 else None
            call("fr_mix_attn_tc", ctypes.byref(a), ptr(batch.tiles), n_tiles, t, batch.max_pos, ptr(scratch), max(size, 0), s)
        return out

    def _rows(self, a: FrMixAttn, n_row: int, keys: int, counters: torch.Tensor, stream, device) -> None:
        lib = _lib.load()
        blocks = (keys + 63) // 64
        splits = max(1, min(blocks, 16, 444 // max(1, n_row * self.kv_heads)))
        if n_row * self.kv_heads > counters.numel():
            splits = 1
        size = lambda n: int(lib.fr_mix_attn_rows_scratch(a.mix, self.heads, self.vdim_p, n, keys, splits))
        step = max(1, min(n_row, 32768, _SCORE_SCRATCH_BYTES // max(1, size(1))))
        scratch = torch.empty(size(step) + 16, dtype=torch.uint8, device=device)
        for r0 in range(0, n_row, step):
            call("fr_mix_attn_rows", ctypes.byref(a), r0, min(step, n_row - r0), keys, splits, ptr(scratch),
                 int(scratch.numel()), ptr(counters), stream)


class LinearScan:
    """Recurrence ``S <- diag(a_t) S + k_t u_t^T``, ``o_t = S^T (scale q_t) + skip v_t`` per head, fp32 state and decays
    (``fr_linear_scan`` in the header). ``decay`` "channel": ``a_t = sigmoid(up . step_t + step_bias) ^ (1 / tau)`` per row
    of S, u = v; "head": step size ``d_t = softplus(step_t + step_bias)``, ``a_t = exp(-rate d_t)``, ``u = d_t v``."""

    def __init__(self, decay: str, heads: int, key_heads: int, dim: int, vdim: int, step_bias: torch.Tensor, *,
                 scale: float = 1.0, tau: float = 1.0, rate: Optional[torch.Tensor] = None, up: Optional[torch.Tensor] = None,
                 skip: Optional[torch.Tensor] = None, device=None):
        if heads % key_heads:
            raise ValueError("heads must be a multiple of key_heads")
        f32 = lambda t: None if t is None else t.to(device=device, dtype=torch.float32).contiguous()
        self._chunks: Optional[bool] = None
        self.step_bias, self.rate, self.up, self.skip = f32(step_bias), f32(rate), f32(up), f32(skip)
        self._args = FrLinearScan(decay=_lib.FR_DECAY_CHANNEL if decay == "channel" else _lib.FR_DECAY_HEAD, heads=heads,
                                  key_heads=key_heads, dim=dim, vdim=vdim, rank=0 if up is None else int(up.shape[1]),
                                  scale=scale, inv_tau=1.0 / tau, step_bias=ptr(self.step_bias), rate=ptr(self.rate),
                                  up=ptr(self.up), skip=ptr(self.skip))

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, step: torch.Tensor, state: torch.Tensor,
                batch: ForwardBatch, out: torch.Tensor) -> torch.Tensor:
        """q, k [T, key_heads * dim], v and out [T, heads * vdim], step fp32; ``state`` [rows, state floats]. bf16 prompts
        run in chunks on the tensor cores, short portions, decode steps and fp32 token after token."""
        require_cuda(q, k, v, step, state)
        a = FrLinearScan.from_buffer_copy(self._args)
        a.dtype = dtype_code(q.dtype)
        a.q, a.ldq, a.k, a.ldk, a.v, a.ldv = ptr(q), q.stride(0), ptr(k), k.stride(0), ptr(v), v.stride(0)
        a.out, a.ldo, a.step, a.ldstep = ptr(out), out.stride(0), ptr(step), step.stride(0)
        a.state, a.state_slots = ptr(state), ptr(batch.req_pool_indices)
        a.qo_indptr, a.pos = ptr(batch.qo_indptr), ptr(batch.positions)
        n_req, t, s = int(batch.req_pool_indices.numel()), int(q.shape[0]), stream_ptr(q.device)
        longest = 1 if batch.one_token else max(batch.extend_seq_lens)
        lib = _lib.load()
        if self._chunks is None:
            self._chunks = bool(lib.fr_linear_scan_chunks_fit(ctypes.byref(a)))
        row_portion = longest
        if self._chunks and a.dtype == 0 and longest > ROW_PORTION:
            row_portion = ROW_PORTION
            size = int(lib.fr_linear_scan_chunks_scratch(ctypes.byref(a), n_req, longest, t))
            scratch = torch.empty(size, dtype=torch.uint8, device=q.device)
            call("fr_linear_scan_chunks", ctypes.byref(a), n_req, longest, t, row_portion + 1, ptr(scratch), size, s)
        if longest <= row_portion or min(batch.extend_seq_lens) <= row_portion:
            call("fr_linear_scan_rows", ctypes.byref(a), n_req, row_portion, t, s)
        return out
