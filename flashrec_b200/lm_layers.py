"""Building blocks of the 16/32-bit decoder models, each a thin wrapper around one C-ABI entry point with its
constants as parameters: merged projections with per-range epilogues, the gated two-part residual update, RMS norm
of the fp32 residual stream, the short causal convolution, and attention that mixes several softmax maps.

``dtype`` (bfloat16 or float32) is the type of weights, activations and caches; the residual stream is fp32 in
both. bfloat16 runs on the tensor cores, float32 is true 32-bit arithmetic throughout."""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import torch

from flashrec_b200 import _lib
from flashrec_b200._lib import FrConvOut, FrGatedPart, FrMixAttn, FrOutSegment, call, ptr, require_cuda, stream_ptr
from flashrec_b200.core import ForwardBatch
from flashrec_b200.kvcache import CacheSpec

SEG = {"store": _lib.FR_SEG_STORE, "swiglu": _lib.FR_SEG_SWIGLU, "sigmoid": _lib.FR_SEG_SIGMOID,
       "store_f32": _lib.FR_SEG_STORE_F32}
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


class MergedProjection:
    """All projections of one input as a single product: one weight ``[N, K]``, column ranges with their own
    epilogues (``fr_dense_proj``)."""

    def __init__(self, k: int):
        self.k = int(k)
        self._parts: List[torch.Tensor] = []
        self.ranges: List[ColumnRange] = []
        self.weight: Optional[torch.Tensor] = None

    def add(self, kind: str, weight: torch.Tensor, n: Optional[int] = None, bias: Optional[torch.Tensor] = None,
            align: int = 32) -> int:
        """Append a range; returns its index. ``swiglu`` takes an interleaved weight and must stay 64-aligned."""
        if kind == "swiglu":
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
        self.ranges.append(ColumnRange(kind, rows, int(n), bias))
        return len(self.ranges) - 1

    def finish(self, dtype: torch.dtype, device) -> None:
        w = torch.cat(self._parts, dim=0)
        self.weight = pad_cols(w, 8).to(device=device, dtype=dtype).contiguous()
        for r in self.ranges:
            if r.bias is not None:
                r.bias = r.bias.to(device=device, dtype=torch.float32).contiguous()
        self._parts = []

    def __call__(self, a: torch.Tensor, outs: Sequence[torch.Tensor],
                 row_maps: Optional[Sequence[Optional[torch.Tensor]]] = None, algo: int = 0) -> None:
        """``a`` [M, lda >= K padded]; ``outs`` one 2-D tensor per range (rows are ``row_maps[i][m]`` if given)."""
        require_cuda(a)
        segs = (FrOutSegment * len(self.ranges))()
        n0 = 0
        for i, r in enumerate(self.ranges):
            o = outs[i]
            rm = row_maps[i] if row_maps is not None else None
            segs[i] = FrOutSegment(SEG[r.kind], n0, r.n, 0, ptr(o), o.stride(0), ptr(rm), ptr(r.bias))
            n0 += r.rows
        w = self.weight
        call("fr_dense_proj", dtype_code(w.dtype), ptr(a), a.stride(0), ptr(w), w.stride(0), int(a.shape[0]), n0,
             int(w.shape[1]), segs, len(segs), algo, stream_ptr(a.device))


@dataclass
class Partials:
    """K shares of a residual update that the next norm adds (``fr_dense_gated_add`` with split K)."""

    buf: torch.Tensor
    n: int


def gated_add(x: torch.Tensor, parts: Sequence[Tuple[torch.Tensor, torch.Tensor, Optional[torch.Tensor]]],
              algo: int = 0, split: bool = True) -> Optional[Partials]:
    """``x += sum gate * (a @ w.T)`` over one or two ``(a, w, gate)`` parts; few-row products may come back as
    partials for the following ``rms_norm`` instead."""
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
    call("fr_dense_gated_add", code, arr, len(parts), ptr(x), x.stride(0), m, n, ptr(buf), n_splits, algo,
         stream_ptr(x.device))
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


def short_conv(u: torch.Tensor, weight: torch.Tensor, outs, state: torch.Tensor, batch: ForwardBatch) -> None:
    """Causal depthwise convolution of ``u`` [T, C] with ``weight`` [C, taps] fp32; ``outs`` = list of
    ``(tensor, row_map or None, first channel, channels)``; ``state`` [rows, taps - 1, C] is read and advanced."""
    require_cuda(u)
    arr = (FrConvOut * len(outs))()
    for i, (o, rm, c0, c) in enumerate(outs):
        arr[i] = FrConvOut(ptr(o), o.stride(0), ptr(rm), c0, c)
    call("fr_short_conv", dtype_code(u.dtype), ptr(u), u.stride(0), ptr(weight), int(weight.shape[1]),
         int(weight.shape[0]), arr, len(outs), ptr(state), ptr(batch.req_pool_indices), ptr(batch.tok_req),
         ptr(batch.qo_indptr), ptr(batch.positions), int(u.shape[0]), int(batch.req_pool_indices.numel()),
         1 if batch.one_token else 0, stream_ptr(u.device))


def alibi_slopes(heads: int) -> List[float]:
    """Distance-bias slopes 2^(-8 (h + 1) / heads)."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


class MixAttention:
    """Attention whose outputs are linear combinations of several softmax maps over the same values
    (``fr_mix_attn`` in the header). ``mix``: "diff" (two maps per head, second one subtracted ``lam`` times, output
    divided by its root mean square, times ``out_scale``) or "talk" (all heads' maps through the matrix ``coef``).
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
        self._args = FrMixAttn(mix=_lib.FR_MIX_DIFF if mix == "diff" else _lib.FR_MIX_TALK,
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
                batch: ForwardBatch, counters: torch.Tensor, max_keys: Optional[int] = None) -> torch.Tensor:
        """q [T, q_cols]; ``k`` / ``v`` the layer's caches (the batch's own keys are in already). bf16 prompts take
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
