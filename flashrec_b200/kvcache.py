"""Cache and state of the 16/32-bit decoder models: paged K/V per layer run, the slot table, the short
convolutions' and the recurrences' state, and the host-side manager that hands pages and rows to requests.

A page is 64 consecutive slots and holds positions ``[64 p, 64 p + 64)`` of one request (the tensor-core
attention loads a page as one tile). The slot table has the layout of ``ReqToTokenPool.req_to_token``
(kvcache/pool.py:142-183), so ``TokenToKVPool`` models and these share it. Slot page 0 and table row 0 are never
handed out: padded rows of a captured decode step write there."""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence

import torch

PAGE = 64


@dataclass(frozen=True)
class CacheSpec:
    """What one layer run keeps per sequence: cache columns, convolution state, a recurrent state matrix per head, and
    which keys stay visible."""

    k_cols: int
    v_cols: int
    conv_channels: int = 0
    conv_taps: int = 1
    # "window": the last `size` positions and the first `keep_first`; "chunk": the own chunk; "none": no keys at all
    mask: str = "window"
    size: int = 0
    keep_first: int = 0
    state_heads: int = 0  # recurrent state [state_dim, state_vdim] per head, fp32
    state_dim: int = 0
    state_vdim: int = 0

    @property
    def state_floats(self) -> int:
        """Per sequence; rows and columns are padded as the scan kernels lay them out."""
        return self.state_heads * ((self.state_dim + 7) // 8 * 8) * ((self.state_vdim + 15) // 16 * 16)

    def lowest_key(self, pos: int) -> int:
        """Lowest visible position (besides the kept first ones) of a query at ``pos``."""
        if self.mask == "none":
            return pos
        if self.mask == "chunk":
            return pos // self.size * self.size
        return max(0, pos - self.size + 1)

    def max_keys(self, pos: int) -> int:
        """Upper bound of the keys that any query at a position <= ``pos`` sees."""
        if self.mask == "none":
            return 0
        return min(self.size + (self.keep_first if self.mask == "window" else 0), pos + 1)


class LayerCaches:
    """Device memory of every layer run: ``k[i]``, ``v[i]`` [slots, cols], ``conv[i]`` [rows, taps - 1, C] and
    ``state[i]`` [rows, state floats], fp32 whatever the dtype.
    Zero-initialised: the tensor-core kernel multiplies unused slots of a page by zero weights."""

    def __init__(self, specs: Sequence[CacheSpec], n_pages: int, n_rows: int, dtype: torch.dtype, device):
        self.specs = list(specs)
        self.num_slots = int(n_pages) * PAGE
        kw = dict(dtype=dtype, device=device)
        self.k = [torch.zeros((self.num_slots, s.k_cols), **kw) for s in specs]
        self.v = [torch.zeros((self.num_slots, s.v_cols), **kw) for s in specs]
        self.conv = [torch.zeros(max(1, n_rows * (s.conv_taps - 1) * s.conv_channels), **kw) for s in specs]
        self.state = [torch.zeros((n_rows, s.state_floats), dtype=torch.float32, device=device) for s in specs]


@dataclass
class SequenceState:
    row: int
    length: int = 0
    pages: Dict[int, int] = field(default_factory=dict)  # page index in the sequence -> page of the pool


class SequenceManager:
    """Pages and table rows of the live requests. ``trim`` gives back the pages that no layer can see any more
    (windows and chunks bound what a sequence holds), so a sequence may be longer than the pool."""

    def __init__(self, specs: Sequence[CacheSpec], n_pages: int, max_requests: int, max_seq: int, device):
        if n_pages < 2 or max_requests < 1:
            raise ValueError("the cache needs a page and a row besides the reserved ones")
        self.specs = list(specs)
        self.max_seq = int(max_seq)
        self.req_to_token = torch.zeros((max_requests + 1, self.max_seq), dtype=torch.int32, device=device)
        self._free_pages: List[int] = list(range(n_pages - 1, 0, -1))
        self._free_rows: List[int] = list(range(max_requests, 0, -1))
        self.live: Dict[object, SequenceState] = {}
        self._keep = max((s.keep_first for s in specs), default=0)

    @property
    def free_pages(self) -> int:
        return len(self._free_pages)

    @property
    def free_rows(self) -> int:
        return len(self._free_rows)

    def pages_needed(self, length: int, extra: int) -> int:
        """New pages for ``extra`` more tokens after ``length``."""
        return (length + extra + PAGE - 1) // PAGE - (length + PAGE - 1) // PAGE

    def open(self, req) -> SequenceState:
        if req in self.live:
            raise KeyError(f"request {req!r} is live already")
        if not self._free_rows:
            raise RuntimeError("no free slot-table row")
        seq = SequenceState(self._free_rows.pop())
        self.live[req] = seq
        return seq

    def extend(self, req, n: int) -> List[int]:
        """Slots of the next ``n`` positions of ``req``; raises (and changes nothing) when the pool is short."""
        seq = self.live[req]
        if seq.length + n > self.max_seq:
            raise RuntimeError(f"request {req!r} would exceed {self.max_seq} tokens")
        if self.pages_needed(seq.length, n) > len(self._free_pages):
            raise RuntimeError("out of cache pages")
        out = []
        for pos in range(seq.length, seq.length + n):
            p = pos // PAGE
            if p not in seq.pages:
                seq.pages[p] = self._free_pages.pop()
            out.append(seq.pages[p] * PAGE + pos % PAGE)
        seq.length += n
        return out

    def trim(self, req) -> int:
        """Give back the pages that the next position sees in no layer. Returns how many."""
        seq = self.live[req]
        low = min((s.lowest_key(seq.length) for s in self.specs), default=0)
        gone = [p for p in seq.pages if (p + 1) * PAGE <= low and p * PAGE >= self._keep]
        for p in gone:
            self._free_pages.append(seq.pages.pop(p))
        return len(gone)

    def close(self, req) -> None:
        seq = self.live.pop(req)
        self._free_pages.extend(seq.pages.values())
        self._free_rows.append(seq.row)

    def length(self, req) -> int:
        seq: Optional[SequenceState] = self.live.get(req)
        return 0 if seq is None else seq.length
