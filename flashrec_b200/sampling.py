"""Choice of the next token from fp32 logits: greedy through the library's row top-k, or a draw from the (top-k)
softmax at a temperature with a per-request seed."""

from __future__ import annotations

from dataclasses import dataclass
from typing import List, Sequence

import torch

from flashrec_b200.logits import topk_rows

_MAX_TOP_K = 1024
_TOPK_COLS = 32768  # columns per call of the row top-k (it keeps a row in shared memory)


def topk_wide(logits: torch.Tensor, k: int):
    """``topk_rows`` for any vocabulary: column blocks first, then their winners. Ties go to the smaller index."""
    n, cols = logits.shape
    if cols <= _TOPK_COLS:
        return topk_rows(logits, k)
    parts = []
    for c in range(0, cols, _TOPK_COLS):
        block = logits[:, c:c + _TOPK_COLS].contiguous()
        v, i = topk_rows(block, min(k, block.shape[1]))
        parts.append((v, i + c))
    vals, idx = torch.cat([p[0] for p in parts], dim=1), torch.cat([p[1] for p in parts], dim=1)
    v, pick = topk_rows(vals, k)
    return v, torch.gather(idx, 1, pick)


@dataclass(frozen=True)
class SamplingParams:
    temperature: float = 0.0  # 0: greedy
    top_k: int = 0            # 0: the most likely 1024
    seed: int = 0


class Sampler:
    """One token per row. A request's draws depend on its own seed and step alone, not on the batch."""

    def __call__(self, logits: torch.Tensor, params: Sequence[SamplingParams], steps: Sequence[int]) -> List[int]:
        vocab = int(logits.shape[1])
        k = 1
        for p in params:
            if p.temperature > 0:
                k = max(k, min(p.top_k or _MAX_TOP_K, _MAX_TOP_K, vocab))
        vals, idx = topk_wide(logits, k)
        vals, idx = vals.cpu(), idx.cpu()
        out = []
        for i, p in enumerate(params):
            if p.temperature <= 0:
                out.append(int(idx[i, 0]))
                continue
            n = min(p.top_k or _MAX_TOP_K, k)
            prob = torch.softmax(vals[i, :n].double() / p.temperature, dim=0)
            g = torch.Generator()
            g.manual_seed(p.seed * 1_000_003 + steps[i])
            out.append(int(idx[i, torch.multinomial(prob, 1, generator=g)]))
        return out
