"""The FP8 Qwen3 model (:mod:`flashrec_b200.decoder`) behind the interface that :class:`flashrec_b200.engine.LMEngine`
drives: the e4m3 pool lives on the engine's pages, the flat slot lists come from the engine's slot table, and the full
vocabulary head runs in bf16 on the rows that are asked for."""

from __future__ import annotations

from typing import List, Optional

import torch

from flashrec_b200.attention import AttentionBackend, TokenToKVPool, gather_kv_indices
from flashrec_b200.core import ForwardBatch
from flashrec_b200.decoder import Qwen3Config, Qwen3ForCausalLM
from flashrec_b200.kvcache import PAGE, CacheSpec
from flashrec_b200.lm_layers import MergedProjection
from flashrec_b200.weights import load_hf_config, load_weights


class Qwen3LM:
    def __init__(self, cfg: Qwen3Config, device):
        self.cfg, self.device = cfg, torch.device(device)
        self.vocab = cfg.vocab_size
        full = 1 << 30  # every key stays visible: nothing is trimmed
        row = cfg.num_key_value_heads * cfg.head_dim
        self.cache_specs = [CacheSpec(row, row, size=full) for _ in range(cfg.num_hidden_layers)]
        pool = TokenToKVPool(1, PAGE, cfg.num_key_value_heads, cfg.head_dim, torch.float8_e4m3fn, self.device)
        self.attn = AttentionBackend(pool, cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim)
        # captured decode steps keep pointing at this buffer: large enough that it is never replaced
        self.attn._shared_len = torch.zeros(4096, dtype=torch.int32, device=self.device)
        self.model = Qwen3ForCausalLM(cfg, self.attn, self.device)
        self.head: Optional[MergedProjection] = None

    def bind_head(self) -> None:
        self.head = MergedProjection(self.cfg.hidden_size)
        self.head.add("store_f32", self.model.lm_head_weight)
        self.head.finish(torch.bfloat16, self.device)

    def new_caches(self, n_pages: int, n_rows: int) -> TokenToKVPool:
        c = self.cfg
        pool = TokenToKVPool(c.num_hidden_layers, n_pages * PAGE, c.num_key_value_heads, c.head_dim, torch.float8_e4m3fn,
                             self.device, page_size=PAGE)
        self.attn.kv_pool = pool
        return pool

    def forward(self, batch: ForwardBatch, caches: TokenToKVPool, req_to_token: torch.Tensor, counters: torch.Tensor,
                static_max_pos: Optional[int] = None, on_layer=None):
        if on_layer is not None:
            raise NotImplementedError("Qwen3LM has no per-layer hook")
        req_to_token.index_put_((batch.tok_rows, batch.positions), batch.out_cache_loc.to(torch.int32))
        n = int(batch.req_pool_indices.numel())
        if static_max_pos is not None:  # captured decode step: buffers sized for any length
            batch.seq_lens = (batch.positions + 1).to(torch.int32)
            cap = n * (static_max_pos + 1)
        else:
            cap = n * (batch.max_pos + 1)
        batch.kv_indptr = torch.empty(n + 1, dtype=torch.int32, device=self.device)
        batch.kv_indices = torch.empty(cap, dtype=torch.int32, device=self.device)
        gather_kv_indices(req_to_token, batch.req_pool_indices, batch.seq_lens, out=batch.kv_indices,
                          indptr_out=batch.kv_indptr)
        batch.is_prefill = not batch.one_token
        self.attn.prepare(batch)
        return self.model.forward(batch), None

    def logits(self, hidden: torch.Tensor, partials, rows: torch.Tensor) -> torch.Tensor:
        out = torch.empty((int(rows.numel()), self.vocab), dtype=torch.float32, device=self.device)
        self.head(hidden.index_select(0, rows), [out])
        return out


def load_qwen3_lm(path: str, device) -> Qwen3LM:
    lm = Qwen3LM(load_hf_config(path), device)
    load_weights(lm.model, path, device, quantize_fp8=True)
    lm.bind_head()
    return lm


def random_qwen3_lm(cfg: Qwen3Config, device, seed: int = 0) -> Qwen3LM:
    """Random weights (benchmarks and tests); the head is the embedding."""
    lm = Qwen3LM(cfg, device)
    lm.model.init_random(seed)
    lm.model.lm_head_weight = lm.model.embed_tokens
    lm.bind_head()
    return lm
