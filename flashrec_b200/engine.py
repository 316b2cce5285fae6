"""Serving of the decoder models: the step function over a ragged batch, and a scheduler with greedy or random
sampling on top of it.

``LMEngine.step`` runs each request's next tokens (a whole prompt, a portion of one, or one decoded token) from the
cache and state that earlier steps left, in one batch, and returns logits at the asked-for places. Batches of single
tokens are captured in CUDA graphs, one per batch size, and replayed. ``Scheduler`` admits requests while pages last,
decodes running requests and feeds prompts in portions within a token budget per step."""

from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from flashrec_b200.core import ForwardBatch
from flashrec_b200.kvcache import PAGE, SequenceManager
from flashrec_b200.lm_layers import ROW_PORTION
from flashrec_b200.sampling import Sampler, SamplingParams

TILE_ROWS = 128          # tokens per tensor-core attention tile


@dataclass
class StepEntry:
    """A request's next tokens and the places among them whose logits are wanted."""

    req: object
    tokens: Sequence[int]
    want: Sequence[int] = ()


@dataclass
class _DecodeGraph:
    graph: torch.cuda.CUDAGraph
    batch: ForwardBatch   # static inputs: every tensor the captured launches read lives here or in `rows`
    rows: torch.Tensor
    logits: torch.Tensor


class LMEngine:
    """Model + caches + slot table. ``max_tokens`` bounds the tokens that live requests hold at a time (a request's
    pages that no layer sees any more are given back), ``max_seq`` the length of one request."""

    GRAPH_SIZES = (1, 2, 4, 8, 16, 24, 32, 48, 64, 96, 128, 192, 256)

    def __init__(self, model, max_tokens: int, max_requests: int = 1, max_seq: Optional[int] = None,
                 use_graphs: bool = True):
        self.model = model
        self.device = torch.device(model.device)
        self.max_seq = int(max_seq if max_seq is not None else max_tokens)
        self.max_requests = int(max_requests)
        n_pages = 1 + self.max_requests + (int(max_tokens) + PAGE - 1) // PAGE
        self.caches = model.new_caches(n_pages, self.max_requests + 1)
        self.seqs = SequenceManager(model.cache_specs, n_pages, self.max_requests, self.max_seq, self.device)
        self.counters = torch.zeros(4096, dtype=torch.int32, device=self.device)
        self.use_graphs = bool(use_graphs)
        self._graphs: Dict[int, _DecodeGraph] = {}
        self._staging: Optional[torch.Tensor] = None

    # -- requests ---------------------------------------------------------------------------------------
    def finish(self, req) -> None:
        """Give back everything the request holds."""
        if req in self.seqs.live:
            self.seqs.close(req)

    def can_extend(self, req, n: int) -> bool:
        length = self.seqs.length(req)
        if req not in self.seqs.live and self.seqs.free_rows == 0:
            return False
        return length + n <= self.max_seq and self.seqs.pages_needed(length, n) <= self.seqs.free_pages

    # -- one step ---------------------------------------------------------------------------------------
    def step(self, entries: Sequence[StepEntry], on_layer=None) -> torch.Tensor:
        """Runs the entries' tokens; fp32 logits [wanted, vocab] in the order of entries and of ``want``. New
        requests are opened; nothing is changed when the batch does not fit."""
        entries = [e for e in entries if len(e.tokens) > 0]
        if not entries:
            return torch.empty((0, self.model.vocab), dtype=torch.float32, device=self.device)
        need = sum(self.seqs.pages_needed(self.seqs.length(e.req), len(e.tokens)) for e in entries)
        fresh = sum(e.req not in self.seqs.live for e in entries)
        if need > self.seqs.free_pages or fresh > self.seqs.free_rows:
            raise RuntimeError("the step does not fit into the cache")
        if len({id(e.req) if e.req is None else e.req for e in entries}) != len(entries):
            raise ValueError("a request appears twice in one step")
        if any(self.seqs.length(e.req) + len(e.tokens) > self.max_seq for e in entries):
            raise RuntimeError(f"a request would exceed {self.max_seq} tokens")
        vocab = self.model.vocab
        if any(not 0 <= int(t) < vocab for e in entries for t in e.tokens):
            raise ValueError("token id outside the vocabulary")
        if any(not 0 <= int(w) < len(e.tokens) for e in entries for w in e.want):
            raise ValueError("want: place outside the entry's tokens")
        # short portions first: their attention runs row by row, the rest in tiles
        order = sorted(range(len(entries)), key=lambda i: len(entries[i].tokens) > ROW_PORTION)
        start: Dict[int, int] = {}
        toks, pos, loc, tok_req, rows, req_rows, qo, pre, ext = [], [], [], [], [], [], [0], [], []
        tiles: List[Tuple[int, int, int]] = []
        n_row = 0
        for b, i in enumerate(order):
            e = entries[i]
            if e.req not in self.seqs.live:
                self.seqs.open(e.req)
            seq = self.seqs.live[e.req]
            n, first, t0 = len(e.tokens), seq.length, len(toks)
            start[i] = t0
            toks += [int(t) for t in e.tokens]
            loc += self.seqs.extend(e.req, n)
            pos += range(first, first + n)
            tok_req += [b] * n
            rows += [seq.row] * n
            req_rows.append(seq.row)
            qo.append(t0 + n)
            pre.append(first)
            ext.append(n)
            if n <= ROW_PORTION:
                n_row = t0 + n
            else:
                tiles += [(b, t0 + s, min(TILE_ROWS, n - s)) for s in range(0, n, TILE_ROWS)]
        want = [start[i] + int(w) for i, e in enumerate(entries) for w in e.want]
        one = len(toks) == len(entries)
        if one and self.use_graphs and on_layer is None and len(entries) <= self.GRAPH_SIZES[-1]:
            out = self._decode(toks, pos, loc, rows, want)
        else:
            batch, want_d = self._stage(toks, pos, loc, rows, req_rows, want, tok_req, qo, pre, ext, tiles, n_row, one)
            x, partials = self.model.forward(batch, self.caches, self.seqs.req_to_token, self.counters, on_layer=on_layer)
            out = self.model.logits(x, partials, want_d) if want else \
                torch.empty((0, vocab), dtype=torch.float32, device=self.device)
        for e in entries:
            self.seqs.trim(e.req)
        return out

    def _upload(self, cols64: Sequence[Sequence[int]], cols32: Sequence[Sequence[int]]) -> Tuple[list, list]:
        """Integer columns to the device in one copy from pinned memory (int64 first, int32 after)."""
        n64 = [len(c) for c in cols64]
        n32 = [(len(c) + 1) // 2 * 2 for c in cols32]
        total = sum(n64) + sum(n32) // 2
        host = torch.empty(total, dtype=torch.int64).pin_memory() if total else torch.empty(0, dtype=torch.int64)
        flat = host.numpy()
        o = 0
        for c, n in zip(cols64, n64):
            flat[o:o + n] = c
            o += n
        v32 = flat.view(np.int32)
        p = 2 * o
        for c, n in zip(cols32, n32):
            v32[p:p + len(c)] = c
            p += n
        dev = host.to(self.device, non_blocking=True)
        self._staging = host  # alive until the next step's copy replaces it
        out64, out32, o = [], [], 0
        for n in n64:
            out64.append(dev[o:o + n])
            o += n
        d32 = dev.view(torch.int32)
        p = 2 * o
        for c, n in zip(cols32, n32):
            out32.append(d32[p:p + len(c)])
            p += n
        return out64, out32

    def _stage(self, toks, pos, loc, rows, req_rows, want, tok_req, qo, pre, ext, tiles, n_row, one):
        (d_tok, d_pos, d_loc, d_rows, d_req, d_want), (d_tr, d_qo, d_tiles, d_len) = self._upload(
            [toks, pos, loc, rows, req_rows, want],
            [tok_req, qo, [v for t in tiles for v in t], [p + n for p, n in zip(pre, ext)]])
        batch = ForwardBatch(input_ids=d_tok, req_pool_indices=d_req, seq_lens=d_len, positions=d_pos,
                             out_cache_loc=d_loc, is_prefill=not one, extend_prefix_lens=pre, extend_seq_lens=ext, qo_indptr=d_qo, tok_req=d_tr, tok_rows=d_rows,
                             n_row_tokens=n_row, tiles=d_tiles.view(-1, 3), one_token=one, max_pos=max(pos))
        return batch, d_want

    # -- captured decode steps --------------------------------------------------------------------------
    def _decode(self, toks, pos, loc, rows, want) -> torch.Tensor:
        n = len(toks)
        size = next(s for s in self.GRAPH_SIZES if s >= n)
        g = self._graphs.get(size)
        if g is None:
            g = self._graphs[size] = self._capture(size)
        pad = [0] * (size - n)
        (cols,), _ = self._upload([toks + pad + pos + pad + loc + pad + rows + pad], [])
        g.batch._static.copy_(cols.view(4, size), non_blocking=True)
        g.graph.replay()
        if not want:
            return g.logits[:0]
        if want == list(range(n)):
            return g.logits[:n].clone()
        return g.logits[torch.tensor(want, dtype=torch.int64, device=self.device)]

    def _capture(self, size: int) -> _DecodeGraph:
        static = torch.zeros((4, size), dtype=torch.int64, device=self.device)
        batch = ForwardBatch(input_ids=static[0], req_pool_indices=static[3],
                             seq_lens=torch.ones(size, dtype=torch.int32, device=self.device), positions=static[1],
                             out_cache_loc=static[2], qo_indptr=torch.arange(size + 1, dtype=torch.int32, device=self.device),
                             tok_req=torch.arange(size, dtype=torch.int32, device=self.device), tok_rows=static[3],
                             n_row_tokens=size, tiles=None, one_token=True, max_pos=self.max_seq - 1)
        batch._static = static
        rows = torch.arange(size, dtype=torch.int64, device=self.device)

        def run():
            x, partials = self.model.forward(batch, self.caches, self.seqs.req_to_token, self.counters,
                                             static_max_pos=self.max_seq - 1)
            return self.model.logits(x, partials, rows)

        # the warm-up and the capture touch only the reserved row, page and state
        side = torch.cuda.Stream(self.device)
        side.wait_stream(torch.cuda.current_stream(self.device))
        with torch.cuda.stream(side):
            run()
        torch.cuda.current_stream(self.device).wait_stream(side)
        torch.cuda.synchronize(self.device)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            logits = run()
        return _DecodeGraph(graph, batch, rows, logits)


# -------------------------------------------------------------------------------------------------------
@dataclass
class Request:
    req: object
    prompt: List[int]
    max_new_tokens: int
    sampling: SamplingParams = field(default_factory=SamplingParams)
    stop_tokens: Tuple[int, ...] = ()
    fed: int = 0                                   # prompt (and, after a preemption, generated) tokens in the cache
    output: List[int] = field(default_factory=list)

    @property
    def context(self) -> List[int]:
        return self.prompt + self.output


class Scheduler:
    """First come, first served. Every step decodes the running requests and spends what is left of
    ``max_step_tokens`` on portions of waiting prompts. When pages run out, the youngest running request gives its
    pages back and starts again later."""

    def __init__(self, engine: LMEngine, max_step_tokens: int = 2048):
        self.engine = engine
        self.max_step_tokens = int(max_step_tokens)
        self.sampler = Sampler()
        self.waiting: deque = deque()
        self.running: List[Request] = []   # whole context in the cache but the last sampled token
        self.prefilling: List[Request] = []
        self.finished: Dict[object, Request] = {}

    def add(self, request: Request) -> None:
        if not request.prompt:
            raise ValueError("a request needs at least one prompt token")
        if len(request.prompt) + request.max_new_tokens > self.engine.max_seq:
            raise ValueError("prompt and new tokens exceed the engine's sequence length")
        if request.max_new_tokens <= 0:
            self.finished[request.req] = request
            return
        self.waiting.append(request)

    @property
    def done(self) -> bool:
        return not (self.waiting or self.running or self.prefilling)

    def _preempt(self) -> bool:
        pool = self.running if self.running else self.prefilling
        if not pool or (len(self.running) + len(self.prefilling)) <= 1:
            return False
        victim = pool.pop()
        self.engine.finish(victim.req)
        victim.fed = 0
        self.waiting.appendleft(victim)
        return True

    def _plan(self) -> List[Tuple[Request, int]]:
        seqs = self.engine.seqs
        while True:
            plan: List[Tuple[Request, int]] = [(r, 1) for r in self.running[: self.max_step_tokens]]
            budget = self.max_step_tokens - len(plan)
            pages = seqs.free_pages - sum(seqs.pages_needed(seqs.length(r.req), 1) for r, _ in plan)
            if pages < 0:
                if not self._preempt():
                    raise RuntimeError("the cache is too small for one request")
                continue
            while self.waiting and len(self.running) + len(self.prefilling) < self.engine.max_requests:
                self.prefilling.append(self.waiting.popleft())
            for r in self.prefilling:
                if budget <= 0:
                    break
                n = min(budget, len(r.context) - r.fed)
                have = seqs.length(r.req)
                while n > 0 and seqs.pages_needed(have, n) > pages:
                    n = min(n - 1, pages * PAGE + (-have) % PAGE)
                if n <= 0:
                    break
                pages -= seqs.pages_needed(have, n)
                budget -= n
                plan.append((r, n))
            if plan:
                return plan
            if not self._preempt():
                raise RuntimeError("the cache is too small for one request")

    def step(self) -> None:
        plan = self._plan()
        entries = []
        for r, n in plan:
            ctx = r.context
            last = r.fed + n == len(ctx)
            entries.append(StepEntry(r.req, ctx[r.fed:r.fed + n], [n - 1] if last else []))
        logits = self.engine.step(entries)
        ready = [r for (r, n), e in zip(plan, entries) if e.want]
        for r, n in plan:
            r.fed += n
        if not ready:
            return
        for r, tok in zip(ready, self.sampler(logits, [r.sampling for r in ready], [len(r.output) for r in ready])):
            r.output.append(tok)
            if r in self.prefilling:
                self.prefilling.remove(r)
                self.running.append(r)
            if len(r.output) >= r.max_new_tokens or tok in r.stop_tokens:
                self.running.remove(r)
                self.engine.finish(r.req)
                self.finished[r.req] = r

    def run(self) -> Dict[object, List[int]]:
        while not self.done:
            self.step()
        return {k: r.output for k, r in self.finished.items()}


def generate(engine: LMEngine, prompts: Sequence[Sequence[int]], max_new_tokens: int,
             sampling: Optional[SamplingParams] = None, max_step_tokens: int = 2048) -> List[List[int]]:
    """Tokens generated after each prompt, all requests scheduled together."""
    sched = Scheduler(engine, max_step_tokens)
    for i, p in enumerate(prompts):
        sched.add(Request(i, [int(t) for t in p], max_new_tokens, sampling or SamplingParams()))
    out = sched.run()
    return [out[i] for i in range(len(prompts))]
