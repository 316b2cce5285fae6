"""Dibepel on the GPU against the plain CPU oracle: every mechanism alone, whole models from whole prompts, portions,
single tokens and mixed batches, cache reuse, greedy generation through the scheduler, the trace runner and the command
line. float32 is compared tightly, bfloat16 within rounding."""

import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from oracle import dibepel_oracle as O
from tests.dibepel_cases import CASES, make, tokens

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = [torch.float32, torch.bfloat16]


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float(((a - b).pow(2).mean() / b.pow(2).mean().clamp_min(1e-30)).sqrt())


def tol(dtype, f32=3e-6, bf16=8e-3):
    return f32 if dtype == torch.float32 else bf16


@pytest.fixture(autouse=True)
def _clean_status():
    yield
    from flashrec_b200 import device_status

    assert device_status() == (0, 0)


# ---- mechanisms -----------------------------------------------------------------------------------------
def _rand(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,algo", [(1, 0), (2, 1), (3, 0), (4, 1), (5, 0), (8, 0), (8, 2), (1, 2), (9, 0), (64, 0), (130, 0),
                                    (700, 0)])
@pytest.mark.parametrize("k", [24, 90, 712])
def test_merged_projection(dtype, m, algo, k):
    from flashrec_b200.lm_layers import MergedProjection, ceil_to, interleave_rows

    dev = "cuda"
    x = _rand(m, k, seed=1).to(dtype)
    ws = {n: _rand(r, k, seed=2 + i, scale=k ** -0.5).to(dtype) for i, (n, r) in
          enumerate((("a", 40), ("kv", 72), ("gate", 90), ("up", 90), ("s", 51)))}
    bias = _rand(51, seed=9)
    proj = MergedProjection(k)
    proj.add("store", ws["a"])
    proj.add("store", ws["kv"])
    proj.add("swiglu", interleave_rows(ws["gate"], ws["up"]))
    proj.add("sigmoid", ws["s"], bias=bias)
    proj.add("store_f32", ws["a"])
    proj.finish(dtype, dev)
    h = torch.zeros((m, ceil_to(k, 8)), dtype=dtype, device=dev)
    h[:, :k] = x.to(dev)
    perm = torch.randperm(m + 5, generator=torch.Generator().manual_seed(3))[:m].to(dev)
    outs = [torch.full((m, 40), 9.0, dtype=dtype, device=dev), torch.full((m + 5, 72), 9.0, dtype=dtype, device=dev),
            torch.full((m, 96), 9.0, dtype=dtype, device=dev), torch.full((m, 56), 9.0, dtype=dtype, device=dev),
            torch.full((m, 41), 9.0, dtype=torch.float32, device=dev)]
    proj(h, outs, [None, perm, None, None, None], algo=algo)
    f = {n: x.double() @ w.double().t() for n, w in ws.items()}
    t = tol(dtype)
    assert rel(outs[0], f["a"]) < t
    assert rel(outs[1][perm], f["kv"]) < t
    untouched = torch.ones(m + 5, dtype=torch.bool)
    untouched[perm.cpu()] = False
    assert (outs[1].cpu()[untouched] == 9.0).all()
    assert rel(outs[2][:, :90], f["gate"] * torch.sigmoid(f["gate"]) * f["up"]) < t and not outs[2][:, 90:].any()
    assert rel(outs[3][:, :51], torch.sigmoid(f["s"] + bias.double())) < t and (outs[3][:, 51:] == 9.0).all()
    assert rel(outs[4][:, :40], f["a"]) < 3e-6 and (outs[4][:, 40:] == 9.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [1, 2, 7, 8, 9, 40, 200, 1500])
@pytest.mark.parametrize("n,ks", [(90, (48, 96)), (320, (1024, 2080)), (128, (64,)), (2048, (256, 512))])
def test_gated_update(dtype, m, n, ks):
    from flashrec_b200.lm_layers import gated_add, rms_norm

    dev = "cuda"
    x = _rand(m, n, seed=1)
    want = x.double().clone()
    parts = []
    for i, k in enumerate(ks):
        a, w = _rand(m, k, seed=2 + i).to(dtype), _rand(n, k, seed=5 + i, scale=k ** -0.5).to(dtype)
        ld = (n + 7) // 8 * 8
        g = torch.rand((m, ld), generator=torch.Generator().manual_seed(i)).to(dtype)
        want += g[:, :n].double() * (a.double() @ w.double().t())
        parts.append((a.to(dev), w.to(dev), g.to(dev) if not (i == 1 and m == 7) else None))
        if parts[-1][2] is None:
            want += (1 - g[:, :n].double()) * (a.double() @ w.double().t())
    xd = x.to(dev)
    pend = gated_add(xd, parts)
    assert (pend is not None) == (dtype == torch.bfloat16 and 8 < m <= 1024 and
                                  -(-m // 128) * -(-n // 64) * 2 <= 148)
    # the following norm adds what is pending
    weight = _rand(n, seed=8).to(dev)
    out = torch.empty((m, (n + 7) // 8 * 8), dtype=dtype, device=dev)
    rms_norm(xd, weight, 1.0, 1e-5, out, pend)
    assert rel(xd, want) < 3e-6
    ref = O.zero_centred_norm(want, weight.double().cpu(), 1e-5)
    assert rel(out[:, :n], ref) < tol(dtype)
    x2 = x.to(dev)
    assert gated_add(x2, parts, split=False) is None
    assert rel(x2, want) < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("w", [8, 77, 90, 320, 2048, 9000])
def test_norm_rows_and_offset(dtype, w):
    from flashrec_b200.lm_layers import Partials, ceil_to, rms_norm

    x, wt = _rand(9, w, seed=1), _rand(w, seed=2)
    pend = _rand(3, 9, w, seed=3)
    rows = torch.tensor([8, 0, 0, 5], device="cuda")
    out = torch.full((4, ceil_to(w, 8)), 5.0, dtype=dtype, device="cuda")
    xd = x.cuda()
    rms_norm(xd, wt.cuda(), 0.0, 1e-2, out, Partials(pend.cuda(), 3), rows)
    full = x.double() + pend.double().sum(0)
    ref = (O.rms(full, 1e-2) * wt.double())[rows.cpu()]
    assert rel(out[:, :w], ref) < tol(dtype) and not out[:, w:].any()
    assert torch.equal(xd.cpu(), x)  # picked rows: the stream itself stays


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_short_convolution_in_portions(dtype, taps):
    from flashrec_b200.core import ForwardBatch
    from flashrec_b200.lm_layers import short_conv

    c, lens = 300, [31, 9, 1]
    us = [_rand(n, c, seed=i).to(dtype) for i, n in enumerate(lens)]
    w = _rand(c, taps, seed=7)
    refs = [O.short_conv(u.double(), w.double()) for u in us]
    state = torch.full((5 * max(1, taps - 1) * c,), 3.0, dtype=dtype, device="cuda")  # stale: position 0 ignores it
    slots, done = [4, 1, 2], [0, 0, 0]
    got = [[], [], []]
    for portion in (2, 1, 7, 1, 1, 3, 40):
        live = [i for i in range(3) if done[i] < lens[i]]
        ns = [min(portion, lens[i] - done[i]) for i in live]
        u = torch.cat([us[i][done[i]:done[i] + n] for i, n in zip(live, ns)]).cuda()
        qo = [0]
        for n in ns:
            qo.append(qo[-1] + n)
        t = qo[-1]
        batch = ForwardBatch(
            input_ids=None, req_pool_indices=torch.tensor([slots[i] for i in live], device="cuda"), seq_lens=None,
            positions=torch.tensor([done[i] + e for i, n in zip(live, ns) for e in range(n)], device="cuda"),
            qo_indptr=torch.tensor(qo, dtype=torch.int32, device="cuda"),
            tok_req=torch.tensor([b for b, n in enumerate(ns) for _ in range(n)], dtype=torch.int32, device="cuda"),
            one_token=max(ns) == 1)
        a, b = torch.empty((t, 104), dtype=dtype, device="cuda"), torch.empty((t + 3, 196), dtype=dtype, device="cuda")
        move = torch.arange(t + 2, 2, -1, device="cuda")
        short_conv(u, w.cuda(), [(a, None, 0, 104), (b, move, 104, 196)], state, batch)
        y = torch.cat([a, b[move]], dim=1).cpu()
        for i, n, q0 in zip(live, ns, qo):
            got[i].append(y[q0:q0 + n])
            done[i] += n
    for g, r in zip(got, refs):
        assert rel(torch.cat(g), r) < tol(dtype)


def _mix_setup(kind, heads, kv, dim, vdim, size, keep, t, seed=0, scale=None, spikes=()):
    """Inputs of one attention layer in float32 on the CPU; ``spikes`` = (query, key) pairs whose score stands out."""
    maps = 2 if kind == "diff" else 1
    q, k = _rand(t, heads, maps, dim, seed=seed), _rand(t, kv, maps, dim, seed=seed + 1)
    v = _rand(t, kv, vdim, seed=seed + 2)
    rep = heads // kv
    for i, j in spikes:
        for h in range(heads):
            q[i, h] = k[j, h // rep] * 4.0
    scale = scale or dim ** -0.5
    mixer = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, diff=0.25,
                 mask=dict(size=size, keep_first=keep) if kind == "diff" else dict(size=size))
    return q, k, v, mixer


def _mix_run(kind, q, k, v, mixer, dtype, coef, lam, eps, portions, tensor_cores=None):
    """The product path over a shuffled page table, in portions; returns [T, heads * vdim]."""
    from flashrec_b200.core import ForwardBatch
    from flashrec_b200.kvcache import PAGE, CacheSpec
    from flashrec_b200.lm_layers import MixAttention, alibi_slopes

    t, heads, maps, dim = q.shape
    kv, vdim = v.shape[1], v.shape[2]
    mask = mixer["mask"]
    spec = CacheSpec(0, 0, mask="window" if kind == "diff" else "chunk", size=mask["size"], keep_first=mask.get("keep_first", 0))
    attn = MixAttention(kind, heads, kv, dim, vdim, mixer["scale"], spec, eps=eps, lam=lam, out_scale=1 - mixer["diff"],
                        coef=coef, slopes=None if kind == "diff" else torch.tensor(alibi_slopes(heads)))
    attn.bind("cuda")
    if tensor_cores is not None:
        assert attn.tensor_cores == tensor_cores
    dp, vp = attn.dim_p, attn.vdim_p
    pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1]))
    qp, kp, vp_ = pad(q, dp).reshape(t, -1).to(dtype).cuda(), pad(k, dp).reshape(t, -1).to(dtype), pad(v, vp).reshape(t, -1).to(dtype)
    n_pages = (t + PAGE - 1) // PAGE
    perm = torch.randperm(n_pages + 2, generator=torch.Generator().manual_seed(5))
    kc = torch.zeros(((n_pages + 2) * PAGE, kp.shape[1]), dtype=dtype)
    vc = torch.zeros(((n_pages + 2) * PAGE, vp_.shape[1]), dtype=dtype)
    slot = torch.tensor([int(perm[i // PAGE]) * PAGE + i % PAGE for i in range(t)])
    table = torch.zeros((3, n_pages * PAGE), dtype=torch.int32)
    table[2, :t] = slot.to(torch.int32)
    kc[slot], vc[slot] = kp, vp_
    kc, vc, table = kc.cuda(), vc.cuda(), table.cuda()
    counters = torch.zeros(4096, dtype=torch.int32, device="cuda")
    out, at, x = [], 0, 0
    while at < t:
        n = min(portions[x % len(portions)], t - at)
        x += 1
        tiles = torch.tensor([(0, s, min(128, n - s)) for s in range(0, n, 128)], dtype=torch.int32).cuda()
        b = ForwardBatch(input_ids=None, req_pool_indices=torch.tensor([2]).cuda(), seq_lens=None,
                         positions=torch.arange(at, at + n).cuda(), tok_req=torch.zeros(n, dtype=torch.int32).cuda(),
                         n_row_tokens=n if n <= 4 else 0, tiles=tiles, max_pos=at + n - 1)
        y = attn.forward(qp[at:at + n], kc, vc, table, b, counters)
        out.append(y.view(n, heads, vp)[:, :, :vdim].reshape(n, -1).float().cpu())
        at += n
    assert not counters.any()
    return torch.cat(out)


DIFF_SHAPES = [  # heads, kv, dim, vdim, window, keep, tokens
    (4, 2, 64, 128, 100, 5, 300), (3, 3, 20, 24, 64, 0, 200), (8, 1, 96, 112, 33, 70, 270), (1, 1, 128, 192, 1000, 1, 150),
    (2, 1, 16, 16, 1, 0, 100), (2, 2, 192, 64, 65, 64, 260), (6, 2, 40, 80, 63, 65, 210), (2, 1, 208, 48, 50, 3, 140),
    (2, 2, 32, 256, 80, 2, 130), (4, 2, 64, 128, 900, 4, 1500),
]
TALK_SHAPES = [  # heads, kv, dim, vdim, chunk, tokens
    (4, 2, 64, 64, 100, 300), (8, 2, 128, 128, 128, 300), (6, 6, 24, 40, 64, 200), (5, 1, 48, 96, 63, 200),
    (1, 1, 16, 192, 65, 150), (3, 1, 192, 176, 1000, 140), (16, 8, 32, 128, 1, 70), (2, 1, 200, 200, 90, 150), (12, 4, 80, 32, 70, 210),
    (4, 2, 128, 128, 700, 1300),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", DIFF_SHAPES)
def test_differential_attention(dtype, shape):
    heads, kv, dim, vdim, size, keep, t = shape
    edge = min(size, t - 2)
    spikes = [(i, j) for i, j in ((t - 1, t - edge), (t - 2, t - 2 - edge), (t - 3, keep), (t - 4, max(0, keep - 1)), (t - 5, 0))
              if 0 <= j <= i]  # just inside / outside the window, the last kept and the first dropped token
    q, k, v, mixer = _mix_setup("diff", heads, kv, dim, vdim, size, keep, t, spikes=spikes)
    if dtype == torch.bfloat16:
        q, k, v = q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float()
    lam, eps = 0.43, 1e-3
    ref = O.differential_attention(q.double(), k.double(), v.double(), mixer, lam, eps)
    for portions in ((t,), (97, 5, 2, 64, 1), (1,)):
        got = _mix_run("diff", q, k, v, mixer, dtype, None, lam, eps, portions, dim <= 192 and vdim <= 192)
        err = (got - ref.float()).pow(2).mean(1).sqrt() / ref.float().pow(2).mean(1).sqrt()
        assert err.max() < tol(dtype, 2e-5, 3e-2), (portions, int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", TALK_SHAPES)
def test_talking_attention(dtype, shape):
    heads, kv, dim, vdim, size, t = shape
    last = (t - 1) // size * size
    spikes = [(i, j) for i, j in ((t - 1, last), (t - 2, last - 1), (last, last - 1 if last else 0), (last - 1, 0)) if 0 <= j <= i]
    q, k, v, mixer = _mix_setup("talk", heads, kv, dim, vdim, size, 0, t, spikes=spikes)
    if dtype == torch.bfloat16:
        q, k, v = q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float()
    coef = _rand(heads, heads, seed=11) * 0.6 + torch.eye(heads)
    ref = O.talking_attention(q[:, :, 0].double(), k[:, :, 0].double(), v.double(), mixer, coef.double())
    for portions in ((t,), (97, 5, 2, 64, 1), (1,)):
        got = _mix_run("talk", q, k, v, mixer, dtype, coef, 0.0, 0.0, portions, dim <= 192 and vdim <= 192)
        err = (got - ref.float()).pow(2).mean(1).sqrt() / ref.float().pow(2).mean(1).sqrt()
        assert err.max() < tol(dtype, 2e-5, 3e-2), (portions, int(err.argmax()), float(err.max()))


# ---- whole models ---------------------------------------------------------------------------------------
_ORACLE = {}


def oracle(name, seed, n):
    key = (name, seed, n)
    if key not in _ORACLE:
        raw, cfg, w = make(name)
        _ORACLE[key] = O.forward(raw, w, tokens(cfg, n, seed))
    return _ORACLE[key]


def engine(name, dtype, max_tokens=1024, reqs=4, **kw):
    from flashrec_b200.dibepel import DibepelForCausalLM
    from flashrec_b200.engine import LMEngine

    raw, cfg, w = make(name)
    return LMEngine(DibepelForCausalLM(cfg, w, dtype, "cuda"), max_tokens, reqs, **kw)


def run_portions(eng, req, toks, portions):
    from flashrec_b200.engine import StepEntry

    out, at, x = [], 0, 0
    while at < len(toks):
        n = min(portions[x % len(portions)], len(toks) - at)
        x += 1
        out.append(eng.step([StepEntry(req, toks[at:at + n], list(range(n)))]).clone())
        at += n
    eng.finish(req)
    return torch.cat(out).cpu()


def check_rows(got, ref, dtype):
    """Every row close, and in bf16 (where the difference of two maps now and then cancels) the rows together closer."""
    err = (got - ref).pow(2).mean(1).sqrt() / ref.pow(2).mean().sqrt()
    assert err.max() < tol(dtype, 3e-5, 0.1), (int(err.argmax()), float(err.max()))
    assert err.pow(2).mean().sqrt() < tol(dtype, 3e-5, 0.03), float(err.pow(2).mean().sqrt())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_model_in_every_cut(name, dtype):
    raw, cfg, _ = make(name)
    n = 230
    ref = oracle(name, 3, n)
    toks = tokens(cfg, n, 3)
    eng = engine(name, dtype)
    for portions in ((n,), (1,), (2,), (64,), (63, 2, 65, 3, 1, 7), (190, 1)):
        check_rows(run_portions(eng, "r", toks, portions), ref, dtype)
    assert eng.seqs.free_rows == 4 and not eng.seqs.live


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_match_one_by_one(dtype):
    from flashrec_b200.engine import StepEntry

    raw, cfg, w = make("ragged")
    toks = tokens(cfg, 90, 4)
    ref = []
    O.forward(raw, w, toks, layers_out=ref)
    eng = engine("ragged", dtype)
    got = []
    eng.step([StepEntry(0, toks, [0])], on_layer=lambda i, x: got.append(x.cpu().clone()))
    assert len(got) == len(raw["layers"])
    for g, r in zip(got, ref):
        assert rel(g, r) < tol(dtype, 3e-6, 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch(dtype):
    from flashrec_b200.engine import StepEntry

    raw, cfg, _ = make("ragged")
    lens = {0: 230, 1: 40, 2: 131, 3: 7}
    eng = engine("ragged", dtype)
    refs = {r: oracle("ragged", 10 + r, n) for r, n in lens.items()}
    toks = {r: tokens(cfg, n, 10 + r) for r, n in lens.items()}
    at, got = {r: 0 for r in lens}, {r: [] for r in lens}
    plan = [{0: 70, 1: 1, 2: 2, 3: 3}, {0: 1, 1: 1, 2: 1, 3: 1}, {0: 130, 2: 64}, {0: 2, 1: 30, 2: 1}, {2: 1, 3: 1}, {0: 9, 1: 8, 2: 70, 3: 2},
            {0: 18}]
    for k, step in enumerate(plan):
        ids = list(step) if k % 2 else list(step)[::-1]
        entries = []
        for r in ids:
            n = min(step[r], lens[r] - at[r])
            if n > 0:
                entries.append(StepEntry(r, toks[r][at[r]:at[r] + n], list(range(n))))
        lg = eng.step(entries).cpu()
        o = 0
        for e in entries:
            got[e.req].append(lg[o:o + len(e.tokens)])
            o += len(e.tokens)
            at[e.req] += len(e.tokens)
    for r in lens:
        g = torch.cat(got[r])
        check_rows(g, refs[r][:g.shape[0]], dtype)
        assert g.shape[0] >= min(lens[r], 7)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_on_recycled_pages(dtype):
    """A sequence several times longer than the pool: pages are trimmed, handed to another request and come back."""
    from flashrec_b200.engine import StepEntry

    raw, cfg, _ = make("narrow" if dtype == torch.bfloat16 else "ragged")
    name = "narrow" if dtype == torch.bfloat16 else "ragged"
    n = 420
    toks, ref = tokens(cfg, n, 5), oracle(name, 5, n)
    other, other_ref = tokens(cfg, 60, 6), oracle(name, 6, 60)
    eng = engine(name, dtype, max_tokens=128, reqs=2, max_seq=n)
    got = [eng.step([StepEntry("long", toks[:20], list(range(20)))]).cpu()]
    k = 0
    for i in range(20, n):
        if i % 100 == 0:  # somebody else takes and returns pages meanwhile
            k += 1
            lg = eng.step([StepEntry(("o", k), other, list(range(60)))]).cpu()
            check_rows(lg, other_ref, dtype)
            eng.finish(("o", k))
        got.append(eng.step([StepEntry("long", [toks[i]], [0])]).cpu().clone())
    check_rows(torch.cat(got), ref, dtype)
    eng.finish("long")
    assert eng.seqs.free_pages == 128 // 64 + 2


def test_step_rejects_what_does_not_fit():
    from flashrec_b200.engine import StepEntry

    eng = engine("equal", torch.float32, max_tokens=128, reqs=1)
    with pytest.raises(ValueError):
        eng.step([StepEntry(0, [10 ** 6], [0])])
    with pytest.raises(ValueError):
        eng.step([StepEntry(0, [1, 2], [2])])
    with pytest.raises(RuntimeError):
        eng.step([StepEntry(0, [1] * 400, [])])
    with pytest.raises(RuntimeError):
        eng.step([StepEntry(0, [1], []), StepEntry(1, [1], [])])
    assert not eng.seqs.live and eng.step([]).shape == (0, 200)


def _greedy(raw, w, prompt, n):
    ctx, margin = list(prompt), []
    for _ in range(n):
        lg = O.forward(raw, w, ctx)[-1]
        top = lg.topk(2).values
        margin.append(float(top[0] - top[1]))
        ctx.append(int(lg.argmax()))
    return ctx[len(prompt):], margin


@pytest.mark.parametrize("budget,max_tokens", [(256, 1024), (20, 1024), (256, 192)])
def test_greedy_generation_through_the_scheduler(budget, max_tokens):
    from flashrec_b200.engine import generate

    raw, cfg, w = make("equal")
    prompts = [tokens(cfg, n, 20 + n) for n in (1, 2, 65, 30, 100)]
    want = [_greedy(raw, w, p, 12) for p in prompts]
    eng = engine("equal", torch.float32, max_tokens=max_tokens, reqs=3, max_seq=256)
    got = generate(eng, prompts, 12, max_step_tokens=budget)
    for g, (ids, margin) in zip(got, want):
        sure = next((i for i, m in enumerate(margin) if m < 1e-3), len(ids))  # ties may go either way
        assert g[:sure] == ids[:sure] and len(g) == 12
    assert not eng.seqs.live


def test_sampling_depends_on_the_request_alone():
    from flashrec_b200.engine import generate
    from flashrec_b200.sampling import Sampler, SamplingParams

    raw, cfg, _ = make("equal")
    prompts = [tokens(cfg, n, 40 + n) for n in (20, 45)]
    eng = engine("equal", torch.float32, reqs=4)
    sp = SamplingParams(temperature=0.8, top_k=20, seed=7)
    both = generate(eng, prompts, 8, sp)
    assert both == [generate(eng, [p], 8, sp)[0] for p in prompts]
    lg = torch.randn(5, 70000, generator=torch.Generator().manual_seed(0)).cuda()  # wider than one row top-k
    assert Sampler()(lg, [SamplingParams()] * 5, [0] * 5) == lg.argmax(1).tolist()
    counts = torch.zeros(3)
    row = torch.tensor([[2.0, 1.0, 0.0]]).cuda()
    for s in range(300):
        counts[Sampler()(row, [SamplingParams(temperature=1.0, seed=s)], [0])[0]] += 1
    assert (counts / 300 - torch.softmax(row.cpu()[0], 0)).abs().max() < 0.1


# ---- entry points ----------------------------------------------------------------------------------------
def _write_checkpoint(path, name):
    from safetensors.torch import save_file

    raw, cfg, w = make(name)
    path.mkdir()
    (path / "config.json").write_text(json.dumps(raw))
    save_file({k: v.contiguous() for k, v in w.items()}, str(path / "model.safetensors"))
    return raw, cfg, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    import numpy as np

    raw, cfg, w = _write_checkpoint(tmp_path / "m", "ragged")
    out = tmp_path / "out"
    out.mkdir()
    toks = tokens(cfg, 70, 8)
    steps = [dict(step=0, entries=[dict(id="a", tokens=toks[:50], want=[0, 49])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=toks[50:52], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=toks[52:53], want=[0])], end=[]),
             dict(step=3, entries=[dict(id="a", tokens=toks[53:], want=[16])], end=["a"]),
             dict(step=4, entries=[dict(id="b", tokens=toks[:9], want=[8])], end=["b"])]
    p = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "80"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True,
                       timeout=300)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    ref = O.forward(raw, w, toks)
    for step, rows in ((0, [0, 49]), (2, [52]), (3, [69]), (4, [8])):
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").copy()).view(len(rows), cfg.vocab)
        check_rows(got, ref[rows], getattr(torch, dtype))
    assert not (out / "1.f32").exists()


def test_command_line_generates(tmp_path):
    raw, cfg, w = _write_checkpoint(tmp_path / "m", "equal")
    prompt = tokens(cfg, 30, 9)
    p = subprocess.run([str(ROOT / "bin" / "generate"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                        "--max-new-tokens", "6", "--prompt", " ".join(map(str, prompt))], capture_output=True, text=True,
                       timeout=300)
    assert p.returncode == 0, p.stderr
    ids, margin = _greedy(raw, w, prompt, 6)
    sure = next((i for i, m in enumerate(margin) if m < 1e-3), 6)
    assert json.loads(p.stdout.splitlines()[-1])["tokens"][:sure] == ids[:sure]


def test_qwen3_runs_through_the_same_engine():
    """The FP8 model behind the step engine: portions, single tokens and batches agree with one whole prompt."""
    from flashrec_b200.decoder import Qwen3Config
    from flashrec_b200.engine import LMEngine, StepEntry, generate
    from flashrec_b200.qwen3_lm import random_qwen3_lm

    cfg = Qwen3Config(hidden_size=256, num_attention_heads=4, num_key_value_heads=2, intermediate_size=512, num_hidden_layers=2,
                      vocab_size=512)
    lm = random_qwen3_lm(cfg, "cuda", seed=3)
    eng = LMEngine(lm, 1024, 3)
    toks = tokens(type("C", (), {"vocab": 512}), 150, 1)
    whole = eng.step([StepEntry(0, toks, list(range(150)))]).cpu()
    eng.finish(0)
    for portions in ((100, 1), (33, 2, 64), (1,)):
        got = run_portions(eng, "p", toks, portions)
        err = (got - whole).pow(2).mean(1).sqrt() / whole.pow(2).mean(1).sqrt()
        assert err.max() < 0.15, (portions, float(err.max()))  # e4m3 roundings flip with the summation order
    out = generate(eng, [toks[:20], toks[20:90], toks[:1]], 5)
    assert [len(o) for o in out] == [5, 5, 5] and not eng.seqs.live
