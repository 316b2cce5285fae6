"""Kotipel on the GPU against the plain CPU oracle: every mechanism alone, whole models from whole prompts, portions,
single tokens and mixed batches, reuse of pages and state rows, greedy generation through the scheduler, the trace runner
and the command line. float32 is compared tightly, bfloat16 within rounding."""

import json
import subprocess
from pathlib import Path

import pytest
import torch

from oracle import kotipel_oracle as O
from tests.kotipel_cases import CASES, make, tokens

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = [torch.float32, torch.bfloat16]


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float(((a - b).pow(2).mean() / b.pow(2).mean().clamp_min(1e-30)).sqrt())


def tol(dtype, f32=3e-6, bf16=8e-3):
    return f32 if dtype == torch.float32 else bf16


def _rand(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


@pytest.fixture(autouse=True)
def _clean_status():
    yield
    from flashrec_b200 import device_status

    assert device_status() == (0, 0)


# ---- mechanisms -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,algo", [(1, 0), (2, 1), (3, 0), (8, 0), (8, 2), (9, 0), (130, 0), (700, 0)])
@pytest.mark.parametrize("k", [24, 90, 712])
def test_clamped_glu_and_gelu_ranges(dtype, m, algo, k):
    from flashrec_b200.lm_layers import MergedProjection, ceil_to, interleave_rows

    x = _rand(m, k, seed=1).to(dtype)
    ws = {n: _rand(r, k, seed=2 + i, scale=2 * k ** -0.5).to(dtype) for i, (n, r) in
          enumerate((("a", 40), ("gate", 90), ("up", 90), ("s", 51)))}
    table, ids = _rand(33, 5, 56, seed=7).to(dtype), torch.arange(m) * 7 % 33
    proj = MergedProjection(k)
    proj.add("store_f32", ws["a"])
    proj.add("glu_clamp", interleave_rows(ws["gate"], ws["up"]), limit=0.7, alpha=1.3, up_bias=0.5)
    proj.add("gelu_mul", ws["s"])
    proj.finish(dtype, "cuda")
    h = torch.zeros((m, ceil_to(k, 8)), dtype=dtype, device="cuda")
    h[:, :k] = x.cuda()
    outs = [torch.empty((m, 40), dtype=torch.float32, device="cuda"), torch.full((m, 96), 9.0, dtype=dtype, device="cuda"),
            torch.full((m, 56), 9.0, dtype=dtype, device="cuda")]
    proj(h, outs, algo=algo, mul=(table.cuda()[:, 3], ids.cuda()))
    f = {n: x.double() @ w.double().t() for n, w in ws.items()}
    g, u = f["gate"].clamp(max=0.7), f["up"].clamp(-0.7, 0.7)
    assert rel(outs[0], f["a"]) < 3e-6
    assert rel(outs[1][:, :90], g * torch.sigmoid(1.3 * g) * (u + 0.5)) < tol(dtype) and not outs[1][:, 90:].any()
    assert rel(outs[2][:, :51], O.gelu_tanh(f["s"]) * table[ids, 3, :51].double()) < tol(dtype)
    assert (outs[2][:, 51:] == 9.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("w", [8, 77, 90, 320, 2048, 4096, 9000])
def test_update_and_norm(dtype, w):
    from flashrec_b200.lm_layers import Partials, Pending, ceil_to, update_norm

    m, eps = 9, 1e-2
    shares = _rand(4, m, w, seed=12)
    x, wt, add = _rand(m, w, seed=1), _rand(w, seed=2), _rand(w, seed=3)
    pend = _rand(3, m, w, seed=4)
    ys = [torch.nn.functional.pad(_rand(m, w, seed=5 + i, scale=0.1 + i), (0, ceil_to(w, 8) - w)).to(dtype) for i in range(2)]
    wy = [_rand(w, seed=8 + i) for i in range(2)]
    dev = lambda ts: [t.cuda() for t in ts]
    for n_parts, use_p, use_add in ((0, False, False), (1, False, True), (2, False, False), (0, True, False), (2, True, True)):
        want = x.double()
        if use_p:
            want = want + pend.double().sum(0)
        for i in range(n_parts):
            want = want + (0.5, 1.0)[i] * O.rms(ys[i][:, :w].double(), eps) * wy[i].double()
        if use_add:
            want = want + add.double()
        p = Pending(Partials(pend.cuda(), 3) if use_p else None,
                    [(y, v, c) for y, v, c in zip(dev(ys), dev(wy), (0.5, 1.0))][:n_parts])
        a = add.cuda() if use_add else None
        out = torch.full((m, ceil_to(w, 8)), 5.0, dtype=dtype, device="cuda")
        xd = x.cuda()
        update_norm(xd, eps, out, wt.cuda(), 0.25, p, a)
        assert rel(xd, want) < 3e-6
        assert rel(out[:, :w], O.rms(want, eps) * (0.25 + wt.double())) < tol(dtype) and not out[:, w:].any()
        xd = x.cuda()
        update_norm(xd, eps, out, None, 0.0, p, a)  # the stream itself, rounded
        assert rel(out[:, :w], want) < tol(dtype)
        xd = x.cuda()
        update_norm(xd, eps, None, pending=p, add=a)
        assert rel(xd, want) < 3e-6
        rows = torch.tensor([8, 0, 0, 5], device="cuda")
        if n_parts == 2:  # one of the vectors as shares of a split product
            p.parts[1] = (Partials(shares.cuda(), 4), p.parts[1][1], 1.0)
            want = want + (O.rms(shares.double().sum(0), eps) - O.rms(ys[1][:, :w].double(), eps)) * wy[1].double()
        xd = x.cuda()
        update_norm(xd, eps, out[:4], wt.cuda(), 0.0, p, a, rows)
        assert torch.equal(xd.cpu(), x) and rel(out[:4, :w], (O.rms(want, eps) * wt.double())[rows.cpu()]) < tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [1, 7, 8, 9, 40, 200, 1500])
@pytest.mark.parametrize("n,k", [(90, 96), (130, 1040), (2048, 512)])
def test_products_that_update_copy_or_come_in_shares(dtype, m, n, k):
    from flashrec_b200.lm_layers import MergedProjection, ceil_to, gated_add, split_product

    a, w = _rand(m, k, seed=1).to(dtype), _rand(n, k, seed=2, scale=k ** -0.5).to(dtype)
    x = _rand(m, n, seed=3)
    ref = a.double() @ w.double().t()
    xd, copy = x.cuda(), torch.full((m, ceil_to(n, 8)), 7.0, dtype=dtype, device="cuda")
    gated_add(xd, [(a.cuda(), w.cuda(), None)], split=False, copy=copy)
    assert rel(xd, x.double() + ref) < 3e-6
    assert torch.equal(copy[:, :n], xd.to(dtype)) and not copy[:, n:].any()
    p = split_product(a.cuda(), w.cuda())
    if p is not None:
        assert p.buf.shape == (p.n, m, n) and rel(p.buf.sum(0), ref) < 3e-6
    proj = MergedProjection(k)
    proj.add("store", w[:n // 2])
    proj.add("sigmoid", w[n // 2:], bias=torch.ones(n - n // 2))
    proj.finish(dtype, "cuda")
    outs = [torch.empty((m, ceil_to(c, 8)), dtype=dtype, device="cuda") for c in (n // 2, n - n // 2)]
    proj(a.cuda(), outs)
    assert rel(outs[0][:, :n // 2], ref[:, :n // 2]) < tol(dtype)
    assert rel(outs[1][:, :n - n // 2], torch.sigmoid(ref[:, n // 2:] + 1)) < tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("groups,size", [(1, 60), (4, 15), (3, 22), (16, 128), (2, 1000), (1, 2048), (3, 4096), (1, 5000), (1, 9001)])
def test_gated_group_norm(dtype, groups, size):
    from flashrec_b200.lm_layers import ceil_to, group_norm

    m, n, eps = 11, groups * size, 1e-3
    ld = ceil_to(n, 8)
    y, z = (torch.nn.functional.pad(_rand(m, n, seed=s), (0, ld - n)).to(dtype) for s in (1, 2))
    yd, zd = y[:, :n].double(), z[:, :n].double()
    norm = lambda u: O.rms(u.view(m, groups, size), eps).reshape(m, n)
    for w in (_rand(size, seed=3), _rand(n, seed=4)):
        full = w.double().repeat(groups if w.numel() != n else 1)
        for gate, first, ref in ((None, False, norm(yd) * full), (z, False, norm(yd) * full * O.silu(zd)),
                                 (z, True, norm(yd * O.silu(zd)) * full)):
            out = torch.full((m, ld), 7.0, dtype=dtype, device="cuda")
            group_norm(y.cuda(), groups, size, w.cuda(), eps, out, None if gate is None else gate.cuda(), first)
            assert rel(out[:, :n], ref) < tol(dtype) and not out[:, n:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,rot", [(6, 2, 20, 12), (2, 2, 64, 64), (1, 1, 16, 2), (16, 4, 128, 96), (3, 1, 33, 0)])
def test_norm_and_rotation_of_queries_and_keys(dtype, heads, kv, dim, rot):
    from flashrec_b200.core import ForwardBatch
    from flashrec_b200.lm_layers import ceil_to, pad_heads, qk_norm_rope, rotary_frequencies, rotary_table

    spec = dict(dims=rot, base=7000.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=128))
    pos = [0, 1, 17, 1000, 31337, 200000]
    t, dp, eps = len(pos), ceil_to(dim, 16), 1e-3
    q, k = _rand(t, heads * dim, seed=1).to(dtype), _rand(t, kv * dim, seed=2, scale=0.3).to(dtype)
    wq, wk = 1 + 0.3 * _rand(heads * dim, seed=3), 1 + 0.3 * _rand(kv * dim, seed=4)
    pad = lambda x, n: pad_heads(x.t(), dim, dp).t().contiguous()
    cache = torch.zeros((20, kv * dp), dtype=dtype, device="cuda")
    loc = torch.tensor([3, 19, 0, 7, 8, 11], device="cuda")
    qd = pad(q, heads).cuda()
    freqs = rotary_frequencies(rot, 7000.0, spec["scaling"]) if rot else torch.zeros((0, 2))
    table = rotary_table(freqs.cuda(), torch.tensor(pos, device="cuda"))
    qk_norm_rope(qd, pad(k, kv).cuda(), heads, kv, dim, pad_heads(wq, dim, dp).cuda(), pad_heads(wk, dim, dp).cuda(), eps, table,
                 ForwardBatch(None, None, None, out_cache_loc=loc), cache)
    fr = O.rotary_frequencies(spec) if rot else []
    for x, w, n, got in ((q, wq, heads, qd), (k, wk, kv, cache[loc])):
        ref = (O.rms(x.double(), eps) * w.double()).view(t, n, dim)
        ref = torch.stack([O.rotate(ref[i], p, fr) for i, p in enumerate(pos)])
        got = got.view(t, n, dp)
        for i in range(t):
            assert rel(got[i, :, :dim], ref[i]) < tol(dtype, 1e-6, 5e-3), pos[i]
        assert not got[:, :, dim:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,c", [(1, 300), (2, 304), (4, 304), (4, 299), (7, 300)])
def test_short_convolution_with_bias_and_silu(dtype, taps, c):
    from flashrec_b200.core import ForwardBatch
    from flashrec_b200.lm_layers import short_conv

    lens = [31, 9, 1]
    us = [_rand(n, c, seed=i).to(dtype) for i, n in enumerate(lens)]
    w, bias = _rand(c, taps, seed=7), _rand(c, seed=8)
    refs = [O.short_conv(u.double(), w.double(), bias.double()) for u in us]
    state = torch.full((5 * max(1, taps - 1) * c,), 3.0, dtype=dtype, device="cuda")  # stale: position 0 ignores it
    slots, done, got = [4, 1, 2], [0, 0, 0], [[], [], []]
    for portion in (2, 1, 7, 1, 1, 3, 40):
        live = [i for i in range(3) if done[i] < lens[i]]
        ns = [min(portion, lens[i] - done[i]) for i in live]
        batch, qo = _batch(slots, live, ns, done)
        ld = (c + 7) // 8 * 8
        u = torch.zeros((qo[-1], ld), dtype=dtype, device="cuda")
        u[:, :c] = torch.cat([us[i][done[i]:done[i] + n] for i, n in zip(live, ns)]).cuda()
        out = torch.empty((qo[-1], ld), dtype=dtype, device="cuda")
        short_conv(u, w.cuda(), [(out, None, 0, c)], state, batch, bias.cuda(), silu=True)
        for i, n, q0 in zip(live, ns, qo):
            got[i].append(out[q0:q0 + n, :c].cpu())
            done[i] += n
    for g, r in zip(got, refs):
        assert rel(torch.cat(g), r) < tol(dtype)


def _batch(slots, live, ns, done):
    from flashrec_b200.core import ForwardBatch

    qo = [0]
    for n in ns:
        qo.append(qo[-1] + n)
    return ForwardBatch(
        input_ids=None, req_pool_indices=torch.tensor([slots[i] for i in live], device="cuda"), seq_lens=None,
        positions=torch.tensor([done[i] + e for i, n in zip(live, ns) for e in range(n)], device="cuda"),
        extend_seq_lens=list(ns), qo_indptr=torch.tensor(qo, dtype=torch.int32, device="cuda"),
        tok_req=torch.tensor([b for b, n in enumerate(ns) for _ in range(n)], dtype=torch.int32, device="cuda"),
        one_token=max(ns) == 1), qo


ATTN_SHAPES = [  # heads, kv, dim, vdim, tokens
    (4, 2, 64, 128, 300), (3, 3, 20, 24, 200), (8, 1, 96, 112, 270), (1, 1, 128, 192, 150), (2, 2, 192, 64, 260), (6, 2, 40, 80, 130),
    (2, 1, 208, 48, 140), (16, 4, 128, 128, 700),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", ATTN_SHAPES)
def test_causal_attention_with_head_gates(dtype, shape):
    """Over a shuffled page table, in portions; single keys stand out: the first, one at a page's edge, the query's own."""
    from flashrec_b200.core import ForwardBatch
    from flashrec_b200.kvcache import PAGE, CacheSpec
    from flashrec_b200.lm_layers import MixAttention

    heads, kv, dim, vdim, t = shape
    rep, scale = heads // kv, 1.3 * dim ** -0.5
    q, k, v = _rand(t, heads, dim, seed=1), _rand(t, kv, dim, seed=2), _rand(t, kv, vdim, seed=3)
    for i, j in ((t - 1, 0), (t - 2, 63), (t - 3, 64), (t - 4, t - 4), (t - 5, t - 4), (70, 0), (127, 128), (128, 127)):
        for h in range(heads):
            q[i, h] = k[j, h // rep] * 4.0  # j > i: a key that must stay hidden
    if dtype == torch.bfloat16:
        q, k, v = q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float()
    gate = _rand(t, heads, seed=4, scale=2.0)
    ref = O.causal_attention(q.double(), k.double(), v.double(), scale) * O.sigmoid(gate.double())[:, :, None]
    attn = MixAttention("plain", heads, kv, dim, vdim, scale, CacheSpec(0, 0, size=1 << 30))
    attn.bind("cuda")
    assert attn.tensor_cores == (dim <= 192 and vdim <= 192)
    dp, vp = attn.dim_p, attn.vdim_p
    pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1])).reshape(t, -1).to(dtype).cuda()
    qp, kp, vpd = pad(q, dp), pad(k, dp), pad(v, vp)
    n_pages = (t + PAGE - 1) // PAGE
    perm = torch.randperm(n_pages + 2, generator=torch.Generator().manual_seed(5))
    slot = torch.tensor([int(perm[i // PAGE]) * PAGE + i % PAGE for i in range(t)])
    kc = torch.zeros(((n_pages + 2) * PAGE, kv * dp), dtype=dtype, device="cuda")
    vc = torch.zeros(((n_pages + 2) * PAGE, kv * vp), dtype=dtype, device="cuda")
    table = torch.zeros((3, n_pages * PAGE), dtype=torch.int32, device="cuda")
    table[2, :t] = slot.to(torch.int32).cuda()
    kc[slot.cuda()], vc[slot.cuda()] = kp, vpd
    counters = torch.zeros(4096, dtype=torch.int32, device="cuda")
    for portions in ((t,), (97, 5, 2, 64, 1), (1,) if t < 200 else (t - 30, 1)):
        out, at, x = [], 0, 0
        while at < t:
            n = min(portions[min(x, len(portions) - 1)] if portions[-1] == 1 else portions[x % len(portions)], t - at)
            x += 1
            tiles = torch.tensor([(0, s, min(128, n - s)) for s in range(0, n, 128)], dtype=torch.int32).cuda()
            b = ForwardBatch(input_ids=None, req_pool_indices=torch.tensor([2]).cuda(), seq_lens=None,
                             positions=torch.arange(at, at + n).cuda(), tok_req=torch.zeros(n, dtype=torch.int32).cuda(),
                             n_row_tokens=n if n <= 4 else 0, tiles=tiles, max_pos=at + n - 1)
            y = attn.forward(qp[at:at + n], kc, vc, table, b, counters, None, gate[at:at + n].cuda())
            out.append(y.view(n, heads, vp)[:, :, :vdim].float().cpu())
            at += n
        got = torch.cat(out).reshape(t, -1)
        want = ref.float().reshape(t, -1)
        err = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean(1).sqrt()
        assert err.max() < tol(dtype, 2e-5, 2e-2), (portions, int(err.argmax()), float(err.max()))
    assert not counters.any()


SCANS = [  # decay, heads, key heads, dim, vdim, strength of the decays
    ("channel", 3, 3, 18, 22, 0.05), ("channel", 2, 2, 64, 64, 0.05), ("channel", 1, 1, 128, 128, 0.02), ("channel", 2, 2, 128, 64, 4.0),
    ("channel", 2, 2, 16, 16, 0.5), ("channel", 1, 1, 200, 96, 0.1), ("channel", 3, 3, 32, 256, 0.7),
    ("head", 6, 2, 12, 10, 0.2), ("head", 4, 1, 128, 64, 0.05), ("head", 4, 4, 64, 128, 1.0), ("head", 2, 1, 16, 16, 5.0),
    ("head", 3, 1, 256, 40, 0.1), ("head", 2, 2, 128, 128, 0.01), ("head", 4, 2, 64, 64, 60.0), ("channel", 3, 3, 32, 48, 1.2),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", SCANS)
def test_matrix_state_recurrences(dtype, case):
    """Three requests in portions of every size, on state rows that hold something else before; decays from nearly none
    to a state that is gone after two tokens."""
    _check_scan(dtype, case, [330, 150, 41], ((400,), (70, 1, 2, 64, 63, 200), (130, 128, 3, 1, 1, 300)))


@pytest.mark.parametrize("case", [SCANS[2], SCANS[3], SCANS[8], SCANS[10], SCANS[12]])
def test_recurrences_in_segments(case):
    """Prompts that are long enough for several CTAs to share one head's tokens."""
    _check_scan(torch.bfloat16, case, [2100, 700, 1030], ((2100,), (1200, 9, 1500)))


def _check_scan(dtype, case, lens, cuts):
    from flashrec_b200.kvcache import CacheSpec
    from flashrec_b200.lm_layers import LinearScan

    kind, heads, kh, dim, vdim, strength = case
    rank, scale, tau = 5, 0.3, 2.0
    bias = _rand(heads * dim if kind == "channel" else heads, seed=1)
    up = _rand(heads * dim, rank, seed=2, scale=0.7) if kind == "channel" else None
    rate, skip = (None, None) if kind == "channel" else (strength * torch.exp(_rand(heads, seed=3)), _rand(heads, seed=4))
    if kind == "channel":  # sigmoid(z) ^ (1 / tau) of about exp(-strength)
        bias = bias * 0.5 + torch.log(1 / torch.expm1(torch.tensor(tau * strength)))
    scan = LinearScan(kind, heads, kh, dim, vdim, bias, scale=scale, tau=tau, rate=rate, up=up, skip=skip, device="cuda")
    ins, refs = [], []
    for r, n in enumerate(lens):
        q, k, v = (_rand(n, h * d, seed=10 * r + s).to(dtype) for s, (h, d) in enumerate(((kh, dim), (kh, dim), (heads, vdim))))
        step = _rand(n, rank if kind == "channel" else heads, seed=10 * r + 5)
        ins.append((q, k, v, step))
        qd, kd, vd = q.double().view(n, kh, dim) * scale, k.double().view(n, kh, dim), v.double().view(n, heads, vdim)
        out = []
        if kind == "channel":
            a = torch.exp(-O.softplus(-(step.double() @ up.double().t() + bias.double())) / tau).view(n, heads, dim)
            out = [O.recurrence(qd[:, h], kd[:, h], vd[:, h], a[:, h]) for h in range(heads)]
        else:
            dt = O.softplus(step.double() + bias.double())
            for h in range(heads):
                o = O.recurrence(qd[:, h // (heads // kh)], kd[:, h // (heads // kh)], vd[:, h] * dt[:, h:h + 1],
                                 torch.exp(-rate.double()[h] * dt[:, h]))
                out.append(o + skip.double()[h] * vd[:, h])
        refs.append(torch.cat(out, dim=1))
    spec = CacheSpec(0, 0, state_heads=heads, state_dim=dim, state_vdim=vdim)
    slots = [5, 0, 3]
    for portions in cuts:
        state = torch.full((6, spec.state_floats), float("nan"), device="cuda")
        done, got, x = [0, 0, 0], [[], [], []], 0
        while any(d < n for d, n in zip(done, lens)):
            live = [i for i in (2, 0, 1) if done[i] < lens[i]]
            ns = [min(portions[(x + i) % len(portions)], lens[i] - done[i]) for i in live]
            x += 1
            batch, qo = _batch(slots, live, ns, done)
            q, k, v, step = (torch.cat([ins[i][j][done[i]:done[i] + n] for i, n in zip(live, ns)]).cuda() for j in range(4))
            out = scan.forward(q, k, v, step, state, batch, torch.empty((qo[-1], heads * vdim), dtype=dtype, device="cuda"))
            for i, n, q0 in zip(live, ns, qo):
                got[i].append(out[q0:q0 + n].cpu())
                done[i] += n
        for g, r in zip(got, refs):
            g = torch.cat(g).double()
            err = (g - r).pow(2).mean(1).sqrt() / (r.pow(2).mean(1).sqrt() + 0.02 * r.pow(2).mean().sqrt())
            assert err.max() < tol(dtype, 1e-5, 1e-2), (portions, int(err.argmax()), float(err.max()))


# ---- whole models ---------------------------------------------------------------------------------------
_ORACLE = {}


def oracle(name, seed, n):
    key = (name, seed, n)
    if key not in _ORACLE:
        raw, cfg, w = make(name)
        _ORACLE[key] = O.forward(raw, w, tokens(cfg, n, seed))
    return _ORACLE[key]


def engine(name, dtype, max_tokens=1024, reqs=4, **kw):
    from flashrec_b200.engine import LMEngine
    from flashrec_b200.kotipel import KotipelForCausalLM

    raw, cfg, w = make(name)
    return LMEngine(KotipelForCausalLM(cfg, w, dtype, "cuda"), max_tokens, reqs, **kw)


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
    """Every row close; in bf16 a row now and then amplifies rounding (a recurrence's output that nearly cancels is
    divided by its own root mean square): one in fifty may be further off."""
    err = (got - ref).pow(2).mean(1).sqrt() / ref.pow(2).mean().sqrt()
    assert err.max() < tol(dtype, 6e-5, 0.3), (int(err.argmax()), float(err.max()))
    assert (err > tol(dtype, 6e-5, 0.1)).sum() <= max(1, len(err) // 50)
    assert err.pow(2).mean().sqrt() < tol(dtype, 3e-5, 0.04), float(err.pow(2).mean().sqrt())


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
@pytest.mark.parametrize("name", ["ragged", "tiles"])
def test_layer_runs_match_one_by_one(name, dtype):
    from flashrec_b200.engine import StepEntry

    raw, cfg, w = make(name)
    toks = tokens(cfg, 90, 4)
    ref, got = [], []
    O.forward(raw, w, toks, layers_out=ref)
    eng = engine(name, dtype)
    eng.step([StepEntry(0, toks, [0])], on_layer=lambda i, x: got.append(x.cpu().clone()))
    assert len(got) == len(ref) == len(cfg.runs())
    for g, r in zip(got, ref):
        assert rel(g, r) < tol(dtype, 6e-6, 3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "tiles"])
def test_unequal_requests_in_one_batch(name, dtype):
    from flashrec_b200.engine import StepEntry

    raw, cfg, _ = make(name)
    lens = {0: 230, 1: 40, 2: 131, 3: 7}
    eng = engine(name, dtype)
    refs = {r: oracle(name, 10 + r, n) for r, n in lens.items()}
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
    assert at == lens
    for r in lens:
        check_rows(torch.cat(got[r]), refs[r], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_rows_and_pages_are_reused(dtype):
    """One request after the other, and one that decodes on while others come and go on freed rows and pages."""
    from flashrec_b200.engine import StepEntry

    name, n = "equal", 300
    raw, cfg, _ = make(name)
    toks, ref = tokens(cfg, n, 5), oracle(name, 5, n)
    other, other_ref = tokens(cfg, 60, 6), oracle(name, 6, 60)
    eng = engine(name, dtype, max_tokens=512, reqs=2)
    got = [eng.step([StepEntry("long", toks[:20], list(range(20)))]).cpu()]
    for i in range(20, n):
        if i % 50 == 0:
            lg = eng.step([StepEntry(("o", i), other, list(range(60)))]).cpu()
            check_rows(lg, other_ref, dtype)
            eng.finish(("o", i))
        got.append(eng.step([StepEntry("long", [toks[i]], [0])]).cpu().clone())
    check_rows(torch.cat(got), ref, dtype)
    eng.finish("long")
    for _ in range(3):
        check_rows(run_portions(eng, "again", other, (59, 1)), other_ref, dtype)
    assert eng.seqs.free_rows == 2


def test_recurrent_model_outgrows_its_pages():
    raw, cfg, _ = make("recurrent")
    n = 400
    eng = engine("recurrent", torch.float32, max_tokens=64, reqs=1, max_seq=n)
    check_rows(run_portions(eng, "r", tokens(cfg, n, 7), (30, 1, 64, 2)), oracle("recurrent", 7, n), torch.float32)


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
    want = [_greedy(raw, w, p, 8) for p in prompts]
    eng = engine("equal", torch.float32, max_tokens=max_tokens, reqs=3, max_seq=256)
    got = generate(eng, prompts, 8, max_step_tokens=budget)
    for g, (ids, margin) in zip(got, want):
        sure = next((i for i, m in enumerate(margin) if m < 1e-3), len(ids))  # ties may go either way
        assert g[:sure] == ids[:sure] and len(g) == 8
    assert not eng.seqs.live


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
