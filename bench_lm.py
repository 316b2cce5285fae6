"""``bench.py --workload dibepel | kotipel``: prefill and decode throughput of a 16-bit decoder at sizes of real models
(random weights), beside the closest other model at equal size through the same engine (Dibepel beside the FP8 Qwen3,
Kotipel beside Dibepel), and the time of every kernel of a layer.

One JSON line: ``sizes[name][model]`` with ``prefill`` (tokens/s by tokens per step), ``decode`` (tokens/s by batch) and
``kernels`` (microseconds, achieved rate and fraction of the measured peak per kernel)."""

from __future__ import annotations

import json
import statistics
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent

# width, heads, kv heads, ff, layers timed
SIZES = {"1.7b": (2048, 16, 8, 6144, 8), "8b": (4096, 32, 8, 12288, 4)}
WINDOW, KEEP, CHUNK, VOCAB = 1024, 4, 1024, 32768


def dibepel_config(width, heads, kv_heads, ff, layers):
    diff = dict(heads=heads, kv_heads=kv_heads, dim=64, vdim=128, scale=64 ** -0.5, diff=0.2,
                mask=dict(size=WINDOW, keep_first=KEEP))
    talk = dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, conv=4, mask=dict(size=CHUNK))
    entries = [dict(type="attention" if i % 2 == 0 else "attention_2", mixer=diff if i % 2 == 0 else talk,
                    mlp=dict(kind="dense", ff=ff)) for i in range(layers)]
    return dict(architecture="Dibepel", vocab=VOCAB, width=width, norm=dict(eps=1e-5), embedding=dict(scale=1.0),
                layers=entries)


# per width: heads of the gated linear attention (64 x 128) and of the state-space recurrence (64 wide, state 128)
RECURRENT = {2048: (16, 64), 4096: (32, 128)}
SIDE = 256


def kotipel_config(width, heads, kv_heads, ff, layers):
    gla, ssm = RECURRENT[width]
    mlp = dict(kind="dense", ff=ff, limit=7.0)
    mamba = dict(type="mamba2", mlp=mlp, mixer=dict(heads=ssm, vdim=64, state=128, groups=8, conv=4, norm_groups=1))
    rot = dict(dims=128, base=5e5, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192))
    par = dict(type="parallel", mlp=mlp, mixer=dict(
        left=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, rot=rot, scale=128 ** -0.5),
        right=dict(heads=gla, dim=64, vdim=128, tau=16.0)))
    return dict(architecture="Kotipel", vocab=VOCAB, width=width, norm=dict(eps=1e-5), token_side=dict(dim=SIDE),
                layers=[mamba if i % 2 == 0 else par for i in range(layers)])


def event_time(torch, fn, iters: int, warmup: int = 3, rest: float = 0.0, flush=None) -> float:
    """Median milliseconds of ``fn(i)``; the caller's working set exceeds L2 or rotates through buffers, or ``flush`` (a
    buffer larger than L2) is written before every call. ``rest``: seconds of idling first, for single kernels that are set
    against the burst peak (the clocks recover from the power cap)."""
    if rest > 0:
        torch.cuda.synchronize()
        time.sleep(rest)
    for i in range(warmup):
        fn(i)
    torch.cuda.synchronize()
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(iters)]
    for i, (a, b) in enumerate(ev):
        if flush is not None:
            flush.zero_()
        a.record()
        fn(i)
        b.record()
    torch.cuda.synchronize()
    return statistics.median(a.elapsed_time(b) for a, b in ev)


def throughput(torch, make_engine, vocab, prefill_tokens, decode_batches, context, iters):
    from flashrec_b200.engine import StepEntry

    out = {"prefill": {}, "decode": {}}
    for n_req, n_tok in prefill_tokens:
        eng = make_engine(n_req * n_tok, n_req, n_tok)
        toks = [[(7 * t + 13 * r) % vocab for t in range(n_tok)] for r in range(n_req)]

        def once(i):
            eng.step([StepEntry(r, toks[r], [n_tok - 1]) for r in range(n_req)])
            for r in range(n_req):
                eng.finish(r)

        # host work (page lists, upload) is part of the step as a user calls it; events bracket the whole call
        ms = event_time(torch, once, max(3, iters // 2))
        out["prefill"][f"{n_req}x{n_tok}"] = {"ms": round(ms, 3), "tokens_per_s": round(n_req * n_tok / ms * 1e3)}
        del eng
        torch.cuda.empty_cache()
    for b in decode_batches:
        eng = make_engine(b * (context + 256), b, context + 256)
        for r0 in range(0, b, 8):
            eng.step([StepEntry(r, [(3 * t + r) % vocab for t in range(context)]) for r in range(r0, min(b, r0 + 8))])
        step = lambda i: eng.step([StepEntry(r, [(i + r) % vocab], [0]) for r in range(b)])
        for i in range(4):
            step(i)
        torch.cuda.synchronize()
        g = eng._graphs[next(s for s in eng.GRAPH_SIZES if s >= b)]
        ms_graph = event_time(torch, lambda i: g.graph.replay(), iters)
        ms = event_time(torch, step, iters)
        out["decode"][str(b)] = {"ms": round(ms, 4), "tokens_per_s": round(b / ms * 1e3), "graph_ms": round(ms_graph, 4)}
        del eng, g
        torch.cuda.empty_cache()
    return out


def kernel_times(torch, model, n_tok, peaks, iters=10):
    """Every kernel of a differential and of a talking layer alone, one prompt of ``n_tok`` tokens."""
    from flashrec_b200.engine import LMEngine, StepEntry
    from flashrec_b200.lm_layers import gated_add, rms_norm, short_conv

    eng = LMEngine(model, n_tok, 1, n_tok)
    grabbed = {}
    orig = type(model).forward

    def grab(self, batch, *a, **k):
        grabbed["batch"] = batch
        return orig(self, batch, *a, **k)

    model.forward = grab.__get__(model)
    eng.step([StepEntry(0, [t % model.vocab for t in range(n_tok)])])
    del model.forward
    batch, table, caches = grabbed["batch"], eng.seqs.req_to_token, eng.caches
    # what the step trimmed from the table's point of view is still there: the pages have not been handed out again
    dev, cfg = model.device, model.cfg
    bf = dict(dtype=torch.bfloat16, device=dev)
    res = {}
    visible = {"diff": sum(min(i + 1, WINDOW) + (KEEP if i >= WINDOW + KEEP else 0) for i in range(n_tok)),
               "talk": sum(i % CHUNK + 1 for i in range(n_tok))}

    def put(name, ms, flops=None, byts=None):
        r = {"us": round(ms * 1e3, 1)}
        if flops is not None:
            r.update(tflops=round(flops / ms / 1e9, 1), frac_of_measured=round(flops / ms / 1e9 / peaks["bf16_tflops"], 3))
        if byts is not None:
            r.update(gbs=round(byts / ms / 1e6), frac_of_measured=round(byts / ms / 1e6 / peaks["hbm_gbs"], 3))
        res[name] = r

    for kind, li in (("diff", 0), ("talk", 1)):
        layers = [l for i, l in enumerate(model.layers) if i % 2 == li]
        l = layers[0]
        w = cfg.width
        x = torch.randn((n_tok, w), device=dev)
        h = torch.empty((n_tok, w), **bf)
        put(f"{kind}.norm", event_time(torch, lambda i: rms_norm(x, l.norm_w, 1.0, cfg.eps, h), iters, rest=0.4), byts=n_tok * w * 6)
        outs, maps = [], []
        for r in l.proj.ranges:
            outs.append(torch.empty((n_tok, r.n), **bf))
            maps.append(None)
        n = sum(r.n * (2 if r.kind == "swiglu" else 1) for r in l.proj.ranges)
        put(f"{kind}.projections", event_time(torch, lambda i: layers[i % len(layers)].proj(h, outs, maps), iters, rest=0.4),
            flops=2 * n_tok * n * w)
        q = torch.randn((n_tok, l.attn.q_cols), device=dev).bfloat16()
        a = l.attn
        hsum = a.heads * (a.maps * a.dim_p + a.maps * a.vdim_p) if kind == "diff" else a.heads * (a.dim_p + a.vdim_p)
        put(f"{kind}.attention", event_time(
            torch, lambda i: a.forward(q, caches.k[li], caches.v[li], table, batch, eng.counters), iters, rest=0.4),
            flops=2 * visible[kind] * hsum)
        if l.conv_w is not None:
            u = outs[0]
            c = int(l.conv_w.shape[0])
            put(f"{kind}.conv", event_time(torch, lambda i: short_conv(
                u, l.conv_w, [(q, None, 0, a.q_cols), (caches.k[li], batch.out_cache_loc, a.q_cols, l.spec.k_cols),
                              (caches.v[li], batch.out_cache_loc, a.q_cols + l.spec.k_cols, l.spec.v_cols)],
                caches.conv[li], batch), iters, rest=0.4), byts=n_tok * c * 4)
        o = torch.randn((n_tok, a.heads * a.vdim_p), device=dev).bfloat16()
        act = torch.randn((n_tok, l.ff_cols), device=dev).bfloat16()
        g1, g2 = torch.rand((n_tok, w), device=dev).bfloat16(), torch.rand((n_tok, w), device=dev).bfloat16()
        put(f"{kind}.update", event_time(torch, lambda i: gated_add(
            x, [(o, layers[i % len(layers)].o_w, g1), (act, layers[i % len(layers)].down_w, g2)]), iters, rest=0.4),
            flops=2 * n_tok * w * (a.heads * a.vdim_p + l.ff_cols))
    return res


def qwen3_kernel_times(torch, lm, n_tok, peaks, iters=10):
    """The closest model's layer GEMMs and causal attention on as many tokens, one prompt."""
    from flashrec_b200.core import ForwardBatch
    from flashrec_b200.kernel.sglops import fp8_scaled_mm_silu_mul, per_token_quant_fp8

    c, dev = lm.cfg, lm.device
    x = torch.randn((n_tok, c.hidden_size), device=dev).bfloat16()
    q8, s = per_token_quant_fp8(x)
    l = lm.model.layers[0]
    res = {}
    peak8 = 2 * peaks["bf16_tflops"]

    def put(name, ms, flops, peak):
        res[name] = {"us": round(ms * 1e3, 1), "tflops": round(flops / ms / 1e9, 1),
                     "frac_of_measured": round(flops / ms / 1e9 / peak, 3)}

    qkv = l.self_attn.qkv_proj
    put("qkv", event_time(torch, lambda i: lm.model.layers[i % len(lm.model.layers)].self_attn.qkv_proj.forward_fp8(
        q8, s, (n_tok, c.hidden_size), torch.bfloat16), iters, rest=0.4), 2 * n_tok * qkv.out_features * c.hidden_size, peak8)
    put("gate_up", event_time(torch, lambda i: fp8_scaled_mm_silu_mul(
        q8, lm.model.layers[i % len(lm.model.layers)].mlp._gu_w, s, lm.model.layers[i % len(lm.model.layers)].mlp._gu_s), iters, rest=0.4),
        4 * n_tok * c.intermediate_size * c.hidden_size, peak8)
    y8, ys = per_token_quant_fp8(torch.randn((n_tok, c.intermediate_size), device=dev).bfloat16())
    r = torch.zeros((n_tok, c.hidden_size), **dict(dtype=torch.bfloat16, device=dev))
    put("down", event_time(torch, lambda i: lm.model.layers[i % len(lm.model.layers)].mlp.down_proj.forward_fp8_add_(y8, ys, r), iters, rest=0.4),
        2 * n_tok * c.intermediate_size * c.hidden_size, peak8)
    pool = lm.new_caches(n_tok // 64 + 2, 2)
    q = torch.randn((n_tok, c.num_attention_heads, c.head_dim), device=dev).bfloat16()
    b = ForwardBatch(input_ids=None, req_pool_indices=None, seq_lens=torch.tensor([n_tok], dtype=torch.int32, device=dev),
                     is_prefill=True, kv_indices=torch.arange(64, 64 + n_tok, dtype=torch.int32, device=dev),
                     kv_indptr=torch.tensor([0, n_tok], dtype=torch.int32, device=dev), extend_prefix_lens=[0],
                     extend_seq_lens=[n_tok], qo_indptr=torch.tensor([0, n_tok], dtype=torch.int32, device=dev))
    put("attention", event_time(torch, lambda i: lm.attn.forward(q, None, None, 0, b, skip_store=True), iters, rest=0.4),
        4 * c.num_attention_heads * c.head_dim * n_tok * (n_tok + 1) // 2, peaks["bf16_tflops"])
    del pool
    return res


def kotipel_kernel_times(torch, model, n_tok, peaks, iters=10):
    """Every kernel of a state-space and of a parallel layer alone, one prompt of ``n_tok`` tokens: the launches of one
    forward are recorded and each is repeated on the buffers it ran on."""
    from flashrec_b200 import lm_layers
    from flashrec_b200.engine import LMEngine, StepEntry

    cfg, w = model.cfg, model.cfg.width
    eng = LMEngine(model, n_tok, 1, n_tok)
    mamba, par = cfg.layers[0].mixer, cfg.layers[1].mixer
    ff, d = cfg.layers[0].ff, cfg.side_dim
    a, g = par.left, par.right
    gemm = lambda n, k: ("flops", 2 * n_tok * n * k)
    move = lambda cols: ("bytes", 2 * n_tok * cols)  # 16-bit columns in and out; the stream counts double
    keys = n_tok * (n_tok + 1) // 2
    mc, gk, gv = mamba.channels, g.heads * g.dim, g.heads * g.vdim
    tail = [("norm2", move(7 * w)), ("gate_up", gemm(2 * ff, w)), ("down", gemm(w, ff)), ("side.gate", gemm(d, w)), ("side.proj", gemm(w, d))]
    names = [("mamba.norm1", move(3 * w)), ("mamba.projections", gemm(mamba.inner + mc + mamba.heads, w)), ("mamba.conv", move(2 * mc)),
             ("mamba.recurrence", move(mc + mamba.inner + 2 * mamba.heads)), ("mamba.norm", move(3 * mamba.inner)),
             ("mamba.out", gemm(w, mamba.inner))]
    names += [("mamba." + n, c) for n, c in tail]
    names[6] = ("mamba.norm2", move(3 * w))
    n_par = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) + 2 * gk + 2 * gv + a.heads + model.layers[1].mixer.rank
    names += [("parallel.norm1", move(6 * w)), ("parallel.projections", gemm(n_par, w)),
              ("parallel.qk_rope", move(2 * (a.heads + a.kv_heads) * a.dim)),
              ("parallel.attention", ("flops", 2 * keys * a.heads * (a.dim + a.vdim))), ("parallel.left_out", gemm(w, a.heads * a.vdim)),
              ("parallel.recurrence", move(2 * gk + 2 * gv)), ("parallel.head_norm", move(3 * gv)), ("parallel.right_out", gemm(w, gv))]
    names += [("parallel." + n, c) for n, c in tail]
    launches, keep = [], []
    orig, empty = lm_layers.call, torch.empty

    def record(name, *args):
        if name not in ("fr_lm_embed", "fr_lm_rotary_table"):  # once a step
            launches.append((name, args))
        orig(name, *args)

    def kept(*args, **kw):
        keep.append(empty(*args, **kw))
        return keep[-1]

    lm_layers.call, torch.empty = record, kept
    try:
        eng.step([StepEntry(0, [t % model.vocab for t in range(n_tok)])])
    finally:
        lm_layers.call, torch.empty = orig, empty
    torch.cuda.synchronize()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=model.device)
    res = {}
    for (name, (what, amount)), (entry, args) in zip(names, launches):
        ms = event_time(torch, lambda _: orig(entry, *args), iters, rest=0.4, flush=flush)
        r = {"us": round(ms * 1e3, 1), "entry": entry}
        if what == "flops":
            r.update(tflops=round(amount / ms / 1e9, 1), frac_of_measured=round(amount / ms / 1e9 / peaks["bf16_tflops"], 3))
        else:
            r.update(gbs=round(amount / ms / 1e6), frac_of_measured=round(amount / ms / 1e6 / peaks["hbm_gbs"], 3))
        res[name] = r
    del keep
    return res


def _peaks():
    if (ROOT / "MEASURED_PEAKS.json").exists():
        p = json.loads((ROOT / "MEASURED_PEAKS.json").read_text())
        return {"bf16_tflops": p["bf16_tflops"], "hbm_gbs": p["hbm_gbs"], "source": "MEASURED_PEAKS.json"}
    return {"bf16_tflops": 1590.0, "hbm_gbs": 6650.0, "source": "fallback"}


def _weight_bytes(tree) -> int:
    """Bytes of the matrices that one pass over the layers reads (norms and tables of the token input aside)."""
    from flashrec_b200.lm_layers import MergedProjection

    n = 0
    for v in vars(tree).values():
        if isinstance(v, MergedProjection):
            n += v.weight.numel() * v.weight.element_size()
        elif hasattr(v, "numel") and getattr(v, "dim", lambda: 0)() == 2 and v.element_size() == 2 and v.is_contiguous():
            n += v.numel() * 2
        elif type(v).__module__.startswith("flashrec_b200.kotipel") and type(v).__name__.endswith("Mixer"):
            n += _weight_bytes(v)
    return n


def run_kotipel(args) -> None:
    import torch

    from bench import ClockSampler
    from flashrec_b200 import device_status
    from flashrec_b200.dibepel import DibepelConfig, DibepelForCausalLM
    from flashrec_b200.dibepel import random_tensors as dibepel_tensors
    from flashrec_b200.engine import LMEngine
    from flashrec_b200.kotipel import KotipelConfig, KotipelForCausalLM, random_tensors

    peaks, dev = _peaks(), torch.device("cuda:0")
    torch.cuda.set_device(dev)
    prefill, decode, iters = [(1, 8192), (8, 1024)], [1, 4, 16, 64, 256], max(args.steps, 10)
    line = {"metric": "kotipel_prefill_decode_tokens_per_s", "unit": "tokens/s", "n_gpus": 1, "data": "synthetic", "dtype": "bf16",
            "higher_is_better": True, "peaks": peaks, "sizes": {},
            "config": {"token_side": SIDE, "recurrent_heads": RECURRENT, "vocab": VOCAB, "context": 1024,
                       "l2": "weights and activations of a step exceed L2"}}
    with ClockSampler(0) as clk:
        for name, (width, heads, kv, ff, layers) in SIZES.items():
            cfg = KotipelConfig.from_json(kotipel_config(width, heads, kv, ff, layers))
            model = KotipelForCausalLM(cfg, random_tensors(cfg, device=dev), torch.bfloat16, dev)
            make = lambda tokens, reqs, seq: LMEngine(model, tokens, reqs, seq)
            rec = {"layers": layers, "width": width, "heads": heads, "kv_heads": kv, "ff": ff,
                   "kotipel": throughput(torch, make, cfg.vocab, prefill, decode, 1024, iters)}
            rec["kotipel"]["kernels_8192"] = kotipel_kernel_times(torch, model, 8192, peaks)
            w = sum(_weight_bytes(l) for l in model.layers) + model.head.weight.numel() * 2
            for b, r in rec["kotipel"]["decode"].items():
                r["weight_stream_frac_of_measured"] = round(w / r["graph_ms"] / 1e6 / peaks["hbm_gbs"], 3)
            del model
            torch.cuda.empty_cache()
            dcfg = DibepelConfig.from_json(dibepel_config(width, heads, kv, ff, layers))
            dib = DibepelForCausalLM(dcfg, dibepel_tensors(dcfg, device=dev), torch.bfloat16, dev)
            make = lambda tokens, reqs, seq: LMEngine(dib, tokens, reqs, seq)
            rec["dibepel"] = throughput(torch, make, dcfg.vocab, prefill, decode, 1024, iters)
            rec["dibepel"]["kernels_8192"] = kernel_times(torch, dib, 8192, peaks)
            w = sum(t.numel() for l in dib.layers for t in (l.proj.weight, l.o_w, l.down_w)) * 2 + dib.head.weight.numel() * 2
            for b, r in rec["dibepel"]["decode"].items():
                r["weight_stream_frac_of_measured"] = round(w / r["graph_ms"] / 1e6 / peaks["hbm_gbs"], 3)
            del dib
            torch.cuda.empty_cache()
            line["sizes"][name] = rec
    line["clocks"] = clk.summary()
    line["value"] = line["sizes"]["1.7b"]["kotipel"]["prefill"]["1x8192"]["tokens_per_s"]
    line["device_status"] = list(device_status())
    print(json.dumps(line), flush=True)


def run(args) -> None:
    import torch

    from bench import ClockSampler
    from flashrec_b200 import device_status
    from flashrec_b200.decoder import Qwen3Config
    from flashrec_b200.dibepel import DibepelConfig, DibepelForCausalLM, random_tensors
    from flashrec_b200.engine import LMEngine
    from flashrec_b200.qwen3_lm import random_qwen3_lm

    peaks = _peaks()
    dev = torch.device("cuda:0")
    torch.cuda.set_device(dev)
    prefill = [(1, 8192), (8, 1024)]
    decode = [1, 4, 16, 64, 256]
    line = {"metric": "dibepel_prefill_decode_tokens_per_s", "unit": "tokens/s", "n_gpus": 1, "data": "synthetic",
            "dtype": "bf16", "higher_is_better": True, "peaks": peaks, "sizes": {},
            "config": {"window": WINDOW, "keep_first": KEEP, "chunk": CHUNK, "vocab": VOCAB, "context": 1024,
                       "l2": "weights and activations of a step exceed L2"}}
    with ClockSampler(0) as clk:
        for name, (width, heads, kv, ff, layers) in SIZES.items():
            cfg = DibepelConfig.from_json(dibepel_config(width, heads, kv, ff, layers))
            model = DibepelForCausalLM(cfg, random_tensors(cfg, device=dev), torch.bfloat16, dev)
            make = lambda tokens, reqs, seq: LMEngine(model, tokens, reqs, seq)
            rec = {"layers": layers, "width": width, "heads": heads, "kv_heads": kv, "ff": ff,
                   "dibepel": throughput(torch, make, cfg.vocab, prefill, decode, 1024, max(args.steps, 10))}
            rec["dibepel"]["kernels_8192"] = kernel_times(torch, model, 8192, peaks)
            w = sum(t.numel() for l in model.layers for t in (l.proj.weight, l.o_w, l.down_w)) * 2
            head = model.head.weight.numel() * 2
            for b, r in rec["dibepel"]["decode"].items():
                r["weight_stream_frac_of_measured"] = round((w + head) / r["graph_ms"] / 1e6 / peaks["hbm_gbs"], 3)
            del model
            torch.cuda.empty_cache()
            qcfg = Qwen3Config(hidden_size=width, num_attention_heads=heads, num_key_value_heads=kv, head_dim=128,
                               intermediate_size=ff, num_hidden_layers=layers, vocab_size=VOCAB)
            lm = random_qwen3_lm(qcfg, dev)
            make = lambda tokens, reqs, seq: LMEngine(lm, tokens, reqs, seq)
            rec["qwen3"] = throughput(torch, make, VOCAB, prefill, decode, 1024, max(args.steps, 10))
            rec["qwen3"]["kernels_8192"] = qwen3_kernel_times(torch, lm, 8192, peaks)
            w8 = sum(l.self_attn.qkv_proj.in_features * l.self_attn.qkv_proj.out_features +
                     l.self_attn.o_proj.in_features * l.self_attn.o_proj.out_features + 3 * width * ff for l in lm.model.layers)
            for b, r in rec["qwen3"]["decode"].items():
                r["weight_stream_frac_of_measured"] = round((w8 + lm.head.weight.numel() * 2) / r["graph_ms"] / 1e6 / peaks["hbm_gbs"], 3)
            del lm
            torch.cuda.empty_cache()
            line["sizes"][name] = rec
    line["clocks"] = clk.summary()
    line["value"] = line["sizes"]["1.7b"]["dibepel"]["prefill"]["1x8192"]["tokens_per_s"]
    line["device_status"] = list(device_status())
    print(json.dumps(line), flush=True)
