"""Host side of the Dibepel serving path on the CPU: configuration, registry, page manager, scheduler, and that the
tests' models are sharp enough for a mistake in a mechanism to show."""

import copy
import json

import pytest
import torch

from flashrec_b200 import registry
from flashrec_b200.dibepel import DibepelConfig
from flashrec_b200.engine import Request, Scheduler
from flashrec_b200.kvcache import PAGE, CacheSpec, SequenceManager
from flashrec_b200.lm_layers import MergedProjection, interleave_rows, pad_heads
from oracle import dibepel_oracle as O
from tests.dibepel_cases import CASES, make, tokens


def test_config_reads_sizes_and_borrowed_weights():
    cfg = DibepelConfig.from_json(CASES["ragged"])
    assert [cfg.owner(i) for i in range(5)] == [0, 1, 2, 0, 1]
    shapes = cfg.tensor_shapes()
    assert shapes["l0.mix.q"] == (6 * 2 * 20, 90) and shapes["l0.mix.k"] == (2 * 2 * 20, 90)
    assert shapes["l1.mix.v.conv"] == (3 * 40, 3) and shapes["l1.mix.talk"] == (6, 6)
    assert "l2.mlp.gate" not in shapes and "l2.rg2" not in shapes and "l3.norm1" not in shapes
    spec = cfg.layers[1].mixer.cache_spec()
    assert (spec.k_cols, spec.v_cols, spec.conv_channels) == (3 * 32, 3 * 48, 6 * 32 + 3 * 32 + 3 * 48)


def test_config_rejects_what_the_design_does_not_have():
    bad = copy.deepcopy(CASES["equal"])
    bad["layers"][0]["type"] = "attention_9"
    with pytest.raises(ValueError):
        DibepelConfig.from_json(bad)
    bad = copy.deepcopy(CASES["equal"])
    bad["layers"][0]["mlp"]["kind"] = "mixture"
    with pytest.raises(ValueError):
        DibepelConfig.from_json(bad)
    bad = copy.deepcopy(CASES["equal"])
    bad["layers"][0]["weights_of"], bad["layers"][1]["weights_of"] = 1, 0
    with pytest.raises(ValueError):
        DibepelConfig.from_json(bad).tensor_shapes() and DibepelConfig.from_json(bad).owner(0)


def test_registry_picks_the_family(tmp_path):
    assert registry.lookup(CASES["equal"]).name == "dibepel"
    assert registry.lookup({"architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3"}).name == "qwen3-fp8"
    with pytest.raises(ValueError):
        registry.lookup({"architecture": "Nothing"})
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "qwen3"}))
    with pytest.raises(NotImplementedError):
        registry.load_model(str(tmp_path), torch.float32)


def test_lowest_key_and_bounds():
    w, c = CacheSpec(1, 1, size=10, keep_first=3), CacheSpec(1, 1, mask="chunk", size=10)
    assert [w.lowest_key(p) for p in (0, 9, 10, 25)] == [0, 0, 1, 16]
    assert [c.lowest_key(p) for p in (0, 9, 10, 25)] == [0, 0, 10, 20]
    for spec in (w, c):
        for p in range(60):
            n = sum(1 for j in range(p + 1) if (spec.mask == "chunk" and j // 10 == p // 10)
                    or (spec.mask == "window" and (p - j < 10 or j < 3)))
            assert n <= spec.max_keys(59) and spec.lowest_key(p) <= p


def test_pages_are_given_back_and_reused():
    specs = [CacheSpec(1, 1, size=100, keep_first=4), CacheSpec(1, 1, mask="chunk", size=150)]
    m = SequenceManager(specs, n_pages=9, max_requests=2, max_seq=4000, device="cpu")
    m.open("a")
    seen = set()
    for _ in range(40):
        slots = m.extend("a", 50)
        assert 0 not in {s // PAGE for s in slots}  # the reserved page is never handed out
        assert all(s % PAGE == (m.length("a") - 50 + i) % PAGE for i, s in enumerate(slots))
        seen |= {s // PAGE for s in slots}
        m.trim("a")
        nxt = m.length("a")
        for spec in specs:  # everything the next position sees is still held
            for j in range(nxt):
                visible = nxt - j < 100 or j < 4 if spec.mask == "window" else j // 150 == nxt // 150
                assert not visible or j // PAGE in m.live["a"].pages
    assert m.length("a") == 2000 and len(seen) <= 8
    m.open("b")
    with pytest.raises(RuntimeError):
        m.extend("b", 64 * 9)
    assert m.length("b") == 0
    with pytest.raises(RuntimeError):
        m.open("c")
    m.close("a")
    m.close("b")
    assert m.free_pages == 8 and m.free_rows == 2


class FakeEngine:
    """Scheduling only: 'logits' name the number of tokens a request has in the cache."""

    vocab = 997

    def __init__(self, pages, rows, max_seq=4096):
        self.seqs = SequenceManager([CacheSpec(1, 1, size=1 << 20)], pages, rows, max_seq, "cpu")
        self.max_seq, self.max_requests = max_seq, rows
        self.cache, self.steps = {}, []

    def finish(self, req):
        if req in self.seqs.live:
            self.seqs.close(req)
            self.cache.pop(req)

    def step(self, entries):
        self.steps.append([len(e.tokens) for e in entries])
        rows = []
        for e in entries:
            if e.req not in self.seqs.live:
                self.seqs.open(e.req)
                self.cache[e.req] = []
            self.seqs.extend(e.req, len(e.tokens))
            self.cache[e.req] += list(e.tokens)
            for w in e.want:
                row = torch.zeros(self.vocab)
                row[sum(self.cache[e.req]) * 7 % self.vocab] = 1.0  # depends on the whole context
                rows.append(row)
        return torch.stack(rows) if rows else torch.empty((0, self.vocab))


def _expected(prompt, n):
    ctx = list(prompt)
    for _ in range(n):
        ctx.append(sum(ctx) * 7 % FakeEngine.vocab)
    return ctx[len(prompt):]


@pytest.mark.parametrize("pages,budget", [(200, 64), (200, 7), (7, 64)])
def test_scheduler_runs_every_request_whatever_the_budget_and_pages(pages, budget):
    eng = FakeEngine(pages, rows=4)
    sched = Scheduler(eng, budget)
    sched.sampler = lambda logits, params, steps: logits.argmax(1).tolist()
    prompts = [[(i * 37 + j) % 101 for j in range(n)] for i, n in enumerate((1, 150, 33, 64, 65, 200, 2))]
    for i, p in enumerate(prompts):
        sched.add(Request(i, p, 70))
    out = sched.run()
    assert {i: out[i] for i in out} == {i: _expected(p, 70) for i, p in enumerate(prompts)}
    assert max(sum(s) for s in eng.steps) <= budget
    assert eng.seqs.free_pages == pages - 1 and eng.seqs.free_rows == 4
    with pytest.raises(ValueError):
        sched.add(Request("x", [], 1))


def test_scheduler_reports_a_request_that_can_never_fit():
    sched = Scheduler(FakeEngine(3, rows=2), 64)
    sched.sampler = lambda logits, params, steps: logits.argmax(1).tolist()
    sched.add(Request(0, list(range(120)), 60))
    with pytest.raises(RuntimeError):
        sched.run()


def test_weight_layouts():
    w = torch.arange(2 * 3 * 5, dtype=torch.float32).view(6, 5)
    p = pad_heads(w, 3, 4)
    assert torch.equal(p.view(2, 4, 5)[:, :3], w.view(2, 3, 5)) and not p.view(2, 4, 5)[:, 3].any()
    g, u = torch.ones(40, 8), 2 * torch.ones(40, 8)
    il = interleave_rows(g, u)
    assert il.shape == (128, 8) and il[:32].eq(1).all() and il[32:64].eq(2).all() and not il[72:96].any()
    m = MergedProjection(8)
    m.add("store", torch.ones(40, 8))
    m.add("swiglu", il)
    m.add("sigmoid", torch.ones(7, 8), bias=torch.ones(7))
    m.finish(torch.float32, "cpu")
    starts = [sum(r.rows for r in m.ranges[:i]) for i in range(3)]
    assert starts == [0, 64, 192] and m.weight.shape == (224, 8)


def _fault(raw, what):
    bad = copy.deepcopy(raw)
    for e in bad["layers"]:
        m = e["mixer"]
        if what == "window" and e["type"] == "attention":
            m["mask"]["size"] += 1
        if what == "keep" and e["type"] == "attention":
            m["mask"]["keep_first"] += 1
        if what == "chunk" and e["type"] == "attention_2":
            m["mask"]["size"] += 1
        if what == "diff" and e["type"] == "attention":
            m["diff"] += 0.1
    return bad


@pytest.mark.parametrize("what", ["window", "keep", "chunk", "diff"])
def test_a_planted_mistake_shows_in_the_oracle(what):
    raw, cfg, w = make("ragged")
    t = tokens(cfg, 120)
    good, bad = O.forward(raw, w, t), O.forward(_fault(raw, what), w, t)
    err = ((good - bad)[60:].pow(2).mean(1) / good[60:].pow(2).mean(1)).sqrt()
    assert err.max() > 0.1, err.max()


@pytest.mark.parametrize("name", list(CASES))
def test_oracle_is_causal(name):
    raw, cfg, w = make(name)
    t = tokens(cfg, 24)
    assert torch.allclose(O.forward(raw, w, t)[:15], O.forward(raw, w, t[:15]), atol=1e-4)
