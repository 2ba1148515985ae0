"""Host side of the layered decoder designs, without a GPU: configuration, registry, slots and step tables, scheduling,
sampling, the trace replay and the engine's request preparation, against a stand-in model."""
import io
import json
import os
import re
from types import SimpleNamespace

import pytest
import torch

from msa_b200 import _cabi_lm
from msa_b200.cache import PackedStep, RecurrentSpec, RingSpec, SequenceStateCache
from msa_b200.generate import choose_tokens
from msa_b200.hybrid_config import HybridConfig
from msa_b200.scheduler import Scheduler, SequenceRequest
from oracle import hybrid_oracle as O
from tests import hybrid_util as U

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_library_exports_what_the_header_declares():
    header = open(os.path.join(ROOT, "include", "msa_b200_lm.h")).read()
    header = re.sub(r"/\*.*?\*/", "", header, flags=re.S)
    declared = set(re.findall(r"\b(msa_lm_[a-z0-9_]+)\s*\(", header))
    assert declared == set(_cabi_lm.EXPORTS)
    from msa_b200.build import build
    build(only="lm")
    for name in _cabi_lm.EXPORTS:
        assert hasattr(_cabi_lm.lib(), name)


def test_configuration_reads_every_choice():
    c = HybridConfig.parse(U.MIXED)
    assert c.width == 88 and c.eps == 3e-4 and c.windows == (17, 33, 9)
    assert c.runs() == [(0, None)] + [(i, t) for t in range(3) for i in (1, 2, 3)] + [(4, None)]
    assert c.layers[0].mixer.channels == 2 * 2 * 24 + 4 * 20 and c.layers[2].mlp is None
    assert c.layers[1].mlp.limit == 1.5 and c.layers[2].mixer.rot_base == 77.0
    assert HybridConfig.parse(U.WIDE).runs() == [(i, None) for i in range(4)]
    bad = json.loads(json.dumps(U.WIDE))
    bad["layers"][0]["type"] = "unknown"
    with pytest.raises(ValueError, match="unknown mixer"):
        HybridConfig.parse(bad)
    bad = json.loads(json.dumps(U.MIXED))
    bad["loop"]["stop"] = 9
    with pytest.raises(ValueError, match="does not fit"):
        HybridConfig.parse(bad)


def test_configuration_of_the_parallel_frame():
    c = HybridConfig.parse(U.PAR_MIXED)
    assert c.structure.block == "parallel" and c.structure.norm_offset == 1.0 and not c.structure.tied
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur, c.logit_softcap) == (61, 31, 5, 9.0)
    assert c.windows == (17, 33) and c.runs() == [(0, None)] + [(i, t) for t in range(3) for i in (1, 2, 3)] + [(4, None)]
    att, ssd = c.layers[1].mixer, c.layers[2].mixer
    assert (att.heads, att.kv_heads, att.dim, att.vdim, att.rot_dims, att.rot_base, att.taps, att.window) == (6, 2, 20, 28, 12, 500.0, 3, 17)
    assert att.sink and att.gate and att.channels == 8 * 20 + 2 * 28
    assert (ssd.inner, ssd.channels, ssd.norm_groups, ssd.taps) == (72, 72 + 2 * 60, 2, 4) and c.layers[2].mlp is None
    odd = HybridConfig.parse(U.PAR_ODD)
    assert odd.bigram is None and odd.logit_softcap is None and odd.layers[3].mixer.rot_dims == 0
    bad = json.loads(json.dumps(U.PAR_MIXED))
    bad["layers"][1]["mixer"]["kv_heads"] = 4
    with pytest.raises(ValueError, match="multiple"):
        HybridConfig.parse(bad)
    bad = json.loads(json.dumps(U.PAR_MIXED))
    bad["layers"][2]["mixer"]["norm_groups"] = 5
    with pytest.raises(ValueError, match="divide"):
        HybridConfig.parse(bad)
    bad = json.loads(json.dumps(U.PAR_MIXED))
    bad["layers"][0]["mlp"] = U.moe(4, 2, 8, 1.0)
    with pytest.raises(ValueError, match="dense"):
        HybridConfig.parse(bad)
    with pytest.raises(ValueError, match="architecture"):
        HybridConfig.parse({**U.PAR_MIXED, "architecture": "Unheard"})


def test_registry_tells_designs_apart(tmp_path):
    from msa_b200.registry import design_of
    (tmp_path / "a").mkdir(), (tmp_path / "b").mkdir(), (tmp_path / "c").mkdir(), (tmp_path / "d").mkdir()
    (tmp_path / "d" / "config.json").write_text(json.dumps(U.PAR_ODD))
    assert design_of(str(tmp_path / "d")).name == "Nazerax" and design_of(str(tmp_path / "d")).serves == "states"
    (tmp_path / "a" / "config.json").write_text(json.dumps(U.ODD))
    (tmp_path / "b" / "config.json").write_text(json.dumps({"architectures": ["MSAForCausalLM"], "msa_config": {}}))
    (tmp_path / "c" / "config.json").write_text(json.dumps({"architectures": ["Something"]}))
    assert design_of(str(tmp_path / "a")).serves == "states"
    assert design_of(str(tmp_path / "b")).serves == "memory"
    with pytest.raises(ValueError, match="unknown architecture"):
        design_of(str(tmp_path / "c"))


def cpu_cache(n_slots=3, max_len=50):
    return SequenceStateCache([RingSpec(6, 8), RecurrentSpec(2, 3, 4, 20, 3), RingSpec(6, None)], n_slots, max_len, "cpu", torch.float32)


def test_slots_are_handed_out_and_taken_back():
    c = cpu_cache()
    assert c.ring[0].shape == (4, 8, 6) and c.ring[2].shape == (4, 50, 6) and c.scratch == 3      # one slot to spare
    assert c.state[1].shape == (4, 2, 3, 4) and c.conv[1].shape == (4, 2, 2, 20)
    slots = {s: c.acquire(s) for s in "abc"}
    assert sorted(slots.values()) == [0, 1, 2] and c.free_slots == 0
    with pytest.raises(RuntimeError):
        c.acquire("d")
    c.advance("b", 7)
    c.release("b")
    assert "b" not in c and c.acquire("d") == slots["b"] and c.length("d") == 0
    with pytest.raises(KeyError):
        c.acquire("d")


def test_state_of_every_kind_of_layer():
    c = SequenceStateCache([RingSpec(6, 8, channels=10, taps=4), RecurrentSpec(2, 3, 3, shift=12), RecurrentSpec(2, 5, 4, 18, 1)], 2, 50, "cpu",
                           torch.float32)
    assert c.conv[0].shape == (3, 2, 3, 10) and c.shift[1].shape == (3, 12) and 1 not in c.conv and c.conv[2].shape == (3, 2, 0, 18)
    assert c.state[1].shape == (3, 2, 3, 3) and c.last_token.shape == (3,) and c.last_token.dtype == torch.int32


def test_step_tables_put_single_tokens_first_and_find_the_wanted_rows():
    c = cpu_cache()
    for s, n in (("a", 20), ("b", 3), ("c", 0)):
        c.acquire(s)
        c.advance(s, n)
    step = PackedStep([("a", [1, 2, 3], [0, 2]), ("b", [4], [0]), ("c", [5, 6], [])], c, (8, None))
    assert step.token.tolist() == [4, 1, 2, 3, 5, 6] and step.pos.tolist() == [3, 20, 21, 22, 0, 1]
    assert step.cu.tolist() == [0, 1, 4, 6] and step.start.tolist() == [3, 20, 0] and step.tok_seq.tolist() == [0, 1, 1, 1, 2, 2]
    assert (step.n_tok, step.n_seq, step.n_decode, step.max_len) == (6, 3, 1, 3)
    assert step.want_rows.tolist() == [1, 3, 0]
    assert step.slot.tolist() == [c.slot("b"), c.slot("a"), c.slot("c")]
    narrow, wide = step.views[8], step.views[None]
    assert narrow.ctx_off.tolist() == [0, 7 + 3, 7 + 3 + 2] and narrow.old_off.tolist() == [0, 7, 7] and narrow.window == 8
    assert wide.ctx_off.tolist() == [0, 23, 25] and wide.n_old == 20 and wide.window == 50
    step.commit(c)
    assert (c.length("a"), c.length("b"), c.length("c")) == (23, 4, 2)
    with pytest.raises(ValueError, match="room"):
        PackedStep([("a", [0] * 28, [])], c, ())
    with pytest.raises(ValueError, match="outside"):
        PackedStep([("a", [0], [1])], c, ())
    with pytest.raises(ValueError, match="twice"):
        PackedStep([("a", [0], []), ("a", [0], [])], c, ())


class CountingModel:
    """Next token = (sum of everything the sequence was fed) mod vocab: any lost, doubled or swapped token shows."""
    config = SimpleNamespace(vocab=23, windows=())
    device = torch.device("cpu")

    def __init__(self):
        self.sums, self.steps = {}, []

    def new_cache(self, n_slots, max_len):
        return SequenceStateCache([RingSpec(1, 4)], n_slots, max_len, "cpu", torch.float32)

    def run(self, entries, cache):
        step = PackedStep(entries, cache, ())
        self.steps.append([(s, len(t)) for s, t, _ in entries])
        rows = []
        for s, toks, want in entries:
            if cache.length(s) == 0:
                self.sums[s] = 0
            for j, t in enumerate(toks):
                self.sums[s] += t
                if j in want:
                    rows.append(self.sums[s] % 23)
        step.commit(cache)
        return torch.nn.functional.one_hot(torch.tensor(rows, dtype=torch.long), 23).float() if rows else torch.zeros(0, 23)

    def check_status(self):
        pass


def counted(prompt, n):
    total, out = sum(prompt), []
    for _ in range(n):
        out.append(total % 23)
        total += out[-1]
    return out


def test_scheduler_batches_unequal_requests_over_few_slots():
    model = CountingModel()
    s = Scheduler(model, max_batch=2, max_len=64, portion=5, step_tokens=7)
    reqs = [SequenceRequest([(i * 7 + j) % 23 for j in range(n)], k) for i, (n, k) in enumerate([(13, 4), (1, 6), (5, 1), (22, 3), (2, 9)])]
    for r in reqs:
        s.submit(r)
    done = s.run()
    assert len(done) == 5 and s.cache.free_slots == 2
    for r in reqs:
        assert r.output == counted(r.tokens, r.max_new_tokens)
    assert all(len(st) <= 2 and sum(n for _, n in st) <= 7 for st in model.steps)
    with pytest.raises(ValueError):
        s.submit(SequenceRequest([1] * 60, 10))
    with pytest.raises(ValueError):
        s.submit(SequenceRequest([99], 1))


def test_scheduler_stops_at_an_end_token_and_cancels():
    model = CountingModel()
    s = Scheduler(model, max_batch=2, max_len=64)
    want = counted([3, 4], 8)
    r = SequenceRequest([3, 4], 8, eos_token_ids=[want[3]])
    gone = SequenceRequest([5], 8)
    s.submit(r), s.submit(gone)
    s.step()
    s.cancel(gone.id)
    s.run()
    assert r.output == want[:want.index(want[3]) + 1] and s.cache.free_slots == 2


def test_sampling_mixes_greedy_and_drawn_rows():
    logits = torch.tensor([[0.0, 5.0, 1.0], [4.0, 0.0, 3.9], [4.0, 0.0, 3.9]])
    g = lambda: torch.Generator().manual_seed(3)
    a = choose_tokens(logits, [0.0, 1.0, None], [None, 0.9, None], [None, g(), None])
    assert a[0] == 1 and a[1] in (0, 2) and a[2] == 0
    assert a == choose_tokens(logits, [0.0, 1.0, None], [None, 0.9, None], [None, g(), None])
    assert choose_tokens(logits[1:2], [1.0], [0.3], [g()]) == [0]            # the nucleus holds one token


def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from msa_b200.trace import replay
    model, said = CountingModel(), []
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": [1], "want": []}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": [2], "want": [0]}], "end": ["y"]}]
    cache = model.new_cache(1, 16)
    replay(model, cache, io.StringIO("\n".join(map(json.dumps, steps))), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and cache.free_slots == 1
    first = torch.frombuffer(bytearray((tmp_path / "0.f32").read_bytes()), dtype=torch.float32).view(2, 23)
    assert first.argmax(-1).tolist() == [5, 18] and not (tmp_path / "1.f32").exists()
    assert (tmp_path / "2.f32").stat().st_size == 4 * 23


def test_engine_prepares_state_requests_without_templates(tmp_path):
    from msa_b200.engine import GenerateConfig, MSAEngine
    from msa_b200.memory import ModelConfig
    from msa_b200.tools import NumberTokenizer
    (tmp_path / "config.json").write_text(json.dumps(U.ODD))
    e = MSAEngine(GenerateConfig(devices=[0, 1], max_generate_tokens=4, max_context=10), ModelConfig(model_path=str(tmp_path)), start=False,
                  tokenizer=NumberTokenizer())
    assert e.serves == "states"
    reqs, pads = e.prepare_requests(["1 2 3", [4, 5], "6"], 1)
    assert pads == 0 and [r.input_ids for r in reqs] == [[[1, 2, 3], [4, 5]], [[6]]]
    with pytest.raises(ValueError, match="max_context"):
        e.prepare_requests([[1] * 7], 2)
    with pytest.raises(ValueError, match="empty"):
        e.prepare_requests([[]], 3)


def test_oracle_state_carries_over_and_window_counts_the_token_itself():
    """The oracle's own corner stones, by hand."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v, gate, beta = r(9, 2, 3), r(9, 2, 3), r(9, 2, 4), torch.rand(9, 2, generator=g).double(), torch.rand(9, 2, generator=g).double()
    whole, s_end = O.delta_rule(q, k, v, gate, beta)
    a, s = O.delta_rule(q[:4], k[:4], v[:4], gate[:4], beta[:4])
    b, s = O.delta_rule(q[4:], k[4:], v[4:], gate[4:], beta[4:], s)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(s, s_end)
    assert O.window_mask(4, 2).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    x = torch.arange(1.0, 5.0).double()[:, None]
    taps = torch.tensor([[10.0, 1.0]]).double()
    assert torch.allclose(O.causal_conv_silu(x, taps), O.silu(torch.tensor([1.0, 12.0, 23.0, 34.0]).double()[:, None]))
    p = O.rotate_interleaved(torch.tensor([[1.0, 0.0, 0.0, 2.0]]).double(), torch.tensor([3]), 100.0)[0]
    c = torch.cos(torch.tensor([3.0, 0.3]).double()), torch.sin(torch.tensor([3.0, 0.3]).double())
    assert torch.allclose(p, torch.stack([c[0][0], c[1][0], -2 * c[1][1], 2 * c[0][1]]))


def test_oracle_of_the_parallel_mechanisms_by_hand():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # a bonus-less read-out sees earlier tokens only; a decay of zero forgets everything but the last one
    q, k, v, w = r(5, 1, 3), r(5, 1, 3), r(5, 1, 3), torch.rand(5, 1, 3, generator=g).double()
    out, _ = O.wkv_recurrence(q, k, v, w, torch.zeros(1, 3).double())
    assert float(out[0].abs().max()) == 0
    want = (q[2, 0] * (w[1, 0] * k[0, 0])).sum() * v[0, 0] + (q[2, 0] * k[1, 0]).sum() * v[1, 0]
    assert torch.allclose(out[2, 0], want)
    out, s = O.wkv_recurrence(q, k, v, torch.zeros_like(w), torch.ones(1, 3).double())
    assert torch.allclose(out[3, 0], (q[3, 0] * k[2, 0]).sum() * v[2, 0] + (q[3, 0] * k[3, 0]).sum() * v[3, 0])
    assert torch.allclose(s[0], torch.outer(k[4, 0], v[4, 0]))
    # the current token is read with its full step
    out, _ = O.ssd_recurrence(q, k, v, torch.log(w[..., 0]), torch.full((5, 1), 2.0).double())
    assert torch.allclose(out[1, 0], 2 * (q[1, 0] * k[1, 0]).sum() * v[1, 0] + 2 * w[1, 0, 0] * (q[1, 0] * k[0, 0]).sum() * v[0, 0])
    p = O.softmax_plus_one(torch.tensor([[0.0, float("-inf"), 0.0], [50.0, 0.0, 0.0]]).double())
    assert torch.allclose(p[0], torch.tensor([1 / 3, 0.0, 1 / 3]).double()) and float(p[1, 0]) > 1 - 1e-9
    x = torch.arange(1.0, 5.0).double()[:, None]
    assert O.causal_conv(x, torch.tensor([[10.0, 1.0]]).double(), torch.tensor([0.5]).double())[:, 0].tolist() == [1.5, 12.5, 23.5, 34.5]
    assert O.shifted(x)[:, 0].tolist() == [0.0, 1.0, 2.0, 3.0]
    y = O.group_norm(torch.tensor([[3.0, 4.0, 0.0, 2.0]]).double(), 2, 0.0)
    assert torch.allclose(y, torch.tensor([[3.0, 4.0, 0.0, 2.0]]).double() / torch.tensor([12.5, 12.5, 2.0, 2.0]).double().sqrt())
    cfg = {"embedding": {"bigram": {"buckets": 5, "mul_prev": 3, "mul_cur": 2}}}
    w = {"embed": torch.zeros(9, 1), "bigram": torch.arange(6.0)[:, None]}
    assert O.embedding(cfg, w, [4, 7, 4], torch.float64)[:, 0].tolist() == [5.0, (12 + 14) % 5, (21 + 8) % 5]
    rot = O.rotate_leading(torch.tensor([[1.0, 0.0, 7.0]]).double(), torch.tensor([2]), 100.0, 2)[0]
    assert torch.allclose(rot, torch.tensor([torch.cos(torch.tensor(2.0)), torch.sin(torch.tensor(2.0)), 7.0]).double())
