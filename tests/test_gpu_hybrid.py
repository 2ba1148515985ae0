"""The layered decoder designs on the GPU against the plain oracle: every mechanism alone, whole prompts, portions,
decoding, mixed batches, slots used again, window edges, long decoding, and greedy generation through the engine."""
import pytest
import torch

from oracle import hybrid_oracle as O
from tests import hybrid_util as U

pytestmark = pytest.mark.gpu
EPS = 1e-5


@pytest.fixture(scope="module", autouse=True)
def exact_products():
    if not torch.cuda.is_available():
        pytest.skip("needs a GPU")
    torch.set_float32_matmul_precision("highest")


_MODELS = {}


def model(name, dtype, seed=0):
    from msa_b200.hybrid import HybridForCausalLM
    from msa_b200.hybrid_config import HybridConfig
    key = (name, dtype, seed)
    if key not in _MODELS:
        cfg = U.CONFIGS[name]
        _MODELS[key] = HybridForCausalLM(HybridConfig.parse(cfg), U.model_weights(name, seed, dtype), "cuda:0", dtype)
    return _MODELS[key]


def feed(m, cache, seq, toks, cuts):
    """Feeds ``toks`` in portions of the given sizes (the last one repeats); logits of every position."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(m.run([(seq, toks[at:at + n], range(n))], cache))
        at, k = at + n, k + 1
    return torch.cat(out)


def close(got, want, dtype):
    """fp32: every row.  bf16: rounding may still flip a close choice between experts for a position, and the recurrent
    states and windows carry that on, so the bulk of the rows is held to the bound."""
    e = U.row_errors(got, want)
    if dtype == torch.float32:
        assert float(e.max()) < 2e-4, (float(e.max()), int(e.argmax()))
    else:
        assert float(e.quantile(0.8)) < 0.06, (float(e.median()), float(e.quantile(0.8)))


DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
NAMES = pytest.mark.parametrize("name", list(U.CONFIGS))
BOTH = pytest.mark.parametrize("name", ["mixed", "par-mixed"])


# ------------------------------------------------------------------------------------------ mechanisms alone
class OneMixer:
    """A single mixer over hand-made inputs: what ``HybridForCausalLM.step`` does around one layer."""

    def __init__(self, kind, spec, weights, width, dtype, eps=EPS):
        from msa_b200 import hybrid as H, hybrid_config as C
        s = C.MIXERS[kind].parse(spec)
        w = H.Weights({"m." + k: v for k, v in weights.items()}, "cuda:0", dtype)
        self.mixer = H.MIXERS[kind](s, w, "m.", width, eps)
        w.check_all_used()
        self.dtype, self.windows = dtype, (s.window,) if hasattr(s, "window") else ()

    def cache(self, n_slots, max_len):
        from msa_b200.cache import SequenceStateCache
        return SequenceStateCache([self.mixer.state_spec], n_slots, max_len, "cuda:0", self.dtype)

    def run(self, cache, entries):
        """``entries`` = [(sequence, rows [n, width])] -> outputs in the same order."""
        from msa_b200 import lm_ops as K
        from msa_b200.cache import PackedStep
        step = PackedStep([(s, [0] * h.shape[0], range(h.shape[0])) for s, h in entries], cache, self.windows)
        packed = torch.empty((step.n_tok, entries[0][1].shape[1]), dtype=self.dtype, device="cuda:0")
        packed[step.want_rows.long()] = torch.cat([h for _, h in entries]).to("cuda:0", self.dtype)
        y = K.matmul(self.mixer.forward(packed, step, cache, 0), self.mixer.w_o)
        step.commit(cache)
        return list(y[step.want_rows.long()].float().cpu().split([h.shape[0] for _, h in entries]))


def mixer_case(kind, spec, width, seed, sharp=2.0):
    cfg = U.config(width, 8, [U.layer(kind, spec, None)])
    w = {k[len("l0.mix."):]: v for k, v in U.make_weights(cfg, seed, sharp).items() if k.startswith("l0.mix.")}
    return w, lambda h, s=spec: O.MIXERS[kind](h.double(), {k: v.double() for k, v in w.items()}, s, EPS)


def bf16_rows(n, width, seed):
    return torch.randn(n, width, generator=torch.Generator().manual_seed(seed)).to(torch.bfloat16).float()


MIXER_CASES = {
    "latent": ("latent_attention", U.latent(3, 20, 12, 28, 44, 17), 72),
    "latent-odd": ("latent_attention", U.latent(2, 7, 2, 5, 11, 6), 33),
    "latent-window1": ("latent_attention", U.latent(2, 8, 4, 8, 16, 1), 32),
    "latent-wide": ("latent_attention", U.latent(4, 128, 64, 128, 256, 150, base=10000.0), 128),
    "latent-64": ("latent_attention", U.latent(16, 64, 32, 64, 512, 70), 128),
    "latent-16": ("latent_attention", U.latent(5, 48, 16, 32, 96, 130), 64),
    "latent-96": ("latent_attention", U.latent(6, 96, 32, 96, 128, 300), 64),
    "delta": ("delta", U.delta(4, 2, 24, 20, 4), 72),
    "delta-odd": ("delta", U.delta(3, 1, 9, 7, 3), 33),
    "delta-taps1": ("delta", U.delta(2, 2, 16, 16, 1), 32),
    "delta-128": ("delta", U.delta(4, 2, 128, 128, 4), 96),
    "delta-64": ("delta", U.delta(6, 2, 64, 96, 4), 96),
    "delta-192": ("delta", U.delta(2, 1, 192, 64, 2), 64),
    "delta-32": ("delta", U.delta(2, 2, 32, 64, 4), 64),
    "group": ("attention", U.attention(6, 2, 20, 28, 17, 12, 3), 72),
    "group-odd": ("attention", U.attention(3, 1, 7, 5, 6, 2, 2), 33),
    "group-window1": ("attention", U.attention(4, 2, 8, 8, 1, 8, 4), 32),
    "group-taps6": ("attention", U.attention(4, 2, 16, 8, 40, 6, 6), 40),
    "group-plain": ("attention", U.attention(5, 5, 24, 16, 70, 0, 1), 40),
    "group-64": ("attention", U.attention(8, 2, 64, 64, 150, 32, 4), 128),
    "group-128": ("attention", U.attention(24, 2, 128, 128, 300, 128, 4), 128),
    "group-unequal": ("attention", U.attention(6, 3, 96, 40, 64, 30, 3), 96),
    "group-192": ("attention", U.attention(2, 1, 192, 160, 90, 64, 2), 64),
    "wkv": ("wkv", U.wkv(3, 24), 72),
    "wkv-odd": ("wkv", U.wkv(3, 7), 33),
    "wkv-16": ("wkv", U.wkv(1, 16), 32),
    "wkv-64": ("wkv", U.wkv(4, 64), 128),
    "wkv-72": ("wkv", U.wkv(2, 72), 64),
    "wkv-128": ("wkv", U.wkv(2, 128), 96),
    "wkv-160": ("wkv", U.wkv(2, 160), 64),
    "mamba2": ("mamba2", U.mamba2(6, 12, 20, 3, 2, 4), 72),
    "mamba2-odd": ("mamba2", U.mamba2(3, 5, 7, 1, 5, 3), 33),
    "mamba2-taps1": ("mamba2", U.mamba2(2, 16, 16, 2, 1, 1), 32),
    "mamba2-taps6": ("mamba2", U.mamba2(4, 16, 24, 2, 4, 6), 40),
    "mamba2-128": ("mamba2", U.mamba2(8, 64, 128, 1, 4, 4), 128),
    "mamba2-wide": ("mamba2", U.mamba2(4, 128, 64, 4, 8, 4), 96),
    "mamba2-192": ("mamba2", U.mamba2(2, 24, 192, 1, 1, 2), 64),
}


def mixer_close(got, want, dtype):
    """bf16: a unit norm or output norm of a nearly vanishing vector magnifies the rounding of a row here and there."""
    e = U.row_errors(got, want)
    if dtype == torch.float32:
        assert float(e.max()) < 5e-5, (float(e.max()), int(e.argmax()))
    else:
        assert float(e.max()) < 0.1 and (len(e) < 10 or float(e.median()) < 0.015), (float(e.max()), int(e.argmax()), float(e.median()))


@DTYPES
@pytest.mark.parametrize("case", list(MIXER_CASES))
def test_mixer_alone(case, dtype):
    """Whole, token by token, portions down to two tokens, and a mixed batch of unequal sequences."""
    kind, spec, width = MIXER_CASES[case]
    w, oracle = mixer_case(kind, spec, width, 5)
    m = OneMixer(kind, spec, w, width, dtype)
    h = [bf16_rows(n, width, 10 + n) for n in (300, 131, 1)]
    want = [oracle(x) for x in h]
    cache = m.cache(4, 320)

    def feed_rows(x, cuts):
        cache.acquire("s")
        out, at, k = [], 0, 0
        while at < x.shape[0]:
            n = min(cuts[k % len(cuts)], x.shape[0] - at)
            out.append(m.run(cache, [("s", x[at:at + n])])[0])
            at, k = at + n, k + 1
        cache.release("s")
        return torch.cat(out)

    for cuts in ((300,), (2, 3), (64, 1, 7), (97, 65, 2, 1, 128)):
        mixer_close(feed_rows(h[0], cuts), want[0], dtype)
    mixer_close(feed_rows(h[1], (1,)), want[1], dtype)
    # unequal sequences side by side, at different places of their lives
    for i in range(3):
        cache.acquire(i)
    at, out = [0, 0, 0], [[], [], []]
    for plan in ((40, 1, 1), (1, 70, 0), (150, 1, 0), (1, 1, 0), (2, 57, 0), (106, 1, 0)):
        entries = [(i, h[i][at[i]:at[i] + n]) for i, n in enumerate(plan) if n]
        for (i, x), y in zip(entries, m.run(cache, entries)):
            out[i].append(y)
            at[i] += x.shape[0]
    assert at == [300, 131, 1]
    for i in range(3):
        mixer_close(torch.cat(out[i]), want[i], dtype)


@DTYPES
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("window", [5, 64, 129])
def test_window_edge_is_exact(window, decode, dtype):
    """One early token's key answers every later query so loudly that the output is that token's value while the window
    holds it and something else one position later."""
    heads, dim, vdim, rank, width = 2, 16, 16, 32, 64
    spec = U.latent(heads, dim, 2, vdim, rank, window, base=1e9)
    w, oracle = mixer_case("latent_attention", spec, width, 3, sharp=0.3)
    n, loud = 3 * window + 7, window // 2 + 1
    h = bf16_rows(n, width, 8)
    h[:, :2] = 0.0
    h[loud, 0] = 60.0                                    # only this row drives latent direction 0
    h[:, 1] = 1.0                                        # every query asks for it
    w["dkv"][:, :2] = 0
    w["dkv"][0, :] = 0
    w["dkv"][0, 0] = 1.0
    w["q"][:, 1] = 0
    for hd in range(heads):
        w["q"][hd * (dim + 2), 1] = 6.0
        w["uk"][hd * dim, :] = 0
        w["uk"][hd * dim, 0] = 4.0
    want = oracle(h)
    wrong_out, wrong_in = oracle(h, {**spec, "mask": {"size": window - 1}}), oracle(h, {**spec, "mask": {"size": window + 1}})
    last_seen, first_gone = loud + window - 1, loud + window
    scale = want.pow(2).mean().sqrt()
    gap = lambda x, i: float((x[i] - want[i]).pow(2).mean().sqrt() / scale)
    assert gap(wrong_out, last_seen) > 0.3 and gap(wrong_in, first_gone) > 0.3        # a window one off would show
    m = OneMixer("latent_attention", spec, w, width, dtype)
    cache = m.cache(1, n)
    cache.acquire(0)
    if decode:
        got = torch.cat([m.run(cache, [(0, h[:loud + 1])])[0]] + [m.run(cache, [(0, h[i:i + 1])])[0] for i in range(loud + 1, n)])
    else:
        got = m.run(cache, [(0, h)])[0]
    e = U.row_errors(got, want)
    assert float(e[last_seen]) < 0.05 and float(e[first_gone]) < 0.05 and float(e.max()) < (1e-4 if dtype == torch.float32 else 0.05)


@DTYPES
def test_delta_state_remembers_a_far_write(dtype):
    """One token writes a large value with slow decay; hundreds of tokens later it is still what the read-out shows."""
    spec, width = U.delta(2, 1, 16, 16, 2), 48
    w, oracle = mixer_case("delta", spec, width, 4)
    w["A_log"][:] = -9.0
    w["b"][:, 0] = -1.0                                  # column 0 of h closes the write gate
    h = bf16_rows(420, width, 2)
    h[:, 0] = 12.0
    h[3, 0] = -12.0
    want = oracle(h)
    erased = h.clone()
    erased[3] = h[4]
    assert float(U.row_errors(oracle(erased)[-1:], want[-1:])) > 0.3                 # a lost state would show
    m = OneMixer("delta", spec, w, width, dtype)
    cache = m.cache(1, 420)
    cache.acquire(0)
    got = torch.cat([m.run(cache, [(0, x)])[0] for x in (h[:200], h[200:202], h[202:203], h[203:419], h[419:])])
    mixer_close(got[4:], want[4:], dtype)


@DTYPES
@pytest.mark.parametrize("spec", [U.moe(7, 2, 36, 1.5), U.moe(3, 1, 11, 3.0), U.moe(5, 5, 9, 0.5), U.moe(16, 4, 64, 2.0), U.moe(40, 6, 128, 1.0)],
                         ids=["7-2", "3-1", "all", "16-4", "40-6"])
@pytest.mark.parametrize("n", [1, 5, 300])
def test_experts_alone(spec, n, dtype):
    from msa_b200 import hybrid as H, hybrid_config as C, lm_ops as K
    width = 64 if spec["expert"]["ff"] % 8 == 0 else 35
    weights = U.make_weights(U.config(width, 8, [U.layer("delta", U.delta(1, 1, 4, 4, 2), spec)]), 6)
    w = {k[len("l0.mlp."):]: v for k, v in weights.items() if k.startswith("l0.mlp.")}
    w["router"] = w["router"] * 2
    h = bf16_rows(n, width, n) * 2                                                     # the clamps bite
    want = O.moe_ff(h.double(), {k: v.double() for k, v in w.items()}, spec)
    z = (h.double() @ w["router"].double().T + w["router.b"].double()).sort(dim=-1, descending=True).values
    top = spec["router"]["top"]
    sure = torch.ones(n, dtype=torch.bool) if top == z.shape[1] else (z[:, top - 1] - z[:, top]) > 1e-3
    ff = H.MixtureFeedForward(C.MoeSpec.parse(spec), H.Weights(w, "cuda:0", dtype), "", width)
    b = ff.branch(h.to("cuda:0", dtype))
    got = torch.empty((n, width), dtype=torch.float32, device="cuda:0")
    K.residual_norm(None, b.pop("y"), None, None, EPS, dtype, x_out=got, want_h=False, **b)
    e = U.row_errors(got, want)
    assert sure.sum() > 0.8 * n and float(e[sure].max()) < (2e-5 if dtype == torch.float32 else 3e-2)


@DTYPES
@pytest.mark.parametrize("width,ff", [(64, 96), (35, 33)])
def test_dense_feed_forward_alone(width, ff, dtype):
    from msa_b200 import hybrid as H, hybrid_config as C
    weights = U.make_weights(U.config(width, 8, [U.layer("delta", U.delta(1, 1, 4, 4, 2), U.dense(ff))]), 7)
    w = {k[len("l0.mlp."):]: v for k, v in weights.items() if k.startswith("l0.mlp.")}
    h = bf16_rows(77, width, 1)
    got = H.DenseFeedForward(C.DenseSpec(ff), H.Weights(w, "cuda:0", dtype), "", width).branch(h.to("cuda:0", dtype))["y"]
    e = U.row_errors(got, O.dense_ff(h.double(), {k: v.double() for k, v in w.items()}))
    assert float(e.max()) < (1e-5 if dtype == torch.float32 else 2e-2)


@DTYPES
@pytest.mark.parametrize("width", [64, 51, 2048])
def test_residual_step_alone(width, dtype):
    """Branch norm + add + next norm, the unnormed branch on a broadcast base, the gathered final norm, the embedding."""
    from msa_b200 import lm_ops as K
    g = torch.Generator().manual_seed(width)
    x, y = torch.randn(9, width, generator=g), torch.randn(9, width, generator=g).to(torch.bfloat16).float() * 2
    wb, wn = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    c = lambda t, d=torch.float32: t.to("cuda:0", d)
    tol = 1e-6 if dtype == torch.float32 else 4e-3
    xd, yd, wbd, wnd = x.double(), y.double(), wb.double(), wn.double()
    out, cat = torch.empty(9, width, device="cuda:0"), torch.zeros(9, 2 * width, device="cuda:0", dtype=dtype)
    h = K.residual_norm(c(x), c(y, dtype), c(wb), c(wn), 1e-3, dtype, x_out=out, cat=cat)
    want = xd + O.rms_norm(yd, wbd, 1e-3)
    assert float(U.row_errors(out, want).max()) < 1e-6 and float(U.row_errors(h, O.rms_norm(want, wnd, 1e-3)).max()) < tol
    assert float(U.row_errors(cat[:, :width], want).max()) < tol and float(cat[:, width:].abs().max()) == 0
    h = K.residual_norm(c(x[0]), c(y), None, c(wn), 1e-3, dtype, x_out=out, broadcast=True)
    assert float(U.row_errors(out, xd[0] + yd).max()) < 1e-6 and float(U.row_errors(h, O.rms_norm(xd[0] + yd, wnd, 1e-3)).max()) < tol
    rows = torch.tensor([7, 0, 7], dtype=torch.int32, device="cuda:0")
    h = K.residual_norm(c(x), None, None, c(wn), 1e-3, dtype, rows=rows)
    assert float(U.row_errors(h, O.rms_norm(xd[[7, 0, 7]], wnd, 1e-3)).max()) < tol
    table, status = c(y, dtype), torch.zeros(4, dtype=torch.int32, device="cuda:0")
    tok = torch.tensor([3, 8, 0, 11], dtype=torch.int32, device="cuda:0")
    x2, h = K.embed(table, tok, c(wn), 1e-3, cat=cat, cat_both=True, status=status)
    assert float(U.row_errors(x2, yd[[3, 8, 0, 0]]).max()) < 1e-6 and status.tolist() == [0, 0, 1, 0]
    assert torch.equal(cat[:4, :width], table[[3, 8, 0, 0]]) and torch.equal(cat[:4, width:], table[[3, 8, 0, 0]])


# ------------------------------------------------------------------------------------------ whole models
@NAMES
@DTYPES
def test_prompt_decode_and_portions_agree_with_the_oracle(name, dtype):
    m, toks = model(name, dtype), U.tokens_of(U.CONFIGS[name], 150, 1)
    want = U.oracle_logits(name, 0, toks, dtype)
    cache = m.new_cache(2, 150)
    for cuts in ((150,), (70, 1), (2,), (33, 5, 64, 2, 1, 9)):
        cache.acquire("a")
        close(feed(m, cache, "a", toks, cuts), want, dtype)
        cache.release("a")
    m.check_status()


@NAMES
def test_token_by_token_from_the_start(name):
    m, toks = model(name, torch.float32), U.tokens_of(U.CONFIGS[name], 40, 2)
    cache = m.new_cache(1, 64)
    cache.acquire("a")
    close(feed(m, cache, "a", toks, (1,)), U.oracle_logits(name, 0, toks), torch.float32)


@NAMES
@DTYPES
def test_unequal_requests_side_by_side_with_slots_used_again(name, dtype):
    """Five requests over three slots, portions and single tokens mixed in every step; each must read as if alone."""
    m, cfg = model(name, dtype), U.CONFIGS[name]
    toks = {i: U.tokens_of(cfg, n, 20 + i) for i, n in enumerate((61, 7, 90, 2, 35))}
    cache, at, got = m.new_cache(3, 96), {}, {i: [] for i in toks}
    waiting, rnd = list(toks), torch.Generator().manual_seed(9)
    while waiting or at:
        while waiting and cache.free_slots:
            i = waiting.pop(0)
            cache.acquire(i)
            at[i] = 0
        entries = []
        for i in at:
            n = min([1, 1, 2, 13, 40][int(torch.randint(0, 5, (1,), generator=rnd))], len(toks[i]) - at[i])
            entries.append((i, toks[i][at[i]:at[i] + n], range(n)))
        logits = m.run(entries, cache)
        for (i, t, _), part in zip(entries, logits.split([len(t) for _, t, _ in entries])):
            got[i].append(part)
            at[i] += len(t)
            if at[i] == len(toks[i]):
                del at[i]
                cache.release(i)
    close(torch.cat([torch.cat(got[i]) for i in toks]), torch.cat([U.oracle_logits(name, 0, toks[i], dtype) for i in toks]), dtype)


@BOTH
def test_batch_mates_do_not_change_a_sequence(name):
    """The same portion alone and beside others differs by rounding at most (fp32)."""
    m, cfg = model(name, torch.float32), U.CONFIGS[name]
    a, b = U.tokens_of(cfg, 50, 31), U.tokens_of(cfg, 77, 32)
    cache = m.new_cache(2, 100)
    cache.acquire("a")
    alone = m.run([("a", a, range(50))], cache)
    cache.release("a")
    cache.acquire("b"), cache.acquire("a")
    both = m.run([("b", b, range(77)), ("a", a, range(50))], cache)[77:]
    assert float(U.row_errors(both, alone).max()) < 2e-5


@BOTH
def test_long_decoding(name):
    m, cfg = model(name, torch.float32), U.CONFIGS[name]
    toks = U.tokens_of(cfg, 420, 41)
    cache = m.new_cache(2, 420)
    cache.acquire("other"), cache.acquire("a")
    got = feed(m, cache, "a", toks, (9, 1))
    close(got, U.oracle_logits(name, 0, toks), torch.float32)


@pytest.mark.parametrize("name", ["wide", "par-wide", "par-mixed"])
def test_graphed_decode_matches_plain_steps(name):
    from msa_b200.hybrid import GraphedDecode
    m, cfg = model(name, torch.bfloat16), U.CONFIGS[name]
    prompts = [U.tokens_of(cfg, n, 50 + n) for n in (5, 130, 64)]
    runs = []
    for graphed in (False, True):
        cache = m.new_cache(3, 200)
        g = GraphedDecode(m, cache, 4) if graphed else None          # one row to fill up
        for i in range(3):
            cache.acquire(i)
        tok = m.run([(i, p, [len(p) - 1]) for i, p in enumerate(prompts)], cache).argmax(-1).tolist()
        rows = []
        for _ in range(12):
            if graphed:
                logits = g.run(tok, [cache.length(i) for i in range(3)], [cache.slot(i) for i in range(3)]).clone()
                for i in range(3):
                    cache.advance(i, 1)
            else:
                logits = m.run([(i, [t], [0]) for i, t in enumerate(tok)], cache)
            tok = U.tokens_of(cfg, 3, len(rows))
            rows.append(logits)
        runs.append(torch.cat(rows))
    assert float(U.row_errors(runs[1], runs[0]).max()) < 1e-2


# ------------------------------------------------------------------------------------------ generation
def oracle_greedy(name, prompt, n):
    toks, cfg = list(prompt), U.CONFIGS[name]
    w = U.make_weights(cfg, 0)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@NAMES
def test_scheduler_generates_what_the_oracle_would(name):
    from msa_b200.scheduler import Scheduler, SequenceRequest
    m, cfg = model(name, torch.float32), U.CONFIGS[name]
    s = Scheduler(m, max_batch=6, max_len=80, portion=11, step_tokens=16)
    reqs = [SequenceRequest(U.tokens_of(cfg, n, 60 + n), 7) for n in (23, 1, 40, 9, 2, 17, 30, 5, 11)]
    for r in reqs:
        s.submit(r)
    s.run()
    assert s.cache.free_slots == 6 and s._graphs          # decode-only steps came from graphs
    for r in reqs:
        assert r.output == oracle_greedy(name, r.tokens, 7)


@BOTH
def test_forward_takes_left_padded_batches(name):
    """The interleave loop's call: padded rows, masked steps, states advanced for unmasked tokens only."""
    m, cfg = model(name, torch.float32), U.CONFIGS[name]
    a, b = U.tokens_of(cfg, 9, 71), U.tokens_of(cfg, 5, 72)
    cache = m.new_cache(2, 32)
    ids = torch.tensor([a[:8], [0] * 4 + b[:4]])
    mask = torch.tensor([[1] * 8, [0] * 4 + [1] * 4])
    first = m(input_ids=ids, attention_mask=mask, past_key_values=cache).logits
    assert first.shape == (2, 1, cfg["vocab"])
    second = m(input_ids=torch.tensor([[a[8]], [0]]), attention_mask=torch.tensor([[1], [0]]), past_key_values=cache).logits
    third = m(input_ids=torch.tensor([[0], [b[4]]]), attention_mask=torch.tensor([[0], [1]]), past_key_values=cache).logits
    wa, wb = U.oracle_logits(name, 0, a), U.oracle_logits(name, 0, b)
    for got, want in ((first[0, 0], wa[7]), (first[1, 0], wb[3]), (second[0, 0], wa[8]), (third[1, 0], wb[4])):
        assert float(U.row_errors(got[None], want[None])) < 2e-4
    assert float(second[1].abs().max()) == 0 and cache.length(0) == 9 and cache.length(1) == 5


@BOTH
@pytest.mark.timeout(300)
def test_engine_and_command_line_generate(name, tmp_path, capfd):
    from msa_b200.__main__ import main
    from msa_b200.engine import GenerateConfig, MSAEngine
    from msa_b200.memory import ModelConfig
    cfg = U.CONFIGS[name]
    U.save(cfg, U.make_weights(cfg, 0), str(tmp_path))
    prompts = [U.tokens_of(cfg, n, 80 + n) for n in (12, 3, 30)]
    want = [" ".join(map(str, oracle_greedy(name, p, 5))) for p in prompts]
    gen = GenerateConfig(devices=[0], max_generate_tokens=5, max_context=64, state_slots=2)
    with MSAEngine(gen, ModelConfig(model_path=str(tmp_path), dtype="float32")) as e:
        texts, _, tag = e.generate([prompts[0], " ".join(map(str, prompts[1])), prompts[2]], userdata="t")
        assert texts == want and tag == "t"
        with pytest.raises(RuntimeError, match="vocabulary"):
            e.generate([[cfg["vocab"]]])
        assert e.generate([prompts[2]])[0] == want[2:]
    assert main(["generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, prompts[0])), "--max-new-tokens", "5",
                 "--max-context", "64", "--dtype", "float32"]) == 0
    assert want[0] in capfd.readouterr().out


def test_sampled_generation_is_reproducible():
    from msa_b200.scheduler import Scheduler, SequenceRequest
    m, cfg = model("odd", torch.float32), U.CONFIGS["odd"]
    outs = []
    for _ in range(2):
        s = Scheduler(m, max_batch=3, max_len=64)
        reqs = [SequenceRequest(U.tokens_of(cfg, 6, 90), 10, temperature=1.0, top_p=0.95, seed=k) for k in (1, 2, 1)]
        for r in reqs:
            s.submit(r)
        s.run()
        outs.append([r.output for r in reqs])
    assert outs[0] == outs[1] and outs[0][0] == outs[0][2] and outs[0][0] != outs[0][1]
