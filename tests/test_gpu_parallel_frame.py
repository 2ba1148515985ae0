"""The mechanisms of the parallel frame (Nazerax) where random weights would hide a fault: window edges, the sink, decays
from very slow to very steep, far memories, the hashed bigram rows, and the small kernels between the products."""
import pytest
import torch

from oracle import hybrid_oracle as O
from tests import hybrid_util as U
from tests.test_gpu_hybrid import DTYPES, EPS, OneMixer, bf16_rows, exact_products, mixer_case, mixer_close  # noqa: F401

pytestmark = pytest.mark.gpu


def gap(x, want, i):
    return float((x[i] - want[i]).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())


def loud_key(w, spec, width, seed, n, loud):
    """Rows whose token ``loud`` has a key that every query asks for: column 0 of the rows drives the last dimension of the
    keys, column 1 that of the queries, both past their convolutions unchanged."""
    h = bf16_rows(n, width, seed)
    h[:, 0], h[:, 1] = 0.0, 1.0
    h[loud, 0] = 60.0
    for name, heads, col, gain in (("q", spec["heads"], 1, 5.0), ("k", spec["kv_heads"], 0, 4.0)):
        w[name][:, :2] = 0
        for hd in range(heads):
            r = hd * spec["dim"] + spec["dim"] - 1
            w[name][r, :] = 0
            w[name][r, col] = gain
            w[name + ".conv"][r, :] = 0
            w[name + ".conv"][r, -1] = 1.0
    w["v"][:, :2] = 0
    return h


@DTYPES
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("sizes", [(4, 2, 18, 10), (8, 2, 64, 64), (20, 2, 128, 64)], ids=["any", "64", "128"])
@pytest.mark.parametrize("window", [5, 64, 130])
def test_window_edge_is_exact(window, sizes, decode, dtype):
    heads, kv, dim, vdim = sizes
    spec, width = U.attention(heads, kv, dim, vdim, window, 8, 3, scale=0.1), 64
    w, oracle = mixer_case("attention", spec, width, 3, sharp=0.3)
    n, loud = 2 * window + 90, window // 2 + 1
    h = loud_key(w, spec, width, 8, n, loud)
    want = oracle(h)
    last_seen, first_gone = loud + window - 1, loud + window
    assert gap(oracle(h, {**spec, "mask": {"size": window - 1}}), want, last_seen) > 0.3          # one off would show
    assert gap(oracle(h, {**spec, "mask": {"size": window + 1}}), want, first_gone) > 0.3
    m = OneMixer("attention", spec, w, width, dtype)
    cache = m.cache(1, n)
    cache.acquire(0)
    if decode:
        got = torch.cat([m.run(cache, [(0, h[:loud + 1])])[0]] + [m.run(cache, [(0, h[i:i + 1])])[0] for i in range(loud + 1, n)])
    else:
        got = m.run(cache, [(0, h)])[0]
    e = U.row_errors(got, want)
    tol = 1e-4 if dtype == torch.float32 else 0.05
    assert float(e[last_seen]) < tol and float(e[first_gone]) < tol and float(e.max()) < tol


@DTYPES
@pytest.mark.parametrize("sizes", [(4, 2, 18, 10), (8, 2, 64, 64)], ids=["any", "64"])
@pytest.mark.parametrize("level", [-1.0, 0.0, 1.0], ids=["quiet", "even", "loud"])
def test_sink_takes_its_share(level, sizes, dtype):
    """All scores far below, around and far above the sink's: its share goes from everything to nothing."""
    heads, kv, dim, vdim = sizes
    spec, width, n = U.attention(heads, kv, dim, vdim, 40, 4, 2, scale=0.25), 64, 170
    w, oracle = mixer_case("attention", spec, width, 9, sharp=0.2)
    h = bf16_rows(n, width, 4)
    h[:, 0] = 1.0
    for name, hs, v in (("q", heads, 5.0), ("k", kv, 5.0 * level)):
        for hd in range(hs):
            r = hd * dim + dim - 1
            w[name][r, :] = 0
            w[name][r, 0] = v
            w[name + ".conv"][r, :] = 0
            w[name + ".conv"][r, -1] = 1.0
    want = oracle(h)
    plain = O.softmax_plus_one
    try:
        O.softmax_plus_one = lambda s: torch.softmax(s, dim=-1)
        without = oracle(h)
    finally:
        O.softmax_plus_one = plain
    share = float((without - want).pow(2).mean().sqrt() / without.pow(2).mean().sqrt())
    assert share > 0.9 if level < 0 else (share > 0.02 if level == 0 else share < 0.01)
    m = OneMixer("attention", spec, w, width, dtype)
    cache = m.cache(1, n)
    cache.acquire(0)
    got = torch.cat([m.run(cache, [(0, x)])[0] for x in (h[:130], *h[130:].split(1))])
    e = U.row_errors(got, want)
    assert float(e.max()) < (1e-4 if dtype == torch.float32 else 0.05)


def run_cuts(m, h, cuts, n_slots=1):
    cache = m.cache(n_slots, h.shape[0])
    cache.acquire("s")
    out, at, k = [], 0, 0
    while at < h.shape[0]:
        n = min(cuts[k % len(cuts)], h.shape[0] - at)
        out.append(m.run(cache, [("s", h[at:at + n])])[0])
        at, k = at + n, k + 1
    return torch.cat(out)


@DTYPES
@pytest.mark.parametrize("dim", [12, 64])
@pytest.mark.parametrize("kind", ["slow", "steep", "all"])
def test_wkv_decays_of_every_size(kind, dim, dtype):
    """log decays per token from -1e-4 to -3000 (the running sums of a chunk then leave the range of 32-bit exponentials)."""
    spec, width = U.wkv(3, dim), 48
    w, oracle = mixer_case("wkv", spec, width, 6)
    inner = 3 * dim
    lo, hi = {"slow": (-9.0, -7.0), "steep": (2.5, 8.0), "all": (-9.0, 8.0)}[kind]
    w["w0"] = (lo + (hi - lo) * torch.rand(inner, generator=torch.Generator().manual_seed(2))).to(torch.bfloat16)
    h = bf16_rows(330, width, 3)
    want = oracle(h)
    m = OneMixer("wkv", spec, w, width, dtype)
    for cuts in ((330,), (100, 1, 2, 65)):
        got = run_cuts(m, h, cuts)
        assert torch.isfinite(got).all()
        mixer_close(got, want, dtype)


@DTYPES
@pytest.mark.parametrize("sizes", [(12, 20), (64, 128)])
@pytest.mark.parametrize("kind", ["slow", "steep", "all"])
def test_ssd_decays_of_every_size(kind, sizes, dtype):
    spec, width = U.mamba2(4, sizes[0], sizes[1], 2, 2, 3), 48
    w, oracle = mixer_case("mamba2", spec, width, 6)
    lo, hi = {"slow": (-9.0, -7.0), "steep": (3.0, 8.0), "all": (-9.0, 8.0)}[kind]
    w["A_log"] = torch.linspace(lo, hi, 4).to(torch.bfloat16)
    w["in"][-4:] *= 4                                                 # steps from next to nothing to large
    h = bf16_rows(330, width, 3)
    want = oracle(h)
    m = OneMixer("mamba2", spec, w, width, dtype)
    for cuts in ((330,), (100, 1, 2, 65)):
        got = run_cuts(m, h, cuts)
        assert torch.isfinite(got).all()
        mixer_close(got, want, dtype)


@pytest.mark.parametrize("dim", [8, 40, 64, 96, 128])
def test_wkv_chunks_match_the_recurrence(dim):
    """The chunked kernels on given operands: what is left is the rounding of the output."""
    from types import SimpleNamespace
    from msa_b200 import lm_ops as K
    from msa_b200.cache import PackedStep, RecurrentSpec, SequenceStateCache
    heads, g = 3, torch.Generator().manual_seed(dim)
    r = lambda *s: torch.randn(*s, generator=g)
    lens = (1, 2, 64, 65, 200)
    cache = SequenceStateCache([RecurrentSpec(heads, dim, dim)], 5, 256, "cuda:0", torch.bfloat16)
    for i in range(5):
        cache.acquire(i)
    cache.advance(4, 30)                                             # one sequence continues from a state
    first = r(heads, dim, dim)
    cache.state[0][cache.slot(4)] = first.cuda()
    step = PackedStep([(i, [0] * n, range(n)) for i, n in enumerate(lens)], cache, ())
    n, inner = step.n_tok, heads * dim
    rkvg = r(4, n, inner).to(torch.bfloat16)
    raw = 3.0 * r(n, inner) - 1.0
    w0, u, norm = r(inner), r(heads, dim), 1 + 0.2 * r(inner)
    dev = lambda t: t.cuda()
    out = torch.empty(n, inner, dtype=torch.bfloat16, device="cuda:0")
    weights = SimpleNamespace(w0=dev(w0), u=dev(u), norm=dev(norm))
    K.wkv_mix(dev(rkvg), dev(raw.clone()), SimpleNamespace(heads=heads, dim=dim), weights, cache.state[0], EPS, step, out)
    order = step.want_rows.cpu().long().split([x for x in lens])
    for i, rows in enumerate(order):
        q, k, v, gate = (rkvg[j][rows].double().view(-1, heads, dim) for j in range(4))
        decay = torch.exp(-torch.exp(raw[rows].double() + w0.double())).view(-1, heads, dim)
        o, end = O.wkv_recurrence(q, k, v, decay, u.double(), first.double() if i == 4 else None)
        want = O.rms_norm(o, None, EPS).reshape(-1, inner) * norm.double() * O.silu(gate.reshape(-1, inner))
        assert float((out[rows.cuda()].double().cpu() - want).abs().max()) < 2e-2 * float(want.abs().max())
        assert float(U.row_errors(out[rows.cuda()], want).max()) < 6e-3
        got = cache.state[0][cache.slot(i)].double().cpu()
        assert float((got - end).abs().max()) < 3e-4 * float(end.abs().max())


@DTYPES
@pytest.mark.parametrize("kind", ["wkv", "mamba2"])
def test_state_remembers_a_far_write(kind, dtype):
    """One token writes a large value and decays hardly at all; hundreds of tokens later it is what the read-out shows."""
    width, n = 48, 420
    spec = U.wkv(2, 24) if kind == "wkv" else U.mamba2(2, 24, 16, 1, 2, 2)
    w, oracle = mixer_case(kind, spec, width, 4)
    if kind == "wkv":
        w["w0"][:], w["w2"][:] = -12.0, 0.0
    else:
        w["A_log"][:], w["conv.b"][:], w["D"][:] = -9.0, 0.0, 0.0
    h = bf16_rows(n, width, 2) * 0.05
    h[3] = 30.0 * h[3]
    want = oracle(h)
    erased = h.clone()
    erased[3] = h[4]
    assert float(U.row_errors(oracle(erased)[-1:], want[-1:])) > 0.3                 # a lost state would show
    m = OneMixer(kind, spec, w, width, dtype)
    mixer_close(run_cuts(m, h, (200, 2, 1, 216, 1)), want, dtype)
    mixer_close(run_cuts(m, h, (2, 64, 1)), want, dtype)


@pytest.mark.parametrize("dtype", [torch.bfloat16], ids=["bf16"])
@pytest.mark.parametrize("width", [64, 51])
def test_embedding_with_bigrams_over_steps(width, dtype):
    """Rows of a step, the first token of a sequence, and the previous token across steps and slots used again."""
    from msa_b200 import lm_ops as K
    from msa_b200.cache import PackedStep, RingSpec, SequenceStateCache
    g = torch.Generator().manual_seed(width)
    buckets, a, b = 37, 13, 1009
    table, pairs = torch.randn(50, width, generator=g).to(dtype), torch.randn(buckets + 1, width, generator=g).to(dtype)
    w1, w2 = (1 + 0.2 * torch.randn(width, generator=g) for _ in range(2))
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": a, "mul_cur": b}}}
    toks = {i: torch.randint(0, 50, (n,), generator=g).tolist() for i, n in enumerate((9, 6, 7))}
    want = {i: O.embedding(cfg, {"embed": table, "bigram": pairs}, t, torch.float64) for i, t in toks.items()}
    cache, status = SequenceStateCache([RingSpec(4, 4)], 2, 32, "cuda:0", dtype), torch.zeros(4, dtype=torch.int32, device="cuda:0")
    at = {0: 0, 1: 0, 2: 0}
    for plan in (((0, 4), (1, 1)), ((0, 1), (1, 3)), ((0, 2), (1, 2)), ((0, 2), (2, 1)), ((2, 1),), ((2, 5),)):
        for i, _ in plan:
            if i not in cache:
                cache.acquire(i)
        step = PackedStep([(i, toks[i][at[i]:at[i] + n], range(n)) for i, n in plan], cache, ())
        copy = torch.empty(step.n_tok, width, device="cuda:0")
        x, h, h2 = K.embed(table.cuda(), step.token, w1.cuda(), 1e-3, status=status, w_next2=w2.cuda(), x_copy=copy,
                           pair=(pairs.cuda(), buckets, a, b), step=step, last_token=cache.last_token)
        rows = step.want_rows.long()
        exp = torch.cat([want[i][at[i]:at[i] + n] for i, n in plan])
        assert float((x[rows].double().cpu() - exp).abs().max()) < 1e-6 and torch.equal(x, copy)
        assert float(U.row_errors(h[rows], O.rms_norm(exp, w1.double(), 1e-3)).max()) < 4e-3
        assert float(U.row_errors(h2[rows], O.rms_norm(exp, w2.double(), 1e-3)).max()) < 4e-3
        step.commit(cache)
        for i, n in plan:
            at[i] += n
            if at[i] == len(toks[i]):
                cache.release(i)
    assert status.tolist() == [0, 0, 0, 0]


@DTYPES
@pytest.mark.parametrize("width", [64, 51, 6000])
def test_residual_step_with_a_second_norm_and_further_rows(width, dtype):
    from msa_b200 import lm_ops as K
    g = torch.Generator().manual_seed(width)
    for n in (5, 600):
        x, y, more = (torch.randn(n, width, generator=g) for _ in range(3))
        w1, w2 = (1 + 0.3 * torch.randn(width, generator=g) for _ in range(2))
        c = lambda t, d=torch.float32: t.to("cuda:0", d)
        yr = y.to(dtype).double()
        xd = c(x)
        h, h2 = K.residual_norm(xd, c(y, dtype), None, c(w1), 1e-3, dtype, x_out=xd, add=c(more), w_next2=c(w2))
        want = x.double() + yr + more.double()
        tol = 1e-6 if dtype == torch.float32 else 4e-3
        assert float(U.row_errors(xd, want).max()) < 1e-6
        assert float(U.row_errors(h, O.rms_norm(want, w1.double(), 1e-3)).max()) < tol
        assert float(U.row_errors(h2, O.rms_norm(want, w2.double(), 1e-3)).max()) < tol


@DTYPES
def test_small_kernels(dtype):
    from msa_b200 import lm_ops as K
    g = torch.Generator().manual_seed(5)
    tol = 1e-6 if dtype == torch.float32 else 4e-3
    z = 40 * torch.randn(7, 33, generator=g)
    assert float((K.softcap(z.cuda(), 12.0).double().cpu() - O.softcap(z.double(), 12.0)).abs().max()) < 1e-5
    t = torch.randn(9, 24, generator=g)
    parts = 2 if dtype == torch.bfloat16 else 1
    got = K.tanh_split(t.cuda(), dtype, parts).view(9, parts, 24).double().sum(1).cpu()
    assert float((got - torch.tanh(t.double())).abs().max()) < 1e-5
    for width, groups in ((96, 4), (35, 5), (40, 1), (12, 12)):
        x, w = torch.randn(6, width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
        out = K.part_norm(x.cuda(), w.cuda(), groups, 1e-3, torch.empty(6, width, dtype=dtype, device="cuda:0"))
        assert float(U.row_errors(out, O.group_norm(x.double(), groups, 1e-3) * w.double()).max()) < tol


@DTYPES
@pytest.mark.parametrize("name", ["par-mixed", "par-wide"])
def test_stream_after_every_layer(name, dtype):
    """The residual stream after every layer run, loop passes included."""
    from msa_b200.hybrid import HybridForCausalLM
    from msa_b200.hybrid_config import HybridConfig
    cfg, w = U.CONFIGS[name], U.make_weights(U.CONFIGS[name], 3)
    m, toks, want, got = HybridForCausalLM(HybridConfig.parse(cfg), w, "cuda:0", dtype), U.tokens_of(cfg, 70, 4), [], []
    O.forward(cfg, w, toks, layers_out=want)
    cache = m.new_cache(1, 70)
    cache.acquire("a")
    m.on_layer = lambda run, x: got.append(x.clone())
    m.run([("a", toks, [])], cache)
    assert len(got) == len(want) == len(m.config.runs())
    for a, b in zip(got, want):
        assert float(U.row_errors(a, b).max()) < (1e-5 if dtype == torch.float32 else 0.05)


def test_checkpoint_must_fit_the_configuration(tmp_path):
    from msa_b200.registry import load_model
    w = U.make_weights(U.PAR_ODD, 0)
    U.save(U.PAR_ODD, {**w, "l0.mix.extra": torch.zeros(2)}, str(tmp_path))
    with pytest.raises(ValueError, match="extra"):
        load_model(str(tmp_path), "cuda:0")
    w.pop("l1.mix.D")
    U.save(U.PAR_ODD, w, str(tmp_path))
    with pytest.raises(KeyError, match="l1.mix.D"):
        load_model(str(tmp_path), "cuda:0")
