"""Small random models of the layered decoder designs, and the comparisons the tests share."""
import json
import os

import torch

from oracle import hybrid_oracle as O


def latent(heads, dim, rot, vdim, rank, window, base=500.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot) ** -0.5,
            "rot": {"base": base, "dims": rot}, "mask": {"size": window}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attention(heads, kv_heads, dim, vdim, window, rot, conv, base=500.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or dim ** -0.5,
            "rot": {"base": base, "dims": rot}, "mask": {"size": window}}


def wkv(heads, dim):
    return {"heads": heads, "dim": dim}


def mamba2(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, loop=None, eps=1e-5):
    return {"architecture": "Mutuvik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": loop}


def parallel(width, vocab, layers, loop=None, eps=1e-5, bigram=None, cap=None):
    pair = None if bigram is None else {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    return {"architecture": "Nazerax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": loop,
            "embedding": {"bigram": pair}, "logit_softcap": cap}


# uneven sizes everywhere, two windows, a layer without a feed-forward, a loop in the middle with a tail behind it
MIXED = config(88, 211, [
    layer("delta", delta(4, 2, 24, 20, 4), dense(112)),
    layer("latent_attention", latent(3, 20, 12, 28, 44, 17), moe(7, 2, 36, 1.5)),
    layer("latent_attention", latent(5, 8, 6, 12, 20, 33, base=77.0), None),
    layer("delta", delta(6, 3, 16, 36, 2), moe(4, 3, 20, 0.7)),
    layer("latent_attention", latent(2, 16, 8, 16, 24, 9), dense(52)),
], loop={"start": 1, "stop": 4, "times": 3}, eps=3e-4)

# odd sizes: nothing is a multiple of 4; the loop starts with the first layer and runs once; window 1 and a wide one
ODD = config(51, 97, [
    layer("latent_attention", latent(3, 5, 2, 7, 13, 1), moe(3, 1, 11, 3.0)),
    layer("delta", delta(3, 1, 9, 7, 3), dense(33)),
    layer("latent_attention", latent(1, 3, 4, 5, 9, 400), moe(5, 5, 9, 1.0)),
], loop={"start": 0, "stop": 2, "times": 1})

# no loop; sizes that the tensor-core kernels take
WIDE = config(256, 320, [
    layer("delta", delta(4, 2, 128, 128, 4), moe(8, 2, 128, 2.5)),
    layer("latent_attention", latent(4, 128, 64, 128, 256, 96, base=10000.0), moe(6, 3, 64, 1.0)),
    layer("delta", delta(2, 2, 64, 64, 4), dense(256)),
    layer("latent_attention", latent(8, 64, 32, 64, 128, 160, base=10000.0), dense(128)),
])

# the parallel frame: uneven sizes, two windows, a convolution of one tap, a layer without a feed-forward, a loop with a tail
PAR_MIXED = parallel(72, 203, [
    layer("wkv", wkv(3, 24), dense(112)),
    layer("attention", attention(6, 2, 20, 28, 17, 12, 3), dense(60)),
    layer("mamba2", mamba2(6, 12, 20, 3, 2, 4), None),
    layer("attention", attention(4, 4, 16, 8, 33, 16, 1, base=77.0), dense(88)),
    layer("wkv", wkv(2, 40), dense(52)),
], loop={"start": 1, "stop": 4, "times": 3}, eps=3e-4, bigram=(61, 31, 5), cap=9.0)

# nothing is a multiple of 4; the loop starts with the first layer; no bigram, no cap; window 1 and a wide one, no rotation
PAR_ODD = parallel(51, 97, [
    layer("wkv", wkv(3, 7), dense(33)),
    layer("mamba2", mamba2(3, 5, 7, 1, 5, 3), dense(9)),
    layer("attention", attention(3, 1, 9, 5, 1, 4, 2), dense(21)),
    layer("attention", attention(3, 3, 5, 7, 400, 0, 6), None),
], loop={"start": 0, "stop": 2, "times": 2})

# sizes that the tensor-core kernels take; a single pass of the loop
PAR_WIDE = parallel(256, 320, [
    layer("wkv", wkv(4, 64), dense(320)),
    layer("attention", attention(8, 2, 64, 128, 100, 32, 4, base=10000.0), dense(256)),
    layer("mamba2", mamba2(6, 64, 128, 2, 3, 4), dense(192)),
    layer("wkv", wkv(2, 128), dense(128)),
    layer("attention", attention(20, 2, 128, 64, 160, 64, 4, base=10000.0), dense(256)),
    layer("mamba2", mamba2(4, 32, 40, 1, 4, 2), dense(64)),
], loop={"start": 2, "stop": 4, "times": 1}, bigram=(127, 11, 3), cap=20.0)

CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE, "par-mixed": PAR_MIXED, "par-odd": PAR_ODD, "par-wide": PAR_WIDE}


def make_weights(cfg, seed=0, sharp=2.0):
    """bf16 tensors by name.  ``sharp`` scales the attention queries: peaked weights let a single wrong key show."""
    g = torch.Generator().manual_seed(seed)
    w, width = {}, cfg["width"]
    mat = lambda n, r, c, s=1.0: w.__setitem__(n, torch.randn(r, c, generator=g) * (s / c ** 0.5))
    vec = lambda n, k, mean, std: w.__setitem__(n, mean + std * torch.randn(k, generator=g))
    w["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    par = cfg["architecture"] == "Nazerax"
    mid = 0.0 if par else 1.0                      # what the frame's norm weights are stored around
    if par:
        mat("head", cfg["vocab"], width, 3.0)
        if cfg["embedding"]["bigram"]:
            w["bigram"] = torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, width, generator=g)
    elif cfg["loop"]:
        mat("loop.in", width, 2 * width)
        w["loop.step"] = 0.5 * torch.randn(cfg["loop"]["times"], width, generator=g)
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        for n in ("norm1", "norm2") if par else ("norm1", "norm1b") + (("norm2", "norm2b") if entry["mlp"] else ()):
            vec(p + n, width, mid, 0.2)
        x = p + "mix."
        if entry["type"] == "delta":
            qk, v = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, r in (("q", qk), ("k", qk), ("v", v)):
                mat(x + n, r, width)
                w[x + n + ".conv"] = torch.randn(r, m["conv"], generator=g) * 0.6
            mat(x + "g", v, width)
            mat(x + "b", m["heads"], width)
            mat(x + "a", m["heads"], width)
            w[x + "A_log"] = torch.rand(m["heads"], generator=g) * 3 - 3.5
            vec(x + "dt_bias", m["heads"], 0.0, 1.0)
            vec(x + "norm", m["vdim"], 1.0, 0.2)
            mat(x + "o", width, v)
        elif entry["type"] == "wkv":
            inner, rank = m["heads"] * m["dim"], 4 + m["dim"] // 8
            for n in "rkvgw":
                w[x + "mu." + n] = torch.rand(width, generator=g)
            for n in "rkvg":
                mat(x + n, inner, width)
            mat(x + "w1", rank, width, 2.0)
            mat(x + "w2", inner, rank, 1.5)
            w[x + "w0"] = torch.rand(inner, generator=g) * 6 - 5
            w[x + "u"] = 0.5 * torch.randn(m["heads"], m["dim"], generator=g)
            vec(x + "norm", inner, 1.0, 0.2)
            mat(x + "o", width, inner)
        elif entry["type"] == "mamba2":
            inner, chan = m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            mat(x + "in", inner + chan + m["heads"], width)
            w[x + "conv"] = torch.randn(chan, m["conv"], generator=g) * 0.6
            vec(x + "conv.b", chan, 0.0, 0.3)
            vec(x + "dt_bias", m["heads"], -1.0, 1.0)
            w[x + "A_log"] = torch.rand(m["heads"], generator=g) * 3 - 2.5
            vec(x + "D", m["heads"], 1.0, 0.5)
            vec(x + "norm", inner, 1.0, 0.2)
            mat(x + "o", width, inner)
        elif entry["type"] == "attention":
            for n, r in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                mat(x + n, r, width, sharp if n == "q" else 1.0)
                w[x + n + ".conv"] = torch.randn(r, m["conv"], generator=g) * 0.6
            mat(x + "g", m["heads"], width)
            mat(x + "o", width, m["heads"] * m["vdim"])
        else:
            mat(x + "q", m["heads"] * (m["dim"] + m["rot_dim"]), width, sharp)
            mat(x + "dkv", m["kv_rank"] + m["rot_dim"], width)
            vec(x + "dkv.norm", m["kv_rank"], 1.0, 0.2)
            mat(x + "uk", m["heads"] * m["dim"], m["kv_rank"])
            mat(x + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(x + "o", width, m["heads"] * m["vdim"])
        f = entry["mlp"]
        if f and f["kind"] == "dense":
            for n, r, c in (("gate", f["ff"], width), ("up", f["ff"], width), ("down", width, f["ff"])):
                mat(p + "mlp." + n, r, c)
        elif f:
            e_ff = f["expert"]["ff"]
            mat(p + "mlp.router", f["router"]["experts"], width)
            vec(p + "mlp.router.b", f["router"]["experts"], 0.0, 0.7)
            for e in range(f["router"]["experts"]):
                for n, r, c in (("gate", e_ff, width), ("up", e_ff, width), ("down", width, e_ff)):
                    mat(f"{p}mlp.e{e}.{n}", r, c, 1.5)
    vec("final.norm", width, mid, 0.2)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def save(cfg, weights, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got, want):
    """Per row: rms of the difference over the rms of the wanted rows."""
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def model_weights(name, seed, dtype):
    """Whole-model comparisons in bf16 cannot rest on close calls of a router: there the biases decide most choices."""
    w = make_weights(CONFIGS[name], seed)
    if dtype == torch.bfloat16:
        for k in w:
            if k.endswith("router.b"):
                w[k] = w[k] * 6
            elif k.endswith("mlp.router"):
                w[k] = w[k] * 0.25
    return w


_ORACLE = {}


def oracle_logits(name, seed, toks, dtype=torch.float32):
    key = (name, seed, tuple(toks), dtype)
    if key not in _ORACLE:
        _ORACLE[key] = O.forward(CONFIGS[name], model_weights(name, seed, dtype), toks)
    return _ORACLE[key]
