"""Plain, slow restatement of the mechanisms of the layered decoder designs.  TEST INFRASTRUCTURE ONLY.

One function per mechanism, written token by token or as whole-sequence matrix algebra, in the dtype of its inputs
(the tests use float64), on the CPU.  Nothing here is shared with the product path: no cache, no portions, no kernels.
A sequence is a 2-D tensor ``[tokens, width]``; positions are its row numbers.

``forward(config, weights, tokens)`` chains them for one sequence; ``config`` is the parsed config.json dictionary,
``weights`` a dictionary tensor name -> tensor.
"""
from __future__ import annotations

import torch


def rms_norm(x, weight, eps):
    """Root-mean-square norm over the last axis with eps inside the root."""
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_interleaved(x, positions, base):
    """x ``[tokens, ..., dims]``: neighbours (2i, 2i+1) form a plane that turns by position * base^(-2i/dims)."""
    dims = x.shape[-1]
    i = torch.arange(dims // 2, dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None] * base ** (-2.0 * i / dims)
    angle = angle.view([x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2])
    even, odd = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = even * torch.cos(angle) - odd * torch.sin(angle)
    out[..., 1::2] = odd * torch.cos(angle) + even * torch.sin(angle)
    return out


def window_mask(n, size):
    """[n, n] boolean: row i may look at column j."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def latent_attention(h, w, spec, eps):
    """Attention over a shared low-rank latent; keys and values of every head are expanded from it."""
    n = h.shape[0]
    heads, dim, rot, vdim, rank = spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"], spec["kv_rank"]
    pos = torch.arange(n)
    q = (h @ w["q"].T).view(n, heads, dim + rot)
    q_plain, q_rot = q[..., :dim], rotate_interleaved(q[..., dim:], pos, spec["rot"]["base"])
    down = h @ w["dkv"].T
    latent = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    k_rot = rotate_interleaved(down[:, rank:], pos, spec["rot"]["base"])
    k_plain = (latent @ w["uk"].T).view(n, heads, dim)
    v = (latent @ w["uv"].T).view(n, heads, vdim)
    score = torch.einsum("ihd,jhd->hij", q_plain, k_plain) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    score = score * spec["scale"]
    mask = window_mask(n, (spec.get("mask") or {}).get("size"))
    weight = torch.softmax(score.masked_fill(~mask, float("-inf")), dim=-1)
    return torch.einsum("hij,jhd->ihd", weight, v).reshape(n, heads * vdim) @ w["o"].T


def causal_conv_silu(x, taps):
    """x ``[tokens, channels]``, taps ``[channels, n]``; the last tap meets the current token."""
    n_taps = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(n_taps):
        back = n_taps - 1 - t
        out[back:] += x[:x.shape[0] - back] * taps[:, t] if back < x.shape[0] else 0
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """q, k ``[tokens, heads, dim]``, v ``[tokens, heads, vdim]``, g and beta ``[tokens, heads]``: decay the state, write
    the correction of what it would answer to k, read with q."""
    n, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(n):
        s = s * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", s, k[t]))
        s = s + torch.einsum("hk,hv->hkv", k[t], u)
        out[t] = torch.einsum("hkv,hk->hv", s, q[t])
    return out, s


def delta_mixer(h, w, spec, eps):
    n = h.shape[0]
    heads, kv_heads, dim, vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = causal_conv_silu(h @ w["q"].T, w["q.conv"]).view(n, kv_heads, dim)
    k = causal_conv_silu(h @ w["k"].T, w["k.conv"]).view(n, kv_heads, dim)
    v = causal_conv_silu(h @ w["v"].T, w["v.conv"]).view(n, heads, vdim)
    q, k = unit(q) * dim ** -0.5, unit(k)
    owner = torch.arange(heads) // (heads // kv_heads)
    beta = sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o, _ = delta_rule(q[:, owner], k[:, owner], v, g, beta)
    o = rms_norm(o, w["norm"], eps) * silu(h @ w["g"].T).view(n, heads, vdim)
    return o.reshape(n, heads * vdim) @ w["o"].T


def dense_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router, bias, top):
    """Chosen experts ``[tokens, top]`` and the softmax over their logits alone."""
    z, idx = torch.topk(h @ router.T + bias, top, dim=-1)
    return idx, torch.softmax(z, dim=-1)


def moe_ff(h, w, spec):
    idx, weight = route(h, w["router"], w["router.b"], spec["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(idx[t].tolist(), weight[t]):
            out[t] += p * clamped_expert(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], spec["expert"]["limit"])[0]
    return out


def _sub(weights, prefix, dtype):
    return {k[len(prefix):]: v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


def layer_runs(config):
    """[(layer index, pass or None)] in order of execution."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[tokens, vocab]`` of one sequence; ``layers_out`` (a list) collects the stream after every layer run."""
    eps = config["norm"]["eps"]
    table = weights["embed"].to(dtype)
    x = table[torch.as_tensor(tokens)]
    x0 = x
    for i, t in layer_runs(config):
        spec = config["layers"][i]
        if t is not None and i == config["loop"]["start"]:
            x = torch.cat([x, x0], dim=-1) @ weights["loop.in"].to(dtype).T + weights["loop.step"][t].to(dtype)
        w = _sub(weights, f"l{i}.", dtype)
        mixer = {"latent_attention": latent_attention, "delta": delta_mixer}[spec["type"]]
        y = mixer(rms_norm(x, w["norm1"], eps), _sub(weights, f"l{i}.mix.", dtype), spec["mixer"], eps)
        x = x + rms_norm(y, w["norm1b"], eps)
        if spec.get("mlp"):
            h, m = rms_norm(x, w["norm2"], eps), _sub(weights, f"l{i}.mlp.", dtype)
            y = dense_ff(h, m) if spec["mlp"]["kind"] == "dense" else moe_ff(h, m, spec["mlp"])
            x = x + rms_norm(y, w["norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, weights["final.norm"].to(dtype), eps) @ table.T
