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


def shifted(h):
    """Row t of the result is row t-1 of h; zeros in front."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_recurrence(r, k, v, decay, bonus, state=None):
    """r, k, decay ``[tokens, heads, dim]``, v ``[tokens, heads, vdim]``, bonus ``[heads, dim]``: read the state with the
    current token added under the bonus, then decay every key channel by its own factor and add the token."""
    n, heads, dim = r.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(n):
        kv = torch.einsum("hk,hv->hkv", k[t], v[t])
        out[t] = torch.einsum("hkv,hk->hv", s + bonus[:, :, None] * kv, r[t])
        s = decay[t][:, :, None] * s + kv
    return out, s


def wkv_mixer(h, w, spec, eps):
    n, heads, dim = h.shape[0], spec["heads"], spec["dim"]
    back = shifted(h) - h
    mixed = {s: h + back * w["mu." + s] for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[s].T).view(n, heads, dim) for s in "rkv")
    decay = torch.exp(-torch.exp(torch.tanh(mixed["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).view(n, heads, dim)
    o, _ = wkv_recurrence(r, k, v, decay, w["u"])
    o = rms_norm(o, None, eps).reshape(n, heads * dim) * w["norm"]
    return (o * silu(mixed["g"] @ w["g"].T)) @ w["o"].T


def causal_conv(x, taps, bias=None):
    """x ``[tokens, channels]``, taps ``[channels, n]``: every output is the weighted sum of the token's own input and the
    n - 1 before it."""
    n, n_taps = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros(n_taps - 1, x.shape[1]), x])
    out = sum(padded[j:j + n] * taps[:, j] for j in range(n_taps))
    return out if bias is None else out + bias


def rotate_leading(x, positions, base, dims):
    """The first ``dims`` of every head turn, the rest pass."""
    if not dims:
        return x
    return torch.cat([rotate_interleaved(x[..., :dims], positions, base), x[..., dims:]], dim=-1)


def softmax_plus_one(score):
    """Softmax over the last axis with one added to the denominator (a silent entry whose score is 0)."""
    top = torch.clamp(score.max(dim=-1, keepdim=True).values, min=0)
    e = torch.exp(score - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def window_attention(h, w, spec, eps=None):
    """Grouped-query attention over a sliding window behind a short convolution, with a silent sink and one gate per head."""
    n, heads, groups, dim, vdim = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    pos, rot = torch.arange(n), spec.get("rot") or {"base": 1.0, "dims": 0}
    q, k, v = (causal_conv(h @ w[s].T, w[s + ".conv"]) for s in "qkv")
    q = rotate_leading(q.view(n, heads, dim), pos, rot["base"], rot["dims"])
    k = rotate_leading(k.view(n, groups, dim), pos, rot["base"], rot["dims"])
    owner = torch.arange(heads) // (heads // groups)
    k, v = k[:, owner], v.view(n, groups, vdim)[:, owner]
    score = torch.einsum("ihd,jhd->hij", q, k) * spec["scale"]
    mask = window_mask(n, (spec.get("mask") or {}).get("size"))
    o = torch.einsum("hij,jhd->ihd", softmax_plus_one(score.masked_fill(~mask, float("-inf"))), v)
    return (o * sigmoid(h @ w["g"].T)[:, :, None]).reshape(n, heads * vdim) @ w["o"].T


def ssd_recurrence(c, b, x, log_decay, step, state=None):
    """c, b ``[tokens, heads, n]``, x ``[tokens, heads, vdim]``, log_decay and step ``[tokens, heads]``: decay the state by
    one factor per head, add the token scaled by its step, read."""
    s = torch.zeros(c.shape[1], c.shape[2], x.shape[-1], dtype=x.dtype) if state is None else state.clone()
    out = torch.empty_like(x)
    for t in range(x.shape[0]):
        s = torch.exp(log_decay[t])[:, None, None] * s + torch.einsum("hn,hv->hnv", b[t] * step[t][:, None], x[t])
        out[t] = torch.einsum("hnv,hn->hv", s, c[t])
    return out, s


def group_norm(x, parts, eps):
    """Equal contiguous parts of the last axis, each divided by its own root mean square."""
    return rms_norm(x.view(*x.shape[:-1], parts, -1), None, eps).reshape(x.shape)


def mamba2_mixer(h, w, spec, eps):
    n, heads, vdim, ns, groups = h.shape[0], spec["heads"], spec["vdim"], spec["state"], spec["groups"]
    inner = heads * vdim
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * groups * ns, heads], dim=-1)
    x, b, c = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, groups * ns, groups * ns], dim=-1)
    x = x.reshape(n, heads, vdim)
    owner = torch.arange(heads) // (heads // groups)
    b, c = b.reshape(n, groups, ns)[:, owner], c.reshape(n, groups, ns)[:, owner]
    step = softplus(dt + w["dt_bias"])
    y, _ = ssd_recurrence(c, b, x, -torch.exp(w["A_log"]) * step, step)
    y = (y + w["D"][:, None] * x).reshape(n, inner) * silu(z)
    return (group_norm(y, spec["norm_groups"], eps) * w["norm"]) @ w["o"].T


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


def embedding(config, weights, tokens, dtype):
    """Rows of the table, plus, with ``embedding.bigram``, the hashed row of (previous token, token)."""
    x = weights["embed"].to(dtype)[torch.as_tensor(tokens)]
    pair = (config.get("embedding") or {}).get("bigram")
    if pair:
        rows = [pair["buckets"]] + [(a * pair["mul_prev"] + b * pair["mul_cur"]) % pair["buckets"] for a, b in zip(tokens, tokens[1:])]
        x = x + weights["bigram"].to(dtype)[torch.tensor(rows)]
    return x


def softcap(z, cap):
    return z if not cap else cap * torch.tanh(z / cap)


def _feed_forward(h, w, spec):
    return dense_ff(h, w) if spec["kind"] == "dense" else moe_ff(h, w, spec)


MIXERS = {"latent_attention": latent_attention, "delta": delta_mixer, "wkv": wkv_mixer, "attention": window_attention,
          "mamba2": mamba2_mixer}


def forward(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[tokens, vocab]`` of one sequence; ``layers_out`` (a list) collects the stream after every layer run."""
    return {"Mutuvik": forward_sandwich, "Nazerax": forward_parallel}[config["architecture"]](config, weights, tokens, dtype, layers_out)


def forward_parallel(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Mixer and feed-forward read the same stream through a norm each; norm weights are stored around zero; every pass
    of the loop but the first starts by adding the embedding again."""
    eps = config["norm"]["eps"]
    norm = lambda x, name: rms_norm(x, 1 + weights[name].to(dtype), eps)
    x = x0 = embedding(config, weights, tokens, dtype)
    for i, t in layer_runs(config):
        spec, p = config["layers"][i], f"l{i}."
        if t and i == config["loop"]["start"]:
            x = x + x0
        y = MIXERS[spec["type"]](norm(x, p + "norm1"), _sub(weights, p + "mix.", dtype), spec["mixer"], eps)
        if spec.get("mlp"):
            y = y + _feed_forward(norm(x, p + "norm2"), _sub(weights, p + "mlp.", dtype), spec["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return softcap(norm(x, "final.norm") @ weights["head"].to(dtype).T, config.get("logit_softcap"))


def forward_sandwich(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Norms on both sides of every sublayer; a looped pass starts from a product over [stream, embedding]."""
    eps = config["norm"]["eps"]
    table = weights["embed"].to(dtype)
    x = x0 = embedding(config, weights, tokens, dtype)
    for i, t in layer_runs(config):
        spec = config["layers"][i]
        if t is not None and i == config["loop"]["start"]:
            x = torch.cat([x, x0], dim=-1) @ weights["loop.in"].to(dtype).T + weights["loop.step"][t].to(dtype)
        w = _sub(weights, f"l{i}.", dtype)
        y = MIXERS[spec["type"]](rms_norm(x, w["norm1"], eps), _sub(weights, f"l{i}.mix.", dtype), spec["mixer"], eps)
        x = x + rms_norm(y, w["norm1b"], eps)
        if spec.get("mlp"):
            y = _feed_forward(rms_norm(x, w["norm2"], eps), _sub(weights, f"l{i}.mlp.", dtype), spec["mlp"])
            x = x + rms_norm(y, w["norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, weights["final.norm"].to(dtype), eps) @ table.T
