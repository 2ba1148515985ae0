"""Functional wrappers of the layered-decoder kernels: torch tensors in, one C-ABI call each."""
from __future__ import annotations

import ctypes as C
from typing import Optional

import torch

from . import _cabi_lm as A


def _rows(t: torch.Tensor) -> int:
    """Row stride of a 2-D tensor with a contiguous last axis."""
    if t.stride(-1) != 1:
        raise A.MsaError("rows with a contiguous last axis expected")
    return t.stride(0)


def matmul(x: torch.Tensor, w: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``x @ w.T`` with 32-bit accumulation; ``out_dtype`` float32 keeps the accumulator's precision."""
    if out_dtype is None or out_dtype == x.dtype:
        return torch.mm(x, w.t())
    return torch.mm(x, w.t(), out_dtype=out_dtype)


def embed(table, token, w_next, eps, cat: Optional[torch.Tensor] = None, cat_both: bool = False, status=None, *, w_next2=None,
          x_copy: Optional[torch.Tensor] = None, pair=None, step=None, last_token=None):
    """``(x fp32, h)``: the embedding rows and, with ``w_next``, their norm (``w_next2``: a second one, ``(x, h, h2)``).
    ``cat`` [n, 2*width]: its right half (with ``cat_both`` its left half too) receives the rows; ``x_copy`` fp32 too.
    ``pair`` = (table, buckets, mul_prev, mul_cur): hashed rows of (previous token, token) join, from the tables of ``step``
    and ``last_token`` [slots]."""
    A.need_cuda(table, token)
    n, width = token.shape[0], table.shape[1]
    x = torch.empty((n, width), dtype=torch.float32, device=table.device)
    h = torch.empty((n, width), dtype=table.dtype, device=table.device) if w_next is not None else None
    h2 = torch.empty_like(h) if w_next2 is not None else None
    args = A.EmbedArgs(table=A.ptr(table), token=A.ptr(token), w_next=A.ptr(w_next), w_next2=A.ptr(w_next2), x_out=A.ptr(x), x_copy=A.ptr(x_copy),
                       h_out=A.ptr(h), h_out2=A.ptr(h2), cat0=A.ptr(cat) if cat is not None and cat_both else 0,
                       cat1=A.ptr(cat) + width * cat.element_size() if cat is not None else 0,
                       cat_stride=_rows(cat) if cat is not None else 0, status=A.ptr(status), n_rows=n, width=width, vocab=table.shape[0],
                       eps=float(eps), dtype=A.dtype_code(table.dtype))
    if pair is not None:
        args.pair_table, args.buckets, args.mul_prev, args.mul_cur = A.ptr(pair[0]), pair[1], pair[2], pair[3]
        args.last_token, args.tok_seq, args.slot = A.ptr(last_token), A.ptr(step.tok_seq), A.ptr(step.slot)
        args.start, args.cu = A.ptr(step.start), A.ptr(step.cu)
    A.call("msa_lm_embed", C.byref(args), A.stream_ptr(table.device))
    return (x, h) if w_next2 is None else (x, h, h2)


def residual_norm(base, y, w_branch, w_next, eps, dtype, *, x_out=None, want_h=True, cat=None, inv=None, mix=None,
                  rows=None, broadcast=False, add=None, w_next2=None):
    """One launch of ``msa_lm_residual_norm``; returns ``h`` (or None; with ``w_next2`` a pair).  ``base`` fp32 rows
    (``broadcast``: one vector), ``y`` the branch or the expert outputs when ``inv`` / ``mix`` [n, top] are given, ``add``
    further fp32 rows."""
    A.need_cuda(base, y)
    width = (base if base is not None else y).shape[-1]
    if rows is not None:
        n = rows.shape[0]
    elif inv is not None:
        n = inv.shape[0]
    else:
        n = y.shape[0] if y is not None else base.shape[0]
    dev = (base if base is not None else y).device
    h = torch.empty((n, width), dtype=dtype, device=dev) if want_h and w_next is not None else None
    h2 = torch.empty_like(h) if h is not None and w_next2 is not None else None
    A.call("msa_lm_residual_norm", A.ptr(base), 0 if broadcast or base is None else _rows(base), A.ptr(y),
           A.dtype_code(y.dtype) if y is not None else 0, _rows(y) if y is not None else 0, A.ptr(inv), A.ptr(mix),
           inv.shape[1] if inv is not None else 0, A.ptr(w_branch), A.ptr(w_next) if h is not None else 0, float(eps),
           A.ptr(rows), n, width, A.ptr(x_out), A.ptr(h), A.ptr(cat), _rows(cat) if cat is not None else 0, A.ptr(add),
           A.ptr(w_next2) if h2 is not None else 0, A.ptr(h2), A.dtype_code(dtype), A.stream_ptr(dev))
    return h if w_next2 is None else (h, h2)


def silu_mul(gu: torch.Tensor, ff: int, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    A.need_cuda(gu)
    if out is None:
        out = torch.empty((gu.shape[0], ff), dtype=gu.dtype, device=gu.device)
    A.call("msa_lm_silu_mul", A.ptr(gu), _rows(gu), gu.shape[0], ff, A.ptr(out), _rows(out), A.dtype_code(gu.dtype), A.stream_ptr(gu.device))
    return out


def softcap(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """In place on fp32 logits."""
    if logits.numel():
        A.call("msa_lm_softcap", A.ptr(logits), logits.numel(), float(cap), A.stream_ptr(logits.device))
    return logits


def token_shift(h, mu, step, shift):
    """``[mixes, n, width]``: every row of ``h`` mixed with its sequence's previous one (``shift`` keeps the last rows)."""
    A.need_cuda(h, mu)
    out = torch.empty((mu.shape[0],) + h.shape, dtype=h.dtype, device=h.device)
    A.call("msa_lm_token_shift", A.ptr(h), A.ptr(mu), mu.shape[0], h.shape[0], h.shape[1], A.ptr(step.tok_seq), A.ptr(step.slot),
           A.ptr(step.start), A.ptr(step.cu), A.ptr(shift), A.ptr(out), A.dtype_code(h.dtype), A.stream_ptr(h.device))
    return out


def tanh_split(x: torch.Tensor, dtype: torch.dtype, parts: int) -> torch.Tensor:
    out = torch.empty((x.shape[0], parts * x.shape[1]), dtype=dtype, device=x.device)
    A.call("msa_lm_tanh_split", A.ptr(x), x.shape[0], x.shape[1], parts, A.ptr(out), A.dtype_code(dtype), A.stream_ptr(x.device))
    return out


def part_norm(x, w, parts, eps, out):
    A.call("msa_lm_part_norm", A.ptr(x), _rows(x), A.ptr(w), x.shape[0], x.shape[1], parts, float(eps), A.ptr(out), _rows(out),
           A.dtype_code(out.dtype), A.stream_ptr(x.device))
    return out


# ---------------------------------------------------------------------------------------------- latent attention
def latent_prep(proj, spec, w_norm, inv_freq, eps, step, view, ring, ctx):
    """Normalise the latent, rotate, and place the rows of a step in ring and context (``view``: the step's context
    bookkeeping for this layer's window)."""
    A.call("msa_lm_latent_prep", A.ptr(proj), _rows(proj), A.ptr(w_norm), float(eps), A.ptr(inv_freq), spec.heads, spec.dim,
           spec.rot_dim, spec.kv_rank, A.ptr(step.pos), A.ptr(step.tok_seq), A.ptr(step.slot), A.ptr(step.start),
           A.ptr(step.cu), A.ptr(view.ctx_off), A.ptr(view.old_off), step.n_tok, step.n_seq, step.n_decode, view.n_old,
           view.window, A.ptr(ring), ring.shape[1], A.ptr(ctx), A.dtype_code(proj.dtype), A.stream_ptr(proj.device))


def ring_store(ctx, step, view, ring):
    A.call("msa_lm_ring_store", A.ptr(ctx), ctx.shape[1], A.ptr(step.slot), A.ptr(step.start), A.ptr(step.cu),
           A.ptr(view.ctx_off), step.n_seq, step.n_decode, step.max_len, view.window, A.ptr(ring), ring.shape[1],
           A.dtype_code(ctx.dtype), A.stream_ptr(ctx.device))


def attn_args(qa, qb, ka, kb, v, out, *, scale, window, start, cu, seq0, seq1, max_len, slot=None, ctx_off=None, ring_rows=0,
              sink=False, gate=None) -> A.AttnArgs:
    """``qa`` / ``qb`` / ``out`` are ``[tokens, heads, d]`` views of the query rows, ``ka`` / ``kb`` / ``v`` ``[rows, kv heads, d]``
    views of the key rows; ``gate`` ``[tokens, heads]`` logits."""
    head = lambda t: 0 if t is None or t.shape[1] == 1 else t.stride(1)
    row = lambda t: 0 if t is None else t.stride(0)
    for t in (qa, qb, ka, kb, v, out):
        if t is not None and t.stride(2) != 1:
            raise A.MsaError("window attention: contiguous last axis expected")
    return A.AttnArgs(
        qa=A.ptr(qa), qa_row=row(qa), qa_head=qa.stride(1), qb=A.ptr(qb), qb_row=row(qb), qb_head=qb.stride(1) if qb is not None else 0,
        ka=A.ptr(ka), ka_row=row(ka), ka_head=head(ka), kb=A.ptr(kb), kb_row=row(kb), kb_head=head(kb),
        v=A.ptr(v), v_row=row(v), v_head=head(v), out=A.ptr(out), out_row=row(out), out_head=out.stride(1),
        gate=A.ptr(gate), gate_row=row(gate), slot=A.ptr(slot), start=A.ptr(start), cu=A.ptr(cu), ctx_off=A.ptr(ctx_off),
        ring_rows=ring_rows, group=qa.shape[1] // max(ka.shape[1], v.shape[1]), sink=1 if sink else 0, seq0=seq0, seq1=seq1,
        max_len=max_len, heads=qa.shape[1], da=qa.shape[2], db=qb.shape[2] if qb is not None else 0, dv=v.shape[2], window=window,
        qa_dtype=A.dtype_code(qa.dtype), out_dtype=A.dtype_code(out.dtype), dtype=A.dtype_code(ka.dtype), scale=float(scale))


def window_attn(qa, qb, ka, kb, v, out, **kw):
    """General windowed attention (any sizes, both dtypes)."""
    A.call("msa_lm_window_attn", C.byref(attn_args(qa, qb, ka, kb, v, out, **kw)), A.stream_ptr(qa.device))


def window_attn_tc_supported(dim, rot, vdim, dtype, scale) -> bool:
    return dtype == torch.bfloat16 and scale > 0 and bool(A.lib().msa_lm_window_attn_tc_supported(dim, rot, vdim))


def window_attn_tc(qa, qb, ka, kb, v, out, *, row0, status, **kw):
    """The portions of a step on the tensor cores: ``qa`` / ``out`` from the first portion row (packed row ``row0``) on."""
    args = attn_args(qa, qb, ka, kb, v, out, **kw)
    A.call("msa_lm_window_attn_tc", C.byref(args), qa.shape[0], ka.shape[0], row0, A.ptr(status), A.stream_ptr(qa.device))


def latent_decode_supported(spec, dtype) -> bool:
    return (dtype == torch.bfloat16 and spec.dim % 8 == 0 and spec.scale > 0
            and bool(A.lib().msa_lm_latent_decode_supported(spec.kv_rank, spec.rot_dim)))


def latent_decode_splits(n: int, heads: int, ring_rows: int, n_sm: int = 148) -> int:
    """CTAs per sequence and head group: fill the GPU once, at least two 64-row tiles each."""
    groups = (heads + 31) // 32 if heads > 16 else 1
    return max(1, min(n_sm // max(n * groups, 1), (ring_rows + 127) // 128, 64))


def latent_decode(qa, qb, ring, slot, pos, out, *, window, scale, status):
    """``qa`` / ``qb`` / ``out`` ``[n, heads, d]`` views, ``ring`` ``[slots, rows, rank + rot]``."""
    n, heads, rank = qa.shape
    rot = 0 if qb is None else qb.shape[2]
    splits = latent_decode_splits(n, heads, ring.shape[1])
    part_o = part_ml = None
    if splits > 1:
        f = dict(dtype=torch.float32, device=qa.device)
        part_o, part_ml = torch.empty((n, heads, splits, rank), **f), torch.empty((n, heads, splits, 2), **f)
    A.call("msa_lm_latent_decode", A.ptr(qa), qa.stride(0), qa.stride(1), A.ptr(qb), 0 if qb is None else qb.stride(0),
           0 if qb is None else qb.stride(1), A.ptr(ring), ring.shape[1], A.ptr(slot), A.ptr(pos), n, heads, rank, rot, window,
           splits, float(scale), A.ptr(out), A.ptr(part_o), A.ptr(part_ml), A.ptr(status), A.stream_ptr(qa.device))


# ---------------------------------------------------------------------------------------------- grouped attention
def group_prep(proj, spec, w, step, view, ring, conv_state, q, ctx):
    """Convolve, rotate and place the rows of a step: queries in ``q`` [n, heads, pitch], keys and values in ring and context."""
    args = A.GroupArgs(proj=A.ptr(proj), proj_stride=_rows(proj), conv_w=A.ptr(w.conv), inv_freq=A.ptr(w.inv_freq), conv_state=A.ptr(conv_state),
                       q_out=A.ptr(q), ring=A.ptr(ring), ctx=A.ptr(ctx), pos=A.ptr(step.pos), tok_seq=A.ptr(step.tok_seq), slot=A.ptr(step.slot),
                       start=A.ptr(step.start), cu=A.ptr(step.cu), ctx_off=A.ptr(view.ctx_off), old_off=A.ptr(view.old_off),
                       ring_rows=ring.shape[1], heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim, vdim=spec.vdim, rot=spec.rot_dims,
                       taps=spec.taps, q_pitch=w.dim, k_pitch=w.dim, v_pitch=w.vdim, n_tok=step.n_tok, n_seq=step.n_seq,
                       n_decode=step.n_decode, n_old=view.n_old, window=view.window, dtype=A.dtype_code(proj.dtype))
    A.call("msa_lm_group_prep", C.byref(args), A.stream_ptr(proj.device))


def conv_store(proj, channels, taps, step, conv_state):
    """The portions' last convolution inputs; ``proj`` from the first convolved column on."""
    if taps > 1 and step.n_seq > step.n_decode:
        A.call("msa_lm_conv_store", A.ptr(proj), _rows(proj), channels, taps, A.ptr(conv_state), A.ptr(step.slot), A.ptr(step.start),
               A.ptr(step.cu), step.n_seq, step.n_decode, A.dtype_code(proj.dtype), A.stream_ptr(proj.device))


def group_decode_supported(dim, vdim, dtype) -> bool:
    return dtype == torch.bfloat16 and bool(A.lib().msa_lm_group_decode_supported(dim, vdim))


def group_decode_splits(n: int, heads: int, kv_heads: int, ring_rows: int, n_sm: int = 148) -> int:
    """CTAs per sequence and head group: two per SM, at least 64 rows each."""
    group = heads // kv_heads
    tiles = kv_heads * ((group + 15) // 16 if group > 8 else 1)
    return max(1, min(2 * n_sm // max(n * tiles, 1), (ring_rows + 63) // 64, 64))


def group_decode(q, ring, kv_heads, step, out, *, window, scale, sink, gate):
    """``q`` [n, heads, dim], ``out`` [n, heads, vdim] views, ``ring`` [slots, rows, kv_heads * (dim + vdim)]."""
    n, heads, dim = q.shape
    vdim = out.shape[2]
    splits = group_decode_splits(n, heads, kv_heads, ring.shape[1])
    part_o = part_ml = None
    if splits > 1:
        f = dict(dtype=torch.float32, device=q.device)
        part_o, part_ml = torch.empty((n, heads, splits, vdim), **f), torch.empty((n, heads, splits, 2), **f)
    A.call("msa_lm_group_decode", A.ptr(q), q.stride(0), A.ptr(ring), ring.shape[1], A.ptr(step.slot), A.ptr(step.start), n, heads, kv_heads, dim,
           vdim, window, splits, float(scale), 1 if sink else 0, A.ptr(gate), gate.stride(0) if gate is not None else 0, A.ptr(out),
           out.stride(0), A.ptr(part_o), A.ptr(part_ml), A.stream_ptr(q.device))


# ---------------------------------------------------------------------------------------------- decaying outer products
def wkv_mix(rkvg, decay, spec, w, state, eps, step, out):
    """``rkvg`` [4, n, heads*dim], ``decay`` fp32 [n, heads*dim] (overwritten); advances the states, fills ``out``."""
    args = A.WkvArgs(r=A.ptr(rkvg[0]), k=A.ptr(rkvg[1]), v=A.ptr(rkvg[2]), g=A.ptr(rkvg[3]), row_stride=rkvg.stride(1), decay=A.ptr(decay),
                     w0=A.ptr(w.w0), u=A.ptr(w.u), norm=A.ptr(w.norm), state=A.ptr(state), tok_seq=A.ptr(step.tok_seq), slot=A.ptr(step.slot),
                     start=A.ptr(step.start), cu=A.ptr(step.cu), n_tok=step.n_tok, n_seq=step.n_seq, n_decode=step.n_decode,
                     heads=spec.heads, dim=spec.dim, eps=float(eps), dtype=A.dtype_code(rkvg.dtype))
    dev, st = rkvg.device, A.stream_ptr(rkvg.device)
    if step.n_decode:
        A.call("msa_lm_wkv_decode", C.byref(args), A.ptr(out), _rows(out), st)
    rows = step.n_tok - step.n_decode
    if not rows:
        return out
    tail, f = out[step.n_decode:], dict(dtype=torch.float32, device=dev)
    if rkvg.dtype == torch.bfloat16 and A.lib().msa_lm_wkv_chunk_supported(spec.dim):
        work = torch.empty((step.n_chunks, spec.heads, spec.dim, spec.dim), **f)
        A.call("msa_lm_wkv_chunk", C.byref(args), A.ptr(step.chunk_off), step.n_chunks, A.ptr(work), A.ptr(tail), _rows(tail), st)
    else:
        o = torch.empty((rows, spec.heads * spec.dim), **f)
        A.call("msa_lm_wkv_scan", C.byref(args), A.ptr(o), A.ptr(tail), _rows(tail), st)
    return out


def ssd_mix(proj, spec, w, conv_state, state, eps, step, out):
    """From the projections to the input of the output product; advances the states, fills ``out``."""
    dev, st, f = proj.device, A.stream_ptr(proj.device), dict(dtype=torch.float32, device=proj.device)
    y = torch.empty((step.n_tok, spec.inner), **f)
    args = A.SsdArgs(proj=A.ptr(proj), proj_stride=_rows(proj), conv_w=A.ptr(w.conv), conv_b=A.ptr(w.conv_b), dt_bias=A.ptr(w.dt_bias),
                     a_log=A.ptr(w.a_log), d_skip=A.ptr(w.d_skip), conv_state=A.ptr(conv_state), state=A.ptr(state), tok_seq=A.ptr(step.tok_seq),
                     slot=A.ptr(step.slot), start=A.ptr(step.start), cu=A.ptr(step.cu), y=A.ptr(y), n_tok=step.n_tok, n_seq=step.n_seq,
                     n_decode=step.n_decode, heads=spec.heads, vdim=spec.vdim, n_state=spec.state, groups=spec.groups, taps=spec.taps,
                     dtype=A.dtype_code(proj.dtype))
    if step.n_decode:
        A.call("msa_lm_ssd_decode", C.byref(args), st)
    rows = step.n_tok - step.n_decode
    if rows:
        xbc, dt = torch.empty((rows, spec.channels), dtype=proj.dtype, device=dev), torch.empty((rows, spec.heads), **f)
        A.call("msa_lm_ssd_prep", C.byref(args), A.ptr(xbc), A.ptr(dt), st)
        conv_store(proj[:, spec.inner:], spec.channels, spec.taps, step, conv_state)
        if proj.dtype == torch.bfloat16 and A.lib().msa_lm_ssd_chunk_supported(spec.state, spec.vdim):
            gcum = torch.empty((rows, spec.heads), dtype=torch.float64, device=dev)
            work = torch.empty((step.n_chunks, spec.heads, spec.state, spec.vdim), **f)
            A.call("msa_lm_ssd_chunk", C.byref(args), A.ptr(xbc), A.ptr(dt), A.ptr(step.chunk_off), step.n_chunks, A.ptr(gcum), A.ptr(work), st)
        else:
            A.call("msa_lm_ssd_scan", C.byref(args), A.ptr(xbc), A.ptr(dt), st)
    return part_norm(y, w.norm, spec.norm_groups, eps, out)


# ---------------------------------------------------------------------------------------------- gated delta rule
def delta_args(proj, spec, w, conv_state, state, eps, step) -> A.DeltaArgs:
    return A.DeltaArgs(proj=A.ptr(proj), proj_stride=_rows(proj), conv_w=A.ptr(w.conv), a_log=A.ptr(w.a_log),
                       dt_bias=A.ptr(w.dt_bias), w_norm=A.ptr(w.norm), conv_state=A.ptr(conv_state), state=A.ptr(state),
                       pos=A.ptr(step.pos), tok_seq=A.ptr(step.tok_seq), slot=A.ptr(step.slot), start=A.ptr(step.start),
                       cu=A.ptr(step.cu), n_tok=step.n_tok, n_seq=step.n_seq, n_decode=step.n_decode, heads=spec.heads,
                       kv_heads=spec.kv_heads, dim=spec.dim, vdim=spec.vdim, taps=spec.taps, eps=float(eps),
                       dtype=A.dtype_code(proj.dtype))


def delta_chunk_supported(spec, dtype) -> bool:
    return dtype == torch.bfloat16 and bool(A.lib().msa_lm_delta_chunk_supported(spec.dim, spec.vdim, spec.taps))


def delta_tile(n_seq: int, heads: int, vdim: int, n_sm: int = 148) -> int:
    """Value columns per CTA of the chunked recurrence: wide ones unless that leaves most of the GPU idle."""
    best = 32
    for t in (128, 64, 32):
        if vdim % t == 0:
            best = t
            if n_seq * heads * (vdim // t) * 2 >= n_sm:
                break
    return best


def delta_portions(args, spec, step, out) -> None:
    """The portions of a step through the chunked kernels."""
    dev, st = out.device, A.stream_ptr(out.device)
    rows, heads = step.n_tok - step.n_decode, spec.heads
    qk = torch.empty((rows, 4 * spec.kv_heads * spec.dim), dtype=torch.bfloat16, device=dev)
    f = dict(dtype=torch.float32, device=dev)
    v = torch.empty((rows, heads * spec.vdim), dtype=torch.bfloat16, device=dev)
    gates = torch.empty((rows, 2 * heads), **f)
    A.call("msa_lm_delta_prep_split", C.byref(args), A.ptr(qk), A.ptr(v), A.ptr(gates), st)
    A.call("msa_lm_delta_conv_store", C.byref(args), st)
    delta_chunks(args, spec, step, qk, v, gates, out)


def delta_chunks(args, spec, step, qk, v, gates, out) -> None:
    dev, heads = out.device, spec.heads
    tile = delta_tile(step.n_seq - step.n_decode, heads, spec.vdim)
    work = torch.empty(A.lib().msa_lm_delta_chunk_workspace(step.n_chunks, heads), dtype=torch.uint8, device=dev)
    o = torch.empty(v.shape, dtype=torch.float32, device=dev) if tile != spec.vdim else None
    A.call("msa_lm_delta_chunk", C.byref(args), A.ptr(qk), A.ptr(v), A.ptr(gates), A.ptr(step.chunk_off), step.n_chunks, tile,
           A.ptr(work), A.ptr(o), A.ptr(out), _rows(out), A.stream_ptr(dev))


def delta_mix(proj, spec, w, conv_state, state, eps, step) -> torch.Tensor:
    """From the projections to the input of the output product, ``[n_tok, heads*vdim]``; advances the states."""
    args = delta_args(proj, spec, w, conv_state, state, eps, step)
    dev, st = proj.device, A.stream_ptr(proj.device)
    out = torch.empty((step.n_tok, spec.heads * spec.vdim), dtype=proj.dtype, device=dev)
    if step.n_decode:
        A.call("msa_lm_delta_decode", C.byref(args), A.ptr(out), _rows(out), st)
    rows = step.n_tok - step.n_decode
    if not rows:
        return out
    tail = out[step.n_decode:]
    if delta_chunk_supported(spec, proj.dtype):
        delta_portions(args, spec, step, tail)
        return out
    f = dict(dtype=torch.float32, device=dev)
    qk = torch.empty((rows, 2 * spec.kv_heads * spec.dim), **f)
    v = torch.empty((rows, spec.heads * spec.vdim), **f)
    gates = torch.empty((rows, 2 * spec.heads), **f)
    o = torch.empty((rows, spec.heads * spec.vdim), **f)
    A.call("msa_lm_delta_prep", C.byref(args), A.ptr(qk), A.ptr(v), A.ptr(gates), st)
    A.call("msa_lm_delta_conv_store", C.byref(args), st)
    A.call("msa_lm_delta_scan", C.byref(args), A.ptr(qk), A.ptr(v), A.ptr(gates), A.ptr(o), st)
    A.call("msa_lm_delta_out", C.byref(args), A.ptr(o), A.ptr(tail), _rows(tail), st)
    return out


# ---------------------------------------------------------------------------------------------- experts
MOE_TILE_ROWS = 32


def moe_topk(logits, bias, top):
    n, experts = logits.shape
    idx = torch.empty((n, top), dtype=torch.int32, device=logits.device)
    weight = torch.empty((n, top), dtype=torch.float32, device=logits.device)
    A.call("msa_lm_moe_topk", A.ptr(logits), _rows(logits), A.ptr(bias), n, experts, top, A.ptr(idx), A.ptr(weight),
           A.stream_ptr(logits.device))
    return idx, weight


def moe_sort(idx, experts, tile_rows=MOE_TILE_ROWS):
    """``(src, inv, off, tiles)``: the choices grouped by expert."""
    n, top = idx.shape
    dev = idx.device
    max_tiles = n * top // tile_rows + min(n * top, experts)
    i = dict(dtype=torch.int32, device=dev)
    src, inv = torch.empty(n * top, **i), torch.empty((n, top), **i)
    off, tiles = torch.empty(experts + 1, **i), torch.empty((max_tiles, 2), **i)
    counts = torch.empty(((n * top + 2047) // 2048, experts), **i) if n * top > 4096 else None
    A.call("msa_lm_moe_sort", A.ptr(idx), n, top, experts, tile_rows, A.ptr(src), A.ptr(inv), A.ptr(off), A.ptr(tiles),
           max_tiles, A.ptr(counts), A.stream_ptr(dev))
    return src, inv, off, tiles


def moe_gemm(x, src, w, off, tiles, *, entries, act, limit=0.0, out_dtype=None):
    experts, n_out, k = w.shape
    cols = n_out // 2 if act else n_out
    out = torch.empty((entries, cols), dtype=out_dtype or x.dtype, device=x.device)
    A.call("msa_lm_moe_gemm", A.ptr(x), _rows(x), A.ptr(src), A.ptr(w), A.ptr(off), A.ptr(tiles), tiles.shape[0], n_out, k,
           1 if act else 0, float(limit), A.ptr(out), _rows(out), A.dtype_code(out.dtype), A.dtype_code(x.dtype),
           A.stream_ptr(x.device))
    return out


MOE_TC_TILE_ROWS = 128
MOE_GATHER_ROWS = 64      # entries per expert from which a copy of the grouped rows beats fetching them four at a time


def gather_rows(x, src):
    out = torch.empty((src.shape[0], x.shape[1]), dtype=x.dtype, device=x.device)
    A.call("msa_lm_gather_rows", A.ptr(x), _rows(x) * x.element_size(), A.ptr(src), src.shape[0], x.shape[1] * x.element_size(),
           A.ptr(out), A.stream_ptr(x.device))
    return out


def moe_tc_supported(dtype, width, ff) -> bool:
    return dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0


def moe_gemm_tc(x, src, w, off, tiles, *, entries, act, limit=0.0, status):
    experts, n_out, k = w.shape
    out = torch.empty((entries, n_out // 2 if act else n_out), dtype=x.dtype, device=x.device)
    A.call("msa_lm_moe_gemm_tc", A.ptr(x), _rows(x), x.shape[0], A.ptr(src), A.ptr(w), experts, A.ptr(off), A.ptr(tiles),
           tiles.shape[0], n_out, k, 1 if act else 0, float(limit), A.ptr(out), _rows(out), A.ptr(status), A.stream_ptr(x.device))
    return out
