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


def embed(table, token, w_next, eps, cat: Optional[torch.Tensor] = None, cat_both: bool = False, status=None):
    """``(x fp32, h)``: the embedding rows and, with ``w_next``, their norm.  ``cat`` [n, 2*width]: its right half (with
    ``cat_both`` its left half too) receives the rows."""
    A.need_cuda(table, token)
    n, width = token.shape[0], table.shape[1]
    x = torch.empty((n, width), dtype=torch.float32, device=table.device)
    h = torch.empty((n, width), dtype=table.dtype, device=table.device) if w_next is not None else None
    cat0 = A.ptr(cat) if cat is not None and cat_both else 0
    cat1 = A.ptr(cat) + width * cat.element_size() if cat is not None else 0
    A.call("msa_lm_embed", A.ptr(table), A.ptr(token), n, width, table.shape[0], A.ptr(w_next), float(eps), A.ptr(x),
           A.ptr(h), cat0, cat1, _rows(cat) if cat is not None else 0, A.ptr(status), A.dtype_code(table.dtype),
           A.stream_ptr(table.device))
    return x, h


def residual_norm(base, y, w_branch, w_next, eps, dtype, *, x_out=None, want_h=True, cat=None, inv=None, mix=None,
                  rows=None, broadcast=False):
    """One launch of ``msa_lm_residual_norm``; returns ``h`` (or None).  ``base`` fp32 rows (``broadcast``: one vector),
    ``y`` the branch or the expert outputs when ``inv`` / ``mix`` [n, top] are given."""
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
    A.call("msa_lm_residual_norm", A.ptr(base), 0 if broadcast or base is None else _rows(base), A.ptr(y),
           A.dtype_code(y.dtype) if y is not None else 0, _rows(y) if y is not None else 0, A.ptr(inv), A.ptr(mix),
           inv.shape[1] if inv is not None else 0, A.ptr(w_branch), A.ptr(w_next) if h is not None else 0, float(eps),
           A.ptr(rows), n, width, A.ptr(x_out), A.ptr(h), A.ptr(cat), _rows(cat) if cat is not None else 0,
           A.dtype_code(dtype), A.stream_ptr(dev))
    return h


def silu_mul(gu: torch.Tensor, ff: int) -> torch.Tensor:
    A.need_cuda(gu)
    out = torch.empty((gu.shape[0], ff), dtype=gu.dtype, device=gu.device)
    A.call("msa_lm_silu_mul", A.ptr(gu), _rows(gu), gu.shape[0], ff, A.ptr(out), A.dtype_code(gu.dtype), A.stream_ptr(gu.device))
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


def window_attn(qa, qb, ka, kb, v, out, *, scale, window, start, cu, seq0, seq1, max_len, slot=None, ctx_off=None, ring_rows=0):
    """General windowed attention.  ``qa`` / ``qb`` / ``out`` are ``[tokens, heads, d]`` views of the query rows,
    ``ka`` / ``kb`` / ``v`` ``[rows, heads or 1, d]`` views of the key rows (1: shared by the heads)."""
    head = lambda t: 0 if t is None or t.shape[1] == 1 else t.stride(1)
    row = lambda t: 0 if t is None else t.stride(0)
    for t in (qa, qb, ka, kb, v, out):
        if t is not None and t.stride(2) != 1:
            raise A.MsaError("window_attn: contiguous last axis expected")
    args = A.AttnArgs(
        qa=A.ptr(qa), qa_row=row(qa), qa_head=qa.stride(1), qb=A.ptr(qb), qb_row=row(qb), qb_head=qb.stride(1) if qb is not None else 0,
        ka=A.ptr(ka), ka_row=row(ka), ka_head=head(ka), kb=A.ptr(kb), kb_row=row(kb), kb_head=head(kb),
        v=A.ptr(v), v_row=row(v), v_head=head(v), out=A.ptr(out), out_row=row(out), out_head=out.stride(1),
        slot=A.ptr(slot), start=A.ptr(start), cu=A.ptr(cu), ctx_off=A.ptr(ctx_off), ring_rows=ring_rows, seq0=seq0, seq1=seq1,
        max_len=max_len, heads=qa.shape[1], da=qa.shape[2], db=qb.shape[2] if qb is not None else 0, dv=v.shape[2], window=window,
        qa_dtype=A.dtype_code(qa.dtype), out_dtype=A.dtype_code(out.dtype), dtype=A.dtype_code(ka.dtype), scale=float(scale))
    A.call("msa_lm_window_attn", C.byref(args), A.stream_ptr(qa.device))


def window_attn_tc_supported(spec, dtype) -> bool:
    return (dtype == torch.bfloat16 and spec.kv_rank % 8 == 0 and spec.scale > 0
            and bool(A.lib().msa_lm_window_attn_tc_supported(spec.dim, spec.rot_dim, spec.vdim)))


def window_attn_tc(proj, kv, ctx, spec, out, step, view, status):
    """The portions of a step on the tensor cores: ``proj`` / ``out`` from the first portion row on."""
    A.call("msa_lm_window_attn_tc", A.ptr(proj), _rows(proj), proj.shape[0], A.ptr(kv), _rows(kv), A.ptr(ctx), _rows(ctx),
           ctx.shape[0], spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank, A.ptr(step.start), A.ptr(step.cu),
           A.ptr(view.ctx_off), step.n_decode, step.n_seq, step.n_decode, step.max_len, view.window, float(spec.scale),
           A.ptr(out), _rows(out), A.ptr(status), A.stream_ptr(proj.device))


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
