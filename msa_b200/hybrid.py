"""Layered decoder designs: a stack whose layers each name their mixer and feed-forward, on the package's kernels.

The configuration (``hybrid_config``) lists the layers; a mixer is a class below with its weights, its per-sequence
state (``state_spec``) and its forward step; ``hybrid_config.Structure`` says how a design frames its layers.  A step works on packed tokens of many sequences (``cache.PackedStep``):
matrix products run over all of them at once, the mixers treat single-token continuations and longer portions by their
own kernels.  The residual stream is fp32; between two products one launch does branch norm, residual add, next norm
and rounding (``lm_ops.residual_norm``), including the weighted sum over a mixture's experts.  Where mixer and feed-forward
read the same stream side by side, that launch writes both of their norms, and their output products are one product over
their joined columns.

``HybridForCausalLM.step`` is the serving entry (scheduler, trace replay, benchmark); ``forward`` takes the keyword
arguments of ``MSAForCausalLM.forward``, so that the interleave loop can drive either.
"""
from __future__ import annotations

import glob
import os
from types import SimpleNamespace
from typing import Dict, List, Optional

import torch

from . import lm_ops as K
from .cache import DecodeStep, PackedStep, RecurrentSpec, RingSpec, SequenceStateCache
from .hybrid_config import HybridConfig


class Weights:
    """Checkpoint tensors by name; every tensor must be taken exactly once."""

    def __init__(self, tensors: Dict[str, torch.Tensor], device, dtype: torch.dtype):
        self._t, self._left, self.device, self.dtype = tensors, set(tensors), torch.device(device), dtype
        self.status = torch.zeros(4, dtype=torch.int32, device=device)     # shared by the kernels that report

    def has(self, name: str) -> bool:
        return name in self._t

    def shape(self, name: str):
        if name not in self._t:
            raise KeyError(f"checkpoint lacks {name}")
        return tuple(self._t[name].shape)

    def raw(self, name: str, *shape: int) -> torch.Tensor:
        if name not in self._t:
            raise KeyError(f"checkpoint lacks {name}")
        t = self._t[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name} has shape {tuple(t.shape)}, the configuration says {shape}")
        self._left.discard(name)
        return t

    def matrix(self, name: str, *shape: int) -> torch.Tensor:
        return self.raw(name, *shape).to(device=self.device, dtype=self.dtype).contiguous()

    def vector(self, name: str, *shape: int) -> torch.Tensor:
        return self.raw(name, *shape).to(device=self.device, dtype=torch.float32).contiguous()

    def stack(self, names_rows, cols: int, pad: bool = False) -> torch.Tensor:
        """Matrices with a common input, stacked by output rows: one product instead of several.  ``pad``: zero rows up to
        a multiple of 8, so that every row of the product starts on a 16-byte boundary."""
        m = torch.cat([self.raw(n, r, cols) for n, r in names_rows])
        if pad and m.shape[0] % 8:
            m = torch.cat([m, m.new_zeros((-m.shape[0] % 8, cols))])
        return m.to(device=self.device, dtype=self.dtype).contiguous()

    def check_all_used(self) -> None:
        if self._left:
            raise ValueError(f"checkpoint tensors the configuration does not name: {sorted(self._left)[:5]}")


class Mixer:
    """``mix`` goes from the input projections (one product with ``w_in``) to the input of the output product (``w_o``)."""

    def forward(self, h: torch.Tensor, step, cache: SequenceStateCache, run: int, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        y = self.mix(K.matmul(h, self.w_in), step, cache, run)
        return y if out is None else out.copy_(y)


class LatentAttention(Mixer):
    """Windowed attention over a cached low-rank latent.  Portions expand keys and values for their context and attend
    per head; single tokens fold the key expansion into the query and attend over the latents themselves."""

    def __init__(self, spec, w: Weights, prefix: str, width: int, eps: float):
        s = self.spec = spec
        self.eps, self.status = eps, w.status
        self.tc_prompt = s.kv_rank % 8 == 0 and K.window_attn_tc_supported(s.dim, s.rot_dim, s.vdim, w.dtype, s.scale)
        self.tc_decode = K.latent_decode_supported(s, w.dtype)
        self.w_in = w.stack([(prefix + "q", s.heads * (s.dim + s.rot_dim)), (prefix + "dkv", s.kv_rank + s.rot_dim)], width, pad=True)
        self.norm = w.vector(prefix + "dkv.norm", s.kv_rank)
        self.w_kv = w.stack([(prefix + "uk", s.heads * s.dim), (prefix + "uv", s.heads * s.vdim)], s.kv_rank)
        self.w_uk = self.w_kv[:s.heads * s.dim].view(s.heads, s.dim, s.kv_rank)
        self.w_uv = self.w_kv[s.heads * s.dim:].view(s.heads, s.vdim, s.kv_rank)
        self.w_o = w.matrix(prefix + "o", width, s.heads * s.vdim)
        i = torch.arange(s.rot_dim // 2, dtype=torch.float64)
        self.inv_freq = (s.rot_base ** (-2.0 * i / max(s.rot_dim, 1))).to(torch.float32).to(self.w_in.device)

    @property
    def state_spec(self) -> RingSpec:
        return RingSpec(self.spec.kv_rank + self.spec.rot_dim, self.spec.window)

    def mix(self, proj: torch.Tensor, step, cache: SequenceStateCache, run: int) -> torch.Tensor:
        s, n, nd = self.spec, step.n_tok, step.n_decode
        ring, view = cache.ring[run], step.views[s.window]
        out = torch.empty((n, s.heads * s.vdim), dtype=proj.dtype, device=proj.device)
        ctx = torch.empty((view.n_ctx, s.kv_rank + s.rot_dim), dtype=proj.dtype, device=proj.device) if n > nd else None
        K.latent_prep(proj, s, self.norm, self.inv_freq, self.eps, step, view, ring, ctx)
        q = proj[:, :s.heads * (s.dim + s.rot_dim)].view(n, s.heads, s.dim + s.rot_dim)
        if nd:
            self._decode(q[:nd], step, view, ring, out[:nd])
        if n > nd:
            kv = K.matmul(ctx[:, :s.kv_rank], self.w_kv)
            k = kv[:, :s.heads * s.dim].view(-1, s.heads, s.dim)
            v = kv[:, s.heads * s.dim:].view(-1, s.heads, s.vdim)
            kr = ctx[:, s.kv_rank:].unsqueeze(1) if s.rot_dim else None
            qp = q[nd:]
            args = (qp[..., :s.dim], qp[..., s.dim:] if s.rot_dim else None, k, kr, v, out[nd:].view(n - nd, s.heads, s.vdim))
            portion_attention(args, self.tc_prompt, self.status, step, view, s.scale)
            K.ring_store(ctx, step, view, ring)
        return out

    def _decode(self, q, step, view, ring, out) -> None:
        s, n = self.spec, q.shape[0]
        if self.tc_decode:
            qa = torch.bmm(q[..., :s.dim].transpose(0, 1), self.w_uk)                     # [heads, n, rank]
            lat = torch.empty((n, s.heads, s.kv_rank), dtype=q.dtype, device=q.device)
            K.latent_decode(qa.transpose(0, 1), q[..., s.dim:] if s.rot_dim else None, ring, step.slot, step.start, lat,
                            window=view.window, scale=s.scale, status=self.status)
            torch.bmm(lat.transpose(0, 1), self.w_uv.transpose(1, 2), out=out.view(n, s.heads, s.vdim).transpose(0, 1))
            return
        f32 = dict(out_dtype=torch.float32) if q.dtype != torch.float32 else {}
        qa = torch.bmm(q[..., :s.dim].transpose(0, 1), self.w_uk, **f32)                  # [heads, n, rank]
        lat = torch.empty((n, s.heads, s.kv_rank), dtype=q.dtype, device=q.device)
        rows = ring.view(-1, 1, s.kv_rank + s.rot_dim)
        K.window_attn(qa.transpose(0, 1), q[..., s.dim:] if s.rot_dim else None, rows[..., :s.kv_rank],
                      rows[..., s.kv_rank:] if s.rot_dim else None, rows[..., :s.kv_rank], lat, scale=s.scale,
                      window=view.window, start=step.start, cu=step.cu, seq0=0, seq1=n, max_len=1, slot=step.slot,
                      ring_rows=ring.shape[1])
        out.view(n, s.heads, s.vdim).copy_(torch.bmm(lat.transpose(0, 1), self.w_uv.transpose(1, 2)).transpose(0, 1))


class GatedDelta(Mixer):
    """Gated delta rule behind a short causal convolution."""

    def __init__(self, spec, w: Weights, prefix: str, width: int, eps: float):
        s = self.spec = spec
        self.eps = eps
        qk, v = s.kv_heads * s.dim, s.heads * s.vdim
        self.w_in = w.stack([(prefix + "q", qk), (prefix + "k", qk), (prefix + "v", v), (prefix + "g", v),
                             (prefix + "b", s.heads), (prefix + "a", s.heads)], width, pad=True)
        self.conv = torch.cat([w.vector(prefix + n + ".conv", r, s.taps) for n, r in (("q", qk), ("k", qk), ("v", v))]).t().contiguous()
        self.a_log, self.dt_bias = w.vector(prefix + "A_log", s.heads), w.vector(prefix + "dt_bias", s.heads)
        self.norm = w.vector(prefix + "norm", s.vdim)
        self.w_o = w.matrix(prefix + "o", width, v)

    @property
    def state_spec(self) -> RecurrentSpec:
        s = self.spec
        return RecurrentSpec(s.heads, s.dim, s.vdim, s.channels, s.taps)

    def mix(self, proj: torch.Tensor, step, cache: SequenceStateCache, run: int) -> torch.Tensor:
        return K.delta_mix(proj, self.spec, self, cache.conv[run], cache.state[run], self.eps, step)


def portion_attention(args, tc: bool, status, step, view, scale, **kw) -> None:
    """The portions of a step (``args``: q parts, k parts, v, out) over their packed context."""
    kw.update(scale=scale, window=view.window, start=step.start, cu=step.cu, seq0=step.n_decode, seq1=step.n_seq, max_len=step.max_len,
              ctx_off=view.ctx_off)
    if tc:
        K.window_attn_tc(*args, row0=step.n_decode, status=status, **kw)
    else:
        K.window_attn(*args, **kw)


class GroupedAttention(Mixer):
    """Grouped-query window attention behind a short convolution, with a silent sink and a gate per head.  Head sizes up to 128
    are stored with zeros up to 64 or 128 in bf16, so that the tensor-core kernels take any of them."""

    def __init__(self, spec, w: Weights, prefix: str, width: int, eps: float):
        s = self.spec = spec
        self.status = w.status
        nq, nk, nv = s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim
        rows = [(prefix + "q", nq), (prefix + "k", nk), (prefix + "v", nv)] + ([(prefix + "g", s.heads)] if s.gate else [])
        self.w_in = w.stack(rows, width, pad=True)
        self.conv = torch.cat([w.vector(prefix + n + ".conv", r, s.taps) for n, r in (("q", nq), ("k", nk), ("v", nv))]).t().contiguous()
        up = lambda d: d if w.dtype != torch.bfloat16 or d > 128 else (64 if d <= 64 else 128)
        self.dim, self.vdim = up(s.dim), up(s.vdim)                  # as stored
        self.tc_prompt = K.window_attn_tc_supported(self.dim, 0, self.vdim, w.dtype, s.scale)
        self.tc_decode = K.group_decode_supported(self.dim, self.vdim, w.dtype)
        w_o = w.matrix(prefix + "o", width, s.heads * s.vdim)
        self.w_o = torch.nn.functional.pad(w_o.view(width, s.heads, s.vdim), (0, self.vdim - s.vdim)).reshape(width, s.heads * self.vdim)
        i = torch.arange(s.rot_dims // 2, dtype=torch.float64)
        self.inv_freq = (s.rot_base ** (-2.0 * i / max(s.rot_dims, 1))).to(torch.float32).to(self.w_in.device)

    @property
    def state_spec(self) -> RingSpec:
        s = self.spec
        return RingSpec(s.kv_heads * (self.dim + self.vdim), s.window, s.channels, s.taps)

    def forward(self, h, step, cache, run, out=None):
        return self.mix(K.matmul(h, self.w_in), step, cache, run, out)

    def mix(self, proj: torch.Tensor, step, cache: SequenceStateCache, run: int, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        s, n, nd = self.spec, step.n_tok, step.n_decode
        ring, view, conv = cache.ring[run], step.views[s.window], cache.conv[run]
        new = torch.empty if (self.dim, self.vdim) == (s.dim, s.vdim) else torch.zeros      # the filling must be zero
        kw = dict(dtype=proj.dtype, device=proj.device)
        q = new((n, s.heads, self.dim), **kw)
        ctx = new((view.n_ctx, s.kv_heads * (self.dim + self.vdim)), **kw) if n > nd else None
        if out is None:
            out = torch.empty((n, s.heads * self.vdim), **kw)
        K.group_prep(proj, s, self, step, view, ring, conv, q, ctx)
        heads_out = out.unflatten(1, (s.heads, self.vdim))
        gate = proj[:, s.channels:s.channels + s.heads] if s.gate else None
        split = s.kv_heads * self.dim
        parts = lambda rows: (rows[:, :split].unflatten(1, (s.kv_heads, self.dim)), rows[:, split:].unflatten(1, (s.kv_heads, self.vdim)))
        if nd and self.tc_decode:
            K.group_decode(q[:nd], ring, s.kv_heads, step, heads_out[:nd], window=view.window, scale=s.scale, sink=s.sink,
                           gate=None if gate is None else gate[:nd])
        elif nd:
            k, v = parts(ring.view(-1, ring.shape[2]))
            K.window_attn(q[:nd], None, k, None, v, heads_out[:nd], scale=s.scale, window=view.window, start=step.start, cu=step.cu, seq0=0,
                          seq1=nd, max_len=1, slot=step.slot, ring_rows=ring.shape[1], sink=s.sink, gate=None if gate is None else gate[:nd])
        if n > nd:
            K.conv_store(proj, s.channels, s.taps, step, conv)
            k, v = parts(ctx)
            portion_attention((q[nd:], None, k, None, v, heads_out[nd:]), self.tc_prompt, self.status, step, view, s.scale, sink=s.sink,
                              gate=None if gate is None else gate[nd:])
            K.ring_store(ctx, step, view, ring)
        return out


class Wkv(Mixer):
    """Decaying outer products with a decay per key channel.  The decays' small products keep 32 bits: their input between the
    two is a pair of bf16 numbers."""

    def __init__(self, spec, w: Weights, prefix: str, width: int, eps: float):
        s = self.spec = spec
        self.eps = eps
        self.mu = torch.stack([w.vector(prefix + "mu." + n, width) for n in "rkvgw"])
        self.w_in = torch.stack([w.matrix(prefix + n, s.inner, width) for n in "rkvg"])
        rank = w.shape(prefix + "w1")[0]
        self.w1 = w.stack([(prefix + "w1", rank)], width, pad=True)
        w2 = torch.nn.functional.pad(w.matrix(prefix + "w2", s.inner, rank), (0, self.w1.shape[0] - rank))
        self.parts = 2 if w.dtype == torch.bfloat16 else 1
        self.w2 = w2.repeat(1, self.parts).contiguous()
        self.w0, self.u = w.vector(prefix + "w0", s.inner), w.vector(prefix + "u", s.heads, s.dim)
        self.norm = w.vector(prefix + "norm", s.inner)
        self.w_o = w.matrix(prefix + "o", width, s.inner)

    @property
    def state_spec(self) -> RecurrentSpec:
        s = self.spec
        return RecurrentSpec(s.heads, s.dim, s.dim, shift=self.mu.shape[1])

    def forward(self, h, step, cache, run, out=None):
        mixes = K.token_shift(h, self.mu, step, cache.shift[run])
        rkvg = torch.bmm(mixes[:4], self.w_in.transpose(1, 2))
        low = K.tanh_split(K.matmul(mixes[4], self.w1, torch.float32), h.dtype, self.parts)
        decay = K.matmul(low, self.w2, torch.float32)
        if out is None:
            out = torch.empty((h.shape[0], self.spec.inner), dtype=h.dtype, device=h.device)
        return K.wkv_mix(rkvg, decay, self.spec, self, cache.state[run], self.eps, step, out)


class Mamba2(Mixer):
    """State-space recurrence behind a short convolution, gated, normalised in parts."""

    def __init__(self, spec, w: Weights, prefix: str, width: int, eps: float):
        s = self.spec = spec
        self.eps = eps
        self.w_in = w.stack([(prefix + "in", s.inner + s.channels + s.heads)], width, pad=True)
        self.conv = w.vector(prefix + "conv", s.channels, s.taps).t().contiguous()
        self.conv_b = w.vector(prefix + "conv.b", s.channels)
        self.dt_bias, self.a_log, self.d_skip = (w.vector(prefix + n, s.heads) for n in ("dt_bias", "A_log", "D"))
        self.norm = w.vector(prefix + "norm", s.inner)
        self.w_o = w.matrix(prefix + "o", width, s.inner)

    @property
    def state_spec(self) -> RecurrentSpec:
        s = self.spec
        return RecurrentSpec(s.heads, s.state, s.vdim, s.channels, s.taps)

    def forward(self, h, step, cache, run, out=None):
        if out is None:
            out = torch.empty((h.shape[0], self.spec.inner), dtype=h.dtype, device=h.device)
        return K.ssd_mix(K.matmul(h, self.w_in), self.spec, self, cache.conv[run], cache.state[run], self.eps, step, out)


class DenseFeedForward:
    def __init__(self, spec, w: Weights, prefix: str, width: int):
        self.ff = spec.ff
        self.w_gate_up = w.stack([(prefix + "gate", spec.ff), (prefix + "up", spec.ff)], width)
        self.w_down = w.matrix(prefix + "down", width, spec.ff)

    def activate(self, h: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        return K.silu_mul(K.matmul(h, self.w_gate_up), self.ff, out)

    def branch(self, h: torch.Tensor) -> dict:
        return dict(y=K.matmul(self.activate(h), self.w_down))


class MixtureFeedForward:
    """Top-k mixture of small clamped experts; the weighted sum over a token's experts is left to the residual step."""

    def __init__(self, spec, w: Weights, prefix: str, width: int):
        s = self.spec = spec
        self.router = w.matrix(prefix + "router", s.experts, width)
        self.bias = w.vector(prefix + "router.b", s.experts)
        dev, dt = w.device, w.dtype
        self.status, self.tc = w.status, K.moe_tc_supported(dt, width, s.ff)
        self.w_gate_up = torch.empty((s.experts, 2 * s.ff, width), dtype=dt, device=dev)
        self.w_down = torch.empty((s.experts, width, s.ff), dtype=dt, device=dev)
        for e in range(s.experts):
            p = f"{prefix}e{e}."
            self.w_gate_up[e, :s.ff] = w.raw(p + "gate", s.ff, width)
            self.w_gate_up[e, s.ff:] = w.raw(p + "up", s.ff, width)
            self.w_down[e] = w.raw(p + "down", width, s.ff)

    def branch(self, h: torch.Tensor) -> dict:
        s, n = self.spec, h.shape[0]
        idx, mix = K.moe_topk(K.matmul(h, self.router, torch.float32), self.bias, s.top)
        if self.tc:
            src, inv, off, tiles = K.moe_sort(idx, s.experts, K.MOE_TC_TILE_ROWS)
            if n * s.top >= s.experts * K.MOE_GATHER_ROWS:
                h, src = K.gather_rows(h, src), None
            act = K.moe_gemm_tc(h, src, self.w_gate_up, off, tiles, entries=n * s.top, act=True, limit=s.limit, status=self.status)
            return dict(y=K.moe_gemm_tc(act, None, self.w_down, off, tiles, entries=n * s.top, act=False, status=self.status),
                        inv=inv, mix=mix)
        src, inv, off, tiles = K.moe_sort(idx, s.experts)
        act = K.moe_gemm(h, src, self.w_gate_up, off, tiles, entries=n * s.top, act=True, limit=s.limit)
        y = K.moe_gemm(act, None, self.w_down, off, tiles, entries=n * s.top, act=False)
        return dict(y=y, inv=inv, mix=mix)


MIXERS = {"latent_attention": LatentAttention, "delta": GatedDelta, "attention": GroupedAttention, "wkv": Wkv, "mamba2": Mamba2}
FEED_FORWARDS = {"dense": DenseFeedForward, "moe": MixtureFeedForward}


class HybridForCausalLM:
    """Weights, layer runs and the packed step."""

    def __init__(self, config: HybridConfig, tensors, device, dtype: torch.dtype = torch.bfloat16):
        """``tensors``: the checkpoint's tensors by name, or a ``Weights`` that hands them out."""
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False     # 32-bit accumulation throughout
        w = tensors if isinstance(tensors, Weights) else Weights(tensors, self.device, dtype)
        c, width = config, config.width
        norm = lambda name: w.vector(name, width) + c.structure.norm_offset
        self.embed = w.matrix("embed", c.vocab, width)
        self.head = self.embed if c.structure.tied else w.matrix("head", c.vocab, width)
        self.pair = None
        if c.bigram is not None:
            self.pair = (w.matrix("bigram", c.bigram.buckets + 1, width), c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur)
        self.final_norm = norm("final.norm")
        if c.loop is not None and c.structure.loop_input == "project":
            self.loop_in = w.matrix("loop.in", width, 2 * width)
            self.loop_step = w.vector("loop.step", c.loop.times, width)
        self.layers: List[SimpleNamespace] = []
        for i, spec in enumerate(c.layers):
            p = f"l{i}."
            layer = SimpleNamespace(mixer=MIXERS[spec.mixer.kind](spec.mixer, w, p + "mix.", width, c.eps), norm1=norm(p + "norm1"),
                                    norm1b=None, norm2=None, norm2b=None, ff=None)
            sandwich = c.structure.block == "sandwich"
            if sandwich:
                layer.norm1b = norm(p + "norm1b")
            if spec.mlp is not None:
                layer.ff = FEED_FORWARDS[spec.mlp.kind](spec.mlp, w, p + "mlp.", width)
                layer.norm2 = norm(p + "norm2")
                if sandwich:
                    layer.norm2b = norm(p + "norm2b")
            else:                          # a layer without a feed-forward has no use for its norms
                for name in (p + "norm2", p + "norm2b"):
                    if w.has(name):
                        norm(name)
            if not sandwich:
                self._join_outputs(layer)
            self.layers.append(layer)
        w.check_all_used()
        self.status = w.status
        self._program = self._compile()
        self.on_layer = None       # hook(run, x): the stream after every layer run (debugging)

    @classmethod
    def from_pretrained(cls, path: str, device, dtype: torch.dtype = torch.bfloat16) -> "HybridForCausalLM":
        from safetensors.torch import load_file
        tensors: Dict[str, torch.Tensor] = {}
        for shard in sorted(glob.glob(os.path.join(path, "*.safetensors"))):
            tensors.update(load_file(shard))
        return cls(HybridConfig.from_pretrained(path), tensors, device, dtype)

    @staticmethod
    def _join_outputs(layer) -> None:
        """One output product for mixer and feed-forward over their joined columns; the parts become views of it."""
        m, ff = layer.mixer, layer.ff
        layer.cols = m.w_o.shape[1]
        layer.w_out = m.w_o if ff is None else torch.cat([m.w_o, ff.w_down], dim=1).contiguous()
        m.w_o = layer.w_out[:, :layer.cols]
        if ff is not None:
            ff.w_down = layer.w_out[:, layer.cols:]

    # ------------------------------------------------------------------ structure
    def _compile(self):
        """The run as a list of (kind, run, layer, pass): what is norm-ed for whom follows from the next entry."""
        prog, loop = [], self.config.loop
        if self.config.structure.block != "sandwich":
            return prog
        for run, (i, t) in enumerate(self.config.runs()):
            if loop is not None and t is not None and i == loop.start:
                prog.append(("enter", run, i, t))
            prog.append(("mix", run, i, t))
            if self.layers[i].ff is not None:
                prog.append(("ff", run, i, t))
        return prog + [("final", None, None, None)]

    def _next_norm(self, k: int) -> Optional[torch.Tensor]:
        kind, _, i, _ = self._program[k]
        return {"mix": lambda: self.layers[i].norm1, "ff": lambda: self.layers[i].norm2}.get(kind, lambda: None)()

    def state_specs(self):
        return [self.layers[i].mixer.state_spec for i, _ in self.config.runs()]

    def new_cache(self, n_slots: int, max_len: int) -> SequenceStateCache:
        return SequenceStateCache(self.state_specs(), n_slots, max_len, self.device, self.dtype)

    # ------------------------------------------------------------------ the step
    @torch.no_grad()
    def step(self, step, cache: SequenceStateCache) -> torch.Tensor:
        """Runs the step's tokens from the states in ``cache`` and advances those; fp32 logits ``[wanted, vocab]``."""
        x = (self._run_sandwich if self.config.structure.block == "sandwich" else self._run_parallel)(step, cache)
        h = K.residual_norm(x, None, None, self.final_norm, self.config.eps, self.dtype, rows=step.want_rows)
        logits = K.matmul(h, self.head, torch.float32)
        return logits if self.config.logit_softcap is None else K.softcap(logits, self.config.logit_softcap)

    def _pair_args(self, step, cache) -> dict:
        return {} if self.pair is None else dict(pair=self.pair, step=step, last_token=cache.last_token)

    def _run_parallel(self, step, cache: SequenceStateCache) -> torch.Tensor:
        c, eps, dt, n = self.config, self.config.eps, self.dtype, step.n_tok
        runs = c.runs()
        again = lambda k: k < len(runs) and bool(runs[k][1]) and runs[k][0] == c.loop.start     # a pass but the first starts
        norms = lambda k: (self.layers[runs[k][0]].norm1, self.layers[runs[k][0]].norm2) if k < len(runs) else (None, None)
        pair_of = lambda h: h if isinstance(h, tuple) else (h, None)
        x0 = torch.empty((n, c.width), dtype=torch.float32, device=self.device) if any(map(again, range(len(runs)))) else None
        w1, w2 = norms(0)
        x, *h = K.embed(self.embed, step.token, w1, eps, status=self.status, w_next2=w2, x_copy=x0, **self._pair_args(step, cache))
        h = pair_of(tuple(h) if len(h) > 1 else h[0])
        for k, (i, _) in enumerate(runs):
            layer = self.layers[i]
            cols = layer.w_out.shape[1]
            act = torch.empty((n, (cols + 7) // 8 * 8), dtype=dt, device=self.device)[:, :cols]
            layer.mixer.forward(h[0], step, cache, k, act[:, :layer.cols])
            if layer.ff is not None:
                layer.ff.activate(h[1], act[:, layer.cols:])
            y = K.matmul(act, layer.w_out)
            w1, w2 = norms(k + 1)
            if self.on_layer is not None:
                K.residual_norm(x, y, None, None, eps, dt, x_out=x, want_h=False)
                self.on_layer(k, x)
                y = None
            h = pair_of(K.residual_norm(x, y, None, w1, eps, dt, x_out=x, add=x0 if again(k + 1) else None, w_next2=w2))
        return x

    def _run_sandwich(self, step, cache: SequenceStateCache) -> torch.Tensor:
        c, eps, dt = self.config, self.config.eps, self.dtype
        cat = torch.empty((step.n_tok, 2 * c.width), dtype=dt, device=self.device) if c.loop is not None else None
        x, h = K.embed(self.embed, step.token, self._next_norm(0), eps, cat=cat, cat_both=self._program[0][0] == "enter",
                       status=self.status, **self._pair_args(step, cache))
        for k, (kind, run, i, t) in enumerate(self._program[:-1]):
            nxt = self._next_norm(k + 1)
            if kind == "enter":
                y = K.matmul(cat, self.loop_in, torch.float32)
                h = K.residual_norm(self.loop_step[t], y, None, nxt, eps, dt, x_out=x, broadcast=True)
                continue
            layer = self.layers[i]
            if kind == "mix":
                branch, wb = dict(y=K.matmul(layer.mixer.forward(h, step, cache, run), layer.mixer.w_o)), layer.norm1b
            else:
                branch, wb = layer.ff.branch(h), layer.norm2b
            left = cat if self._program[k + 1][0] == "enter" else None
            h = K.residual_norm(x, branch.pop("y"), wb, nxt, eps, dt, x_out=x, cat=left, **branch)
            if self.on_layer is not None and self._program[k + 1][1] != run:
                self.on_layer(run, x)
        return x

    def run(self, entries, cache: SequenceStateCache) -> torch.Tensor:
        """``entries`` = (sequence, tokens, wanted places): one step, states advanced."""
        step = PackedStep(entries, cache, self.config.windows)
        logits = self.step(step, cache)
        step.commit(cache)
        return logits

    # ------------------------------------------------------------------ the call of the interleave loop
    @torch.no_grad()
    def forward(self, input_ids=None, attention_mask=None, position_ids=None, past_key_values=None, doc_ids=None,
                use_cache=True, logits_to_keep: int = 1, **unused):
        """``MSAForCausalLM.forward``'s call on a batch of rows: row b continues sequence b of ``past_key_values`` (a
        ``SequenceStateCache``) with its unmasked tokens; returns the logits of the last ``logits_to_keep`` columns
        (masked columns: zeros).  Positions follow from the sequence; ``doc_ids`` has no meaning here."""
        bsz, width = input_ids.shape
        mask = torch.ones_like(input_ids) if attention_mask is None else attention_mask[:, -width:]
        ids, mask = input_ids.tolist(), mask.bool().tolist()
        keep = logits_to_keep or width
        entries, places = [], []
        for b in range(bsz):
            cols = [j for j in range(width) if mask[b][j]]
            if not cols:
                continue
            if b not in past_key_values:
                past_key_values.acquire(b)
            want = [n for n, j in enumerate(cols) if j >= width - keep]
            entries.append((b, [ids[b][j] for j in cols], want))
            places += [(b, cols[n] - (width - keep)) for n in want]
        logits = torch.zeros((bsz, keep, self.config.vocab), dtype=torch.float32, device=self.device)
        if entries:
            got = self.run(entries, past_key_values)
            if places:
                b, j = zip(*places)
                logits[list(b), list(j)] = got
        return SimpleNamespace(logits=logits, past_key_values=past_key_values if use_cache else None)

    __call__ = forward

    def check_status(self) -> None:
        """Raises if a step met token ids outside the vocabulary or a kernel gave up waiting."""
        st = self.status.tolist()
        if st[0] or st[2]:
            self.status.zero_()
            raise RuntimeError(f"kernel status {st}: wait code {st[0]}, {st[2]} token ids outside the vocabulary")


class GraphedDecode:
    """Decode steps of up to ``n`` sequences as one CUDA graph.  ``run`` feeds tokens from the host (missing rows work in
    the cache's scratch slot), ``replay`` continues all ``n`` on the device with what the last step chose (greedy)."""

    def __init__(self, model: HybridForCausalLM, cache: SequenceStateCache, n: int, pool=None):
        self.model, self.cache, self.n = model, cache, n
        self.tables = DecodeStep(n, cache, model.config.windows)
        self.graph = torch.cuda.CUDAGraph()
        side = torch.cuda.Stream(model.device)
        side.wait_stream(torch.cuda.current_stream(model.device))

        def body():
            logits = model.step(self.tables, cache)
            return logits, logits.argmax(dim=-1).to(torch.int32)
        self.tables.fill([0] * n, [0] * n, [cache.scratch] * n)
        with torch.cuda.stream(side):
            for _ in range(2):
                body()
        torch.cuda.current_stream(model.device).wait_stream(side)
        with torch.cuda.graph(self.graph, pool=pool):
            self.logits, self.next = body()

    def run(self, tokens, positions, slots) -> torch.Tensor:
        k = self.n - len(tokens)
        self.tables.fill(list(tokens) + [0] * k, list(positions) + [0] * k, list(slots) + [self.cache.scratch] * k)
        self.graph.replay()
        return self.logits[:len(tokens)]

    def replay(self) -> torch.Tensor:
        self.tables.token.copy_(self.next)
        self.tables.pos.add_(1)
        self.graph.replay()
        return self.next
