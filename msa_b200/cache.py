"""The cache object the attention layer talks to (mirror of ``CustomDynamicCache``,
src/utils/cache.py:14-137, and of its CPU-offloading subclass :139-172).

Only the protocol the path uses is kept -- per-layer ``cache_kwargs``, ``meta``, ``record_kwargs``
(merge), ``update``, ``update_router_kcache``, ``get_kvcache``, ``get_router_kcache``,
``clear_kvcache`` -- implemented on plain dictionaries instead of HF ``DynamicCache`` internals
(which changed between transformers releases)."""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import torch


class SparseCache:
    def __init__(self):
        self.cache_kwargs = {}
        self.meta = {}
        self.key_cache = {}
        self.value_cache = {}
        self.router_key_cache = {}

    def record_kwargs(self, layer_idx, kwargs):
        if layer_idx in self.cache_kwargs:
            self.cache_kwargs[layer_idx].update(kwargs)
        else:
            self.cache_kwargs[layer_idx] = dict(kwargs)

    def get_layer_length(self):
        return len(self.cache_kwargs)

    def update(self, key_states, value_states, layer_idx, cache_kwargs=None):
        self.key_cache[layer_idx], self.value_cache[layer_idx] = key_states, value_states
        return key_states, value_states

    def update_router_kcache(self, key_states, layer_idx):
        self.router_key_cache[layer_idx] = key_states
        return key_states

    def get_kvcache(self, layer_idx):
        return self.key_cache[layer_idx], self.value_cache[layer_idx]

    def get_router_kcache(self, layer_idx):
        return self.router_key_cache.get(layer_idx)

    def clear_kvcache(self):
        self.key_cache, self.value_cache = {}, {}


class SparseCacheOnCPU(SparseCache):
    """Moves everything it is handed to host memory, as the stage-1 worker's cache does."""

    @staticmethod
    def _cpu(t):
        return t.cpu() if torch.is_tensor(t) and t.is_cuda else t

    def record_kwargs(self, layer_idx, kwargs):
        super().record_kwargs(layer_idx, {k: (self._cpu(v) if torch.is_tensor(v) and v.is_cuda else
                                              (v.clone() if torch.is_tensor(v) else v)) for k, v in kwargs.items()})

    def update(self, key_states, value_states, layer_idx, cache_kwargs=None):
        return super().update(self._cpu(key_states), self._cpu(value_states), layer_idx)

    def update_router_kcache(self, key_states, layer_idx):
        return super().update_router_kcache(self._cpu(key_states), layer_idx)


@dataclass(frozen=True)
class RingSpec:
    """A windowed layer's state: the last rows of ``width`` elements (``window`` None: every row) and, where a short
    convolution feeds them, its last ``taps - 1`` inputs over ``channels`` channels."""
    width: int
    window: Optional[int]
    channels: int = 0
    taps: int = 1


@dataclass(frozen=True)
class RecurrentSpec:
    """A recurrent layer's state: a ``[heads, dim, vdim]`` fp32 matrix per head and the last ``taps - 1`` inputs of its
    convolution over ``channels`` channels (double-buffered by the parity of the sequence's position); ``shift``: width of
    the layer's input if the previous token's is kept."""
    heads: int
    dim: int
    vdim: int
    channels: int = 0
    taps: int = 1
    shift: int = 0


class SequenceStateCache(SparseCache):
    """Slots of per-sequence state for models whose layers keep bounded state (rings, recurrent matrices).

    One slot holds a sequence's state in every layer run; ``acquire`` / ``release`` hand slots out and take them back.
    Nothing is cleared: the kernels take a sequence at position 0 as empty and never read a ring row that the sequence
    has not written.  One more slot than asked for exists, ``scratch``: rows that only fill up a step work there.  ``specs`` lists the runs in order (``model.state_specs()``); a ring has
    ``min(window, max_len)`` rows.  ``last_token`` keeps every sequence's previous token (for embeddings that read it).  The protocol of ``SparseCache`` (``meta``, ``record_kwargs``) stays usable, so the
    interleave loop drives a model on this cache unchanged."""

    def __init__(self, specs: Sequence, n_slots: int, max_len: int, device, dtype: torch.dtype):
        super().__init__()
        if n_slots < 1 or max_len < 1:
            raise ValueError("SequenceStateCache needs at least one slot and one position")
        self.specs, self.n_slots, self.max_len, self.device, self.dtype = list(specs), n_slots, max_len, torch.device(device), dtype
        self.scratch, rows_all = n_slots, n_slots + 1
        self.ring: Dict[int, torch.Tensor] = {}
        self.state: Dict[int, torch.Tensor] = {}
        self.conv: Dict[int, torch.Tensor] = {}
        self.shift: Dict[int, torch.Tensor] = {}
        self.last_token = torch.zeros(rows_all, dtype=torch.int32, device=device)
        for i, s in enumerate(self.specs):
            if isinstance(s, RingSpec):
                rows = max_len if s.window is None else min(s.window, max_len)
                self.ring[i] = torch.zeros((rows_all, rows, s.width), dtype=dtype, device=device)
            else:
                self.state[i] = torch.zeros((rows_all, s.heads, s.dim, s.vdim), dtype=torch.float32, device=device)
                if s.shift:
                    self.shift[i] = torch.zeros((rows_all, s.shift), dtype=dtype, device=device)
            if s.channels:
                self.conv[i] = torch.zeros((rows_all, 2, s.taps - 1, s.channels), dtype=dtype, device=device)
        self._free: List[int] = list(range(n_slots - 1, -1, -1))
        self._slot: Dict[Hashable, int] = {}
        self._length: Dict[Hashable, int] = {}

    @property
    def free_slots(self) -> int:
        return len(self._free)

    def __contains__(self, seq: Hashable) -> bool:
        return seq in self._slot

    def acquire(self, seq: Hashable) -> int:
        if seq in self._slot:
            raise KeyError(f"sequence {seq!r} already holds a slot")
        if not self._free:
            raise RuntimeError(f"all {self.n_slots} slots are taken")
        self._slot[seq], self._length[seq] = self._free.pop(), 0
        return self._slot[seq]

    def release(self, seq: Hashable) -> None:
        self._free.append(self._slot.pop(seq))
        del self._length[seq]

    def slot(self, seq: Hashable) -> int:
        return self._slot[seq]

    def length(self, seq: Hashable) -> int:
        return self._length[seq]

    def advance(self, seq: Hashable, n: int) -> None:
        self._length[seq] += n

    def state_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for d in (self.ring, self.state, self.conv, self.shift) for t in d.values())


@dataclass
class ContextView:
    """Context bookkeeping of one step for one attention window: where each portion's context starts (``ctx_off``,
    prefix sums) and how many earlier rows it begins with (``old_off``, prefix sums)."""
    window: int
    ctx_off: Optional[torch.Tensor]
    old_off: Optional[torch.Tensor]
    n_ctx: int
    n_old: int


class PackedStep:
    """The tokens of one step, packed: single-token continuations (decode) first, then the portions.

    ``entries`` = ``(sequence, token ids, wanted places)``; the sequences must hold slots in ``cache``.  ``want_rows``
    lists the packed rows whose logits are asked for, in the order of the entries."""

    def __init__(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]], cache: SequenceStateCache, windows: Sequence[Optional[int]]):
        entries = [(s, list(t), list(w)) for s, t, w in entries]
        if len({s for s, _, _ in entries}) != len(entries):
            raise ValueError("a sequence appears twice in one step")
        for s, t, w in entries:
            if not t:
                raise ValueError(f"sequence {s!r} brings no tokens")
            if cache.length(s) + len(t) > cache.max_len:
                raise ValueError(f"sequence {s!r} would hold {cache.length(s) + len(t)} tokens, the cache has room for {cache.max_len}")
            if any(not 0 <= i < len(t) for i in w):
                raise ValueError(f"sequence {s!r}: a wanted place lies outside its {len(t)} tokens")
        order = sorted(range(len(entries)), key=lambda i: len(entries[i][1]) > 1)      # stable: decode entries first
        token, pos, tok_seq, slot, start, cu, row0 = [], [], [], [], [], [0], {}
        for k, i in enumerate(order):
            s, t, _ = entries[i]
            p0 = cache.length(s)
            row0[i] = len(token)
            token += t
            pos += range(p0, p0 + len(t))
            tok_seq += [k] * len(t)
            slot.append(cache.slot(s))
            start.append(p0)
            cu.append(len(token))
        self.seqs = [(s, len(t)) for s, t, _ in entries]
        self.n_tok, self.n_seq = len(token), len(order)
        self.n_decode = sum(len(t) == 1 for _, t, _ in entries)
        self.max_len = max([len(t) for _, t, _ in entries if len(t) > 1], default=0)
        want = [row0[i] + w for i, (_, _, ws) in enumerate(entries) for w in ws]
        views = []
        for window in windows:
            size = cache.max_len if window is None else min(window, cache.max_len)
            ctx, old = [0], [0]
            for k in range(self.n_decode, self.n_seq):
                o = min(start[k], size - 1)
                old.append(old[-1] + o)
                ctx.append(ctx[-1] + o + cu[k + 1] - cu[k])
            views.append((window, size, ctx, old))
        chunk_off = [0]                       # chunks of 64 tokens of the portions (the recurrent layers walk those)
        for k in range(self.n_decode, self.n_seq):
            chunk_off.append(chunk_off[-1] + (cu[k + 1] - cu[k] + 63) // 64)
        self.n_chunks = chunk_off[-1]
        # one host-to-device copy for all tables
        parts = [token, pos, tok_seq, slot, start, cu, want, chunk_off] + [x for v in views for x in v[2:]]
        flat = torch.tensor([x for p in parts for x in p], dtype=torch.int32)
        if cache.device.type == "cuda":
            flat = flat.pin_memory()
        flat = flat.to(cache.device, non_blocking=True)
        at, dev = 0, []
        for p in parts:
            dev.append(flat[at:at + len(p)])
            at += len(p)
        self.token, self.pos, self.tok_seq, self.slot, self.start, self.cu, self.want_rows, self.chunk_off = dev[:8]
        self.views = {w: ContextView(size, dev[8 + 2 * i], dev[9 + 2 * i], ctx[-1], old[-1])
                      for i, (w, size, ctx, old) in enumerate(views)}

    def commit(self, cache: SequenceStateCache) -> None:
        """The step has been launched: its sequences have grown."""
        for s, n in self.seqs:
            cache.advance(s, n)


class DecodeStep:
    """A step of one token for each of ``n`` sequences with tables that stay at fixed device addresses, so that a CUDA
    graph of the step can be replayed: ``fill`` rewrites them, the sampled tokens may be fed back on the device."""

    def __init__(self, n: int, cache: SequenceStateCache, windows: Sequence[Optional[int]]):
        dev = cache.device
        i = dict(dtype=torch.int32, device=dev)
        self.n_tok = self.n_seq = self.n_decode = n
        self.max_len = self.n_chunks = 0
        self.chunk_off = None
        self.table = torch.zeros((3, n), **i)
        self.token, self.pos, self.slot = self.table[0], self.table[1], self.table[2]
        self.start = self.pos
        self.tok_seq = torch.arange(n, **i)
        self.cu = torch.arange(n + 1, **i)
        self.want_rows = torch.arange(n, **i)
        self.views = {w: ContextView(cache.max_len if w is None else min(w, cache.max_len), None, None, 0, 0) for w in windows}
        self._host = torch.zeros((3, n), dtype=torch.int32)
        self._copied = None
        if dev.type == "cuda":
            self._host, self._copied = self._host.pin_memory(), torch.cuda.Event()

    def fill(self, tokens: Sequence[int], positions: Sequence[int], slots: Sequence[int]) -> None:
        if self._copied is not None:
            self._copied.synchronize()        # the copy of the last fill has left the host buffer
        self._host.copy_(torch.tensor([tokens, positions, slots], dtype=torch.int32))
        self.table.copy_(self._host, non_blocking=True)
        if self._copied is not None:
            self._copied.record()


class SharedPooledCache:
    """One stage-1 block's pooled tensors in a shared-memory file, in the bank's own layouts.

    The reference's stage-1 worker hands its CPU cache object to the service through a ``multiprocessing.Queue``
    (src/prefill.py:124-131), i.e. pickles every pooled tensor and copies it twice.  Here the worker writes, per
    router layer, ``kv [C, 2, Hkv, D]`` (K then V per chunk) and ``rk [C, Hkv, D]`` once into a file under
    ``/dev/shm``; what travels through the queue is this small object (path, shapes, the per-layer ``cache_kwargs``
    with the template prefix and ``pooled_doc_ids``).  The receiver maps the file: ``kv_chunk_major`` / ``rk_chunk_major``
    give the mapped tensors for a straight copy into the bank, ``get_kvcache`` / ``get_router_kcache`` the
    reference-shaped ``[1, Hkv, C, D]`` views of the same bytes.  ``clear_kvcache`` (which the receive loop calls
    per block, src/msa_service.py:569) unmaps and removes the file."""

    def __init__(self, path: str, dtype: torch.dtype, n_kv_heads: int, head_dim: int, layer_chunks: dict, has_rk: dict,
                 cache_kwargs: dict, meta: dict):
        self.path, self.dtype, self.n_kv_heads, self.head_dim = path, dtype, n_kv_heads, head_dim
        self.layer_chunks, self.has_rk = dict(layer_chunks), dict(has_rk)
        self.cache_kwargs, self.meta = cache_kwargs, meta
        self._raw = None

    @staticmethod
    def _layer_bytes(c, h, d, esize, has_rk):
        return c * 2 * h * d * esize, (c * h * d * esize if has_rk else 0)

    @classmethod
    def write(cls, path: str, cache: SparseCache, router_layer_ids):
        """Move the pooled K / V / K_r of ``cache`` (``[1, Hkv, C, D]`` per router layer) into ``path``."""
        first_k = cache.key_cache[router_layer_ids[0]]
        dtype, h, d = first_k.dtype, first_k.shape[1], first_k.shape[3]
        layer_chunks, has_rk = {}, {}
        with open(path, "wb") as f:
            for layer in router_layer_ids:
                k, v = cache.get_kvcache(layer)
                rk = cache.get_router_kcache(layer)
                kv = torch.stack([k[0].permute(1, 0, 2), v[0].permute(1, 0, 2)], dim=1).contiguous().cpu()    # [C, 2, Hkv, D]
                f.write(kv.view(torch.uint8).numpy().tobytes() if kv.numel() else b"")
                if rk is not None:
                    f.write(rk[0].permute(1, 0, 2).contiguous().cpu().view(torch.uint8).numpy().tobytes())
                layer_chunks[layer], has_rk[layer] = int(k.shape[2]), rk is not None
            if f.tell() == 0:
                f.write(b"\0" * 16)
        meta = {k: v for k, v in cache.meta.items() if not str(k).startswith("_msa_b200_")}   # per-process scratch stays behind
        return cls(path, dtype, h, d, layer_chunks, has_rk, cache.cache_kwargs, meta)

    def __getstate__(self):
        state = dict(self.__dict__)
        state["_raw"] = None          # the mapping is per process
        return state

    def _map(self):
        if self._raw is None:
            self._raw = torch.from_file(self.path, shared=True, size=max(os.path.getsize(self.path), 1), dtype=torch.uint8)
        return self._raw

    def _offsets(self, layer_idx):
        esize = torch.empty((), dtype=self.dtype).element_size()
        off = 0
        for layer, c in self.layer_chunks.items():
            n_kv, n_rk = self._layer_bytes(c, self.n_kv_heads, self.head_dim, esize, self.has_rk[layer])
            if layer == layer_idx:
                return off, n_kv, n_rk, c
            off += n_kv + n_rk
        raise KeyError(layer_idx)

    def kv_chunk_major(self, layer_idx):
        off, n_kv, _, c = self._offsets(layer_idx)
        return self._map()[off:off + n_kv].view(self.dtype).view(c, 2, self.n_kv_heads, self.head_dim)

    def rk_chunk_major(self, layer_idx):
        off, n_kv, n_rk, c = self._offsets(layer_idx)
        if not n_rk:
            return None
        return self._map()[off + n_kv:off + n_kv + n_rk].view(self.dtype).view(c, self.n_kv_heads, self.head_dim)

    def get_kvcache(self, layer_idx):
        kv = self.kv_chunk_major(layer_idx)
        return kv[:, 0].permute(1, 0, 2).unsqueeze(0), kv[:, 1].permute(1, 0, 2).unsqueeze(0)

    def get_router_kcache(self, layer_idx):
        rk = self.rk_chunk_major(layer_idx)
        return None if rk is None else rk.permute(1, 0, 2).unsqueeze(0)

    def record_kwargs(self, layer_idx, kwargs):
        self.cache_kwargs.setdefault(layer_idx, {}).update(kwargs)

    def clear_kvcache(self):
        self._raw = None
        if os.path.exists(self.path):
            os.unlink(self.path)


def create_cache():
    return SparseCache()
