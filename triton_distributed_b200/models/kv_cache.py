"""KV caches: dense per-sequence (``KV_Cache``, as python/triton_dist/models/kv_cache.py:29-66) and paged
(``PagedKVCache``, as mega_triton_kernel/models/paged_kv_cache.py:28-58).  Both expose the paged view the attention
kernels take: ``layer(i) -> (k, v) [pages, page_size, Hkv, D]`` plus an int32 ``block_table [B, max_pages]``.
Offsets live on the device so a CUDA graph of one decode step can be replayed while they advance."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from ..ops.attention import decode_workspace, pick_kv_splits
from ..ops.gla import gla_chunk_tables


class KV_Cache:
    def __init__(self, num_layers: int, batch_size: int, max_length: int, kv_heads: int, head_dim: int,
                 dtype: torch.dtype = torch.bfloat16, device=None, world_size: int = 1):
        self.num_layers, self.batch_size, self.max_length = num_layers, batch_size, max_length
        self.kv_heads, self.head_dim = kv_heads, head_dim
        dev = device or "cuda"
        self.k_cache = torch.zeros(num_layers, batch_size, max_length, kv_heads, head_dim, dtype=dtype, device=dev)
        self.v_cache = torch.zeros_like(self.k_cache)
        self.kv_offset = torch.zeros(batch_size, dtype=torch.int32, device=dev)
        self.block_table = torch.arange(batch_size, dtype=torch.int32, device=dev).unsqueeze(1).contiguous()
        self._row_base = (torch.arange(batch_size, dtype=torch.int64, device=dev) * max_length)
        self._ws = None
        self.kv_splits = pick_kv_splits(batch_size, kv_heads, 1, max_length)

    # -- views used by the attention layer --------------------------------------------------------------------
    def layer(self, i: int) -> Tuple[torch.Tensor, torch.Tensor]:
        return self.k_cache[i], self.v_cache[i]

    def slots_for(self, position_ids: torch.Tensor, bsz: int, q_len: int) -> torch.Tensor:
        """Flat cache row of every token: ``b * max_length + position``."""
        return (self._row_base[:bsz, None] + position_ids.reshape(bsz, q_len).to(torch.int64)).reshape(-1)

    def kv_lens_after(self, q_len: int, bsz: int) -> torch.Tensor:
        return (self.kv_offset[:bsz] + q_len).to(torch.int32)

    def cu_seqlens(self, bsz: int, q_len: int) -> torch.Tensor:
        return torch.arange(0, (bsz + 1) * q_len, q_len, dtype=torch.int32, device=self.kv_offset.device)

    def decode_workspace(self, num_q_heads: int, head_dim: int) -> torch.Tensor:
        need = self.batch_size * num_q_heads * self.kv_splits * (head_dim + 1)
        if self._ws is None or self._ws.numel() < need:
            self._ws = decode_workspace(self.batch_size, num_q_heads, head_dim, self.kv_splits, self.kv_offset.device)
        return self._ws

    # -- per-step values shared by all layers (computed once instead of once per layer) ----------------------
    def begin_step(self, position_ids: torch.Tensor, bsz: int, q_len: int):
        self._step = (self.slots_for(position_ids, bsz, q_len), self.kv_lens_after(q_len, bsz), bsz, q_len)

    def end_step(self):
        self._step = None

    def step_values(self, position_ids: torch.Tensor, bsz: int, q_len: int):
        """(cache rows of the new tokens, kv lengths after the step): the values of ``begin_step`` when a step is
        open for the same shape, else computed here."""
        st = getattr(self, "_step", None)
        if st is not None and st[2] == bsz and st[3] == q_len:
            return st[0], st[1]
        return self.slots_for(position_ids, bsz, q_len), self.kv_lens_after(q_len, bsz)

    # -- bookkeeping ------------------------------------------------------------------------------------------
    def inc_offset(self, n: int = 1):
        self.kv_offset += n

    def clear(self):
        self.kv_offset.zero_()

    def rand_fill(self, length: int):
        """Pretend ``length`` tokens are cached (random contents): used by decode benchmarks."""
        self.k_cache[:, :, :length].normal_()
        self.v_cache[:, :, :length].normal_()
        self.kv_offset.fill_(length)


class PagedKVCache:
    """Pages of ``page_size`` tokens with a (random by default) block table, same interface as ``KV_Cache``."""

    def __init__(self, num_layers: int, batch_size: int, max_length: int, kv_heads: int, head_dim: int,
                 page_size: int = 16, dtype: torch.dtype = torch.bfloat16, device=None, shuffle: bool = True):
        dev = device or "cuda"
        self.num_layers, self.batch_size, self.max_length = num_layers, batch_size, max_length
        self.kv_heads, self.head_dim, self.page_size = kv_heads, head_dim, page_size
        self.pages_per_seq = (max_length + page_size - 1) // page_size
        n_pages = batch_size * self.pages_per_seq
        self.k_cache = torch.zeros(num_layers, n_pages, page_size, kv_heads, head_dim, dtype=dtype, device=dev)
        self.v_cache = torch.zeros_like(self.k_cache)
        order = torch.randperm(n_pages, device=dev) if shuffle else torch.arange(n_pages, device=dev)
        self.block_table = order.to(torch.int32).reshape(batch_size, self.pages_per_seq).contiguous()
        self.kv_offset = torch.zeros(batch_size, dtype=torch.int32, device=dev)
        self._ws = None
        self.kv_splits = pick_kv_splits(batch_size, kv_heads, 1, max_length)

    def layer(self, i: int):
        return self.k_cache[i], self.v_cache[i]

    def slots_for(self, position_ids: torch.Tensor, bsz: int, q_len: int) -> torch.Tensor:
        pos = position_ids.reshape(bsz, q_len).to(torch.int64)
        page = torch.gather(self.block_table[:bsz].to(torch.int64), 1, pos // self.page_size)
        return (page * self.page_size + pos % self.page_size).reshape(-1)

    kv_lens_after = KV_Cache.kv_lens_after
    cu_seqlens = KV_Cache.cu_seqlens
    decode_workspace = KV_Cache.decode_workspace
    inc_offset = KV_Cache.inc_offset
    clear = KV_Cache.clear
    begin_step = KV_Cache.begin_step
    end_step = KV_Cache.end_step
    step_values = KV_Cache.step_values

    def rand_fill(self, length: int):
        self.k_cache.normal_()
        self.v_cache.normal_()
        self.kv_offset.fill_(length)


# ------------------------------------------------------------------ layered decoders: per-layer storage, packed steps
@dataclass(frozen=True)
class TiedKVSpec:
    """A layer that caches raw keys (which are also its values) and one fp32 factor per token.  ``block`` > 0: attention is
    local to blocks of that many positions, so a sequence keeps ``block`` rows, position p at row ``p % block``."""
    kv_heads: int
    head_dim: int
    block: int = 0

    def rows(self, max_length: int) -> int:
        return min(self.block, max_length) if self.block > 0 else max_length


@dataclass(frozen=True)
class StateSpec:
    """A recurrent layer: fp32 state [heads, dk, dv] per sequence."""
    heads: int
    dk: int
    dv: int


@dataclass(frozen=True)
class LatentSpec:
    """A layer that caches one row per token, shared by all heads: ``rank`` elements of a latent and ``rot`` of a rotated key
    part."""
    rank: int
    rot: int


@dataclass(frozen=True)
class KVSpec:
    """A layer that caches a key and a value per token and KV head, both of ``head_dim`` elements."""
    kv_heads: int
    head_dim: int


@dataclass(frozen=True)
class WindowKVSpec:
    """A layer that caches a key of ``key_dim`` and a value of ``value_dim`` elements per token and KV head.  ``window`` > 0: position i sees
    the positions j with i - j < window, so a sequence keeps ``window`` rows, position p at row ``p % window``."""
    kv_heads: int
    key_dim: int
    value_dim: int
    window: int = 0

    def rows(self, max_length: int) -> int:
        return min(self.window, max_length) if self.window > 0 else max_length


@dataclass(frozen=True)
class DeltaSpec:
    """A recurrent layer behind short convolutions: fp32 state [heads, dk, dv] and the convolutions' last inputs, a ring of ``taps``
    rows (position p at row ``p % taps``) of ``channels`` elements."""
    heads: int
    dk: int
    dv: int
    channels: int
    taps: int


@dataclass(frozen=True)
class GroupSpec:
    """A layer of several mixers side by side, each with its own storage under its own names."""
    parts: tuple


@dataclass(frozen=True)
class SharedSpec:
    """A layer without storage of its own: it reads that of layer ``source``."""
    source: int


@dataclass
class KVPlan:
    """What layers with a key and a value per token need to know about a step (see ``StepPlan.kv``): a sequence's rows are one page of
    ``max_length`` rows, the page of its slot."""
    home_rows: torch.Tensor                         # int64 [T] cache row of every token
    row0: torch.Tensor                              # int64 [T] cache row of the sequence's first token
    n_keys: torch.Tensor                            # int32 [T]
    kv_lens: torch.Tensor                           # int32 [sequences]
    block_table: torch.Tensor                       # int32 [sequences, 1]
    q_pos0: Optional[torch.Tensor] = None           # int32 [sequences] (prompts)
    max_q: int = 1
    max_kv: int = 0                                 # longest sequence after the step (prompts)


class WindowPlan:
    """What a layer with a window needs to know about a step (see ``StepPlan.window``); ``rows`` is the length of its rings.  A decode step
    reads the rings; a prompt reads packed rows: per sequence, what the ring held of earlier steps and is still visible, then the
    new tokens."""

    def __init__(self, plan: "StepPlan", window: int, rows: int):
        self.plan, self.window, self.rows = plan, window, rows
        self._visible = None
        base = plan.slots.to(torch.int64) * rows
        if plan.decode:
            self.row0 = base
            self.home_rows = base + plan.positions % rows            # int64 [T] cache row of every token, -1 = not kept after the step
            return
        slots, starts, lens = plan.host
        home, packed, src, dst, shift, at = [], [], [], [], [], 0
        for slot, start, n in zip(slots, starts, lens):
            first = max(0, start - window + 1) if window > 0 else 0  # oldest position that the step still sees
            p = torch.arange(start, start + n)
            home.append(torch.where(p >= start + n - rows, p % rows + slot * rows, -1))
            packed.append(p - first + at)
            if start > first:
                old = torch.arange(first, start)
                src.append(old % rows + slot * rows)
                dst.append(old - first + at)
            shift.append(at - first)
            at += start + n - first
        dev, T, N = plan.slots.device, plan.num_tokens, len(lens)
        nc = sum(int(t.numel()) for t in src)
        big = torch.cat(home + packed + src + dst).to(torch.int64).to(dev)
        small = torch.tensor(list(starts) + shift, dtype=torch.int32).to(dev)
        self.home_rows, self.packed_rows = big[:T], big[T:2 * T]      # packed_rows int64 [T]
        self.carry_src = big[2 * T:2 * T + nc] if nc else None        # cache rows of earlier steps ...
        self.carry_dst = big[2 * T + nc:] if nc else None             # ... and their packed rows
        self.q_pos0, self.shift = small[:N], small[N:]                # int32 [sequences]; position p is packed row p + shift
        self.total, self.max_q = at, max(lens)

    def visible(self):
        """Per token: first row it sees (int64; cache rows in a decode step, else packed rows), number of rows, and its own row among
        them (int32)."""
        if self._visible is None:
            pos = self.plan.positions
            if self.plan.decode:
                n = (pos + 1).clamp(max=self.rows)
                self._visible = (self.row0, n.to(torch.int32), (pos % self.rows).to(torch.int32))
            else:
                n = (pos + 1).clamp(max=self.window) if self.window > 0 else pos + 1
                self._visible = (self.packed_rows - n + 1, n.to(torch.int32), (n - 1).to(torch.int32))
        return self._visible


@dataclass
class LatentPlan:
    """What the latent-attention layers need to know about a step (see ``StepPlan.latent``)."""
    home_rows: torch.Tensor                         # int64 [T] cache row of every token (slot * max_length + position)
    row0: torch.Tensor                              # int64 [T] cache row of the sequence's first token
    n_keys: torch.Tensor                            # int32 [T]
    kv_lens: torch.Tensor                           # int32 [sequences]
    # prompts only: the visible rows of all sequences packed one after the other, each start a multiple of 64
    ctx_len: int = 0
    ctx_rows: Optional[torch.Tensor] = None         # int64 [T] packed row of every token
    ctx0: Optional[torch.Tensor] = None             # int32 [sequences]
    q_pos0: Optional[torch.Tensor] = None           # int32 [sequences]
    max_q: int = 0
    carry_src: Optional[torch.Tensor] = None        # cache rows of earlier steps ...
    carry_dst: Optional[torch.Tensor] = None        # ... and their packed rows


@dataclass
class BlockPlan:
    """What a tied-KV layer needs to know about a step (see ``StepPlan.blocks``); ``rows`` is the page size of its cache."""
    home_rows: torch.Tensor                         # int64 [T] cache row of every token, -1 = not kept after the step
    block_table: torch.Tensor                       # int32 [virtual sequences, 1]
    row0: torch.Tensor                              # int64 [T] first visible row of every token (of the page pool used)
    n_keys: torch.Tensor                            # int32 [T]
    kv_lens: torch.Tensor                           # int32 [virtual sequences]
    # prompts only: every (sequence, block) pair is a virtual sequence of its own with a page of a scratch pool
    scratch_rows: Optional[torch.Tensor] = None     # int64 [T]
    cu: Optional[torch.Tensor] = None               # int32 [virtual sequences + 1]
    q_pos0: Optional[torch.Tensor] = None           # int32 [virtual sequences] position of the first query in its block
    pages: int = 0
    page_rows: int = 0
    max_q: int = 0
    max_kv: int = 0
    carry_src: Optional[torch.Tensor] = None        # cache rows of earlier steps that a continued block still needs ...
    carry_dst: Optional[torch.Tensor] = None        # ... and where they go in the scratch pool


class StepPlan:
    """The tokens of one step, packed sequence after sequence.  Built by the cache; the per-layer tables are derived once
    per distinct block size.  A decode plan (one token per sequence) is made of device tensors only, so it can be captured
    in a CUDA graph."""

    def __init__(self, cache: "HybridCache", slots: torch.Tensor, positions: torch.Tensor, pos0: torch.Tensor,
                 host: Optional[Tuple[List[int], List[int], List[int]]] = None):
        self.cache, self.slots, self.positions, self.pos0, self.host = cache, slots, positions, pos0, host
        self.num_seqs, self.num_tokens = slots.numel(), positions.numel()
        self.decode = host is None
        self.cu = None
        self._blocks: Dict[int, BlockPlan] = {}
        self._chunks = None
        self._latent: Optional[LatentPlan] = None
        self._kv: Optional[KVPlan] = None
        self._windows: Dict[int, WindowPlan] = {}
        self.contexts: Dict[int, torch.Tensor] = {}  # packed rows of the layers that later layers of the step read as well
        if not self.decode:
            cu = [0]
            for n in host[2]:
                cu.append(cu[-1] + n)
            self.cu_host = cu
            self.cu = torch.tensor(cu, dtype=torch.int32).to(slots.device)
            self.last_rows = torch.tensor([c - 1 for c in cu[1:]], dtype=torch.int64).to(slots.device)

    def chunk_tables(self):
        """Chunks of the recurrent layers' kernels (None for a decode step)."""
        if self._chunks is None and not self.decode:
            self._chunks = gla_chunk_tables(self.cu_host, self.slots.device)
        return self._chunks

    def kv(self) -> KVPlan:
        if self._kv is None:
            M = self.cache.max_length
            pages = self.slots.unsqueeze(1).contiguous()
            n = (self.positions + 1).to(torch.int32)
            if self.decode:
                row0 = self.slots.to(torch.int64) * M
                self._kv = KVPlan(row0 + self.positions, row0, n, n, pages)
            else:
                slots, starts, lens = self.host
                row0 = torch.cat([torch.full((k,), s * M, dtype=torch.int64) for s, k in zip(slots, lens)]).to(self.slots.device)
                ends = [a + k for a, k in zip(starts, lens)]
                small = torch.tensor(ends + list(starts), dtype=torch.int32).to(self.slots.device)
                self._kv = KVPlan(row0 + self.positions, row0, n, small[:len(lens)], pages, small[len(lens):], max(lens), max(ends))
        return self._kv

    def window(self, spec: WindowKVSpec) -> WindowPlan:
        if spec.window not in self._windows:
            self._windows[spec.window] = WindowPlan(self, spec.window, spec.rows(self.cache.max_length))
        return self._windows[spec.window]

    def latent(self) -> LatentPlan:
        if self._latent is None:
            self._latent = self._decode_latent() if self.decode else self._prompt_latent()
        return self._latent

    def _decode_latent(self) -> LatentPlan:
        row0 = self.slots.to(torch.int64) * self.cache.max_length
        n = (self.positions + 1).to(torch.int32)
        return LatentPlan(home_rows=row0 + self.positions, row0=row0, n_keys=n, kv_lens=n)

    def _prompt_latent(self) -> LatentPlan:
        slots, starts, lens = self.host
        M, at = self.cache.max_length, 0
        home, row0, ctx_rows, src, dst, ctx0 = [], [], [], [], [], []
        for slot, start, n in zip(slots, starts, lens):
            r = torch.arange(start, start + n)
            home.append(r + slot * M)
            row0.append(torch.full((n,), slot * M))
            ctx_rows.append(r + at)
            if start > 0:
                src.append(torch.arange(start) + slot * M)
                dst.append(torch.arange(start) + at)
            ctx0.append(at)
            at += (start + n + 63) // 64 * 64
        T, N = self.num_tokens, len(lens)
        nc = sum(starts)
        big = torch.cat(home + row0 + ctx_rows + src + dst).to(torch.int64).to(self.slots.device)
        small = torch.tensor([a + n for a, n in zip(starts, lens)] + ctx0 + list(starts), dtype=torch.int32).to(self.slots.device)
        return LatentPlan(home_rows=big[:T], row0=big[T:2 * T], ctx_rows=big[2 * T:3 * T], n_keys=(self.positions + 1).to(torch.int32),
                          carry_src=big[3 * T:3 * T + nc] if nc else None, carry_dst=big[3 * T + nc:] if nc else None,
                          kv_lens=small[:N], ctx0=small[N:2 * N], q_pos0=small[2 * N:], ctx_len=at, max_q=max(lens))

    def blocks(self, spec: TiedKVSpec) -> BlockPlan:
        rows = spec.rows(self.cache.max_length)
        if rows not in self._blocks:
            self._blocks[rows] = self._decode_blocks(rows) if self.decode else self._prompt_blocks(rows)
        return self._blocks[rows]

    def _decode_blocks(self, rows: int) -> BlockPlan:
        base = self.slots.to(torch.int64) * rows
        off = self.positions % rows
        return BlockPlan(home_rows=base + off, block_table=self.slots.unsqueeze(1).contiguous(), row0=base,
                         n_keys=(off + 1).to(torch.int32), kv_lens=(self.positions + 1).to(torch.int32))

    def _prompt_blocks(self, rows: int) -> BlockPlan:
        slots, starts, lens = self.host
        virt = []                                    # (first token, tokens, position inside the block, slot or -1 = not last)
        tok = 0
        for slot, start, n in zip(slots, starts, lens):
            at, left = start, n
            while left > 0:
                take = min(left, rows - at % rows)
                virt.append((tok, take, at % rows, slot, left == take))
                tok, at, left = tok + take, at + take, left - take
        max_kv = max(off + n for _, n, off, _, _ in virt)
        page_rows = min(rows, (max_kv + 7) // 8 * 8)
        home, scratch, row0, keys = [], [], [], []
        src, dst = [], []
        for i, (_, n, off, slot, last) in enumerate(virt):
            r = torch.arange(off, off + n)
            home.append(r + slot * rows if last else torch.full((n,), -1))
            scratch.append(r + i * page_rows)
            row0.append(torch.full((n,), i * page_rows))
            keys.append(r + 1)
            if off > 0:                              # the block began in an earlier step
                src.append(torch.arange(off) + slot * rows)
                dst.append(torch.arange(off) + i * page_rows)
        dev = self.slots.device
        T = self.num_tokens
        big = torch.cat([torch.cat(x) for x in (home, scratch, row0)] + src + dst).to(torch.int64).to(dev)
        nv, nc = len(virt), sum(int(x.numel()) for x in src)
        small = torch.tensor([v[0] for v in virt] + [T] + [v[2] for v in virt] + [v[2] + v[1] for v in virt] + list(range(nv)),
                             dtype=torch.int32)
        small = torch.cat([small, torch.cat(keys).to(torch.int32)]).to(dev)
        return BlockPlan(home_rows=big[:T], scratch_rows=big[T:2 * T], row0=big[2 * T:3 * T],
                         carry_src=big[3 * T:3 * T + nc] if nc else None, carry_dst=big[3 * T + nc:] if nc else None,
                         cu=small[:nv + 1], q_pos0=small[nv + 1:2 * nv + 1], kv_lens=small[2 * nv + 1:3 * nv + 1],
                         block_table=small[3 * nv + 1:4 * nv + 1].unsqueeze(1), n_keys=small[4 * nv + 1:], pages=nv,
                         page_rows=page_rows, max_q=max(v[1] for v in virt), max_kv=max_kv)


class HybridCache:
    """Cache of a layered decoder: one storage per layer run (``KVSpec``, ``WindowKVSpec``, ``TiedKVSpec``, ``LatentSpec``, ``StateSpec``, ``DeltaSpec``, or a
    ``GroupSpec`` of several; ``SharedSpec`` layers share another layer's), indexed by a sequence's slot.

    Slots are handed out by ``alloc`` and given back by ``free``; nothing is cleared in between, because a sequence that
    starts at position 0 neither reads its state row nor any row it has not written.  ``kv_offset`` (device) and ``lens``
    (host) count the tokens each slot holds; a step's plan starts there.  The first ``batch_size`` slots are allocated at
    construction, which is what :class:`Engine` uses for a rectangular batch."""

    def __init__(self, specs: Sequence, batch_size: int, max_length: int, dtype: torch.dtype = torch.bfloat16, device=None,
                 allocate: bool = True):
        self.specs, self.batch_size, self.max_length, self.dtype = list(specs), batch_size, max_length, dtype
        self.device = device or "cuda"
        self.capacity = 0
        self.layers: List[dict] = [{} for _ in self.specs]
        self.kv_offset = torch.zeros(0, dtype=torch.int32, device=self.device)
        self.lens: List[int] = []
        self._free: List[int] = []
        self._grow(max(1, batch_size))
        if allocate:
            for _ in range(batch_size):
                self.alloc()
        self.batch_slots = torch.arange(batch_size, dtype=torch.int32, device=self.device)

    # -- slots ------------------------------------------------------------------------------------------------
    def _grow(self, capacity: int):
        def widen(t, *shape, dtype):
            new = torch.zeros(capacity, *shape, dtype=dtype, device=self.device)
            if t is not None:
                new[:self.capacity] = t
            return new

        for i, (spec, st) in enumerate(zip(self.specs, self.layers)):
            if isinstance(spec, SharedSpec):
                if not 0 <= spec.source < i or isinstance(self.specs[spec.source], SharedSpec):
                    raise ValueError(f"layer {i} cannot share the cache of layer {spec.source}")
                self.layers[i] = self.layers[spec.source]
                continue
            parts = spec.parts if isinstance(spec, GroupSpec) else (spec,)
            names = [n for s in parts for n in self._tensors(s)]
            if len(set(names)) != len(names):
                raise ValueError(f"layer {i}: mixers side by side need storage of different names")
            for s in parts:
                for name, (shape, dtype) in self._tensors(s).items():
                    st[name] = widen(st.get(name), *shape, dtype=dtype)
        self.kv_offset = widen(self.kv_offset, dtype=torch.int32)
        self._free = list(range(capacity - 1, self.capacity - 1, -1)) + self._free
        self.lens += [0] * (capacity - self.capacity)
        self.capacity = capacity

    def _tensors(self, spec) -> Dict[str, tuple]:
        """Storage of one slot: name -> (shape, dtype)."""
        M, act = self.max_length, self.dtype
        if isinstance(spec, LatentSpec):
            return {"latent": ((M, spec.rank + spec.rot), act)}
        if isinstance(spec, TiedKVSpec):
            rows = spec.rows(M)
            return {"k": ((rows, spec.kv_heads, spec.head_dim), act), "scale": ((rows,), torch.float32)}
        if isinstance(spec, KVSpec):
            return {n: ((M, spec.kv_heads, spec.head_dim), act) for n in ("k", "v")}
        if isinstance(spec, WindowKVSpec):
            rows = spec.rows(M)
            return {"k": ((rows, spec.kv_heads, spec.key_dim), act), "v": ((rows, spec.kv_heads, spec.value_dim), act)}
        state = {"state": ((spec.heads, spec.dk, spec.dv), torch.float32)}
        return {**state, "conv": ((spec.taps, spec.channels), act)} if isinstance(spec, DeltaSpec) else state

    def alloc(self) -> int:
        """A slot for a new sequence (the storage doubles when none is free; captured graphs do not survive that)."""
        if not self._free:
            self._grow(2 * self.capacity)
        slot = self._free.pop()
        self._set_len(slot, 0)
        return slot

    def free(self, slot: int):
        if slot in self._free or not 0 <= slot < self.capacity:
            raise ValueError(f"slot {slot} is not in use")
        self._free.append(slot)

    def _set_len(self, slot: int, n: int):
        self.lens[slot] = n
        self.kv_offset[slot] = n

    # -- step plans -------------------------------------------------------------------------------------------
    def plan(self, slots: Sequence[int], lens: Sequence[int]) -> StepPlan:
        """A step that brings ``lens[i]`` new tokens of the sequence in ``slots[i]``.  Raises ``ValueError`` when a sequence
        would outgrow ``max_length``."""
        slots, lens = list(slots), list(lens)
        if not slots or len(slots) != len(lens) or min(lens) < 1 or len(set(slots)) != len(slots):
            raise ValueError("a step needs distinct sequences with at least one token each")
        starts = [self.lens[s] for s in slots]
        for s, a, n in zip(slots, starts, lens):
            if a + n > self.max_length:
                raise ValueError(f"sequence of {a + n} tokens exceeds max_length ({self.max_length})")
        dev_slots = torch.tensor(slots, dtype=torch.int32).to(self.device)
        pos0 = torch.tensor(starts, dtype=torch.int64).to(self.device)
        if max(lens) == 1:
            return StepPlan(self, dev_slots, pos0, pos0)
        pos = torch.cat([torch.arange(a, a + n) for a, n in zip(starts, lens)]).to(self.device)
        return StepPlan(self, dev_slots, pos, pos0, (slots, starts, lens))

    def decode_plan(self, positions: torch.Tensor) -> StepPlan:
        """One token for each of the first ``len(positions)`` slots; ``positions`` int64 on the device."""
        pos = positions.reshape(-1).to(torch.int64)
        return StepPlan(self, self.batch_slots[:pos.numel()], pos, pos)

    def advance(self, slots: Sequence[int], lens: Sequence[int]):
        """The tokens of a step have been computed."""
        for s, n in zip(slots, lens):
            self.lens[s] += n
        idx = torch.tensor(list(slots), dtype=torch.int64).to(self.device)
        self.kv_offset[idx] += torch.tensor(list(lens), dtype=torch.int32).to(self.device)

    # -- the rectangular-batch interface of the engine ----------------------------------------------------------
    def inc_offset(self, n=1):
        """Advance the engine's batch by ``n`` tokens (one number, or one per sequence)."""
        per = [n] * self.batch_size if isinstance(n, int) else list(n)
        for s, k in enumerate(per):
            self.lens[s] += k
        if isinstance(n, int):
            self.kv_offset[:self.batch_size] += n
        else:
            self.kv_offset[:self.batch_size] += torch.tensor(per, dtype=torch.int32).to(self.device)

    def clear(self):
        self.kv_offset.zero_()
        self.lens = [0] * self.capacity

    def snapshot(self):
        """Copies of what a decode step changes besides the rows it writes (recurrent states): a step run for warm-up must
        not count.  (Writing a row again, of a ring as well, writes the same values.)"""
        return [st["state"].clone() if "state" in st else None for st in self.layers]

    def restore(self, snap):
        for st, old in zip(self.layers, snap):
            if old is not None:
                st["state"].copy_(old)

    def rand_fill(self, length: int):
        """Pretend ``length`` tokens are cached (random contents): used by decode benchmarks."""
        for st in self.layers:
            for name, t in st.items():
                if name == "scale":
                    t.fill_(1.0)
                else:
                    t.normal_()
        self.kv_offset.fill_(length)
        self.lens = [length] * self.capacity
