"""Device-resident paged KV pool and per-sequence block tables.

One allocation holds every layer's K and V blocks: [layers, 2, blocks, kv_heads_local, block_size, head_dim]
(sized for the 180 GB of a B200 up front instead of the reference's doubling growth,
candle-llm/src/primitives/paged_kv_cache.rs:101-140). Block ids are handed out by the refcounted
allocator policy (copy-on-write prefix sharing), so a block id is valid across all layers.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from ..policy.paging import BlockAllocator


class PagedKvPool:
    def __init__(self, num_layers: int, num_blocks: int, kv_heads: int, head_dim: int, block_size: int = 16,
                 device: torch.device | str = "cuda", dtype: torch.dtype = torch.bfloat16):
        self.num_layers, self.num_blocks, self.block_size = num_layers, num_blocks, block_size
        self.kv_heads, self.head_dim = kv_heads, head_dim
        self.data = torch.zeros((num_layers, 2, num_blocks, kv_heads, block_size, head_dim), dtype=dtype,
                                device=device)
        self.allocator = BlockAllocator(num_blocks)

    @property
    def bytes(self) -> int:
        return self.data.numel() * self.data.element_size()

    def copy_block(self, src: int, dst: int) -> None:
        """Copy-on-write: duplicate one block across all layers (K and V)."""
        self.data[:, :, dst].copy_(self.data[:, :, src])

    @staticmethod
    def blocks_for_budget(bytes_budget: int, num_layers: int, kv_heads: int, head_dim: int, block_size: int = 16,
                          elem: int = 2) -> int:
        per_block = num_layers * 2 * kv_heads * block_size * head_dim * elem
        return max(1, bytes_budget // per_block)


@dataclass(frozen=True)
class KvGeometry:
    """K / V pages of one cache-owning layer run. v_heads: value heads, where they are not cached like the keys (0: like the keys)."""
    kv_heads: int
    k_dim: int
    v_dim: int
    v_heads: int = 0

    def page_shapes(self, block_size: int) -> list[tuple[int, ...]]:
        return [(self.kv_heads, block_size, self.k_dim), (self.v_heads or self.kv_heads, block_size, self.v_dim)]


@dataclass(frozen=True)
class LatentGeometry:
    """Pages of a latent-attention layer: one row of `width` numbers per token, shared by all heads."""
    width: int

    def page_shapes(self, block_size: int) -> list[tuple[int, ...]]:
        return [(block_size, self.width)]


@dataclass(frozen=True)
class TokenGeometry:
    """Pages of token ids, for models whose input at a position depends on the ids in front of it. Paged like keys, so that rollbacks,
    forks and shared prefixes need nothing else."""

    def page_shapes(self, block_size: int) -> list[tuple[int, ...]]:
        return [(block_size,)]


@dataclass(frozen=True)
class StateGeometry:
    """Recurrent layer: per sequence a fp32 state and a window of recent inputs in the activation type; no pages."""
    state: tuple[int, ...]
    window: tuple[int, ...]

    def page_shapes(self, block_size: int) -> list[tuple[int, ...]]:
        return []


@dataclass(frozen=True)
class WindowGeometry:
    """Short convolution over time: per sequence a window of recent inputs in the activation type; no pages."""
    window: tuple[int, ...]

    def page_shapes(self, block_size: int) -> list[tuple[int, ...]]:
        return []


PER_SEQUENCE = (StateGeometry, WindowGeometry)      # what a state slot holds


class LayeredKvPool:
    """Paged pool of a model whose layers differ in what they keep, or run more than once: every run owns its page tensors
    [blocks, ...] (K and V, latent rows, or token ids), or several such entries. Block ids are shared by all runs (one allocator), so sequences, forks and
    rollbacks work as on the uniform pool. Recurrent layers and short convolutions own tensors [state_slots, ...] instead; a sequence holds one slot
    for all of them from its first token to its release. A slot needs no clearing: the kernels take the state of a sequence
    as zero at position 0."""

    def __init__(self, geometry: list[KvGeometry | LatentGeometry | TokenGeometry | StateGeometry | WindowGeometry], num_blocks: int, block_size: int = 16,
                 device: torch.device | str = "cuda", dtype: torch.dtype = torch.bfloat16, state_slots: int = 0):
        self.geometry, self.num_layers = list(geometry), len(geometry)
        self.num_blocks, self.block_size = num_blocks, block_size
        self.has_state = any(isinstance(g, PER_SEQUENCE) for g in geometry)
        if self.has_state and state_slots < 1:
            raise ValueError("a pool with recurrent layers needs state slots")

        def tensors(g) -> tuple[torch.Tensor, ...]:
            if isinstance(g, StateGeometry):
                return (torch.zeros((state_slots, *g.state), dtype=torch.float32, device=device),
                        torch.zeros((state_slots, *g.window), dtype=dtype, device=device))
            if isinstance(g, WindowGeometry):
                return (torch.zeros((state_slots, *g.window), dtype=dtype, device=device),)
            kind = torch.int32 if isinstance(g, TokenGeometry) else dtype
            return tuple(torch.zeros((num_blocks, *s), dtype=kind, device=device) for s in g.page_shapes(block_size))
        self.data = [tensors(g) for g in geometry]
        self.allocator = BlockAllocator(num_blocks)
        self.slots = BlockAllocator(state_slots) if self.has_state else None

    @property
    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for kv in self.data for t in kv)

    def copy_block(self, src: int, dst: int) -> None:
        for g, kv in zip(self.geometry, self.data):
            if not isinstance(g, PER_SEQUENCE):
                for t in kv:
                    t[dst].copy_(t[src])

    def copy_state(self, src: int, dst: int) -> None:
        for g, kv in zip(self.geometry, self.data):
            if isinstance(g, PER_SEQUENCE):
                for t in kv:
                    t[dst].copy_(t[src])

    @staticmethod
    def block_bytes(geometry, block_size: int = 16, elem: int = 2) -> int:
        return sum(math.prod(s) * (4 if isinstance(g, TokenGeometry) else elem) for g in geometry for s in g.page_shapes(block_size))


class PagedSequence:
    """Block table of one sequence over a pool: token i lives in blocks[i // bs] at offset i % bs."""

    _next_uid = 1

    def __init__(self, pool: PagedKvPool):
        self.pool = pool
        self.blocks: list[int] = []
        self.length = 0  # tokens whose K/V are (or are being) written
        self.uid = PagedSequence._next_uid  # never reused; with `epoch` it keys cached device block tables
        PagedSequence._next_uid += 1
        self.epoch = 0   # bumped whenever an already-published block id changes (COW unshare, truncate)
        self.state_slot = -1                    # recurrent layers: slot of this sequence's state (held while length > 0)
        self.tokens: list[int] | None = []      # recurrent layers: what was fed, to rebuild the state of a rollback; None
        #                                         once tokens were chosen on the device
        self.checkpoint: tuple[int, int] | None = None   # (length, slot): copy of the state before the last verify step

    @classmethod
    def seeded(cls, pool: PagedKvPool, blocks: list[int], length: int) -> "PagedSequence":
        """Share an existing prefix copy-on-write: retains the full blocks covering `length` tokens."""
        s = cls(pool)
        for b in blocks:
            pool.allocator.retain(b)
        s.blocks = list(blocks)
        s.length = length
        return s

    def reserve(self, n_tokens: int) -> list[int]:
        """Make room for n_tokens more tokens and return their flat cache slots (block * bs + offset)."""
        bs = self.pool.block_size
        slots = []
        if self.state_slot < 0 and self.stateful:
            self.state_slot = self.pool.slots.alloc()
        for _ in range(n_tokens):
            bi, off = divmod(self.length, bs)
            if bi == len(self.blocks):
                self.blocks.append(self.pool.allocator.alloc())
            elif off == 0 or self.pool.allocator.refcount(self.blocks[bi]) > 1:
                # writing into a shared block: unshare it first (copy-on-write)
                if self.pool.allocator.refcount(self.blocks[bi]) > 1:
                    fresh = self.pool.allocator.alloc()
                    self.pool.copy_block(self.blocks[bi], fresh)
                    self.pool.allocator.release(self.blocks[bi])
                    self.blocks[bi] = fresh
                    self.epoch += 1
            slots.append(self.blocks[bi] * bs + off)
            self.length += 1
        return slots

    @property
    def stateful(self) -> bool:
        return getattr(self.pool, "has_state", False)

    def fed(self, tokens: list[int] | None) -> None:
        """Remembers the tokens of a step (None: they are known to the device only)."""
        if self.stateful:
            self.tokens = None if tokens is None or self.tokens is None else self.tokens + tokens

    def drop_checkpoint(self) -> None:
        if self.checkpoint is not None:
            self.pool.slots.release(self.checkpoint[1])
            self.checkpoint = None

    def truncate(self, length: int) -> None:
        """Roll back to `length` tokens (speculative rejection); frees blocks past the boundary. A recurrent state cannot
        run backwards: there the caller restores or rebuilds it for `length` tokens (`GpuBackend.truncate`)."""
        bs = self.pool.block_size
        keep = (length + bs - 1) // bs
        for b in self.blocks[keep:]:
            self.pool.allocator.release(b)
        self.blocks = self.blocks[:keep]
        self.length = length
        self.epoch += 1
        if self.stateful and self.tokens is not None:
            self.tokens = self.tokens[:length]

    def shareable_prefix_blocks(self, n_tokens: int) -> list[int]:
        """Blocks fully covered by the first n_tokens tokens (only whole blocks are shareable)."""
        return self.blocks[: n_tokens // self.pool.block_size]

    def release(self) -> None:
        for b in self.blocks:
            self.pool.allocator.release(b)
        self.blocks = []
        self.length = 0
        self.drop_checkpoint()
        if self.state_slot >= 0:
            self.pool.slots.release(self.state_slot)
            self.state_slot = -1
        self.tokens = []
