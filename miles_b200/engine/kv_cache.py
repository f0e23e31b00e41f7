"""Paged KV cache: fixed-size blocks, per-request block tables, a free-list allocator.

The allocator has a C++ implementation (`miles_b200.native`, lock-free free list + ref counts for
shared prefixes) that is used when the native runtime library is built; the python class below is
the same algorithm and the CPU-test path.  The engine the reference drives (SGLang, radix/paged KV)
is external to it; sizing follows its `--sglang-mem-fraction-static` knob.
"""
from __future__ import annotations

import math

import torch


class BlockAllocator:
    def __init__(self, num_blocks: int):
        self.num_blocks = num_blocks
        self.free: list[int] = list(range(num_blocks - 1, -1, -1))
        self.refcnt = [0] * num_blocks

    @property
    def num_free(self) -> int:
        return len(self.free)

    def alloc(self, n: int) -> list[int] | None:
        if n > len(self.free):
            return None
        out = [self.free.pop() for _ in range(n)]
        for b in out:
            self.refcnt[b] = 1
        return out

    def share(self, blocks: list[int]):
        for b in blocks:
            self.refcnt[b] += 1

    def release(self, blocks: list[int]):
        for b in blocks:
            self.refcnt[b] -= 1
            if self.refcnt[b] == 0:
                self.free.append(b)
            assert self.refcnt[b] >= 0

    def reset(self):
        self.free = list(range(self.num_blocks - 1, -1, -1))
        self.refcnt = [0] * self.num_blocks


def make_allocator(num_blocks: int):
    try:
        from ..native import runtime as rt

        if rt.available():
            return rt.NativeBlockAllocator(num_blocks)
    except Exception:
        pass
    return BlockAllocator(num_blocks)


class KVCache:
    """Paged tensors per layer, each [num_blocks, block_size, *row]: K and V rows (Hkv, D) by default, or what a model's
    `kv_rows()` lists per layer (one latent row; nothing for a layer that keeps no tokens or reads another layer's)."""

    def __init__(self, num_layers: int, num_blocks: int, block_size: int, num_kv_heads: int, head_dim: int,
                 dtype, device, layer_ids: list[int] | None = None, rows: "dict[int, tuple] | None" = None):
        self.num_blocks, self.block_size = num_blocks, block_size
        self.dtype, self.device = dtype, device
        if rows is None:
            ids = layer_ids if layer_ids is not None else list(range(num_layers))
            rows = {l: ((num_kv_heads, head_dim), (num_kv_heads, head_dim)) for l in ids}
        self.rows = rows
        self.layer_ids = list(rows)
        self.layers: dict[int, tuple[torch.Tensor, ...]] = {}
        self.live = False
        self.allocate()

    def allocate(self):
        for l, shapes in self.rows.items():
            self.layers[l] = tuple(torch.zeros((self.num_blocks, self.block_size, *s), dtype=self.dtype, device=self.device) for s in shapes)
        self.live = True

    def free(self):
        """Release the cache memory (engine `release_memory_occupation(tags=['kv_cache'])`)."""
        self.layers = {}
        self.live = False
        if torch.cuda.is_available():
            torch.cuda.empty_cache()

    @property
    def allocated(self) -> bool:
        return self.live

    def bytes(self) -> int:
        return self.num_blocks * self.bytes_per_block(self.rows, self.block_size, self.dtype)

    @staticmethod
    def bytes_per_block(rows: "dict[int, tuple]", block_size: int, dtype) -> int:
        return block_size * sum(math.prod(s) for shapes in rows.values() for s in shapes) * torch.empty((), dtype=dtype).element_size()

    @staticmethod
    def blocks_for_budget(bytes_budget: int, num_layers: int, block_size: int, num_kv_heads: int, head_dim: int, dtype,
                          rows: "dict[int, tuple] | None" = None) -> int:
        if rows is None:
            rows = {l: ((num_kv_heads, head_dim), (num_kv_heads, head_dim)) for l in range(num_layers)}
        return max(1, bytes_budget // max(1, KVCache.bytes_per_block(rows, block_size, dtype)))


class StateCache:
    """Per-sequence fp32 state of recurrent layers: one [slots, *shape] tensor per layer and a free list of slots.  A sequence
    holds one slot from its admission to its end; the kernels start a sequence from zero state at position 0, so a slot that is
    used again needs no clearing."""

    def __init__(self, shapes: dict[int, tuple], num_slots: int, device):
        self.shapes, self.num_slots, self.device = shapes, num_slots, device
        self.layers: dict[int, torch.Tensor] = {}
        self.allocate()
        self.reset()

    def allocate(self):
        self.layers = {l: torch.zeros((self.num_slots, *s), dtype=torch.float32, device=self.device) for l, s in self.shapes.items()}

    def free(self):
        self.layers = {}

    @property
    def num_free(self) -> int:
        return len(self.free_slots)

    def alloc(self) -> int:
        return self.free_slots.pop()

    def release(self, slot: int):
        assert 0 <= slot < self.num_slots and slot not in self.free_slots
        self.free_slots.append(slot)

    def reset(self):
        self.free_slots = list(range(self.num_slots - 1, -1, -1))

    def copy(self, src: list[int], dst: list[int]):
        """The states of slots `src` into slots `dst`, every layer."""
        s = torch.tensor(src, dtype=torch.int64, device=self.device)
        d = torch.tensor(dst, dtype=torch.int64, device=self.device)
        for t in self.layers.values():
            t.index_copy_(0, d, t.index_select(0, s))
