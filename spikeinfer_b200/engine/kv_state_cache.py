"""Cache of a decoder that mixes paged attention with recurrent layers.

Per layer any of: a pair of dense K/V page pools (:class:`PagedKVPool`, addressed by the same block tables and slots as
the spike pools), and named per-row states in 32 bits (one slot per batch row; a request keeps its row, and with it its
slot, from its first token to its release).  A slot is never cleared when it is handed on: a portion that starts at position
0 does not read it.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class KVSpec:
    """One layer's attention cache: ``kv_heads`` heads of ``dim`` key and ``vdim`` value channels per token."""

    kv_heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class LayerCacheSpec:
    kv: KVSpec | None = None
    states: tuple[tuple[str, tuple[int, ...]], ...] = ()
    """(name, shape) of every per-row state."""


class PagedKVPool:
    """One K or V pool ``[num_blocks, kv_heads, block_size, pad]`` in the model dtype.

    16-bit pools of up to 128 channels and pages of a multiple of sixteen rows are *tiled*: ``pad`` is the next multiple of 64
    and a page is stored in the 128-byte-swizzled order the tensor core reads shared memory in, so that a page copied as it
    is becomes part of an operand tile.  Other pools are plain rows.  Channels beyond ``dim`` stay zero."""

    def __init__(self, num_blocks: int, kv_heads: int, block_size: int, dim: int, dtype: torch.dtype, device) -> None:
        self.dim, self.block_size = dim, block_size
        self.tiled = dtype == torch.bfloat16 and dim <= 128 and block_size % 16 == 0
        self.pad = -(-dim // 64) * 64 if self.tiled else dim
        self.data = torch.zeros((num_blocks, kv_heads, block_size, self.pad), dtype=dtype, device=device)

    def rows(self) -> torch.Tensor:
        """The pool as ``[num_blocks * block_size, kv_heads, dim]`` in plain order (for checks)."""
        nb, heads, bs, pad = self.data.shape
        x = self.data
        if self.tiled:
            x = x.view(nb, heads, pad // 64, bs, 8, 8)
            r = torch.arange(bs, device=x.device)
            group = torch.arange(8, device=x.device)[None, :] ^ (r[:, None] & 7)  # stored place of group c in row r
            x = x.gather(4, group.view(1, 1, 1, bs, 8, 1).expand(x.shape)).permute(0, 1, 3, 2, 4, 5).reshape(nb, heads, bs, pad)
        return x[..., : self.dim].permute(0, 2, 1, 3).reshape(nb * bs, heads, self.dim)


class LayerCache:
    def __init__(self, spec: LayerCacheSpec, num_blocks: int, block_size: int, max_rows: int, dtype: torch.dtype, device) -> None:
        self.k = self.v = None
        if spec.kv is not None:
            self.k = PagedKVPool(num_blocks, spec.kv.kv_heads, block_size, spec.kv.dim, dtype, device)
            self.v = PagedKVPool(num_blocks, spec.kv.kv_heads, block_size, spec.kv.vdim, dtype, device)
        self.states = {name: torch.zeros((max_rows, *shape), dtype=torch.float32, device=device) for name, shape in spec.states}


class PagedKVStateCache:
    def __init__(self, specs: list[LayerCacheSpec], num_blocks: int, block_size: int, max_rows: int, dtype: torch.dtype,
                 device: str | torch.device = "cuda") -> None:
        if num_blocks < 2:
            raise ValueError("need at least 2 blocks (one is reserved for padding)")
        if block_size < 1 or block_size & (block_size - 1):
            raise ValueError(f"block_size must be a power of two, got {block_size}")
        self.num_blocks, self.block_size, self.max_rows = num_blocks, block_size, max_rows
        self.device = torch.device(device)
        self.layers = [LayerCache(s, num_blocks, block_size, max_rows, dtype, self.device) for s in specs]

    @property
    def pad_block(self) -> int:
        return self.num_blocks - 1

    @property
    def capacity_tokens(self) -> int:
        return (self.num_blocks - 1) * self.block_size

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for layer in self.layers
                   for t in (*(p.data for p in (layer.k, layer.v) if p is not None), *layer.states.values()))

    def recurrent_tensors(self) -> tuple:
        """State that a replayed step would not rewrite by itself (snapshots save it)."""
        return tuple(t for layer in self.layers for t in layer.states.values())
