"""Cache of a decoder that mixes paged attention with recurrent layers.

Per layer any of: a pair of dense K/V page pools (:class:`PagedKVPool`, addressed by the same block tables and slots as
the spike pools), a pool of shared-latent rows (:class:`PagedLatentPool`; a layer may read an earlier layer's), and named per-row states in 32 bits (one slot per batch row; a request keeps its row, and with it its
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
class LatentSpec:
    """One layer's shared-latent cache: ``rank`` latent and ``rot_dim`` rotated channels per token, read by all heads."""

    rank: int
    rot_dim: int


@dataclass(frozen=True)
class LayerCacheSpec:
    kv: KVSpec | None = None
    states: tuple[tuple[str, tuple[int, ...]], ...] = ()
    """(name, shape) of every per-row state."""
    latent: LatentSpec | None = None
    latent_from: int | None = None
    """The (earlier) layer whose latent pool this layer reads."""


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


class PagedLatentPool(PagedKVPool):
    """A pool of shared-latent cache rows: ``rank`` latent channels at 0, ``rot_dim`` rotated ones at ``rank_pad``; one pool head.
    In 16 bits pages are tiled and both parts padded to 64 channels: eight rows after the other, of eight rows 64 channels after
    the other, swizzled as in :class:`PagedKVPool`, so that pages laid end to end are one operand.  Plain without padding otherwise."""

    def __init__(self, num_blocks: int, block_size: int, rank: int, rot_dim: int, dtype: torch.dtype, device) -> None:
        self.rank, self.rot_dim, self.block_size = rank, rot_dim, block_size
        self.tiled = dtype == torch.bfloat16 and block_size % 16 == 0
        self.rank_pad, self.rot_pad = (-(-x // 64) * 64 if self.tiled else x for x in (rank, rot_dim))
        self.pad = self.dim = self.rank_pad + self.rot_pad
        self.data = torch.zeros((num_blocks, 1, block_size, self.pad), dtype=dtype, device=device)

    def rows(self) -> torch.Tensor:
        """``[num_blocks * block_size, rank + rot_dim]`` in plain order (for checks)."""
        nb, _, bs, pad = self.data.shape
        x = self.data.view(nb * bs, pad)
        if self.tiled:
            x = self.data.view(nb, bs // 8, pad // 64, 8, 8, 8)
            r = torch.arange(8, device=x.device)
            group = r[None, :] ^ r[:, None]  # stored place of group c in row r
            x = x.gather(4, group.view(1, 1, 1, 8, 8, 1).expand(x.shape)).transpose(2, 3).reshape(nb * bs, pad)
        return torch.cat((x[:, : self.rank], x[:, self.rank_pad: self.rank_pad + self.rot_dim]), dim=1)


class LayerCache:
    def __init__(self, spec: LayerCacheSpec, num_blocks: int, block_size: int, max_rows: int, dtype: torch.dtype, device,
                 earlier: list["LayerCache"] = ()) -> None:
        self.latent = None
        if spec.latent_from is not None:
            if not 0 <= spec.latent_from < len(earlier) or earlier[spec.latent_from].latent is None:
                raise ValueError(f"layer {spec.latent_from} holds no latent pool to share")
            self.latent = earlier[spec.latent_from].latent
        elif spec.latent is not None:
            self.latent = PagedLatentPool(num_blocks, block_size, spec.latent.rank, spec.latent.rot_dim, dtype, device)
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
        self.layers: list[LayerCache] = []
        for s in specs:
            self.layers.append(LayerCache(s, num_blocks, block_size, max_rows, dtype, self.device, self.layers))

    @property
    def pad_block(self) -> int:
        return self.num_blocks - 1

    @property
    def capacity_tokens(self) -> int:
        return (self.num_blocks - 1) * self.block_size

    @property
    def nbytes(self) -> int:
        tensors = {id(t): t for layer in self.layers
                   for t in (*(p.data for p in (layer.k, layer.v, layer.latent) if p is not None), *layer.states.values())}
        return sum(t.numel() * t.element_size() for t in tensors.values())  # a shared pool counts once

    def recurrent_tensors(self) -> tuple:
        """State that a replayed step would not rewrite by itself (snapshots save it)."""
        return tuple(t for layer in self.layers for t in layer.states.values())
