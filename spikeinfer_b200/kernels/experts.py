"""Experts chosen by the token's id (CUDA): routing, and the experts' products on matrices sorted by expert.

A *sorted matrix* holds one row per (token, choice) pair, grouped by expert; every expert's segment starts at a multiple of eight rows.
In bf16 it is stored as tensor-core operand tiles: ``[ceil(columns / 64)][rows][64]``, the 16-byte group ``g`` of row ``r`` at group
``g ^ (r & 7)``, columns beyond the width zero.  In fp32 it is plain ``[rows, columns]``."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import _lib
from .dense import _call, _ptr


def operand_tiles(w: torch.Tensor) -> torch.Tensor:
    """``[rows, k]`` (rows a multiple of eight) -> ``[ceil(k / 64), rows, 64]`` in operand order."""
    rows, k = w.shape
    kt = -(-k // 64)
    x = torch.zeros((rows, kt * 64), dtype=w.dtype, device=w.device)
    x[:, :k] = w
    x = x.view(rows, kt, 8, 8)
    r = torch.arange(rows, device=w.device)
    source = torch.arange(8, device=w.device)[None, :] ^ (r[:, None] & 7)
    x = x.gather(2, source.view(rows, 1, 8, 1).expand(x.shape))
    return x.permute(1, 0, 2, 3).reshape(kt, rows, 64).contiguous()


def plain_rows(tiles: torch.Tensor, k: int) -> torch.Tensor:
    """Inverse of :func:`operand_tiles` (for checks)."""
    kt, rows, _ = tiles.shape
    x = tiles.view(kt, rows, 8, 8)
    r = torch.arange(rows, device=tiles.device)
    stored = torch.arange(8, device=tiles.device)[None, :] ^ (r[:, None] & 7)
    x = x.gather(2, stored.view(1, rows, 8, 1).expand(x.shape))
    return x.reshape(kt, rows, 64).permute(1, 0, 2).reshape(rows, kt * 64)[:, :k]


def _blocks(w: torch.Tensor, per: int) -> torch.Tensor:
    """``[out, k]`` -> ``[ceil(out / per), ktiles, per, 64]`` operand tiles, rows beyond ``out`` zero."""
    out, k = w.shape
    blocks = -(-out // per)
    x = torch.zeros((blocks * per, k), dtype=w.dtype, device=w.device)
    x[:out] = w
    t = operand_tiles(x)
    return t.view(t.shape[0], blocks, per, 64).transpose(0, 1).contiguous()


class ExpertWeights:
    """Gate, up and down matrices of a layer's experts in the layout of their kernels, and the table that names a token's experts."""

    def __init__(self, gates, ups, downs, table: torch.Tensor) -> None:
        self.experts, self.ff, self.width = len(gates), gates[0].shape[0], gates[0].shape[1]
        self.top = table.shape[1]
        dtype, device = gates[0].dtype, gates[0].device
        if int(table.min()) < 0 or int(table.max()) >= self.experts:
            raise ValueError("the expert table names experts that do not exist")
        self.table = table.to(device=device, dtype=torch.int32).contiguous()
        self.dtype, self.tiled = dtype, dtype == torch.bfloat16
        if self.tiled:
            # [experts][blocks][ktiles][gate | up][128][64] and [experts][blocks][ktiles][256][64]
            first = torch.stack((_blocks(gates[0], 128), _blocks(ups[0], 128)), dim=2)
            self.w_in = torch.empty((self.experts, *first.shape), dtype=dtype, device=device)
            down = _blocks(downs[0], 256)
            self.w_out = torch.empty((self.experts, *down.shape), dtype=dtype, device=device)
            for e in range(self.experts):
                self.w_in[e] = torch.stack((_blocks(gates[e], 128), _blocks(ups[e], 128)), dim=2)
                self.w_out[e] = _blocks(downs[e], 256)
        else:
            self.w_in = torch.stack([torch.cat((g, u)) for g, u in zip(gates, ups)])
            self.w_out = torch.stack(list(downs))

    def rows(self, n: int) -> int:
        return int(_lib.load().spk_expert_rows(n, self.top, self.experts))

    def sorted_matrix(self, n: int, columns: int) -> torch.Tensor:
        shape = (-(-columns // 64), self.rows(n), 64) if self.tiled else (self.rows(n), columns)
        return torch.empty(shape, dtype=self.dtype, device=self.w_in.device)


@dataclass
class LayerRoute:
    slots: torch.Tensor
    """int32 ``[n, top]``: the rows of a token in the sorted matrix, -1 where it takes no part."""
    segs: torch.Tensor
    """int32 ``[experts, 2]``: first row and rows of every expert."""


class ExpertRouter:
    """Routing of all expert layers of a model: ids are all it needs, so one launch at the head of a step serves every layer."""

    def __init__(self, layers: list[ExpertWeights], vocab: int) -> None:
        self.layers, self.vocab = layers, vocab
        rows, self.tops, self.entries = [], 0, 0
        for w in layers:
            if w.table.shape[0] != vocab:
                raise ValueError("the expert table needs one row per token id")
            rows.append([w.table.data_ptr(), w.top, w.experts, self.tops, 2 * self.entries, 0, 0, 0])
            self.tops += w.top
            self.entries += w.experts
        self.desc = torch.tensor(rows, dtype=torch.int64, device=layers[0].table.device)

    def __call__(self, ids: torch.Tensor, active: torch.Tensor | None = None, status: torch.Tensor | None = None) -> list[LayerRoute]:
        n = ids.numel()
        slots = torch.empty(n * self.tops, dtype=torch.int32, device=ids.device)
        segs = torch.empty((self.entries, 2), dtype=torch.int32, device=ids.device)
        a = _lib.ExpertRouteArgs(layers=self.desc.data_ptr(), ids=ids.data_ptr(), active=_ptr(active), slots=slots.data_ptr(),
                                 segs=segs.data_ptr(), n=n, vocab=self.vocab, n_layers=len(self.layers),
                                 max_experts=max(w.experts for w in self.layers), status=_ptr(status))
        _call("spk_expert_route", a, ids.device)
        out, s, e = [], 0, 0
        for w in self.layers:
            out.append(LayerRoute(slots[n * s: n * (s + w.top)].view(n, w.top), segs[e: e + w.experts]))
            s, e = s + w.top, e + w.experts
        return out


def experts_forward(x: torch.Tensor, w: ExpertWeights, route: LayerRoute, status: torch.Tensor | None = None) -> torch.Tensor:
    """Every expert's feed-forward on its rows of the sorted matrix ``x``: fp32 ``[rows, width]``, unweighted."""
    _lib.require_cuda(x, "experts_forward input")
    n = route.slots.shape[0]
    rows = w.rows(n)
    hidden = w.sorted_matrix(n, w.ff)
    out = torch.empty((rows, w.width), dtype=torch.float32, device=x.device)
    common = dict(segs=route.segs.data_ptr(), rows=rows, pairs=n * w.top, experts=w.experts, dtype=_lib.dtype_code(w.dtype), status=_ptr(status))
    _call("spk_experts", _lib.ExpertsArgs(x=x.data_ptr(), w=w.w_in.data_ptr(), out=hidden.data_ptr(), k=w.width, out_features=w.ff, gated=1, **common),
          x.device)
    _call("spk_experts", _lib.ExpertsArgs(x=hidden.data_ptr(), w=w.w_out.data_ptr(), out=out.data_ptr(), k=w.ff, out_features=w.width, gated=0,
                                          **common), x.device)
    return out
