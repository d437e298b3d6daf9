"""Attention over a shared latent (CUDA): what is cached per token is a normalised latent and one rotated key part; queries are taken
into the latent space, sums of latents back out of it.

``pool`` is a :class:`~spikeinfer_b200.engine.kv_state_cache.PagedLatentPool`.  Tensors are fp32 or bf16; norms, rotations, scores and
key weights are 32-bit."""
from __future__ import annotations

import torch

from .. import _lib
from .dense import _call, _f32, _ptr


def latent_prepare(cq: torch.Tensor, w_q: torch.Tensor, *, eps: float, kv: torch.Tensor | None = None, w_kv: torch.Tensor | None = None, pool=None,
                   rot_table: torch.Tensor | None = None, positions: torch.Tensor | None = None, slot_mapping: torch.Tensor | None = None,
                   status: torch.Tensor | None = None) -> torch.Tensor:
    """Norm of the query latent (returned, ``[n, q_rank]``); with ``kv`` also norm, rotation and page write of the cached row.  ``cq`` and
    ``kv`` are column ranges of one projection output."""
    _lib.require_cuda(cq, "latent_prepare input")
    n, q_rank = cq.shape
    _f32(w_q, "w_q", q_rank)
    out = torch.empty((n, q_rank), dtype=cq.dtype, device=cq.device)
    a = _lib.LatentPrepareArgs(cq=cq.data_ptr(), ld=cq.stride(0), w_q=w_q.data_ptr(), cq_out=out.data_ptr(), n=n, q_rank=q_rank,
                               dtype=_lib.dtype_code(cq.dtype), eps=eps, status=_ptr(status))
    if kv is not None:
        _f32(w_kv, "w_kv", pool.rank)
        if kv.shape != (n, pool.rank + pool.rot_dim) or kv.stride(0) != cq.stride(0) or rot_table.shape[1] * 2 != pool.rot_dim:
            raise ValueError("kv must be [n, rank + rot_dim] in the matrix cq lies in, with a table of its rotation")
        a.kv, a.w_kv, a.pool, a.rot_table = kv.data_ptr(), w_kv.data_ptr(), pool.data.data_ptr(), rot_table.data_ptr()
        a.positions, a.slot_mapping, a.rot_positions, a.num_blocks = positions.data_ptr(), slot_mapping.data_ptr(), rot_table.shape[0], pool.data.shape[0]
        a.rank, a.rot_dim, a.rank_pad, a.rot_pad = pool.rank, pool.rot_dim, pool.rank_pad, pool.rot_pad
        a.tiled, a.block_size = int(pool.tiled), pool.block_size
    _call("spk_latent_prepare", a, cq.device)
    return out


def latent_query(q: torch.Tensor, w_uk: torch.Tensor, pool, rot_table: torch.Tensor, positions: torch.Tensor, *, heads: int, dim: int,
                 status: torch.Tensor | None = None) -> torch.Tensor:
    """``q [n, heads * (dim + rot_dim)]`` -> queries over cache rows ``[n, heads, pool.pad]``: ``W_uk^T`` of the unrotated part, the rotated
    part turned."""
    _lib.require_cuda(q, "latent_query input")
    n = q.shape[0]
    if not q.is_contiguous() or q.shape[1] != heads * (dim + pool.rot_dim) or w_uk.shape != (heads * dim, pool.rank) or not w_uk.is_contiguous():
        raise ValueError("q and w_uk do not fit the head sizes")
    out = torch.empty((n, heads, pool.pad), dtype=q.dtype, device=q.device)
    a = _lib.LatentQueryArgs(q=q.data_ptr(), w_uk=w_uk.data_ptr(), out=out.data_ptr(), rot_table=rot_table.data_ptr(), positions=positions.data_ptr(),
                             rot_positions=rot_table.shape[0], n=n, heads=heads, dim=dim, rank=pool.rank, rot_dim=pool.rot_dim,
                             rank_pad=pool.rank_pad, rot_pad=pool.rot_pad, dtype=_lib.dtype_code(q.dtype), status=_ptr(status))
    _call("spk_latent_query", a, q.device)
    return out


def latent_attention(q: torch.Tensor, pool, tables: torch.Tensor, sink: torch.Tensor, w_uv: torch.Tensor, gate: torch.Tensor, out: torch.Tensor, *,
                     vdim: int, scale: float, seq_lens: torch.Tensor | None = None, active: torch.Tensor | None = None,
                     token_rows: torch.Tensor | None = None, positions: torch.Tensor | None = None, most_keys: int | None = None,
                     status: torch.Tensor | None = None) -> torch.Tensor:
    """``out[t, h vdim :] = sigmoid(gate) * W_uv[h] (softmax with sink over the visible cache rows)`` for queries of :func:`latent_query`.
    ``token_rows`` / ``positions``: tokens of prefill portions (token t sees ``positions[t] + 1`` keys of its row); without them the
    decode form over ``seq_lens`` / ``active``."""
    _lib.require_cuda(q, "latent_attention query")
    n, heads, _ = q.shape
    _f32(sink, "sink", heads)
    if out.shape != (n, heads * vdim) or gate.shape != out.shape or out.stride(1) != 1 or gate.stride(1) != 1 or out.dtype != q.dtype or gate.dtype != q.dtype:
        raise ValueError("out and gate must be [n, heads * vdim] in the dtype of q with unit column stride")
    lib = _lib.load()
    code = _lib.dtype_code(q.dtype)
    keys = tables.shape[1] * pool.block_size if most_keys is None else most_keys
    splits = int(lib.spk_latent_attn_splits(code, pool.rank, pool.rot_dim, pool.rank_pad, pool.rot_pad, int(pool.tiled), pool.block_size, n, heads, keys))
    partials = torch.empty((n, splits, heads, pool.rank), dtype=torch.float32, device=q.device)
    stats = torch.empty((n, splits, heads, 2), dtype=torch.float32, device=q.device)
    prefill = token_rows is not None
    a = _lib.LatentAttnArgs(
        q=q.data_ptr(), pool=pool.data.data_ptr(), tables=tables.data_ptr(), seq_lens=_ptr(seq_lens), active=_ptr(active), token_rows=_ptr(token_rows),
        positions=_ptr(positions), partials=partials.data_ptr(), stats=stats.data_ptr(), table_stride=tables.stride(0), table_rows=tables.shape[0],
        max_blocks=tables.shape[1], n=n, num_blocks=pool.data.shape[0], splits=splits, heads=heads, rank=pool.rank, rot_dim=pool.rot_dim,
        rank_pad=pool.rank_pad, rot_pad=pool.rot_pad, tiled=int(pool.tiled), block_size=pool.block_size, dtype=code, scale=scale, status=_ptr(status))
    _call("spk_latent_attn", a, q.device)
    b = _lib.LatentOutArgs(
        partials=partials.data_ptr(), stats=stats.data_ptr(), sink=sink.data_ptr(), w_uv=w_uv.data_ptr(), gate=gate.data_ptr(), out=out.data_ptr(),
        seq_lens=None if prefill else seq_lens.data_ptr(), active=_ptr(active), positions=_ptr(positions), gate_stride=gate.stride(0),
        out_stride=out.stride(0), n=n, splits=splits, heads=heads, vdim=vdim, rank=pool.rank, dtype=code, status=_ptr(status))
    _call("spk_latent_out", b, q.device)
    return out
