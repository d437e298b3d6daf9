"""Attention over a shared latent (CUDA): what is cached per token is a normalised latent and one rotated key part; queries are taken
into the latent space, sums of latents back out of it.

``pool`` is a :class:`~spikeinfer_b200.engine.kv_state_cache.PagedLatentPool`.  Tensors are fp32 or bf16; norms, rotations, scores and
key weights are 32-bit."""
from __future__ import annotations

import torch
import torch.nn.functional as F

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
                     token_rows: torch.Tensor | None = None, positions: torch.Tensor | None = None, most_keys: int | None = None, overlap_previous: bool = False,
                     status: torch.Tensor | None = None) -> torch.Tensor:
    """``out[t, h vdim :] = sigmoid(gate) * W_uv[h] (softmax with sink over the visible cache rows)`` for queries of :func:`latent_query`.
    ``token_rows`` / ``positions``: tokens of prefill portions (token t sees ``positions[t] + 1`` keys of its row); without them the
    decode form over ``seq_lens`` / ``active``.  ``overlap_previous``: this call directly follows :func:`latent_query` and may be placed while
    that still runs (tables and lengths were complete before it began)."""
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
        rank_pad=pool.rank_pad, rot_pad=pool.rot_pad, tiled=int(pool.tiled), block_size=pool.block_size, dtype=code, overlap=int(overlap_previous), scale=scale, status=_ptr(status))
    _call("spk_latent_attn", a, q.device)
    b = _lib.LatentOutArgs(
        partials=partials.data_ptr(), stats=stats.data_ptr(), sink=sink.data_ptr(), w_uv=w_uv.data_ptr(), gate=gate.data_ptr(), out=out.data_ptr(),
        seq_lens=None if prefill else seq_lens.data_ptr(), active=_ptr(active), positions=_ptr(positions), gate_stride=gate.stride(0),
        out_stride=out.stride(0), n=n, splits=splits, heads=heads, vdim=vdim, rank=pool.rank, dtype=code, overlap=1,
        status=_ptr(status))
    _call("spk_latent_out", b, q.device)
    return out


PREFILL_TILE = 128          # query tokens per tile of the spelled-out form
PREFILL_MIN_TOKENS = 64     # fewer tokens in a call are taken into the latent space one by one
PREFILL_CONTEXT_RATIO = 32  # spelling keys and values out pays off up to this many cache rows per query token
PREFILL_MAX_BYTES = 8 << 30


def spelled_out_weights(w_uk: torch.Tensor, w_uv: torch.Tensor, heads: int) -> torch.Tensor:
    """Key and value matrices of all heads stacked, every head padded to a multiple of 64 channels with zeros."""
    def pad(w):
        d = w.shape[0] // heads
        return F.pad(w.view(heads, d, -1), (0, 0, 0, -d % 64)).flatten(0, 1)
    return torch.cat((pad(w_uk), pad(w_uv))).contiguous()


def latent_prefill(q: torch.Tensor, pool, tables: torch.Tensor, w_uk: torch.Tensor, w_uv: torch.Tensor, w_kv: torch.Tensor | None, sink: torch.Tensor,
                   gate: torch.Tensor, out: torch.Tensor, *, rot_table: torch.Tensor, positions: torch.Tensor, token_rows: torch.Tensor, plan, heads: int,
                   dim: int, vdim: int, scale: float, spelled_out: bool | None = None, status: torch.Tensor | None = None) -> torch.Tensor:
    """Attention of the tokens of prefill portions (``plan``), ``q [n, heads * (dim + rot_dim)]`` as projected.  Long portions spell keys and
    values out (``w_kv`` from :func:`spelled_out_weights`; ``spelled_out`` overrides the choice), others take the queries into the latent
    space.  The rest as in :func:`latent_attention`."""
    lib = _lib.load()
    n = q.shape[0]
    code = _lib.dtype_code(q.dtype)
    possible = w_kv is not None and scale > 0 and bool(lib.spk_latent_prefill_form(code, dim, pool.rot_pad, vdim, int(pool.tiled)))
    if spelled_out is None:
        rows = sum(plan.contexts_before) + sum(plan.lens)
        spelled_out = possible and n >= PREFILL_MIN_TOKENS and rows <= PREFILL_CONTEXT_RATIO * n and rows * w_kv.shape[0] * 2 <= PREFILL_MAX_BYTES
    if not spelled_out:
        ql = latent_query(q, w_uk, pool, rot_table, positions, heads=heads, dim=dim, status=status)
        return latent_attention(ql, pool, tables, sink, w_uv, gate, out, vdim=vdim, scale=scale, token_rows=token_rows, positions=positions,
                                most_keys=plan.most_keys, status=status)
    if not possible:
        raise ValueError("these sizes have no spelled-out form")
    _f32(sink, "sink", heads)
    if not q.is_contiguous() or q.shape[1] != heads * (dim + pool.rot_dim) or out.shape != (n, heads * vdim) or gate.shape != out.shape:
        raise ValueError("q, gate and out do not fit the head sizes")
    _, total, rows = plan.contexts()
    latents = torch.empty((total, pool.rank_pad), dtype=q.dtype, device=q.device)
    rotated = torch.empty((total, 64), dtype=q.dtype, device=q.device)
    g = _lib.LatentGatherArgs(pool=pool.data.data_ptr(), tables=tables.data_ptr(), rows=rows.data_ptr(), latents=latents.data_ptr(), rotated=rotated.data_ptr(),
                              table_stride=tables.stride(0), table_rows=tables.shape[0], max_blocks=tables.shape[1], num_blocks=pool.data.shape[0],
                              n_ctx=total, n_rows=rows.shape[0], rank_pad=pool.rank_pad, block_size=pool.block_size, status=_ptr(status))
    _call("spk_latent_gather", g, q.device)
    kv = F.linear(latents[:, : pool.rank], w_kv)
    tiles = plan.context_tiles(PREFILL_TILE)
    a = _lib.LatentPrefillArgs(
        q=q.data_ptr(), kv=kv.data_ptr(), kr=rotated.data_ptr(), tiles=tiles.data_ptr(), sink=sink.data_ptr(), gate=gate.data_ptr(), out=out.data_ptr(),
        rot_table=rot_table.data_ptr(), rot_positions=rot_table.shape[0], n=n, n_ctx=total, gate_stride=gate.stride(0), out_stride=out.stride(0),
        n_tiles=tiles.shape[0], heads=heads, dim=dim, rot_dim=pool.rot_dim, vdim=vdim, dim_pad=-(-dim // 64) * 64, vdim_pad=-(-vdim // 64) * 64,
        dtype=code, scale=scale, status=_ptr(status))
    _call("spk_latent_prefill", a, q.device)
    return out
