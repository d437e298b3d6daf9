"""Operators of the dense (non-spiking) decoders (CUDA): post-norm and pre-norm residual boundaries, activations, paged
attention with element-wise key weights, linear attention with a decaying state.

Tensors are fp32 or bf16; 32-bit arithmetic throughout.  The decode forms (token t = batch row t) have fixed arguments and
can be captured in a CUDA graph."""
from __future__ import annotations

from ctypes import byref

import torch

from .. import _lib

_ptr = _lib.ptr


def _call(name: str, args, device: torch.device) -> None:
    lib = _lib.load()
    with torch.cuda.device(device):
        rc = getattr(lib, name)(byref(args), _lib.current_stream(device))
    _lib.check(rc, name)


def _f32(t: torch.Tensor | None, name: str, numel: int | None = None) -> None:
    if t is not None and (t.dtype != torch.float32 or not t.is_contiguous() or (numel is not None and t.numel() != numel)):
        raise ValueError(f"{name} must be contiguous fp32" + ("" if numel is None else f" with {numel} elements"))


def residual_norm(out: torch.Tensor, *, eps: float, x: torch.Tensor | None = None, delta: torch.Tensor | None = None,
                  weight: torch.Tensor | None = None, alpha: float = 1.0, ids: torch.Tensor | None = None,
                  embed: torch.Tensor | None = None, x_out: torch.Tensor | None = None, second_weight: torch.Tensor | None = None,
                  mix: torch.Tensor | None = None, prev: torch.Tensor | None = None, commit: torch.Tensor | None = None,
                  positions: torch.Tensor | None = None, token_rows: torch.Tensor | None = None,
                  token_edges: torch.Tensor | None = None, active: torch.Tensor | None = None,
                  status: torch.Tensor | None = None) -> torch.Tensor:
    """One sublayer boundary: ``y = layernorm(alpha * x + delta) * weight`` (or ``y = embed[ids]``), written to ``x_out``
    (fp32) and, through the token shift ``mix``, the second norm or as it is, to ``out``.  ``prev`` / ``commit`` are
    per-row states ``[rows, width]``: the previous token of a portion's first token, and where the old ``x`` of its last token
    goes.  ``token_rows`` / ``token_edges`` None: decode form, gated by ``active``."""
    _lib.require_cuda(out, "residual_norm output")
    n, width = out.shape
    if not out.is_contiguous():
        raise ValueError("out must be contiguous")
    for t, name in ((weight, "weight"), (second_weight, "second_weight"), (mix, "mix")):
        _f32(t, name, width)
    for t, name in ((x, "x"), (x_out, "x_out")):
        _f32(t, name, n * width)
    for t, name in ((prev, "prev"), (commit, "commit")):
        _f32(t, name)
    if delta is not None and (delta.shape != out.shape or not delta.is_contiguous()):
        raise ValueError("delta must be contiguous and of the shape of out")
    if ids is not None and (embed is None or embed.dtype != out.dtype or not embed.is_contiguous() or embed.shape[1] != width or ids.numel() != n):
        raise ValueError("embed must be a contiguous [vocab, width] table in the dtype of out, ids one entry per row of out")
    state = prev if prev is not None else commit
    a = _lib.ResidualNormArgs(
        x=_ptr(x), x_out=_ptr(x_out), delta=_ptr(delta), embed=_ptr(embed), ids=_ptr(ids), vocab=0 if embed is None else embed.shape[0],
        w=_ptr(weight), w2=_ptr(second_weight), mix=_ptr(mix), prev=_ptr(prev), commit=_ptr(commit),
        state_rows=0 if state is None else state.shape[0], positions=_ptr(positions), token_rows=_ptr(token_rows),
        token_edges=_ptr(token_edges), active=_ptr(active), out=out.data_ptr(), n=n, width=width, alpha=alpha, eps=eps,
        dtype=_lib.dtype_code(out.dtype), delta_dtype=0 if delta is None else _lib.dtype_code(delta.dtype), status=_ptr(status))
    _call("spk_residual_norm", a, out.device)
    return out


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float, out: torch.Tensor | None = None) -> torch.Tensor:
    """``c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3`` per row, ``N`` = division by the root mean square (``out`` may be ``z``)."""
    _lib.require_cuda(z, "poly_norm input")
    _f32(coef, "coef", 4)
    out = torch.empty_like(z) if out is None else out
    if not z.is_contiguous() or not out.is_contiguous() or out.shape != z.shape or out.dtype != z.dtype:
        raise ValueError("z and out must be contiguous, same shape and dtype")
    lib = _lib.load()
    with torch.cuda.device(z.device):
        rc = lib.spk_poly_norm(z.data_ptr(), coef.data_ptr(), eps, out.data_ptr(), z.shape[0], z.shape[1],
                               _lib.dtype_code(z.dtype), _lib.current_stream(z.device))
    _lib.check(rc, "spk_poly_norm")
    return out


def _same_rows(*views: torch.Tensor) -> int:
    ld = views[0].stride(0)
    if any(v.stride(0) != ld or v.stride(1) != 1 for v in views):
        raise ValueError("the projections must be column ranges of one row-major matrix")
    return ld


def qk_prepare(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, k_pool, v_pool, slot_mapping: torch.Tensor, *, heads: int,
               kv_heads: int, dim: int, vdim: int, eps: float, unit_norm: bool = True, rot_table: torch.Tensor | None = None,
               positions: torch.Tensor | None = None, status: torch.Tensor | None = None) -> torch.Tensor:
    """Rotary embedding (``rot_table`` fp32 ``[positions, rot_dims / 2, 2]``) and unit norm of q and k, k and v into their
    pages.  ``q``, ``k``, ``v`` are column ranges of one projection output.  Returns q ``[n, heads, k_pool.pad]``."""
    _lib.require_cuda(q, "qk_prepare input")
    n = q.shape[0]
    ld = _same_rows(q, k, v)
    if q.shape[1] != heads * dim or k.shape[1] != kv_heads * dim or v.shape[1] != kv_heads * vdim:
        raise ValueError("projection widths do not fit the head sizes")
    _f32(rot_table, "rot_table")
    out = torch.empty((n, heads, k_pool.pad), dtype=q.dtype, device=q.device)
    a = _lib.QkPrepareArgs(
        q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(), ld=ld, q_out=out.data_ptr(), k_pool=k_pool.data.data_ptr(),
        v_pool=v_pool.data.data_ptr(), rot_table=_ptr(rot_table), positions=_ptr(positions), slot_mapping=slot_mapping.data_ptr(),
        rot_positions=0 if rot_table is None else rot_table.shape[0], n=n, num_blocks=k_pool.data.shape[0], heads=heads,
        kv_heads=kv_heads, dim=dim, vdim=vdim, k_pad=k_pool.pad, v_pad=v_pool.pad, k_tiled=int(k_pool.tiled),
        v_tiled=int(v_pool.tiled), block_size=k_pool.block_size, rot_dims=0 if rot_table is None else 2 * rot_table.shape[1],
        unit_norm=int(unit_norm), dtype=_lib.dtype_code(q.dtype), eps=eps, status=_ptr(status))
    _call("spk_qk_prepare", a, q.device)
    return out


def sigmoid_attention(q: torch.Tensor, k_pool, v_pool, tables: torch.Tensor, head_bias: torch.Tensor, out: torch.Tensor, *,
                      heads: int, kv_heads: int, dim: int, vdim: int, scale: float, out_scale: float = 1.0,
                      plan=None, seq_lens: torch.Tensor | None = None, active: torch.Tensor | None = None,
                      status: torch.Tensor | None = None, partial_sums: bool = False, overlap_previous: bool = False) -> torch.Tensor | None:
    """``out[t, h * vdim :] = out_scale * sum_j sigmoid(scale * q.k_j + head_bias[h]) v_j`` over the keys up to token t's own
    position, read through ``tables``.  ``out`` is a column range of a row-major matrix in the model dtype.  ``plan`` (a
    ``PrefillPlan``): prefill form; None: decode form over ``seq_lens`` / ``active``.

    ``partial_sums`` (decode form): where the sizes allow it, leave ``out`` alone and return fp32 partial sums
    ``[n, splits, heads * vdim]`` of key ranges, for :func:`gated_norm` to add up; otherwise ``out`` is written and None
    returned.  ``overlap_previous``: this call directly follows :func:`decay_attention` and may run beside it."""
    _lib.require_cuda(q, "sigmoid_attention query")
    _f32(head_bias, "head_bias", heads)
    n = q.shape[0]
    if out.shape != (n, heads * vdim) or out.stride(1) != 1 or out.dtype != q.dtype:
        raise ValueError("out must be [n, heads * vdim] in the dtype of q with unit column stride")
    lib = _lib.load()
    form = (_lib.dtype_code(q.dtype), k_pool.pad, v_pool.pad, int(k_pool.tiled), int(v_pool.tiled), k_pool.block_size)
    tiles = None if plan is None else plan.tiles(int(lib.spk_sigmoid_attn_tile_tokens(*form)))
    partials, splits = None, 0
    if partial_sums and plan is None:
        splits = int(lib.spk_sigmoid_attn_splits(*form, n, heads, kv_heads, tables.shape[1] * k_pool.block_size))
        if splits:
            partials = torch.empty((n, splits, heads * vdim), dtype=torch.float32, device=q.device)
    a = _lib.SigmoidAttnArgs(
        q=q.data_ptr(), k_pool=k_pool.data.data_ptr(), v_pool=v_pool.data.data_ptr(), tables=tables.data_ptr(),
        seq_lens=_ptr(seq_lens), active=_ptr(active), tiles=_ptr(tiles), head_bias=head_bias.data_ptr(), out=out.data_ptr(),
        out_stride=out.stride(0), table_stride=tables.stride(0), table_rows=tables.shape[0], max_blocks=tables.shape[1], n=n,
        num_blocks=k_pool.data.shape[0], partials=_ptr(partials), n_tiles=0 if tiles is None else tiles.shape[0], splits=splits,
        heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, k_pad=k_pool.pad, v_pad=v_pool.pad, k_tiled=int(k_pool.tiled),
        v_tiled=int(v_pool.tiled), block_size=k_pool.block_size, dtype=form[0], scale=scale, out_scale=out_scale,
        overlap=int(overlap_previous and partials is not None), status=_ptr(status))
    _call("spk_sigmoid_attn", a, q.device)
    return partials


def decay_powers(decay, device) -> torch.Tensor:
    """fp32 ``[heads, powers]``: the powers 0, 1, 2 ... of every head's decay, evaluated in double precision."""
    d = torch.tensor(list(decay), dtype=torch.float64)
    n = torch.arange(int(_lib.load().spk_decay_powers()), dtype=torch.float64)
    return (d[:, None] ** n[None, :]).to(torch.float32).to(device).contiguous()


def decay_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, state: torch.Tensor, powers: torch.Tensor, *,
                    plan=None, active: torch.Tensor | None = None, silu: bool = True,
                    status: torch.Tensor | None = None, overlap_previous: bool = False) -> torch.Tensor:
    """``S <- decay S + k v^T, o = S^T q`` per head, silu on q, k and v first.  ``q``, ``k``, ``v`` are column ranges of one
    projection output; ``state`` fp32 ``[rows, heads, dim, vdim]`` is updated in place; ``powers`` from :func:`decay_powers`.
    Returns fp32 ``[n, heads * vdim]``.  ``plan``: prefill form, None: decode form gated by ``active``.
    ``overlap_previous`` (decode form): this call directly follows :func:`qk_prepare` of the same step, everything it reads was
    complete before that began, and it may be placed while that still runs."""
    _lib.require_cuda(q, "decay_attention query")
    n = q.shape[0]
    rows, heads, dim, vdim = state.shape
    ld = _same_rows(q, k, v)
    if q.shape[1] != heads * dim or k.shape[1] != heads * dim or v.shape[1] != heads * vdim:
        raise ValueError("projection widths do not fit the state")
    _f32(state, "state")
    _f32(powers, "powers")
    lib = _lib.load()
    out = torch.empty((n, heads * vdim), dtype=torch.float32, device=q.device)
    a = _lib.DecayAttnArgs(
        q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(), ld=ld, state=state.data_ptr(), state_stride=state.stride(0), state_rows=rows,
        decay_pow=powers.data_ptr(), out=out.data_ptr(), active=_ptr(active), n=n, heads=heads, dim=dim, vdim=vdim,
        silu=int(silu), dtype=_lib.dtype_code(q.dtype), overlap=int(overlap_previous and plan is None), status=_ptr(status))
    if plan is None:
        _call("spk_decay_attn_step", a, q.device)
        return out
    chunks, seqs = plan.chunks(int(lib.spk_decay_chunk_tokens(a.dtype, dim, vdim, n, heads)))
    need = int(lib.spk_decay_attn_workspace_bytes(chunks.shape[0], heads, dim, vdim))
    ws = torch.empty(need, dtype=torch.uint8, device=q.device)
    a.chunks, a.seqs, a.n_chunks, a.n_seqs = chunks.data_ptr(), seqs.data_ptr(), chunks.shape[0], seqs.shape[0]
    a.workspace, a.workspace_bytes = ws.data_ptr(), need
    _call("spk_decay_attn_chunks", a, q.device)
    return out


def gated_norm(x: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, out: torch.Tensor, out_offset: int, *, eps: float,
               scale: float = 1.0, partials: torch.Tensor | None = None, left_scale: float = 1.0,
               seq_lens: torch.Tensor | None = None, active: torch.Tensor | None = None) -> torch.Tensor:
    """``out[:, out_offset:] = scale * rmsnorm(x) * weight * sigmoid(gate)`` over the whole width of ``x`` (fp32); with
    ``partials`` of :func:`sigmoid_attention` also ``out[:, :left_width] = left_scale * (their sum)``."""
    _lib.require_cuda(x, "gated_norm input")
    n, width = x.shape
    _f32(x, "x")
    _f32(weight, "weight", width)
    _f32(partials, "partials")
    if gate.shape != (n, width) or gate.stride(1) != 1 or gate.dtype != out.dtype or out.stride(1) != 1 or out.shape[1] < out_offset + width:
        raise ValueError("gate and out must be row-major in the model dtype and wide enough")
    a = _lib.GatedNormArgs(x=x.data_ptr(), w=weight.data_ptr(), gate=gate.data_ptr(), gate_stride=gate.stride(0), out=out.data_ptr(),
                           out_stride=out.stride(0), partials=_ptr(partials), seq_lens=_ptr(seq_lens), active=_ptr(active), n=n,
                           width=width, out_offset=out_offset, splits=0 if partials is None else partials.shape[1],
                           left_width=0 if partials is None else partials.shape[2], dtype=_lib.dtype_code(out.dtype), eps=eps,
                           scale=scale, left_scale=left_scale)
    _call("spk_gated_norm", a, x.device)
    return out


def rms_residual(*, eps: float, x: torch.Tensor | None = None, delta: torch.Tensor | None = None, ids: torch.Tensor | None = None,
                 embed: torch.Tensor | None = None, embed_scale: float = 1.0, x_out: torch.Tensor | None = None,
                 pairs: torch.Tensor | None = None, pair_slots: torch.Tensor | None = None, pair_scale: float = 1.0,
                 w1: torch.Tensor | None = None, out1: torch.Tensor | None = None, w2: torch.Tensor | None = None,
                 out2: torch.Tensor | None = None, out2_slots: torch.Tensor | None = None, out2_tiled: bool = False,
                 status: torch.Tensor | None = None) -> None:
    """One layer boundary: ``y = x + delta + pair_scale * (rows pair_slots[t] of pairs)`` (or ``embed_scale * embed[ids]``), to
    ``x_out`` (fp32, may be ``x``); ``out1 = rmsnorm(y) * w1`` and ``out2 = rmsnorm(y) * w2``.  ``out2_slots`` int32 ``[n, top]``:
    ``out2`` is a sorted matrix of experts (:mod:`.experts`) and a row goes to all of its slots, as operand tiles with
    ``out2_tiled``."""
    some = x if x is not None else x_out if x_out is not None else out1
    _lib.require_cuda(some, "rms_residual")
    n, width = some.shape
    for t, name in ((x, "x"), (x_out, "x_out")):
        _f32(t, name, n * width)
    for t, name in ((w1, "w1"), (w2, "w2")):
        _f32(t, name, width)
    _f32(pairs, "pairs")
    if delta is not None and (delta.shape != (n, width) or not delta.is_contiguous()):
        raise ValueError("delta must be contiguous [n, width]")
    if ids is not None and (embed is None or not embed.is_contiguous() or embed.shape[1] != width or ids.numel() != n):
        raise ValueError("embed must be a contiguous [vocab, width] table, ids one entry per row")
    for o in (out1, out2 if out2_slots is None else None):
        if o is not None and (o.shape != (n, width) or not o.is_contiguous()):
            raise ValueError("out1 and out2 must be contiguous [n, width]")
    outs = [t.dtype for t in (out1, out2, embed) if t is not None]
    if len(set(outs)) > 1:
        raise ValueError("outputs and embedding table must share one dtype")
    for s in (pair_slots, out2_slots):
        if s is not None and (s.dtype != torch.int32 or not s.is_contiguous() or s.shape[0] != n):
            raise ValueError("slots must be contiguous int32 [n, top]")
    a = _lib.RmsResidualArgs(
        x=_ptr(x), x_out=_ptr(x_out), delta=_ptr(delta), embed=_ptr(embed), ids=_ptr(ids), vocab=0 if embed is None else embed.shape[0],
        pairs=_ptr(pairs), pair_slots=_ptr(pair_slots), w1=_ptr(w1), out1=_ptr(out1), w2=_ptr(w2), out2=_ptr(out2),
        out2_slots=_ptr(out2_slots), pair_rows=0 if pairs is None else pairs.shape[0],
        out2_rows=0 if out2_slots is None else out2.numel() // out2.shape[-1] // (out2.shape[0] if out2_tiled else 1), n=n, width=width,
        pair_top=0 if pair_slots is None else pair_slots.shape[1], out2_top=0 if out2_slots is None else out2_slots.shape[1],
        out2_tiled=int(out2_tiled), dtype=_lib.dtype_code(outs[0] if outs else torch.float32),
        delta_dtype=0 if delta is None else _lib.dtype_code(delta.dtype), embed_scale=embed_scale, pair_scale=pair_scale, eps=eps,
        status=_ptr(status))
    _call("spk_rms_residual", a, some.device)


def gelu_tanh(z: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out = gelu(z)``, the tanh form; ``out`` may be a column range of a row-major matrix."""
    _lib.require_cuda(z, "gelu_tanh input")
    if not z.is_contiguous() or out.shape != z.shape or out.dtype != z.dtype or out.stride(1) != 1:
        raise ValueError("z must be contiguous, out of the same shape and dtype with unit column stride")
    lib = _lib.load()
    with torch.cuda.device(z.device):
        rc = lib.spk_gelu_tanh(z.data_ptr(), out.data_ptr(), out.stride(0), z.shape[0], z.shape[1], _lib.dtype_code(z.dtype),
                               _lib.current_stream(z.device))
    _lib.check(rc, "spk_gelu_tanh")
    return out
