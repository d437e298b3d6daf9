"""Gated delta rule with one decay per head and key channel (CUDA), with the short convolutions, unit vectors, decays and the output
norm and gate around it."""
from __future__ import annotations

import torch

from .. import _lib
from .dense import _call, _f32, _ptr, _same_rows


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, b: torch.Tensor, a: torch.Tensor, gate: torch.Tensor, *, conv, a_log: torch.Tensor,
               dt_bias: torch.Tensor, norm: torch.Tensor, state: torch.Tensor, conv_state: torch.Tensor, out: torch.Tensor, kv_heads: int, eps: float,
               positions: torch.Tensor | None = None, active: torch.Tensor | None = None, plan=None, status: torch.Tensor | None = None) -> torch.Tensor:
    """``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q`` per head, ``out = rmsnorm(o) * norm * sigmoid(gate)``.

    ``q``, ``k``, ``v``, ``b`` are column ranges of one projection output, ``a`` (the decays' raw values) and ``gate`` of another; ``conv``
    are the three fp32 ``[channels, taps]`` filters.  ``state`` fp32 ``[rows, heads, dim, vdim]`` and ``conv_state`` fp32 ``[rows, taps,
    channels]`` are updated in place.  ``plan`` (a ``PrefillPlan``): prefill form; None: decode form over ``positions`` / ``active``."""
    _lib.require_cuda(q, "delta_rule query")
    n = q.shape[0]
    rows, heads, dim, vdim = state.shape
    taps = conv[0].shape[1]
    ld, ld2 = _same_rows(q, k, v, b), _same_rows(a, gate)
    if (q.shape[1], k.shape[1], v.shape[1], b.shape[1], a.shape[1], gate.shape[1]) != (kv_heads * dim, kv_heads * dim, heads * vdim, heads,
                                                                                        heads * dim, heads * vdim):
        raise ValueError("projection widths do not fit the state")
    if conv_state.shape != (rows, taps, 2 * kv_heads * dim + heads * vdim):
        raise ValueError("conv_state must be [rows, taps, channels of q, k and v]")
    for t, name, numel in ((state, "state", None), (conv_state, "conv_state", None), (a_log, "a_log", heads), (dt_bias, "dt_bias", heads * dim),
                           (norm, "norm", vdim), (conv[0], "conv of q", q.shape[1] * taps), (conv[1], "conv of k", k.shape[1] * taps),
                           (conv[2], "conv of v", v.shape[1] * taps)):
        _f32(t, name, numel)
    if out.shape != (n, heads * vdim) or out.stride(1) != 1 or out.dtype != q.dtype:
        raise ValueError("out must be [n, heads * vdim] in the dtype of q with unit column stride")
    args = _lib.DeltaArgs(
        q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(), b=b.data_ptr(), a=a.data_ptr(), gate=gate.data_ptr(), ld=ld, ld2=ld2,
        conv_q=conv[0].data_ptr(), conv_k=conv[1].data_ptr(), conv_v=conv[2].data_ptr(), a_log=a_log.data_ptr(), dt_bias=dt_bias.data_ptr(),
        w_norm=norm.data_ptr(), state=state.data_ptr(), conv_state=conv_state.data_ptr(), state_rows=rows, positions=_ptr(positions),
        active=_ptr(active), out=out.data_ptr(), out_stride=out.stride(0), n=n, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, taps=taps,
        dtype=_lib.dtype_code(q.dtype), eps=eps, status=_ptr(status))
    if plan is None:
        _call("spk_delta_step", args, q.device)
        return out
    lib = _lib.load()
    chunks, seqs = plan.chunks(int(lib.spk_delta_chunk_tokens(args.dtype, dim, vdim)))
    portions = plan.portions()
    need = int(lib.spk_delta_workspace_bytes(args.dtype, n, chunks.shape[0], heads, kv_heads, dim, vdim))
    ws = torch.empty(need, dtype=torch.uint8, device=q.device)
    args.seqs = seqs.data_ptr()
    args.chunks, args.portions, args.n_chunks, args.n_portions = chunks.data_ptr(), portions.data_ptr(), chunks.shape[0], portions.shape[0]
    args.workspace, args.workspace_bytes = ws.data_ptr(), need
    _call("spk_delta_prefill", args, q.device)
    return out
