"""Manirax: a decoder with post-norm residuals, token shift and a two-branch mixer, for the paged engine (CUDA).

Every layer reads its input mixed with the previous token's (token shift), runs two mixers side by side on it and adds
``left_scale * left + right_scale * right`` to ``alpha`` times the residual before the layer norm; an optional dense
feed-forward with a polynomial norm activation follows in the same way.

* left: grouped-query attention whose key weights are sigmoids (no softmax), q and k rotated and brought to unit RMS,
  over the paged K/V pools;
* right: linear attention with a per-head decay, its state one 32-bit matrix per head and batch row.

How a layer runs: one GEMM for all seven input projections; one launch that rotates, normalises and writes K/V pages; the
attention; the recurrence; one launch for the right branch's gated norm.  Both branches write column ranges of ONE matrix,
already multiplied by their scale, so a single GEMM over the concatenated output weights yields the mixer's sum.  Every
residual add + layer norm + (token shift | final norm) is one launch.  The residual stream, all norms, angles, key
weights and states are 32-bit; GEMMs stay cuBLAS through torch, with 32-bit accumulation and 32-bit outputs where they feed
the residual or are logits.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _lib
from .attention import AttentionMetadata
from .engine.kv_state_cache import KVSpec, LayerCacheSpec, PagedKVStateCache
from .kernels.dense import (decay_attention, decay_powers, gated_norm, poly_norm, qk_prepare, residual_norm,
                            sigmoid_attention)
from .rotary import RotaryConfig


@dataclass(frozen=True)
class SigmoidAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotaryConfig | None


@dataclass(frozen=True)
class DecayAttentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]


@dataclass(frozen=True)
class ManiraxLayerConfig:
    left: SigmoidAttentionConfig
    right: DecayAttentionConfig
    left_scale: float
    right_scale: float
    ff: int | None

    @classmethod
    def from_dict(cls, d: dict) -> "ManiraxLayerConfig":
        if d["type"] != "parallel":
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mlp = d.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        m = d["mixer"]
        lf, rt = m["left"], m["right"]
        left = SigmoidAttentionConfig(heads=lf["heads"], kv_heads=lf["kv_heads"], dim=lf["dim"], vdim=lf["vdim"],
                                      scale=float(lf["scale"]), rot=RotaryConfig.from_dict(lf.get("rot")))
        right = DecayAttentionConfig(heads=rt["heads"], dim=rt["dim"], vdim=rt["vdim"], decay=tuple(float(x) for x in rt["decay"]))
        if left.heads % left.kv_heads:
            raise ValueError("query heads must be a multiple of the key/value heads")
        if len(right.decay) != right.heads:
            raise ValueError("one decay per recurrent head")
        return cls(left=left, right=right, left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"]),
                   ff=mlp["ff"] if mlp else None)


@dataclass(frozen=True)
class ManiraxConfig:
    vocab: int
    width: int
    eps: float
    alpha: float
    layers: tuple[ManiraxLayerConfig, ...]

    @classmethod
    def from_dict(cls, d: dict) -> "ManiraxConfig":
        return cls(vocab=d["vocab"], width=d["width"], eps=float(d["norm"]["eps"]), alpha=float(d["postln_alpha"]),
                   layers=tuple(ManiraxLayerConfig.from_dict(x) for x in d["layers"]))


class _Layer:
    """One layer's weights on the device: GEMM operands in the model dtype, everything else fp32."""

    def __init__(self, cfg: ManiraxLayerConfig, get, f32, device) -> None:
        self.cfg = cfg
        lf, rt = cfg.left, cfg.right
        parts = [get(f"mix.left.{n}") for n in "qkv"] + [get(f"mix.right.{n}") for n in "qkvg"]
        self.widths = [lf.heads * lf.dim, lf.kv_heads * lf.dim, lf.kv_heads * lf.vdim,
                       rt.heads * rt.dim, rt.heads * rt.dim, rt.heads * rt.vdim, rt.heads * rt.vdim]
        if [p.shape[0] for p in parts] != self.widths:
            raise ValueError(f"projection rows {[p.shape[0] for p in parts]} do not fit the configured sizes {self.widths}")
        self.w_in = torch.cat(parts).contiguous()
        self.left_width, self.right_width = lf.heads * lf.vdim, rt.heads * rt.vdim
        self.w_out = torch.cat([get("mix.left.o"), get("mix.right.o")], dim=1).contiguous()
        self.head_bias = f32("mix.left.pb")
        self.right_norm = f32("mix.right.norm")
        self.decay = decay_powers(rt.decay, device)
        self.shift, self.norm1 = f32("shift"), f32("norm1")
        if cfg.ff is not None:
            self.up, self.down = get("mlp.up"), get("mlp.down")
            self.act, self.norm2 = f32("mlp.act"), f32("norm2")


class ManiraxModel:
    """Inference-only model over a weights dict; every tensor lives on ``device``.  ``dtype`` fp32 computes everything in
    32 bits, bf16 takes 16-bit GEMM and attention operands."""

    def __init__(self, config: ManiraxConfig, weights: dict, device: str | torch.device = "cuda",
                 dtype: torch.dtype | None = None) -> None:
        self.config = config
        self.device = torch.device(device)
        _lib.require_cuda(torch.empty(0, device=self.device), "ManiraxModel device")
        self.dtype = dtype or weights["embed"].dtype
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"{self.dtype} is not supported: fp32 or bf16")
        # sums stay 32-bit: no TF32 products for fp32, no bf16 partial sums in split reductions for bf16
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        get = lambda k: weights[k].to(device=self.device, dtype=self.dtype).contiguous()
        f32 = lambda k: weights[k].to(device=self.device, dtype=torch.float32).contiguous()
        self.embed = get("embed")
        if tuple(self.embed.shape) != (config.vocab, config.width):
            raise ValueError(f"embedding table {tuple(self.embed.shape)} does not fit the configuration")
        self.final_norm = f32("final.norm")
        self.layers = [_Layer(c, lambda k, i=i: get(f"l{i}.{k}"), lambda k, i=i: f32(f"l{i}.{k}"), self.device)
                       for i, c in enumerate(config.layers)]
        self._rot: dict[RotaryConfig, torch.Tensor] = {}

    def prepare(self, max_positions: int) -> None:
        """Engine hook: positions ``0 .. max_positions - 1`` may be fed (tabulates the rotary factors)."""
        for layer in self.config.layers:
            rot = layer.left.rot
            if rot is not None and (rot not in self._rot or self._rot[rot].shape[0] < max_positions):
                self._rot[rot] = rot.table(max_positions, self.device)

    def new_cache(self, num_blocks: int, block_size: int, max_rows: int) -> PagedKVStateCache:
        """Engine hook: K/V pages of the left mixers, and per row the right mixers' states and the last token's residual."""
        specs = [LayerCacheSpec(kv=KVSpec(c.left.kv_heads, c.left.dim, c.left.vdim),
                                states=(("decay", (c.right.heads, c.right.dim, c.right.vdim)), ("shift", (self.config.width,))))
                 for c in self.config.layers]
        return PagedKVStateCache(specs, num_blocks, block_size, max_rows, self.dtype, self.device)

    def _matmul(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """``x w^T`` in the model dtype."""
        return F.linear(x, w)

    def _matmul_f32(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """``x w^T`` with the 32-bit sums as they are."""
        if x.dtype == torch.float32:
            return F.linear(x, w)
        return torch.mm(x, w.t(), out_dtype=torch.float32)

    def _mixer(self, L: _Layer, h: torch.Tensor, positions: torch.Tensor, cache, meta: AttentionMetadata) -> torch.Tensor:
        lf, rt, eps = L.cfg.left, L.cfg.right, self.config.eps
        n = h.shape[0]
        lq, lk, lv, rq, rk, rv, rg = self._matmul(h, L.w_in).split(L.widths, dim=1)
        both = torch.empty((n, L.left_width + L.right_width), dtype=self.dtype, device=h.device)
        heads = dict(heads=lf.heads, kv_heads=lf.kv_heads, dim=lf.dim, vdim=lf.vdim)
        q = qk_prepare(lq, lk, lv, cache.k, cache.v, meta.slot_mapping, eps=eps, rot_table=None if lf.rot is None else self._rot[lf.rot],
                       positions=positions, status=meta.status, **heads)
        common = dict(scale=lf.scale, out_scale=L.cfg.left_scale, status=meta.status, **heads)
        left = both[:, : L.left_width]
        if meta.num_prefills:
            plan = meta.prefill_plan()
            o = decay_attention(rq, rk, rv, cache.states["decay"], L.decay, plan=plan, status=meta.status)
            sigmoid_attention(q, cache.k, cache.v, meta.row_tables, L.head_bias, left, plan=plan, **common)
            partials = None
        else:
            # three launches in a row: the recurrence is placed while K/V are being written, the attention runs beside it
            o = decay_attention(rq, rk, rv, cache.states["decay"], L.decay, active=meta.row_active,
                                overlap_previous=meta.tables_settled, status=meta.status)
            partials = sigmoid_attention(q, cache.k, cache.v, meta.block_tables, L.head_bias, left, seq_lens=meta.seq_lens,
                                         active=meta.row_active, partial_sums=True, overlap_previous=meta.tables_settled, **common)
        gated_norm(o, L.right_norm, rg, both, L.left_width, eps=eps, scale=L.cfg.right_scale, partials=partials,
                   left_scale=L.cfg.left_scale, seq_lens=meta.seq_lens, active=meta.row_active)
        return self._matmul_f32(both, L.w_out)

    @torch.no_grad()
    def forward_paged(self, input_ids: torch.Tensor, positions: torch.Tensor, caches, meta: AttentionMetadata,
                      residuals: list | None = None) -> torch.Tensor:
        """One step over ``[n]`` tokens: all decode rows, or all prefill portions.  Returns what the output projection reads,
        ``[n, width]``; ``residuals`` (optional) receives a copy of the residual stream after every layer."""
        if meta.num_prefills and meta.num_decode_tokens:
            raise ValueError("a step holds decode rows or prefill portions, not both")
        c = self.config
        n = input_ids.shape[0]
        x, x_next = torch.empty((2, n, c.width), dtype=torch.float32, device=self.device)
        h = torch.empty((n, c.width), dtype=self.dtype, device=self.device)
        place = dict(eps=c.eps, positions=positions, token_rows=meta.token_rows, token_edges=meta.token_edges,
                     active=meta.row_active, status=meta.status)

        def reads(i: int) -> dict:
            """What the boundary before layer i hands on: the shifted stream, or the model's output norm."""
            if i == len(self.layers):
                return dict(second_weight=self.final_norm)
            return dict(mix=self.layers[i].shift, prev=caches[i].states["shift"])

        residual_norm(h, ids=input_ids, embed=self.embed, x_out=x, **reads(0), **place)
        for i, L in enumerate(self.layers):
            delta = self._mixer(L, h, positions, caches[i], meta)
            # the launch that ends the mixer still reads the layer's input: it leaves the last token's for the next portion
            norm1 = dict(x=x, delta=delta, weight=L.norm1, alpha=c.alpha, x_out=x_next, commit=caches[i].states["shift"])
            if L.cfg.ff is None:
                residual_norm(h, **norm1, **reads(i + 1), **place)
            else:
                residual_norm(h, **norm1, **place)
                x, x_next = x_next, x
                z = self._matmul(h, L.up)
                delta = self._matmul_f32(poly_norm(z, L.act, c.eps, out=z), L.down)
                residual_norm(h, x=x, delta=delta, weight=L.norm2, alpha=c.alpha, x_out=x_next, **reads(i + 1), **place)
            x, x_next = x_next, x
            if residuals is not None:
                residuals.append(x.clone())
        return h

    @torch.no_grad()
    def compute_logits(self, hidden: torch.Tensor, indices: torch.Tensor | None = None) -> torch.Tensor:
        """fp32 logits of the rows that are sampled (the output projection is the embedding table)."""
        if indices is not None:
            hidden = hidden.index_select(0, indices)
        return self._matmul_f32(hidden, self.embed)
