"""Gotunex: a pre-norm decoder whose mixer and feed-forward read one residual stream side by side, for the paged engine (CUDA).

``x <- x + mixer(norm1(x)) + ff(norm2(x))``.  A layer's mixer is one of

* latent attention: what is cached per token is a normalised latent and one rotated key part shared by all heads (paged); a layer may
  read an earlier layer's cache; softmax with a learned sink per head, sigmoid output gate;
* channel delta: gated delta rule with one decay per head and key channel behind short causal convolutions; a 32-bit state matrix
  per head and the convolutions' last inputs live in the batch row's slot.

Its feed-forward is dense (gelu) or a mixture of experts that a table names by token id.  No routing depends on activations, so one launch
at the head of a step sorts the step's tokens for every layer, and the launch that ends a layer writes the next layer's
feed-forward input straight to the rows its experts read.

How a layer runs: one GEMM for all projections that read norm1; the mixer's kernels; the feed-forward's; one GEMM whose 32-bit sums feed
the residual (mixer and dense feed-forward share it, as column ranges of one matrix); one launch that adds everything up and
takes both norms for the next layer.  The residual stream, norms, angles, scores, key weights, decays and states are 32-bit."""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _lib
from .attention import AttentionMetadata
from .engine.kv_state_cache import LatentSpec, LayerCacheSpec, PagedKVStateCache
from .kernels.delta import delta_rule
from .kernels.dense import gelu_tanh, rms_residual
from .kernels.experts import ExpertRouter, ExpertWeights, experts_forward
from .kernels.latent import latent_attention, latent_prefill, latent_prepare, latent_query, spelled_out_weights
from .rotary import RotaryConfig


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotaryConfig
    kv_from: int | None

    @classmethod
    def from_dict(cls, m: dict) -> "LatentAttentionConfig":
        rot = RotaryConfig.from_dict(m["rot"])
        if rot is None or rot.dims != m["rot_dim"]:
            raise ValueError("the rotation covers the rotated key part")
        return cls(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"],
                   scale=float(m["scale"]), rot=rot, kv_from=m.get("kv_from"))


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @classmethod
    def from_dict(cls, m: dict) -> "ChannelDeltaConfig":
        if m["heads"] % m["kv_heads"]:
            raise ValueError("heads must be a multiple of the query/key heads")
        return cls(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], taps=m["conv"])


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class GotunexLayerConfig:
    mixer: LatentAttentionConfig | ChannelDeltaConfig
    mlp: DenseConfig | ExpertsConfig | None

    @classmethod
    def from_dict(cls, d: dict) -> "GotunexLayerConfig":
        kinds = {"latent_attention": LatentAttentionConfig, "channel_delta": ChannelDeltaConfig}
        if d["type"] not in kinds:
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mixer, m = kinds[d["type"]].from_dict(d["mixer"]), d.get("mlp")
        if m is None:
            mlp = None
        elif m["kind"] == "dense":
            mlp = DenseConfig(ff=m["ff"])
        elif m["kind"] == "moe":
            mlp = ExpertsConfig(experts=m["router"]["experts"], top=m["router"]["top"], ff=m["expert"]["ff"])
        else:
            raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
        return cls(mixer=mixer, mlp=mlp)


@dataclass(frozen=True)
class GotunexConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: tuple[GotunexLayerConfig, ...]

    @classmethod
    def from_dict(cls, d: dict) -> "GotunexConfig":
        layers = tuple(GotunexLayerConfig.from_dict(x) for x in d["layers"])
        for i, layer in enumerate(layers):
            j = getattr(layer.mixer, "kv_from", None)
            if j is None:
                continue
            src = layers[j].mixer if 0 <= j < i else None
            if not isinstance(src, LatentAttentionConfig) or src.kv_from is not None:
                raise ValueError(f"layer {i} reads the cache of layer {j}, which has none of its own")
            if (src.kv_rank, src.rot_dim, src.rot) != (layer.mixer.kv_rank, layer.mixer.rot_dim, layer.mixer.rot):
                raise ValueError(f"layer {i} and layer {j} differ in the shape of the cache they share")
        return cls(vocab=d["vocab"], width=d["width"], eps=float(d["norm"]["eps"]), embed_scale=float(d["embedding"]["scale"]), layers=layers)


def _stack(parts: dict[str, torch.Tensor]) -> tuple[torch.Tensor, dict[str, slice]]:
    """Matrices over one input as one matrix; every part starts at a multiple of eight rows (zero rows in between), so that the parts'
    column ranges of the product start on 16-byte boundaries."""
    rows, ranges, at = [], {}, 0
    for name, w in parts.items():
        ranges[name] = slice(at, at + w.shape[0])
        pad = -w.shape[0] % 8
        rows += [w, w.new_zeros((pad, w.shape[1]))] if pad else [w]
        at += w.shape[0] + pad
    return torch.cat(rows).contiguous(), ranges


def _expect(name: str, w: torch.Tensor, *shape: int) -> torch.Tensor:
    if tuple(w.shape) != shape:
        raise ValueError(f"{name} is {tuple(w.shape)}, the configuration says {shape}")
    return w


class _LatentAttention:
    def __init__(self, cfg: LatentAttentionConfig, width: int, get, f32) -> None:
        self.cfg = c = cfg
        parts = {"dq": _expect("dq", get("mix.dq"), c.q_rank, width)}
        self.kv_norm = None
        if c.kv_from is None:
            parts["dkv"] = _expect("dkv", get("mix.dkv"), c.kv_rank + c.rot_dim, width)
            self.kv_norm = _expect("dkv.norm", f32("mix.dkv.norm"), c.kv_rank)
        parts["g"] = _expect("g", get("mix.g"), c.heads * c.vdim, width)
        self.w_in, self.at = _stack(parts)
        self.q_norm = _expect("dq.norm", f32("mix.dq.norm"), c.q_rank)
        self.w_uq = _expect("uq", get("mix.uq"), c.heads * (c.dim + c.rot_dim), c.q_rank)
        self.w_uk = _expect("uk", get("mix.uk"), c.heads * c.dim, c.kv_rank)
        self.w_uv = _expect("uv", get("mix.uv"), c.heads * c.vdim, c.kv_rank)
        self.w_kv = spelled_out_weights(self.w_uk, self.w_uv, c.heads) if self.w_uk.dtype == torch.bfloat16 else None
        self.sink = _expect("sink", f32("mix.sink"), c.heads)
        self.out_width = c.heads * c.vdim
        self.w_o = _expect("o", get("mix.o"), width, self.out_width)

    def cache_spec(self) -> LayerCacheSpec:
        c = self.cfg
        return LayerCacheSpec(latent=LatentSpec(c.kv_rank, c.rot_dim) if c.kv_from is None else None, latent_from=c.kv_from)

    def forward(self, model: "GotunexModel", h, out, positions, cache, meta: AttentionMetadata) -> None:
        c = self.cfg
        z = model._matmul(h, self.w_in)
        rot, pool = model._rot[c.rot], cache.latent
        own = {} if c.kv_from is not None else dict(kv=z[:, self.at["dkv"]], w_kv=self.kv_norm, pool=pool, rot_table=rot, positions=positions,
                                                    slot_mapping=meta.slot_mapping)
        cq = latent_prepare(z[:, self.at["dq"]], self.q_norm, eps=model.config.eps, status=meta.status, **own)
        q, gate = model._matmul(cq, self.w_uq), z[:, self.at["g"]]
        common = dict(vdim=c.vdim, scale=c.scale, status=meta.status)
        if meta.num_prefills:
            latent_prefill(q, pool, meta.row_tables, self.w_uk, self.w_uv, self.w_kv, self.sink, gate, out, rot_table=rot, positions=positions,
                           token_rows=meta.token_rows, plan=meta.prefill_plan(), heads=c.heads, dim=c.dim, **common)
            return
        ql = latent_query(q, self.w_uk, pool, rot, positions, heads=c.heads, dim=c.dim, status=meta.status)
        latent_attention(ql, pool, meta.block_tables, self.sink, self.w_uv, gate, out, seq_lens=meta.seq_lens, active=meta.row_active,
                         overlap_previous=meta.tables_settled, **common)


class _ChannelDelta:
    def __init__(self, cfg: ChannelDeltaConfig, width: int, get, f32) -> None:
        self.cfg = c = cfg
        qk, v = c.kv_heads * c.dim, c.heads * c.vdim
        a1, g1 = get("mix.a1"), get("mix.g1")
        self.w_in, self.at = _stack({"q": _expect("q", get("mix.q"), qk, width), "k": _expect("k", get("mix.k"), qk, width),
                                     "v": _expect("v", get("mix.v"), v, width), "b": _expect("b", get("mix.b"), c.heads, width), "a1": a1, "g1": g1})
        # both second steps as one product: block-diagonal over the adjacent ranges of the first steps
        self.low = slice(self.at["a1"].start, self.w_in.shape[0])
        a2 = _expect("a2", get("mix.a2"), c.heads * c.dim, a1.shape[0])
        g2 = _expect("g2", get("mix.g2"), v, g1.shape[0])
        self.gate_at = a2.shape[0] + (-a2.shape[0] % 8)
        self.w_low = a2.new_zeros((self.gate_at + v, self.w_in.shape[0] - self.low.start))
        self.w_low[: a2.shape[0], : a1.shape[0]] = a2
        first = self.at["g1"].start - self.low.start
        self.w_low[self.gate_at:, first: first + g1.shape[0]] = g2
        self.conv = [_expect(f"{n}.conv", f32(f"mix.{n}.conv"), rows, c.taps) for n, rows in (("q", qk), ("k", qk), ("v", v))]
        self.a_log, self.dt_bias = _expect("A_log", f32("mix.A_log"), c.heads), _expect("dt_bias", f32("mix.dt_bias"), c.heads * c.dim)
        self.norm = _expect("norm", f32("mix.norm"), c.vdim)
        self.out_width = v
        self.w_o = _expect("o", get("mix.o"), width, v)

    def cache_spec(self) -> LayerCacheSpec:
        c = self.cfg
        return LayerCacheSpec(states=(("delta", (c.heads, c.dim, c.vdim)), ("conv", (c.taps, 2 * c.kv_heads * c.dim + c.heads * c.vdim))))

    def forward(self, model: "GotunexModel", h, out, positions, cache, meta: AttentionMetadata) -> None:
        c = self.cfg
        z = model._matmul(h, self.w_in)
        low = model._matmul(z[:, self.low], self.w_low)
        where = dict(plan=meta.prefill_plan()) if meta.num_prefills else dict(positions=positions, active=meta.row_active)
        delta_rule(z[:, self.at["q"]], z[:, self.at["k"]], z[:, self.at["v"]], z[:, self.at["b"]], low[:, : c.heads * c.dim], low[:, self.gate_at:],
                   conv=self.conv, a_log=self.a_log, dt_bias=self.dt_bias, norm=self.norm, state=cache.states["delta"],
                   conv_state=cache.states["conv"], out=out, kv_heads=c.kv_heads, eps=model.config.eps, status=meta.status, **where)


class _Layer:
    """One layer's weights on the device: GEMM operands in the model dtype, everything else fp32."""

    def __init__(self, cfg: GotunexLayerConfig, width: int, vocab: int, get, f32, ints) -> None:
        self.cfg = cfg
        self.norm1 = _expect("norm1", f32("norm1"), width)
        mixer = _LatentAttention if isinstance(cfg.mixer, LatentAttentionConfig) else _ChannelDelta
        self.mixer = mixer(cfg.mixer, width, get, f32)
        self.norm2 = None if cfg.mlp is None else _expect("norm2", f32("norm2"), width)
        self.up = self.experts = self.route_index = None
        self.w_out = self.mixer.w_o
        if isinstance(cfg.mlp, DenseConfig):
            self.up = _expect("up", get("mlp.up"), cfg.mlp.ff, width)
            self.w_out = torch.cat([self.mixer.w_o, _expect("down", get("mlp.down"), width, cfg.mlp.ff)], dim=1).contiguous()
        elif cfg.mlp is not None:
            m = cfg.mlp
            part = lambda name, *shape: [_expect(name, get(f"mlp.e{e}.{name}"), *shape) for e in range(m.experts)]
            self.experts = ExpertWeights(part("gate", m.ff, width), part("up", m.ff, width), part("down", width, m.ff),
                                         _expect("table", ints("mlp.table"), vocab, m.top))


class GotunexModel:
    """Inference-only model over a weights dict; every tensor lives on ``device``.  ``dtype`` fp32 computes everything in
    32 bits, bf16 takes 16-bit GEMM and attention operands."""

    def __init__(self, config: GotunexConfig, weights: dict, device: str | torch.device = "cuda", dtype: torch.dtype | None = None) -> None:
        self.config = config
        self.device = torch.device(device)
        _lib.require_cuda(torch.empty(0, device=self.device), "GotunexModel device")
        self.dtype = dtype or weights["embed"].dtype
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"{self.dtype} is not supported: fp32 or bf16")
        # sums stay 32-bit: no TF32 products for fp32, no bf16 partial sums in split reductions for bf16
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        get = lambda k: weights[k].to(device=self.device, dtype=self.dtype).contiguous()
        f32 = lambda k: weights[k].to(device=self.device, dtype=torch.float32).contiguous()
        ints = lambda k: weights[k].to(device=self.device)
        c = config
        self.embed, self.head = _expect("embed", get("embed"), c.vocab, c.width), _expect("head", get("head"), c.vocab, c.width)
        self.final_norm = _expect("final.norm", f32("final.norm"), c.width)
        self.layers = [_Layer(layer, c.width, c.vocab, *(lambda k, f=f, i=i: f(f"l{i}.{k}") for f in (get, f32, ints)))
                       for i, layer in enumerate(c.layers)]
        routed = [layer for layer in self.layers if layer.experts is not None]
        for i, layer in enumerate(routed):
            layer.route_index = i
        self.router = ExpertRouter([layer.experts for layer in routed], c.vocab) if routed else None
        self._rot: dict[RotaryConfig, torch.Tensor] = {}
        # the feed-forward reads the same x as the mixer: steps of up to this many tokens run it on a stream of its own beside it
        self.side_tokens = 1024
        self._side = torch.cuda.Stream(device=self.device)

    def prepare(self, max_positions: int) -> None:
        """Engine hook: positions ``0 .. max_positions - 1`` may be fed (tabulates the rotary factors)."""
        for layer in self.config.layers:
            rot = getattr(layer.mixer, "rot", None)
            if rot is not None and (rot not in self._rot or self._rot[rot].shape[0] < max_positions):
                self._rot[rot] = rot.table(max_positions, self.device)

    def new_cache(self, num_blocks: int, block_size: int, max_rows: int) -> PagedKVStateCache:
        """Engine hook: pages of latents and rotated keys, and per row the delta states and the convolutions' last inputs."""
        return PagedKVStateCache([layer.mixer.cache_spec() for layer in self.layers], num_blocks, block_size, max_rows, self.dtype, self.device)

    def _matmul(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """``x w^T`` in the model dtype."""
        return F.linear(x, w)

    def _matmul_f32(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """``x w^T`` with the 32-bit sums as they are."""
        if x.dtype == torch.float32:
            return F.linear(x, w)
        return torch.mm(x, w.t(), out_dtype=torch.float32)

    @torch.no_grad()
    def forward_paged(self, input_ids: torch.Tensor, positions: torch.Tensor, caches, meta: AttentionMetadata,
                      residuals: list | None = None) -> torch.Tensor:
        """One step over ``[n]`` tokens: all decode rows, or all prefill portions.  Returns what the output projection reads,
        ``[n, width]``; ``residuals`` (optional) receives a copy of the residual stream after every layer."""
        if meta.num_prefills and meta.num_decode_tokens:
            raise ValueError("a step holds decode rows or prefill portions, not both")
        c = self.config
        n = input_ids.shape[0]
        x = torch.empty((n, c.width), dtype=torch.float32, device=self.device)
        h = torch.empty((n, c.width), dtype=self.dtype, device=self.device)
        routes = self.router(input_ids, meta.row_active, meta.status) if self.router is not None else []
        common = dict(eps=c.eps, x_out=x, out1=h, status=meta.status)

        def reads(i: int) -> dict:
            """What the boundary before layer i hands on: both norms, or the model's output norm."""
            if i == len(self.layers):
                return dict(w1=self.final_norm)
            L = self.layers[i]
            out = dict(w1=L.norm1, w2=L.norm2)
            if L.experts is not None:
                out.update(out2=L.experts.sorted_matrix(n, c.width), out2_slots=routes[L.route_index].slots, out2_tiled=L.experts.tiled)
            elif L.up is not None:
                out["out2"] = torch.empty_like(h)
            return out

        hand = reads(0)
        rms_residual(ids=input_ids, embed=self.embed, embed_scale=c.embed_scale, **hand, **common)
        for i, L in enumerate(self.layers):
            mixed = L.mixer.out_width
            both = torch.empty((n, L.w_out.shape[1]), dtype=self.dtype, device=self.device)
            added = {}
            main, beside = torch.cuda.current_stream(self.device), n <= self.side_tokens and L.norm2 is not None
            if beside:
                self._side.wait_stream(main)
            with torch.cuda.stream(self._side if beside else main):
                if L.up is not None:
                    gelu_tanh(self._matmul(hand["out2"], L.up), both[:, mixed:])
                elif L.experts is not None:
                    route = routes[L.route_index]
                    added = dict(pairs=experts_forward(hand["out2"], L.experts, route, meta.status), pair_slots=route.slots, pair_scale=1.0 / L.experts.top)
            L.mixer.forward(self, h, both[:, :mixed], positions, caches[i], meta)
            if beside and L.up is not None:
                main.wait_stream(self._side)
            delta = self._matmul_f32(both, L.w_out)
            if beside and L.experts is not None:
                main.wait_stream(self._side)
            hand = reads(i + 1)
            rms_residual(x=x, delta=delta, **added, **hand, **common)
            if residuals is not None:
                residuals.append(x.clone())
        return h

    @torch.no_grad()
    def compute_logits(self, hidden: torch.Tensor, indices: torch.Tensor | None = None) -> torch.Tensor:
        """fp32 logits of the rows that are sampled."""
        if indices is not None:
            hidden = hidden.index_select(0, indices)
        return self._matmul_f32(hidden, self.head)
