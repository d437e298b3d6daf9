"""Plain, slow CPU restatement of the Gotunex decoder (TEST INFRASTRUCTURE ONLY).

One function per mechanism, written straight from the equations: no cache, no chunks, no batching, the recurrence one token at a
time, attention one query at a time with keys and values spelled out per head, experts one token at a time.  Shares no code with the
product path.  Everything runs in the dtype of the weights it is handed (float64 by default, which makes the oracle's own rounding
negligible).

Weights are a ``dict[str, Tensor]`` under the checkpoint's tensor names; the configuration is the parsed ``config.json`` dictionary.
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def rotate(x: torch.Tensor, position: int, rot: dict) -> torch.Tensor:
    """``x [..., >= dims]`` at one position: channel i turns with channel i + dims/2, the rest stays."""
    out = x.clone()
    half = rot["dims"] // 2
    for i in range(half):
        a = position * rot["base"] ** (-2.0 * i / rot["dims"])
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * math.cos(a) - v * math.sin(a)
        out[..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def causal_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """``x [n, channels]``, ``taps [channels, T]``: the last tap is the current token's, zeros before the first token."""
    T = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(T):
            s = t - (T - 1 - j)
            if s >= 0:
                out[t] = out[t] + x[s] * taps[:, j]
    return out


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, log_decay):
    """One head: ``q, k, log_decay [n, dim]``, ``v [n, vdim]``, ``beta [n]`` -> ``o [n, vdim]`` (and the final state)."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = torch.exp(log_decay[t])[:, None] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.t() @ q[t]
    return out, S


def channel_delta(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    act = lambda name: silu(causal_conv(h @ w[p + name].t(), w[p + name + ".conv"]))
    q = unit(act("q").view(n, G, D)) * D ** -0.5
    k = unit(act("k").view(n, G, D))
    v = act("v").view(n, H, V)
    beta = torch.sigmoid(h @ w[p + "b"].t())
    raw = (h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "dt_bias"]
    log_decay = -torch.exp(w[p + "A_log"])[None, :, None] * softplus(raw).view(n, H, D)
    gate = torch.sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t()).view(n, H, V)
    out = torch.zeros(n, H, V, dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        o, _ = delta_rule(q[:, g], k[:, g], v[:, i], beta[:, i], log_decay[:, i])
        out[:, i] = rms(o, eps) * w[p + "norm"] * gate[:, i]
    return out.reshape(n, H * V) @ w[p + "o"].t()


def latent_and_key(h: torch.Tensor, w, p: str, m: dict, eps: float):
    """What a layer caches: the normalised latent ``[n, kv_rank]`` and the rotated shared key part ``[n, rot_dim]``."""
    both = h @ w[p + "dkv"].t()
    c = rms(both[:, : m["kv_rank"]], eps) * w[p + "dkv.norm"]
    kr = torch.stack([rotate(both[t, m["kv_rank"]:], t, m["rot"]) for t in range(h.shape[0])])
    return c, kr


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Weights of the keys: the denominator also counts exp(sink)."""
    top = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(sink - top))


def latent_attention(h: torch.Tensor, w, p: str, m: dict, eps: float, cached) -> torch.Tensor:
    n, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = cached
    q = (rms(h @ w[p + "dq"].t(), eps) * w[p + "dq.norm"]) @ w[p + "uq"].t()
    q = q.view(n, H, D + R)
    keys = (c @ w[p + "uk"].t()).view(n, H, D)
    values = (c @ w[p + "uv"].t()).view(n, H, V)
    out = torch.zeros(n, H, V, dtype=h.dtype)
    for t in range(n):
        qr = rotate(q[t, :, D:], t, m["rot"])
        for i in range(H):
            scores = (keys[: t + 1, i] @ q[t, i, :D] + kr[: t + 1] @ qr[i]) * m["scale"]
            out[t, i] = sink_softmax(scores, w[p + "sink"][i]) @ values[: t + 1, i]
    gate = torch.sigmoid(h @ w[p + "g"].t())
    return (out.reshape(n, H * V) * gate) @ w[p + "o"].t()


def dense_feed_forward(h: torch.Tensor, w, p: str) -> torch.Tensor:
    return gelu_tanh(h @ w[p + "up"].t()) @ w[p + "down"].t()


def table_experts(h: torch.Tensor, tokens, w, p: str, m: dict) -> torch.Tensor:
    """The token's id names its experts; equal weights."""
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        chosen = w[p + "table"][tok].tolist()
        for e in chosen:
            q = f"{p}e{e}."
            out[t] += ((silu(h[t] @ w[q + "gate"].t()) * (h[t] @ w[q + "up"].t())) @ w[q + "down"].t()) / m["router"]["top"]
    return out


def embed(tokens, w, cfg: dict) -> torch.Tensor:
    return w["embed"][torch.tensor(list(tokens))] * cfg["embedding"]["scale"]


def forward(tokens, w, cfg: dict, layers: list | None = None) -> torch.Tensor:
    """Logits ``[n, vocab]`` of a whole sequence; ``layers`` receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w, cfg)
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h1 = rms(x, eps) * w[p + "norm1"]
        if layer["type"] == "channel_delta":
            y = channel_delta(h1, w, p + "mix.", m, eps)
        else:
            src = m.get("kv_from")
            if src is None:
                cached[i] = latent_and_key(h1, w, p + "mix.", m, eps)
            y = latent_attention(h1, w, p + "mix.", m, eps, cached[i if src is None else src])
        if mlp is not None:
            h2 = rms(x, eps) * w[p + "norm2"]
            y = y + (dense_feed_forward(h2, w, p + "mlp.") if mlp["kind"] == "dense" else table_experts(h2, tokens, w, p + "mlp.", mlp))
        x = x + y
        if layers is not None:
            layers.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].t()


def greedy(prompt, steps: int, w, cfg: dict):
    """Greedy continuation, and at every step the margin of the best logit over the second best."""
    tokens, out, margins = list(prompt), [], []
    for _ in range(steps):
        top = torch.topk(forward(tokens, w, cfg)[-1], 2)
        out.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
        tokens.append(out[-1])
    return out, margins


def as_float(weights, dtype: torch.dtype = torch.float64) -> dict:
    return {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}


def random_weights(cfg: dict, seed: int, low_rank: int = 12, dtype: torch.dtype = torch.bfloat16) -> dict:
    """Seeded weights of a configuration, of a size at which every mechanism shows in the logits.  ``low_rank``: rank of the decay's and
    the gate's two-step projections (not part of the configuration)."""
    g = torch.Generator().manual_seed(seed)
    mat = lambda o, i, s=1.0: (torch.randn(o, i, generator=g) * s / math.sqrt(i)).to(dtype)
    vec = lambda n, lo=0.6, hi=1.4: (lo + (hi - lo) * torch.rand(n, generator=g)).to(dtype)
    width, vocab = cfg["width"], cfg["vocab"]
    w = {"embed": (torch.randn(vocab, width, generator=g) / cfg["embedding"]["scale"]).to(dtype), "final.norm": vec(width), "head": mat(vocab, width)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        a = p + "mix."
        w[p + "norm1"] = vec(width)
        if layer["type"] == "channel_delta":
            H, G, D, V, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                w[a + name] = mat(rows, width)
                w[a + name + ".conv"] = (torch.randn(rows, T, generator=g) * 0.6).to(dtype)
            w[a + "b"] = mat(H, width)
            w[a + "A_log"] = vec(H, -2.5, 1.0)
            w[a + "dt_bias"] = vec(H * D, -5.0, 0.5)
            w[a + "a1"], w[a + "a2"] = mat(low_rank, width), mat(H * D, low_rank)
            w[a + "g1"], w[a + "g2"] = mat(low_rank + 3, width), mat(H * V, low_rank + 3)
            w[a + "norm"] = vec(V)
            w[a + "o"] = mat(width, H * V)
        else:
            H, D, R, V, K, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w[a + "dq"], w[a + "dq.norm"] = mat(Q, width), vec(Q)
            w[a + "uq"] = mat(H * (D + R), Q, 1.5)
            if m.get("kv_from") is None:
                w[a + "dkv"], w[a + "dkv.norm"] = mat(K + R, width), vec(K)
            w[a + "uk"], w[a + "uv"] = mat(H * D, K, 1.5), mat(H * V, K)
            w[a + "sink"] = vec(H, -1.0, 3.0)
            w[a + "g"], w[a + "o"] = mat(H * V, width), mat(width, H * V)
        if mlp is None:
            continue
        w[p + "norm2"] = vec(width)
        b = p + "mlp."
        if mlp["kind"] == "dense":
            w[b + "up"], w[b + "down"] = mat(mlp["ff"], width), mat(width, mlp["ff"])
        else:
            E, top, ff = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            for e in range(E):
                w[f"{b}e{e}.gate"], w[f"{b}e{e}.up"], w[f"{b}e{e}.down"] = mat(ff, width), mat(ff, width), mat(width, ff)
            w[b + "table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).to(torch.int32)
    return w
