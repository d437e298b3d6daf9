"""Plain, slow CPU restatement of the Manirax decoder (TEST INFRASTRUCTURE ONLY).

One function per mechanism, written straight from the equations: no cache, no chunks, no batching, the recurrence
one token at a time, attention one query at a time.  Shares no code with the product path.  Everything runs in
the dtype of the weights it is handed (float64 by default, which makes the oracle's own rounding negligible).

Weights are a ``dict[str, Tensor]`` under the checkpoint's tensor names; the configuration is the parsed
``config.json`` dictionary.
"""
from __future__ import annotations

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """Mean removed, divided by the deviation, scaled; no bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def token_shift(h: torch.Tensor, mix: torch.Tensor) -> torch.Tensor:
    """Every token moves towards its predecessor (zeros before the first) by ``mix``, per channel."""
    out = torch.empty_like(h)
    before = torch.zeros_like(h[0])
    for t in range(h.shape[0]):
        out[t] = h[t] + (before - h[t]) * mix
        before = h[t]
    return out


def rotary_frequencies(rot: dict) -> list[float]:
    dims = rot["dims"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    return [rot["base"] ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate(x: torch.Tensor, position: int, rot: dict | None) -> torch.Tensor:
    """``x [heads, dim]`` at one position: channel i turns with channel i + dims/2, the rest stays."""
    if not rot:
        return x
    out = x.clone()
    half = rot["dims"] // 2
    for i, f in enumerate(rotary_frequencies(rot)):
        a = torch.tensor(position * f, dtype=torch.float64)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[:, i], x[:, i + half]
        out[:, i] = u * c - v * s
        out[:, i + half] = v * c + u * s
    return out


def sigmoid_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, head_bias: torch.Tensor) -> torch.Tensor:
    """``q [n, H, d]``, ``k [n, G, d]``, ``v [n, G, dv]``: the last query positions line up with the last keys; every
    visible key weighs sigmoid(score + bias of the head), without normalisation."""
    n, H = q.shape[:2]
    total, G = k.shape[:2]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        last = total - n + i
        for h in range(H):
            g = h // (H // G)
            w = torch.sigmoid(k[: last + 1, g] @ q[i, h] * scale + head_bias[h])
            out[i, h] = w @ v[: last + 1, g]
    return out


def decay_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: list[float],
                     state: torch.Tensor | None = None):
    """``q, k [n, H, d]``, ``v [n, H, dv]``: S <- decay S + k v^T, o = S^T q.  Returns ``(o, S)``."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for t in range(n):
        for h in range(H):
            S[h] = decay[h] * S[h] + torch.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def silu(x: torch.Tensor) -> torch.Tensor:
    return x / (1 + torch.exp(-x))


def poly_norm(z: torch.Tensor, act: torch.Tensor, eps: float) -> torch.Tensor:
    """a N(z) + b N(z^2) + c N(z^3) + e with N the division by the root mean square over the last axis."""
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def left_mixer(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(n, H, d)
    k = (h @ w[p + "k"].T).reshape(n, G, d)
    v = (h @ w[p + "v"].T).reshape(n, G, dv)
    q = rms(torch.stack([rotate(q[t], t, m.get("rot")) for t in range(n)]), eps)
    k = rms(torch.stack([rotate(k[t], t, m.get("rot")) for t in range(n)]), eps)
    o = sigmoid_attention(q, k, v, m["scale"], w[p + "pb"])
    return o.reshape(n, H * dv) @ w[p + "o"].T


def right_mixer(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(n, H, d)
    k = silu(h @ w[p + "k"].T).reshape(n, H, d)
    v = silu(h @ w[p + "v"].T).reshape(n, H, dv)
    o, _ = decay_recurrence(q, k, v, m["decay"])
    o = rms(o.reshape(n, H * dv), eps) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def forward(tokens: list[int], w: dict, config: dict, layers_out: list | None = None) -> torch.Tensor:
    """Logits ``[len(tokens), vocab]`` of one sequence; ``layers_out`` receives the residual stream after every layer."""
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.int64)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        h = token_shift(x, w[p + "shift"])
        mixed = (m["left_scale"] * left_mixer(h, w, p + "mix.left.", m["left"], eps)
                 + m["right_scale"] * right_mixer(h, w, p + "mix.right.", m["right"], eps))
        x = layer_norm(alpha * x + mixed, w[p + "norm1"], eps)
        if layer.get("mlp"):
            ff = poly_norm(x @ w[p + "mlp.up"].T, w[p + "mlp.act"], eps) @ w[p + "mlp.down"].T
            x = layer_norm(alpha * x + ff, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(prompt: list[int], steps: int, w: dict, config: dict) -> tuple[list[int], list[float]]:
    """``steps`` greedy tokens and the margin between the two best logits at each of them."""
    seq, margins = list(prompt), []
    for _ in range(steps):
        top = forward(seq, w, config)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        seq.append(int(top.indices[0]))
    return seq[len(prompt):], margins


def random_weights(config: dict, seed: int, dtype: torch.dtype = torch.bfloat16) -> dict:
    """Seeded weights under the checkpoint's names, scaled so that activations stay near one."""
    g = torch.Generator().manual_seed(seed)
    width, vocab = config["width"], config["vocab"]
    lin = lambda o, i, s=1.0: (torch.randn(o, i, generator=g) * s / i ** 0.5).to(dtype)
    near = lambda n, c, s: (c + s * torch.randn(n, generator=g)).to(dtype)
    w = {"embed": torch.randn(vocab, width, generator=g).to(dtype), "final.norm": near(width, 1.0, 0.2)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        L, R = m["left"], m["right"]
        w[p + "norm1"] = near(width, 1.0, 0.2)
        w[p + "shift"] = torch.rand(width, generator=g).to(dtype)
        a = p + "mix.left."
        w[a + "q"], w[a + "k"] = lin(L["heads"] * L["dim"], width), lin(L["kv_heads"] * L["dim"], width)
        w[a + "v"] = lin(L["kv_heads"] * L["vdim"], width)
        w[a + "pb"] = near(L["heads"], -2.0, 1.0)
        w[a + "o"] = lin(width, L["heads"] * L["vdim"])
        a = p + "mix.right."
        for n in ("q", "k"):
            w[a + n] = lin(R["heads"] * R["dim"], width)
        for n in ("v", "g"):
            w[a + n] = lin(R["heads"] * R["vdim"], width)
        w[a + "norm"] = near(R["heads"] * R["vdim"], 1.0, 0.2)
        w[a + "o"] = lin(width, R["heads"] * R["vdim"])
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            w[p + "norm2"] = near(width, 1.0, 0.2)
            w[p + "mlp.up"], w[p + "mlp.down"] = lin(ff, width, 1.5), lin(width, ff)
            w[p + "mlp.act"] = torch.tensor([0.6, 0.4, -0.3, 0.1]).to(dtype)
    return w


def as_float(w: dict, dtype: torch.dtype = torch.float64) -> dict:
    return {k: t.to(dtype) for k, t in w.items()}
