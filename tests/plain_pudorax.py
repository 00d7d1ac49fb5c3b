"""A plain, slow Pudorax: whole sequences, no cache, one function per mechanism.

The yardstick for the engine's Pudorax parts.  It shares no code with the package: config.json
is read with ``json``, the weights with the ``safetensors`` library, and everything is
elementary torch arithmetic on the CPU in float64 (or float32).

Notation: ``x`` [S, D] is the residual stream of one sequence of S tokens at positions
0 .. S-1; a linear map is stored [out, in] and applied as ``x @ W.T``;
``unit(x) = x / sqrt(mean(x**2) + eps)`` and
``centred(x) = (x - mean(x)) / sqrt(mean((x - mean(x))**2) + eps)`` over the last axis.

* input: ``x = x0 = c * embed[id]``;
* block: ``x += mixer(norm1(x))``; where it has one, ``x += ff(norm2(x))``; where the model has
  it, ``x += unit(P (gelu(G x) * e)) * n`` with e the layer's part of a second embedding of the token.
  ``norm(x) = centred(x) * w + b``;
* a span of blocks runs several times in a row, each pass behind ``x = L [x; x0]``;
* mixers: grouped-query attention whose projections pass a short convolution and whose queries
  and keys are normed over the whole projection, with a gate per channel; and the Mamba-2
  recurrence;
* the feed-forward: routed experts with clamped gates, and one that every token uses;
* logits: ``c2 * tanh(head (norm(x)) / c2)``.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List

import torch


def read_model_folder(model_dir: str):
    from safetensors import safe_open
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as f:
        cfg = json.load(f)
    weights = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            weights[name] = f.get_tensor(name).to(torch.float64)
    return cfg, weights


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def centred(x: torch.Tensor, eps: float) -> torch.Tensor:
    """``unit`` of what is left when the mean is taken off."""
    return unit(x - x.mean(dim=-1, keepdim=True), eps)


def layer_norm(x, W, name, eps):
    return centred(x, eps) * W[name] + W[name + ".b"]


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(u, w):
    """u [S, C] over time with taps w [C, K]: the last tap is the present row's, rows before the
    sequence's start are zero."""
    S, K = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(S):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def rotate_pairs(z, base: float, dims: int):
    """z [S, heads, d]: channels 2i and 2i + 1 of the first ``dims`` are turned by
    ``t * base^(-2i/dims)``; the rest pass."""
    S = z.shape[0]
    i = torch.arange(dims // 2, dtype=torch.float64)
    freq = torch.tensor(float(base), dtype=torch.float64) ** (-2.0 * i / dims)
    ang = torch.arange(S, dtype=torch.float64)[:, None] * freq[None, :]
    c, s = torch.cos(ang).to(z.dtype)[:, None, :], torch.sin(ang).to(z.dtype)[:, None, :]
    u, v = z[..., 0:dims:2], z[..., 1:dims:2]
    out = z.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def attention(q, k, v, scale):
    """Causal softmax attention, q [S, H, d], k [S, G, d], v [S, G, e] -> [S, H, e]."""
    S, H, _ = q.shape
    G = k.shape[1]
    seen = torch.ones(S, S, dtype=torch.bool).tril()
    out = torch.zeros(S, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out[:, h] = (e / e.sum(dim=-1, keepdim=True)) @ v[:, g]
    return out


def mixer_attention(h, W, p, m, eps):
    S = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q = (unit(q, eps) * W[p + "q.norm"]).reshape(S, H, d)
    k = (unit(k, eps) * W[p + "k.norm"]).reshape(S, G, d)
    rot = m["rot"]
    o = attention(rotate_pairs(q, rot["base"], rot["dims"]), rotate_pairs(k, rot["base"], rot["dims"]),
                  v.reshape(S, G, e), m["scale"]).reshape(S, H * e)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def state_space(x, B, C, dt, a, D):
    """x [S, H, e], B and C [S, G, N], dt [S, H] step sizes, a [H] decay rates, D [H] -> y [S, H, e].
    Per head a state M [N, e], zero at the start: ``M <- exp(-a dt) M + dt B x^T``,
    ``y = M^T C + D x``."""
    S, H, e = x.shape
    G, N = B.shape[1:]
    y = torch.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        M = torch.zeros(N, e, dtype=x.dtype)
        for t in range(S):
            M = torch.exp(-a[h] * dt[t, h]) * M + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = M.T @ C[t, g] + D[h] * x[t, h]
    return y


def gated_parts_norm(y, z, parts: int, w, eps):
    """``y * silu(z)``, then each of ``parts`` equal parts over its own root mean square, times w."""
    S, n = y.shape
    return unit((y * silu(z)).reshape(S, parts, n // parts), eps).reshape(S, n) * w


def mixer_mamba2(h, W, p, m, eps):
    S = h.shape[0]
    H, e, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, C = H * e, H * e + 2 * G * N
    u = h @ W[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:inner + C], u[:, inner + C:]
    xbc = silu(causal_conv(xbc, W[p + "conv"]) + W[p + "conv.b"])
    y = state_space(xbc[:, :inner].reshape(S, H, e), xbc[:, inner:inner + G * N].reshape(S, G, N),
                    xbc[:, inner + G * N:].reshape(S, G, N), softplus(dt + W[p + "dt_bias"]),
                    torch.exp(W[p + "A_log"]), W[p + "D"]).reshape(S, inner)
    return gated_parts_norm(y, z, m["norm_groups"], W[p + "norm"], eps) @ W[p + "o"].T


def clamped_expert(h, W, p, limit: float):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def choose(z, top: int):
    """z [E] the logits of one token -> (the experts with the largest, the softmax over those)."""
    ids = sorted(range(z.shape[0]), key=lambda j: -float(z[j]))[:top]
    e = torch.exp(z[ids] - z[ids].max())
    return ids, e / e.sum()


def routed(h, W, p, mlp):
    r = mlp["router"]
    z = h @ W[p + "router"].T + W[p + "router.b"]
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j, w in zip(*choose(z[t], r["top"])):
            y[t] += w * clamped_expert(h[t], W, f"{p}e{j}.", mlp["expert"]["limit"])
    if mlp.get("shared"):
        y = y + clamped_expert(h, W, p + "shared.", mlp["shared"]["limit"])
    return y


def token_side(x, ids, W, p, i: int, dim: int, eps):
    e = torch.stack([W["side.embed"][t, i * dim:(i + 1) * dim] for t in ids])
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return unit(y, eps) * W[p + "side.norm"]


MIXERS = {"attention": mixer_attention, "mamba2": mixer_mamba2}


def run_order(cfg):
    """(layer, first of a pass) in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    span = list(range(loop["start"], loop["stop"]))
    return [(i, False) for i in range(loop["start"])] \
        + [(i, i == span[0]) for _ in range(loop["times"]) for i in span] \
        + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], ids: List[int], dtype=torch.float64,
            streams=None) -> torch.Tensor:
    """Logits [S, vocab] of one whole sequence.  ``streams``, a list, receives the residual
    stream after every layer run."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x0 = torch.stack([W["embed"][t] for t in ids]) * cfg["embedding"]["scale"]
    x = x0
    for i, merge in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if merge:
            x = torch.cat([x, x0], dim=1) @ W["loop.in"].T
        x = x + MIXERS[layer["type"]](layer_norm(x, W, p + "norm1", eps), W, p + "mix.",
                                      layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + routed(layer_norm(x, W, p + "norm2", eps), W, p + "mlp.", layer["mlp"])
        if cfg.get("token_side"):
            x = x + token_side(x, ids, W, p, i, cfg["token_side"]["dim"], eps)
        if streams is not None:
            streams.append(x.clone())
    logits = layer_norm(x, W, "final.norm", eps) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def greedy(cfg, weights, prompt: List[int], n: int, dtype=torch.float64) -> List[int]:
    ids, out = list(prompt), []
    for _ in range(n):
        logits = forward(cfg, weights, ids, dtype)[-1]
        best = int(torch.nonzero(logits == logits.max())[0])
        out.append(best)
        ids.append(best)
    return out
